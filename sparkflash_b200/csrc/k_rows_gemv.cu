// Matrix products of one to four rows, bf16 weights streamed once: out = x W^T (+ bias), to bf16 or 32-bit, or act(x Wg^T) * (x Wu^T)
// with gate and up stacked, or act(x W^T), or gelu(x W^T) times the token's row of a table.  Paced by memory: a warp (or two, four, eight of them, each on a share of K) owns two weight rows, whose first
// 16-byte words are requested before the previous kernel has finished - weights do not depend on it; x sits in shared memory.
#include "k_rows.cuh"

namespace sfb {
namespace rgemv {

constexpr int U = 4;          // 256-element steps of K in flight per weight row

struct Args {
  const __nv_bfloat16* w;     // [M, K] ([2 M, K] with act: gate rows, then up rows)
  const __nv_bfloat16* x;     // [n, K]
  const __nv_bfloat16* bias;  // [M] or null
  void* out;                  // [n, M] bf16 (or float)
  int M, K, n, wk, f32, act, single;     // act: of gate and up; single: of one product
  int64_t out_stride;         // elements between the rows of out
  float alpha, limit;         // of the clamped gate; the single activation's numbers
  const __nv_bfloat16* table; // [vocab, table_stride] or null: out = gelu(x W^T) * table[token][col0 + .]
  int64_t table_stride;
  const int* tokens;
  int col0, vocab;
  Status* status;
};

template <int N>
__global__ void __launch_bounds__(256, 2) gemv_kernel(Args a) {
  extern __shared__ __align__(16) uint8_t raw[];
  __shared__ float part[2][8][2][N];
  __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(raw);      // [N][K]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int groups = 8 / a.wk, g = warp / a.wk, pk = warp % a.wk;
  const int outs = a.act ? a.M : (a.M + 1) / 2;                 // pairs of weight rows
  const int stride = gridDim.x * groups, first = blockIdx.x * groups;
  const int rounds = first < outs ? (outs - first + stride - 1) / stride : 0;      // the same for every warp of the block
  const int steps = (a.K + 255) / 256, mine = (steps + a.wk - 1) / a.wk, batches = (mine + U - 1) / U;
  uint4 c0[U], c1[U];
  // batch b of the warp's pair in round t (the stream of batches runs on over the rounds)
  auto fetch = [&](int t, int b) {
    const int o = first + t * stride + g;
    const bool v0 = a.act ? o < a.M : 2 * o < a.M, v1 = a.act ? o < a.M : 2 * o + 1 < a.M;
    const uint4* w0 = reinterpret_cast<const uint4*>(a.w + (size_t)(a.act ? o : 2 * o) * a.K);
    const uint4* w1 = reinterpret_cast<const uint4*>(a.w + (size_t)(a.act ? o + a.M : 2 * o + 1) * a.K);
#pragma unroll
    for (int i = 0; i < U; ++i) {
      const int k = (pk + (b * U + i) * a.wk) * 32 + lane;       // 16-byte word of the row
      const bool in = t < rounds && k * 8 < a.K;
      c0[i] = in && v0 ? ldg_nc(w0 + k) : make_uint4(0u, 0u, 0u, 0u);
      c1[i] = in && v1 ? ldg_nc(w1 + k) : make_uint4(0u, 0u, 0u, 0u);
    }
  };
  fetch(0, 0);
  pdl_launch_dependents();
  pdl_wait();
  const int words = a.K / 8;
  for (int i = tid; i < N * words; i += 256) {
    const int r = i / words;
    reinterpret_cast<uint4*>(xs)[i] = r < a.n ? reinterpret_cast<const uint4*>(a.x)[i] : make_uint4(0u, 0u, 0u, 0u);
  }
  __syncthreads();
  float acc[2][N];
#pragma unroll
  for (int i = 0; i < N; ++i) acc[0][i] = acc[1][i] = 0.f;
  for (int t = 0; t < rounds; ++t) {
    for (int b = 0; b < batches; ++b) {
      uint4 d0[U], d1[U];
#pragma unroll
      for (int i = 0; i < U; ++i) { d0[i] = c0[i]; d1[i] = c1[i]; }
      if (b + 1 < batches) fetch(t, b + 1);
      else fetch(t + 1, 0);
#pragma unroll
      for (int i = 0; i < U; ++i) {
        const int k = (pk + (b * U + i) * a.wk) * 32 + lane;
        if (k * 8 >= a.K) continue;
        const uint32_t p[4] = {d0[i].x, d0[i].y, d0[i].z, d0[i].w}, q[4] = {d1[i].x, d1[i].y, d1[i].z, d1[i].w};
#pragma unroll
        for (int r = 0; r < N; ++r) {
          const uint4 xv = reinterpret_cast<const uint4*>(xs)[r * words + k];
          const uint32_t xw[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float x0 = __uint_as_float(xw[j] << 16), x1 = __uint_as_float(xw[j] & 0xffff0000u);
            acc[0][r] = fmaf(__uint_as_float(p[j] << 16), x0, acc[0][r]);
            acc[0][r] = fmaf(__uint_as_float(p[j] & 0xffff0000u), x1, acc[0][r]);
            acc[1][r] = fmaf(__uint_as_float(q[j] << 16), x0, acc[1][r]);
            acc[1][r] = fmaf(__uint_as_float(q[j] & 0xffff0000u), x1, acc[1][r]);
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < N; ++r) {
      acc[0][r] = warp_sum(acc[0][r]);
      acc[1][r] = warp_sum(acc[1][r]);
    }
    if (a.wk > 1) {
      if (lane == 0) {
#pragma unroll
        for (int r = 0; r < N; ++r) { part[t & 1][warp][0][r] = acc[0][r]; part[t & 1][warp][1][r] = acc[1][r]; }
      }
      __syncthreads();       // the other half of `part` was read before this round's barrier
      if (pk == 0) {
        for (int k = 1; k < a.wk; ++k) {
#pragma unroll
          for (int r = 0; r < N; ++r) { acc[0][r] += part[t & 1][warp + k][0][r]; acc[1][r] += part[t & 1][warp + k][1][r]; }
        }
      }
    }
    if (pk == 0 && lane < a.n) {
      float s0 = acc[0][0], s1 = acc[1][0];
#pragma unroll
      for (int r = 1; r < N; ++r)
        if (lane == r) { s0 = acc[0][r]; s1 = acc[1][r]; }
      const int o = first + t * stride + g;
      const size_t at = (size_t)lane * a.out_stride;
      if (a.act) {
        if (o < a.M)
          ((__nv_bfloat16*)a.out)[at + o] = __float2bfloat16_rn(a.act == rows::ACT_CLAMP ? rows::gate_clamp<float>(s0, s1, a.alpha, a.limit)
                                                                : (a.act == rows::ACT_GELU ? rows::gelu_tanh_f(s0) : s0 * rows::sigmoid_f(s0)) * s1);
      } else {
        const int r0 = 2 * o, r1 = r0 + 1;
        if (a.bias) { if (r0 < a.M) s0 += __bfloat162float(a.bias[r0]); if (r1 < a.M) s1 += __bfloat162float(a.bias[r1]); }
        if (a.single) { s0 = rows::act_single<float>(s0, a.single, a.alpha, a.limit); s1 = rows::act_single<float>(s1, a.single, a.alpha, a.limit); }
        if (a.table) {
          int tok = a.tokens[lane];
          if (tok < 0 || tok >= a.vocab) { status_set(a.status, ST_BOUNDS, 76, tok, a.vocab); tok = 0; }
          const __nv_bfloat16* e = a.table + (size_t)tok * a.table_stride + a.col0;
          s0 = r0 < a.M ? rows::gelu_tanh_f(s0) * __bfloat162float(e[r0]) : 0.f;
          s1 = r1 < a.M ? rows::gelu_tanh_f(s1) * __bfloat162float(e[r1]) : 0.f;
        }
        if (a.f32) {
          if (r0 < a.M) ((float*)a.out)[at + r0] = s0;
          if (r1 < a.M) ((float*)a.out)[at + r1] = s1;
        } else {
          if (r0 < a.M) ((__nv_bfloat16*)a.out)[at + r0] = __float2bfloat16_rn(s0);
          if (r1 < a.M) ((__nv_bfloat16*)a.out)[at + r1] = __float2bfloat16_rn(s1);
        }
      }
    }
#pragma unroll
    for (int r = 0; r < N; ++r) acc[0][r] = acc[1][r] = 0.f;
  }
}

template <int N>
static int launch(const Args& a, int blocks, cudaStream_t st) {
  const size_t smem = (size_t)N * a.K * 2;
  static size_t granted = 40 * 1024;
  if (smem > granted) {
    const cudaError_t e = cudaFuncSetAttribute(gemv_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    granted = smem;
  }
  return (int)sfb_launch(gemv_kernel<N>, dim3(blocks), dim3(256), smem, st, a);
}

}  // namespace rgemv
}  // namespace sfb

using namespace sfb;
using namespace sfb::rgemv;

static int run(Args a, cudaStream_t stream) {
  const int N = a.n <= 1 ? 1 : a.n <= 2 ? 2 : 4;
  if (a.n < 1 || a.n > 4 || a.M < 1 || a.K < 8 || a.K % 8 || (size_t)N * a.K * 2 > 200 * 1024) return (int)cudaErrorInvalidValue;
  const int pairs = a.act ? a.M : (a.M + 1) / 2, steps = (a.K + 255) / 256;
  a.wk = 1;                // enough pairs of rows for every SM, at least a batch of K per warp
  while (a.wk < 8 && (long long)pairs * a.wk / 8 < 296 && steps / (a.wk * 2) >= 2) a.wk *= 2;
  const int needed = (pairs + 8 / a.wk - 1) / (8 / a.wk), blocks = needed < 296 ? needed : 296;
  return N == 1 ? launch<1>(a, blocks, stream) : N == 2 ? launch<2>(a, blocks, stream) : launch<4>(a, blocks, stream);
}

extern "C" {

// n <= 4 rows, K a multiple of 8, n K bounded by shared memory (4 K rows of 200 KB).  act (1 silu, 2 gelu, 3 clamped): w holds 2 M rows; the
// ungated ones (4, 5): M rows.
int sfb_rows_gemv(const void* w, const void* x, const void* bias, void* out, int64_t out_stride, int n, int M, int K, int f32, int act, float alpha, float limit,
                  cudaStream_t stream) {
  Args a{};
  a.w = (const __nv_bfloat16*)w; a.x = (const __nv_bfloat16*)x; a.bias = (const __nv_bfloat16*)bias; a.out = out; a.M = M; a.K = K; a.n = n; a.f32 = f32;
  if (act == rows::ACT_RELU2 || act == rows::ACT_XIELU) a.single = act;
  else a.act = act;
  a.out_stride = out_stride; a.alpha = alpha; a.limit = limit;
  return run(a, stream);
}

// out [n, M] = gelu(x w^T) * table[token][col0 + .]
int sfb_rows_gemv_token(const void* w, const void* x, void* out, const void* table, int64_t table_stride, const int* tokens, int col0, int vocab, int n, int M, int K,
                        void* status, cudaStream_t stream) {
  Args a{};
  a.w = (const __nv_bfloat16*)w; a.x = (const __nv_bfloat16*)x; a.out = out; a.M = M; a.K = K; a.n = n; a.out_stride = M; a.table = (const __nv_bfloat16*)table;
  a.table_stride = table_stride; a.tokens = tokens; a.col0 = col0; a.vocab = vocab; a.status = (Status*)status;
  return run(a, stream);
}

}  // extern "C"
