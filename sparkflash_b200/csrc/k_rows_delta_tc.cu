// The gated delta rule of k_rows_state.cu for long runs of rows, on tcgen05.  With unit vectors q and k of a head,
//
//   S = a_t S_(t-1),   u_t = b_t (v_t - S^T k_t),   S_t = S + k_t u_t^T,   y_t = S_t^T q_t
//
// A run is cut into chunks of 128 rows.  With c_t the running sum of log a inside a chunk, S_0 the state at its start and
// A_ij = b_i exp(c_i - c_j) (k_i . k_j) for j < i, the writes of a chunk solve (I + A) U = X, so that
//
//   U = (I + A)^-1 X,   X_i = b_i (v_i - exp(c_i) S_0^T k_i),
//   S_0 of the next chunk = exp(c_last) S_0 + sum_j exp(c_last - c_j) k_j u_j^T,
//   y_i = sum_{j <= i} exp(c_i - c_j) (q_i . k_j) u_j + exp(c_i) S_0^T q_i
//
//   delta_prep    per (chunk, group of heads): K K^T, the numbers of the rows (RATES), and (I + A)^-1 of every head in 32-bit: diagonal blocks
//                 of 32 by substitution, the others from pairs of blocks
//   delta_chain   per (head, 32 value dims), chunk after chunk: three products (K S_0, inverse X, K^T U), the state in registers; U and S_0
//                 leave for chunk_out as tiles of two terms, [2, chunks, H, 128, P] and [2, chunks, H, N, P]
//   chunk_out     the third line, all chunks at once (k_rows_state_tc.cu)
//
// q and k stay the bf16 vectors they come as; what makes them unit vectors is a factor per row on a product's result or on its other
// operand.  Everything else that enters a product is a 32-bit value taken as two bf16 terms (16 mantissa bits): state, X, U, the inverse
// (whose product with X leaves out lower times lower).  Accumulators, decays, the inverse and the state are 32-bit.  Every wait is bounded
// and reports through the status word; no cluster, no multicast.
#include "k_rows_state_tc.cuh"

namespace sfb {
namespace rdelta {
using namespace rst;

struct Args {
  const int *c_row0, *c_rows;      // chunks
  const int *seg, *first;          // runs: segment, first chunk (one entry more than runs)
  const int *seg_src, *seg_dst;
  const __nv_bfloat16* qkv;        // [n, stride]: q, k, v from the columns below
  int64_t stride;
  const __nv_bfloat16 *dt, *beta;  // [n, .] raw step sizes, raw write strengths
  int64_t dt_stride, beta_stride;
  const float *dt_bias, *a;        // [H]
  float* S;                        // [slots, H, P, Np]
  float* rates;                    // [chunks, H, RATES, 128]
  float* dec;                      // [chunks, H] decay over the whole chunk
  __nv_bfloat16* inv;              // [chunks, H, 2, 128, 128]: upper terms, lower terms (columns 64.. of rows below 64 are not written)
  int H, G, N, P, Np, ns, hpc, chunks;
  int q_col, k_col, v_col;
  float q_scale, unit_eps;
  Status* status;
};

constexpr int LD = 132;            // row stride of the matrix that is inverted

// One warp, one head: running sums of log2 of the decays (a lane takes four rows; past the end: decay 1) and write strengths (past the end: 0).
__device__ __forceinline__ void head_rates(const Args& a, int chunk, int h, int row0, int rows, float* cs, float* bs) {
  const int lane = threadIdx.x & 31;
  const float ah = a.a[h] * LOG2E, bias = a.dt_bias[h];
  float z[4], b[4], c[4], t = 0.f;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int i = min(lane * 4 + k, rows - 1);
    z[k] = __bfloat162float(a.dt[(size_t)(row0 + i) * a.dt_stride + h]) + bias;
    b[k] = __bfloat162float(a.beta[(size_t)(row0 + i) * a.beta_stride + h]);
  }
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const bool in = lane * 4 + k < rows;
    b[k] = in ? 1.f / (1.f + expf(-b[k])) : 0.f;
    t += in ? ah * (log1pf(expf(-fabsf(z[k]))) + fmaxf(z[k], 0.f)) : 0.f;
    c[k] = t;
  }
  float s = t;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, s, o); if (lane >= o) s += v; }
  const float last = __shfl_sync(0xffffffffu, s, 31), before = s - t;
#pragma unroll
  for (int k = 0; k < 4; ++k) c[k] += before;
  rows::store_v<float, 4>(cs + lane * 4, c);
  rows::store_v<float, 4>(bs + lane * 4, b);
  if (lane == 0) a.dec[(size_t)chunk * a.H + h] = ex2(last);
}

// acc[r][c] += sum over k in [k0, k1) of x[r][k] y[k][c], four by four; x, y: rows of LD floats, k0 and k1 multiples of four
__device__ __forceinline__ void micro(float (&acc)[4][4], const float* x, const float* y, int k0, int k1) {
  for (int k = k0; k < k1; k += 4) {
    float4 l[4], r[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      l[i] = *reinterpret_cast<const float4*>(x + i * LD + k);
      r[i] = *reinterpret_cast<const float4*>(y + (k + i) * LD);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float lv[4] = {l[i].x, l[i].y, l[i].z, l[i].w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[i][0] = fmaf(lv[j], r[j].x, acc[i][0]); acc[i][1] = fmaf(lv[j], r[j].y, acc[i][1]);
        acc[i][2] = fmaf(lv[j], r[j].z, acc[i][2]); acc[i][3] = fmaf(lv[j], r[j].w, acc[i][3]);
      }
    }
  }
}

// The block below a pair of inverted diagonal blocks of B rows at `b0`: -T22 (A21 T11).  A warp takes 16 rows (from `r0`) x 32 columns (from
// `c0`), four by four a thread.  The block above the diagonal holds the inner product.  Two calls, a barrier in between.
template <int B>
__device__ __forceinline__ void pair_inner(float* A, int b0, int r0, int c0) {
  const int r = r0 + (threadIdx.x >> 3 & 3) * 4, c = c0 + (threadIdx.x & 7) * 4;
  float acc[4][4] = {};
  micro(acc, A + (b0 + B + r) * LD + b0, A + b0 * LD + b0 + c, c0, B);      // T11 is lower triangular
#pragma unroll
  for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(A + (b0 + r + i) * LD + b0 + B + c) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
}
template <int B>
__device__ __forceinline__ void pair_outer(float* A, int b0, int r0, int c0) {
  const int r = r0 + (threadIdx.x >> 3 & 3) * 4, c = c0 + (threadIdx.x & 7) * 4;
  float acc[4][4] = {};
  micro(acc, A + (b0 + B + r) * LD + b0 + B, A + b0 * LD + b0 + B + c, 0, r0 + 16);
#pragma unroll
  for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(A + (b0 + B + r + i) * LD + b0 + c) = make_float4(-acc[i][0], -acc[i][1], -acc[i][2], -acc[i][3]);
}

// grid (groups x parts of a group's heads, chunks); 256 threads
__global__ void __launch_bounds__(WORK, 3) delta_prep_kernel(const __grid_constant__ CUtensorMap mk, Args a) {
  extern __shared__ __align__(1024) uint8_t sm[];
  uint8_t* ks = sm;                                       // k, two slabs; after k k^T:
  float* A = reinterpret_cast<float*>(sm);                // [128][LD]
  float* rk = A + L * LD;                                 // [128] each: factors to unit length
  float *rq = rk + L, *css = rq + L, *bss = css + a.hpc * L;      // [hpc][128]: running sums, write strengths
  Ctl& C = *reinterpret_cast<Ctl*>(bss + a.hpc * L);
  setup(C, 128);
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.y, rep = a.H / a.G, parts = (rep + a.hpc - 1) / a.hpc, g = blockIdx.x / parts;
  const int h0 = g * rep + (blockIdx.x % parts) * a.hpc, nh = min(a.hpc, (g + 1) * rep - h0), row0 = a.c_row0[chunk], rows = a.c_rows[chunk];
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;
  volatile int* dead = &C.dead;
  if (warp == 0) {
    if (elect_one()) {
      mbar_expect(&C.full[0], a.ns * SLAB);
      for (int s = 0; s < a.ns; ++s) tma2d(ks + s * SLAB, &mk, a.k_col + g * a.N + 64 * s, row0, &C.full[0]);
    }
    wait_warp(&C.full[0], 0, dead, 2);
    if (elect_one()) {
      const uint32_t id = idesc(128, 0, 0);
      const uint64_t dk = desc(smem_u32(ks), 16);
      for (int t = 0; t < a.N / 16; ++t) {
        const uint64_t o = (uint64_t)(t >> 2) * (SLAB >> 4) + (t & 3) * 2;
        mma_ss(C.tmem, dk + o, dk + o, id, t ? 1u : 0u);
      }
      commit(&C.done[0]);
    }
    __syncwarp();
  }
  for (int x = WORK / 32 - 1 - warp; x < nh; x += WORK / 32) head_rates(a, chunk, h0 + x, row0, rows, css + x * L, bss + x * L);
  {   // eight lanes per row and vector: its factor to unit length
    const int sub = lane & 7, words = a.N / 8;
#pragma unroll
    for (int t0 = 0; t0 < 8; t0 += 4) {
      uint4 v[4][2];
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        const int rv = warp * 32 + (t0 + t) * 4 + (lane >> 3), i = rv & (L - 1);      // the first 128: q, then k
        const uint4* p = reinterpret_cast<const uint4*>(a.qkv + (size_t)(row0 + min(i, rows - 1)) * a.stride + (rv >> 7 ? a.k_col : a.q_col) + g * a.N);
#pragma unroll
        for (int q = 0; q < 2; ++q) v[t][q] = sub + 8 * q < words ? p[sub + 8 * q] : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        float s = 0.f;
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const uint32_t x[4] = {v[t][q].x, v[t][q].y, v[t][q].z, v[t][q].w};
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float f0 = __uint_as_float(x[k] << 16), f1 = __uint_as_float(x[k] & 0xffff0000u);
            s = fmaf(f0, f0, s);
            s = fmaf(f1, f1, s);
          }
        }
        s += __shfl_xor_sync(0xffffffffu, s, 1);
        s += __shfl_xor_sync(0xffffffffu, s, 2);
        s += __shfl_xor_sync(0xffffffffu, s, 4);
        const int rv = warp * 32 + (t0 + t) * 4 + (lane >> 3);
        if (sub == 0) (rv >> 7 ? rk : rq)[rv & (L - 1)] = (rv >> 7 ? 1.f : a.q_scale) / sqrtf(s + a.unit_eps);
      }
    }
  }
  const int w4 = warp & 3, half = warp >> 2, i = w4 * 32 + lane;
  wait_warp(&C.done[0], 0, dead, 3);
  fence_after();
  for (int x = 0; x < nh; ++x) {
    const int h = h0 + x;
    const float *cs = css + x * L, *bs = bss + x * L;
    __syncthreads();                                      // the numbers are there; the matrix of the head before has been written out
    if (tid < L) {
      float* o = a.rates + ((size_t)chunk * a.H + h) * RATES * L + tid;
      const bool in = tid < rows;
      const float c = cs[tid], f = rk[tid];
      o[0] = c;
      o[L] = in ? c - __log2f(f) : INFINITY;              // its exponential: 0
      o[2 * L] = rq[tid];
      o[3 * L] = in ? ex2(c) * f : 0.f;
      o[4 * L] = bs[tid];
      o[5 * L] = in ? ex2(cs[L - 1] - c) * f : 0.f;
    }
    {
      const float ci = cs[i], bi = i < rows ? bs[i] * rk[i] : 0.f;
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        const int j0 = half * 64 + b * 32;
        if (j0 > w4 * 32 + 31) continue;                  // above the diagonal: not read below
        float s[32];
        ld32(C.tmem + j0 + ((uint32_t)(w4 * 32) << 16), s);
        wait_ld();
#pragma unroll
        for (int q = 0; q < 8; ++q) {
          float o[4], cj[4], rj[4];
          rows::load_v<float, 4>(cs + j0 + 4 * q, cj);
          rows::load_v<float, 4>(rk + j0 + 4 * q, rj);
#pragma unroll
          for (int k = 0; k < 4; ++k) o[k] = j0 + 4 * q + k < i && i < rows ? s[4 * q + k] * bi * rj[k] * ex2(ci - cj[k]) : 0.f;
          *reinterpret_cast<float4*>(A + i * LD + j0 + 4 * q) = make_float4(o[0], o[1], o[2], o[3]);
        }
      }
    }
    __syncthreads();
    if (warp < 4) {   // a diagonal block: lane = column, row after row
      float t[32];
      float* B = A + (warp * 32) * LD + warp * 32;
#pragma unroll
      for (int r = 0; r < 32; ++r) {
        float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
        for (int k = 0; k < r; k += 4) {                  // elements at and past the diagonal are 0
          const float4 v = *reinterpret_cast<const float4*>(B + r * LD + k);
          s0 = fmaf(v.x, t[k], s0);
          if (k + 1 < r) s1 = fmaf(v.y, t[k + 1], s1);
          if (k + 2 < r) s2 = fmaf(v.z, t[k + 2], s2);
          if (k + 3 < r) s3 = fmaf(v.w, t[k + 3], s3);
        }
        t[r] = r == lane ? 1.f : -((s0 + s1) + (s2 + s3));
      }
      __syncwarp();
#pragma unroll
      for (int r = 0; r < 32; ++r) B[r * LD + lane] = t[r];
    }
    __syncthreads();
    if (warp < 4) pair_inner<32>(A, (warp >> 1) * 64, (warp & 1) * 16, 0);
    __syncthreads();
    if (warp < 4) pair_outer<32>(A, (warp >> 1) * 64, (warp & 1) * 16, 0);
    __syncthreads();
    {                 // the two blocks of 32 above the diagonal inside the blocks of 64
      const int p = tid >> 7, r = tid >> 2 & 31, c = (tid & 3) * 8;
#pragma unroll
      for (int k = 0; k < 8; k += 4) *reinterpret_cast<float4*>(A + (p * 64 + r) * LD + p * 64 + 32 + c + k) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pair_inner<64>(A, 0, (warp >> 1) * 16, (warp & 1) * 32);
    __syncthreads();
    pair_outer<64>(A, 0, (warp >> 1) * 16, (warp & 1) * 32);
    __syncthreads();
    __nv_bfloat16* hi = a.inv + ((size_t)chunk * a.H + h) * 2 * L * L;
#pragma unroll 4
    for (int k = 0; k < 12; ++k) {       // a warp: two of the first 64 rows (their first half) at a time, then one of the others
      const int r = k < 4 ? (warp * 4 + k) * 2 + (lane >> 4) : 64 + warp * 8 + k - 4, c = (k < 4 ? lane & 15 : lane) * 4;
      const float4 v = *reinterpret_cast<const float4*>(A + r * LD + c);
      uint2 u, l;
      split2(v.x, v.y, u.x, l.x);
      split2(v.z, v.w, u.y, l.y);
      *reinterpret_cast<uint2*>(hi + r * L + c) = u;
      *reinterpret_cast<uint2*>(hi + (L + r) * L + c) = l;
    }
  }
  fence_before();
  if (*dead) drain(C);
  teardown(C, 128, a.status, 73);
}

// sixteen 32-bit values as two bf16 terms: 16-byte words of the upper and of the lower ones
__device__ __forceinline__ void split16(const float* f, uint4 (&hi)[2], uint4 (&lo)[2]) {
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    split2(f[8 * q], f[8 * q + 1], hi[q].x, lo[q].x); split2(f[8 * q + 2], f[8 * q + 3], hi[q].y, lo[q].y);
    split2(f[8 * q + 4], f[8 * q + 5], hi[q].z, lo[q].z); split2(f[8 * q + 6], f[8 * q + 7], hi[q].w, lo[q].w);
  }
}

constexpr int PT = 32, TILE = L * PT * 2;             // value dims of a block; bytes of 128 rows of them

// grid (heads x tiles of 32 value dims, runs).  Operands with the value dims along a row (state, X, U) are 128 rows of 128 bytes: the upper terms
// of the tile, then the lower ones, so that one product takes both (64 columns, whose halves are added up as they are read).
__global__ void __launch_bounds__(THREADS, 1)
delta_chain_kernel(const __grid_constant__ CUtensorMap mk, const __grid_constant__ CUtensorMap mt, const __grid_constant__ CUtensorMap mt64,
                   const __grid_constant__ CUtensorMap mv, const __grid_constant__ CUtensorMap mu, const __grid_constant__ CUtensorMap ms, Args a) {
  extern __shared__ __align__(1024) uint8_t sm[];
  uint8_t* ks = sm;                                       // two stages of two slabs
  uint8_t* ts = ks + 4 * SLAB;                            // inverse: upper terms (two slabs), lower terms
  uint8_t* ss = ts + 4 * SLAB;                            // state
  uint8_t* xs = ss + SLAB;                                // X, then U
  uint8_t* vs = xs + SLAB;                                // values, two stages of a tile (128 rows of 64 bytes)
  uint8_t* us = vs + 2 * TILE;                            // U and the state on their way out: tiles of the upper and of the lower terms
  uint8_t* so = us + 2 * TILE;
  Ctl& C = *reinterpret_cast<Ctl*>(so + 2 * TILE);
  setup(C, 256);
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;
  // columns 64.. of the inverse's rows below 64 are zero and never loaded
  for (int x = tid; x < 2 * HSLAB / 16; x += THREADS)
    reinterpret_cast<uint4*>(ts + (x / (HSLAB / 16)) * 2 * SLAB + SLAB)[x % (HSLAB / 16)] = make_uint4(0u, 0u, 0u, 0u);
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();
  const int tiles = (a.P + PT - 1) / PT, h = blockIdx.x / tiles, pt = blockIdx.x % tiles, g = h / (a.H / a.G);
  const int run = blockIdx.y, seg = a.seg[run], c0 = a.first[run], nc = a.first[run + 1] - c0;
  const bool issuer = warp == WORK / 32;
  volatile int* dead = &C.dead;
  const uint32_t t_ks = C.tmem, t_u = t_ks + 2 * PT, t_d = t_u + 2 * PT, t_l = t_d + 2 * PT;      // t_l: lower terms of the inverse
  if (issuer) {
    auto load_k = [&](int c) {
      const int y = a.c_row0[c0 + c];
      mbar_expect(&C.full[c & 1], a.ns * SLAB + TILE);
      for (int s = 0; s < a.ns; ++s) tma2d(ks + ((c & 1) * 2 + s) * SLAB, &mk, a.k_col + g * a.N + 64 * s, y, &C.full[c & 1]);
      tma2d(vs + (c & 1) * TILE, &mv, a.v_col + h * a.P + pt * PT, y, &C.full[c & 1]);
    };
    auto load_t = [&](int c) {
      const int y = ((c0 + c) * a.H + h) * 2 * L;
      mbar_expect(&C.full[2], 2 * (SLAB + HSLAB));
      for (int t = 0; t < 2; ++t) {
        tma2d(ts + t * 2 * SLAB, &mt, 0, y + t * L, &C.full[2]);
        tma2d(ts + t * 2 * SLAB + SLAB + HSLAB, &mt64, 64, y + t * L + 64, &C.full[2]);
      }
    };
    const bool leader = elect_one();
    if (leader) {
      load_k(0);
      load_t(0);
      if (nc > 1) load_k(1);
    }
    __syncwarp();
    const uint32_t id = idesc(2 * PT, 0, 1), id1 = idesc(PT, 0, 1), idt = idesc(2 * PT, 1, 1);
    const uint64_t dt = desc(smem_u32(ts), 16), ds = desc(smem_u32(ss), SLAB), dx = desc(smem_u32(xs), SLAB);
    const int kst = a.N / 16;
    auto store_u = [&](int c) {
      for (int t = 0; t < 2; ++t) tma_store2d(&mu, pt * PT, ((t * a.chunks + c0 + c) * a.H + h) * L, us + t * TILE);
      bulk_commit();
    };
    for (int c = 0; c < nc; ++c) {
      const uint64_t dk = desc(smem_u32(ks) + (c & 1) * 2 * SLAB, 16), dkt = desc(smem_u32(ks) + (c & 1) * 2 * SLAB, SLAB);
      wait_warp(&C.full[c & 1], (c >> 1) & 1, dead, 4);
      if (leader) bulk_wait_read();                       // the tile of the state before has left
      __syncwarp();
      __syncthreads();                                    // the state is in place (and the tile of U before)
      if (leader) {
        fence_after();
#pragma unroll
        for (int t = 0; t < 8; ++t)
          if (t < kst) mma_ss(t_ks, dk + (uint64_t)(t >> 2) * (SLAB >> 4) + (t & 3) * 2, ds + (uint64_t)t * (2048 >> 4), id, t ? 1u : 0u);
        commit(&C.done[0]);
        if (c > 0) store_u(c - 1);
      }
      __syncwarp();
      wait_warp(&C.full[2], c & 1, dead, 5);
      __syncthreads();                                    // X is in place (and the tile of the state)
      if (leader) {
        bulk_wait_read();                                 // the tile of U before has left
        fence_after();
#pragma unroll
        for (int t = 0; t < 8; ++t) {
          const uint64_t ta = dt + (uint64_t)(t >> 2) * (SLAB >> 4) + (t & 3) * 2, xb = dx + (uint64_t)t * (2048 >> 4);
          mma_ss(t_u, ta, xb, id, t ? 1u : 0u);
          mma_ss(t_l, ta + 2 * (SLAB >> 4), xb, id1, t ? 1u : 0u);
        }
        commit(&C.done[1]);
        for (int t = 0; t < 2; ++t) tma_store2d(&ms, pt * PT, ((t * a.chunks + c0 + c) * a.H + h) * a.N, so + t * TILE);
        bulk_commit();
      }
      __syncwarp();
      wait_warp(&C.done[1], c & 1, dead, 6);
      if (c + 1 < nc && leader) load_t(c + 1);
      __syncwarp();
      __syncthreads();                                    // U is in place
      if (leader) {
        fence_after();
#pragma unroll
        for (int t = 0; t < 8; ++t) {
          const uint64_t o = (uint64_t)t * (2048 >> 4);
          mma_ss(t_d, dkt + o, dx + o, idt, t ? 1u : 0u);
        }
        commit(&C.done[2]);
      }
      __syncwarp();
      wait_warp(&C.done[2], c & 1, dead, 7);
      if (c + 2 < nc && leader) load_k(c + 2);
      __syncwarp();
    }
    __syncthreads();                                      // the last tile of U is in place
    if (leader) {
      store_u(nc - 1);
      bulk_wait();
    }
    __syncwarp();
  } else {
    // a thread has one row (of the chunk, or of the state) and sixteen value dims
    const int w4 = warp & 3, half = warp >> 2, i = w4 * 32 + lane, p0 = pt * PT + half * 16, width = min(16, a.P - p0);      // width: a multiple of 8, or none
    const uint32_t at = ((uint32_t)(w4 * 32) << 16) + half * 16;
    const size_t slot = (size_t)a.H * a.P * a.Np;
    const bool in_n = i < a.N;
    float S[16];
    {
      const int src = a.seg_src[seg];
      const float* s0 = a.S + (size_t)(src >= 0 ? src : 0) * slot + ((size_t)h * a.P + p0) * a.Np + i;
#pragma unroll
      for (int k = 0; k < 16; ++k) S[k] = src >= 0 && in_n && k < width ? s0[(size_t)k * a.Np] : 0.f;
    }
    auto put = [&](uint8_t* op, const uint4 (&hi)[2], const uint4 (&lo)[2]) {      // row i, 128-byte swizzle
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        *reinterpret_cast<uint4*>(op + i * 128 + (((half * 2 + q) ^ (i & 7)) << 4)) = hi[q];
        *reinterpret_cast<uint4*>(op + i * 128 + (((half * 2 + q + 4) ^ (i & 7)) << 4)) = lo[q];
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      fence_before();
      __syncthreads();
    };
    auto read = [&](uint32_t t, float (&f)[16]) {                                   // the sum of both terms' products
      float l[16];
      ld16(t + at, f);
      ld16(t + PT + at, l);
      wait_ld();
#pragma unroll
      for (int k = 0; k < 16; ++k) f[k] += l[k];
    };
    auto put_out = [&](uint8_t* tile, const uint4 (&h2)[2], const uint4 (&l2)[2]) {      // row i of the tiles on their way out, 64-byte swizzle
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int o = i * 64 + (((half * 2 + q) ^ (i >> 1 & 3)) << 4);
        *reinterpret_cast<uint4*>(tile + o) = h2[q];
        *reinterpret_cast<uint4*>(tile + TILE + o) = l2[q];
      }                                                   // (the next `put` orders them ahead of the copy)
    };
    uint4 hi[2], lo[2];
    auto put_state = [&]() {
      split16(S, hi, lo);
      put(ss, hi, lo);
      put_out(so, hi, lo);                                // under the product
    };
    float ek, b, ue, dec;
    int rows = a.c_rows[c0], rows1 = nc > 1 ? a.c_rows[c0 + 1] : 0;                 // this chunk's, the next one's
    auto fetch = [&](int c, float& x, float& y, float& z, float& d) {               // numbers of chunk c
      const float* n = a.rates + ((size_t)(c0 + c) * a.H + h) * RATES * L + i;
      x = n[3 * L]; y = n[4 * L]; z = n[5 * L];
      d = a.dec[(size_t)(c0 + c) * a.H + h];
    };
    fetch(0, ek, b, ue, dec);
    put_state();
    for (int c = 0; c < nc; ++c) {
      float f[16], ek1 = 0.f, b1 = 0.f, ue1 = 0.f, dec1 = 0.f;
      int rows2 = 0;
      uint4 v[2];
      wait_warp(&C.full[c & 1], (c >> 1) & 1, dead, 11);
#pragma unroll
      for (int q = 0; q < 2; ++q) v[q] = *reinterpret_cast<const uint4*>(vs + (c & 1) * TILE + i * 64 + (((half * 2 + q) ^ (i >> 1 & 3)) << 4));
      if (c + 1 < nc) {                                   // requested a chunk ahead
        fetch(c + 1, ek1, b1, ue1, dec1);
        if (c + 2 < nc) rows2 = a.c_rows[c0 + c + 2];
      }
      wait_warp(&C.done[0], c & 1, dead, 8);
      fence_after();
      read(t_ks, f);
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const uint32_t vw[4] = {v[q].x, v[q].y, v[q].z, v[q].w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          float* x = f + 8 * q + 2 * k;
          x[0] = i < rows ? b * (__uint_as_float(vw[k] << 16) - ek * x[0]) : 0.f;
          x[1] = i < rows ? b * (__uint_as_float(vw[k] & 0xffff0000u) - ek * x[1]) : 0.f;
        }
      }
      split16(f, hi, lo);
      put(xs, hi, lo);
      wait_warp(&C.done[1], c & 1, dead, 9);
      fence_after();
      {
        float l[16];
        ld16(t_l + at, l);
        read(t_u, f);
#pragma unroll
        for (int k = 0; k < 16; ++k) f[k] += l[k];
      }
      {
        float x[16];
#pragma unroll
        for (int k = 0; k < 16; ++k) x[k] = i < rows ? f[k] * ue : 0.f;
        split16(x, hi, lo);
      }
      put(xs, hi, lo);
      split16(f, hi, lo);
      put_out(us, hi, lo);                                // under the product
      wait_warp(&C.done[2], c & 1, dead, 10);
      fence_after();
      read(t_d, f);
#pragma unroll
      for (int k = 0; k < 16; ++k) S[k] = in_n ? fmaf(dec, S[k], f[k]) : 0.f;
      if (c + 1 < nc) put_state();
      ek = ek1; b = b1; ue = ue1; dec = dec1; rows = rows1; rows1 = rows2;
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    fence_before();
    __syncthreads();
    if (in_n) {
      float* s1 = a.S + (size_t)a.seg_dst[seg] * slot + ((size_t)h * a.P + p0) * a.Np + i;
#pragma unroll
      for (int k = 0; k < 16; ++k)
        if (k < width) s1[(size_t)k * a.Np] = S[k];
    }
  }
  drain(C);
  teardown(C, 256, a.status, 74);
}

}  // namespace rdelta
}  // namespace sfb

using namespace sfb;
using namespace sfb::rdelta;

extern "C" {

// mk: rows of q | k | v, box 128 rows; mt, mt64: inv seen as [256 chunks H, 128], boxes of 128 and 64 rows; with 32 columns: mv: as mk; mu: u seen as
// [2 chunks H 128, P], box 128 rows; ms: starts seen as [2 chunks H N, P], box N rows.  N: a multiple of 16 up to 128; P: a
// multiple of 8; first columns and stride multiples of 8.  The rows between N and Np of the stored states are not written.
int sfb_rows_delta_tc(const void* mk, const void* mt, const void* mt64, const void* mv, const void* mu, const void* ms, const int* c_row0, const int* c_rows, const int* seg, const int* first, const int* seg_src,
                      const int* seg_dst, const void* qkv, int64_t stride, const void* dt, int64_t dt_stride, const void* beta, int64_t beta_stride,
                      const void* dt_bias, const void* la, void* S, void* rates, void* dec, void* inv, int runs, int chunks, int H,
                      int G, int N, int P, int Np, int q_col, int k_col, int v_col, float q_scale, float unit_eps, void* status, cudaStream_t stream) {
  if (runs < 1 || runs > 65535 || chunks < 1 || chunks > 65535 || G < 1 || H % G || N < 16 || N % 16 || N > 128 || P < 8 || P % 8 || Np < N ||
      (q_col | k_col | v_col) % 8 || stride % 8 || (uintptr_t)qkv % 16)
    return (int)cudaErrorInvalidValue;
  Args a{c_row0, c_rows, seg, first, seg_src, seg_dst, (const __nv_bfloat16*)qkv, stride, (const __nv_bfloat16*)dt, (const __nv_bfloat16*)beta, dt_stride,
         beta_stride, (const float*)dt_bias, (const float*)la, (float*)S, (float*)rates, (float*)dec, (__nv_bfloat16*)inv,
         H, G, N, P, Np, (N + 63) / 64, 1, chunks, q_col, k_col, v_col, q_scale, unit_eps, (Status*)status};
  const int rep = H / G;
  a.hpc = rep < 8 ? rep : 8;                 // heads that share a block's K K^T: fewer where that leaves SMs empty
  while (a.hpc > 1 && (long long)G * ((rep + a.hpc - 1) / a.hpc) * chunks < 296) a.hpc = (a.hpc + 1) / 2;
  static size_t granted[2] = {0, 0};
  const size_t prep = ((size_t)L * LD + (2 + 2 * a.hpc) * L) * sizeof(float) + sizeof(Ctl), chain = (size_t)10 * SLAB + 6 * TILE + sizeof(Ctl);
  cudaError_t rc = grant(delta_prep_kernel, prep, granted[0]);
  if (rc == cudaSuccess) rc = grant(delta_chain_kernel, chain, granted[1]);
  if (rc == cudaSuccess)
    rc = sfb_launch(delta_prep_kernel, dim3(G * ((rep + a.hpc - 1) / a.hpc), chunks), dim3(WORK), prep, stream, *(const CUtensorMap*)mk, a);
  if (rc == cudaSuccess)
    rc = sfb_launch(delta_chain_kernel, dim3(H * ((P + PT - 1) / PT), runs), dim3(THREADS), chain, stream, *(const CUtensorMap*)mk, *(const CUtensorMap*)mt,
                    *(const CUtensorMap*)mt64, *(const CUtensorMap*)mv, *(const CUtensorMap*)mu, *(const CUtensorMap*)ms, a);
  return (int)rc;
}

}  // extern "C"
