// Products of a mixture of experts on tcgen05, bf16: the tiles of k_rows_moe.cu's plan (up to 128 pairs of one expert) against that expert's
// weights, 32-bit accumulators.
//
//   gated   act(x Wg^T, x Wu^T): 128 pairs x 128 gate columns beside their 128 up columns; results in plan order.  With few rows the pairs' rows
//           are gathered by TMA straight from the layer's input (four rows a copy); many are brought into plan order first (`pick`)
//   single  act(x W^T): the same with 256 columns of one matrix
//   down    128 pairs x 256 columns; rows in plan order; every result row goes to its [row][choice]
//
// The shared expert's rows (all of the step, in order, with sizes of their own) are tiles of the same launches, ahead of the others.
//
// Persistent: one CTA per SM takes every gridDim-th of the tiles x column blocks (the column blocks of a tile side by side, so that its rows
// and its expert's weights stay in L2).  Warp 0 copies (K in steps of 64 through a ring of four stages), warp 1 issues the products, warps
// 2-5 take the results out of tensor memory, where two accumulators of 256 columns take turns, so that a tile's results leave under the
// next tile's products.  Every wait is bounded and reports through the status word; no cluster, no multicast.
#include "k_rows_tc.cuh"

namespace sfb {
namespace rmoetc {
using namespace tc;

constexpr int THREADS = 192, ROWS = 128, COLS = 256, KS = 64, ST = 4, XSLAB = ROWS * 128, WSLAB = COLS * 128;

constexpr int DOWN = 0, GATED = 1, SINGLE = 2;

struct Args {
  const int *order, *tiles, *count;
  __nv_bfloat16 *out, *sout; // first product: [pairs, M], the shared expert's [n, SM]; down: [n, slots, M]
  int M, K, SM, SK, top, slots, act, cblocks, sblocks;     // cblocks, sblocks: blocks of 128 (gated) or 256 columns
  int stotal, n;             // tiles x column blocks of the shared expert (0: none), its rows
  float alpha, limit, slimit;
  Status* status;
};

// what one turn of a CTA works on
struct Job {
  int4 t;                    // expert, first place (shared: row), pairs, -
  int c0, M, K, shared;
};
template <int KIND>
__device__ __forceinline__ Job job(const Args& a, int b) {
  Job j;
  j.shared = b < a.stotal;
  const int x = j.shared ? b : b - a.stotal, blocks = j.shared ? a.sblocks : a.cblocks, ti = x / blocks;
  j.t = j.shared ? make_int4(0, ti * 128, min(128, a.n - ti * 128), 0) : reinterpret_cast<const int4*>(a.tiles)[ti];
  j.c0 = (x % blocks) * (KIND == GATED ? 128 : 256);
  j.M = j.shared ? a.SM : a.M;
  j.K = j.shared ? a.SK : a.K;
  return j;
}

struct Smem {
  alignas(1024) uint8_t x[ST * XSLAB];
  alignas(1024) uint8_t w[ST * WSLAB];
  alignas(8) uint64_t full[ST], empty[ST], acc_full[2], acc_empty[2];
  uint32_t tmem;
  int dead;
};

// rows y[0..3] of the map, 64 columns from x on, one after another
__device__ __forceinline__ void gather4(void* dst, const CUtensorMap* map, int x, int4 y, uint64_t* bar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cta.global.tile::gather4.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5, %6}], [%7];"
               ::"r"(smem_u32(dst)), "l"(map), "r"(x), "r"(y.x), "r"(y.y), "r"(y.z), "r"(y.w), "r"(smem_u32(bar)) : "memory");
}

// the layer's input rows in plan order, 16-byte words; a warp per pair
__global__ void __launch_bounds__(256) moe_pick_kernel(const uint4* x, const int* order, uint4* out, int pairs, int top, int words) {
  pdl_launch_dependents();
  pdl_wait();
  const int place = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (place >= pairs) return;
  const uint4* src = x + (size_t)(order[place] / top) * words;
  uint4* dst = out + (size_t)place * words;
  for (int w = lane; w < words; w += 256) {
    uint4 v[8];
#pragma unroll
    for (int k = 0; k < 8; ++k)
      if (w + 32 * k < words) v[k] = src[w + 32 * k];
#pragma unroll
    for (int k = 0; k < 8; ++k)
      if (w + 32 * k < words) dst[w + 32 * k] = v[k];
  }
}

template <int KIND, bool GATHER>
__global__ void __launch_bounds__(THREADS, 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap mx, const __grid_constant__ CUtensorMap mw, const __grid_constant__ CUtensorMap msx,
                const __grid_constant__ CUtensorMap msw, Args a) {
  extern __shared__ uint8_t raw[];
  Smem& S = *reinterpret_cast<Smem*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~(uintptr_t)1023);
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;
  volatile int* dead = &S.dead;
  if (tid == 0) {
    S.dead = 0;
    for (int i = 0; i < ST; ++i) { mbar_init(&S.full[i], 1); mbar_init(&S.empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&S.acc_full[i], 1); mbar_init(&S.acc_empty[i], 128); }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], 512;" ::"r"(smem_u32(&S.tmem)) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_launch_dependents();
  fence_before();
  __syncthreads();
  fence_after();
  pdl_wait();
  const uint32_t tmem = S.tmem;
  const int total = a.stotal + *a.count * a.cblocks;

  if (warp == 0) {
    int it = 0;              // stages filled so far
    for (int b = blockIdx.x; b < total && !*dead; b += gridDim.x) {
      const Job j = job<KIND>(a, b);
      const int4 t = j.t;
      const bool gather = GATHER && !j.shared;
      int4 rows = make_int4(0, 0, 0, 0);      // a lane gathers four rows, the tile's last one again past its end; lanes past it none
      if (gather) {
        int* r = reinterpret_cast<int*>(&rows);
#pragma unroll
        for (int k = 0; k < 4; ++k) r[k] = a.order[t.y + min(lane * 4 + k, t.z - 1)] / a.top;
      }
      const int wrow = t.x * (KIND == GATED ? 2 : 1) * j.M + j.c0, steps = (j.K + KS - 1) / KS;
      const CUtensorMap *x = j.shared ? &msx : &mx, *w = j.shared ? &msw : &mw;
      for (int k = 0; k < steps; ++k, ++it) {
        const int st = it % ST, ph = (it / ST) & 1;
        const bool ok = mbar_wait(&S.empty[st], ph ^ 1, dead);
        if (!__all_sync(0xffffffffu, ok)) break;
        if (lane == 0) mbar_expect(&S.full[st], (gather ? (t.z + 3) / 4 * 512 : XSLAB) + WSLAB);
        __syncwarp();
        if (gather && lane * 4 < t.z) gather4(S.x + st * XSLAB + lane * 512, &mx, k * KS, rows, &S.full[st]);
        if (lane == 0) {
          if (!gather) tma2d(S.x + st * XSLAB, x, k * KS, t.y, &S.full[st]);
          tma2d(S.w + st * WSLAB, w, k * KS, wrow, &S.full[st]);
          tma2d(S.w + st * WSLAB + XSLAB, w, k * KS, wrow + (KIND == GATED ? j.M : 128), &S.full[st]);
        }
      }
    }
    if (*dead && lane == 0) {       // copies still in flight must land before the CTA ends
      for (int k = max(0, it - ST); k < it; ++k)
        for (int i = 0; i < 100000 && !mbar_try(&S.full[k % ST], (k / ST) & 1); ++i) __nanosleep(64);
    }
  } else if (warp == 1) {
    if (elect_one()) {
      const uint32_t id = idesc(COLS, 0, 0);
      const uint64_t dx = desc(smem_u32(S.x), 16), dw = desc(smem_u32(S.w), 16);
      int it = 0, n = 0;
      bool ok = true;
      for (int b = blockIdx.x; ok && b < total; b += gridDim.x, ++n) {
        const int acc = n & 1, steps = ((b < a.stotal ? a.SK : a.K) + KS - 1) / KS;
        if (!(ok = mbar_wait(&S.acc_empty[acc], ((n >> 1) & 1) ^ 1, dead))) break;
        fence_after();
        for (int k = 0; k < steps; ++k, ++it) {
          const int st = it % ST;
          if (!(ok = mbar_wait(&S.full[st], (it / ST) & 1, dead))) break;
          fence_after();
          const uint64_t x = dx + (uint64_t)st * (XSLAB >> 4), w = dw + (uint64_t)st * (WSLAB >> 4);
#pragma unroll
          for (int q = 0; q < KS / 16; ++q) mma_ss(tmem + acc * COLS, x + q * 2, w + q * 2, id, (k | q) ? 1u : 0u);
          commit(&S.empty[st]);
        }
        if (ok) commit(&S.acc_full[acc]);
      }
      // no arrival may be under way when the CTA ends
      for (int k = max(0, it - ST); ok && k < it; ++k) ok = mbar_wait(&S.empty[k % ST], (k / ST) & 1, dead);
    }
  } else {
    const int w4 = warp & 3, r = w4 * 32 + lane;      // tensor memory lanes of this warp
    const uint32_t lanes = (uint32_t)(w4 * 32) << 16;
    int n = 0;
    for (int b = blockIdx.x; b < total; b += gridDim.x, ++n) {
      const Job j = job<KIND>(a, b);
      const int acc = n & 1;
      const bool in = r < j.t.z;
      size_t row = 0;
      if (KIND != DOWN) row = (size_t)(j.t.y + r);
      else if (j.shared) row = (size_t)(j.t.y + r) * a.slots + a.top;
      else if (in) { const int pair = a.order[j.t.y + r]; row = (size_t)(pair / a.top) * a.slots + pair % a.top; }
      __nv_bfloat16* o = (KIND != DOWN && j.shared ? a.sout : a.out) + row * j.M + j.c0;
      const float limit = j.shared ? a.slimit : a.limit;
      const bool ok = mbar_wait(&S.acc_full[acc], (n >> 1) & 1, dead);
      if (!__all_sync(0xffffffffu, ok)) break;
      fence_after();
      const uint32_t ta = tmem + acc * COLS + lanes;
      const int width = min(KIND == GATED ? 128 : 256, j.M - j.c0);
      for (int c = 0; c < width; c += 32) {
        float f[32];
        ld32(ta + c, f);
        if constexpr (KIND == GATED) {
          float u[32];
          ld32(ta + 128 + c, u);
          wait_ld();
#pragma unroll
          for (int k = 0; k < 32; ++k) f[k] = rows::gate_clamp<__nv_bfloat16>(f[k], u[k], a.alpha, limit);
        } else {
          wait_ld();
          if constexpr (KIND == SINGLE) {
            if (a.act == rows::ACT_RELU2) {
#pragma unroll
              for (int k = 0; k < 32; ++k) { const float p = fmaxf(f[k], 0.f); f[k] = p * p; }
            } else {
#pragma unroll
              for (int k = 0; k < 32; ++k) f[k] = rows::act_single<__nv_bfloat16>(f[k], rows::ACT_XIELU, a.alpha, limit);
            }
          }
        }
        if (in) {
#pragma unroll
          for (int k = 0; k < 32; k += 8)
            if (c + k < width) rows::store_v<__nv_bfloat16, 8>(o + c + k, f + k);      // M is a multiple of eight
        }
      }
      fence_before();
      mbar_arrive(&S.acc_empty[acc]);
    }
  }
  fence_before();
  __syncthreads();
  if (tid == 0 && *dead) status_set(a.status, ST_TIMEOUT, 75, blockIdx.x, KIND);
  if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, 512;" ::"r"(tmem) : "memory");
}

template <int KIND, bool GATHER>
static int launch(const CUtensorMap* mx, const CUtensorMap* mw, const CUtensorMap* msx, const CUtensorMap* msw, const Args& a, int most, cudaStream_t st) {
  const size_t smem = sizeof(Smem) + 1024;
  static bool done = false;
  if (!done) {
    const cudaError_t e = cudaFuncSetAttribute(moe_gemm_kernel<KIND, GATHER>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    done = true;
  }
  int dev = 0, sms = 148;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  const long long blocks = (long long)most * a.cblocks + a.stotal;
  return (int)sfb_launch(moe_gemm_kernel<KIND, GATHER>, dim3((unsigned)(blocks < sms ? blocks : sms)), dim3(THREADS), smem, st, *mx, *mw, *msx, *msw, a);
}

}  // namespace rmoetc
}  // namespace sfb

using namespace sfb;
using namespace sfb::rmoetc;

extern "C" {

// x [n, K] to out [pairs, K] in plan order; K a multiple of 8
int sfb_rows_moe_pick(const void* x, const void* order, void* out, int pairs, int top, int K, cudaStream_t stream) {
  if (pairs < 1 || top < 1 || K < 8 || K % 8) return (int)cudaErrorInvalidValue;
  return (int)sfb_launch(moe_pick_kernel, dim3((pairs + 7) / 8), dim3(256), 0, stream, (const uint4*)x, (const int*)order, (uint4*)out, pairs, top, K / 8);
}

// mx: rows [pairs, K] in plan order, box 128 rows, or (gather) rows [n, K], box of one row; mw: weights [E (2) M, K], box 128 rows.  msx, msw: the
// same of the shared expert (rows in order), or null.  M, K, SM and SK: multiples of 8; most: the most tiles (of up to 128 pairs) that the plan
// can hold.  act: 0 down, ACT_CLAMP (gated) or an ungated activation with the numbers alpha, limit.
int sfb_rows_moe_gemm(const void* mx, const void* mw, const void* msx, const void* msw, const void* order, const void* tiles, const void* count, void* out, void* sout,
                      int most, int n, int M, int K, int SM, int SK, int top, int slots, int act, int gather, float alpha, float limit, float slimit, void* status,
                      cudaStream_t stream) {
  if (most < 1 || n < 1 || M < 8 || M % 8 || K < 8 || K % 8 || top < 1 || (gather && !act) || (act && act != rows::ACT_CLAMP && act != rows::ACT_RELU2 && act != rows::ACT_XIELU) || (msx && (SM < 8 || SM % 8 || SK < 8 || SK % 8 || slots <= top)) ||
      (uintptr_t)out % 16 || (uintptr_t)sout % 16)
    return (int)cudaErrorInvalidValue;
  const int gated = act == rows::ACT_CLAMP, per = gated ? 128 : 256;
  Args a{(const int*)order, (const int*)tiles, (const int*)count, (__nv_bfloat16*)out, (__nv_bfloat16*)sout, M, K, SM, SK, top, slots, act, (M + per - 1) / per,
         (SM + per - 1) / per, 0, n, alpha, limit, slimit, (Status*)status};
  if (msx) a.stotal = (n + 127) / 128 * a.sblocks;
  const CUtensorMap *x = (const CUtensorMap*)mx, *w = (const CUtensorMap*)mw, *sx = msx ? (const CUtensorMap*)msx : x, *sw = msw ? (const CUtensorMap*)msw : w;
  if (gather) return gated ? launch<GATED, true>(x, w, sx, sw, a, most, stream) : launch<SINGLE, true>(x, w, sx, sw, a, most, stream);
  if (act) return gated ? launch<GATED, false>(x, w, sx, sw, a, most, stream) : launch<SINGLE, false>(x, w, sx, sw, a, most, stream);
  return launch<DOWN, false>(x, w, sx, sw, a, most, stream);
}

}  // extern "C"
