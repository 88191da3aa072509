// Mixture of experts on a step's rows: every row goes through `top` of E feed-forwards (gated, or with one activation), and through a
// shared one.
//
//   moe_route   the chosen experts of a row and their weights, and the shared expert's weight (sigmoid of one more logit); one warp per row.
//               Either the largest logits and the softmax over them; or scores s = sigmoid(logit), the largest s + correction among the
//               groups of neighbouring experts whose two best sum highest, weighted by their s over its sum
//   moe_plan    (row, choice) pairs in order of their expert, cut into tiles of `tile` pairs of one expert; chooses as well when rows are few
//   moe_tile    one tile x 64 output columns on CUDA cores: any sizes, bf16 or 32-bit (k_rows_moe_tc.cu takes bf16 on tcgen05)
//   moe_gemv    one to four rows, bf16: a block per (pair, share of the output), weights streamed; the shared expert's rows beside the
//               pairs; every block of the first product chooses for its row
//
// Both products of an expert go through the same kernels: the first (rows picked by the plan; gate and up rows stacked, act(gate) * up, or one
// matrix and act) and down (rows of the first product in plan order, results at [row][choice], where the seam sums them with their weights).
#include "k_rows.cuh"

namespace sfb {
namespace rmoe {
using namespace rows;

constexpr int MAX_E = 1024, MAX_TOP = 32;

// ---- choice ---------------------------------------------------------------------------------------------------------------
struct RouteArgs {
  const float* z;           // [n, ld] router logits, then (shared) the shared expert's
  int64_t ld;
  int* ids;                 // [n, top]
  float* wts;               // [n, top + shared]
  int n, E, top, shared;
  const float* corr;        // [E]: choice by sigmoid(logit) + corr, weights by the sigmoids; null: by logits and their softmax
  int groups, keep;         // (corr) runs of E / groups experts, of which the best `keep` are open
  float scale;              // (corr) of the weights
};
constexpr int HELD = 8;     // scores a lane holds, the rest is read again
constexpr int MAX_GROUPS = 256;
// bits that compare as the numbers do; above 0 for every number
__device__ __forceinline__ uint32_t rank_bits(float v) {
  const uint32_t b = __float_as_uint(v);
  return b & 0x80000000u ? ~b : b | 0x80000000u;
}
__device__ __forceinline__ float choice_score(const RouteArgs& a, const float* z, int e) { return a.corr ? sigmoid_f(z[e]) + a.corr[e] : z[e]; }

// The warp's largest of v[k] (number k * 32 + lane; 0: none), the lower number among equal ones; it becomes 0.
template <int N> __device__ __forceinline__ int take_best(uint32_t (&v)[N], int none) {
  const int lane = threadIdx.x & 31;
  uint32_t best = 0;
  int at = none;
#pragma unroll
  for (int k = 0; k < N; ++k)
    if (v[k] > best) { best = v[k]; at = k * 32 + lane; }
  const uint32_t top = __reduce_max_sync(0xffffffffu, best);
  at = (int)__reduce_min_sync(0xffffffffu, (unsigned)(best == top ? at : none));
#pragma unroll
  for (int k = 0; k < N; ++k)
    if (at == k * 32 + lane) v[k] = 0u;
  return at;
}

// Groups of 2, 4 .. 32 experts whose scores c the lanes hold: a group is a run of lanes, and its two largest meet in it.  Bit k of the result: this
// lane's expert k * 32 + lane cannot be chosen.
__device__ __forceinline__ uint32_t shut_held(const RouteArgs& a, const float (&c)[HELD], int size) {
  const int lane = threadIdx.x & 31;
  uint32_t v[HELD];
#pragma unroll
  for (int k = 0; k < HELD; ++k) {
    v[k] = 0u;
    if (k * 32 >= a.E) continue;
    float m0 = c[k], m1 = -INFINITY;
    for (int o = 1; o < size; o <<= 1) {
      const float x0 = __shfl_xor_sync(0xffffffffu, m0, o), x1 = __shfl_xor_sync(0xffffffffu, m1, o);
      m1 = fmaxf(fmaxf(m1, x1), fminf(m0, x0));
      m0 = fmaxf(m0, x0);
    }
    if (k * 32 + lane < a.E) v[k] = rank_bits(m0 + m1);
  }
  uint32_t shut = 0xffffffffu;
  for (int i = 0; i < a.keep; ++i) {
    uint32_t best = 0;
    int at = a.groups - 1;
#pragma unroll
    for (int k = 0; k < HELD; ++k)
      if (v[k] > best) { best = v[k]; at = (k * 32 + lane) / size; }
    const uint32_t top = __reduce_max_sync(0xffffffffu, best);
    at = (int)__reduce_min_sync(0xffffffffu, (unsigned)(best == top ? at : a.groups - 1));
#pragma unroll
    for (int k = 0; k < HELD; ++k)
      if (k * 32 + lane < a.E && (k * 32 + lane) / size == at) { v[k] = 0u; shut &= ~(1u << k); }
  }
  return shut;
}
// The same for groups of any size.
__device__ __forceinline__ uint32_t shut_experts(const RouteArgs& a, const float* z) {
  const int lane = threadIdx.x & 31, size = a.E / a.groups;
  constexpr int N = MAX_GROUPS / 32;
  uint32_t v[N];
#pragma unroll
  for (int k = 0; k < N; ++k) v[k] = 0u;
  for (int g = 0; g < a.groups; ++g) {
    float m0 = -INFINITY, m1 = -INFINITY;       // the two largest of the group
    for (int e = lane; e < size; e += 32) {
      const float s = choice_score(a, z, g * size + e);
      m1 = fmaxf(m1, fminf(m0, s));
      m0 = fmaxf(m0, s);
    }
    for (int o = 1; o < 32 && o < size; o <<= 1) {
      const float x0 = __shfl_xor_sync(0xffffffffu, m0, o), x1 = __shfl_xor_sync(0xffffffffu, m1, o);
      m1 = fmaxf(fmaxf(m1, x1), fminf(m0, x0));
      m0 = fmaxf(m0, x0);
    }
    const uint32_t bits = __shfl_sync(0xffffffffu, rank_bits(size > 1 ? m0 + m1 : m0), 0);
#pragma unroll
    for (int k = 0; k < N; ++k)
      if (g == k * 32 + lane) v[k] = bits;
  }
  uint32_t shut = 0xffffffffu;
  for (int i = 0; i < a.keep; ++i) {
    const int g = take_best<N>(v, a.groups - 1);
    for (int k = 0, e = lane; e < a.E; ++k, e += 32)
      if (e / size == g) shut &= ~(1u << k);
  }
  return shut;
}

// One warp, one row: lane j ends up with choice j and its weight (the lower number wins among equal scores); `shared_w`: the shared expert's.
__device__ __forceinline__ void choose(const RouteArgs& a, const float* z, int& id, float& weight, float& shared_w) {
  const int lane = threadIdx.x & 31;
  float c[HELD];
#pragma unroll
  for (int k = 0; k < HELD; ++k) c[k] = k * 32 + lane < a.E ? choice_score(a, z, k * 32 + lane) : -INFINITY;
  uint32_t taken = 0u;      // bit k: this lane's expert k * 32 + lane
  if (a.corr && a.keep < a.groups) {
    const int size = a.E / a.groups;
    taken = a.E <= HELD * 32 && size > 1 && size <= 32 && (size & (size - 1)) == 0 ? shut_held(a, c, size) : shut_experts(a, z);
  }
  uint32_t v[HELD];         // 0: taken, or past the end
#pragma unroll
  for (int k = 0; k < HELD; ++k) v[k] = k * 32 + lane < a.E && !(taken >> k & 1) ? rank_bits(c[k]) : 0u;
  const float zs = a.shared ? z[a.E] : 0.f;
  id = 0;
  for (int j = 0; j < a.top; ++j) {
    uint32_t best = 0;
    int at = a.E;
#pragma unroll
    for (int k = 0; k < HELD; ++k)
      if (v[k] > best) { best = v[k]; at = k * 32 + lane; }
    for (int e = HELD * 32 + lane, k = HELD; e < a.E; e += 32, ++k) {
      const uint32_t x = taken >> k & 1 ? 0u : rank_bits(choice_score(a, z, e));
      if (x > best) { best = x; at = e; }
    }
    const uint32_t top = __reduce_max_sync(0xffffffffu, best);
    at = (int)min(__reduce_min_sync(0xffffffffu, (unsigned)(best == top ? at : a.E)), (unsigned)(a.E - 1));
    if ((at & 31) == lane) {
      taken |= 1u << (at >> 5);
#pragma unroll
      for (int k = 0; k < HELD; ++k)
        if (at >> 5 == k) v[k] = 0u;
    }
    if (lane == j) id = at;
  }
  const float mz = lane < a.top ? z[id] : 0.f;
  if (a.corr) {
    const float s = lane < a.top ? sigmoid_f(mz) : 0.f;
    weight = s / (warp_sum(s) + 1e-20f) * a.scale;
  } else {
    const float top = __shfl_sync(0xffffffffu, mz, 0), e = lane < a.top ? expf(mz - top) : 0.f;
    weight = e / warp_sum(e);
  }
  shared_w = sigmoid_f(zs);
}
__device__ __forceinline__ void route_row(const RouteArgs& a, int row) {
  const int lane = threadIdx.x & 31;
  int id;
  float w, sw;
  choose(a, a.z + (size_t)row * a.ld, id, w, sw);
  float* o = a.wts + (size_t)row * (a.top + a.shared);
  if (lane < a.top) { a.ids[(size_t)row * a.top + lane] = id; o[lane] = w; }
  if (a.shared && lane == 0) o[a.top] = sw;
}
__global__ void __launch_bounds__(256) moe_route_kernel(RouteArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row < a.n) route_row(a, row);
}

// ---- plan -----------------------------------------------------------------------------------------------------------------
struct PlanArgs {
  RouteArgs r;              // r.z null: ids are there
  int* order;               // [pairs] pair at every place
  int* tiles;               // [max tiles][4]: expert, first place, pairs, -
  int* count;               // number of tiles
  int pairs, E, tile;
};
constexpr int BATCH = 16;   // pairs a thread holds: their expert, and how many of it came before (20 bits)

// one block of at least E threads
__global__ void __launch_bounds__(1024) moe_plan_kernel(PlanArgs a) {
  __shared__ int cnt[MAX_E], base[MAX_E], wsum[2][32];
  const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5;
  cnt[tid] = 0;
  pdl_launch_dependents();
  pdl_wait();
  if (a.r.z)
    for (int row = warp; row < a.r.n; row += nt >> 5) route_row(a.r, row);
  __syncthreads();          // (orders the block's own ids too)
  uint32_t held[BATCH];
  // a place inside its expert for every pair
  auto places = [&](int p0) {
#pragma unroll
    for (int k = 0; k < BATCH; ++k) {
      if (p0 + k * nt >= a.pairs) break;
      held[k] = p0 + k * nt + tid < a.pairs ? (uint32_t)a.r.ids[p0 + k * nt + tid] : 0u;
    }
#pragma unroll
    for (int k = 0; k < BATCH; ++k) {
      if (p0 + k * nt >= a.pairs) break;
      if (p0 + k * nt + tid < a.pairs) held[k] = held[k] << 20 | (uint32_t)atomicAdd(&cnt[held[k]], 1);
    }
  };
  for (int p0 = 0; p0 < a.pairs; p0 += BATCH * nt) places(p0);
  __syncthreads();
  const int c = cnt[tid], t = (c + a.tile - 1) / a.tile;
  int sc = c, st = t;       // inclusive sums of pairs and of tiles over the experts
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int x = __shfl_up_sync(0xffffffffu, sc, o), y = __shfl_up_sync(0xffffffffu, st, o);
    if (lane >= o) { sc += x; st += y; }
  }
  if (lane == 31) { wsum[0][warp] = sc; wsum[1][warp] = st; }
  __syncthreads();
  for (int w = 0; w < warp; ++w) { sc += wsum[0][w]; st += wsum[1][w]; }
  for (int k = 0; k < t; ++k) reinterpret_cast<int4*>(a.tiles)[st - t + k] = make_int4(tid, sc - c + k * a.tile, min(a.tile, c - k * a.tile), 0);
  if (tid == nt - 1) *a.count = st;
  base[tid] = sc - c;
  cnt[tid] = 0;             // more pairs than the threads hold: they take their places again
  __syncthreads();
  for (int p0 = 0; p0 < a.pairs; p0 += BATCH * nt) {
    if (a.pairs > BATCH * nt) places(p0);
#pragma unroll
    for (int k = 0; k < BATCH; ++k) {
      if (p0 + k * nt >= a.pairs) break;
      if (p0 + k * nt + tid < a.pairs) a.order[base[held[k] >> 20] + (int)(held[k] & 0xfffffu)] = p0 + k * nt + tid;
    }
  }
}

// ---- tiles on CUDA cores ----------------------------------------------------------------------------------------------------
struct TileArgs {
  const void* x;            // first: [n, K] rows; down: [pairs, K] in plan order
  const void* w;            // [E, M, K], gated: [E, 2 M, K]
  void* out;                // first: [pairs, M] in plan order; down: [n, slots, M]
  const int *order, *tiles, *count;
  int M, K, top, slots, act, gated;      // act: 0 down, ACT_CLAMP (gated), or an ungated one
  float alpha, limit;
};
constexpr int TR = 32, TC = 64, TK = 16;

template <typename T>
__global__ void __launch_bounds__(256) moe_tile_kernel(TileArgs a) {
  __shared__ float xs[TK][TR + 1], ws[2][TK][TC + 1];
  pdl_launch_dependents();
  pdl_wait();
  if ((int)blockIdx.y >= *a.count) return;
  const int4 t = reinterpret_cast<const int4*>(a.tiles)[blockIdx.y];
  const int e = t.x, p0 = t.y, rows = t.z, c0 = blockIdx.x * TC, tid = threadIdx.x;
  const int tr = tid >> 4, tc = tid & 15;            // rows tr, tr + 16; columns tc + 16 i
  const int xr = tid >> 3, xk = (tid & 7) * 2;       // staged: row xr, two of its elements
  const int place = p0 + min(xr, rows - 1);
  const T* xp = (const T*)a.x + (size_t)(a.act ? a.order[place] / a.top : place) * a.K;
  const T* wp = (const T*)a.w + (size_t)e * (a.gated ? 2 : 1) * a.M * a.K;
  float acc[2][2][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += TK) {
#pragma unroll
    for (int i = 0; i < 2; ++i) xs[xk + i][xr] = k0 + xk + i < a.K ? to_f<T>(xp[k0 + xk + i]) : 0.f;
    for (int i = tid; i < (a.gated ? 2 : 1) * TC * TK; i += 256) {
      const int g = i / (TC * TK), c = (i / TK) % TC, k = i % TK;
      ws[g][k][c] = c0 + c < a.M && k0 + k < a.K ? to_f<T>(wp[((size_t)g * a.M + c0 + c) * a.K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      const float x0 = xs[k][tr], x1 = xs[k][tr + 16];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float w0 = ws[0][k][tc + 16 * i];
        acc[0][0][i] = fmaf(x0, w0, acc[0][0][i]);
        acc[0][1][i] = fmaf(x1, w0, acc[0][1][i]);
        if (a.gated) {
          const float w1 = ws[1][k][tc + 16 * i];
          acc[1][0][i] = fmaf(x0, w1, acc[1][0][i]);
          acc[1][1][i] = fmaf(x1, w1, acc[1][1][i]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = tr + 16 * r;
    if (row >= rows) continue;
    size_t o;
    if (a.act) o = (size_t)(p0 + row);
    else { const int pair = a.order[p0 + row]; o = (size_t)(pair / a.top) * a.slots + pair % a.top; }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = c0 + tc + 16 * i;
      if (c >= a.M) continue;
      const float f = acc[0][r][i];
      ((T*)a.out)[o * a.M + c] = from_f<T>(a.gated ? gate_clamp<T>(f, acc[1][r][i], a.alpha, a.limit) : a.act ? act_single<T>(f, a.act, a.alpha, a.limit) : f);
    }
  }
}

// ---- few rows -----------------------------------------------------------------------------------------------------------------
struct GemvArgs {
  RouteArgs r;                // r.z: the first product chooses the experts (and leaves them in r.ids and r.wts)
  const __nv_bfloat16* x;     // first: [n, K]; down: [pairs, K]
  const __nv_bfloat16* w;     // [E, M, K], gated: [E, 2 M, K]
  __nv_bfloat16* out;         // first: [pairs, M]; down: [n, slots, M]
  const __nv_bfloat16 *sx, *sw;     // the shared expert: first [n, SK], down [n, SK]; null: none
  __nv_bfloat16* sout;        // first: [n, SM]
  int pairs, n, M, K, SM, SK, top, slots, act, gated;      // act: 0 down, ACT_CLAMP (gated), or an ungated one
  float alpha, limit, slimit;
};
constexpr int GU = 4;         // 256-element steps in flight per weight row

__global__ void __launch_bounds__(256) moe_gemv_kernel(GemvArgs a) {
  extern __shared__ __align__(16) uint8_t raw[];
  __shared__ int chosen;
  __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(raw);
  pdl_launch_dependents();
  pdl_wait();
  const int job = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool sh = job >= a.pairs;
  if (a.r.z && !sh) {
    if (warp == 0) {
      int id;
      float w, sw;
      choose(a.r, a.r.z + (size_t)(job / a.top) * a.r.ld, id, w, sw);
      if (lane == job % a.top) chosen = id;
      if (blockIdx.x == 0 && job % a.top == 0) {
        float* o = a.r.wts + (size_t)(job / a.top) * a.slots;
        if (lane < a.top) { a.r.ids[job + lane] = id; o[lane] = w; }
        if (a.r.shared && lane == 0) o[a.top] = sw;
      }
    }
    __syncthreads();
  }
  const int expert = sh ? 0 : a.r.z ? chosen : a.r.ids[job];
  const int row = sh ? job - a.pairs : job / a.top, M = sh ? a.SM : a.M, K = sh ? a.SK : a.K, words = K / 8;
  const __nv_bfloat16* w = sh ? a.sw : a.w + (size_t)expert * (a.gated ? 2 : 1) * M * K;
  const __nv_bfloat16* x = a.act ? (sh ? a.sx : a.x) + (size_t)row * K : (sh ? a.sx + (size_t)row * K : a.x + (size_t)job * K);
  __nv_bfloat16* out = a.act ? (sh ? a.sout + (size_t)row * M : a.out + (size_t)job * M)
                               : a.out + ((size_t)row * a.slots + (sh ? a.top : job % a.top)) * M;
  const int outs = a.gated ? M : (M + 1) / 2, stride = gridDim.x * 8;
  uint4 c0[GU], c1[GU];
  auto fetch = [&](int o, int b) {
    const int r0 = a.gated ? o : 2 * o, r1 = a.gated ? o + M : 2 * o + 1;
    const uint4 *w0 = reinterpret_cast<const uint4*>(w + (size_t)r0 * K), *w1 = reinterpret_cast<const uint4*>(w + (size_t)r1 * K);
    const bool v = o < outs, v1 = v && (a.gated || r1 < M);
#pragma unroll
    for (int i = 0; i < GU; ++i) {
      const int k = (b * GU + i) * 32 + lane;
      c0[i] = v && k < words ? ldg_nc(w0 + k) : make_uint4(0u, 0u, 0u, 0u);
      c1[i] = v1 && k < words ? ldg_nc(w1 + k) : make_uint4(0u, 0u, 0u, 0u);
    }
  };
  int o = blockIdx.x * 8 + warp;
  fetch(o, 0);
  for (int i = threadIdx.x; i < words; i += 256) reinterpret_cast<uint4*>(xs)[i] = reinterpret_cast<const uint4*>(x)[i];
  __syncthreads();
  const int batches = (words + 32 * GU - 1) / (32 * GU);
  for (; o < outs; o += stride) {
    float s0 = 0.f, s1 = 0.f;
    for (int b = 0; b < batches; ++b) {
      uint4 d0[GU], d1[GU];
#pragma unroll
      for (int i = 0; i < GU; ++i) { d0[i] = c0[i]; d1[i] = c1[i]; }
      if (b + 1 < batches) fetch(o, b + 1);
      else fetch(o + stride, 0);
#pragma unroll
      for (int i = 0; i < GU; ++i) {
        const int k = (b * GU + i) * 32 + lane;
        if (k >= words) continue;
        const uint4 xv = reinterpret_cast<const uint4*>(xs)[k];
        const uint32_t xw[4] = {xv.x, xv.y, xv.z, xv.w}, p[4] = {d0[i].x, d0[i].y, d0[i].z, d0[i].w}, q[4] = {d1[i].x, d1[i].y, d1[i].z, d1[i].w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float x0 = __uint_as_float(xw[j] << 16), x1 = __uint_as_float(xw[j] & 0xffff0000u);
          s0 = fmaf(__uint_as_float(p[j] << 16), x0, s0);
          s0 = fmaf(__uint_as_float(p[j] & 0xffff0000u), x1, s0);
          s1 = fmaf(__uint_as_float(q[j] << 16), x0, s1);
          s1 = fmaf(__uint_as_float(q[j] & 0xffff0000u), x1, s1);
        }
      }
    }
    s0 = warp_sum(s0);
    s1 = warp_sum(s1);
    if (lane == 0) {
      if (a.gated) out[o] = __float2bfloat16_rn(gate_clamp<float>(s0, s1, a.alpha, sh ? a.slimit : a.limit));
      else {
        if (a.act) { s0 = act_single<float>(s0, a.act, a.alpha, a.limit); s1 = act_single<float>(s1, a.act, a.alpha, a.limit); }
        out[2 * o] = __float2bfloat16_rn(s0);
        if (2 * o + 1 < M) out[2 * o + 1] = __float2bfloat16_rn(s1);
      }
    }
  }
}

}  // namespace rmoe
}  // namespace sfb

using namespace sfb;
using namespace sfb::rmoe;

static bool route_ok(const RouteArgs& a) {
  return a.n >= 1 && a.E >= 1 && a.E <= MAX_E && a.top >= 1 && a.top <= MAX_TOP && a.top <= a.E &&
         (!a.corr || (a.groups >= 1 && a.groups <= MAX_GROUPS && a.E % a.groups == 0 && a.keep >= 1 && a.keep <= a.groups && a.top <= a.E / a.groups * a.keep));
}
// a first product's activation (0: down)
static bool act_ok(int act) { return act == 0 || act == ACT_CLAMP || act == ACT_RELU2 || act == ACT_XIELU; }

extern "C" {

// corr, groups, keep, scale: see RouteArgs
int sfb_rows_moe_route(const void* z, int64_t ld, void* ids, void* wts, int n, int E, int top, int shared, const void* corr, int groups, int keep, float scale,
                       cudaStream_t stream) {
  RouteArgs a{(const float*)z, ld, (int*)ids, (float*)wts, n, E, top, shared, (const float*)corr, groups, keep, scale};
  if (!route_ok(a)) return (int)cudaErrorInvalidValue;
  return (int)sfb_launch(moe_route_kernel, dim3((n + 7) / 8), dim3(256), 0, stream, a);
}

// tiles: 4 ints each, at most pairs / tile + min(E, pairs) of them.  z: the choice is made here (few rows), null: ids are there.
int sfb_rows_moe_plan(const void* z, int64_t ld, void* ids, void* wts, void* order, void* tiles, void* count, int n, int E, int top, int shared, int tile,
                      const void* corr, int groups, int keep, float scale, cudaStream_t stream) {
  RouteArgs r{(const float*)z, ld, (int*)ids, (float*)wts, n, E, top, shared, (const float*)corr, groups, keep, scale};
  if (!route_ok(r) || tile < 1 || (long long)n * top >= 1 << 20) return (int)cudaErrorInvalidValue;
  PlanArgs a{r, (int*)order, (int*)tiles, (int*)count, n * top, E, tile};
  return (int)sfb_launch(moe_plan_kernel, dim3(1), dim3(E > 256 || n * top > 2048 ? 1024 : 256), 0, stream, a);
}

// tiles of at most 32 pairs
int sfb_rows_moe_tile(const void* x, const void* w, void* out, const void* order, const void* tiles, const void* count, int max_tiles, int M, int K, int top,
                      int slots, int act, float alpha, float limit, int fp32, cudaStream_t stream) {
  if (!act_ok(act) || max_tiles < 1 || max_tiles > 65535 || M < 1 || K < 1) return (int)cudaErrorInvalidValue;
  TileArgs a{x, w, out, (const int*)order, (const int*)tiles, (const int*)count, M, K, top, slots, act, act == ACT_CLAMP, alpha, limit};
  const dim3 g((M + TC - 1) / TC, max_tiles), b(256);
  return (int)(fp32 ? sfb_launch(moe_tile_kernel<float>, g, b, 0, stream, a) : sfb_launch(moe_tile_kernel<__nv_bfloat16>, g, b, 0, stream, a));
}

// bf16, K and SK multiples of 8; z: the choice of E experts is made here (first product), null: ids are there
int sfb_rows_moe_gemv(const void* z, int64_t ld, int E, void* ids, void* wts, const void* corr, int groups, int keep, float scale, const void* x, const void* w, void* out,
                      const void* sx, const void* sw, void* sout, int pairs, int n, int M, int K, int SM, int SK, int top, int slots, int act, float alpha, float limit,
                      float slimit, cudaStream_t stream) {
  const int kmax = sw && SK > K ? SK : K, gated = act == ACT_CLAMP;
  if (n < 1 || pairs != n * top || pairs + n > 65535 || M < 1 || K < 8 || K % 8 || (sw && (SM < 1 || SK < 8 || SK % 8)) || kmax * 2 > 200 * 1024 || !act_ok(act))
    return (int)cudaErrorInvalidValue;
  RouteArgs r{(const float*)z, ld, (int*)ids, (float*)wts, n, E, top, slots - top, (const float*)corr, groups, keep, scale};
  if (z && (!act || slots < top || !route_ok(r))) return (int)cudaErrorInvalidValue;
  GemvArgs a{r, (const __nv_bfloat16*)x, (const __nv_bfloat16*)w, (__nv_bfloat16*)out, (const __nv_bfloat16*)sx, (const __nv_bfloat16*)sw,
             (__nv_bfloat16*)sout, pairs, n, M, K, SM, SK, top, slots, act, gated, alpha, limit, slimit};
  const int jobs = pairs + (sw ? n : 0), big = sw && SM > M ? SM : M, outs = gated ? big : (big + 1) / 2;
  int bx = (outs + 7) / 8, cap = (148 * 4 + jobs - 1) / jobs;
  if (bx > cap) bx = cap;
  static size_t granted = 40 * 1024;
  const size_t smem = (size_t)kmax * 2;
  if (smem > granted) {
    const cudaError_t e = cudaFuncSetAttribute(moe_gemv_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    granted = smem;
  }
  return (int)sfb_launch(moe_gemv_kernel, dim3(bx, jobs), dim3(256), smem, stream, a);
}

}  // extern "C"
