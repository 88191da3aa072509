// The matrix-state recurrence of k_rows_state.cu for long runs of rows, on tcgen05: S_t = a_t S_(t-1) + w_t k_t v_t^T, y_t = S_t^T q_t + D v_t.
//
// A run is cut into chunks of 128 rows.  With c_t the running sum of log a inside a chunk and S_0 the state at its start,
//
//   y_i = sum_{j <= i} exp(c_i - c_j) w_j (q_i . k_j) v_j + exp(c_i) S_0^T q_i + D v_i,
//   S_0 of the next chunk = exp(c_last) S_0 + sum_j exp(c_last - c_j) w_j k_j v_j^T
//
//   state_turn     rotated (and scaled) q and k as two bf16 terms each, where the recurrence turns them
//   chunk_sums     the sum in the second line of every (chunk, head):  K^T (weight V)
//   chunk_starts   S_0 of every chunk, element by element along the run, as two bf16 terms; the run's final state, 32-bit
//   chunk_out      the first line: scores Q K^T, weighted in registers, back through tensor memory for the product with V; Q S_0 beside it
//
// Inputs are bf16.  Everything else that enters a product is a 32-bit value taken as two bf16 terms (16 mantissa bits): weighted scores,
// weighted values, states, turned q and k.  Accumulators, decays, weights and states are 32-bit.  Every wait is bounded and reports
// through the status word; no cluster, no multicast.
#include "k_rows_state_tc.cuh"

namespace sfb {
namespace rst {

constexpr int HEADS = 8;         // most heads per block

struct Args {
  const int *c_row0, *c_rows;      // chunks
  const int *seg, *first;          // runs: segment, first chunk (one entry more than runs)
  const int *seg_src, *seg_dst;
  const __nv_bfloat16* dt;         // [n, dt_stride] raw step sizes or null
  int64_t dt_stride;
  const float *dt_bias, *a;        // [H]: A with dt, else the logarithm of the decay
  const float* D;                  // [H] or null
  float* S;                        // [slots, H, P, Np]
  float* sums;                     // [chunks, H, P, Np]
  float* dec;                      // [chunks, H] decay over the whole chunk
  float* rates;                    // [chunks, H, 2, 128] running sum of log2 a; the same less log2 of the weight; delta rule: see RATES
  __nv_bfloat16* starts;           // [2, chunks, H, P, Np]: upper terms, then lower terms; delta rule: [2, chunks, H, N, P]
  __nv_bfloat16* y;                // [n, H P]
  int H, G, N, P, Np, ns, terms;   // ns: 64-element slabs of a q / k row
  int q_col, k_col, v_col;         // first columns in the maps
  int q_lo, k_lo;                  // distance to the columns of the lower terms
  int chunks, hpc;                 // hpc: heads per block
  int wide;                        // outputs lie on 32-byte boundaries
  Status* status;
};

// One warp, one head: running sums of log2 a over the chunk's rows (a lane takes four), weights; past the end: decay 1, weight 0.  The
// numbers go to memory for chunk_out, the factors of the values (decay to the chunk's end times weight) to `wt`.
__device__ __forceinline__ void head_rates(const Args& a, int chunk, int h, int row0, int rows, float* wt) {
  const int lane = threadIdx.x & 31;
  const float ah = a.a[h] * LOG2E, bias = a.dt ? a.dt_bias[h] : 0.f;
  float z[4], w[4], c[4], t = 0.f;
#pragma unroll
  for (int k = 0; k < 4; ++k) z[k] = a.dt && lane * 4 + k < rows ? __bfloat162float(a.dt[(size_t)(row0 + lane * 4 + k) * a.dt_stride + h]) + bias : 0.f;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    w[k] = lane * 4 + k >= rows ? 0.f : a.dt ? log1pf(expf(-fabsf(z[k]))) + fmaxf(z[k], 0.f) : 1.f;
    t += ah * w[k];
    c[k] = t;
  }
  float s = t;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, s, o); if (lane >= o) s += v; }
  const float last = __shfl_sync(0xffffffffu, s, 31), before = s - t;
  float* out = a.rates + ((size_t)chunk * a.H + h) * 2 * L + lane * 4;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    c[k] += before;
    wt[lane * 4 + k] = ex2(last - c[k]) * w[k];
  }
  rows::store_v<float, 4>(out, c);
#pragma unroll
  for (int k = 0; k < 4; ++k) c[k] -= __log2f(w[k]);       // weight 0: infinity, and its exponential below 0
  rows::store_v<float, 4>(out + L, c);
  if (lane == 0) a.dec[(size_t)chunk * a.H + h] = ex2(last);
}

// grid (groups x parts of a group's heads, chunks): k stays in shared memory while the heads (and their tiles of 64 value dims) go by
template <int TERMS>
__global__ void __launch_bounds__(THREADS)
chunk_sums_kernel(const __grid_constant__ CUtensorMap mk, const __grid_constant__ CUtensorMap mv, Args a) {
  extern __shared__ __align__(1024) uint8_t sm[];
  const int nb = (a.ns + 1) / 2;                          // blocks of 128 state rows
  uint8_t* ks = sm;                                       // [terms][2 nb] slabs
  uint8_t* vh = ks + (size_t)TERMS * 2 * nb * SLAB;       // weighted values, upper terms (the copy lands here): two stages
  uint8_t* vl = vh + 2 * SLAB;                            // lower terms
  float* wts = reinterpret_cast<float*>(vl + SLAB);       // [hpc][L] factors of the values
  Ctl& C = *reinterpret_cast<Ctl*>(wts + a.hpc * L);
  setup(C, nb > 1 ? 256 : 128);
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.y, rep = a.H / a.G, parts = (rep + a.hpc - 1) / a.hpc, g = blockIdx.x / parts;
  const int h0 = g * rep + (blockIdx.x % parts) * a.hpc, nh = min(a.hpc, (g + 1) * rep - h0), row0 = a.c_row0[chunk], rows = a.c_rows[chunk];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pts = (a.P + 63) / 64, items = nh * pts;
  const bool issuer = __shfl_sync(0xffffffffu, warp, 0) == WORK / 32;  // uniform: the elected thread's operands stay in uniform registers
  volatile int* dead = &C.dead;
  auto fetch = [&](int it) {
    mbar_expect(&C.full[it & 1], SLAB);
    tma2d(vh + (it & 1) * SLAB, &mv, a.v_col + (h0 + it / pts) * a.P + 64 * (it % pts), row0, &C.full[it & 1]);
  };
  if (issuer && elect_one()) {
    mbar_expect(&C.full[2], TERMS * a.ns * SLAB);
    for (int t = 0; t < TERMS; ++t)
      for (int s = 0; s < a.ns; ++s) tma2d(ks + (size_t)(t * 2 * nb + s) * SLAB, &mk, a.k_col + t * a.k_lo + g * a.N + 64 * s, row0, &C.full[2]);
    fetch(0);
  }
  const uint32_t id = idesc(64, 1, 1), cols = 64 * nb;
  const int w4 = warp & 3, half = warp >> 2;
  auto store = [&](int it) {       // lane = state row: columns of the tile go out as runs of consecutive state rows
    const int h = h0 + it / pts, pt = it % pts;
    for (int b = 0; b < nb; ++b) {
      float f[32];
      ld32(C.tmem + (it & 1) * cols + b * 64 + half * 32 + ((uint32_t)(w4 * 32) << 16), f);
      wait_ld();
      const int n = b * 128 + w4 * 32 + lane;
      if (n < a.Np) {
        float* o = a.sums + (((size_t)chunk * a.H + h) * a.P + pt * 64 + half * 32) * a.Np + n;
        const int m = min(32, a.P - pt * 64 - half * 32);
        if (m == 32 && n < a.N) {
#pragma unroll
          for (int c = 0; c < 32; ++c) o[(size_t)c * a.Np] = f[c];
        } else {
#pragma unroll
          for (int c = 0; c < 32; ++c)
            if (c < m) o[(size_t)c * a.Np] = n < a.N ? f[c] : 0.f;
        }
      }
    }
    fence_before();
  };
  if (!issuer) {
    for (int x = warp; x < nh; x += WORK / 32) head_rates(a, chunk, h0 + x, row0, rows, wts + x * L);
  }
  wait_warp(&C.full[2], 0, dead, 2);
  for (int it = 0; it < items; ++it) {
    uint8_t* vs = vh + (it & 1) * SLAB;
    wait_warp(&C.full[it & 1], (it >> 1) & 1, dead, 3);
    if (it > 0) wait_warp(&C.done[0], (it - 1) & 1, dead, 4);               // the other stage and the lower terms are free
    __syncthreads();
    if (issuer) {
      if (it + 1 < items && elect_one()) fetch(it + 1);
    } else {
      const float* wt = wts + it / pts * L;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int u = tid + i * WORK;                                // a 16-byte unit; its row is u / 8
        const float wr = wt[u >> 3];
        float f[8];
        uint4 hv, lv;
        rows::load_v<__nv_bfloat16, 8>(reinterpret_cast<const __nv_bfloat16*>(vs) + u * 8, f);
#pragma unroll
        for (int k = 0; k < 8; ++k) f[k] *= wr;
        split2(f[0], f[1], hv.x, lv.x); split2(f[2], f[3], hv.y, lv.y); split2(f[4], f[5], hv.z, lv.z); split2(f[6], f[7], hv.w, lv.w);
        reinterpret_cast<uint4*>(vs)[u] = hv;
        reinterpret_cast<uint4*>(vl)[u] = lv;
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __syncthreads();
    if (issuer) {
      if (elect_one()) {
        fence_after();
        const uint64_t dh = desc(smem_u32(vs), SLAB), dl = desc(smem_u32(vl), SLAB);
        for (int b = 0; b < nb; ++b) {
          const uint32_t d = C.tmem + (it & 1) * cols + b * 64;
          const uint64_t k0 = desc(smem_u32(ks) + (2 * b) * SLAB, SLAB), k1 = desc(smem_u32(ks) + (2 * nb + 2 * b) * SLAB, SLAB);
#pragma unroll
          for (int t = 0; t < 8; ++t) {
            const uint64_t o = (uint64_t)t * (2048 >> 4);
            mma_ss(d, k0 + o, dh + o, id, t ? 1u : 0u);
            mma_ss(d, k0 + o, dl + o, id, 1u);
            if (TERMS > 1) mma_ss(d, k1 + o, dh + o, id, 1u);
          }
        }
        commit(&C.done[0]);
      }
      __syncwarp();
    } else if (it > 0) {
      fence_after();
      store(it - 1);                                                 // while the products run
    }
  }
  wait_warp(&C.done[0], (items - 1) & 1, dead, 5);
  fence_after();
  if (!issuer) store(items - 1);
  drain(C);
  teardown(C, nb > 1 ? 256 : 128, a.status, 69);
}

// grid (elements / 1024, runs): a thread follows four elements through the run's chunks
constexpr int AHEAD = 4;
__global__ void __launch_bounds__(256) chunk_starts_kernel(Args a) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t per = (size_t)a.H * a.P * a.Np, e = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4;
  if (e >= per) return;
  const int h = (int)(e / ((size_t)a.P * a.Np)), run = blockIdx.y, seg = a.seg[run], c0 = a.first[run], c1 = a.first[run + 1];
  const int src = a.seg_src[seg];
  float4 S = src >= 0 ? *reinterpret_cast<const float4*>(a.S + (size_t)src * per + e) : make_float4(0.f, 0.f, 0.f, 0.f);
  __nv_bfloat16 *hi = a.starts + e, *lo = a.starts + (size_t)a.chunks * per + e;
  float4 E[AHEAD];
  float d[AHEAD];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i)
    if (c0 + i < c1) { E[i] = *reinterpret_cast<const float4*>(a.sums + (size_t)(c0 + i) * per + e); d[i] = a.dec[(size_t)(c0 + i) * a.H + h]; }
  for (int c = c0; c < c1; c += AHEAD) {
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (c + i >= c1) break;
      const float4 x = E[i];
      const float dd = d[i];
      if (c + i + AHEAD < c1) {
        E[i] = *reinterpret_cast<const float4*>(a.sums + (size_t)(c + i + AHEAD) * per + e);
        d[i] = a.dec[(size_t)(c + i + AHEAD) * a.H + h];
      }
      uint2 u, v;
      split2(S.x, S.y, u.x, v.x);
      split2(S.z, S.w, u.y, v.y);
      *reinterpret_cast<uint2*>(hi + (size_t)(c + i) * per) = u;
      *reinterpret_cast<uint2*>(lo + (size_t)(c + i) * per) = v;
      S.x = fmaf(dd, S.x, x.x); S.y = fmaf(dd, S.y, x.y); S.z = fmaf(dd, S.z, x.z); S.w = fmaf(dd, S.w, x.w);
    }
  }
  *reinterpret_cast<float4*>(a.S + (size_t)a.seg_dst[seg] * per + e) = S;
}

// grid as chunk_sums: q and k stay in shared memory while the heads go by; the scores are computed again for every head (their tensor
// memory is where the weighted scores go).  DELTA: one head per block; the values are u (two terms), the state lies with its N rows one after
// another and takes k's place in shared memory once the scores are done; rows are scaled at the end.
template <int NS, int TERMS, bool DELTA>
__global__ void __launch_bounds__(THREADS, 2)
chunk_out_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mk, const __grid_constant__ CUtensorMap mv,
                 const __grid_constant__ CUtensorMap ms, Args a) {
  extern __shared__ __align__(1024) uint8_t sm[];
  uint8_t* qs = sm;                                      // [terms][ns] slabs
  uint8_t* ks = qs + (size_t)TERMS * NS * SLAB;
  uint8_t* vs = ks + (size_t)TERMS * NS * SLAB;      // one slab (DELTA: two)
  uint8_t* ss = DELTA ? ks : vs + SLAB;                  // start state, [2][ns] slabs of 64 rows
  Ctl& C = *reinterpret_cast<Ctl*>(DELTA ? vs + 2 * SLAB : ss + (size_t)2 * NS * HSLAB);
  constexpr int RW = DELTA ? RATES : 2;
  setup(C, 256);
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.y, rep = a.H / a.G, parts = (rep + a.hpc - 1) / a.hpc, g = blockIdx.x / parts;
  const int h0 = g * rep + (blockIdx.x % parts) * a.hpc, nh = min(a.hpc, (g + 1) * rep - h0), row0 = a.c_row0[chunk], rows = a.c_rows[chunk];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pts = (a.P + 63) / 64, items = nh * pts, w4 = warp & 3, half = warp >> 2;
  const bool issuer = __shfl_sync(0xffffffffu, warp, 0) == WORK / 32;  // uniform: the elected thread's operands stay in uniform registers
  volatile int* dead = &C.dead;
  const uint32_t tp = C.tmem, ta = tp + 128, tb = tp + 192, lanes = (uint32_t)(w4 * 32) << 16;
  auto tile = [&](int it) {                              // values and start state of a tile of 64 value dims
    const int h = h0 + it / pts, pt = it % pts;
    mbar_expect(&C.full[0], (DELTA ? 2 : 1) * SLAB + 2 * NS * HSLAB);
    if constexpr (DELTA) {
      for (int t = 0; t < 2; ++t) tma2d(vs + t * SLAB, &mv, 64 * pt, ((t * a.chunks + chunk) * a.H + h) * L, &C.full[0]);
    } else {
      tma2d(vs, &mv, a.v_col + h * a.P + 64 * pt, row0, &C.full[0]);
    }
  };
  auto state = [&](int it) {
    const int h = h0 + it / pts, pt = it % pts, rows1 = DELTA ? a.N : a.P, y = (chunk * a.H + h) * rows1 + (DELTA ? 0 : 64 * pt);
    for (int t = 0; t < 2; ++t)
      for (int s = 0; s < NS; ++s)
        tma2d(ss + (size_t)(t * NS + s) * HSLAB, &ms, DELTA ? 64 * pt : 64 * s, t * a.chunks * a.H * rows1 + y + (DELTA ? 64 * s : 0), &C.full[0]);
  };
  const int kst = a.N / 16;
  const uint64_t lo = (uint64_t)NS * (SLAB >> 4), dq = desc(smem_u32(qs), 16), dk = desc(smem_u32(ks), 16);
  auto scores = [&]() {
    const uint32_t id = idesc(128, 0, 0);
#pragma unroll
    for (int t = 0; t < 4 * NS; ++t) {
      if (t >= kst) break;
      const uint64_t o = (uint64_t)(t >> 2) * (SLAB >> 4) + (t & 3) * 2;
      mma_ss(tp, dq + o, dk + o, id, t ? 1u : 0u);
      if (TERMS > 1) {
        mma_ss(tp, dq + o, dk + lo + o, id, 1u);
        mma_ss(tp, dq + lo + o, dk + o, id, 1u);
      }
    }
    commit(&C.done[1]);
  };
  if (issuer && elect_one()) {
    mbar_expect(&C.full[2], 2 * TERMS * NS * SLAB);
    for (int t = 0; t < TERMS; ++t)
      for (int s = 0; s < NS; ++s) {
        tma2d(qs + (size_t)(t * NS + s) * SLAB, &mq, a.q_col + t * a.q_lo + g * a.N + 64 * s, row0, &C.full[2]);
        tma2d(ks + (size_t)(t * NS + s) * SLAB, &mk, a.k_col + t * a.k_lo + g * a.N + 64 * s, row0, &C.full[2]);
      }
    tile(0);
    if (!DELTA) state(0);
  }
  const int i = w4 * 32 + lane;
  const float* rates = a.rates + ((size_t)chunk * a.H + h0) * RW * L;
  wait_warp(&C.full[2], 0, dead, 6);
  if (issuer) {
    // after every barrier of the workers below comes what it makes possible
    if (elect_one()) scores();
    __syncwarp();
    if constexpr (DELTA) {
      wait_warp(&C.done[1], 0, dead, 11);
      if (elect_one()) state(0);
      __syncwarp();
    }
    for (int it = 0; it < items; ++it) {
      const bool next = it + 1 < items, head_ends = (it + 1) % pts == 0;
      wait_warp(&C.full[0], it & 1, dead, 7);
      __syncthreads();
      if (elect_one()) {
        fence_after();
        const uint32_t ia = idesc(64, 0, 1), ib = idesc(64, 0, DELTA);
        const uint64_t dv = desc(smem_u32(vs), SLAB), ds = desc(smem_u32(ss), DELTA ? SLAB : 16), sl = (uint64_t)NS * (HSLAB >> 4);
        // the two sums by turns: products on one accumulator follow each other slowly at this size
        auto weighted = [&](int t) {                     // eight steps of 16 rows with the upper terms, then with the lower ones
          const int lower = t >> 3 & 1, vl = t >> 4;     // of the weights, of the values
          mma_ts(ta, tp + ((t & 7) >> 1) * 32 + (t & 1) * 8 + lower * 16, dv + (uint64_t)vl * (SLAB >> 4) + (uint64_t)(t & 7) * (2048 >> 4), ia, t ? 1u : 0u);
        };
        constexpr int PER = 16 / (4 * NS);               // weighted products for every step of the other sum
#pragma unroll
        for (int t = 0; t < 4 * NS; ++t) {
          const uint64_t o = (uint64_t)(t >> 2) * (SLAB >> 4) + (t & 3) * 2, os = DELTA ? (uint64_t)t * (2048 >> 4) : (uint64_t)(t >> 2) * (HSLAB >> 4) + (t & 3) * 2;
          if (t < kst) mma_ss(tb, dq + o, ds + os, ib, t ? 1u : 0u);
          weighted(PER * t);
          if (t < kst) mma_ss(tb, dq + o, ds + sl + os, ib, 1u);
          if (PER > 1) weighted(PER * t + 1);
          if (TERMS > 1 && t < kst) mma_ss(tb, dq + lo + o, ds + os, ib, 1u);
#pragma unroll
          for (int u = 2; u < PER; ++u) weighted(PER * t + u);
        }
#pragma unroll
        for (int t = PER * 4 * NS; t < (DELTA ? 24 : 16); ++t) weighted(t);
        commit(&C.done[0]);
      }
      __syncwarp();
      wait_warp(&C.done[0], it & 1, dead, 8);
      if (next && elect_one()) {
        fence_after();
        tile(it + 1);
        state(it + 1);
        if (!DELTA && head_ends) scores();                         // of the next head
      }
      __syncwarp();
    }
  } else {
    float next_ci = rates[i], ei = 0.f;
    const float scale = DELTA ? rates[2 * L + i] : 1.f;
    for (int it = 0; it < items; ++it) {
      const int hi = it / pts, h = h0 + hi, pt = it % pts;
      if (pt == 0) {
        const float ci = next_ci, D = a.D ? a.D[h] : 0.f;
        const float* cs = rates + (size_t)hi * RW * L + L;
        ei = ex2(ci);
        if (hi + 1 < nh) next_ci = rates[(size_t)(hi + 1) * RW * L + i];
        wait_warp(&C.done[1], hi & 1, dead, 9);
        fence_after();
        // Blocks of 32 columns: before the warp's diagonal block all are visible, after it none.  A thread's weights take the place of the
        // scores it has read: upper terms in the block's first 16 columns, lower terms in the others.
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          const int blk = 2 * half + b;
          uint32_t hv[16], lv[16];
          if (blk <= w4) {
            float s[32];
            ld32(tp + blk * 32 + lanes, s);
            float4 cj[8];
#pragma unroll
            for (int q = 0; q < 8; ++q) cj[q] = *reinterpret_cast<const float4*>(cs + blk * 32 + 4 * q);
            wait_ld();
#pragma unroll
            for (int q = 0; q < 8; ++q) {
              const float c4[4] = {cj[q].x, cj[q].y, cj[q].z, cj[q].w};
#pragma unroll
              for (int k = 0; k < 4; ++k) s[4 * q + k] *= ex2(ci - c4[k]);
            }
            if (blk == w4) {
#pragma unroll
              for (int k = 0; k < 32; ++k) {
                if (k > lane) s[k] = 0.f;
                if (k == lane) s[k] += D;                // D v_i
              }
            }
#pragma unroll
            for (int q = 0; q < 16; ++q) split2(s[2 * q], s[2 * q + 1], hv[q], lv[q]);
          } else {
#pragma unroll
            for (int q = 0; q < 16; ++q) hv[q] = lv[q] = 0u;
          }
          st16(tp + blk * 32 + lanes, hv);
          st16(tp + blk * 32 + 16 + lanes, lv);
        }
        wait_st();
        fence_before();
      }
      __syncthreads();                                   // weights are in place, accumulators have been read
      wait_warp(&C.done[0], it & 1, dead, 10);
      fence_after();
      __nv_bfloat16* o = a.y + ((size_t)(row0 + i) * a.H + h) * a.P + pt * 64 + half * 32;
      const int cols = min(32, a.P - pt * 64 - half * 32);
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        float x[16], z[16];
        ld16(ta + half * 32 + 16 * b + lanes, x);
        ld16(tb + half * 32 + 16 * b + lanes, z);
        wait_ld();
        if (i < rows) {
#pragma unroll
          for (int k = 0; k < 16; ++k) x[k] = fmaf(ei, z[k], x[k]) * scale;
          if (a.wide && 16 * b + 16 <= cols) store32(o + 16 * b, x);
          else {
#pragma unroll
            for (int u = 0; u < 2; ++u)
              if (16 * b + 8 * u < cols) rows::store_v<__nv_bfloat16, 8>(o + 16 * b + 8 * u, x + 8 * u);      // P is a multiple of eight
          }
        }
      }
      fence_before();
    }
  }
  drain(C);
  teardown(C, 256, a.status, 70);
}

// q and k of a row, turned by its position, k scaled: out [n][q hi | q lo | k hi | k lo], each [H, N]
struct TurnArgs {
  const __nv_bfloat16 *q, *k;
  int64_t q_stride, k_stride;
  const float2* rot;
  const int* row_pos;
  __nv_bfloat16* out;
  int n, H, N, dims;
  float k_scale;
};
__global__ void __launch_bounds__(256) state_turn_kernel(TurnArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, half = a.dims >> 1, HN = a.H * a.N, N2 = a.N >> 1;
  const float2* cs = a.rot + (size_t)a.row_pos[row] * half;
  const __nv_bfloat16 *q = a.q + (size_t)row * a.q_stride, *k = a.k + (size_t)row * a.k_stride;
  __nv_bfloat16* o = a.out + (size_t)row * 4 * HN;
  // a thread takes two neighbouring dims of a head (half is even or the pair is handled element by element below)
  for (int x = blockIdx.y * 256 + threadIdx.x; x < a.H * N2; x += gridDim.y * 256) {
    const int h = x / N2, d = (x - h * N2) * 2;
    float qf[2], kf[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int n = d + e, at = h * a.N + n;
      qf[e] = __bfloat162float(q[at]);
      kf[e] = __bfloat162float(k[at]);
      if (n < a.dims) {
        const int i = n < half ? n : n - half, p = n < half ? at + half : at - half;
        const float2 t = cs[i];
        const float s = n < half ? -t.y : t.y;
        qf[e] = qf[e] * t.x + __bfloat162float(q[p]) * s;
        kf[e] = kf[e] * t.x + __bfloat162float(k[p]) * s;
      }
      kf[e] *= a.k_scale;
    }
    uint32_t qh, ql, kh, kl;
    split2(qf[0], qf[1], qh, ql);
    split2(kf[0], kf[1], kh, kl);
    uint32_t* w = reinterpret_cast<uint32_t*>(o + h * a.N + d);
    w[0] = qh; w[HN / 2] = ql; w[HN] = kh; w[HN + HN / 2] = kl;
  }
}

static size_t sums_smem(const Args& a) { return (size_t)(a.terms * 2 * ((a.ns + 1) / 2) + 3) * SLAB + a.hpc * L * sizeof(float) + sizeof(Ctl); }
static size_t out_smem(const Args& a, bool delta) { return (size_t)(2 * a.terms * a.ns + (delta ? 2 : 1)) * SLAB + (size_t)(delta ? 0 : 2 * a.ns * HSLAB) + sizeof(Ctl); }

template <int TERMS>
static cudaError_t launch_sums(const CUtensorMap* k, const CUtensorMap* v, const Args& a, dim3 grid, cudaStream_t st) {
  static size_t granted = 0;
  const size_t smem = sums_smem(a);
  const cudaError_t e = grant(chunk_sums_kernel<TERMS>, smem, granted);
  return e != cudaSuccess ? e : sfb_launch(chunk_sums_kernel<TERMS>, grid, dim3(THREADS), smem, st, *k, *v, a);
}
template <int NS, int TERMS, bool DELTA = false>
static cudaError_t launch_out(const CUtensorMap* q, const CUtensorMap* k, const CUtensorMap* v, const CUtensorMap* s, const Args& a, dim3 grid, cudaStream_t st) {
  static size_t granted = 0;
  const size_t smem = out_smem(a, DELTA);
  const cudaError_t e = grant(chunk_out_kernel<NS, TERMS, DELTA>, smem, granted);
  return e != cudaSuccess ? e : sfb_launch(chunk_out_kernel<NS, TERMS, DELTA>, grid, dim3(THREADS), smem, st, *q, *k, *v, *s, a);
}

}  // namespace rst
}  // namespace sfb

using namespace sfb;
using namespace sfb::rst;

extern "C" {

int sfb_rows_state_turn(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* rot, const int* row_pos, void* out, int n, int H, int N,
                        int dims, float k_scale, cudaStream_t stream) {
  if (n < 1 || N < 2 || N % 2 || dims % 2 || dims > N) return (int)cudaErrorInvalidValue;
  TurnArgs a{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, q_stride, k_stride, (const float2*)rot, row_pos, (__nv_bfloat16*)out, n, H, N, dims, k_scale};
  return (int)sfb_launch(state_turn_kernel, dim3(n, (H * N / 2 + 1023) / 1024), dim3(256), 0, stream, a);
}

// mq, mk: rows of q / k terms, box 128 rows; mv: values, box 128 rows; ms: starts seen as [2 chunks H P, Np], box 64 rows.  N: a multiple of
// 16 up to 256 (128 with two terms); P: a multiple of 8; first columns multiples of 8.
int sfb_rows_state_tc(const void* mq, const void* mk, const void* mv, const void* ms, const int* c_row0, const int* c_rows, const int* seg, const int* first,
                      const int* seg_src, const int* seg_dst, const void* dt, int64_t dt_stride, const void* dt_bias, const void* la, const void* D, void* S,
                      void* sums, void* dec, void* rates, void* starts, void* y, int runs, int chunks, int H, int G, int N, int P, int Np, int terms, int q_col, int k_col,
                      int v_col, int q_lo, int k_lo, void* status, cudaStream_t stream) {
  const int ns = (N + 63) / 64;
  if (runs < 1 || runs > 65535 || chunks < 1 || chunks > 65535 || G < 1 || H % G || N % 16 || P % 8 || ns > (terms > 1 ? 2 : 4) || Np < N || Np % 32 ||
      terms < 1 || terms > 2 || (q_col | k_col | v_col | q_lo | k_lo | N) % 8)
    return (int)cudaErrorInvalidValue;
  Args a{c_row0, c_rows, seg, first, seg_src, seg_dst, (const __nv_bfloat16*)dt, dt_stride, (const float*)dt_bias, (const float*)la, (const float*)D, (float*)S,
         (float*)sums, (float*)dec, (float*)rates, (__nv_bfloat16*)starts, (__nv_bfloat16*)y, H, G, N, P, Np, ns, terms, q_col, k_col, v_col, q_lo, k_lo, chunks, 1, (H * P) % 16 == 0 && P % 16 == 0 && (uintptr_t)y % 32 == 0,
         (Status*)status};
  const int rep = H / G;
  a.hpc = rep < HEADS ? rep : HEADS;         // fewer heads per block where that leaves SMs empty
  while (a.hpc > 1 && (long long)G * ((rep + a.hpc - 1) / a.hpc) * chunks < 148) a.hpc = (a.hpc + 1) / 2;
  const int blocks = G * ((rep + a.hpc - 1) / a.hpc);
  const CUtensorMap *q = (const CUtensorMap*)mq, *k = (const CUtensorMap*)mk, *v = (const CUtensorMap*)mv, *s = (const CUtensorMap*)ms;
  const dim3 grid(blocks, chunks);
  cudaError_t rc = terms > 1 ? launch_sums<2>(k, v, a, grid, stream) : launch_sums<1>(k, v, a, grid, stream);
  if (rc != cudaSuccess) return (int)rc;
  const size_t per = (size_t)H * P * Np;
  rc = sfb_launch(chunk_starts_kernel, dim3((unsigned)((per / 4 + 255) / 256), runs), dim3(256), 0, stream, a);
  if (rc != cudaSuccess) return (int)rc;
  if (terms > 1) return (int)(ns == 1 ? launch_out<1, 2>(q, k, v, s, a, grid, stream) : launch_out<2, 2>(q, k, v, s, a, grid, stream));
  switch (ns) {
    case 1: return (int)launch_out<1, 1>(q, k, v, s, a, grid, stream);
    case 2: return (int)launch_out<2, 1>(q, k, v, s, a, grid, stream);
    case 3: return (int)launch_out<3, 1>(q, k, v, s, a, grid, stream);
    default: return (int)launch_out<4, 1>(q, k, v, s, a, grid, stream);
  }
}

// The outputs of the delta rule, after sfb_rows_delta_tc: mq, mk: rows of q / k, box 128 rows; mu: u seen as [2 chunks H 128, P], box 128
// rows; ms: starts seen as [2 chunks H N, P], box 64 rows.  N: a multiple of 16 up to 128; P: a multiple of 8.
int sfb_rows_delta_out(const void* mq, const void* mk, const void* mu, const void* ms, const int* c_row0, const int* c_rows, void* rates, void* starts, void* y,
                       int chunks, int H, int G, int N, int P, int q_col, int k_col, void* status, cudaStream_t stream) {
  if (chunks < 1 || chunks > 65535 || G < 1 || H % G || N % 16 || N < 16 || N > 128 || P % 8 || P < 8 || (q_col | k_col) % 8) return (int)cudaErrorInvalidValue;
  Args a{};
  a.c_row0 = c_row0; a.c_rows = c_rows; a.rates = (float*)rates; a.starts = (__nv_bfloat16*)starts; a.y = (__nv_bfloat16*)y; a.H = H; a.G = G; a.N = N; a.P = P;
  a.ns = (N + 63) / 64; a.terms = 1; a.q_col = q_col; a.k_col = k_col; a.chunks = chunks; a.hpc = 1;
  a.wide = (H * P) % 16 == 0 && P % 16 == 0 && (uintptr_t)y % 32 == 0; a.status = (Status*)status;
  const dim3 grid(H, chunks);
  const CUtensorMap *q = (const CUtensorMap*)mq, *k = (const CUtensorMap*)mk, *u = (const CUtensorMap*)mu, *s = (const CUtensorMap*)ms;
  return (int)(a.ns == 1 ? launch_out<1, 1, true>(q, k, u, s, a, grid, stream) : launch_out<2, 1, true>(q, k, u, s, a, grid, stream));
}

}  // extern "C"
