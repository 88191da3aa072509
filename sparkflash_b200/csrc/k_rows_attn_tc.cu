// Softmax attention over the paged cache for long runs of rows, on tcgen05: score = (q . k) * scale - bias[head][distance],
// causal, the last `window` positions, bf16 queries / keys / values, 32-bit scores, softmax and accumulators.  Optionally
// cap * tanh(score / cap) (no bias then), a sink per head whose exponential is in the softmax's denominator only, and a
// sigmoid gate on the output.
//
// One CTA: 256 consecutive query rows of one segment (two halves of 128) x one head.  Key tiles of one cache page (64 positions)
// stream through shared memory by TMA: a (page, head) block is contiguous, so 64 dims of a tile are one box copy.
//
//   warps 0-3, 4-7   softmax of half 0 / half 1: one thread per query row (no exchange between threads)
//   warps 8, 10      issue the MMAs of half 0 / half 1:   S = Q K^T (shared x shared),   O += P V (P from tensor memory, V MN-major)
//   warp 9           TMA: the queries once, key and value tiles through a ring of stages
//   warp 11          stages the tile's window of the bias row (319 distances, four copies shifted by one element each, so that a
//                    thread reads its row's values, one distance down per key, as aligned 16-byte words without bank
//                    conflicts)
//
// Tensor memory: S0, S1 (64 columns each), P0, P1 (64 columns each), O0, O1 (128 each).  S and P are separate, so the next tile's
// scores are computed while this tile's are exponentiated.  The softmax weights stay 32-bit up to the product, which takes them as
// two bf16 terms (hi = the upper half of the float in columns 0..31, lo = the remainder in 32..63): P V sees 16 mantissa bits.
// The output accumulator is rescaled only when a row's maximum grew by more than 2^8.
//
// Keys come from the page pool through the page table, or (`offs`) from rows that were multiplied out for this step: page p of a
// tile's lane is then page p + offs[tile], heads k_head rows apart.  A key may have a second part that all heads share (template RS:
// its own map, one 64-element slab), matched by the last columns of the head's query; there is no bias then.  Template MODE: what
// happens to a scaled score (nothing, the bias, the cap).
//
// No cluster, no multicast; every wait is bounded and reports through the status word.
#include "k_rows_tc.cuh"

namespace sfb {
namespace rtc {
using namespace tc;

constexpr int THREADS = 384, ROWS = 256, HALF = 128, KT = 64, QSLAB = HALF * 128, SLAB = KT * 128, BST = 4;
constexpr int PLAIN = 0, BIAS = 1, CAP = 2;
constexpr int BW = 328;                       // bias copy stride: 319 values, = 8 mod 32 banks

struct Args {
  const int* tiles;          // (row0, rows) pairs
  const int* table;
  const int *row_lane, *row_pos;
  const int* offs;           // page offset of every tile, or null: through the table
  const float* bias;         // [H, bias_len] or null
  int64_t bias_len;
  const float* sink;         // [H] or null
  float cap;
  __nv_bfloat16* out;        // [n, H vdim]
  const __nv_bfloat16* gate; // [n, gate_row]: outputs are multiplied by its sigmoid; or null
  int64_t gate_row;
  int max_pages, n_pages, H, G, dim, vdim, rot;    // n_pages: of the pool, or of the rows multiplied out
  int k_page, k_head;        // rows between the pages and between the heads of the keys and values
  int window;
  float scale;
  Status* status;
};

// tanh for |x| <= 1/2: the Taylor polynomial to x^13 (the next term is below 2^-24)
__device__ __forceinline__ float2 tanh_small2(float2 x) {
  const float2 t = fma2(x, x, make_float2(0.f, 0.f));
  auto c = [](float v) { return make_float2(v, v); };
  float2 p = fma2(t, c(21844.f / 6081075.f), c(-1382.f / 155925.f));
  p = fma2(p, t, c(62.f / 2835.f));
  p = fma2(p, t, c(-17.f / 315.f));
  p = fma2(p, t, c(2.f / 15.f));
  p = fma2(p, t, c(-1.f / 3.f));
  return fma2(fma2(p, t, c(0.f)), x, x);
}
__device__ __forceinline__ float tanh_any(float x) {
  const float e = ex2(-2.f * LOG2E * fabsf(x));
  return copysignf(__fdividef(1.f - e, 1.f + e), x);
}

template <int DS, int VS, int RS, int MODE>    // 64-element slabs of a query / key row, of a value row, and of the shared key part
struct Smem {
  static constexpr int ST = RS ? 3 : 4, QS = DS + RS;
  alignas(1024) uint8_t q[2 * QS * QSLAB];
  alignas(1024) uint8_t k[ST * QS * SLAB];
  alignas(1024) uint8_t v[ST * VS * SLAB];
  alignas(16) float bias[MODE == BIAS ? BST * 4 * BW : 4];
  alignas(8) uint64_t q_full, k_full[ST], k_empty[ST], v_full[ST], v_empty[ST], s_full[2], s_free[2], p_full[2], pv_done[2], b_full[BST], b_empty[BST];
  uint32_t tmem;
  int dead;
};

template <int DS, int VS, int RS, int MODE>
__global__ void __launch_bounds__(THREADS, 1)
attn_run_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mk, const __grid_constant__ CUtensorMap mv,
                const __grid_constant__ CUtensorMap mr, Args a) {
  extern __shared__ uint8_t raw[];
  using SM = Smem<DS, VS, RS, MODE>;
  constexpr int ST = SM::ST, QS = SM::QS;
  SM& S = *reinterpret_cast<SM*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~(uintptr_t)1023);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  volatile int* dead = &S.dead;
  if (tid == 0) {
    S.dead = 0;
    mbar_init(&S.q_full, 1);
    for (int i = 0; i < ST; ++i) { mbar_init(&S.k_full[i], 1); mbar_init(&S.k_empty[i], 2); mbar_init(&S.v_full[i], 1); mbar_init(&S.v_empty[i], 2); }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&S.s_full[i], 1); mbar_init(&S.s_free[i], HALF); mbar_init(&S.p_full[i], HALF); mbar_init(&S.pv_done[i], 1);
    }
    for (int i = 0; i < BST; ++i) { mbar_init(&S.b_full[i], 32); mbar_init(&S.b_empty[i], ROWS); }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 8) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], 512;" ::"r"(smem_u32(&S.tmem)) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_launch_dependents();
  fence_before();
  __syncthreads();
  fence_after();
  pdl_wait();
  const uint32_t tmem = S.tmem;
  const int h = blockIdx.x, g = h / (a.H / a.G);
  const int row0 = a.tiles[2 * blockIdx.y], rows = a.tiles[2 * blockIdx.y + 1];
  const int pos0 = a.row_pos[row0];
  // key tiles of each half: up to the position of its last row that exists (a half without rows has none)
  const int j0 = max(0, pos0 - a.window + 1) / KT;           // tiles before the first row's window are not visited
  const int n0 = (pos0 + min(rows, HALF) - 1) / KT + 1 - j0;
  const int n1 = rows > HALF ? (pos0 + rows - 1) / KT + 1 - j0 : 0;
  const int nt = max(n0, n1);
  const int* tab = a.offs ? nullptr : a.table + (size_t)a.row_lane[row0] * a.max_pages + j0;
  const int off = a.offs ? a.offs[blockIdx.y] + j0 : 0;

  if (warp == 9) {
    if (elect_one()) {
      mbar_expect(&S.q_full, 2 * QS * QSLAB);
      for (int w = 0; w < 2; ++w)
        for (int s = 0; s < QS; ++s)
          tma2d(S.q + (w * QS + s) * QSLAB, &mq, h * (a.dim + a.rot) + (s < DS ? 64 * s : a.dim), row0 + w * HALF, &S.q_full);
      int issued = 0;
      for (int j = 0; j < nt; ++j) {
        const int st = j % ST, ph = (j / ST) & 1;
        int page = a.offs ? off + j : tab[j];
        if (page < 0 || page >= a.n_pages) { status_set(a.status, ST_BOUNDS, 63, page, a.n_pages); page = 0; }
        const int y = page * a.k_page + g * a.k_head;
        if (!mbar_wait(&S.k_empty[st], ph ^ 1, dead)) break;
        mbar_expect(&S.k_full[st], QS * SLAB);
        for (int s = 0; s < DS; ++s) tma2d(S.k + (st * QS + s) * SLAB, &mk, 64 * s, y, &S.k_full[st]);
        if constexpr (RS > 0) tma2d(S.k + (st * QS + DS) * SLAB, &mr, 0, page * KT, &S.k_full[st]);
        issued = 2 * j + 1;
        if (!mbar_wait(&S.v_empty[st], ph ^ 1, dead)) break;
        mbar_expect(&S.v_full[st], VS * SLAB);
        for (int s = 0; s < VS; ++s) tma2d(S.v + (st * VS + s) * SLAB, &mv, 64 * s, y, &S.v_full[st]);
        issued = 2 * j + 2;
      }
      if (*dead) {               // nobody may have waited for the copies in flight: do so, with a limit, before the CTA ends
        for (int c = max(0, issued - 2 * ST); c < issued; ++c) {
          const int j = c >> 1;
          uint64_t* b = (c & 1) ? &S.v_full[j % ST] : &S.k_full[j % ST];
          for (int i = 0; i < 100000 && !mbar_try(b, (j / ST) & 1); ++i) __nanosleep(64);
        }
        for (int i = 0; i < 100000 && !mbar_try(&S.q_full, 0); ++i) __nanosleep(64);
      }
    }
  } else if (warp == 8 || warp == 10) {
    if (elect_one()) {
      const int w = warp == 10, nw = w ? n1 : n0;
      const int ks = (a.dim + 15) / 16, rs = (a.rot + 15) / 16, nv = (a.vdim + 15) / 16 * 16;
      const uint32_t id_s = idesc(KT, 0, 0), id_o = idesc(nv, 0, 1);
      const uint32_t ts = tmem + w * 64, tp = tmem + 128 + w * 64, to = tmem + 256 + w * 128;
      const uint32_t vb = smem_u32(S.v);
      const uint64_t dq = desc(smem_u32(S.q) + w * QS * QSLAB, 16), dk = desc(smem_u32(S.k), 16), dv = desc(vb, SLAB);
      auto scores = [&](int j) {          // descriptors step in units of 16 bytes
        const uint64_t kd = dk + (uint64_t)((j % ST) * QS * (SLAB >> 4));
#pragma unroll
        for (int t = 0; t < QS * 4; ++t)
          if (t < DS * 4 ? t < ks : t - DS * 4 < rs) mma_ss(ts, dq + (t >> 2) * (QSLAB >> 4) + (t & 3) * 2, kd + (t >> 2) * (SLAB >> 4) + (t & 3) * 2, id_s, t ? 1u : 0u);
        commit(&S.s_full[w]);
        commit(&S.k_empty[j % ST]);
      };
      bool ok = mbar_wait(&S.q_full, 0, dead);
      for (int j = 0; ok && j < nt; ++j) {
        const int st = j % ST, ph = (j / ST) & 1;
        if (j == 0 && nw > 0) {
          if (!(ok = mbar_wait(&S.k_full[0], 0, dead))) break;
          fence_after();
          scores(0);
        }
        if (j + 1 < nw) {                 // the next tile's scores as soon as this tile's have been read
          ok = mbar_wait(&S.k_full[(j + 1) % ST], ((j + 1) / ST) & 1, dead) && mbar_wait(&S.s_free[w], j & 1, dead);
          if (!ok) break;
          fence_after();
          scores(j + 1);
        }
        if (j < nw) {
          ok = mbar_wait(&S.v_full[st], ph, dead) && mbar_wait(&S.p_full[w], j & 1, dead);
          if (!ok) break;
          fence_after();
          const uint64_t vd = dv + (uint64_t)(st * VS * (SLAB >> 4));
#pragma unroll
          for (int t = 0; t < 8; ++t)     // four k-steps of the hi term, then of the lo term
            mma_ts(to, tp + t * 8, vd + (t & 3) * (2048 >> 4), id_o, (j | t) ? 1u : 0u);
          commit(&S.pv_done[w]);
          commit(&S.v_empty[st]);
        } else {                          // a tile that only the other half uses
          ok = mbar_wait(&S.k_full[st], ph, dead) && mbar_wait(&S.v_full[st], ph, dead);
          if (!ok) break;
          mbar_arrive(&S.k_empty[st]);
          mbar_arrive(&S.v_empty[st]);
        }
      }
      // no arrival may be under way when the CTA ends: every stage's last use has been released
      for (int j = max(0, nt - ST); ok && j < nt; ++j)
        ok = mbar_wait(&S.k_empty[j % ST], (j / ST) & 1, dead) && mbar_wait(&S.v_empty[j % ST], (j / ST) & 1, dead);
    }
  } else if (warp == 11) {
    if constexpr (MODE == BIAS) {
    const float* brow = a.bias ? a.bias + (size_t)h * a.bias_len : nullptr;
    for (int j = 0; j < nt; ++j) {
      const int st = j % BST, ph = (j / BST) & 1;
      float v[10];                         // requested before the buffer is free
      const int d0 = pos0 + ROWS - 1 - j * KT;         // the window's entries step down in distance, as a row's keys do
#pragma unroll
      for (int i = 0; i < 10; ++i) {
        const int d = d0 - i * 32 - lane;
        v[i] = (brow && d >= 0 && d < a.bias_len) ? -brow[d] * LOG2E : 0.f;
      }
      if (!mbar_wait(&S.b_empty[st], ph ^ 1, dead)) break;
      float* dst = S.bias + st * 4 * BW;
#pragma unroll
      for (int i = 0; i < 10; ++i)
#pragma unroll
        for (int s = 0; s < 4; ++s)
          if (i * 32 + lane >= s) dst[s * BW + i * 32 + lane - s] = v[i];
      mbar_arrive(&S.b_full[st]);
    }
    }
  } else {
    const int w = warp >> 2, r = (warp & 3) * 32 + lane, nw = w ? n1 : n0;
    const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t ts = tmem + w * 64 + lanes, tp = tmem + 128 + w * 64 + lanes, to = tmem + 256 + w * 128 + lanes;
    const int pos = pos0 + w * HALF + r, rr = w * HALF + r, shift = (ROWS - 1 - rr) & 3;
    const float sl2 = MODE == CAP ? a.scale / a.cap : a.scale * LOG2E;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < nt; ++j) {
      const int st = j % BST, ph = (j / BST) & 1;
      if constexpr (MODE == BIAS) {
        ok = mbar_wait(&S.b_full[st], ph, dead);
        if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
      }
      if (j >= nw) {
        if constexpr (MODE == BIAS) mbar_arrive(&S.b_empty[st]);
        continue;
      }
      ok = mbar_wait(&S.s_full[w], j & 1, dead);
      if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
      fence_after();
      float s[KT];
      ld32(ts, s); ld32(ts + 32, s + 32);
      wait_ld();
      fence_before();
      mbar_arrive(&S.s_free[w]);
      const float* bp = S.bias + (MODE == BIAS ? st * 4 * BW + shift * BW + (ROWS - 1 - rr - shift) : 0);
      if constexpr (MODE == CAP) {       // sl2: scale over cap
        float big = 0.f;
#pragma unroll
        for (int c = 0; c < KT; ++c) big = fmaxf(big, fabsf(s[c]));
        const float2 to2 = make_float2(sl2, sl2), back = make_float2(a.cap * LOG2E, a.cap * LOG2E), zero = make_float2(0.f, 0.f);
        if (__all_sync(0xffffffffu, big * fabsf(sl2) <= 0.5f)) {
#pragma unroll
          for (int c = 0; c < KT; c += 2) {
            const float2 t = fma2(tanh_small2(fma2(make_float2(s[c], s[c + 1]), to2, zero)), back, zero);
            s[c] = t.x; s[c + 1] = t.y;
          }
        } else {
#pragma unroll
          for (int c = 0; c < KT; ++c) s[c] = tanh_any(s[c] * sl2) * back.x;
        }
      } else
#pragma unroll
      for (int q = 0; q < KT / 4; ++q) {
        const float4 b = MODE != BIAS ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(bp + 4 * q);
        const float2 x = fma2(make_float2(s[4 * q], s[4 * q + 1]), make_float2(sl2, sl2), make_float2(b.x, b.y));
        const float2 y = fma2(make_float2(s[4 * q + 2], s[4 * q + 3]), make_float2(sl2, sl2), make_float2(b.z, b.w));
        s[4 * q] = x.x; s[4 * q + 1] = x.y; s[4 * q + 2] = y.x; s[4 * q + 3] = y.y;
      }
      if constexpr (MODE == BIAS) mbar_arrive(&S.b_empty[st]);
      const int k0 = (j0 + j) * KT, vis = pos - k0, out = vis - a.window;      // keys out + 1 .. vis of the tile are visible
      if (k0 + KT - 1 > pos0 + w * HALF || k0 <= pos0 + w * HALF + HALF - 1 - a.window) {
#pragma unroll
        for (int c = 0; c < KT; ++c) s[c] = c <= vis && c > out ? s[c] : -INFINITY;
      }
      float mx[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int c = 4; c < KT; ++c) mx[c & 3] = fmaxf(mx[c & 3], s[c]);
      float m_new = fmaxf(m, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])));
      if (j > 0 && m_new - m <= 8.f) m_new = m;
      const float ref = m_new == -INFINITY ? 0.f : m_new;      // no visible key yet
      const float corr = ex2(m - ref);
      float2 ls[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
      const float2 mneg = make_float2(-ref, -ref);
      uint32_t hi[KT / 2], lo[KT / 2];
#pragma unroll
      for (int i = 0; i < KT / 2; ++i) {
        const float2 t = add2(make_float2(s[2 * i], s[2 * i + 1]), mneg);
        const float p0 = ex2(t.x), p1 = ex2(t.y);
        ls[i & 1] = add2(ls[i & 1], make_float2(p0, p1));
        hi[i] = __byte_perm(__float_as_uint(p0), __float_as_uint(p1), 0x7632);      // the upper halves
        const float2 rest = add2(make_float2(p0, p1), make_float2(__uint_as_float((__float_as_uint(p0) & 0xffff0000u) ^ 0x80000000u),
                                                                  __uint_as_float((__float_as_uint(p1) & 0xffff0000u) ^ 0x80000000u)));
        const __nv_bfloat162 lb = __floats2bfloat162_rn(rest.x, rest.y);
        lo[i] = *reinterpret_cast<const uint32_t*>(&lb);
      }
      if (j > 0) {                         // P and O are free once the previous tile's product is done
        ok = mbar_wait(&S.pv_done[w], (j - 1) & 1, dead);
        if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
        fence_after();
      }
      st16(tp, hi); st16(tp + 16, hi + 16); st16(tp + 32, lo); st16(tp + 48, lo + 16);
      if (j > 0 && __any_sync(0xffffffffu, corr != 1.f)) {
        for (int c = 0; c < VS * 64; c += 16) {
          float o[16];
          ld16(to + c, o);
          wait_ld();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[i] *= corr;
          st16(to + c, reinterpret_cast<const uint32_t*>(o));
        }
      }
      wait_st();
      l = l * corr + (ls[0].x + ls[0].y) + (ls[1].x + ls[1].y);
      m = m_new;
      fence_before();
      mbar_arrive(&S.p_full[w]);
    }
    if (ok && nw > 0) {
      ok = mbar_wait(&S.pv_done[w], (nw - 1) & 1, dead);
      if (__all_sync(0xffffffffu, ok)) {
        fence_after();
        const float inv = 1.f / (a.sink ? l + ex2(a.sink[h] * LOG2E - m) : l);
        const bool valid = rr < rows;
        __nv_bfloat16* o = a.out + ((size_t)(row0 + rr) * a.H + h) * a.vdim;
        for (int c = 0; c < a.vdim; c += 16) {
          float f[16];
          ld16(to + c, f);
          wait_ld();
          uint32_t u[8];
          if (a.gate && valid) {
            const __nv_bfloat16* gp = a.gate + (size_t)(row0 + rr) * a.gate_row + (size_t)h * a.vdim + c;
#pragma unroll
            for (int i = 0; i < 16; i += 8) {
              if (c + i >= a.vdim) break;
              float z[8];
              rows::load_v<__nv_bfloat16, 8>(gp + i, z);
#pragma unroll
              for (int k = 0; k < 8; ++k) f[i + k] *= rows::gate_sigmoid<__nv_bfloat16>(z[k]);
            }
          }
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const __nv_bfloat162 t = __floats2bfloat162_rn(f[2 * i] * inv, f[2 * i + 1] * inv);
            u[i] = *reinterpret_cast<const uint32_t*>(&t);
          }
          if (valid) {             // vdim is a multiple of eight: whole 16-byte words
            *reinterpret_cast<uint4*>(o + c) = make_uint4(u[0], u[1], u[2], u[3]);
            if (c + 8 < a.vdim) *reinterpret_cast<uint4*>(o + c + 8) = make_uint4(u[4], u[5], u[6], u[7]);
          }
        }
      }
    }
  }
  fence_before();
  __syncthreads();
  if (tid == 0 && *dead) status_set(a.status, ST_TIMEOUT, 64, blockIdx.x, blockIdx.y);
  if (warp == 8) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, 512;" ::"r"(tmem) : "memory");
}

typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                             const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

template <int DS, int VS, int RS, int MODE>
static int launch_mode(const CUtensorMap* mq, const CUtensorMap* mk, const CUtensorMap* mv, const CUtensorMap* mr, const Args& a, int n_tiles, cudaStream_t st) {
  const size_t smem = sizeof(Smem<DS, VS, RS, MODE>) + 1024;
  static bool done = false;
  if (!done) {
    const cudaError_t e = cudaFuncSetAttribute(attn_run_kernel<DS, VS, RS, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    done = true;
  }
  return (int)sfb_launch(attn_run_kernel<DS, VS, RS, MODE>, dim3(a.H, n_tiles), dim3(THREADS), smem, st, *mq, *mk, *mv, *mr, a);
}
template <int DS, int VS, int RS>
static int launch(const CUtensorMap* mq, const CUtensorMap* mk, const CUtensorMap* mv, const CUtensorMap* mr, const Args& a, int n_tiles, cudaStream_t st) {
  if constexpr (RS == 0) {
    if (a.cap > 0.f) return launch_mode<DS, VS, RS, CAP>(mq, mk, mv, mr, a, n_tiles, st);
    if (a.bias) return launch_mode<DS, VS, RS, BIAS>(mq, mk, mv, mr, a, n_tiles, st);
  }
  return launch_mode<DS, VS, RS, PLAIN>(mq, mk, mv, mr, a, n_tiles, st);
}

}  // namespace rtc
}  // namespace sfb

using namespace sfb;
using namespace sfb::rtc;

extern "C" {

// 2-D bf16 map over [rows, cols] (row stride in bytes, a multiple of 16) with a box of 64 columns x box_rows, 128-byte swizzled, or of 32
// columns, 64-byte swizzled; columns past the row's end read as zero and are not stored.  0, a CUresult, or -1 without the driver entry point.
int sfb_rows_tmap(void* out_map, const void* base, int64_t rows, int64_t cols, int64_t row_bytes, int box_rows, int box_cols) {
  if (box_cols != 64 && box_cols != 32) return (int)CUDA_ERROR_INVALID_VALUE;
  static EncodeFn fn = nullptr;
  if (!fn) {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess) fn = (EncodeFn)p;
  }
  if (!fn) return -1;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)row_bytes};
  cuuint32_t box[2] = {(cuuint32_t)box_cols, (cuuint32_t)box_rows}, estr[2] = {1u, 1u};
  return (int)fn((CUtensorMap*)out_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                 CU_TENSOR_MAP_INTERLEAVE_NONE, box_cols == 64 ? CU_TENSOR_MAP_SWIZZLE_128B : CU_TENSOR_MAP_SWIZZLE_64B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
}

// mq: queries [rows, H (dim + rot)], box 128 rows; mk, mv: keys and values [rows, dim / vdim], box 64 rows, page p of head g at row
// p k_page + g k_head (through the page table, or p + offs[tile]); mr: the shared key part [rows, rot] or null.  dim and vdim: multiples
// of 8 up to 128; rot: a multiple of 8 up to 64.  gate: as in Args, rows on 16-byte boundaries.
int sfb_rows_attn_tc(const void* mq, const void* mk, const void* mv, const void* mr, const int* table, const int* row_lane, const int* row_pos,
                     const int* tiles, const int* offs, int n_tiles, const void* bias, int64_t bias_len, const void* sink, float cap, void* out,
                     const void* gate, int64_t gate_row, int max_pages, int n_pages, int H, int G,
                     int dim, int vdim, int rot, int k_page, int k_head, int window, float scale, void* status, cudaStream_t stream) {
  if (n_tiles < 1 || n_tiles > 65535 || G < 1 || H % G || dim % 8 || vdim % 8 || dim < 8 || dim > 128 || vdim < 8 || vdim > 128 || rot % 8 || rot > 64 ||
      (rot > 0) != (mr != nullptr) || (rot && bias) || (cap > 0.f && (bias || rot)) || window < 1 || (gate && (gate_row % 8 || (uintptr_t)gate % 16)))
    return (int)cudaErrorInvalidValue;
  Args a{tiles, table, row_lane, row_pos, offs, (const float*)bias, bias_len, (const float*)sink, cap, (__nv_bfloat16*)out, (const __nv_bfloat16*)gate, gate_row, max_pages, n_pages, H, G, dim, vdim, rot, k_page, k_head,
         window, scale, (Status*)status};
  const CUtensorMap *q = (const CUtensorMap*)mq, *k = (const CUtensorMap*)mk, *v = (const CUtensorMap*)mv, *r = mr ? (const CUtensorMap*)mr : k;
  if (rot) {
    if (dim <= 64) return vdim <= 64 ? launch<1, 1, 1>(q, k, v, r, a, n_tiles, stream) : launch<1, 2, 1>(q, k, v, r, a, n_tiles, stream);
    return vdim <= 64 ? launch<2, 1, 1>(q, k, v, r, a, n_tiles, stream) : launch<2, 2, 1>(q, k, v, r, a, n_tiles, stream);
  }
  if (dim <= 64) return vdim <= 64 ? launch<1, 1, 0>(q, k, v, r, a, n_tiles, stream) : launch<1, 2, 0>(q, k, v, r, a, n_tiles, stream);
  return vdim <= 64 ? launch<2, 1, 0>(q, k, v, r, a, n_tiles, stream) : launch<2, 2, 0>(q, k, v, r, a, n_tiles, stream);
}

}  // extern "C"
