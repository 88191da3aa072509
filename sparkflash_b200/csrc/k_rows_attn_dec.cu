// Softmax attention of single rows over the paged cache, bf16, paced by memory: score = (q . k) * scale - bias[head][distance], the last
// `window` positions; optionally cap * tanh(score / cap), and a sink per head whose exponential is in the denominator only.
//
// The pages of all (row, head group) units of the launch form one sequence that is cut evenly over a fixed number of CTAs, so
// rows of any lengths keep every SM busy to the end.  A CTA's producer warp streams its pages (a page of one head's keys and of
// its values: two bulk copies) through a ring of shared-memory stages; eight warps take eight keys of every page each and keep
// their own online softmax, so no barrier is needed per page.  Scores: four lanes per key; values: a lane owns four dims.  The
// warps' results are merged where a unit ends; a unit that is cut leaves (maximum, sum, output) partials for a merge kernel.
//
// Every wait is bounded; a role that gives up lets the others run through (with a status code) instead of leaving a barrier.
#include "k_rows.cuh"

namespace sfb {
namespace rdec {

constexpr int PAGE = 64, WARPS = 8, THREADS = (WARPS + 1) * 32, MAX_ROWS = 1024, MIN_PAGES = 2;
constexpr float LOG2E = 1.4426950408889634f;

struct Args {
  const __nv_bfloat16* q;       // [n, H dim]
  const __nv_bfloat16 *kpool, *vpool;
  const int* table;
  const int *row_lane, *row_pos;
  const int* rows;              // row indices or null
  const float* bias;            // [H, bias_len] or null
  int64_t bias_len;
  const float* sink;            // [H] or null
  float cap;                    // 0: none
  int window;                   // keys a row sees: itself and the window - 1 before it
  __nv_bfloat16* out;           // [n, H vdim]
  float* part;                  // [2 CTAs, R, vdim]
  float* ml;                    // [2 CTAs, R, 2]
  int max_pages, n_pages, n_rows, H, G, dim, vdim, hgroups, ctas, stages;
  float scale;
  Status* status;
};

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ bool mbar_try(uint64_t* b, uint32_t parity) {
  uint32_t ok;
  asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
               : "=r"(ok) : "r"(smem_u32(b)), "r"(parity) : "memory");
  return ok != 0;
}
__device__ __forceinline__ void mbar_wait(uint64_t* b, uint32_t parity, volatile int* dead) {
  for (uint32_t i = 0; i < (1u << 22); ++i) {
    if (mbar_try(b, parity)) return;
    if (i > 256) {
      if (*dead) return;
      if (i > 4096) __nanosleep(64);
    }
  }
  *dead = 1;
}
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ int first_page(const Args& a, int pos) { return max(0, pos - a.window + 1) / PAGE; }
__device__ __forceinline__ int row_pages(const Args& a, int r) {
  const int pos = a.row_pos[a.rows ? a.rows[r] : r];
  return pos / PAGE + 1 - first_page(a, pos);
}
// cap * tanh(x / cap) without cancellation that would show next to the cap's rounding
__device__ __forceinline__ float capped(float x, float cap) {
  const float e = __expf(-2.f * fabsf(x) / cap);
  return copysignf(cap * __fdividef(1.f - e, 1.f + e), x);
}
// a finished unit: output relative to the larger of the scores' maximum and the sink (both in units of log2)
__device__ __forceinline__ float finish(const Args& a, int head, float o, float m, float l) {
  if (!a.sink) return o / l;
  const float sk = a.sink[head] * LOG2E, top = fmaxf(m, sk), f = ex2(m - top);
  return o * f / (l * f + ex2(sk - top));
}
// pages per CTA: even shares, but no CTA for less than a couple of pages
__device__ __forceinline__ int share(int total, int ctas) { return max((total + ctas - 1) / ctas, MIN_PAGES); }

// position in the page sequence: row, unit of the row, page of the unit
struct Cursor {
  int r, u, p, pages;
};

template <int KC, int NVV, int R>      // 32-element groups of a key row; 128-element groups of a value row; heads per unit
__global__ void __launch_bounds__(THREADS, KC * R <= 8 && NVV == 1 ? 2 : 1) attn_stream_kernel(Args a) {
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ int base[MAX_ROWS + 1];
  __shared__ __align__(8) uint64_t full[4], empty[4];
  __shared__ float wm[WARPS][R], wl[WARPS][R];
  __shared__ int dead_flag;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  volatile int* dead = &dead_flag;
  const int kbytes = PAGE * a.dim * 2, vbytes = PAGE * a.vdim * 2, sbytes = kbytes + vbytes;
  if (tid == 0) {
    dead_flag = 0;
    for (int i = 0; i < a.stages; ++i) {
      asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(smem_u32(&full[i])));
      asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(&empty[i])), "r"(WARPS));
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  pdl_launch_dependents();
  pdl_wait();
  const int units = a.G * a.hgroups, rep = a.H / a.G;
  if (warp == 0) {                       // pages before every row
    int carry = 0;
    for (int r0 = 0; r0 < a.n_rows; r0 += 32) {
      const int r = r0 + lane;
      int v = r < a.n_rows ? row_pages(a, r) * units : 0;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const int t = __shfl_up_sync(0xffffffffu, v, o); if (lane >= o) v += t; }
      if (r < a.n_rows) base[r + 1] = carry + v;
      carry += __shfl_sync(0xffffffffu, v, 31);
    }
    if (lane == 0) base[0] = 0;
  }
  __syncthreads();
  const int total = base[a.n_rows], per = share(total, a.ctas);
  const int begin = min((int)blockIdx.x * per, total), end = min(begin + per, total);
  Cursor c{0, 0, 0, 1};
  if (begin < end) {
    int lo = 0, hi = a.n_rows - 1;
    while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (base[mid] <= begin) lo = mid; else hi = mid - 1; }
    c.r = lo; c.pages = (base[lo + 1] - base[lo]) / units;
    c.u = (begin - base[lo]) / c.pages; c.p = (begin - base[lo]) % c.pages;
  }
  auto next = [&](Cursor& k) {
    if (++k.p == k.pages) {
      k.p = 0;
      if (++k.u == units) {
        k.u = 0;
        if (++k.r < a.n_rows) k.pages = (base[k.r + 1] - base[k.r]) / units;
      }
    }
  };
  if (warp == WARPS) {
    if (lane == 0) {
      int i = 0;
      for (int at = begin; at < end; ++at, ++i, next(c)) {
        const int st = i % a.stages, ph = (i / a.stages) & 1;
        const int row = a.rows ? a.rows[c.r] : c.r;
        int page = a.table[(size_t)a.row_lane[row] * a.max_pages + first_page(a, a.row_pos[row]) + c.p];
        if (page < 0 || page >= a.n_pages) { status_set(a.status, ST_BOUNDS, 65, page, a.n_pages); page = 0; }
        const size_t blk = (size_t)page * a.G + c.u / a.hgroups;
        mbar_wait(&empty[st], ph ^ 1, dead);
        if (*dead) break;
        uint8_t* dst = smem + (size_t)st * sbytes;
        asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(&full[st])), "r"(sbytes) : "memory");
        bulk_load(dst, a.kpool + blk * PAGE * a.dim, kbytes, &full[st]);
        bulk_load(dst + kbytes, a.vpool + blk * PAGE * a.vdim, vbytes, &full[st]);
      }
      if (*dead) {          // copies still in flight must land before the CTA ends
        for (int k = max(0, i - a.stages); k < i; ++k)
          for (int t = 0; t < 100000 && !mbar_try(&full[k % a.stages], (k / a.stages) & 1); ++t) __nanosleep(64);
      }
    }
  } else {
    const int key = warp * 8 + (lane >> 2), ql = lane & 3;
    constexpr int KP_MAX = 4;
    const int vl = min(32, a.vdim / 4), kp = vl <= 8 ? KP_MAX : vl <= 16 ? 2 : 1;      // lanes per value row, keys per pass
    const int vsub = kp == 1 ? 0 : lane / vl, vlane = kp == 1 ? lane : lane % vl;
    const bool vact = kp == 1 ? lane < vl : vsub < kp;
    float* pbuf = reinterpret_cast<float*>(smem + (size_t)a.stages * sbytes) + warp * R * 8;      // [R][8] weights of the warp's keys
    float* red = reinterpret_cast<float*>(smem + (size_t)a.stages * sbytes) + WARPS * R * 8;      // [8][R][vdim]
    uint32_t qr[R][KC][4];                 // the lane's query dims as bf16 pairs
    float m[R], l[R], acc[R][NVV][4];
    int i = 0;
    bool fresh = true, from_start = false;
    for (int at = begin; at < end; ++at, ++i) {
      const int st = i % a.stages, ph = (i / a.stages) & 1;
      const int row = a.rows ? a.rows[c.r] : c.r, pos = a.row_pos[row];
      const int h0 = (c.u / a.hgroups) * rep + (c.u % a.hgroups) * R, nh = min(R, rep - (c.u % a.hgroups) * R);
      if (fresh) {
        fresh = false;
        from_start = c.p == 0;
#pragma unroll
        for (int r = 0; r < R; ++r) {
          m[r] = -INFINITY; l[r] = 0.f;
#pragma unroll
          for (int v = 0; v < NVV; ++v)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[r][v][k] = 0.f;
          const __nv_bfloat16* qp = a.q + ((size_t)row * a.H + h0 + (r < nh ? r : 0)) * a.dim;
#pragma unroll
          for (int g = 0; g < KC; ++g) {
            const int gg = (KC & 1) ? g : g ^ ((lane >> 2) & 1);        // neighbouring keys read the other 64-byte half first
            const uint4 t = *reinterpret_cast<const uint4*>(qp + gg * 32 + ql * 8);
            qr[r][g][0] = t.x; qr[r][g][1] = t.y; qr[r][g][2] = t.z; qr[r][g][3] = t.w;
          }
        }
      }
      const int dist = pos - ((first_page(a, pos) + c.p) * PAGE + key);
      float b[R];
#pragma unroll
      for (int r = 0; r < R; ++r) b[r] = (a.bias && dist >= 0 && r < nh) ? a.bias[(size_t)(h0 + r) * a.bias_len + dist] : 0.f;
      mbar_wait(&full[st], ph, dead);
      const uint8_t* kt = smem + (size_t)st * sbytes;
      float dot[R];
#pragma unroll
      for (int r = 0; r < R; ++r) dot[r] = 0.f;
#pragma unroll
      for (int g = 0; g < KC; ++g) {
        const int gg = (KC & 1) ? g : g ^ ((lane >> 2) & 1);
        const uint4 t = *reinterpret_cast<const uint4*>(kt + (size_t)key * a.dim * 2 + gg * 64 + ql * 16);
        const uint32_t w[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float k0 = __uint_as_float(w[k] << 16), k1 = __uint_as_float(w[k] & 0xffff0000u);
#pragma unroll
          for (int r = 0; r < R; ++r) {
            dot[r] = fmaf(__uint_as_float(qr[r][g][k] << 16), k0, dot[r]);
            dot[r] = fmaf(__uint_as_float(qr[r][g][k] & 0xffff0000u), k1, dot[r]);
          }
        }
      }
      float corr[R];
#pragma unroll
      for (int r = 0; r < R; ++r) {
        float s = dot[r];
        s += __shfl_xor_sync(0xffffffffu, s, 1);
        s += __shfl_xor_sync(0xffffffffu, s, 2);
        s = s * a.scale - b[r];
        if (a.cap > 0.f) s = capped(s, a.cap);
        s = dist >= 0 && dist < a.window ? s * LOG2E : -INFINITY;
        float mx = s;
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
        const float mn = fmaxf(m[r], mx), ref = mn == -INFINITY ? 0.f : mn;      // the warp's keys may all lie past the row
        const float p = ex2(s - ref);
        corr[r] = ex2(m[r] - ref);
        l[r] = l[r] * corr[r] + p;           // per key; the four lanes of a key hold the same sum
        m[r] = mn;
        if (ql == 0) pbuf[r * 8 + (lane >> 2)] = p;
      }
      __syncwarp();
      const uint8_t* vt = kt + kbytes + (size_t)warp * 8 * a.vdim * 2;
#pragma unroll
      for (int r = 0; r < R; ++r)
#pragma unroll
        for (int v = 0; v < NVV; ++v)
#pragma unroll
          for (int k = 0; k < 4; ++k) acc[r][v][k] *= corr[r];
      if (vact) {
#pragma unroll 4
        for (int k8 = vsub; k8 < 8; k8 += kp) {
          float pr[R];
#pragma unroll
          for (int r = 0; r < R; ++r) pr[r] = pbuf[r * 8 + k8];
#pragma unroll
          for (int v = 0; v < NVV; ++v) {
            if (NVV > 1 && v * 128 + vlane * 4 >= a.vdim) break;
            float f[4];
            rows::load_v<__nv_bfloat16, 4>(reinterpret_cast<const __nv_bfloat16*>(vt) + (size_t)k8 * a.vdim + v * 128 + vlane * 4, f);
#pragma unroll
            for (int r = 0; r < R; ++r)
#pragma unroll
              for (int k = 0; k < 4; ++k) acc[r][v][k] = fmaf(pr[r], f[k], acc[r][v][k]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&empty[st])) : "memory");
      const bool unit_end = c.p + 1 == c.pages;
      if (unit_end || at + 1 == end) {
        // merge the warps: keys of a pass, then the eight warps
#pragma unroll
        for (int r = 0; r < R; ++r) {
          float t = l[r];
          t += __shfl_xor_sync(0xffffffffu, t, 4);
          t += __shfl_xor_sync(0xffffffffu, t, 8);
          t += __shfl_xor_sync(0xffffffffu, t, 16);
          if (lane == 0) { wm[warp][r] = m[r]; wl[warp][r] = t; }
#pragma unroll
          for (int v = 0; v < NVV; ++v)
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              float t2 = acc[r][v][k];
              if (kp == 4) t2 += __shfl_xor_sync(0xffffffffu, t2, 8);
              if (kp > 1) t2 += __shfl_xor_sync(0xffffffffu, t2, 16);
              acc[r][v][k] = t2;
            }
          if (vsub == 0 && lane < vl) {
#pragma unroll
            for (int v = 0; v < NVV; ++v)
              if (v * 128 + lane * 4 < a.vdim)
                *reinterpret_cast<float4*>(red + ((size_t)warp * R + r) * a.vdim + v * 128 + lane * 4) =
                    make_float4(acc[r][v][0], acc[r][v][1], acc[r][v][2], acc[r][v][3]);
          }
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        const bool whole = from_start && unit_end;
        // partial slot: 2c when the unit is the CTA's first, 2c + 1 otherwise
        const int slot = 2 * blockIdx.x + (at - c.p > begin ? 1 : 0);
        for (int x = tid; x < nh * a.vdim; x += WARPS * 32) {
          const int r = x / a.vdim, v = x - r * a.vdim;
          float mm = wm[0][r];
#pragma unroll
          for (int w = 1; w < WARPS; ++w) mm = fmaxf(mm, wm[w][r]);
          float o = 0.f, ll = 0.f;
#pragma unroll
          for (int w = 0; w < WARPS; ++w) {
            const float f = ex2(wm[w][r] - mm);
            o += red[((size_t)w * R + r) * a.vdim + v] * f;
            ll += wl[w][r] * f;
          }
          if (whole) a.out[((size_t)row * a.H + h0 + r) * a.vdim + v] = __float2bfloat16_rn(finish(a, h0 + r, o, mm, ll));
          else {
            a.part[((size_t)slot * R + r) * a.vdim + v] = o;
            if (v == 0) { a.ml[((size_t)slot * R + r) * 2] = mm; a.ml[((size_t)slot * R + r) * 2 + 1] = ll; }
          }
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        fresh = true;
      }
      next(c);
    }
  }
  __syncthreads();
  if (tid == 0 && *dead) status_set(a.status, ST_TIMEOUT, 66, blockIdx.x, 0);
}

// the partials of one cut unit; grid (units, rows)
template <int R>
__global__ void __launch_bounds__(128) attn_stream_merge_kernel(Args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.y, u = blockIdx.x, units = a.G * a.hgroups, rep = a.H / a.G;
  int lo = 0, all = 0;
  for (int k = threadIdx.x; k < a.n_rows; k += 128) {
    const int v = row_pages(a, k) * units;
    all += v;
    if (k < r) lo += v;
  }
  __shared__ int sums[2][4];
  for (int o = 16; o > 0; o >>= 1) { lo += __shfl_xor_sync(0xffffffffu, lo, o); all += __shfl_xor_sync(0xffffffffu, all, o); }
  if ((threadIdx.x & 31) == 0) { sums[0][threadIdx.x >> 5] = lo; sums[1][threadIdx.x >> 5] = all; }
  __syncthreads();
  lo = sums[0][0] + sums[0][1] + sums[0][2] + sums[0][3];
  all = sums[1][0] + sums[1][1] + sums[1][2] + sums[1][3];
  const int per = share(all, a.ctas), pages = row_pages(a, r), start = lo + u * pages;
  const int c0 = start / per, c1 = (start + pages - 1) / per;
  if (c0 == c1) return;
  const int h0 = (u / a.hgroups) * rep + (u % a.hgroups) * R, nh = min(R, rep - (u % a.hgroups) * R);
  const int row = a.rows ? a.rows[r] : r;
  // weight of every partial: one warp per head, lanes over the partials
  extern __shared__ float wts[];             // [R][partials]
  __shared__ float lsum[R];
  const int parts = c1 - c0 + 1, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int k = warp; k < nh; k += 4) {
    float m = -INFINITY, l = 0.f;
    for (int c = lane; c < parts; c += 32) m = fmaxf(m, a.ml[((size_t)(2 * (c0 + c) + (start > (c0 + c) * per)) * R + k) * 2]);
    m = warp_max(m);
    if (a.sink) {
      m = fmaxf(m, a.sink[h0 + k] * LOG2E);
      if (lane == 0) l = ex2(a.sink[h0 + k] * LOG2E - m);
    }
    for (int c = lane; c < parts; c += 32) {
      const size_t s = (size_t)(2 * (c0 + c) + (start > (c0 + c) * per)) * R + k;
      const float f = ex2(a.ml[2 * s] - m);
      wts[k * parts + c] = f;
      l += a.ml[2 * s + 1] * f;
    }
    l = warp_sum(l);
    if (lane == 0) lsum[k] = l;
  }
  __syncthreads();
  // a warp takes every fourth partial, a lane four dims of it; the warps' sums meet in shared memory
  __shared__ float4 red[4][R * 64];
  const int quads = nh * a.vdim / 4;
  for (int x = lane; x < quads; x += 32) {
    const int k = x / (a.vdim / 4), v = (x - k * (a.vdim / 4)) * 4;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int c = warp; c < parts; c += 4) {
      const float4 p = *reinterpret_cast<const float4*>(a.part + ((size_t)(2 * (c0 + c) + (start > (c0 + c) * per)) * R + k) * a.vdim + v);
      const float w = wts[k * parts + c];
      o.x += p.x * w; o.y += p.y * w; o.z += p.z * w; o.w += p.w * w;
    }
    red[warp][x] = o;
  }
  __syncthreads();
  for (int x = threadIdx.x; x < quads; x += 128) {
    const int k = x / (a.vdim / 4), v = (x - k * (a.vdim / 4)) * 4;
    const float inv = 1.f / lsum[k];
    const float4 p = red[0][x], q = red[1][x], r2 = red[2][x], t = red[3][x];
    const float f[4] = {(p.x + q.x + r2.x + t.x) * inv, (p.y + q.y + r2.y + t.y) * inv, (p.z + q.z + r2.z + t.z) * inv, (p.w + q.w + r2.w + t.w) * inv};
    rows::store_v<__nv_bfloat16, 4>(a.out + ((size_t)row * a.H + h0 + k) * a.vdim + v, f);
  }
}

template <int KC, int NVV, int R>
static int launch(Args a, int max_total, cudaStream_t st) {
  a.hgroups = (a.H / a.G + R - 1) / R;
  const size_t stage = (size_t)PAGE * (a.dim + a.vdim) * 2, extra = (size_t)WARPS * R * (8 + a.vdim) * 4;
  a.stages = 4;
  while (a.stages > 2 && a.stages * stage + extra > 110 * 1024) --a.stages;
  const size_t smem = a.stages * stage + extra;
  if (smem > 220 * 1024) return (int)cudaErrorInvalidValue;
  static size_t granted = 0;
  if (smem > granted) {
    const cudaError_t e = cudaFuncSetAttribute(attn_stream_kernel<KC, NVV, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    granted = smem;
  }
  int per_sm = 0, dev = 0, sms = 148;
  cudaError_t e = cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, attn_stream_kernel<KC, NVV, R>, THREADS, smem);
  if (e != cudaSuccess) return (int)e;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  a.ctas = sms * (per_sm < 1 ? 1 : per_sm > 4 ? 4 : per_sm);
  const long long pages = (long long)max_total * a.G * a.hgroups;      // an upper bound of the launch's pages
  if (pages < (long long)a.ctas * MIN_PAGES) a.ctas = (int)((pages + MIN_PAGES - 1) / MIN_PAGES);
  const int rc = (int)sfb_launch(attn_stream_kernel<KC, NVV, R>, dim3(a.ctas), dim3(THREADS), smem, st, a);
  if (rc) return rc;
  return (int)sfb_launch(attn_stream_merge_kernel<R>, dim3(a.G * a.hgroups, a.n_rows), dim3(128), (size_t)R * a.ctas * sizeof(float), st, a);
}
template <int KC, int R>
static int launch_v(const Args& a, int max_total, cudaStream_t st) {
  return a.vdim <= 128 ? launch<KC, 1, R>(a, max_total, st) : launch<KC, 2, R>(a, max_total, st);
}
template <int KC>
static int launch_r(const Args& a, int R, int max_total, cudaStream_t st) {
  return R == 1 ? launch_v<KC, 1>(a, max_total, st) : R == 2 ? launch_v<KC, 2>(a, max_total, st) : launch_v<KC, 4>(a, max_total, st);
}

}  // namespace rdec
}  // namespace sfb

using namespace sfb;
using namespace sfb::rdec;

extern "C" {

// bf16 only; dim and vdim multiples of 32 up to 256 (dim: 32, 64, 96, 128, 256), at most 1,024 rows.  heads_per_unit: 1, 2 or 4.
// page_bound: upper bound of the sum of the rows' pages.  part / ml: 2 x 592 x heads_per_unit x vdim (x 2) floats.
int sfb_rows_attn_stream(const void* q, const void* kpool, const void* vpool, const int* table, const int* row_lane, const int* row_pos,
                         const int* rows, const void* bias, int64_t bias_len, const void* sink, float cap, int window, void* out, void* part, void* ml, int max_pages, int n_pages,
                         int n_rows, int H, int G, int dim, int vdim, int heads_per_unit, int page_bound, float scale, void* status,
                         cudaStream_t stream) {
  if (n_rows < 1 || n_rows > MAX_ROWS || G < 1 || H % G || window < 1 || vdim % 32 || vdim < 32 || vdim > 256) return (int)cudaErrorInvalidValue;
  Args a{};
  a.q = (const __nv_bfloat16*)q; a.kpool = (const __nv_bfloat16*)kpool; a.vpool = (const __nv_bfloat16*)vpool; a.table = table;
  a.row_lane = row_lane; a.row_pos = row_pos; a.rows = rows; a.bias = (const float*)bias; a.bias_len = bias_len; a.sink = (const float*)sink; a.cap = cap; a.window = window; a.out = (__nv_bfloat16*)out;
  a.part = (float*)part; a.ml = (float*)ml; a.max_pages = max_pages; a.n_pages = n_pages; a.n_rows = n_rows; a.H = H; a.G = G; a.dim = dim;
  a.vdim = vdim; a.scale = scale; a.status = (Status*)status;
  switch (dim) {
    case 32: return launch_r<1>(a, heads_per_unit, page_bound, stream);
    case 64: return launch_r<2>(a, heads_per_unit, page_bound, stream);
    case 96: return launch_r<3>(a, heads_per_unit, page_bound, stream);
    case 128: return launch_r<4>(a, heads_per_unit, page_bound, stream);
    case 256: return launch_r<8>(a, heads_per_unit > 2 ? 2 : heads_per_unit, page_bound, stream);
    default: return (int)cudaErrorInvalidValue;
  }
}

}  // extern "C"
