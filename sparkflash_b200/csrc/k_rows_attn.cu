// Softmax attention over the paged cache for single rows and short runs of rows (k_rows_attn_tc.cu takes long runs), in bf16
// or true 32-bit, any head sizes: score = (q . k) * scale - bias[head][distance], causal, the last `window` positions; optionally
// cap * tanh(score / cap), and a sink: a number per head whose exponential is in the softmax's denominator only.
//
// Values may be the first columns of the keys (vpool null): then only key pages are read.  The bias is a table over the distance i - j ([heads, table length], 32-bit), so any distance-only bias is one row of
// numbers per head; null: none.
//
// One block: one row x up to R query heads that share a key/value head x one range of pages.  A page (64 keys) is staged in
// shared memory with cp.async, two pages in flight when they fit; scores: two lanes per key; online softmax: one warp per
// head; values: a thread owns four output dims of every head over a share of the keys.  With more than one range the
// partial (maximum, sum, output) triples are merged by a second kernel.
#include "k_rows.cuh"

namespace sfb {
namespace rows {

struct AttnRowsArgs {
  const void* q;            // [n, H dim] (T)
  const void *kpool, *vpool;  // [pages, G, 64, dim] / [pages, G, 64, vdim] (T)
  const int* table;         // [lanes, max_pages]
  const int *row_lane, *row_pos;
  const int* rows;          // [rows in this launch] row indices, or null: identity
  const float* bias;        // [H, bias_len] or null
  int64_t bias_len;
  const float* sink;        // [H] or null
  float cap;                // 0: none
  void* out;                // [n, H vdim] (T)
  float* part;              // [launch rows, H, splits, vdim]
  float* ml;                // [launch rows, H, splits, 2]
  int max_pages, n_pages, H, G, dim, vdim, splits, hgroups, stages;
  int window;               // keys a row sees: itself and the window - 1 before it
  int compact;              // q and out hold the launch's rows one after another
  int ldk, ldv;             // shared-memory row strides in elements
  float scale;
  Status* status;
};
constexpr int AP = 64;       // keys per page
constexpr int ATHREADS = 128;

__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// 64 rows of `width` elements -> shared rows of `ld` elements; the tail up to a multiple of eight is zeroed
template <typename T>
__device__ __forceinline__ void stage_page(T* dst, const T* src, int width, int ld) {
  const int per16 = 16 / (int)sizeof(T);
  if (width % per16 == 0) {
    const int cpr = width / per16;
    for (int i = threadIdx.x; i < AP * cpr; i += ATHREADS) {
      const int r = i / cpr, c = (i - r * cpr) * per16;
      cp16(dst + r * ld + c, src + (size_t)r * width + c);
    }
    if (width & 7) {
      const int pad = 8 - (width & 7);
      for (int i = threadIdx.x; i < AP * pad; i += ATHREADS) dst[(i / pad) * ld + width + i % pad] = from_f<T>(0.f);
    }
  } else {
    const int w8 = (width + 7) & ~7;
    for (int i = threadIdx.x; i < AP * w8; i += ATHREADS) {
      const int r = i / w8, c = i - r * w8;
      dst[r * ld + c] = c < width ? src[(size_t)r * width + c] : from_f<T>(0.f);
    }
  }
}

template <typename T, int R>
__global__ void __launch_bounds__(ATHREADS) attn_rows_kernel(AttnRowsArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int hg = blockIdx.x % a.hgroups, g = blockIdx.x / a.hgroups;
  const int rep = a.H / a.G, h0 = g * rep + hg * R, nh = min(R, rep - hg * R);
  const int row = a.rows ? a.rows[blockIdx.y] : blockIdx.y;
  const int pos = a.row_pos[row], lane_id = a.row_lane[row];
  const int first = max(0, pos - a.window + 1) / AP, pages = pos / AP + 1 - first, per = (pages + a.splits - 1) / a.splits;
  const int p0 = first + blockIdx.z * per, p1 = min(p0 + per, first + pages);
  const size_t io = a.compact ? blockIdx.y : row;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dim8 = (a.dim + 7) & ~7;
  T* kt = reinterpret_cast<T*>(smem);
  T* vt = a.vpool ? kt + (size_t)a.stages * AP * a.ldk : kt;
  float* qs = reinterpret_cast<float*>(kt + (size_t)a.stages * AP * (a.ldk + (a.vpool ? a.ldv : 0)));   // [R][dim8]
  float* ps = qs + R * dim8;                                                  // [R][64]
  float* fac = ps + R * AP;                                                   // [R] rescale of the running output
  float* msum = fac + R;                                                      // [R][2]
  const int* tab = a.table + (size_t)lane_id * a.max_pages;
  const int cols = (a.vdim + 3) >> 2, groups = ATHREADS / cols, grp = tid / cols, vc = (tid - grp * cols) * 4;
  float acc[R][4];
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int k = 0; k < 4; ++k) acc[r][k] = 0.f;
  float m_run[(R + 3) / 4], l_run[(R + 3) / 4];     // warp w keeps heads w, w + 4, ...
#pragma unroll
  for (int i = 0; i < (R + 3) / 4; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }

  auto stage = [&](int p) {
    int page = tab[p];
    if (page < 0 || page >= a.n_pages) { if (tid == 0) status_set(a.status, ST_BOUNDS, 62, page, a.n_pages); page = 0; }
    const int s = (p - p0) % a.stages;
    stage_page<T>(kt + (size_t)s * AP * a.ldk, (const T*)a.kpool + ((size_t)page * a.G + g) * AP * a.dim, a.dim, a.ldk);
    if (a.vpool) stage_page<T>(vt + (size_t)s * AP * a.ldv, (const T*)a.vpool + ((size_t)page * a.G + g) * AP * a.vdim, a.vdim, a.ldv);
  };
  if (p0 < p1) stage(p0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int i = tid; i < R * dim8; i += ATHREADS) {
    const int r = i / dim8, c = i - r * dim8;
    qs[i] = (r < nh && c < a.dim) ? to_f<T>(((const T*)a.q)[io * a.H * a.dim + (size_t)(h0 + r) * a.dim + c]) * a.scale : 0.f;
  }
  for (int p = p0; p < p1; ++p) {
    if (a.stages > 1) {
      if (p + 1 < p1) stage(p + 1);
      asm volatile("cp.async.commit_group;" ::: "memory");
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int s = (p - p0) % a.stages;
    {  // scores: lanes 2k and 2k + 1 of the block's 128 threads share key k, alternating groups of eight dims
      const int key = tid >> 1, half = tid & 1;
      const T* kr = kt + (size_t)s * AP * a.ldk + (size_t)key * a.ldk;
      float dot[R];
#pragma unroll
      for (int r = 0; r < R; ++r) dot[r] = 0.f;
      for (int c = half * 8; c < dim8; c += 16) {
        float kf[8];
        load_v<T, 8>(kr + c, kf);
#pragma unroll
        for (int r = 0; r < R; ++r) {
          const float4 q0 = *reinterpret_cast<const float4*>(qs + r * dim8 + c), q1 = *reinterpret_cast<const float4*>(qs + r * dim8 + c + 4);
          dot[r] += q0.x * kf[0] + q0.y * kf[1] + q0.z * kf[2] + q0.w * kf[3] + q1.x * kf[4] + q1.y * kf[5] + q1.z * kf[6] + q1.w * kf[7];
        }
      }
      const int dist = pos - (p * AP + key);
#pragma unroll
      for (int r = 0; r < R; ++r) {
        dot[r] += __shfl_xor_sync(0xffffffffu, dot[r], 1);
        if (half == (r & 1) && r < nh) {
          float v = -INFINITY;
          if (dist >= 0 && dist < a.window) {
            v = a.bias ? dot[r] - a.bias[(size_t)(h0 + r) * a.bias_len + dist] : dot[r];
            if (a.cap > 0.f) v = a.cap * tanhf(v / a.cap);
          }
          ps[r * AP + key] = v;
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < (R + 3) / 4; ++i) {
      const int r = warp + i * 4;
      if (r < nh) {
        const float s0 = ps[r * AP + lane], s1 = ps[r * AP + 32 + lane];
        const float m_new = fmaxf(m_run[i], warp_max(fmaxf(s0, s1)));      // every page of the range holds a visible key
        const float e0 = expf(s0 - m_new), e1 = expf(s1 - m_new);
        const float corr = expf(m_run[i] - m_new);
        ps[r * AP + lane] = e0; ps[r * AP + 32 + lane] = e1;
        l_run[i] = l_run[i] * corr + warp_sum(e0 + e1);
        m_run[i] = m_new;
        if (lane == 0) fac[r] = corr;
      }
    }
    __syncthreads();
    if (grp < groups) {
      const T* vb = vt + (size_t)s * AP * a.ldv;
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const float f = r < nh ? fac[r] : 0.f;
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[r][k] *= f;
      }
      for (int key = grp; key < AP; key += groups) {
        float v[4];
        load_v<T, 4>(vb + (size_t)key * a.ldv + vc, v);
#pragma unroll
        for (int r = 0; r < R; ++r) {
          if (r >= nh) break;
          const float pr = ps[r * AP + key];
#pragma unroll
          for (int k = 0; k < 4; ++k) acc[r][k] += pr * v[k];
        }
      }
    }
    __syncthreads();
    if (a.stages == 1 && p + 1 < p1) {
      stage(p + 1);
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
  }
  // ---- sum the key groups, normalise or leave a partial ----
#pragma unroll
  for (int i = 0; i < (R + 3) / 4; ++i) {
    const int r = warp + i * 4;
    if (r < nh && lane == 0) { msum[2 * r] = m_run[i]; msum[2 * r + 1] = l_run[i]; }
  }
  float* red = reinterpret_cast<float*>(smem);                 // [groups][R][cols * 4], the tiles are no longer needed
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  if (grp < groups) {
#pragma unroll
    for (int r = 0; r < R; ++r)
      *reinterpret_cast<float4*>(red + ((size_t)grp * R + r) * cols * 4 + vc) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
  }
  __syncthreads();
  for (int i = tid; i < nh * a.vdim; i += ATHREADS) {
    const int r = i / a.vdim, v = i - r * a.vdim;
    float t = 0.f;
    for (int k = 0; k < groups; ++k) t += red[((size_t)k * R + r) * cols * 4 + v];
    if (a.splits == 1) {
      float l = msum[2 * r + 1];
      if (a.sink) {                       // relative to the larger of the sink and the scores' maximum
        const float sk = a.sink[h0 + r], m = fmaxf(msum[2 * r], sk), f = expf(msum[2 * r] - m);
        t *= f;
        l = l * f + expf(sk - m);
      }
      ((T*)a.out)[(io * a.H + h0 + r) * a.vdim + v] = from_f<T>(t / l);
    }
    else a.part[(((size_t)blockIdx.y * a.H + h0 + r) * a.splits + blockIdx.z) * a.vdim + v] = t;
  }
  if (a.splits > 1 && tid < 2 * nh) a.ml[(((size_t)blockIdx.y * a.H + h0 + (tid >> 1)) * a.splits + blockIdx.z) * 2 + (tid & 1)] = msum[tid];
}

// merge the ranges of one (row, head)
template <typename T>
__global__ void __launch_bounds__(128) attn_rows_merge_kernel(AttnRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, row = a.rows && !a.compact ? a.rows[blockIdx.y] : blockIdx.y;
  const float* ml = a.ml + ((size_t)blockIdx.y * a.H + h) * a.splits * 2;
  const float* part = a.part + ((size_t)blockIdx.y * a.H + h) * a.splits * a.vdim;
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < a.splits; ++s) m = fmaxf(m, ml[2 * s]);
  if (a.sink) { m = fmaxf(m, a.sink[h]); l = expf(a.sink[h] - m); }
  for (int s = 0; s < a.splits; ++s) l += ml[2 * s + 1] * expf(ml[2 * s] - m);
  for (int v = threadIdx.x; v < a.vdim; v += blockDim.x) {
    float t = 0.f;
    for (int s = 0; s < a.splits; ++s) t += part[(size_t)s * a.vdim + v] * expf(ml[2 * s] - m);
    ((T*)a.out)[((size_t)row * a.H + h) * a.vdim + v] = from_f<T>(t / l);
  }
}

template <typename T, int R>
static int launch_attn(AttnRowsArgs a, int n_rows, cudaStream_t st) {
  const int unit = 16 / (int)sizeof(T);
  // rows of shared memory: a whole number of 16-byte units, two more than a multiple of eight, so that the two lanes of
  // four neighbouring keys read eight different bank groups
  auto ld = [&](int w) { const int u = (((w + 7) & ~7) + unit - 1) / unit; return ((u + 7) / 8 * 8 + 2) * unit; };
  a.ldk = ld(a.dim); a.ldv = a.vpool ? ld(a.vdim) : a.ldk;
  const int rep = a.H / a.G, cols = (a.vdim + 3) / 4, groups = ATHREADS / cols;
  a.hgroups = (rep + R - 1) / R;
  const size_t tile = (size_t)AP * (a.ldk + (a.vpool ? a.ldv : 0)) * sizeof(T);
  const size_t extra = ((size_t)R * ((a.dim + 7) & ~7) + R * AP + 3 * R) * sizeof(float);
  const size_t red = (size_t)groups * R * cols * 4 * sizeof(float);
  a.stages = 2 * tile + extra <= 100 * 1024 ? 2 : 1;
  const size_t smem = a.stages * tile + extra;
  if (a.stages * tile < red || smem > 227 * 1024) return (int)cudaErrorInvalidValue;      // the final reduction reuses the tiles
  static size_t granted = 0;
  if (smem > granted) {
    const cudaError_t e = cudaFuncSetAttribute(attn_rows_kernel<T, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    granted = smem;
  }
  return (int)sfb_launch(attn_rows_kernel<T, R>, dim3(a.G * a.hgroups, n_rows, a.splits), dim3(ATHREADS), smem, st, a);
}
template <typename T>
static int launch_attn_r(const AttnRowsArgs& a, int n_rows, cudaStream_t st) {
  const int rep = a.H / a.G;
  int rc;
  if (rep <= 1) rc = launch_attn<T, 1>(a, n_rows, st);
  else if (rep <= 2) rc = launch_attn<T, 2>(a, n_rows, st);
  else if (rep <= 4) rc = launch_attn<T, 4>(a, n_rows, st);
  else rc = launch_attn<T, 8>(a, n_rows, st);
  if (rc || a.splits == 1) return rc;
  return (int)sfb_launch(attn_rows_merge_kernel<T>, dim3(a.H, n_rows), dim3(128), 0, st, a);
}

}  // namespace rows
}  // namespace sfb

using namespace sfb;
using namespace sfb::rows;

extern "C" {

int sfb_rows_attn(const void* q, const void* kpool, const void* vpool, const int* table, const int* row_lane, const int* row_pos,
                  const int* rows, const void* bias, int64_t bias_len, const void* sink, float cap, void* out, void* part, void* ml, int max_pages, int n_pages,
                  int n_rows, int H, int G, int dim, int vdim, int splits, int window, int compact, float scale, int fp32, void* status, cudaStream_t stream) {
  if (n_rows < 1 || n_rows > 65535 || G < 1 || H % G || vdim > 4 * ATHREADS || dim < 1 || vdim < 1 || splits < 1 || window < 1 || (!vpool && vdim > dim)) return (int)cudaErrorInvalidValue;
  AttnRowsArgs a{};
  a.q = q; a.kpool = kpool; a.vpool = vpool; a.table = table; a.row_lane = row_lane; a.row_pos = row_pos; a.rows = rows;
  a.bias = (const float*)bias; a.bias_len = bias_len; a.sink = (const float*)sink; a.cap = cap; a.out = out; a.part = (float*)part; a.ml = (float*)ml; a.max_pages = max_pages;
  a.n_pages = n_pages; a.H = H; a.G = G; a.dim = dim; a.vdim = vdim; a.splits = splits; a.scale = scale; a.status = (Status*)status;
  a.window = window; a.compact = compact;
  return fp32 ? launch_attn_r<float>(a, n_rows, stream) : launch_attn_r<__nv_bfloat16>(a, n_rows, stream);
}

}  // extern "C"
