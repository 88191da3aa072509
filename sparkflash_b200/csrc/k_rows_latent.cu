// Row kernels of latent attention (models/mixers.py): keys and values of all heads are products of one cached vector per token, the
// RMS-normed latent c, beside one rotated key part that the heads share.
//
//   latent_append  norm of the latent, rotation of the shared key part (both to the page pool) and of every head's rotated query part
//                  (in place), pairs (2i, 2i + 1) or (i, i + half); or, where the queries come out of a latent of their own, the norm of that
//                  latent
//   latent_turn    rotation of the queries' part alone, in place
//   head_proj      out[row][h] = x[row][h] W[h] for few rows, W [H, K, M]: the query into the latent space (with the rotation of its other
//                  part), and the attention output out of it (with a sigmoid gate on the result)
//   gather_pages   pages of the pool -> consecutive rows (the keys of a prompt portion, before they are multiplied out)
#include "k_rows.cuh"

namespace sfb {
namespace rows {

struct LatentArgs {
  void* q;                  // [n, q_stride] (T): [H, dim + rot], turned in place; null: the queries are not here
  int64_t q_stride;
  const void* c;            // [n, stride] (T): latent [rank], shared key part [rot]
  const void* cq;           // [n, stride] (T): the queries' latent [q_rank], or null
  void* cqo;                // [n, q_rank] (T): that latent normed
  int64_t stride;
  const float *w, *wq;      // [rank], [q_rank]
  const float2* cs;         // [positions, rot / 2] (cos, sin)
  void* pool;               // [pages, 64, rank + rot] (T)
  const int* table;
  const int *row_lane, *row_pos;
  int max_pages, n_pages, H, dim, rot, rank, q_rank;
  float eps;
  Status* status;
};

// V elements at x (4, or two one by one)
template <typename T, int V> __device__ __forceinline__ void load_few(const T* x, float (&f)[V]) {
  if constexpr (V == 4) load_v<T, 4>(x, f);
  else { f[0] = to_f<T>(x[0]); f[1] = to_f<T>(x[1]); }
}
template <typename T, int V> __device__ __forceinline__ void store_few(T* x, const float (&f)[V]) {
  if constexpr (V == 4) store_v<T, 4>(x, f);
  else { x[0] = from_f<T>(f[0]); x[1] = from_f<T>(f[1]); }
}
// V elements' worth of pairs of a rotated part of `rot` elements, unit u of rot / V: x to o, which may be the same.  HALVES: element i turns with
// i + rot / 2 (units of V / 2 such pairs), else neighbours turn.
template <typename T, int V, bool HALVES>
__device__ __forceinline__ void turn_unit(const T* x, T* o, int u, int half, const float2* cs) {
  if constexpr (HALVES && V == 8) {
    float a[4], b[4];
    const int k = u * 4;
    load_v<T, 4>(x + k, a);
    load_v<T, 4>(x + k + half, b);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 t = cs[k + i];
      const float f = a[i];
      a[i] = f * t.x - b[i] * t.y;
      b[i] = b[i] * t.x + f * t.y;
    }
    store_v<T, 4>(o + k, a);
    store_v<T, 4>(o + k + half, b);
  } else if constexpr (HALVES) {
#pragma unroll
    for (int i = 0; i < V / 2; ++i) {
      const int k = u * (V / 2) + i;
      const float2 t = cs[k];
      const float a = to_f<T>(x[k]), b = to_f<T>(x[k + half]);
      o[k] = from_f<T>(a * t.x - b * t.y);
      o[k + half] = from_f<T>(b * t.x + a * t.y);
    }
  } else {
    float f[V], g[V];
    const int k = u * V;
    load_few<T, V>(x + k, f);
#pragma unroll
    for (int i = 0; i < V; i += 2) {
      const float2 t = cs[(k + i) >> 1];
      g[i] = f[i] * t.x - f[i + 1] * t.y;
      g[i + 1] = f[i + 1] * t.x + f[i] * t.y;
    }
    store_few<T, V>(o + k, g);
  }
}
// the latent's (T) sum of squares, this thread's share of it
template <typename T, int V> __device__ __forceinline__ float squares(const T* c, int rank) {
  float s = 0.f;
  if constexpr (V == 4) {
    for (int i = threadIdx.x * 4; i < rank; i += 512) {
      float f[V];
      load_few<T, V>(c + i, f);
#pragma unroll
      for (int k = 0; k < V; ++k) s += f[k] * f[k];
    }
  } else {
    for (int i = threadIdx.x; i < rank; i += 128) { const float f = to_f<T>(c[i]); s += f * f; }
  }
  return s;
}
template <typename T, int V> __device__ __forceinline__ void normed(const T* c, T* o, const float* w, int rank, float r) {
  if constexpr (V == 4) {
    for (int i = threadIdx.x * 4; i < rank; i += 512) {
      float f[V], g[V];
      load_few<T, V>(c + i, f);
      load_v<float, 4>(w + i, g);
#pragma unroll
      for (int k = 0; k < V; ++k) f[k] *= r * g[k];
      store_few<T, V>(o + i, f);
    }
  } else {
    for (int i = threadIdx.x; i < rank; i += 128) o[i] = from_f<T>(to_f<T>(c[i]) * r * w[i]);
  }
}

// V: elements a thread takes together (4: every width and offset is a multiple of four; 2 otherwise: pairs, element by element)
template <typename T, int V, bool HALVES>
__global__ void __launch_bounds__(128) latent_append_kernel(LatentArgs a) {
  __shared__ float sh[2 * 2 * 32];
  int phase = 0;
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, pos = a.row_pos[row], qd = a.dim + a.rot, half = a.rot >> 1;
  const T* c = (const T*)a.c + (size_t)row * a.stride;
  const T* cq = a.cq ? (const T*)a.cq + (size_t)row * a.stride : nullptr;
  const float2* cs = a.cs + (size_t)pos * half;
  float s[2] = {squares<T, V>(c, a.rank), cq ? squares<T, V>(cq, a.q_rank) : 0.f};
  const int per = a.rot / V;
  if (a.q) {
    T* p = (T*)a.q + (size_t)row * a.q_stride;
#pragma unroll 4
    for (int i = threadIdx.x; i < a.H * per; i += 128) {
      const int h = i / per;
      T* x = p + (size_t)h * qd + a.dim;
      turn_unit<T, V, HALVES>(x, x, i - h * per, half, cs);
    }
  }
  block_sums<2>(s, sh, phase);
  if (cq) normed<T, V>(cq, (T*)a.cqo + (size_t)row * a.q_rank, a.wq, a.q_rank, 1.f / sqrtf(s[1] / (float)a.q_rank + a.eps));
  const int page = a.table[(size_t)a.row_lane[row] * a.max_pages + pos / 64];
  if (page < 0 || page >= a.n_pages) {
    if (threadIdx.x == 0) status_set(a.status, ST_BOUNDS, 67, page, a.n_pages);
    return;
  }
  T* o = (T*)a.pool + ((size_t)page * 64 + pos % 64) * (a.rank + a.rot);
  normed<T, V>(c, o, a.w, a.rank, 1.f / sqrtf(s[0] / (float)a.rank + a.eps));
  for (int u = 127 - threadIdx.x; u < per; u += 128) turn_unit<T, V, HALVES>(c + a.rank, o + a.rank, u, half, cs);
}

// one thread per (row, head, unit)
template <typename T, int V, bool HALVES>
__global__ void __launch_bounds__(256) latent_turn_kernel(T* q, int64_t stride, const float2* cs, const int* row_pos, int n, int H, int dim, int rot) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = rot / V, half = rot >> 1;
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  const int row = (int)(i / (H * per)), j = (int)(i - (int64_t)row * (H * per)), h = j / per;
  if (row >= n) return;
  T* x = q + (size_t)row * stride + (size_t)h * (dim + rot) + dim;
  turn_unit<T, V, HALVES>(x, x, j - h * per, half, cs + (size_t)row_pos[row] * half);
}

struct HeadProjArgs {
  const void* x;            // (T) x of (row, head): row * x_row + head * x_head elements in
  int64_t x_row, x_head;
  const void* w;            // [H, K, M] (T)
  void* out;                // (T)
  int64_t out_row, out_head;
  const int* rows;          // row of x (x_list) or of out (out_list) for every launch row, or null: identity
  const float *part, *ml;   // or x is to be merged: [places, H, K] and (log2 maximum, sum) of every partial result
  const int2* parts;        // first place and number of places of every launch row
  int most;                 // at least the places of a row
  const int* row_pos;       // (cs)
  int x_list, out_list, n, H, K, M, tail;   // tail: elements after x's K that are copied after out's M
  const float2* cs;         // [positions, tail / 2]: the tail is turned (element i with i + tail / 2) by its row's position, or null
  const void* gate;         // (T) outputs are multiplied by sigmoid(gate[row of out][h M + m]), or null
  int64_t gate_row;
};
constexpr int HP_R = 4, HP_T = 256;                    // rows and threads per block

// MG threads x 8 outputs side by side, the others share K
template <typename T, int V, int MG>
__global__ void __launch_bounds__(HP_T) head_proj_kernel(HeadProjArgs a) {
  extern __shared__ __align__(16) float sm[];          // x [HP_R][K], then partials [KG][HP_R][HP_M] (before that: merge weights)
  constexpr int HP_M = MG * 8, KG = HP_T / MG, PRE = 8;
  float* xs = sm;
  float* red = sm + ((HP_R * a.K + 3) & ~3);
  const int tid = threadIdx.x, mg = tid % MG, kg = tid / MG;
  const int mt = (a.M + HP_M - 1) / HP_M, h = blockIdx.x / mt, m0 = (blockIdx.x % mt) * HP_M + mg * 8;
  const int r0 = blockIdx.y * HP_R, nr = min(HP_R, a.n - r0);
  const T* w = (const T*)a.w + (size_t)h * a.K * a.M + m0;
  auto weights = [&](int k, float (&f)[8]) {
    if constexpr (V == 8) load_v<T, 8>(w + (size_t)k * a.M, f);
    else {
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = m0 + j < a.M ? to_f<T>(w[(size_t)k * a.M + j]) : 0.f;
    }
  };
  // the first weights are requested before the previous kernel has finished: they do not depend on it
  float pre[PRE][8];
#pragma unroll
  for (int p = 0; p < PRE; ++p)
    if (m0 < a.M && kg + p * KG < a.K) weights(kg + p * KG, pre[p]);
  pdl_launch_dependents();
  pdl_wait();
  if (a.part) {
    __shared__ int wn[HP_R], w0[HP_R];
    float* wt = red;                                   // [HP_R][most], then the groups' sums [groups][HP_R][K]
    const int warp = tid >> 5, lane = tid & 31;
    if (warp < nr) {
      const int2 places = a.parts[r0 + warp];
      const int place = places.x, nb = places.y;
      const float* ml = a.ml + ((size_t)place * a.H + h) * 2;
      const size_t step = (size_t)a.H * 2;
      float m = -INFINITY, l = 0.f;
      for (int b = lane; b < nb; b += 32) m = fmaxf(m, ml[b * step]);
      m = warp_max(m);
      for (int b = lane; b < nb; b += 32) l += ml[b * step + 1] * exp2f(ml[b * step] - m);
      const float inv = 1.f / warp_sum(l);
      for (int b = lane; b < nb; b += 32) wt[warp * a.most + b] = exp2f(ml[b * step] - m) * inv;
      if (lane == 0) { wn[warp] = nb; w0[warp] = place; }
    }
    __syncthreads();
    // threads in groups of K / 4: a group per row, several on the places of a row where there are more groups than rows
    const int K4 = a.K >> 2, groups = HP_T / K4;       // K (the latent's size) is a multiple of eight, up to 512
    const int across = min(groups, nr), along = groups / across;
    const int grp = tid / K4, k = (tid - grp * K4) * 4, part0 = grp / across;
    float* gs = along > 1 ? red + ((HP_R * a.most + 3) & ~3) : xs;      // [along][HP_R][K]
    if (part0 < along) {
      for (int r = grp % across; r < nr; r += across) {
        float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
        const int nb = wn[r];
        const float* p = a.part + ((size_t)w0[r] * a.H + h) * a.K + k;
        const size_t step = (size_t)a.H * a.K;
#pragma unroll 8
        for (int b = part0; b < nb; b += along) {
          const float wb = wt[r * a.most + b];
          const float4 v = *reinterpret_cast<const float4*>(p + b * step);
          f.x = fmaf(wb, v.x, f.x); f.y = fmaf(wb, v.y, f.y); f.z = fmaf(wb, v.z, f.z); f.w = fmaf(wb, v.w, f.w);
        }
        *reinterpret_cast<float4*>(gs + (size_t)(part0 * HP_R + r) * a.K + k) = f;
      }
    }
    for (int i = nr * a.K + tid; i < HP_R * a.K; i += HP_T) xs[i] = 0.f;
    if (along > 1) {
      __syncthreads();
      for (int i = tid; i < nr * a.K; i += HP_T) {
        float f = 0.f;
        for (int q = 0; q < along; ++q) f += gs[(size_t)q * HP_R * a.K + i];
        xs[i] = f;
      }
    }
  } else {
    for (int i = tid; i < HP_R * a.K; i += HP_T) {
      const int r = i / a.K, k = i - r * a.K;
      float f = 0.f;
      if (r < nr) {
        const int row = a.rows && a.x_list ? a.rows[r0 + r] : r0 + r;
        f = to_f<T>(((const T*)a.x)[(size_t)row * a.x_row + (size_t)h * a.x_head + k]);
      }
      xs[i] = f;
    }
  }
  if (a.cs && blockIdx.x % mt == 0) {
    const int half = a.tail >> 1;
    for (int i = tid; i < nr * half; i += HP_T) {
      const int r = i / half, k = i - r * half;
      const int xr = a.rows && a.x_list ? a.rows[r0 + r] : r0 + r, orow = a.rows && a.out_list ? a.rows[r0 + r] : r0 + r;
      turn_unit<T, 2, true>((const T*)a.x + (size_t)xr * a.x_row + (size_t)h * a.x_head + a.K,
                            (T*)a.out + (size_t)orow * a.out_row + (size_t)h * a.out_head + a.M, k, half, a.cs + (size_t)a.row_pos[xr] * half);
    }
  } else if (a.tail && blockIdx.x % mt == 0) {
    for (int i = tid; i < nr * a.tail; i += HP_T) {
      const int r = i / a.tail, k = i - r * a.tail;
      const int xr = a.rows && a.x_list ? a.rows[r0 + r] : r0 + r, orow = a.rows && a.out_list ? a.rows[r0 + r] : r0 + r;
      ((T*)a.out)[(size_t)orow * a.out_row + (size_t)h * a.out_head + a.M + k] = ((const T*)a.x)[(size_t)xr * a.x_row + (size_t)h * a.x_head + a.K + k];
    }
  }
  __syncthreads();
  float acc[HP_R][8];
#pragma unroll
  for (int r = 0; r < HP_R; ++r)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[r][j] = 0.f;
  auto add = [&](int k, const float (&f)[8]) {
#pragma unroll
    for (int r = 0; r < HP_R; ++r) {
      const float xv = xs[r * a.K + k];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[r][j] = fmaf(xv, f[j], acc[r][j]);
    }
  };
  if (m0 < a.M) {
#pragma unroll
    for (int p = 0; p < PRE; ++p)
      if (kg + p * KG < a.K) add(kg + p * KG, pre[p]);
#pragma unroll 4
    for (int k = kg + PRE * KG; k < a.K; k += KG) {
      float f[8];
      weights(k, f);
      add(k, f);
    }
  }
#pragma unroll
  for (int r = 0; r < HP_R; ++r) {
    *reinterpret_cast<float4*>(red + ((size_t)kg * HP_R + r) * HP_M + mg * 8) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
    *reinterpret_cast<float4*>(red + ((size_t)kg * HP_R + r) * HP_M + mg * 8 + 4) = make_float4(acc[r][4], acc[r][5], acc[r][6], acc[r][7]);
  }
  __syncthreads();
  for (int i = tid; i < nr * HP_M; i += HP_T) {
    const int r = i / HP_M, c = i - r * HP_M, m = (blockIdx.x % mt) * HP_M + c;
    if (m >= a.M) continue;
    float t = 0.f;
#pragma unroll
    for (int q = 0; q < KG; ++q) t += red[((size_t)q * HP_R + r) * HP_M + c];
    const int row = a.rows && a.out_list ? a.rows[r0 + r] : r0 + r;
    if (a.gate) t *= gate_sigmoid<T>(to_f<T>(((const T*)a.gate)[(size_t)row * a.gate_row + (size_t)h * a.M + m]));
    ((T*)a.out)[(size_t)row * a.out_row + (size_t)h * a.out_head + m] = from_f<T>(t);
  }
}

__global__ void __launch_bounds__(256) gather_pages_kernel(const uint4* pool, const int* pages, uint4* out, int words, int n_pages, Status* status) {
  pdl_launch_dependents();
  pdl_wait();
  int page = pages[blockIdx.x];
  if (page < 0 || page >= n_pages) { if (threadIdx.x == 0) status_set(status, ST_BOUNDS, 68, page, n_pages); page = 0; }
  const uint4* s = pool + (size_t)page * words;
  uint4* d = out + (size_t)blockIdx.x * words;
#pragma unroll 4
  for (int i = blockIdx.y * 256 + threadIdx.x; i < words; i += gridDim.y * 256) d[i] = s[i];
}

template <typename T, int V, int MG>
static int launch_head_proj(const HeadProjArgs& a, cudaStream_t st) {
  const size_t red = (size_t)HP_T * HP_R * 8, wts = ((size_t)HP_R * a.most + 3) / 4 * 4 + HP_T * 4 * HP_R;
  const size_t smem = (((size_t)HP_R * a.K + 3) / 4 * 4 + (red > wts ? red : wts)) * sizeof(float);
  if (smem > 220 * 1024) return (int)cudaErrorInvalidValue;
  static size_t granted = 48 * 1024;
  if (smem > granted) {
    const cudaError_t e = cudaFuncSetAttribute(head_proj_kernel<T, V, MG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    granted = smem;
  }
  return (int)sfb_launch(head_proj_kernel<T, V, MG>, dim3(a.H * ((a.M + MG * 8 - 1) / (MG * 8)), (a.n + HP_R - 1) / HP_R), dim3(HP_T), smem, st, a);
}
template <typename T>
static int launch_head_proj_t(const HeadProjArgs& a, cudaStream_t st) {
  if (a.M % 8) return launch_head_proj<T, 1, 16>(a, st);
  // long sums: fewer outputs per block and more threads on each
  return a.K > 256 ? launch_head_proj<T, 8, 4>(a, st) : launch_head_proj<T, 8, 16>(a, st);
}

}  // namespace rows
}  // namespace sfb

using namespace sfb;
using namespace sfb::rows;

extern "C" {

// q null: the queries are turned elsewhere; cq: the queries' latent (normed to cqo), or null; halves: element i turns with i + rot / 2
int sfb_rows_latent_append(void* q, int64_t q_stride, const void* c, const void* cq, void* cqo, int64_t stride, const void* w, const void* wq, const void* cs, void* pool, const int* table,
                           const int* row_lane, const int* row_pos, int max_pages, int n_pages, int n, int H, int dim, int rot, int rank, int q_rank, int halves,
                           float eps, int fp32, void* status, cudaStream_t stream) {
  if (n < 1 || H < 1 || dim < 1 || rot < 0 || rot % 2 || rank < 1 || (cq && (q_rank < 1 || !cqo))) return (int)cudaErrorInvalidValue;
  LatentArgs a{q, q_stride, c, cq, cqo, stride, (const float*)w, (const float*)wq, (const float2*)cs, pool, table, row_lane, row_pos, max_pages, n_pages, H, dim, rot, rank,
               q_rank, eps, (Status*)status};
  const size_t part = fp32 ? 16 : 8;
  const bool v4 = (dim | rot | rank | (cq ? q_rank : 0)) % 4 == 0 && stride % 4 == 0 && (!q || q_stride % 4 == 0) && (uintptr_t)c % part == 0 && (uintptr_t)cq % part == 0;
  const dim3 g(n), b(128);
  if (halves) {
    if (fp32) return (int)(v4 ? sfb_launch(latent_append_kernel<float, 4, true>, g, b, 0, stream, a) : sfb_launch(latent_append_kernel<float, 2, true>, g, b, 0, stream, a));
    return (int)(v4 ? sfb_launch(latent_append_kernel<__nv_bfloat16, 4, true>, g, b, 0, stream, a)
                    : sfb_launch(latent_append_kernel<__nv_bfloat16, 2, true>, g, b, 0, stream, a));
  }
  if (fp32) return (int)(v4 ? sfb_launch(latent_append_kernel<float, 4, false>, g, b, 0, stream, a) : sfb_launch(latent_append_kernel<float, 2, false>, g, b, 0, stream, a));
  return (int)(v4 ? sfb_launch(latent_append_kernel<__nv_bfloat16, 4, false>, g, b, 0, stream, a)
                  : sfb_launch(latent_append_kernel<__nv_bfloat16, 2, false>, g, b, 0, stream, a));
}

// q [n, stride]: heads of dim + rot, the last rot of each turned in place (halves: element i with i + rot / 2, else neighbours)
int sfb_rows_latent_turn(void* q, int64_t stride, const void* cs, const int* row_pos, int n, int H, int dim, int rot, int halves, int fp32, cudaStream_t stream) {
  if (n < 1 || H < 1 || rot < 2 || rot % 2) return (int)cudaErrorInvalidValue;
  const int V = !halves || rot % 8 || dim % 4 || stride % 4 ? 2 : 8;
  const dim3 g((unsigned)(((int64_t)n * H * (rot / V) + 255) / 256)), b(256);
  const float2* t = (const float2*)cs;
  if (fp32) {
    float* f = (float*)q;
    return (int)(V == 8 ? sfb_launch(latent_turn_kernel<float, 8, true>, g, b, 0, stream, f, stride, t, row_pos, n, H, dim, rot)
                 : halves ? sfb_launch(latent_turn_kernel<float, 2, true>, g, b, 0, stream, f, stride, t, row_pos, n, H, dim, rot)
                          : sfb_launch(latent_turn_kernel<float, 2, false>, g, b, 0, stream, f, stride, t, row_pos, n, H, dim, rot));
  }
  __nv_bfloat16* f = (__nv_bfloat16*)q;
  return (int)(V == 8 ? sfb_launch(latent_turn_kernel<__nv_bfloat16, 8, true>, g, b, 0, stream, f, stride, t, row_pos, n, H, dim, rot)
               : halves ? sfb_launch(latent_turn_kernel<__nv_bfloat16, 2, true>, g, b, 0, stream, f, stride, t, row_pos, n, H, dim, rot)
                        : sfb_launch(latent_turn_kernel<__nv_bfloat16, 2, false>, g, b, 0, stream, f, stride, t, row_pos, n, H, dim, rot));
}

// list: 0 = rows ignored, 1 = it names x's rows, 2 = it names out's rows.  part (then x is null), cs, gate: see HeadProjArgs; with part, list
// is 2 or 0.
int sfb_rows_head_proj(const void* x, int64_t x_row, int64_t x_head, const void* w, void* out, int64_t out_row, int64_t out_head, const int* rows, int list,
                       const void* part, const void* ml, const void* parts, int most, const int* row_pos, int n, int H, int K, int M, int tail, const void* cs,
                       const void* gate, int64_t gate_row, int fp32, cudaStream_t stream) {
  if (n < 1 || n > 65535 * HP_R || H < 1 || K < 1 || M < 1 || K > 8192 || (part && (K % 8 || K > 512 || most < 1 || !parts || tail || list == 1)) ||
      (cs && (tail < 2 || tail % 2 || !row_pos)))
    return (int)cudaErrorInvalidValue;
  HeadProjArgs a{x, x_row, x_head, w, out, out_row, out_head, list ? rows : nullptr, (const float*)part, (const float*)ml, (const int2*)parts, part ? most : 0, row_pos,
                 list == 1, list == 2, n, H, K, M, tail, (const float2*)cs, gate, gate_row};
  return fp32 ? launch_head_proj_t<float>(a, stream) : launch_head_proj_t<__nv_bfloat16>(a, stream);
}

// bytes of a page: a multiple of 16
int sfb_rows_gather_pages(const void* pool, const int* pages, void* out, int count, int64_t page_bytes, int n_pages, void* status, cudaStream_t stream) {
  if (count < 1 || page_bytes < 16 || page_bytes % 16) return (int)cudaErrorInvalidValue;
  const int words = (int)(page_bytes / 16);
  return (int)sfb_launch(gather_pages_kernel, dim3(count, min(8, (words + 1023) / 1024)), dim3(256), 0, stream, (const uint4*)pool, pages, (uint4*)out, words,
                         n_pages, (Status*)status);
}

}  // extern "C"
