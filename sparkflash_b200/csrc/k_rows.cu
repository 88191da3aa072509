// Row kernels of the layered decoders (models/layered.py): everything of a layer between its matrix products except
// attention.  A step holds n rows of any mix of lanes; the rows of one lane are a *segment* (consecutive, in position order).
//
//   seam       residual += norm(sublayer output), then the next sublayer's norm, in one pass over a row; options: the output is
//              half the sum of two branches with an RMS norm each, or a weighted sum of several parts; it is scaled element by element
//              instead of normed; norms are layer norms or RMS norms; the row starts from the embedding table; a loop pass adds
//              the embedding output and a vector; a step of single-row segments also applies the input convolution; the embedding is
//              scaled; without a next norm h is the residual at activation precision.
//   conv       causal depthwise convolution with carried inputs, optionally added to its input or followed by silu, optionally with a
//              bias.
//   qk_append  RMS norm over a whole query / key projection, keys and values into the paged cache.
//   head_append  RMS norm of every query and key head with a weight that the heads share, keys and values into the paged cache.
//   rot_append rotated queries and keys, values mixed with another layer's, into the paged cache.
//   token_gate gelu(projection) * the token's row of a table.
//   gated scan real-gated linear recurrence S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with a = exp(-c r softplus(lam)):
//              two passes over chunks of rows for prompts (the chunks' start states in between), one fused kernel (convolution, gates, recurrence,
//              output gate) for single rows.
//   act_mul    act(gate) * up, act = silu, the tanh form of gelu, or the clamped gate.
//   act        the ungated activations: xIELU, the square of relu.
//
// Recurrent state (scan state, convolution inputs) has two versions per lane.  A segment reads version `src` (-1: zeros) and
// writes version `dst`, so every block of a launch sees the state before the step, a replayed graph repeats the same result,
// and a step can be undone by going back to `src`.
#include "k_rows_seam.cuh"

namespace sfb {
namespace rows {

// ---- seam ------------------------------------------------------------------------------------------------------------
struct SeamArgs {
  float* x;                 // [rows, d] residual, 32-bit
  const void* y;            // [rows, d] sublayer output (T) or null: no residual update
  const void* y2;           // second branch (T) or null
  const float *mw, *mw2;    // RMS weights of the two branches
  const float* parts_w;     // [rows, parts]: y is [rows, parts, d] and the output their weighted sum; or null
  const float *pw, *pb;     // post-norm (pb null: no bias), or the scale
  const void* embed;        // [vocab, d] (T)
  const int* tokens;        // [rows]
  const float* step_vec;    // [d] or null: added after the update
  float* tap;               // [rows, d] or null: the residual right after the update
  const float *nw, *nb;     // next norm, or null: h is the residual itself
  void* h;                  // [rows, d] (T) its output, or null
  const int* row_map;       // null: row = block; otherwise the residual row of output row `block`
  const float* cw;          // [taps, d] input convolution, or null
  void* hist;               // [slots, taps - 1, d] (T)
  const int *src, *dst;     // [rows] state versions of single-row segments
  int from_embed, add_embed, taps, d, vocab;
  int parts, post, rms;     // post: POST_*; rms: the next norm is an RMS norm
  float eps, embed_scale;
  Status* status;
};

constexpr int POST_LAYER = 0, POST_RMS = 1, POST_SCALE = 2;

// Mean and sum of squared deviations of a row held as x[NV][V] per thread (`wcnt` = how many of the elements are this warp's):
// each warp takes both about its own mean, then the warps' pairs are combined - one barrier.
template <int V, int NV>
__device__ __forceinline__ void row_moments(const float (&x)[NV][V], int c0, int step, int d, float wcnt, float winv, float inv_d, float* sh, int& phase,
                                            float& mu, float& m2) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  float* s = sh + (phase & 1) * 96;
  phase ^= 1;
  float t = 0.f, q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (c0 + i * step < d) {
#pragma unroll
      for (int k = 0; k < V; ++k) t += x[i][k];
    }
  const float wm = warp_sum(t) * winv;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (c0 + i * step < d) {
#pragma unroll
      for (int k = 0; k < V; ++k) { const float e = x[i][k] - wm; q += e * e; }
    }
  q = warp_sum(q);
  if (lane == 0) { s[w] = wm; s[32 + w] = q; s[64 + w] = wcnt; }
  __syncthreads();
  mu = m2 = 0.f;
  for (int i = 0; i < nw; ++i) mu += s[i] * s[64 + i];
  mu *= inv_d;
  for (int i = 0; i < nw; ++i) { const float e = s[i] - mu; m2 += s[32 + i] + s[64 + i] * e * e; }
}

// AHEAD (few rows): weights and the convolution's carried inputs are requested before they are needed, the former before the
// previous kernel has finished; with many rows that only costs registers.
template <typename T, int V, int NV, bool AHEAD>
__global__ void __launch_bounds__(NV < 8 ? 256 : 512, !AHEAD && NV == 4 ? 4 : 1) seam_kernel(SeamArgs a) {
  __shared__ float sh[2 * 96], sh2[2 * 2 * 32];
  int phase = 0, phase2 = 0;
  const int d = a.d, step = blockDim.x * V, c0 = threadIdx.x * V;
  const float inv_d = 1.f / (float)d;
  constexpr int TW = AHEAD ? 4 : 1;      // taps held ahead
  float pw[NV][V], pb[NV][V], nw[NV][V], nb[NV][V], cw[TW][NV][V], cg[TW][NV][V];
  const bool ahead_conv = AHEAD && a.cw && a.taps <= TW;
  if constexpr (AHEAD) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c >= d) continue;
#pragma unroll
      for (int k = 0; k < V; ++k) pb[i][k] = nb[i][k] = 0.f;
      if (a.y) { load_v<float, V>(a.pw + c, pw[i]); if (a.pb) load_v<float, V>(a.pb + c, pb[i]); }
      if (a.nw) { load_v<float, V>(a.nw + c, nw[i]); if (a.nb) load_v<float, V>(a.nb + c, nb[i]); }
      if (ahead_conv) {
#pragma unroll
        for (int j = 0; j < TW; ++j)
          if (j < a.taps) load_v<float, V>(a.cw + (size_t)j * d + c, cw[j][i]);
      }
    }
  }
  pdl_launch_dependents();
  pdl_wait();
  const int out_row = blockIdx.x, row = a.row_map ? a.row_map[out_row] : out_row;
  int mine = 0;
#pragma unroll
  for (int i = 0; i < NV; ++i) mine += max(0, min(V, d - (c0 + i * step)));
  const float wcnt = warp_sum((float)mine), winv = wcnt > 0.f ? 1.f / wcnt : 0.f;
  const int W = a.taps - 1;
  const int src = a.cw ? a.src[row] : -1;
  T* hd = a.cw ? (T*)a.hist + (size_t)a.dst[row] * W * d : nullptr;
  const T* hs = src >= 0 ? (const T*)a.hist + (size_t)src * W * d : nullptr;
  if constexpr (AHEAD) {
    if (ahead_conv) {
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int j = 0; j < TW - 1; ++j) {
          if (j < W && hs && c0 + i * step < d) load_v<T, V>(hs + (size_t)j * d + c0 + i * step, cg[j][i]);
          else {
#pragma unroll
            for (int k = 0; k < V; ++k) cg[j][i][k] = 0.f;
          }
        }
    }
  }
  float x[NV][V];
  const T* er = nullptr;
  if (a.from_embed || a.add_embed) {
    int tok = a.tokens[row];
    if (tok < 0 || tok >= a.vocab) { if (threadIdx.x == 0) status_set(a.status, ST_BOUNDS, 60, tok, a.vocab); tok = 0; }
    er = (const T*)a.embed + (size_t)tok * d;
  }
  float* xr = a.x + (size_t)row * d;
  if (!a.from_embed) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (c0 + i * step < d) load_v<float, V>(xr + c0 + i * step, x[i]);
  }
  if (a.y) {
    float y[NV][V];
    const T* yr = (const T*)a.y + (size_t)row * d;
    if (a.y2) {
      float s[2] = {0.f, 0.f};
      const T* zr = (const T*)a.y2 + (size_t)row * d;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (c0 + i * step < d) {
          float z[V];
          load_v<T, V>(yr + c0 + i * step, y[i]);
          load_v<T, V>(zr + c0 + i * step, z);
#pragma unroll
          for (int k = 0; k < V; ++k) { s[0] += y[i][k] * y[i][k]; s[1] += z[k] * z[k]; }
        }
      block_sums<2>(s, sh2, phase2);
      const float r0 = 0.5f / sqrtf(s[0] * inv_d + a.eps), r1 = 0.5f / sqrtf(s[1] * inv_d + a.eps);
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (c0 + i * step < d) {
          float w0[V], w1[V], z[V];
          load_v<T, V>(zr + c0 + i * step, z);           // again, out of L1
          load_v<float, V>(a.mw + c0 + i * step, w0);
          load_v<float, V>(a.mw2 + c0 + i * step, w1);
#pragma unroll
          for (int k = 0; k < V; ++k) y[i][k] = y[i][k] * r0 * w0[k] + z[k] * r1 * w1[k];
        }
    } else if (a.parts_w) {
      const float* wr = a.parts_w + (size_t)row * a.parts;
      yr = (const T*)a.y + (size_t)row * a.parts * d;
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int k = 0; k < V; ++k) y[i][k] = 0.f;
#pragma unroll 2
      for (int j = 0; j < a.parts; ++j) {
        const float wj = wr[j];
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (c0 + i * step < d) {
            float z[V];
            load_v<T, V>(yr + (size_t)j * d + c0 + i * step, z);
#pragma unroll
            for (int k = 0; k < V; ++k) y[i][k] = fmaf(wj, z[k], y[i][k]);
          }
      }
    } else {
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (c0 + i * step < d) load_v<T, V>(yr + c0 + i * step, y[i]);
    }
    float mu = 0.f, rs = 1.f;
    if (a.post != POST_SCALE) {
      float m2;
      row_moments<V, NV>(y, c0, step, d, wcnt, winv, inv_d, sh, phase, mu, m2);
      rs = 1.f / sqrtf((a.post == POST_RMS ? fmaf(mu, mu, m2 * inv_d) : m2 * inv_d) + a.eps);
      if (a.post == POST_RMS) mu = 0.f;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (c0 + i * step < d) {
        if constexpr (!AHEAD) {
          float w[V], b[V];
          load_v<float, V>(a.pw + c0 + i * step, w);
#pragma unroll
          for (int k = 0; k < V; ++k) b[k] = 0.f;
          if (a.pb) load_v<float, V>(a.pb + c0 + i * step, b);
#pragma unroll
          for (int k = 0; k < V; ++k) x[i][k] += (y[i][k] - mu) * rs * w[k] + b[k];
        } else {
#pragma unroll
          for (int k = 0; k < V; ++k) x[i][k] += (y[i][k] - mu) * rs * pw[i][k] + pb[i][k];
        }
        if (a.tap) store_v<float, V>(a.tap + (size_t)row * d + c0 + i * step, x[i]);
      }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (c0 + i * step < d) {
      if (er) {
        float e[V];
        load_v<T, V>(er + c0 + i * step, e);
#pragma unroll
        for (int k = 0; k < V; ++k) x[i][k] = a.from_embed ? e[k] * a.embed_scale : fmaf(e[k], a.embed_scale, x[i][k]);
      }
      if (a.step_vec) {
        float sv[V];
        load_v<float, V>(a.step_vec + c0 + i * step, sv);
#pragma unroll
        for (int k = 0; k < V; ++k) x[i][k] += sv[k];
      }
      store_v<float, V>(xr + c0 + i * step, x[i]);
      if (!a.nw && a.h) store_v<T, V>((T*)a.h + (size_t)out_row * d + c0 + i * step, x[i]);
    }
  if (!a.nw) return;
  float mu, m2;
  row_moments<V, NV>(x, c0, step, d, wcnt, winv, inv_d, sh, phase, mu, m2);
  const float rs = 1.f / sqrtf((a.rms ? fmaf(mu, mu, m2 * inv_d) : m2 * inv_d) + a.eps);
  if (a.rms) mu = 0.f;
  T* hr = (T*)a.h + (size_t)out_row * d;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = c0 + i * step;
    if (c >= d) continue;
    float o[V];
    if constexpr (!AHEAD) {
      load_v<float, V>(a.nw + c, nw[i]);
#pragma unroll
      for (int k = 0; k < V; ++k) nb[i][k] = 0.f;
      if (a.nb) load_v<float, V>(a.nb + c, nb[i]);
    }
#pragma unroll
    for (int k = 0; k < V; ++k) o[k] = (x[i][k] - mu) * rs * nw[i][k] + nb[i][k];
    if (a.cw) step_conv<T, V, TW, NV>(o, i, c, d, W, a.cw, hs, hd, ahead_conv, cw, cg);
    store_v<T, V>(hr + c, o);
  }
}

// ---- causal depthwise convolution over segments -------------------------------------------------------------------------
struct ConvRowsArgs {
  const void* x;            // [n, x_stride] (T)
  int64_t x_stride;
  const float* w;           // [taps, C], last = current row
  const float* bias;        // [C] or null
  void* y;                  // [n, C] (T)
  void* hist;               // [slots, taps - 1, C] (T), oldest first
  const int *row_seg, *seg_row0, *seg_len, *seg_src, *seg_dst;
  int n, C, mode;           // 1: y = x + conv(x), 2: y = silu(conv(x))
};
constexpr int CONV_RT = 8;  // most rows per block: their loads are all in flight before the first product

template <typename T, int V, int TAPS, int RT>
__global__ void __launch_bounds__(128) conv_rows_kernel(ConvRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= a.C) return;
  constexpr int W = TAPS - 1;
  const int r0 = blockIdx.y * RT, r1 = min(r0 + RT, a.n);
  const T* X = (const T*)a.x;
  float in[RT][V], w[TAPS][V], win[W > 0 ? W : 1][V], bias[V];
#pragma unroll
  for (int i = 0; i < RT; ++i)
    if (r0 + i < r1) load_v<T, V>(X + (size_t)(r0 + i) * a.x_stride + c, in[i]);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load_v<float, V>(a.w + (size_t)j * a.C + c, w[j]);
#pragma unroll
  for (int k = 0; k < V; ++k) bias[k] = 0.f;
  if (a.bias) load_v<float, V>(a.bias + c, bias);
  int seg = a.row_seg[r0], s0 = a.seg_row0[seg], s1 = s0 + a.seg_len[seg];
  {
    const int src = a.seg_src[seg];
#pragma unroll
    for (int j = 0; j < W; ++j) {         // win[j] = the input of row r0 - W + j
      const int r = r0 - W + j;
      if (r >= s0) load_v<T, V>(X + (size_t)r * a.x_stride + c, win[j]);
      else if (src >= 0) load_v<T, V>((const T*)a.hist + ((size_t)src * W + (W - (s0 - r))) * a.C + c, win[j]);
      else {
#pragma unroll
        for (int k = 0; k < V; ++k) win[j][k] = 0.f;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < RT; ++i) {
    const int r = r0 + i;
    if (r >= r1) break;
    if (r == s1) {                        // next segment: its window comes from its own state
      seg = a.row_seg[r]; s0 = r; s1 = s0 + a.seg_len[seg];
      const int src = a.seg_src[seg];
#pragma unroll
      for (int j = 0; j < W; ++j) {
        if (src >= 0) load_v<T, V>((const T*)a.hist + ((size_t)src * W + j) * a.C + c, win[j]);
        else {
#pragma unroll
          for (int k = 0; k < V; ++k) win[j][k] = 0.f;
        }
      }
    }
    float o[V];
#pragma unroll
    for (int k = 0; k < V; ++k) {
      float acc = bias[k] + w[W][k] * in[i][k];
#pragma unroll
      for (int j = 0; j < W; ++j) acc += w[j][k] * win[j][k];
      o[k] = a.mode == 1 ? in[i][k] + acc : a.mode == 2 ? acc * gate_sigmoid<T>(acc) : acc;
    }
    store_v<T, V>((T*)a.y + (size_t)r * a.C + c, o);
#pragma unroll
    for (int j = 0; j < W; ++j) {
#pragma unroll
      for (int k = 0; k < V; ++k) win[j][k] = j + 1 < W ? win[j + 1 < W ? j + 1 : j][k] : in[i][k];
    }
    if (r == s1 - 1) {
      const int dst = a.seg_dst[seg];
#pragma unroll
      for (int j = 0; j < W; ++j) store_v<T, V>((T*)a.hist + ((size_t)dst * W + j) * a.C + c, win[j]);
    }
  }
}

// ---- query / key norm over the whole projection, cache append -------------------------------------------------------------
struct QkAppendArgs {
  const void* proj;         // [n, stride] (T): q at 0, k at HD, v at HD + GD
  int64_t stride;
  const float *qw, *kw;     // [HD], [GD]
  void* q;                  // [n, HD] (T)
  void *kpool, *vpool;      // [pages, G, 64, dim] / [pages, G, 64, vdim] (T)
  const int* table;         // [lanes, max_pages]
  const int *row_lane, *row_pos;
  int max_pages, n_pages, H, G, dim, vdim;
  float eps;
  Status* status;
};
constexpr int PAGE = 64;

template <typename T, int V>
__global__ void __launch_bounds__(256) qk_append_kernel(QkAppendArgs a) {
  __shared__ float sh[2 * 2 * 32];
  int phase = 0;
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  const int HD = a.H * a.dim, GD = a.G * a.dim, GV = a.G * a.vdim;
  const T* p = (const T*)a.proj + (size_t)row * a.stride;
  float s[2] = {0.f, 0.f};
  for (int c = threadIdx.x * V; c < HD + GD; c += blockDim.x * V) {
    float f[V];
    load_v<T, V>(p + c, f);
    float t = 0.f;
#pragma unroll
    for (int k = 0; k < V; ++k) t += f[k] * f[k];
    if (c < HD) s[0] += t; else s[1] += t;
  }
  block_sums<2>(s, sh, phase);
  const float rq = 1.f / sqrtf(s[0] / (float)HD + a.eps), rk = 1.f / sqrtf(s[1] / (float)GD + a.eps);
  const int pos = a.row_pos[row];
  const int page = a.table[(size_t)a.row_lane[row] * a.max_pages + pos / PAGE], slot = pos % PAGE;
  const bool ok = page >= 0 && page < a.n_pages;
  if (!ok && threadIdx.x == 0) status_set(a.status, ST_BOUNDS, 61, page, a.n_pages);
  for (int c = threadIdx.x * V; c < HD + GD + GV; c += blockDim.x * V) {
    float f[V], w[V];
    load_v<T, V>(p + c, f);
    if (c < HD) {
      load_v<float, V>(a.qw + c, w);
#pragma unroll
      for (int k = 0; k < V; ++k) f[k] = f[k] * rq * w[k];
      store_v<T, V>((T*)a.q + (size_t)row * HD + c, f);
    } else if (c < HD + GD) {
      const int cc = c - HD, g = cc / a.dim, x = cc - g * a.dim;
      load_v<float, V>(a.kw + cc, w);
#pragma unroll
      for (int k = 0; k < V; ++k) f[k] = f[k] * rk * w[k];
      if (ok) store_v<T, V>((T*)a.kpool + (((size_t)page * a.G + g) * PAGE + slot) * a.dim + x, f);
    } else {
      const int cc = c - HD - GD, g = cc / a.vdim, x = cc - g * a.vdim;
      if (ok) store_v<T, V>((T*)a.vpool + (((size_t)page * a.G + g) * PAGE + slot) * a.vdim + x, f);
    }
  }
}

// ---- query / key norm head by head, cache append ---------------------------------------------------------------------------
// Lanes in groups of `per` (a power of two) own a head each; a lane holds NV times V of its elements.  The other lanes copy the values.
template <typename T, int V, int NV>
__global__ void __launch_bounds__(256) head_append_kernel(QkAppendArgs a, int per) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, HG = a.H + a.G, GV = a.G * a.vdim;
  const T* p = (const T*)a.proj + (size_t)row * a.stride;
  const int pos = a.row_pos[row];
  const int page = a.table[(size_t)a.row_lane[row] * a.max_pages + pos / PAGE], slot = pos % PAGE;
  const bool ok = page >= 0 && page < a.n_pages;
  if (!ok && threadIdx.x == 0) status_set(a.status, ST_BOUNDS, 78, page, a.n_pages);
  const int groups = 32 / per, at = lane & (per - 1);
  const float inv_d = 1.f / (float)a.dim;
  for (int h0 = warp * groups; h0 < HG; h0 += 8 * groups) {        // the same for every lane of the warp
    const int h = h0 + lane / per;
    const T* src = p + (size_t)h * a.dim;
    float f[NV][V], w[NV][V], t = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * per + at) * V;
      if (h < HG && c < a.dim) {
        load_v<T, V>(src + c, f[i]);
        load_v<float, V>((h < a.H ? a.qw : a.kw) + c, w[i]);
#pragma unroll
        for (int k = 0; k < V; ++k) t = fmaf(f[i][k], f[i][k], t);
      }
    }
    for (int o = 1; o < per; o <<= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
    const float r = 1.f / sqrtf(t * inv_d + a.eps);
    if (h >= HG || (h >= a.H && !ok)) continue;
    T* dst = h < a.H ? (T*)a.q + ((size_t)row * a.H + h) * a.dim : (T*)a.kpool + (((size_t)page * a.G + h - a.H) * PAGE + slot) * a.dim;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * per + at) * V;
      if (c >= a.dim) continue;
#pragma unroll
      for (int k = 0; k < V; ++k) f[i][k] *= r * w[i][k];
      store_v<T, V>(dst + c, f[i]);
    }
  }
  if (!ok) return;
  for (int c = (255 - threadIdx.x) * V; c < GV; c += 256 * V) {
    const int g = c / a.vdim, x = c - g * a.vdim;
    float f[V];
    load_v<T, V>(p + (size_t)HG * a.dim + c, f);
    store_v<T, V>((T*)a.vpool + (((size_t)page * a.G + g) * PAGE + slot) * a.vdim + x, f);
  }
}

// ---- rotated queries and keys, mixed values, cache append -------------------------------------------------------------------
struct RotAppendArgs {
  const void* proj;         // [n, stride] (T): q, k, v side by side
  int64_t stride;
  const float2* cs;         // [positions, half] (cos, sin)
  void* q;                  // [n, H dim] (T)
  void *kpool, *vpool;      // [pages, G, 64, dim] / [pages, G, 64, vdim] (T)
  void* v_first;            // [n, G vdim] (T) or null: values of the layer that the others mix with
  const float* lam;         // its share, or null: this layer is that one and leaves its values there
  const int* table;
  const int *row_lane, *row_pos;
  int max_pages, n_pages, H, G, dim, vdim, half;
  Status* status;
};

template <typename T, int V>
__global__ void __launch_bounds__(256) rot_append_kernel(RotAppendArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, HG = a.H + a.G, GV = a.G * a.vdim;
  const T* p = (const T*)a.proj + (size_t)row * a.stride;
  const int pos = a.row_pos[row];
  const int page = a.table[(size_t)a.row_lane[row] * a.max_pages + pos / PAGE], slot = pos % PAGE;
  const bool ok = page >= 0 && page < a.n_pages;
  if (!ok && threadIdx.x == 0) status_set(a.status, ST_BOUNDS, 71, page, a.n_pages);
  const float2* cs = a.cs + (size_t)pos * a.half;
  // a head's units: V pairs of dims that turn together, then V dims that pass
  const int turn = a.half / V, units = turn + (a.dim - 2 * a.half) / V;
  for (int u = threadIdx.x; u < HG * units + GV / V; u += blockDim.x) {
    if (u < HG * units) {
      const int h = u / units, i = u - h * units;
      const T* src = p + (size_t)h * a.dim;
      T* dst = h < a.H ? (T*)a.q + ((size_t)row * a.H + h) * a.dim : (T*)a.kpool + (((size_t)page * a.G + h - a.H) * PAGE + slot) * a.dim;
      if (h >= a.H && !ok) continue;
      if (i < turn) {
        float x[V], y[V], c[2 * V];
        const int d = i * V;
        load_v<T, V>(src + d, x);
        load_v<T, V>(src + a.half + d, y);
        if constexpr (V == 1) { const float2 t = cs[d]; c[0] = t.x; c[1] = t.y; }
        else {
#pragma unroll
          for (int k = 0; k < V / 2; ++k) load_v<float, 4>(reinterpret_cast<const float*>(cs + d + 2 * k), c + 4 * k);
        }
#pragma unroll
        for (int k = 0; k < V; ++k) {
          const float t = x[k];
          x[k] = t * c[2 * k] - y[k] * c[2 * k + 1];
          y[k] = y[k] * c[2 * k] + t * c[2 * k + 1];
        }
        store_v<T, V>(dst + d, x);
        store_v<T, V>(dst + a.half + d, y);
      } else {
        const int d = 2 * a.half + (i - turn) * V;
        float x[V];
        load_v<T, V>(src + d, x);
        store_v<T, V>(dst + d, x);
      }
    } else {
      const int c = (u - HG * units) * V, g = c / a.vdim, d = c - g * a.vdim;
      float x[V];
      load_v<T, V>(p + (size_t)HG * a.dim + c, x);
      if (a.lam) {
        const float lam = *a.lam;
        float f[V];
        load_v<T, V>((const T*)a.v_first + (size_t)row * GV + c, f);
#pragma unroll
        for (int k = 0; k < V; ++k) x[k] = (1.f - lam) * x[k] + lam * f[k];
      } else if (a.v_first) {
        store_v<T, V>((T*)a.v_first + (size_t)row * GV + c, x);
      }
      if (ok) store_v<T, V>((T*)a.vpool + (((size_t)page * a.G + g) * PAGE + slot) * a.vdim + d, x);
    }
  }
}

// ---- gelu(projection) * a part of the token's row of a table ----------------------------------------------------------------
template <typename T, int V>
__global__ void __launch_bounds__(256) token_gate_kernel(const T* z, const T* table, const int* tokens, T* out, int n, int dim, int64_t table_stride, int col0, int vocab,
                                                         Status* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = dim / V;
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  const int row = (int)(i / per), c = (int)(i - (int64_t)row * per) * V;
  if (row >= n) return;
  int tok = tokens[row];
  if (tok < 0 || tok >= vocab) { status_set(status, ST_BOUNDS, 72, tok, vocab); tok = 0; }
  float f[V], e[V];
  load_v<T, V>(z + (size_t)row * dim + c, f);
  load_v<T, V>(table + (size_t)tok * table_stride + col0 + c, e);
#pragma unroll
  for (int k = 0; k < V; ++k) f[k] = gate_gelu<T>(f[k]) * e[k];
  store_v<T, V>(out + (size_t)row * dim + c, f);
}
template <typename T, int V>
static int launch_token_gate(const void* z, const void* table, const int* tokens, void* out, int n, int dim, int64_t table_stride, int col0, int vocab, Status* status,
                             cudaStream_t st) {
  const int64_t blocks = ((int64_t)n * (dim / V) + 255) / 256;
  return (int)sfb_launch(token_gate_kernel<T, V>, dim3((unsigned)blocks), dim3(256), 0, st, (const T*)z, (const T*)table, tokens, (T*)out, n, dim, table_stride, col0,
                         vocab, status);
}

// ---- real-gated linear recurrence -------------------------------------------------------------------------------------------
struct ScanArgs {
  const float* gates;       // [blocks, n, 2 bs]: pre-activations of r, then of i; the two-pass form leaves a and b there
  const float *rb, *ib;     // [width] gate biases
  const float* decay;       // [width] c * softplus(lam)
  const void* u;            // [n, width] (T)
  const void* y;            // [n, y_stride] (T) output branch before its gelu
  int64_t y_stride;
  void* out;                // [n, width] (T)
  float* S;                 // [slots, width]
  float2* sums;             // [chunks, width] (product of a, end value from a zero start), then (start state, -)
  const int *chunk_seg, *chunk_row0, *chunk_rows, *chunk_first;   // chunk_first: first chunk of the same segment
  const int *seg_src, *seg_dst, *seg_row0, *seg_len;
  int n, width, bs, chunks;
};

// 1 - exp(t) for t <= 0: a polynomial near 0, where 1 - exp would cancel (Taylor, remainder below 2^-25 of the result)
__device__ __forceinline__ float one_minus_exp(float t, float e) {
  float p = 1.f / 40320.f;
  p = fmaf(p, t, 1.f / 5040.f); p = fmaf(p, t, 1.f / 720.f); p = fmaf(p, t, 1.f / 120.f); p = fmaf(p, t, 1.f / 24.f);
  p = fmaf(p, t, 1.f / 6.f); p = fmaf(p, t, 0.5f); p = fmaf(p, t, 1.f);
  return t > -0.5f ? -t * p : 1.f - e;
}
// decay a and input b of one step from the gate pre-activations
template <typename T> __device__ __forceinline__ void gate_step(float zr, float zi, float decay, float u, float& a, float& b) {
  const float la = -decay * gate_sigmoid<T>(zr);
  if constexpr (sizeof(T) == 4) a = expf(la);
  else a = __expf(la);
  const float m = one_minus_exp(2.f * la, a * a);
  if constexpr (sizeof(T) == 4) b = sqrtf(m) * (gate_sigmoid<T>(zi) * u);
  else {
    float r;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(r) : "f"(m));
    b = r * (gate_sigmoid<T>(zi) * u);
  }
}
// One chunk per segment: gates, recurrence and output gate in one pass.
template <typename T>
__global__ void __launch_bounds__(128) scan_short_kernel(ScanArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= a.width) return;
  const int ch = blockIdx.y, seg = a.chunk_seg[ch], row0 = a.chunk_row0[ch], rows = a.chunk_rows[ch];
  const int src = a.seg_src[seg];
  float S = src >= 0 ? a.S[(size_t)src * a.width + c] : 0.f;
  const int b = c / a.bs, j = c - b * a.bs;
  const float* g = a.gates + ((size_t)b * a.n + row0) * 2 * a.bs + j;
  const T* U = (const T*)a.u + (size_t)row0 * a.width + c;
  const T* Y = (const T*)a.y + (size_t)row0 * a.y_stride + c;
  T* O = (T*)a.out + (size_t)row0 * a.width + c;
  const float rb = a.rb[c], ib = a.ib[c], dec = a.decay[c];
#pragma unroll 4
  for (int t = 0; t < rows; ++t) {
    float at, bt;
    gate_step<T>(g[(size_t)t * 2 * a.bs] + rb, g[(size_t)t * 2 * a.bs + a.bs] + ib, dec, to_f<T>(U[(size_t)t * a.width]), at, bt);
    S = fmaf(at, S, bt);
    O[(size_t)t * a.width] = from_f<T>(S * gate_gelu<T>(to_f<T>(Y[(size_t)t * a.y_stride])));
  }
  a.S[(size_t)a.seg_dst[seg] * a.width + c] = S;
}

// Longer segments, pass 1: (a, b) of every step, in place of the gate pre-activations, and every chunk's summary.
constexpr int SCAN_T = 8;    // rows whose loads are in flight together
template <typename T>
__device__ __forceinline__ void chunk_gates(const ScanArgs& a, int c) {
  const int ch = blockIdx.y, row0 = a.chunk_row0[ch], rows = a.chunk_rows[ch];
  const int b = c / a.bs, j = c - b * a.bs;
  float* g = const_cast<float*>(a.gates) + ((size_t)b * a.n + row0) * 2 * a.bs + j;
  const T* U = (const T*)a.u + (size_t)row0 * a.width + c;
  const float rb = a.rb[c], ib = a.ib[c], dec = a.decay[c];
  float S = 0.f, P = 1.f;
  for (int t0 = 0; t0 < rows; t0 += SCAN_T) {
    float zr[SCAN_T], zi[SCAN_T], u[SCAN_T];
#pragma unroll
    for (int i = 0; i < SCAN_T; ++i)
      if (t0 + i < rows) {
        const float* gp = g + (size_t)(t0 + i) * 2 * a.bs;
        zr[i] = gp[0]; zi[i] = gp[a.bs]; u[i] = to_f<T>(U[(size_t)(t0 + i) * a.width]);
      }
#pragma unroll
    for (int i = 0; i < SCAN_T; ++i)
      if (t0 + i < rows) {
        float at, bt;
        gate_step<T>(zr[i] + rb, zi[i] + ib, dec, u[i], at, bt);
        float* gp = g + (size_t)(t0 + i) * 2 * a.bs;
        gp[0] = at; gp[a.bs] = bt;
        S = fmaf(at, S, bt);
        P *= at;
      }
  }
  a.sums[(size_t)ch * a.width + c] = make_float2(P, S);
}

template <typename T>
__global__ void __launch_bounds__(128) scan_gates_kernel(ScanArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c < a.width) chunk_gates<T>(a, c);
}

// Start state of every chunk and the segments' final states.  A chunk maps its start state S to P S + E; these maps compose, so a
// column's chunks are shared by START_G threads: each composes its own run of chunks, takes its start from the runs before it,
// and goes over its run again.
constexpr int START_G = 16, START_B = 8;
__global__ void __launch_bounds__(32 * START_G) scan_starts_kernel(ScanArgs a) {
  __shared__ float mp[START_G][32], me[START_G][32];
  pdl_launch_dependents();
  pdl_wait();
  const int x = threadIdx.x, g = threadIdx.y, c = blockIdx.x * 32 + x;
  const bool on = c < a.width;
  const int per = (a.chunks + START_G - 1) / START_G, k0 = g * per, k1 = min(k0 + per, a.chunks);
  float2 t[START_B];
  float P = 1.f, E = 0.f;
  for (int pass = 0; pass < 2; ++pass) {
    float S = 0.f;
    if (pass) {
      for (int q = 0; q < g; ++q) S = fmaf(mp[q][x], S, me[q][x]);
    }
    for (int kb = k0; kb < k1; kb += START_B) {
      int seg[START_B + 1];
      if (pass == 0 || per > START_B) {
#pragma unroll
        for (int i = 0; i < START_B; ++i)
          if (on && kb + i < k1) t[i] = a.sums[(size_t)(kb + i) * a.width + c];
      }
#pragma unroll
      for (int i = 0; i <= START_B; ++i) seg[i] = kb + i < a.chunks ? a.chunk_first[kb + i] : kb + i;      // its own index: a segment begins
#pragma unroll
      for (int i = 0; i < START_B; ++i) {
        const int k = kb + i;
        if (k >= k1 || !on) break;
        if (seg[i] == k) {
          const int src = a.seg_src[a.chunk_seg[k]];
          S = src >= 0 ? a.S[(size_t)src * a.width + c] : 0.f;
          P = 0.f; E = S;
        }
        if (pass) a.sums[(size_t)k * a.width + c].x = S;
        S = fmaf(t[i].x, S, t[i].y);
        P *= t[i].x;
        E = fmaf(t[i].x, E, t[i].y);
        if (pass && seg[i + 1] == k + 1) a.S[(size_t)a.seg_dst[a.chunk_seg[k]] * a.width + c] = S;
      }
    }
    if (!pass) {
      mp[g][x] = P; me[g][x] = E;
      __syncthreads();
    }
  }
}

// Pass 2: the recurrence from the chunk's start state, and the output gate.
template <typename T>
__global__ void __launch_bounds__(128) scan_apply_kernel(ScanArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= a.width) return;
  const int ch = blockIdx.y, row0 = a.chunk_row0[ch], rows = a.chunk_rows[ch];
  float S = a.sums[(size_t)ch * a.width + c].x;
  const int b = c / a.bs, j = c - b * a.bs;
  const float* g = a.gates + ((size_t)b * a.n + row0) * 2 * a.bs + j;
  const T* Y = (const T*)a.y + (size_t)row0 * a.y_stride + c;
  T* O = (T*)a.out + (size_t)row0 * a.width + c;
  float at[SCAN_T], bt[SCAN_T], y[SCAN_T];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < SCAN_T; ++i)
      if (t0 + i < rows) {
        const float* gp = g + (size_t)(t0 + i) * 2 * a.bs;
        at[i] = gp[0]; bt[i] = gp[a.bs]; y[i] = to_f<T>(Y[(size_t)(t0 + i) * a.y_stride]);
      }
  };
  for (int t0 = 0; t0 < rows; t0 += SCAN_T) {
    fetch(t0);
#pragma unroll
    for (int i = 0; i < SCAN_T; ++i)
      if (t0 + i < rows) {
        S = fmaf(at[i], S, bt[i]);
        O[(size_t)(t0 + i) * a.width] = from_f<T>(S * gate_gelu<T>(y[i]));
      }
  }
}

// Single-row segments: convolution, gates, recurrence and output gate of one part of the width in one kernel.
// grid (parts * tiles, row groups of RB); 8 warps, a warp owns one output channel at a time.
struct GatedRowArgs {
  const void* x;            // [n, x_stride] (T) convolution input
  const void* y;            // [n, y_stride] (T)
  int64_t x_stride, y_stride;
  const float *cw, *cb;     // [taps, width], [width]
  void* hist;               // [slots, taps - 1, width] (T)
  const void* wg;           // [parts, 2 bs, bs] (T): rows of r, then rows of i
  const float *rb, *ib, *decay;
  float* S;
  void* out;                // [n, width] (T)
  const int *src, *dst;     // [n]
  int n, width, bs, taps, tiles, per_tile;
};
constexpr int GATED_RB = 4;

template <typename T, int V>
__global__ void __launch_bounds__(256, 2) gated_row_kernel(GatedRowArgs a) {
  extern __shared__ float us[];             // [RB][bs rounded up to 8]
  const int part = blockIdx.x / a.tiles, tile = blockIdx.x % a.tiles;
  const int r0 = blockIdx.y * GATED_RB, nr = min(GATED_RB, a.n - r0);
  const int W = a.taps - 1, ld = (a.bs + 7) & ~7;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int j0 = tile * a.per_tile + warp, j1 = min((tile + 1) * a.per_tile, a.bs);
  // the first weight rows are requested before the previous kernel has finished: they do not depend on it
  float wr0[V], wi0[V];
  const bool pre = V == 8 && j0 < j1 && lane * V < a.bs;
  if (pre) {
    const T* w = (const T*)a.wg + ((size_t)part * 2 * a.bs + j0) * a.bs + lane * V;
    if constexpr (V == 8) { load_v<T, 8>(w, wr0); load_v<T, 8>(w + (size_t)a.bs * a.bs, wi0); }
  }
  pdl_launch_dependents();
  pdl_wait();
  for (int idx = threadIdx.x; idx < GATED_RB * a.bs; idx += blockDim.x) {
    const int i = idx / a.bs, j = idx - i * a.bs, c = part * a.bs + j;
    float acc = 0.f;
    if (i < nr) {
      const int row = r0 + i, src = a.src[row];
      const T xt = ((const T*)a.x)[(size_t)row * a.x_stride + c];
      acc = a.cb[c] + a.cw[(size_t)W * a.width + c] * to_f<T>(xt);
      T* hd = (T*)a.hist + (size_t)a.dst[row] * W * a.width + c;
      const T* hs = (const T*)a.hist + (size_t)(src >= 0 ? src : 0) * W * a.width + c;
      for (int k = 0; k < W; ++k) {
        const T g = src >= 0 ? hs[(size_t)k * a.width] : from_f<T>(0.f);
        acc += a.cw[(size_t)k * a.width + c] * to_f<T>(g);
        if (tile == 0 && k > 0) hd[(size_t)(k - 1) * a.width] = g;
      }
      if (tile == 0 && W > 0) hd[(size_t)(W - 1) * a.width] = xt;
      acc = to_f<T>(from_f<T>(acc));        // activation precision, as the many-row convolution stores it
    }
    us[i * ld + j] = acc;
  }
  __syncthreads();
  for (int j = j0; j < j1; j += 8) {
    const T* wr = (const T*)a.wg + ((size_t)part * 2 * a.bs + j) * a.bs;
    const T* wi = wr + (size_t)a.bs * a.bs;
    float dr[GATED_RB], di[GATED_RB];
#pragma unroll
    for (int i = 0; i < GATED_RB; ++i) dr[i] = di[i] = 0.f;
    for (int k = lane * V; k < a.bs; k += 32 * V) {
      float fr[V], fi[V];
      if (V == 8 && j == j0 && k == lane * V) {
#pragma unroll
        for (int v = 0; v < V; ++v) { fr[v] = wr0[v]; fi[v] = wi0[v]; }
      } else if constexpr (V == 8) { load_v<T, 8>(wr + k, fr); load_v<T, 8>(wi + k, fi); }
      else { load_v<T, 1>(wr + k, fr); load_v<T, 1>(wi + k, fi); }
#pragma unroll
      for (int i = 0; i < GATED_RB; ++i) {
#pragma unroll
        for (int v = 0; v < V; ++v) { dr[i] += fr[v] * us[i * ld + k + v]; di[i] += fi[v] * us[i * ld + k + v]; }
      }
    }
    float zr = 0.f, zi = 0.f;
#pragma unroll
    for (int i = 0; i < GATED_RB; ++i) {
      const float a0 = warp_sum(dr[i]), b0 = warp_sum(di[i]);
      if (lane == i) { zr = a0; zi = b0; }
    }
    if (lane < nr) {
      const int row = r0 + lane, c = part * a.bs + j, src = a.src[row];
      float at, bt;
      gate_step<T>(zr + a.rb[c], zi + a.ib[c], a.decay[c], us[lane * ld + j], at, bt);
      const float S = fmaf(at, src >= 0 ? a.S[(size_t)src * a.width + c] : 0.f, bt);
      a.S[(size_t)a.dst[row] * a.width + c] = S;
      ((T*)a.out)[(size_t)row * a.width + c] = from_f<T>(S * gate_gelu<T>(to_f<T>(((const T*)a.y)[(size_t)row * a.y_stride + c])));
    }
  }
}

// ---- act(gate) * up --------------------------------------------------------------------------------------------------------
template <typename T, int V>
__global__ void __launch_bounds__(256) act_mul_kernel(const T* gu, T* out, int ff, int64_t out_stride, int act, float alpha, float limit) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= ff) return;
  const size_t row = blockIdx.x;
  float g[V], u[V];
  load_v<T, V>(gu + row * 2 * ff + c, g);
  load_v<T, V>(gu + row * 2 * ff + ff + c, u);
#pragma unroll
  for (int k = 0; k < V; ++k)
    g[k] = act == ACT_CLAMP ? gate_clamp<T>(g[k], u[k], alpha, limit) : (act == ACT_GELU ? gate_gelu<T>(g[k]) : g[k] * gate_sigmoid<T>(g[k])) * u[k];
  store_v<T, V>(out + row * out_stride + c, g);
}

// ---- ungated activations ---------------------------------------------------------------------------------------------------
constexpr int ACT_U = 2;    // groups of V per thread, requested together
template <typename T, int V>
__global__ void __launch_bounds__(256) act_kernel(const T* z, T* out, int64_t count, int act, float p0, float p1) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t c0 = ((int64_t)blockIdx.x * ACT_U * blockDim.x + threadIdx.x) * V;
  float f[ACT_U][V];
#pragma unroll
  for (int u = 0; u < ACT_U; ++u)
    if (c0 + (int64_t)u * 256 * V < count) load_v<T, V>(z + c0 + (int64_t)u * 256 * V, f[u]);
#pragma unroll
  for (int u = 0; u < ACT_U; ++u) {
    const int64_t c = c0 + (int64_t)u * 256 * V;
    if (c >= count) break;
#pragma unroll
    for (int k = 0; k < V; ++k) f[u][k] = act_single<T>(f[u][k], act, p0, p1);
    store_v<T, V>(out + c, f[u]);
  }
}

// ---- dispatch ---------------------------------------------------------------------------------------------------------------
template <typename T, int V>
static int launch_seam(const SeamArgs& a, int n, cudaStream_t st) {
  const int vecs = (a.d + V - 1) / V;
  const bool few = n <= 296;
  int nv = 1;                              // few rows: many threads per row; many rows: more of the row per thread
  while (nv < 8 && (vecs + nv - 1) / nv > (few ? 256 : nv < 4 ? 128 : 256)) nv *= 2;
  const int threads = ((vecs + nv - 1) / nv + 31) / 32 * 32;
  if (threads > 512) return (int)cudaErrorInvalidValue;
  const dim3 g(n), b(threads);
  switch (nv) {
    case 1: return (int)(few ? sfb_launch(seam_kernel<T, V, 1, true>, g, b, 0, st, a) : sfb_launch(seam_kernel<T, V, 1, false>, g, b, 0, st, a));
    case 2: return (int)(few ? sfb_launch(seam_kernel<T, V, 2, true>, g, b, 0, st, a) : sfb_launch(seam_kernel<T, V, 2, false>, g, b, 0, st, a));
    case 4: return (int)sfb_launch(seam_kernel<T, V, 4, false>, g, b, 0, st, a);
    default: return (int)sfb_launch(seam_kernel<T, V, 8, false>, g, b, 0, st, a);
  }
}
template <typename T, int V, int RT>
static int launch_conv_rt(const ConvRowsArgs& a, int taps, cudaStream_t st) {
  const dim3 g((a.C + 128 * V - 1) / (128 * V), (a.n + RT - 1) / RT), b(128);
  switch (taps) {
    case 1: return (int)sfb_launch(conv_rows_kernel<T, V, 1, RT>, g, b, 0, st, a);
    case 2: return (int)sfb_launch(conv_rows_kernel<T, V, 2, RT>, g, b, 0, st, a);
    case 3: return (int)sfb_launch(conv_rows_kernel<T, V, 3, RT>, g, b, 0, st, a);
    case 4: return (int)sfb_launch(conv_rows_kernel<T, V, 4, RT>, g, b, 0, st, a);
    case 5: return (int)sfb_launch(conv_rows_kernel<T, V, 5, RT>, g, b, 0, st, a);
    case 6: return (int)sfb_launch(conv_rows_kernel<T, V, 6, RT>, g, b, 0, st, a);
    case 7: return (int)sfb_launch(conv_rows_kernel<T, V, 7, RT>, g, b, 0, st, a);
    case 8: return (int)sfb_launch(conv_rows_kernel<T, V, 8, RT>, g, b, 0, st, a);
    default: return (int)cudaErrorInvalidValue;
  }
}
template <typename T, int V>
static int launch_conv(const ConvRowsArgs& a, int taps, cudaStream_t st) {
  // few rows are mostly decoded ones, each with its own carried inputs: side by side instead of one after another
  return a.n <= 128 ? launch_conv_rt<T, V, 1>(a, taps, st) : launch_conv_rt<T, V, CONV_RT>(a, taps, st);
}

}  // namespace rows
}  // namespace sfb

using namespace sfb;
using namespace sfb::rows;

extern "C" {

// fp32: 1 = float activations, 0 = bf16.  See SeamArgs for the rest; null pointers switch the parts off.
int sfb_rows_seam(void* x, const void* y, const void* y2, const void* mw, const void* mw2, const void* parts_w, const void* pw, const void* pb, const void* embed,
                  const int* tokens, const void* step_vec, void* tap, const void* nw, const void* nb, void* h, const int* row_map,
                  const void* cw, void* hist, const int* src, const int* dst, int from_embed, int add_embed, int taps, int parts, int post, int rms, int n, int d,
                  int vocab, float eps, float embed_scale, int fp32, void* status, cudaStream_t stream) {
  if (n < 1 || d < 1 || (parts_w && (parts < 1 || y2))) return (int)cudaErrorInvalidValue;
  SeamArgs a{(float*)x, y, y2, (const float*)mw, (const float*)mw2, (const float*)parts_w, (const float*)pw, (const float*)pb, embed, tokens, (const float*)step_vec,
             (float*)tap, (const float*)nw, (const float*)nb, h, row_map, (const float*)cw, hist, src, dst, from_embed, add_embed, taps, d,
             vocab, parts, post, rms, eps, embed_scale, (Status*)status};
  if (fp32) return d % 4 ? launch_seam<float, 1>(a, n, stream) : launch_seam<float, 4>(a, n, stream);
  return d % 4 ? launch_seam<__nv_bfloat16, 1>(a, n, stream) : launch_seam<__nv_bfloat16, 4>(a, n, stream);
}

int sfb_rows_conv(const void* x, int64_t x_stride, const void* w, const void* bias, void* y, void* hist, const int* row_seg, const int* seg_row0,
                  const int* seg_len, const int* seg_src, const int* seg_dst, int n, int C, int taps, int mode, int fp32,
                  cudaStream_t stream) {
  if (n < 1 || C < 1) return (int)cudaErrorInvalidValue;
  ConvRowsArgs a{x, x_stride, (const float*)w, (const float*)bias, y, hist, row_seg, seg_row0, seg_len, seg_src, seg_dst, n, C, mode};
  const bool v4 = C % 4 == 0 && x_stride % 4 == 0 && ((uintptr_t)x % (fp32 ? 16 : 8)) == 0;
  if (fp32) return v4 ? launch_conv<float, 4>(a, taps, stream) : launch_conv<float, 1>(a, taps, stream);
  return v4 ? launch_conv<__nv_bfloat16, 4>(a, taps, stream) : launch_conv<__nv_bfloat16, 1>(a, taps, stream);
}

int sfb_rows_qk_append(const void* proj, int64_t stride, const void* qw, const void* kw, void* q, void* kpool, void* vpool, const int* table,
                       const int* row_lane, const int* row_pos, int max_pages, int n_pages, int n, int H, int G, int dim, int vdim, float eps,
                       int fp32, void* status, cudaStream_t stream) {
  if (n < 1) return (int)cudaErrorInvalidValue;
  QkAppendArgs a{proj, stride, (const float*)qw, (const float*)kw, q, kpool, vpool, table, row_lane, row_pos, max_pages, n_pages, H, G, dim, vdim,
                 eps, (Status*)status};
  const bool v4 = dim % 4 == 0 && vdim % 4 == 0 && stride % 4 == 0;
  if (!fp32 && dim % 8 == 0 && vdim % 8 == 0 && stride % 8 == 0)
    return (int)sfb_launch(qk_append_kernel<__nv_bfloat16, 8>, dim3(n), dim3(256), 0, stream, a);
  if (fp32) return (int)(v4 ? sfb_launch(qk_append_kernel<float, 4>, dim3(n), dim3(256), 0, stream, a)
                            : sfb_launch(qk_append_kernel<float, 1>, dim3(n), dim3(256), 0, stream, a));
  return (int)(v4 ? sfb_launch(qk_append_kernel<__nv_bfloat16, 4>, dim3(n), dim3(256), 0, stream, a)
                  : sfb_launch(qk_append_kernel<__nv_bfloat16, 1>, dim3(n), dim3(256), 0, stream, a));
}

// qw, kw: [dim]; heads up to 512 wide
int sfb_rows_head_append(const void* proj, int64_t stride, const void* qw, const void* kw, void* q, void* kpool, void* vpool, const int* table,
                         const int* row_lane, const int* row_pos, int max_pages, int n_pages, int n, int H, int G, int dim, int vdim, float eps,
                         int fp32, void* status, cudaStream_t stream) {
  if (n < 1 || G < 1 || dim < 1 || dim > 512) return (int)cudaErrorInvalidValue;
  QkAppendArgs a{proj, stride, (const float*)qw, (const float*)kw, q, kpool, vpool, table, row_lane, row_pos, max_pages, n_pages, H, G, dim, vdim,
                 eps, (Status*)status};
  const int all = dim | vdim | (int)(stride & 1023), V = all % 4 ? 1 : fp32 || all % 8 ? 4 : 8;
  int per = 1;             // lanes of a head
  while (per < 32 && per * V < dim) per *= 2;
  const dim3 g(n), b(256);
  if (fp32) return (int)(V == 4 ? sfb_launch(head_append_kernel<float, 4, 4>, g, b, 0, stream, a, per)
                                : sfb_launch(head_append_kernel<float, 1, 16>, g, b, 0, stream, a, per));
  if (V == 8) return (int)(dim <= 256 ? sfb_launch(head_append_kernel<__nv_bfloat16, 8, 1>, g, b, 0, stream, a, per)
                                      : sfb_launch(head_append_kernel<__nv_bfloat16, 8, 2>, g, b, 0, stream, a, per));
  return (int)(V == 4 ? sfb_launch(head_append_kernel<__nv_bfloat16, 4, 4>, g, b, 0, stream, a, per)
                      : sfb_launch(head_append_kernel<__nv_bfloat16, 1, 16>, g, b, 0, stream, a, per));
}

// summaries: a segment has more than one chunk (two passes; the gates are overwritten); otherwise one pass
int sfb_rows_scan(const void* gates, const void* rb, const void* ib, const void* decay, const void* u, const void* y, int64_t y_stride, void* out,
                  void* S, void* sums, const int* chunk_seg, const int* chunk_row0, const int* chunk_rows, const int* chunk_first,
                  const int* seg_src, const int* seg_dst, const int* seg_row0, const int* seg_len, int chunks, int summaries, int n, int width,
                  int bs, int fp32, cudaStream_t stream) {
  if (n < 1 || chunks < 1 || chunks > 65535) return (int)cudaErrorInvalidValue;
  ScanArgs a{(const float*)gates, (const float*)rb, (const float*)ib, (const float*)decay, u, y, y_stride, out, (float*)S, (float2*)sums,
             chunk_seg, chunk_row0, chunk_rows, chunk_first, seg_src, seg_dst, seg_row0, seg_len, n, width, bs, chunks};
  const dim3 g((width + 127) / 128, chunks), b(128);
  if (!summaries)
    return (int)(fp32 ? sfb_launch(scan_short_kernel<float>, g, b, 0, stream, a) : sfb_launch(scan_short_kernel<__nv_bfloat16>, g, b, 0, stream, a));
  cudaError_t rc = fp32 ? sfb_launch(scan_gates_kernel<float>, g, b, 0, stream, a) : sfb_launch(scan_gates_kernel<__nv_bfloat16>, g, b, 0, stream, a);
  if (rc != cudaSuccess) return (int)rc;
  rc = sfb_launch(scan_starts_kernel, dim3((width + 31) / 32), dim3(32, START_G), 0, stream, a);
  if (rc != cudaSuccess) return (int)rc;
  rc = fp32 ? sfb_launch(scan_apply_kernel<float>, g, b, 0, stream, a) : sfb_launch(scan_apply_kernel<__nv_bfloat16>, g, b, 0, stream, a);
  return (int)rc;
}

int sfb_rows_gated_step(const void* x, int64_t x_stride, const void* y, int64_t y_stride, const void* cw, const void* cb, void* hist,
                        const void* wg, const void* rb, const void* ib, const void* decay, void* S, void* out, const int* src, const int* dst,
                        int n, int width, int bs, int taps, int fp32, cudaStream_t stream) {
  if (n < 1 || bs < 1 || width % bs || taps < 1) return (int)cudaErrorInvalidValue;
  const int parts = width / bs, groups = (n + GATED_RB - 1) / GATED_RB;
  // enough blocks to fill the machine without repeating the convolution more than needed
  int tiles = 1;
  while (tiles < 16 && parts * groups * tiles < 148 && bs / (tiles * 2) >= 8) tiles *= 2;
  GatedRowArgs a{x, y, x_stride, y_stride, (const float*)cw, (const float*)cb, hist, wg, (const float*)rb, (const float*)ib, (const float*)decay,
                 (float*)S, out, src, dst, n, width, bs, taps, tiles, (bs + tiles - 1) / tiles};
  const size_t smem = (size_t)GATED_RB * ((bs + 7) & ~7) * sizeof(float);
  if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  const dim3 g(parts * tiles, groups), b(256);
  const bool v8 = bs % 8 == 0;
  if (fp32) return (int)(v8 ? sfb_launch(gated_row_kernel<float, 8>, g, b, smem, stream, a) : sfb_launch(gated_row_kernel<float, 1>, g, b, smem, stream, a));
  return (int)(v8 ? sfb_launch(gated_row_kernel<__nv_bfloat16, 8>, g, b, smem, stream, a)
                  : sfb_launch(gated_row_kernel<__nv_bfloat16, 1>, g, b, smem, stream, a));
}

int sfb_rows_rot_append(const void* proj, int64_t stride, const void* cs, void* q, void* kpool, void* vpool, void* v_first, const void* lam,
                        const int* table, const int* row_lane, const int* row_pos, int max_pages, int n_pages, int n, int H, int G, int dim, int vdim,
                        int dims, int fp32, void* status, cudaStream_t stream) {
  if (n < 1 || G < 1 || dims % 2 || dims < 0 || dims > dim || (lam && !v_first)) return (int)cudaErrorInvalidValue;
  RotAppendArgs a{proj, stride, (const float2*)cs, q, kpool, vpool, v_first, (const float*)lam, table, row_lane, row_pos, max_pages, n_pages, H, G, dim, vdim,
                  dims / 2, (Status*)status};
  const int all = (dims / 2) | dim | vdim | (int)(stride & 1023);
  const dim3 g(n), b(256);
  if (!fp32 && all % 8 == 0) return (int)sfb_launch(rot_append_kernel<__nv_bfloat16, 8>, g, b, 0, stream, a);
  const bool v4 = all % 4 == 0;
  if (fp32) return (int)(v4 ? sfb_launch(rot_append_kernel<float, 4>, g, b, 0, stream, a) : sfb_launch(rot_append_kernel<float, 1>, g, b, 0, stream, a));
  return (int)(v4 ? sfb_launch(rot_append_kernel<__nv_bfloat16, 4>, g, b, 0, stream, a) : sfb_launch(rot_append_kernel<__nv_bfloat16, 1>, g, b, 0, stream, a));
}

int sfb_rows_token_gate(const void* z, const void* table, const int* tokens, void* out, int n, int dim, int64_t table_stride, int col0, int vocab, int fp32,
                        void* status, cudaStream_t stream) {
  if (n < 1 || dim < 1) return (int)cudaErrorInvalidValue;
  const int all = dim | col0 | (int)(table_stride & 1023);
  Status* s = (Status*)status;
  if (fp32) return all % 4 ? launch_token_gate<float, 1>(z, table, tokens, out, n, dim, table_stride, col0, vocab, s, stream)
                           : launch_token_gate<float, 4>(z, table, tokens, out, n, dim, table_stride, col0, vocab, s, stream);
  if (all % 8 == 0) return launch_token_gate<__nv_bfloat16, 8>(z, table, tokens, out, n, dim, table_stride, col0, vocab, s, stream);
  return all % 4 ? launch_token_gate<__nv_bfloat16, 1>(z, table, tokens, out, n, dim, table_stride, col0, vocab, s, stream)
                 : launch_token_gate<__nv_bfloat16, 4>(z, table, tokens, out, n, dim, table_stride, col0, vocab, s, stream);
}

int sfb_rows_act_mul(const void* gu, void* out, int64_t out_stride, int n, int ff, int act, float alpha, float limit, int fp32, cudaStream_t stream) {
  if (n < 1 || ff < 1) return (int)cudaErrorInvalidValue;
  const int all = ff | (int)(out_stride & 1023), V = all % 4 ? 1 : (fp32 || all % 8) ? 4 : 8;
  const dim3 g(n, (ff + 256 * V - 1) / (256 * V)), b(256);
  if (fp32) return (int)(V == 4 ? sfb_launch(act_mul_kernel<float, 4>, g, b, 0, stream, (const float*)gu, (float*)out, ff, out_stride, act, alpha, limit)
                                : sfb_launch(act_mul_kernel<float, 1>, g, b, 0, stream, (const float*)gu, (float*)out, ff, out_stride, act, alpha, limit));
  const __nv_bfloat16* i = (const __nv_bfloat16*)gu;
  __nv_bfloat16* o = (__nv_bfloat16*)out;
  if (V == 8) return (int)sfb_launch(act_mul_kernel<__nv_bfloat16, 8>, g, b, 0, stream, i, o, ff, out_stride, act, alpha, limit);
  return (int)(V == 4 ? sfb_launch(act_mul_kernel<__nv_bfloat16, 4>, g, b, 0, stream, i, o, ff, out_stride, act, alpha, limit)
                      : sfb_launch(act_mul_kernel<__nv_bfloat16, 1>, g, b, 0, stream, i, o, ff, out_stride, act, alpha, limit));
}

// out = act(z), `count` elements (z and out may be the same)
int sfb_rows_act(const void* z, void* out, int64_t count, int act, float p0, float p1, int fp32, cudaStream_t stream) {
  if (count < 1 || (act != ACT_RELU2 && act != ACT_XIELU)) return (int)cudaErrorInvalidValue;
  const int V = count % 4 ? 1 : fp32 || count % 8 ? 4 : 8;
  const int64_t blocks = (count + 256 * ACT_U * V - 1) / (256 * ACT_U * V);
  if (blocks > 0x7fffffff) return (int)cudaErrorInvalidValue;
  const dim3 g((unsigned)blocks), b(256);
  if (fp32) return (int)(V == 4 ? sfb_launch(act_kernel<float, 4>, g, b, 0, stream, (const float*)z, (float*)out, count, act, p0, p1)
                                : sfb_launch(act_kernel<float, 1>, g, b, 0, stream, (const float*)z, (float*)out, count, act, p0, p1));
  const __nv_bfloat16* i = (const __nv_bfloat16*)z;
  __nv_bfloat16* o = (__nv_bfloat16*)out;
  if (V == 8) return (int)sfb_launch(act_kernel<__nv_bfloat16, 8>, g, b, 0, stream, i, o, count, act, p0, p1);
  return (int)(V == 4 ? sfb_launch(act_kernel<__nv_bfloat16, 4>, g, b, 0, stream, i, o, count, act, p0, p1)
                      : sfb_launch(act_kernel<__nv_bfloat16, 1>, g, b, 0, stream, i, o, count, act, p0, p1));
}

}  // extern "C"
