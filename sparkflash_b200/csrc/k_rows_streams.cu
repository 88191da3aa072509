// Seam of the layered decoders whose residual is several streams (hyper-connections: Zhu et al., "Hyper-Connections"): one pass over a row
// brings a sublayer's output into the streams and makes the next sublayer's input.
//
//   x_t  <- sum_s mix[s][t] x_s + out[t] y      (the right side holds the streams before the pass); y may be a weighted sum of several parts
//   u     = sum_t in[t] x_t                     the streams as the next sublayer reads them (in null: their sum)
//   h     = RMS(u) w                            with, on a step of single-row segments, the input convolution h + conv(h)
//
// A row begins with every stream equal to the scaled embedding.  Streams are 32-bit; one block per row, every stream of a channel in the
// same thread, so that the streams cross memory once in each direction.
#include "k_rows_seam.cuh"

namespace sfb {
namespace rows {

struct StreamArgs {
  float* x;                 // [rows, S, d] streams
  const void* y;            // [rows, d] sublayer output (T) or null: no update
  const float* parts_w;     // [rows, parts]: y is [rows, parts, d] and the output their weighted sum; or null
  const float *mix, *out;   // [S, S] from, to; [S]
  const void* embed;        // [vocab, d] (T): the row begins with it (y null)
  const int* tokens;        // [rows]
  float* tap;               // [rows, d] or null: the sum of the new streams
  const float* in;          // [S] or null: ones
  const float* nw;          // [d]
  void* h;                  // [rows, d] (T)
  const int* row_map;       // null: row = block; otherwise the residual row of output row `block`
  const float* cw;          // [taps, d] input convolution, or null
  void* hist;               // [slots, taps - 1, d] (T)
  const int *src, *dst;     // [rows] state versions of single-row segments
  int S, d, parts, taps, vocab, keep;    // keep: the streams are stored
  float eps, embed_scale;
  Status* status;
};

// SM: most streams.  AHEAD (few rows): weights and the convolution's carried inputs are requested before they are needed.
template <typename T, int V, int NV, int SM, bool AHEAD>
__global__ void __launch_bounds__(NV < 4 ? 256 : 512) stream_seam_kernel(StreamArgs a) {
  __shared__ float sh[2 * 2 * 32];
  int phase = 0;
  const int d = a.d, step = blockDim.x * V, c0 = threadIdx.x * V, S = SM <= 4 ? SM : a.S;
  constexpr int TW = AHEAD ? 4 : 1;      // taps held ahead
  float nw[NV][V], cw[TW][NV][V], cg[TW][NV][V], mix[SM][SM], out[SM], in[SM];
  const bool ahead_conv = AHEAD && a.cw && a.taps <= TW;
#pragma unroll
  for (int s = 0; s < SM; ++s) {
    in[s] = s < S ? (a.in ? a.in[s] : 1.f) : 0.f;
    out[s] = a.y && s < S ? a.out[s] : 0.f;
#pragma unroll
    for (int t = 0; t < SM; ++t) mix[s][t] = a.y && s < S && t < S ? a.mix[s * S + t] : 0.f;
  }
  if constexpr (AHEAD) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c >= d) continue;
      load_v<float, V>(a.nw + c, nw[i]);
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
  const int W = a.taps - 1;
  const int src = a.cw ? a.src[row] : -1;
  T* hd = a.cw ? (T*)a.hist + (size_t)a.dst[row] * W * d : nullptr;
  const T* hs = src >= 0 ? (const T*)a.hist + (size_t)src * W * d : nullptr;
  float* xr = a.x + (size_t)row * S * d;
  float x[SM][NV][V], u[NV][V];
  if (a.y) {
#pragma unroll
    for (int s = 0; s < SM; ++s)
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (s < S && c0 + i * step < d) load_v<float, V>(xr + (size_t)s * d + c0 + i * step, x[s][i]);
  }
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
  float ss[1] = {0.f};
  if (a.y) {
    float y[NV][V];
    const T* yr = (const T*)a.y + (size_t)row * (a.parts_w ? a.parts : 1) * d;
    if (a.parts_w) {
      const float* wr = a.parts_w + (size_t)row * a.parts;
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
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c >= d) continue;
      float sum[V];
#pragma unroll
      for (int k = 0; k < V; ++k) u[i][k] = sum[k] = 0.f;
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) break;
        float n[V];
#pragma unroll
        for (int k = 0; k < V; ++k) {
          n[k] = out[t] * y[i][k];
#pragma unroll
          for (int s = 0; s < SM; ++s)
            if (s < S) n[k] = fmaf(mix[s][t], x[s][i][k], n[k]);
          u[i][k] = fmaf(in[t], n[k], u[i][k]);
          sum[k] += n[k];
        }
        if (a.keep) store_v<float, V>(xr + (size_t)t * d + c, n);
      }
      if (a.tap) store_v<float, V>(a.tap + (size_t)row * d + c, sum);
    }
  } else {
    int tok = a.tokens[row];
    if (tok < 0 || tok >= a.vocab) { if (threadIdx.x == 0) status_set(a.status, ST_BOUNDS, 77, tok, a.vocab); tok = 0; }
    const T* er = (const T*)a.embed + (size_t)tok * d;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c >= d) continue;
      float e[V];
      load_v<T, V>(er + c, e);
#pragma unroll
      for (int k = 0; k < V; ++k) { e[k] *= a.embed_scale; u[i][k] = 0.f; }
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) break;
        store_v<float, V>(xr + (size_t)t * d + c, e);
#pragma unroll
        for (int k = 0; k < V; ++k) u[i][k] = fmaf(in[t], e[k], u[i][k]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (c0 + i * step < d) {
#pragma unroll
      for (int k = 0; k < V; ++k) ss[0] = fmaf(u[i][k], u[i][k], ss[0]);
    }
  block_sums<1>(ss, sh, phase);
  const float rs = 1.f / sqrtf(ss[0] / (float)d + a.eps);
  T* hr = (T*)a.h + (size_t)out_row * d;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = c0 + i * step;
    if (c >= d) continue;
    if constexpr (!AHEAD) load_v<float, V>(a.nw + c, nw[i]);
    float o[V];
#pragma unroll
    for (int k = 0; k < V; ++k) o[k] = u[i][k] * rs * nw[i][k];
    if (a.cw) step_conv<T, V, TW, NV>(o, i, c, d, W, a.cw, hs, hd, ahead_conv, cw, cg);
    store_v<T, V>(hr + c, o);
  }
}

template <typename T, int V, int NV, bool AHEAD>
static int launch_streams_s(const StreamArgs& a, int n, int threads, cudaStream_t st) {
  const dim3 g(n), b(threads);
  switch (a.S) {
    case 1: return (int)sfb_launch(stream_seam_kernel<T, V, NV, 1, AHEAD>, g, b, 0, st, a);
    case 2: return (int)sfb_launch(stream_seam_kernel<T, V, NV, 2, AHEAD>, g, b, 0, st, a);
    case 3: return (int)sfb_launch(stream_seam_kernel<T, V, NV, 3, AHEAD>, g, b, 0, st, a);
    case 4: return (int)sfb_launch(stream_seam_kernel<T, V, NV, 4, AHEAD>, g, b, 0, st, a);
    default: return (int)sfb_launch(stream_seam_kernel<T, V, NV, 8, AHEAD>, g, b, 0, st, a);
  }
}
template <typename T, int V>
static int launch_streams(const StreamArgs& a, int n, cudaStream_t st) {
  const int vecs = (a.d + V - 1) / V;
  const bool few = n <= 296;
  int nv = 1;                              // few rows: many threads per row; many rows: more of the row per thread
  while (nv < 8 && (vecs + nv - 1) / nv > (nv >= 4 ? 512 : few || nv >= 2 ? 256 : 128)) nv *= 2;
  const int threads = ((vecs + nv - 1) / nv + 31) / 32 * 32;
  if (threads > 512) return (int)cudaErrorInvalidValue;
  switch (nv) {
    case 1: return few ? launch_streams_s<T, V, 1, true>(a, n, threads, st) : launch_streams_s<T, V, 1, false>(a, n, threads, st);
    case 2: return few ? launch_streams_s<T, V, 2, true>(a, n, threads, st) : launch_streams_s<T, V, 2, false>(a, n, threads, st);
    case 4: return launch_streams_s<T, V, 4, false>(a, n, threads, st);
    default: return launch_streams_s<T, V, 8, false>(a, n, threads, st);
  }
}

}  // namespace rows
}  // namespace sfb

using namespace sfb;
using namespace sfb::rows;

extern "C" {

// fp32: 1 = float activations, 0 = bf16.  y null: the row begins with the embedding.  Up to 8 streams.  See StreamArgs for the rest.
int sfb_rows_streams(void* x, const void* y, const void* parts_w, const void* mix, const void* out, const void* embed, const int* tokens, void* tap, const void* in,
                     const void* nw, void* h, const int* row_map, const void* cw, void* hist, const int* src, const int* dst, int streams, int parts, int taps,
                     int keep, int n, int d, int vocab, float eps, float embed_scale, int fp32, void* status, cudaStream_t stream) {
  if (n < 1 || d < 1 || streams < 1 || streams > 8 || (parts_w && (parts < 1 || !y)) || (y ? !mix || !out : !embed || !tokens) || !nw || !h ||
      (cw && (taps < 1 || row_map || (taps > 1 && !hist) || !src || !dst)))
    return (int)cudaErrorInvalidValue;
  StreamArgs a{(float*)x, y, (const float*)parts_w, (const float*)mix, (const float*)out, embed, tokens, (float*)tap, (const float*)in, (const float*)nw, h, row_map,
               (const float*)cw, hist, src, dst, streams, d, parts, taps, vocab, keep, eps, embed_scale, (Status*)status};
  if (fp32) return d % 4 ? launch_streams<float, 1>(a, n, stream) : launch_streams<float, 4>(a, n, stream);
  return d % 4 ? launch_streams<__nv_bfloat16, 1>(a, n, stream) : launch_streams<__nv_bfloat16, 4>(a, n, stream);
}

}  // extern "C"
