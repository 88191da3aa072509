// What the seam kernels of the layered decoders share (k_rows.cu: one residual; k_rows_streams.cu: several streams of it).
#pragma once
#include "k_rows.cuh"

namespace sfb {
namespace rows {

// Input convolution of a step of single-row segments: o (channels c .. of a norm's output) becomes o + conv(o) over the carried inputs hs
// (null: zeros), whose next version is hd.  `ahead`: weights and carried inputs are held in registers (rw, rg: [taps][i][V]).
template <typename T, int V, int TW, int NV>
__device__ __forceinline__ void step_conv(float (&o)[V], int i, int c, int d, int W, const float* w, const T* hs, T* hd, bool ahead,
                                          const float (&rw)[TW][NV][V], const float (&rg)[TW][NV][V]) {
  // the convolution sees the norm's output at activation precision, as the many-row kernel does
  float acc[V], t[V];
#pragma unroll
  for (int k = 0; k < V; ++k) o[k] = to_f<T>(from_f<T>(o[k]));
  if (ahead) {
#pragma unroll
    for (int k = 0; k < V; ++k) acc[k] = 0.f;
#pragma unroll
    for (int j = 0; j < TW; ++j) {
      if (j < W) {
#pragma unroll
        for (int k = 0; k < V; ++k) acc[k] += rw[j][i][k] * rg[j][i][k];
        if (j > 0) store_v<T, V>(hd + (size_t)(j - 1) * d + c, rg[j][i]);
      } else if (j == W) {
#pragma unroll
        for (int k = 0; k < V; ++k) acc[k] += rw[j][i][k] * o[k];
      }
    }
  } else {
    load_v<float, V>(w + (size_t)W * d + c, t);
#pragma unroll
    for (int k = 0; k < V; ++k) acc[k] = t[k] * o[k];
#pragma unroll 4
    for (int j = 0; j < W; ++j) {
      float g[V];
      if (hs) load_v<T, V>(hs + (size_t)j * d + c, g);
      else {
#pragma unroll
        for (int k = 0; k < V; ++k) g[k] = 0.f;
      }
      load_v<float, V>(w + (size_t)j * d + c, t);
#pragma unroll
      for (int k = 0; k < V; ++k) acc[k] += t[k] * g[k];
      if (j > 0) store_v<T, V>(hd + (size_t)(j - 1) * d + c, g);
    }
  }
  if (W > 0) store_v<T, V>(hd + (size_t)(W - 1) * d + c, o);
#pragma unroll
  for (int k = 0; k < V; ++k) o[k] += acc[k];
}

}  // namespace rows
}  // namespace sfb
