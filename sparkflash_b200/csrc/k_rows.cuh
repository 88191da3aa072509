// Element access shared by the kernels of the layered decoders (k_rows.cu, k_rows_attn.cu, k_rows_attn_tc.cu): the activation
// type T is bf16 (serving) or float (every step in true 32-bit); arithmetic is always 32-bit.
#pragma once
#include "k_common.cuh"

namespace sfb {
namespace rows {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// V consecutive elements (V = 1, 4 or 8; the address of a group is a multiple of its size, at most 16 bytes)
template <typename T, int V> __device__ __forceinline__ void load_v(const T* p, float* f) {
  if constexpr (V == 1) {
    f[0] = to_f<T>(*p);
  } else if constexpr (V == 8 && sizeof(T) == 2) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
  } else if constexpr (V == 8) {
    load_v<T, 4>(p, f); load_v<T, 4>(p + 4, f + 4);
  } else if constexpr (sizeof(T) == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
  }
}
template <typename T, int V> __device__ __forceinline__ void store_v(T* p, const float* f) {
  if constexpr (V == 1) {
    *p = from_f<T>(f[0]);
  } else if constexpr (V == 8 && sizeof(T) == 2) {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) { const __nv_bfloat162 t = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]); w[i] = *reinterpret_cast<const uint32_t*>(&t); }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  } else if constexpr (V == 8) {
    store_v<T, 4>(p, f); store_v<T, 4>(p + 4, f + 4);
  } else if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
  }
}
// Block sum of N values at once; one barrier per call: successive calls alternate between the two halves of `sh`
// ([2][N * 32] floats), and every thread has read a half before it arrives at the next call's barrier.
template <int N> __device__ __forceinline__ void block_sums(float (&v)[N], float* sh, int& phase) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  float* s = sh + (phase & 1) * (2 * 32);
  phase ^= 1;
#pragma unroll
  for (int k = 0; k < N; ++k) v[k] = warp_sum(v[k]);
  if (lane == 0) {
#pragma unroll
    for (int k = 0; k < N; ++k) s[k * 32 + w] = v[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < N; ++k) {
    float t = 0.f;
    for (int i = 0; i < nw; ++i) t += s[k * 32 + i];
    v[k] = t;
  }
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}


constexpr int ACT_SILU = 1, ACT_GELU = 2, ACT_CLAMP = 3;      // activations of the gated products
constexpr int ACT_RELU2 = 4, ACT_XIELU = 5;                   // of the ungated ones

// exp, reciprocal and square root of the gates, all 32-bit: library-accurate with float activations; with bf16 activations the
// hardware approximations (relative error below 2^-21), whose error is far below the rounding of u
template <typename T> __device__ __forceinline__ float gate_sigmoid(float z) {
  if constexpr (sizeof(T) == 4) return sigmoid_f(z);
  else return __fdividef(1.f, 1.f + __expf(-z));
}
template <typename T> __device__ __forceinline__ float gate_gelu(float z) {
  if constexpr (sizeof(T) == 4) return gelu_tanh_f(z);
  else {   // 0.5 (1 + tanh(k)) = sigmoid(2 k)
    const float k = 1.5957691216057308f * (z + 0.044715f * z * z * z);
    return z * gate_sigmoid<T>(k);
  }
}

// clamped gate: g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(alpha g) (u + 1)
template <typename T> __device__ __forceinline__ float gate_clamp(float g, float u, float alpha, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * gate_sigmoid<T>(alpha * g) * (u + 1.f);
}

// exp(z) - 1 - z for z <= 0: the series near 0, where the difference would cancel.  32-bit activations: the first term left out is below 2^-28 of
// the sum; bf16: the difference is taken from where it is good to 2^-13.
template <typename T> __device__ __forceinline__ float expm1_minus(float z) {
  if constexpr (sizeof(T) == 4) {
    float p = 1.f / 3628800.f;
    p = fmaf(p, z, 1.f / 362880.f); p = fmaf(p, z, 1.f / 40320.f); p = fmaf(p, z, 1.f / 5040.f); p = fmaf(p, z, 1.f / 720.f); p = fmaf(p, z, 1.f / 120.f);
    p = fmaf(p, z, 1.f / 24.f); p = fmaf(p, z, 1.f / 6.f); p = fmaf(p, z, 0.5f);
    return z > -0.75f ? z * z * p : expf(z) - 1.f - z;
  } else {
    const float p = fmaf(fmaf(fmaf(1.f / 120.f, z, 1.f / 24.f), z, 1.f / 6.f), z, 0.5f);
    return z > -0.0625f ? z * z * p : __expf(z) - 1.f - z;
  }
}

// One input.  RELU2: max(z, 0)^2.  XIELU (Huang and Schlag, "Deriving Activation Functions Using Integration"): a z^2 + z / 2 above 0,
// b (exp(z) - 1 - z) + z / 2 below it.
template <typename T> __device__ __forceinline__ float act_single(float z, int act, float a, float b) {
  if (act == ACT_RELU2) { const float r = fmaxf(z, 0.f); return r * r; }
  return (z > 0.f ? a * z * z : b * expm1_minus<T>(fminf(z, 0.f))) + 0.5f * z;
}

}  // namespace rows
}  // namespace sfb
