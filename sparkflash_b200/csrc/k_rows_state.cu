// Linear recurrence with a matrix state and one decay per head (models/mixers.py: state-space duality, retention, delta rule):
//
//   S_t = a_t S_(t-1) + w_t k_t v_t^T,   y_t = S_t^T q_t + D v_t        S: N x P per head, 32-bit
//
// a_t = exp(A dt_t), w_t = dt_t with dt_t = softplus(raw_t + bias) per token and head, or a_t a constant of the head and w_t = 1.
// q and k belong to groups of heads; they may be turned by their position (rotate-half layout) and k scaled.
//
// Delta rule: q and k are unit vectors (q scaled), and what is written is what the state does not yet say about k:
//
//   S = a_t S_(t-1),   u_t = b_t (v_t - S^T k_t),   S_t = S + k_t u_t^T,   y_t = S_t^T q_t        b_t = sigmoid(raw_t)
//
//   state_rows    one block per (segment, head, tile of P): the state stays in registers while the segment's rows go by.  Any
//                 sizes, bf16 or 32-bit; decode steps and short runs.  Steps of single rows also apply the causal convolution
//                 and silu that q, k and v come from.  (k_rows_state_tc.cu takes long runs in bf16.)
//   gated_norm    RMS norm of equal parts of a row with a silu gate before it (weighted) or after it.
//
// States are stored [slot][head][P][N rounded up to 32], so that eight lanes read 128 consecutive bytes.
#include "k_rows.cuh"

namespace sfb {
namespace rows {

struct StateArgs {
  const void *q, *k, *v;            // (T) first element of row 0; rows are q_stride, k_stride, v_stride elements apart
  int64_t q_stride, k_stride, v_stride;
  const void* dt;                   // (T) [n, dt_stride] raw step sizes, or null: constant decay
  int64_t dt_stride;
  const float* dt_bias;             // [H]
  const float* a;                   // [H]: A with dt, else the decay itself
  const float* D;                   // [H] or null
  const void* beta;                 // (T) [n, beta_stride] raw write strengths: delta rule; or null
  int64_t beta_stride;
  const float2* rot;                // [positions, rot_dims / 2] (cos, sin) or null
  const int* row_pos;
  void* y;                          // [n, H P] (T)
  float* S;                         // [slots, H, P, Np]
  const float *cw, *cb;             // [taps, C], [C]: convolution of single rows, or null
  void* hist;                       // [slots, taps - 1, C] (T)
  const int *segs, *seg_row0, *seg_len, *seg_src, *seg_dst;      // segs: segment of every blockIdx.y, or null: identity
  int rot_dims, taps, C, q_ch, k_ch, v_ch;                       // *_ch: first convolution channel of q, k, v
  int H, G, N, P, Np;
  float k_scale, q_scale, unit_eps; // q_scale, unit_eps: of the delta rule's unit vectors
};
constexpr int STB = 8;              // rows whose q, k, v are staged together

__device__ __forceinline__ float softplus_f(float z) { return log1pf(expf(-fabsf(z))) + fmaxf(z, 0.f); }

// the convolution's output at one channel of a single row, rounded to activation precision; `keep`: this block carries the inputs on
constexpr int ST_TAPS = 4;           // taps requested together
template <typename T>
__device__ __forceinline__ float conv_silu(const StateArgs& a, T x, int ch, int src, int dst, bool keep) {
  const int W = a.taps - 1;
  const T* hs = (const T*)a.hist + (size_t)(src >= 0 ? src : 0) * W * a.C + ch;
  T* hd = (T*)a.hist + (size_t)dst * W * a.C + ch;
  float acc = (a.cb ? a.cb[ch] : 0.f) + a.cw[(size_t)W * a.C + ch] * to_f<T>(x);
  for (int j0 = 0; j0 < W; j0 += ST_TAPS) {
    T gv[ST_TAPS];
    float w[ST_TAPS];
#pragma unroll
    for (int j = 0; j < ST_TAPS; ++j) {
      gv[j] = src >= 0 && j0 + j < W ? hs[(size_t)(j0 + j) * a.C] : from_f<T>(0.f);
      w[j] = j0 + j < W ? a.cw[(size_t)(j0 + j) * a.C + ch] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < ST_TAPS; ++j) {
      acc += w[j] * to_f<T>(gv[j]);
      if (keep && j0 + j > 0 && j0 + j < W) hd[(size_t)(j0 + j - 1) * a.C] = gv[j];
    }
  }
  if (keep && W > 0) hd[(size_t)(W - 1) * a.C] = x;
  return to_f<T>(from_f<T>(acc * sigmoid_f(acc)));
}

template <typename T, int NI, bool DELTA>
__global__ void __launch_bounds__(256, NI <= 4 ? (DELTA ? 4 : 5) : NI <= 8 ? 3 : 1) state_rows_kernel(StateArgs a) {
  extern __shared__ __align__(16) float sm[];
  const int PT = blockDim.x >> 3, tiles = (a.P + PT - 1) / PT;
  const int h = blockIdx.x / tiles, tile = blockIdx.x % tiles, g = h / (a.H / a.G);
  const int tid = threadIdx.x, ng = tid & 7, pl = tid >> 3, p = tile * PT + pl;
  float* qs = sm;                     // [STB][Np]
  float* ks = qs + STB * a.Np;
  float* vs = ks + STB * a.Np;        // [STB][PT]
  float* av = vs + STB * PT;          // [STB] decay
  float* wv = av + STB;               // [STB] input scale (delta rule: write strength)
  float* qr = wv + STB;               // [STB], [STB] delta rule: factors that make q and k unit vectors
  float* kr = qr + STB;
  pdl_launch_dependents();
  pdl_wait();
  const int seg = a.segs ? a.segs[blockIdx.y] : blockIdx.y;
  const int row0 = a.seg_row0[seg], len = a.seg_len[seg], src = a.seg_src[seg], dst = a.seg_dst[seg];
  const bool on = p < a.P;
  float4 S[NI];
  const size_t at = ((size_t)h * a.P + (on ? p : 0)) * a.Np + ng * 4, slot = (size_t)a.H * a.P * a.Np;
#pragma unroll
  for (int i = 0; i < NI; ++i)
    S[i] = (src >= 0 && on) ? *reinterpret_cast<const float4*>(a.S + (size_t)src * slot + at + i * 32) : make_float4(0.f, 0.f, 0.f, 0.f);
  const float D = a.D ? a.D[h] : 0.f;
  const int half = a.rot_dims >> 1;
  const bool keep_g = a.cw && tile == 0 && h == g * (a.H / a.G);
  for (int t0 = 0; t0 < len; t0 += STB) {
    const int nb = min(STB, len - t0);
    if (t0) __syncthreads();
    if (a.cw) {                       // one row: channels of q, then k, then the tile's v, one per thread
      const int span = 2 * a.Np + PT;
      for (int x = tid; x < span; x += blockDim.x) {
        const bool isv = x >= 2 * a.Np, isk = !isv && x >= a.Np;
        const int n = isv ? tile * PT + x - 2 * a.Np : isk ? x - a.Np : x, base = isv ? h * a.P : g * a.N;
        float f = 0.f;
        if (n < (isv ? a.P : a.N)) {
          const T r = isv ? ((const T*)a.v)[(size_t)row0 * a.v_stride + base + n]
                          : isk ? ((const T*)a.k)[(size_t)row0 * a.k_stride + base + n] : ((const T*)a.q)[(size_t)row0 * a.q_stride + base + n];
          f = conv_silu<T>(a, r, (isv ? a.v_ch : isk ? a.k_ch : a.q_ch) + base + n, src, dst, isv || keep_g);
        }
        if (isv) vs[x - 2 * a.Np] = f;
        else if (isk) ks[n] = f * a.k_scale;
        else qs[n] = f;
      }
    } else {
      for (int x = tid; x < nb * a.Np; x += blockDim.x) {
        const int t = x / a.Np, n = x - t * a.Np, row = row0 + t0 + t;
        float qf = 0.f, kf = 0.f;
        if (n < a.N) {
          const T* qp = (const T*)a.q + (size_t)row * a.q_stride + (size_t)g * a.N;
          const T* kp = (const T*)a.k + (size_t)row * a.k_stride + (size_t)g * a.N;
          qf = to_f<T>(qp[n]); kf = to_f<T>(kp[n]);
          if (n < a.rot_dims) {
            const int i = n < half ? n : n - half, o = n < half ? n + half : n - half;
            const float2 cs = a.rot[(size_t)a.row_pos[row] * half + i];
            const float sn = n < half ? -cs.y : cs.y;
            qf = qf * cs.x + to_f<T>(qp[o]) * sn;
            kf = kf * cs.x + to_f<T>(kp[o]) * sn;
          }
        }
        qs[x] = qf; ks[x] = kf * a.k_scale;
      }
      for (int x = tid; x < nb * PT; x += blockDim.x) {
        const int t = x / PT, c = tile * PT + x - t * PT;
        vs[x] = c < a.P ? to_f<T>(((const T*)a.v)[(size_t)(row0 + t0 + t) * a.v_stride + (size_t)h * a.P + c]) : 0.f;
      }
    }
    if (tid < nb) {
      if (a.dt) {
        const float dt = softplus_f(to_f<T>(((const T*)a.dt)[(size_t)(row0 + t0 + tid) * a.dt_stride + h]) + a.dt_bias[h]);
        av[tid] = expf(a.a[h] * dt);
        wv[tid] = DELTA ? sigmoid_f(to_f<T>(((const T*)a.beta)[(size_t)(row0 + t0 + tid) * a.beta_stride + h])) : dt;
      } else {
        av[tid] = a.a[h]; wv[tid] = 1.f;
      }
    }
    __syncthreads();
    if constexpr (DELTA) {
      for (int x = tid >> 5; x < 2 * nb; x += blockDim.x >> 5) {
        const float* p0 = (x & 1 ? ks : qs) + (x >> 1) * a.Np;
        float s = 0.f;
        for (int n = tid & 31; n < a.Np; n += 32) s = fmaf(p0[n], p0[n], s);
        s = warp_sum(s);
        if ((tid & 31) == 0) (x & 1 ? kr : qr)[x >> 1] = (x & 1 ? 1.f : a.q_scale) / sqrtf(s + a.unit_eps);
      }
      __syncthreads();
    }
    for (int t = 0; t < nb; ++t) {
      const float dec = av[t], v = vs[t * PT + pl];
      float in = v * wv[t];
      if constexpr (DELTA) {              // what the decayed state says about k
        float m = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const float4 kk = *reinterpret_cast<const float4*>(ks + t * a.Np + i * 32 + ng * 4);
          m = fmaf(S[i].x, kk.x, m); m = fmaf(S[i].y, kk.y, m); m = fmaf(S[i].z, kk.z, m); m = fmaf(S[i].w, kk.w, m);
        }
        m += __shfl_xor_sync(0xffffffffu, m, 1);
        m += __shfl_xor_sync(0xffffffffu, m, 2);
        m += __shfl_xor_sync(0xffffffffu, m, 4);
        in = wv[t] * (v - dec * kr[t] * m) * kr[t];
      }
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float4 kk = *reinterpret_cast<const float4*>(ks + t * a.Np + i * 32 + ng * 4);
        const float4 qq = *reinterpret_cast<const float4*>(qs + t * a.Np + i * 32 + ng * 4);
        S[i].x = fmaf(dec, S[i].x, kk.x * in); S[i].y = fmaf(dec, S[i].y, kk.y * in);
        S[i].z = fmaf(dec, S[i].z, kk.z * in); S[i].w = fmaf(dec, S[i].w, kk.w * in);
        y = fmaf(S[i].x, qq.x, y); y = fmaf(S[i].y, qq.y, y); y = fmaf(S[i].z, qq.z, y); y = fmaf(S[i].w, qq.w, y);
      }
      y += __shfl_xor_sync(0xffffffffu, y, 1);
      y += __shfl_xor_sync(0xffffffffu, y, 2);
      y += __shfl_xor_sync(0xffffffffu, y, 4);
      if constexpr (DELTA) y *= qr[t];
      if (ng == 0 && on) ((T*)a.y)[((size_t)(row0 + t0 + t) * a.H + h) * a.P + p] = from_f<T>(fmaf(D, v, y));
    }
  }
  if (on) {
#pragma unroll
    for (int i = 0; i < NI; ++i) *reinterpret_cast<float4*>(a.S + (size_t)dst * slot + at + i * 32) = S[i];
  }
}

// ---- RMS norm of equal parts with a silu gate ---------------------------------------------------------------------------
struct GatedNormArgs {
  const void* y;            // [n, width] (T)
  const void* gate;         // [n, gate_stride] (T)
  int64_t gate_stride;
  const float* w;           // [width] or null
  void* out;                // [n, width] (T)
  int width, part, before;  // before: the gate multiplies ahead of the norm
  float eps;
};

// A part belongs to a warp (parts side by side in a block) or to the whole block; a thread holds NV vectors of it.
template <typename T, int V, int NV, bool WARP>
__global__ void __launch_bounds__(256) gated_norm_kernel(GatedNormArgs a) {
  __shared__ float sh[2 * 2 * 32];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = WARP ? blockIdx.y * (blockDim.x >> 5) + warp : blockIdx.y, x0 = (WARP ? lane : threadIdx.x) * V, step = (WARP ? 32 : blockDim.x) * V;
  if (WARP && g * a.part >= a.width) return;
  const T* y = (const T*)a.y + (size_t)blockIdx.x * a.width + (size_t)g * a.part;
  const T* z = (const T*)a.gate + (size_t)blockIdx.x * a.gate_stride + (size_t)g * a.part;
  T* o = (T*)a.out + (size_t)blockIdx.x * a.width + (size_t)g * a.part;
  float f[NV][V], gt[NV][V], s[1] = {0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (x0 + i * step < a.part) { load_v<T, V>(y + x0 + i * step, f[i]); load_v<T, V>(z + x0 + i * step, gt[i]); }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (x0 + i * step < a.part) {
#pragma unroll
      for (int k = 0; k < V; ++k) {
        gt[i][k] *= gate_sigmoid<T>(gt[i][k]);
        if (a.before) f[i][k] *= gt[i][k];
        s[0] += f[i][k] * f[i][k];
      }
    }
  if constexpr (WARP) s[0] = warp_sum(s[0]);
  else { int phase = 0; block_sums<1>(s, sh, phase); }
  const float r = 1.f / sqrtf(s[0] / (float)a.part + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = x0 + i * step;
    if (c >= a.part) continue;
    float w[V];
    if (a.w) load_v<float, V>(a.w + (size_t)g * a.part + c, w);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      f[i][k] *= r;
      if (a.w) f[i][k] *= w[k];
      if (!a.before) f[i][k] *= gt[i][k];
    }
    store_v<T, V>(o + c, f[i]);
  }
}

template <typename T, bool DELTA>
static int launch_state(const StateArgs& a, int segs, cudaStream_t st) {
  const int threads = a.P > 16 ? 256 : 128, PT = threads / 8, tiles = (a.P + PT - 1) / PT;
  const dim3 g(a.H * tiles, segs), b(threads);
  const size_t smem = ((size_t)2 * STB * a.Np + STB * PT + 4 * STB) * sizeof(float);
#define SFB_STATE(NI) case NI: return (int)sfb_launch(state_rows_kernel<T, NI, DELTA>, g, b, smem, st, a)
  switch (a.Np / 32) {
    SFB_STATE(1); SFB_STATE(2); SFB_STATE(3); SFB_STATE(4); SFB_STATE(5); SFB_STATE(6); SFB_STATE(7); SFB_STATE(8);
    SFB_STATE(12); SFB_STATE(16);
    default: return (int)cudaErrorInvalidValue;
  }
#undef SFB_STATE
}
template <typename T, int V>
static int launch_gated_norm(const GatedNormArgs& a, int n, cudaStream_t st) {
  const int parts = a.width / a.part, vecs = (a.part + V - 1) / V;
  if (vecs <= 64) {
    const dim3 g(n, (parts + 7) / 8), b(parts < 8 ? 32 * parts : 256);
    return (int)(vecs <= 32 ? sfb_launch(gated_norm_kernel<T, V, 1, true>, g, b, 0, st, a) : sfb_launch(gated_norm_kernel<T, V, 2, true>, g, b, 0, st, a));
  }
  int nv = 1;
  while (nv < 16 && (vecs + nv - 1) / nv > 256) nv *= 2;
  const dim3 g(n, parts), b(((vecs + nv - 1) / nv + 31) / 32 * 32);
  if (b.x > 256) return (int)cudaErrorInvalidValue;
  switch (nv) {
    case 1: return (int)sfb_launch(gated_norm_kernel<T, V, 1, false>, g, b, 0, st, a);
    case 2: return (int)sfb_launch(gated_norm_kernel<T, V, 2, false>, g, b, 0, st, a);
    case 4: return (int)sfb_launch(gated_norm_kernel<T, V, 4, false>, g, b, 0, st, a);
    case 8: return (int)sfb_launch(gated_norm_kernel<T, V, 8, false>, g, b, 0, st, a);
    default: return (int)sfb_launch(gated_norm_kernel<T, V, 16, false>, g, b, 0, st, a);
  }
}

}  // namespace rows
}  // namespace sfb

using namespace sfb;
using namespace sfb::rows;

extern "C" {

// Np: N rounded up to 32 (up to 256), then 384 or 512.  cw: every segment of the launch is one row and q, k, v are the convolution's inputs.
int sfb_rows_state(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t v_stride, const void* dt, int64_t dt_stride,
                   const void* dt_bias, const void* a, const void* D, const void* beta, int64_t beta_stride, const void* rot, const int* row_pos, void* y, void* S, const void* cw,
                   const void* cb, void* hist, const int* segs, const int* seg_row0, const int* seg_len, const int* seg_src, const int* seg_dst,
                   int n_segs, int rot_dims, int taps, int C, int q_ch, int k_ch, int v_ch, int H, int G, int N, int P, int Np, float k_scale,
                   float q_scale, float unit_eps, int fp32, cudaStream_t stream) {
  if (n_segs < 1 || n_segs > 65535 || G < 1 || H % G || (beta && (!dt || rot || D || k_scale != 1.f)) || N < 1 || P < 1 || Np % 32 || Np < N || (rot_dims && (!rot || rot_dims > N || rot_dims % 2)))
    return (int)cudaErrorInvalidValue;
  StateArgs s{q, k, v, q_stride, k_stride, v_stride, dt, dt_stride, (const float*)dt_bias, (const float*)a, (const float*)D, beta, beta_stride, (const float2*)rot, row_pos, y,
              (float*)S, (const float*)cw, (const float*)cb, hist, segs, seg_row0, seg_len, seg_src, seg_dst, rot_dims, taps, C, q_ch, k_ch, v_ch,
              H, G, N, P, Np, k_scale, q_scale, unit_eps};
  if (beta) return fp32 ? launch_state<float, true>(s, n_segs, stream) : launch_state<__nv_bfloat16, true>(s, n_segs, stream);
  return fp32 ? launch_state<float, false>(s, n_segs, stream) : launch_state<__nv_bfloat16, false>(s, n_segs, stream);
}

int sfb_rows_gated_norm(const void* y, const void* gate, int64_t gate_stride, const void* w, void* out, int n, int width, int part, int before, float eps,
                        int fp32, cudaStream_t stream) {
  if (n < 1 || part < 1 || width % part || width / part > 65535) return (int)cudaErrorInvalidValue;
  GatedNormArgs a{y, gate, gate_stride, (const float*)w, out, width, part, before, eps};
  const int v = part % 8 == 0 && part > 128 && gate_stride % 8 == 0 && (uintptr_t)gate % 16 == 0 ? 8 : part % 4 == 0 && gate_stride % 4 == 0 && (uintptr_t)gate % (fp32 ? 16 : 8) == 0 ? 4 : 1;
  if (fp32) return v >= 4 ? launch_gated_norm<float, 4>(a, n, stream) : launch_gated_norm<float, 1>(a, n, stream);
  return v == 8 ? launch_gated_norm<__nv_bfloat16, 8>(a, n, stream) : v == 4 ? launch_gated_norm<__nv_bfloat16, 4>(a, n, stream)
                                                                            : launch_gated_norm<__nv_bfloat16, 1>(a, n, stream);
}

}  // extern "C"
