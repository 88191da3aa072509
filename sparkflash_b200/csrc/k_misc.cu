// Embedding gather, taps for the drafter and synthetic weight fill.
//
// Reference behaviour: kernels/opt_rows_sm121.cu embed_own:2564, crates/sparkflash-model-deepseek-v41/src/synthetic.rs (weights from a hash of name and seed).
#include "k_common.cuh"

namespace sfb {

// h[row, c, :] = embed[token[row], :] for every hc copy
__global__ void embed_kernel(const __nv_bfloat16* embed, const int* tokens, __nv_bfloat16* h, int n, int hc,
                             int d, int vocab, Status* st) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.y;
  int tok = tokens[row];
  if (tok < 0 || tok >= vocab) { if (threadIdx.x == 0 && blockIdx.x == 0) status_set(st, ST_BOUNDS, 3, tok, vocab); tok = 0; }
  const int col = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (col >= d) return;
  const uint4 v = *reinterpret_cast<const uint4*>(embed + (size_t)tok * d + col);
  for (int c = 0; c < hc; ++c) *reinterpret_cast<uint4*>(h + ((size_t)row * hc + c) * d + col) = v;
}

// rows flagged in `mask` take their input embedding from `override` (image tokens: the vision tower's output or
// one of the learned delimiter vectors) instead of the embedding table
__global__ void embed_override_kernel(const __nv_bfloat16* override_rows, const uint8_t* mask, __nv_bfloat16* h, int hc, int d) {
  const int row = blockIdx.y;
  if (!mask[row]) return;
  const int col = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (col >= d) return;
  const uint4 v = *reinterpret_cast<const uint4*>(override_rows + (size_t)row * d + col);
  for (int c = 0; c < hc; ++c) *reinterpret_cast<uint4*>(h + ((size_t)row * hc + c) * d + col) = v;
}

// Markov head of the draft block: logits[row, v] += dot(head[v, :], embed[prev, :]) with prev read from device memory
// (the token sampled for the previous block position), one warp per vocabulary entry.
__global__ void __launch_bounds__(256) markov_bias_kernel(float* logits, const __nv_bfloat16* head, const __nv_bfloat16* embed,
                                                         const int* prev, int vl, int r, int vocab) {
  const int v = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (v >= vl) return;
  int p = *prev;
  if (p < 0 || p >= vocab) p = 0;
  float s = 0.f;
  for (int i = lane; i < r; i += 32) s += bf16_to_f(head[(size_t)v * r + i]) * bf16_to_f(embed[(size_t)p * r + i]);
  s = warp_sum(s);
  if (lane == 0) logits[v] += s;
}

// tap[row, :] = bf16(mean over copies of h[row, c, :])
__global__ void tap_mean_kernel(const __nv_bfloat16* h, __nv_bfloat16* tap, int64_t tap_stride, int hc, int d) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.y;
  const int col = blockIdx.x * blockDim.x + threadIdx.x;
  if (col >= d) return;
  float s = 0.f;
  for (int c = 0; c < hc; ++c) s += bf16_to_f(h[((size_t)row * hc + c) * d + col]);
  tap[(size_t)row * tap_stride + col] = __float2bfloat16_rn(s / (float)hc);
}

// rope[row, v, p] = (cos, sin)(angle) with angle = ((pos / ratio_v) * ratio_v) * inv_freq_v[p], evaluated in
// double once per step; every layer's kernels read this table instead of calling sincos themselves.
struct RopeTableArgs {
  const double* inv_freq[4];
  int ratio[4];
  int V, half;
  const int* row_pos;
  float2* out;  // [n, V, half]
};
__global__ void rope_table_kernel(RopeTableArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  const int pos = a.row_pos[row];
  for (int i = threadIdx.x; i < a.V * a.half; i += blockDim.x) {
    const int v = i / a.half, p = i - v * a.half;
    const int pp = (pos / a.ratio[v]) * a.ratio[v];
    double s, c;
    sincos((double)pp * a.inv_freq[v][p], &s, &c);
    a.out[((size_t)row * a.V + v) * a.half + p] = make_float2((float)c, (float)s);
  }
}

// L2 prefetch of a weight range: decode kernels are short and latency-bound, so the next kernel's weights are
// pulled into L2 on a side stream while the current one runs (reference: kernels/prefetch_sm121.cuh:44,
// opt_rows prefetch_l2:2508 - the same instruction, there issued under the all-reduce).
__global__ void prefetch_l2_kernel(const uint8_t* p, size_t bytes) {
  const size_t off = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 2048;
  if (off >= bytes) return;
  size_t sz = bytes - off < 2048 ? bytes - off : 2048;
  sz &= ~(size_t)15;
  if (sz) asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(p + off), "r"((uint32_t)sz) : "memory");
}
// the same for the experts a row selected: expert e occupies [base + e*stride, +bytes)
__global__ void prefetch_experts_kernel(const uint8_t* base, size_t stride, size_t bytes, const int* ids, int k) {
  const int e = ids[blockIdx.y];  // blockIdx.y indexes (row, slot) pairs: ids is [rows*k] flattened
  const size_t off = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 2048;
  if (off >= bytes) return;
  size_t sz = bytes - off < 2048 ? bytes - off : 2048;
  sz &= ~(size_t)15;
  if (sz) asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(base + (size_t)e * stride + off), "r"((uint32_t)sz) : "memory");
}

// ---- synthetic weights: bytes from a hash of (tensor seed, element index) ----------------------------------
// fp8: E4M3 codes of ~N(0, sigma) values pre-divided by the block scale 2^(scale_code-127).
__global__ void synth_fp8_kernel(uint8_t* q, int64_t count, uint64_t seed, float sigma_over_scale) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i * 4 >= count) return;
  uint64_t h = splitmix64(seed ^ (uint64_t)i);
  // four values per hash: each from the sum of four 4-bit uniforms (approximately normal)
  uint32_t packed = 0;
  for (int j = 0; j < 4; ++j) {
    uint32_t bits = (uint32_t)(h >> (16 * j)) & 0xffffu;
    float s = (float)((bits & 15) + ((bits >> 4) & 15) + ((bits >> 8) & 15) + ((bits >> 12) & 15)) - 30.f;
    float v = s * (1.f / 9.2195f) * sigma_over_scale;  // var of the sum = 4 * (255/12) = 85 -> std 9.2195
    packed |= (uint32_t)enc_e4m3(v) << (8 * j);
  }
  if (i * 4 + 3 < count) *reinterpret_cast<uint32_t*>(q + i * 4) = packed;
  else for (int j = 0; i * 4 + j < count; ++j) q[i * 4 + j] = (uint8_t)(packed >> (8 * j));
}

// fp4: packed E2M1 codes of ~N(0, sigma)/scale values, 8 per 32-bit word
__global__ void synth_fp4_kernel(uint32_t* q, int64_t words, uint64_t seed, float sigma_over_scale) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= words) return;
  uint64_t h0 = splitmix64(seed ^ (uint64_t)(2 * i)), h1 = splitmix64(seed ^ (uint64_t)(2 * i + 1));
  uint32_t packed = 0;
  for (int j = 0; j < 8; ++j) {
    uint32_t bits = (uint32_t)((j < 4 ? h0 : h1) >> (16 * (j & 3))) & 0xffffu;
    float s = (float)((bits & 15) + ((bits >> 4) & 15) + ((bits >> 8) & 15) + ((bits >> 12) & 15)) - 30.f;
    float v = s * (1.f / 9.2195f) * sigma_over_scale;
    packed |= (uint32_t)f32_to_e2m1(v) << (4 * j);
  }
  q[i] = packed;
}

__global__ void synth_bf16_kernel(__nv_bfloat16* w, int64_t count, uint64_t seed, float sigma, float mean) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= count) return;
  uint64_t h = splitmix64(seed ^ (uint64_t)i);
  uint32_t bits = (uint32_t)h;
  float s = 0.f;
  for (int j = 0; j < 8; ++j) s += (float)((bits >> (4 * j)) & 15);
  w[i] = __float2bfloat16_rn(mean + (s - 60.f) * (1.f / 13.038f) * sigma);  // std of sum of 8 = 13.038
}

__global__ void synth_f32_kernel(float* w, int64_t count, uint64_t seed, float sigma, float mean) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= count) return;
  uint64_t h = splitmix64(seed ^ (uint64_t)i);
  uint32_t bits = (uint32_t)h;
  float s = 0.f;
  for (int j = 0; j < 8; ++j) s += (float)((bits >> (4 * j)) & 15);
  w[i] = mean + (s - 60.f) * (1.f / 13.038f) * sigma;
}

}  // namespace sfb

using namespace sfb;

extern "C" {

int sfb_embed(const void* embed, const int* tokens, void* h, int n, int hc, int d, int vocab, void* status,
              cudaStream_t stream) {
  if (d % 8) return (int)cudaErrorInvalidValue;
  embed_kernel<<<dim3((d / 8 + 127) / 128, n), 128, 0, stream>>>((const __nv_bfloat16*)embed, tokens,
                                                               (__nv_bfloat16*)h, n, hc, d, vocab, (Status*)status);
  return SFB_CHECK_LAUNCH();
}

int sfb_markov_bias(void* logits_row, const void* head, const void* embed, const int* prev, int vl, int r, int vocab, cudaStream_t stream) {
  markov_bias_kernel<<<(vl + 7) / 8, 256, 0, stream>>>((float*)logits_row, (const __nv_bfloat16*)head, (const __nv_bfloat16*)embed, prev, vl, r, vocab);
  return SFB_CHECK_LAUNCH();
}

int sfb_embed_override(const void* override_rows, const void* mask, void* h, int n, int hc, int d, cudaStream_t stream) {
  if (d % 8) return (int)cudaErrorInvalidValue;
  embed_override_kernel<<<dim3((d / 8 + 127) / 128, n), 128, 0, stream>>>((const __nv_bfloat16*)override_rows, (const uint8_t*)mask,
                                                                        (__nv_bfloat16*)h, hc, d);
  return SFB_CHECK_LAUNCH();
}

// variants: V <= 4 (inv_freq device pointer, ratio) pairs
int sfb_rope_table(const double* const* inv_freq, const int* ratio, int V, int half, const int* row_pos, void* out,
                   int n, cudaStream_t stream) {
  if (V < 1 || V > 4) return (int)cudaErrorInvalidValue;
  RopeTableArgs a{};
  for (int v = 0; v < V; ++v) { a.inv_freq[v] = inv_freq[v]; a.ratio[v] = ratio[v] > 0 ? ratio[v] : 1; }
  a.V = V; a.half = half; a.row_pos = row_pos; a.out = (float2*)out;
  return (int)sfb_launch(rope_table_kernel, dim3(n), dim3(128), 0, stream, a);
}

int sfb_prefetch_l2(const void* p, int64_t bytes, cudaStream_t stream) {
  if (bytes <= 0) return 0;
  const int64_t threads = (bytes + 2047) / 2048;
  prefetch_l2_kernel<<<(unsigned)((threads + 127) / 128), 128, 0, stream>>>((const uint8_t*)p, (size_t)bytes);
  return SFB_CHECK_LAUNCH();
}

int sfb_prefetch_experts(const void* base, int64_t stride, int64_t bytes, const int* ids, int n_ids, cudaStream_t stream) {
  if (bytes <= 0 || n_ids <= 0) return 0;
  const int64_t threads = (bytes + 2047) / 2048;
  prefetch_experts_kernel<<<dim3((unsigned)((threads + 127) / 128), n_ids), 128, 0, stream>>>(
      (const uint8_t*)base, (size_t)stride, (size_t)bytes, ids, 0);
  return SFB_CHECK_LAUNCH();
}

int sfb_tap_mean(const void* h, void* tap, int64_t tap_stride, int n, int hc, int d, cudaStream_t stream) {
  return (int)sfb_launch(tap_mean_kernel, dim3((d + 255) / 256, n), dim3(256), 0, stream, (const __nv_bfloat16*)h,
                         (__nv_bfloat16*)tap, tap_stride, hc, d);
}

// kind: 0 fp8 bytes, 1 fp4 bytes (count = bytes), 2 bf16 elements, 3 f32 elements
int sfb_synth_fill(int kind, void* dst, int64_t count, uint64_t seed, float sigma, float mean,
                   cudaStream_t stream) {
  const int T = 256;
  if (kind == 0) {
    int64_t thr = (count + 3) / 4;
    synth_fp8_kernel<<<(unsigned)((thr + T - 1) / T), T, 0, stream>>>((uint8_t*)dst, count, seed, sigma);
  } else if (kind == 1) {
    if (count % 4) return (int)cudaErrorInvalidValue;
    int64_t words = count / 4;
    synth_fp4_kernel<<<(unsigned)((words + T - 1) / T), T, 0, stream>>>((uint32_t*)dst, words, seed, sigma);
  } else if (kind == 2) {
    synth_bf16_kernel<<<(unsigned)((count + T - 1) / T), T, 0, stream>>>((__nv_bfloat16*)dst, count, seed, sigma, mean);
  } else if (kind == 3) {
    synth_f32_kernel<<<(unsigned)((count + T - 1) / T), T, 0, stream>>>((float*)dst, count, seed, sigma, mean);
  } else return (int)cudaErrorInvalidValue;
  return SFB_CHECK_LAUNCH();
}

int sfb_device_info(int* sm_count, int* cc_major, int* cc_minor, int64_t* total_mem) {
  cudaDeviceProp p;
  int dev = 0;
  int e = (int)cudaGetDevice(&dev);
  if (e) return e;
  e = (int)cudaGetDeviceProperties(&p, dev);
  if (e) return e;
  *sm_count = p.multiProcessorCount; *cc_major = p.major; *cc_minor = p.minor; *total_mem = (int64_t)p.totalGlobalMem;
  return 0;
}

}  // extern "C"
