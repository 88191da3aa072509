// Stateless Gumbel-max sampling over a vocabulary slice and the fold of several ranks' winners.
//
// Reference behaviour: kernels/opt_rows_sm121.cu argmax_fold:1810 / argmax_pick:1834, kernels/opt_sample_sm121.cuh (noise keyed
// on seed, position, token id).
#include <cooperative_groups.h>

#include "k_common.cuh"

namespace sfb {

__device__ __forceinline__ float gumbel(uint64_t base, int id) {
  const uint64_t h = splitmix64(base ^ ((uint64_t)id * 0x9E3779B97F4A7C15ull));
  const double u = ((double)(h >> 40) + 0.5) * (1.0 / 16777216.0);
  return (float)(-log(-log(u)));
}

struct SampleArgs {
  const float* logits;    // [n, V] this rank's vocabulary slice
  int64_t stride;
  const int* row_pos;     // sampling position = row_pos + 1 (the position the new token will occupy)
  const float* temperature;  // [n]
  const uint64_t* seed;      // [n]
  const uint8_t* mask;    // optional [n, mask_stride] allowed-token bytes (constrained decoding), 0 = banned
  int64_t mask_stride;
  float* best_val;        // [n]
  int* best_id;           // [n] global token id
  int V, vocab_offset;
};

constexpr int SAMPLE_CLUSTER = 8;   // CTAs per row: each scans an eighth of the vocabulary slice, CTA 0 merges through DSMEM

__global__ void __cluster_dims__(SAMPLE_CLUSTER, 1, 1) __launch_bounds__(1024) sample_kernel(SampleArgs a) {
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sv[32];
  __shared__ int si[32];
  __shared__ float cv[SAMPLE_CLUSTER];
  __shared__ int ci[SAMPLE_CLUSTER];
  const int row = blockIdx.y, part = blockIdx.x;   // part == rank in the cluster
  const float T = a.temperature[row];
  const bool greedy = T < 1e-5f;
  const uint64_t base = splitmix64(a.seed[row] ^ splitmix64((uint64_t)(a.row_pos[row] + 1)));
  float bv = -INFINITY;
  int bi = 0x7fffffff;
  // (value, lowest id) is a total order, so the winner does not depend on how the slice is cut
  for (int i = part * 1024 + threadIdx.x; i < a.V; i += 1024 * SAMPLE_CLUSTER) {
    const int id = a.vocab_offset + i;
    if (a.mask && a.mask[(size_t)row * a.mask_stride + id] == 0) continue;
    float v = a.logits[(size_t)row * a.stride + i];
    if (!greedy) v = v / T + gumbel(base, id);
    if (v > bv || (v == bv && id < bi)) { bv = v; bi = id; }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
  }
  if ((threadIdx.x & 31) == 0) { sv[threadIdx.x >> 5] = bv; si[threadIdx.x >> 5] = bi; }
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int w = 1; w < 32; ++w)
      if (sv[w] > bv || (sv[w] == bv && si[w] < bi)) { bv = sv[w]; bi = si[w]; }
    *cluster.map_shared_rank(&cv[part], 0) = bv;
    *cluster.map_shared_rank(&ci[part], 0) = bi;
  }
  cluster.sync();
  if (part == 0 && threadIdx.x == 0) {
    bv = cv[0]; bi = ci[0];
    for (int p = 1; p < SAMPLE_CLUSTER; ++p)
      if (cv[p] > bv || (cv[p] == bv && ci[p] < bi)) { bv = cv[p]; bi = ci[p]; }
    a.best_val[row] = bv;
    a.best_id[row] = bi;
  }
}

// Fold W ranks' (value, id) winners: larger value wins, ties to the lower id.  vals / ids are [W, stride].
// With flags the kernel first waits (bounded) until every rank's winners have arrived.
struct FoldBestArgs {
  const float* vals;
  const int* ids;
  int W, n, stride;
  int* out_tokens;
  const uint32_t* flags[8];
  const uint32_t* epoch_ptr;
  uint32_t epoch_add;
  uint64_t wait_ns;
  Status* status;
};
__global__ void sample_fold_kernel(FoldBestArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  if (a.flags[0] != nullptr) {
    const uint32_t want = *a.epoch_ptr + a.epoch_add;
    if (threadIdx.x < a.W && !wait_flag_ge(a.flags[threadIdx.x], want, a.wait_ns))
      status_set(a.status, ST_TIMEOUT, 4, threadIdx.x, (int)want);
    __syncthreads();
  }
  for (int row = threadIdx.x; row < a.n; row += blockDim.x) {
    float bv = a.vals[row];
    int bi = a.ids[row];
    for (int r = 1; r < a.W; ++r) {
      const float v = a.vals[(size_t)r * a.stride + row];
      const int id = a.ids[(size_t)r * a.stride + row];
      if (v > bv || (v == bv && id < bi)) { bv = v; bi = id; }
    }
    a.out_tokens[row] = bi;
  }
}

}  // namespace sfb

using namespace sfb;

extern "C" {

int sfb_sample(const float* logits, int64_t stride, const int* row_pos, const float* temperature,
               const void* seed, const void* mask, int64_t mask_stride, float* best_val, int* best_id, int n,
               int V, int vocab_offset, cudaStream_t stream) {
  SampleArgs a{logits, stride, row_pos, temperature, (const uint64_t*)seed, (const uint8_t*)mask, mask_stride,
               best_val, best_id, V, vocab_offset};
  return (int)sfb_launch(sample_kernel, dim3(SAMPLE_CLUSTER, n), dim3(1024), 0, stream, a);
}

int sfb_sample_fold(const void* vals, const void* ids, int W, int n, int stride, int* out_tokens,
                    const void* const* flag_ptrs, const void* epoch_ptr, uint32_t epoch_add, uint64_t wait_ns,
                    void* status, cudaStream_t stream) {
  if (W < 1 || W > 8) return (int)cudaErrorInvalidValue;
  FoldBestArgs a{};
  a.vals = (const float*)vals; a.ids = (const int*)ids; a.W = W; a.n = n; a.stride = stride; a.out_tokens = out_tokens;
  for (int r = 0; r < 8; ++r) a.flags[r] = (flag_ptrs && r < W) ? (const uint32_t*)flag_ptrs[r] : nullptr;
  a.epoch_ptr = (const uint32_t*)epoch_ptr; a.epoch_add = epoch_add; a.wait_ns = wait_ns ? wait_ns : 2000000000ull;
  a.status = (Status*)status;
  return (int)sfb_launch(sample_fold_kernel, dim3(1), dim3(64), 0, stream, a);
}

}  // extern "C"
