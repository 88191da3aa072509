// What the tensor-core kernels of the matrix-state recurrences share (k_rows_state_tc.cu, k_rows_delta_tc.cu): chunk sizes, barriers, bounded
// waits of whole warps, tensor memory.
#pragma once
#include "k_rows_tc.cuh"

namespace sfb {
namespace rst {
using namespace tc;

constexpr int L = 128, SLAB = L * 128, HSLAB = 64 * 128;         // rows of a chunk; bytes of 128 / 64 rows of 64 elements
constexpr int WORK = 256, THREADS = WORK + 32;                   // threads that compute, and one warp that issues copies and products

// Numbers per (chunk, head) of the delta rule, [RATES][128]: running sum c of log2 of the decays; c less log2 of k's factor to unit length;
// q's factor; 2^c times k's factor; write strength; decay to the chunk's end times k's factor
constexpr int RATES = 6;

struct Ctl {
  uint64_t full[3], done[3];       // copies; products (chunk_out: weighted ones, scores - a barrier each, since the next head's scores are issued
                                   // before every thread has seen the products end)
  uint32_t tmem;
  int dead;
};

__device__ __forceinline__ void setup(Ctl& C, uint32_t cols) {
  if (threadIdx.x == 0) {
    C.dead = 0;
    for (int i = 0; i < 3; ++i) mbar_init(&C.full[i], 1);
    for (int i = 0; i < 3; ++i) mbar_init(&C.done[i], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (threadIdx.x < 32) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&C.tmem)), "r"(cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  fence_before();
  __syncthreads();
  fence_after();
}
__device__ __forceinline__ void teardown(Ctl& C, uint32_t cols, Status* status, int where) {
  fence_before();
  __syncthreads();
  if (threadIdx.x == 0 && C.dead) status_set(status, ST_TIMEOUT, where, C.dead, blockIdx.y << 16 | blockIdx.x);
  if (threadIdx.x < 32) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(C.tmem), "r"(cols) : "memory");
}

// a wait of whole warps: what follows it is executed by all lanes together
// `id`: what the status word says if the wait gives up.
__device__ __forceinline__ void wait_warp(uint64_t* b, uint32_t parity, volatile int* dead, int id) {
  if (!mbar_wait(b, parity, dead) && *dead == 1) *dead = id;
  __syncwarp();
}
// sixteen values as one 32-byte store (a whole sector)
__device__ __forceinline__ void store32(__nv_bfloat16* p, const float* f) {
  uint32_t w[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) { const __nv_bfloat162 t = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]); w[i] = *reinterpret_cast<const uint32_t*>(&t); }
  asm volatile("st.global.v8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(p), "r"(w[0]), "r"(w[1]), "r"(w[2]), "r"(w[3]), "r"(w[4]), "r"(w[5]), "r"(w[6]),
               "r"(w[7]) : "memory");
}
// after a wait that gave up: copies and products under way must end before the CTA does (bounded: a phase that never comes is not waited for)
__device__ __forceinline__ void drain(Ctl& C) {
  if (!C.dead) return;
  if (threadIdx.x == 0)
    for (int i = 0; i < 100000; ++i) __nanosleep(64);
}

template <typename K>
static cudaError_t grant(K kernel, size_t smem, size_t& granted) {
  if (smem <= granted) return cudaSuccess;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e == cudaSuccess) granted = smem;
  return e;
}
}  // namespace rst
}  // namespace sfb
