// Latent attention of single rows and short runs, bf16, on tcgen05: every head of a row scores the same cached vectors (latent and shared
// key part), and sums the latents, so a block of 128 keys is one operand for all of them.
//
// One CTA: one row x one block of two pages (128 positions) x up to NH heads.  The keys are the M = 128 side of both products and lie in
// shared memory once, in 64-dim slabs that TMA fetches page by page:
//   scores   S [128 keys x NH] = K [128 x (rank + rot)] Q^T            keys K-major, queries [NH rows] K-major
//   output   O [rank x NH]     = C^T [rank x 128 keys] P^T             the same slabs MN-major, 128 latent dims per product
// Scores go through shared memory to the threads of a head, 32-bit softmax over the block, and the weights return as two bf16 terms (16
// mantissa bits).  A block leaves (maximum, sum, output); head_proj (k_rows_latent.cu) merges the blocks of a row on its way through W_uv.
//
// Every wait is bounded and reports through the status word; no cluster, no multicast.
#include "k_rows_tc.cuh"

namespace sfb {
namespace rld {
using namespace tc;

constexpr int KEYS = 128, SLAB = KEYS * 128, PSLAB = 64 * 128, THREADS = 128;

struct Args {
  const int* table;
  const int *row_lane, *row_pos;
  const int* rows;          // row of every launch row, or null
  float* part;              // [launch rows, H, blocks, rank]
  float* ml;                // [launch rows, H, blocks, 2]
  int max_pages, n_pages, H, rank, rot, window, blocks, q_row0;     // q_row0: row of the maps where the launch's queries begin
  float scale;
  Status* status;
};

struct Ctl {
  uint64_t full, done;
  uint32_t tmem;
  int dead;
};

template <int NH>
__global__ void __launch_bounds__(THREADS)
latent_block_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mqr, const __grid_constant__ CUtensorMap mc,
                    const __grid_constant__ CUtensorMap mr, Args a) {
  extern __shared__ __align__(1024) uint8_t sm[];
  const int nl = (a.rank + 63) / 64, nsl = nl + 1, nb = (nl + 1) / 2;       // latent slabs, all slabs, blocks of 128 latent dims
  constexpr int QSLAB = NH * 128, SROW = KEYS + 4;
  uint8_t* ks = sm;                                       // [nsl] slabs
  uint8_t* qs = ks + (size_t)nsl * SLAB;                  // [nsl] slabs of NH rows
  uint8_t* ph = qs + (size_t)nsl * QSLAB;                 // weights: [2 terms][2] slabs of NH rows
  float* sc = reinterpret_cast<float*>(ph + 4 * QSLAB);   // [NH][SROW]
  Ctl& C = *reinterpret_cast<Ctl*>(sc + NH * SROW);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  volatile int* dead = &C.dead;
  if (tid == 0) {
    C.dead = 0;
    mbar_init(&C.full, 1);
    mbar_init(&C.done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], 256;" ::"r"(smem_u32(&C.tmem)) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_launch_dependents();
  fence_before();
  __syncthreads();
  fence_after();
  pdl_wait();
  const int lr = blockIdx.y, h0 = blockIdx.z * NH, nh = min(NH, a.H - h0);
  const int row = a.rows ? a.rows[lr] : lr, pos = a.row_pos[row], first = max(0, pos - a.window + 1);
  const int p0 = first / 64 + 2 * blockIdx.x, pl = pos / 64;               // first page of the block, last page of the row
  bool ok = true;
  if (p0 <= pl) {
    const uint32_t ts = C.tmem, to = ts + NH, lanes = (uint32_t)(warp * 32) << 16;
    if (warp == 0 && elect_one()) {
      mbar_expect(&C.full, nsl * (SLAB + QSLAB));
      const int* tab = a.table + (size_t)a.row_lane[row] * a.max_pages;
      for (int w = 0; w < 2; ++w) {
        int page = tab[min(p0 + w, pl)];                  // a page past the row's last is masked: the last one stands in for it
        if (page < 0 || page >= a.n_pages) { status_set(a.status, ST_BOUNDS, 71, page, a.n_pages); page = 0; }
        for (int s = 0; s < nl; ++s) tma2d(ks + (size_t)s * SLAB + w * PSLAB, &mc, 64 * s, page * 64, &C.full);
        tma2d(ks + (size_t)nl * SLAB + w * PSLAB, &mr, 0, page * 64, &C.full);
      }
      for (int s = 0; s < nl; ++s) tma2d(qs + (size_t)s * QSLAB, &mq, 64 * s, a.q_row0 + lr * a.H + h0, &C.full);
      tma2d(qs + (size_t)nl * QSLAB, &mqr, 0, a.q_row0 + lr * a.H + h0, &C.full);
    }
    ok = __syncthreads_and(mbar_wait(&C.full, 0, dead));
    if (ok) {
      fence_after();
      if (warp == 0 && elect_one()) {
        const uint64_t dk = desc(smem_u32(ks), 16), dq = desc(smem_u32(qs), 16);
        const uint32_t id = idesc(NH, 0, 0);
        const int kl = (a.rank + 15) / 16, kr = (a.rot + 15) / 16;
        for (int t = 0; t < kl; ++t) mma_ss(ts, dk + (t >> 2) * (SLAB >> 4) + (t & 3) * 2, dq + (t >> 2) * (QSLAB >> 4) + (t & 3) * 2, id, t ? 1u : 0u);
        for (int t = 0; t < kr; ++t) mma_ss(ts, dk + nl * (SLAB >> 4) + t * 2, dq + nl * (QSLAB >> 4) + t * 2, id, 1u);
        commit(&C.done);
      }
      ok = __syncthreads_and(mbar_wait(&C.done, 0, dead));
    }
    if (ok) {
      fence_after();
      {  // lane = key
        const int j = p0 * 64 + tid, dist = pos - j;
        const bool vis = dist >= 0 && dist < a.window;
        const float sl = a.scale * LOG2E;
#pragma unroll
        for (int b = 0; b < NH / 16; ++b) {
          float s[16];
          ld16(ts + 16 * b + lanes, s);
          wait_ld();
#pragma unroll
          for (int k = 0; k < 16; ++k) sc[(16 * b + k) * SROW + tid] = vis ? s[k] * sl : -INFINITY;
        }
      }
      __syncthreads();
      // TPH neighbouring threads per head, KPT keys each, in units of eight keys that lie TPH units apart
      constexpr int TPH = THREADS / NH, KPT = KEYS / TPH;
      const int hh = tid / TPH, q = tid % TPH;
      float v[KPT], m = -INFINITY, l = 0.f;
#pragma unroll
      for (int u = 0; u < KPT / 8; ++u)
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          v[8 * u + k] = sc[hh * SROW + (u * TPH + q) * 8 + k];
          m = fmaxf(m, v[8 * u + k]);
        }
#pragma unroll
      for (int o = 1; o < TPH; o <<= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float ref = m == -INFINITY ? 0.f : m;         // a second page without visible keys cannot be: the block's first page has one
#pragma unroll
      for (int k = 0; k < KPT; ++k) { v[k] = ex2(v[k] - ref); l += v[k]; }
#pragma unroll
      for (int o = 1; o < TPH; o <<= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
#pragma unroll
      for (int u = 0; u < KPT / 8; ++u) {
        const int c = u * TPH + q;                        // unit of eight keys: slab c / 8, unit c % 8 of the slab's row
        uint4 hi, lo;
        split2(v[8 * u], v[8 * u + 1], hi.x, lo.x); split2(v[8 * u + 2], v[8 * u + 3], hi.y, lo.y);
        split2(v[8 * u + 4], v[8 * u + 5], hi.z, lo.z); split2(v[8 * u + 6], v[8 * u + 7], hi.w, lo.w);
        uint8_t* d = ph + (c >> 3) * QSLAB + hh * 128 + (((c & 7) ^ (hh & 7)) * 16);
        *reinterpret_cast<uint4*>(d) = hi;
        *reinterpret_cast<uint4*>(d + 2 * QSLAB) = lo;
      }
      const size_t at = ((size_t)lr * a.H + h0 + hh) * a.blocks + blockIdx.x;
      if (q == 0 && hh < nh) { a.ml[2 * at] = m; a.ml[2 * at + 1] = l; }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      fence_before();
      __syncthreads();
      fence_after();
      if (warp == 0 && elect_one()) {
        const uint64_t dp = desc(smem_u32(ph), 16);
        const uint32_t id = idesc(NH, 1, 0);
        for (int b = 0; b < nb; ++b) {
          const uint64_t dc = desc(smem_u32(ks) + 2 * b * SLAB, SLAB);
          for (int t = 0; t < 16; ++t)                    // eight steps of 16 keys with the upper terms, then with the lower ones
            mma_ss(to + b * NH, dc + (uint64_t)(t & 7) * (2048 >> 4), dp + ((t >> 3) * 2 + ((t & 7) >> 2)) * (QSLAB >> 4) + (t & 3) * 2, id, t ? 1u : 0u);
        }
        commit(&C.done);
      }
      ok = __syncthreads_and(mbar_wait(&C.done, 1, dead));
    }
    if (ok) {
      fence_after();
      for (int b = 0; b < nb; ++b) {
        const int d = b * 128 + tid;
#pragma unroll
        for (int c = 0; c < NH / 16; ++c) {
          float o[16];
          ld16(to + b * NH + 16 * c + lanes, o);
          wait_ld();
          if (d < a.rank) {
#pragma unroll
            for (int k = 0; k < 16; ++k)
              if (16 * c + k < nh) a.part[(((size_t)lr * a.H + h0 + 16 * c + k) * a.blocks + blockIdx.x) * a.rank + d] = o[k];
          }
        }
      }
    }
    if (C.dead && tid == 0)
      for (int i = 0; i < 100000; ++i) __nanosleep(64);   // copies and products under way end before the CTA does
  }
  fence_before();
  __syncthreads();
  if (tid == 0 && C.dead) status_set(a.status, ST_TIMEOUT, 72, blockIdx.x, blockIdx.y);
  if (warp == 0) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, 256;" ::"r"(C.tmem) : "memory");
}

template <int NH>
static size_t smem_bytes(const Args& a) {
  const size_t nsl = (a.rank + 63) / 64 + 1;
  return nsl * (SLAB + NH * 128) + 4 * NH * 128 + (size_t)NH * (KEYS + 4) * 4 + sizeof(Ctl);
}
template <int NH>
static int launch(const CUtensorMap* q, const CUtensorMap* qr, const CUtensorMap* c, const CUtensorMap* r, const Args& a, int n, cudaStream_t st) {
  const size_t smem = smem_bytes<NH>(a);
  static size_t granted = 0;
  if (smem > granted) {
    const cudaError_t e = cudaFuncSetAttribute(latent_block_kernel<NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    granted = smem;
  }
  return (int)sfb_launch(latent_block_kernel<NH>, dim3(a.blocks, n, (a.H + NH - 1) / NH), dim3(THREADS), smem, st, *q, *qr, *c, *r, a);
}

}  // namespace rld
}  // namespace sfb

using namespace sfb;
using namespace sfb::rld;

extern "C" {

// heads (16 or 32) a block takes: the box height of mq and mqr
int sfb_rows_latent_heads(int H) { return H <= 16 ? 16 : 32; }

// mq, mqr: latent and shared parts of the queries, rows = launch row x H + head; mc, mr: the same of the pool, rows = page x 64 + slot, boxes
// of 64 rows.  blocks: at least the pairs of pages that a row's window touches.  rank: a multiple of 8 up to 512, rot a multiple of 8 up to 64.
int sfb_rows_latent_decode(const void* mq, const void* mqr, const void* mc, const void* mr, const int* table, const int* row_lane, const int* row_pos,
                           const int* rows, void* part, void* ml, int max_pages, int n_pages, int n, int H, int rank, int rot, int window, int blocks, int q_row0,
                           float scale, void* status, cudaStream_t stream) {
  if (n < 1 || n > 65535 || H < 1 || rank < 8 || rank % 8 || rank > 512 || rot < 8 || rot % 8 || rot > 64 || window < 1 || blocks < 1)
    return (int)cudaErrorInvalidValue;
  Args a{table, row_lane, row_pos, rows, (float*)part, (float*)ml, max_pages, n_pages, H, rank, rot, window, blocks, q_row0, scale, (Status*)status};
  const CUtensorMap *q = (const CUtensorMap*)mq, *qr = (const CUtensorMap*)mqr, *c = (const CUtensorMap*)mc, *r = (const CUtensorMap*)mr;
  return sfb_rows_latent_heads(H) == 16 ? launch<16>(q, qr, c, r, a, n, stream) : launch<32>(q, qr, c, r, a, n, stream);
}

}  // extern "C"
