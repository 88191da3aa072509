// Latent attention of single rows and short runs, bf16, on tcgen05: every head of a row scores the same cached vectors (latent and shared
// key part), and sums the latents, so a page of 64 keys is one operand for all of them.
//
// The work is a list: the pages that the rows see, row after row, shared equally among the CTAs, so that rows of any lengths fill the machine.  A
// CTA takes up to NH heads of its pages one after another and leaves one partial result per row it touches, at place CTA + launch row: walking the
// list, either the CTA or the row goes up by one.  The keys are the M side of both products and lie in shared memory once, in 64-dim slabs that TMA
// fetches; two latent slabs are a ring stage, and two pages and more fit:
//   scores   S [64 keys x NH]  = K [64 x (rank + rot)] Q^T             keys K-major, queries [NH rows] K-major
//   output   O [rank x 2 NH]  += C^T [rank x 64 keys] P^T              the same slabs MN-major, 128 latent dims (a stage) per product
// Warp 4 copies, warp 5 issues the products (the next page's scores ahead of this page's output), warps 0-3 hold the softmax: scores go through
// shared memory to the threads of a head, 32-bit softmax over the page, and the weights return as two bf16 terms (16 mantissa bits), side by side, whose sums are added at the end.  The output stays
// in tensor memory while pages of a row go by and is rescaled only when a head's maximum grew by more than 2^8.  head_proj (k_rows_latent.cu) merges
// the (maximum, sum, output) of a row's places on its way through W_uv.
//
// Every wait is bounded and reports through the status word; no cluster, no multicast.
#include "k_rows_tc.cuh"

namespace sfb {
namespace rld {
using namespace tc;

constexpr int KEYS = 64, SLAB = KEYS * 128, STAGE = 2 * SLAB, THREADS = 192, SOFT = 128, MAX_STAGES = 12, ROWS = 256, SINGLE = 64;

struct Args {
  const int* table;
  const int *row_lane, *row_pos;
  const int* rows;          // row of every launch row, or null
  float* part;              // [places, H, rank]
  float* ml;                // [places, H, 2]
  int2* parts;              // [n] first place and number of places of every launch row
  int max_pages, n_pages, n, H, rank, rot, window, stages, q_row0;     // q_row0: row of the maps where the launch's queries begin
  float scale;
  Status* status;
};

struct Ctl {
  uint64_t full[MAX_STAGES], empty[MAX_STAGES], r_full[2], r_empty[2], q_full, q_empty, s_full[2], p_full, o_done;
  uint32_t tmem;
  int dead;
  int pre[ROWS + 1], pos[ROWS], lane[ROWS];     // pages of the rows before; position and cache lane of every row
};

// with more than SINGLE pages a share is two at least: one alone is hardly faster, and its partial result has to be merged
__host__ __device__ __forceinline__ int shares_of(int total, int ctas) {
  const int s = total > SINGLE ? (total + 1) / 2 : total;
  return s < ctas ? s : ctas;
}

// barriers of the softmax warps alone
__device__ __forceinline__ void soft_sync() { asm volatile("barrier.cta.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ bool soft_all(bool p) {
  uint32_t r;
  asm volatile("{\n\t.reg .pred a, b;\n\tsetp.ne.u32 a, %1, 0;\n\tbarrier.cta.red.and.pred b, 1, 128, a;\n\tselp.u32 %0, 1, 0, b;\n\t}" : "=r"(r) : "r"((uint32_t)p) : "memory");
  return r != 0;
}

// a place in the ring, and the parity of its round
struct Turn {
  int at = 0;
  uint32_t par = 0;
  __device__ __forceinline__ void next(int stages) {
    if (++at == stages) { at = 0; par ^= 1; }
  }
};

template <int NH>
__global__ void __launch_bounds__(THREADS, 1)
latent_pages_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mqr, const __grid_constant__ CUtensorMap mc,
                    const __grid_constant__ CUtensorMap mr, Args a) {
  extern __shared__ __align__(1024) uint8_t sm[];
  const int nl = (a.rank + 63) / 64, nsl = nl + 1, nb = (nl + 1) / 2;       // latent slabs, all slabs of a query, stages of a page
  constexpr int QSLAB = NH * 128, SROW = KEYS + 4, COLS = NH <= 16 ? 256 : 512;      // columns of tensor memory
  uint8_t* ks = sm;                                       // [stages] pairs of latent slabs
  uint8_t* kr = ks + (size_t)a.stages * STAGE;            // [2] slabs of the shared key part
  uint8_t* qs = kr + 2 * SLAB;                            // [nsl] slabs of NH rows
  uint8_t* ph = qs + (size_t)nsl * QSLAB;                 // weights: NH rows of upper terms, NH rows of lower ones
  float* sc = reinterpret_cast<float*>(ph + 2 * QSLAB);   // [NH][SROW]
  float* cr = sc + NH * SROW;                             // [NH] rescaling of the output
  Ctl& C = *reinterpret_cast<Ctl*>(cr + NH);
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;
  volatile int* dead = &C.dead;
  pdl_launch_dependents();
  if (warp == 4 && lane == 0) {
    C.dead = 0;
    for (int i = 0; i < MAX_STAGES; ++i) { mbar_init(&C.full[i], 1); mbar_init(&C.empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&C.r_full[i], 1); mbar_init(&C.r_empty[i], 1); mbar_init(&C.s_full[i], 1); }
    mbar_init(&C.q_full, 1); mbar_init(&C.q_empty, 1); mbar_init(&C.p_full, SOFT); mbar_init(&C.o_done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 5) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&C.tmem)), "n"(COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_wait();
  if (warp == 0) {
    int sum = 0;
    for (int i0 = 0; i0 < a.n; i0 += 32) {
      const int i = i0 + lane;
      int x = 0;
      if (i < a.n) {
        const int row = a.rows ? a.rows[i] : i, pos = a.row_pos[row];
        C.pos[i] = pos;
        C.lane[i] = a.row_lane[row];
        x = pos / 64 - max(0, pos - a.window + 1) / 64 + 1;
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, x, o);
        if (lane >= o) x += y;
      }
      if (i < a.n) C.pre[i + 1] = sum + x;
      sum += __shfl_sync(0xffffffffu, x, 31);
    }
    if (lane == 0) C.pre[0] = 0;
  }
  fence_before();
  __syncthreads();
  fence_after();
  const int total = C.pre[a.n], shares = shares_of(total, gridDim.x), cta = blockIdx.x, h0 = blockIdx.y * NH, nh = min(NH, a.H - h0);
  auto begin = [&](int c) { return (int)((int64_t)c * total / shares); };
  const int g0 = cta < shares ? begin(cta) : 0, g1 = cta < shares ? begin(cta + 1) : 0;
  int r0 = 0;                                             // first row of the share
  while (r0 + 1 < a.n && C.pre[r0 + 1] <= g0) ++r0;
  if (cta == 0 && blockIdx.y == 0 && warp < 4) {
    auto owner = [&](int g) { return (int)(((int64_t)(g + 1) * shares - 1) / total); };
    for (int i = tid; i < a.n; i += SOFT) {
      const int c = owner(C.pre[i]);
      a.parts[i] = make_int2(c + i, owner(C.pre[i + 1] - 1) - c + 1);
    }
  }
  const uint32_t ts = C.tmem, to = ts + 2 * NH;

  if (warp == 4) {
    if (elect_one()) {
      int n = 0, seg = 0;
      Turn turn;
      bool ok = true;
      for (int r = r0; ok && r < a.n && C.pre[r] < g1; ++r, ++seg) {
        const int b0 = max(g0 - C.pre[r], 0), b1 = min(g1, C.pre[r + 1]) - C.pre[r];
        const int* tab = a.table + (size_t)C.lane[r] * a.max_pages + max(0, C.pos[r] - a.window + 1) / 64;
        int next = tab[b0];
        if (!(ok = mbar_wait(&C.q_empty, (seg & 1) ^ 1, dead))) break;
        mbar_expect(&C.q_full, nsl * QSLAB);
        for (int s = 0; s < nl; ++s) tma2d(qs + (size_t)s * QSLAB, &mq, 64 * s, a.q_row0 + r * a.H + h0, &C.q_full);
        tma2d(qs + (size_t)nl * QSLAB, &mqr, 0, a.q_row0 + r * a.H + h0, &C.q_full);
        for (int b = b0; ok && b < b1; ++b, ++n) {
          int page = next;
          if (b + 1 < b1) next = tab[b + 1];
          if (page < 0 || page >= a.n_pages) { status_set(a.status, ST_BOUNDS, 71, page, a.n_pages); page = 0; }
          for (int j = 0; j < nb; ++j, turn.next(a.stages)) {
            const int st = turn.at, ns = min(2, nl - 2 * j);
            if (!(ok = mbar_wait(&C.empty[st], turn.par ^ 1, dead))) break;
            mbar_expect(&C.full[st], ns * SLAB);
            for (int s = 0; s < ns; ++s) tma2d(ks + (size_t)st * STAGE + s * SLAB, &mc, 64 * (2 * j + s), page * 64, &C.full[st]);
          }
          if (!ok || !(ok = mbar_wait(&C.r_empty[n & 1], ((n >> 1) & 1) ^ 1, dead))) break;
          mbar_expect(&C.r_full[n & 1], SLAB);
          tma2d(kr + (n & 1) * SLAB, &mr, 0, page * 64, &C.r_full[n & 1]);
        }
      }
    }
  } else if (warp == 5) {
    if (elect_one()) {
      const uint64_t dk = desc(smem_u32(ks), 16), dr = desc(smem_u32(kr), 16), dq = desc(smem_u32(qs), 16), dc = desc(smem_u32(ks), SLAB), dp = desc(smem_u32(ph), 16);
      const uint32_t id_s = idesc(NH, 0, 0, KEYS), id_o = idesc(2 * NH, 1, 0);
      const int kl = (a.rank + 15) / 16, krot = (a.rot + 15) / 16, pages = g1 - g0;
      int rs = r0, seg = 0;                               // row of the page whose scores are issued next
      Turn in, out;                                       // stages of the scores, of the output
      bool ok = true;
      auto scores = [&](int n) {                          // of the share's page n
        if (n == 0 || g0 + n == C.pre[rs + 1]) {
          if (n) { ++rs; ++seg; }
          if (!mbar_wait(&C.q_full, seg & 1, dead)) return false;
        }
        const uint32_t d = ts + (n & 1) * NH;
        for (int j = 0; j < nb; ++j, in.next(a.stages)) {
          const int st = in.at;
          if (!mbar_wait(&C.full[st], in.par, dead)) return false;
          fence_after();
          const uint64_t k = dk + st * (STAGE >> 4), q = dq + j * (2 * QSLAB >> 4);
#pragma unroll
          for (int t = 0; t < 8; ++t)
            if (8 * j + t < kl) mma_ss(d, k + (t >> 2) * (SLAB >> 4) + (t & 3) * 2, q + (t >> 2) * (QSLAB >> 4) + (t & 3) * 2, id_s, (j | t) ? 1u : 0u);
        }
        if (!mbar_wait(&C.r_full[n & 1], (n >> 1) & 1, dead)) return false;
        fence_after();
        const uint64_t k = dr + (n & 1) * (SLAB >> 4), q = dq + nl * (QSLAB >> 4);
#pragma unroll
        for (int t = 0; t < 4; ++t)
          if (t < krot) mma_ss(d, k + t * 2, q + t * 2, id_s, 1u);
        commit(&C.r_empty[n & 1]);
        if (g0 + n + 1 == C.pre[rs + 1] || n + 1 == pages) commit(&C.q_empty);
        commit(&C.s_full[n & 1]);
        return true;
      };
      int ro = r0;                                        // row of the page whose output is issued next
      if (pages > 0) ok = scores(0);
      for (int n = 0; ok && n < pages; ++n) {
        if (n + 1 < pages && !(ok = scores(n + 1))) break;
        if (!(ok = mbar_wait(&C.p_full, n & 1, dead))) break;
        fence_after();
        const bool fresh = n == 0 || g0 + n == C.pre[ro + 1];
        if (fresh && n) ++ro;
        for (int j = 0; j < nb; ++j, out.next(a.stages)) {
          const int st = out.at;
          const uint64_t c = dc + st * (STAGE >> 4);
#pragma unroll
          for (int t = 0; t < 4; ++t)                     // 16 keys at a time, the weights' upper and lower terms side by side
            mma_ss(to + j * 2 * NH, c + t * (2048 >> 4), dp + t * 2, id_o, t ? 1u : fresh ? 0u : 1u);
          commit(&C.empty[st]);
        }
        commit(&C.o_done);
      }
      // no arrival may be under way when the CTA ends
      for (int i = max(0, pages * nb - a.stages); ok && i < pages * nb; ++i) ok = mbar_wait(&C.empty[i % a.stages], (i / a.stages) & 1, dead);
      for (int n = max(0, pages - 2); ok && n < pages; ++n) ok = mbar_wait(&C.r_empty[n & 1], (n >> 1) & 1, dead);
      if (ok && pages > 0) ok = mbar_wait(&C.q_empty, seg & 1, dead);
    }
  } else {
    // TPH neighbouring threads per head, KPT keys each, in units of eight keys that lie TPH units apart
    constexpr int TPH = SOFT / NH, KPT = KEYS / TPH;
    const int hh = tid / TPH, q = tid % TPH;
    const uint32_t lanes = (uint32_t)(warp * 32) << 16;
    const float sl = a.scale * LOG2E;
    int n = 0;
    bool ok = true;
    for (int r = r0; ok && r < a.n && C.pre[r] < g1; ++r) {
      const int pos = C.pos[r], p0 = max(0, pos - a.window + 1) / 64;
      const int b0 = max(g0 - C.pre[r], 0), b1 = min(g1, C.pre[r + 1]) - C.pre[r];
      float m = -INFINITY, l = 0.f;                       // of this thread's head
      for (int b = b0; b < b1; ++b, ++n) {
        if (!(ok = soft_all(mbar_wait(&C.s_full[n & 1], (n >> 1) & 1, dead)))) break;
        fence_after();
        {  // the first 16 lanes of a warp are keys
          const int key = warp * 16 + lane, dist = pos - ((p0 + b) * 64 + key);
          const bool vis = dist >= 0 && dist < a.window;
#pragma unroll
          for (int k0 = 0; k0 < NH; k0 += 16) {
            float s[16];
            ld16(ts + (n & 1) * NH + k0 + lanes, s);
            wait_ld();
            if (lane < 16) {
#pragma unroll
              for (int k = 0; k < 16; ++k) sc[(k0 + k) * SROW + key] = vis ? s[k] * sl : -INFINITY;
            }
          }
        }
        fence_before();
        soft_sync();
        float v[KPT], mb = -INFINITY, lb = 0.f;
#pragma unroll
        for (int u = 0; u < KPT / 8; ++u) {
          const float4 x = *reinterpret_cast<const float4*>(sc + hh * SROW + (u * TPH + q) * 8), y = *reinterpret_cast<const float4*>(sc + hh * SROW + (u * TPH + q) * 8 + 4);
          v[8 * u] = x.x; v[8 * u + 1] = x.y; v[8 * u + 2] = x.z; v[8 * u + 3] = x.w;
          v[8 * u + 4] = y.x; v[8 * u + 5] = y.y; v[8 * u + 6] = y.z; v[8 * u + 7] = y.w;
        }
#pragma unroll
        for (int k = 0; k < KPT; ++k) mb = fmaxf(mb, v[k]);
#pragma unroll
        for (int o = 1; o < TPH; o <<= 1) mb = fmaxf(mb, __shfl_xor_sync(0xffffffffu, mb, o));
        // (every page of the list has a visible key)
        float corr = 1.f;
        const bool grew = mb - m > 8.f;                   // the first page of a row too
        if (grew) { corr = ex2(m - mb); m = mb; }
        if (q == 0) cr[hh] = corr;
        const bool rescale = !soft_all(!grew) && b > b0;
#pragma unroll
        for (int k = 0; k < KPT; ++k) { v[k] = ex2(v[k] - m); lb += v[k]; }
#pragma unroll
        for (int o = 1; o < TPH; o <<= 1) lb += __shfl_xor_sync(0xffffffffu, lb, o);
        l = fmaf(l, corr, lb);
        if (b > b0) {                                     // the previous page's output: its weights have been read, its sums are there
          if (!(ok = soft_all(mbar_wait(&C.o_done, (n - 1) & 1, dead)))) break;
          if (rescale) {
            fence_after();
            for (int c = 0; c < nb * 2 * NH; c += 16) {
              float o[16];
              ld16(to + c + lanes, o);
              wait_ld();
#pragma unroll
              for (int k = 0; k < 16; ++k) o[k] *= cr[(c + k) % NH];
              st16(to + c + lanes, reinterpret_cast<const uint32_t*>(o));
            }
            wait_st();
          }
        }
#pragma unroll
        for (int u = 0; u < KPT / 8; ++u) {
          const int c = u * TPH + q;                      // unit of eight keys of the head's row
          uint4 hi, lo;
          split2(v[8 * u], v[8 * u + 1], hi.x, lo.x); split2(v[8 * u + 2], v[8 * u + 3], hi.y, lo.y);
          split2(v[8 * u + 4], v[8 * u + 5], hi.z, lo.z); split2(v[8 * u + 6], v[8 * u + 7], hi.w, lo.w);
          uint8_t* d = ph + hh * 128 + ((c ^ (hh & 7)) * 16);
          *reinterpret_cast<uint4*>(d) = hi;
          *reinterpret_cast<uint4*>(d + QSLAB) = lo;
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        fence_before();
        mbar_arrive(&C.p_full);
      }
      if (!ok || !(ok = soft_all(mbar_wait(&C.o_done, (n - 1) & 1, dead)))) break;
      fence_after();
      const size_t place = (size_t)(cta + r) * a.H + h0;
      if (q == 0 && hh < nh) { a.ml[2 * (place + hh)] = m; a.ml[2 * (place + hh) + 1] = l; }
      for (int j = 0; j < nb; ++j) {
        const int d = j * 128 + tid;
#pragma unroll
        for (int c = 0; c < NH; c += 16) {
          float o[16], o2[16];
          ld16(to + j * 2 * NH + c + lanes, o);
          ld16(to + j * 2 * NH + NH + c + lanes, o2);
          wait_ld();
          if (d < a.rank) {
#pragma unroll
            for (int k = 0; k < 16; ++k)
              if (c + k < nh) a.part[(place + c + k) * a.rank + d] = o[k] + o2[k];
          }
        }
      }
      fence_before();                                     // read before the next row's products (ordered by its weights' barrier)
    }
  }
  fence_before();
  __syncthreads();
  if (tid == 0 && *dead) {
    status_set(a.status, ST_TIMEOUT, 72, blockIdx.x, blockIdx.y);
    for (int i = 0; i < 100000; ++i) __nanosleep(64);     // copies and products under way end before the CTA does
  }
  __syncthreads();
  if (warp == 5) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(ts), "n"(COLS) : "memory");
}

template <int NH>
static int launch(const CUtensorMap* q, const CUtensorMap* qr, const CUtensorMap* c, const CUtensorMap* r, Args a, int ctas, int bound, cudaStream_t st) {
  const size_t nl = (a.rank + 63) / 64, nb = (nl + 1) / 2, most = 227 * 1024;
  const size_t rest = 2 * SLAB + (nl + 1) * NH * 128 + 2 * NH * 128 + (size_t)NH * (KEYS + 4) * 4 + NH * 4 + sizeof(Ctl);
  // the most pages of a share, up to three: two need room for both, more take what there is (less leaves room for the kernels before and after)
  const int b = bound > SINGLE && bound < 2 * SINGLE ? 2 * SINGLE : bound, per = (b + shares_of(b, ctas) - 1) / shares_of(b, ctas);
  size_t stages = (most - rest) / STAGE;
  if (stages > MAX_STAGES) stages = MAX_STAGES;
  if (stages > 4 * nb) stages = 4 * nb;
  if (per <= 2 && stages > per * nb) stages = per * nb;
  if (stages < (per < 2 ? 1 : 2) * nb) return (int)cudaErrorInvalidValue;
  a.stages = (int)stages;
  const size_t smem = stages * STAGE + rest;
  static size_t granted = 0;
  if (smem > granted) {
    const cudaError_t e = cudaFuncSetAttribute(latent_pages_kernel<NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    granted = smem;
  }
  return (int)sfb_launch(latent_pages_kernel<NH>, dim3(ctas, (a.H + NH - 1) / NH), dim3(THREADS), smem, st, *q, *qr, *c, *r, a);
}

}  // namespace rld
}  // namespace sfb

using namespace sfb;
using namespace sfb::rld;

extern "C" {

// heads (16 or 32) a block takes: the box height of mq and mqr
int sfb_rows_latent_heads(int H) { return H <= 16 ? 16 : 32; }

// mq, mqr: latent and shared parts of the queries, rows = launch row x H + head; mc, mr: the same of the pool, rows = page x 64 + slot, boxes
// of 64 rows.  ctas: how many share the pages, of which there are `bound` at most; part and ml hold ctas + n places, parts n pairs.  n up to 256; rank: a multiple of 8 up to 512, rot a multiple of 8 up to 64.
int sfb_rows_latent_decode(const void* mq, const void* mqr, const void* mc, const void* mr, const int* table, const int* row_lane, const int* row_pos,
                           const int* rows, void* part, void* ml, void* parts, int max_pages, int n_pages, int n, int H, int rank, int rot, int window, int ctas, int bound, int q_row0,
                           float scale, void* status, cudaStream_t stream) {
  if (n < 1 || n > ROWS || H < 1 || rank < 8 || rank % 8 || rank > 512 || rot < 8 || rot % 8 || rot > 64 || window < 1 || ctas < 1 || bound < 1)
    return (int)cudaErrorInvalidValue;
  Args a{table, row_lane, row_pos, rows, (float*)part, (float*)ml, (int2*)parts, max_pages, n_pages, n, H, rank, rot, window, 0, q_row0, scale, (Status*)status};
  const CUtensorMap *q = (const CUtensorMap*)mq, *qr = (const CUtensorMap*)mqr, *c = (const CUtensorMap*)mc, *r = (const CUtensorMap*)mr;
  return sfb_rows_latent_heads(H) == 16 ? launch<16>(q, qr, c, r, a, ctas, bound, stream) : launch<32>(q, qr, c, r, a, ctas, bound, stream);
}

}  // extern "C"
