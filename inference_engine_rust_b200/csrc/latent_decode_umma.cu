// One-token steps of latent attention on the 5th-generation tensor cores: the attention over the cached rows, in the
// absorbed form (latent_decode_tc.cu has the absorption of the queries before it and the merge behind it).  A cached row
// [latent | rotated key part] is the key of every head and, in its latent part, the value of every head, so a page of 64
// rows comes into shared memory once and is an operand of both products:
//
//   S = Qa C^T      [heads x keys]   A = the absorbed queries, from tensor memory,       B = the page, K-major
//   L^T += C^T P^T  [rank x heads]   A = the same page, MN-major (its columns are rows),  B = the probabilities
//
//   What an instruction costs here is the shared memory it reads (about 64 bytes a cycle), so the queries, which every
//   page meets, live in TMEM: 128 lanes hold 128 / NH copies of the NH heads, every warp of the softmax finds all heads in
//   its own 32 lanes and takes 16 of the page's 64 keys.  Their way there is through the last stage of the page ring,
//   which is filled with pages once they have moved on.
//   grid (sequences, runs of pages, groups of NH heads); a CTA walks its run of the sequence's pages.
//   warp 4      TMA producer: the queries once, then pages into a ring of `stages`; the first pages, unless one is the
//               newest, are asked for before the wait on the kernel in front.
//   warp 5      MMA issuer: the scores of the next page as soon as it has landed, the weighted sum of this one as soon as
//               its probabilities are there, whichever comes first.
//   warps 0-3   softmax, a head per lane and 16 keys per warp: mask, the page's maximum per head through shared memory,
//               exponentials against a reference maximum that moves only when it has grown by more than 2^8 (L^T is
//               rescaled in TMEM then), probabilities as bf16 into (swizzled) shared memory.  A row of the page that does
//               not count (outside the window, beyond the newest position, a page that is not there) is cleared first: its
//               weight is zero, but zero times whatever the page held need not be.
//   Every wait is bounded; on expiry the kernel records IERT_ERR_WAIT_EXPIRED, waits (bounded) for its copies and MMAs,
//   frees its TMEM and returns.
#include "common.cuh"
#include "sm100.cuh"
#include "tma_host.cuh"

using namespace iert;
using namespace sm100;

namespace {

constexpr int BK = 64;                         // keys per page
constexpr int BOX = BK * 128;                  // 64 rows x 64 columns of bf16
constexpr int THREADS = 192, SOFT = 128;
constexpr uint32_t WAIT_LIMIT = 1u << 22;
constexpr uint32_t POLL_LIMIT = 1u << 25;      // polls that do not suspend the thread: about as long a wait
constexpr int MAX_STAGES = 4;

struct LatentUmmaParams {
  int Hpad, H, rank, nbox, qcols, mblocks, splits, stages;
  uint32_t tmem_cols;
  float scale_log2e;
  float* part_m;
  float* part_l;
  float* part_acc;
  int* err;
};

__device__ __forceinline__ bool wait_bar(uint64_t* bar, uint32_t parity, volatile int* abort_flag) {
  for (uint32_t i = 0; i < WAIT_LIMIT; ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 255u) == 255u && *abort_flag) return false;
  }
  return false;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// The MMAs and commits of a whole converged warp of which one lane acts (`leader` != 0): the operands stay warp-uniform,
// which is what lets one instruction follow another without moving them between register files first.
__device__ __forceinline__ uint32_t elect_leader() {
  uint32_t l;
  asm volatile("{\n\t.reg .pred p;\n\telect.sync _|p, 0xffffffff;\n\tselp.u32 %0, 1, 0, p;\n\t}" : "=r"(l));
  return l;
}
__device__ __forceinline__ void mma_ts(uint32_t leader, uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.b32 p, %4, 0;\n\tsetp.ne.b32 q, %5, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d), "r"(a), "l"(b), "r"(idesc), "r"(accumulate), "r"(leader) : "memory");
}
__device__ __forceinline__ void mma_ss(uint32_t leader, uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.b32 p, %4, 0;\n\tsetp.ne.b32 q, %5, 0;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(accumulate), "r"(leader) : "memory");
}
__device__ __forceinline__ void mma_commit(uint32_t leader, uint64_t* bar) {
  asm volatile(
      "{\n\t.reg .pred q;\n\tsetp.ne.b32 q, %1, 0;\n\t"
      "@q tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}"
      ::"r"(smem_addr(bar)), "r"(leader) : "memory");
}
__device__ __forceinline__ void soft_sync() { asm volatile("bar.sync 1, %0;" ::"n"(SOFT) : "memory"); }

template <int NH>
__global__ void __launch_bounds__(THREADS, 1)
latent_decode_umma_kernel(const __grid_constant__ CUtensorMap map_c, const __grid_constant__ CUtensorMap map_q, LatentUmmaParams p,
                          IertBatchView b, IertKvView kv) {
  extern __shared__ __align__(1024) uint8_t smem[];     // no static shared memory: the window starts 1024-byte aligned
  constexpr int QBOX = NH * 128, PBUF = NH * 128;
  uint8_t* c_s = smem;                                   // stages x nbox boxes of 64 rows
  uint8_t* q_s = c_s + (p.stages - 1) * p.nbox * BOX;    // nbox boxes of NH rows, in the last stage until they are in TMEM
  uint8_t* p_s = c_s + p.stages * p.nbox * BOX;          // 2 buffers: NH rows (heads) of 64 probabilities
  uint8_t* tail = p_s + (2 * PBUF > BOX ? 2 * PBUF : BOX);      // (an MMA may read one box beyond the last page)
  float* wmax = reinterpret_cast<float*>(tail);          // [2][4][32]
  float* wsum = wmax + 8 * 32;                           // [4][32]
  uint64_t* bars = reinterpret_cast<uint64_t*>(wsum + 4 * 32);
  uint64_t* q_full = bars;
  uint64_t* c_full = bars + 1;                           // MAX_STAGES
  uint64_t* c_empty = c_full + MAX_STAGES;               // MAX_STAGES
  uint64_t* q_moved = c_empty + MAX_STAGES;              // the queries are in TMEM
  uint64_t* s_full = q_moved + 1;
  uint64_t* s_empty = s_full + 1;                        // every thread has read its scores
  uint64_t* p_ready = s_empty + 1;                       // 2
  uint64_t* pv_done = p_ready + 2;                       // 2
  uint64_t* drained = pv_done + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(drained + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  volatile int* armed = abort_flag + 1;                  // pages the producer has asked for; -1: not even the queries
  volatile int* stop = armed + 1;                        // [2]: the flag as warp 0 saw it in front of a barrier, so that all agree

  const int s = blockIdx.x, split = blockIdx.y, rows0 = blockIdx.z * NH;
  const int tid = threadIdx.x, lane = tid & 31;
  const int warp = __shfl_sync(0xffffffffu, tid >> 5, 0);          // known to be the same for the whole warp
  const int slot = b.slot_ids[s];
  if (slot < 0) { pdl_wait(); return; }
  const int pos = b.pos0[s];                             // one token per sequence: its own row is in the cache
  const IertPageWalk walk = iert_page_walk(kv, pos, BK);
  const int t_lo = (int)((long long)split * walk.n / p.splits), t_hi = (int)((long long)(split + 1) * walk.n / p.splits);
  const int n_tiles = t_hi - t_lo;
  const size_t part_row0 = ((size_t)s * p.splits + split) * p.Hpad + rows0;
  if (n_tiles <= 0) {                                    // an empty run: a partial that the merge skips
    pdl_wait();
    if (tid < NH) { p.part_m[part_row0 + tid] = -INFINITY; p.part_l[part_row0 + tid] = 0.f; }
    return;
  }
  if (smem_addr(smem) & 1023u) {                         // never expected; refuse rather than compute garbage
    if (tid == 0) atomicOr(p.err, IERT_ERR_WAIT_EXPIRED);
    return;
  }
  if (tid == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < MAX_STAGES; ++i) { mbar_init(&c_full[i], 1); mbar_init(&c_empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&p_ready[i], SOFT); mbar_init(&pv_done[i], 1); }
    mbar_init(q_moved, SOFT);
    mbar_init(s_full, 1);
    mbar_init(s_empty, SOFT);
    mbar_init(drained, 1);
    *abort_flag = 0;
    *armed = -1;
    mbar_fence_init();
    tma_prefetch_desc(&map_c);
    tma_prefetch_desc(&map_q);
  }
  if (warp == 5) tmem_alloc(tmem_slot, p.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();                               // (a later kernel must not take the TMEM this CTA still waits for)
  const uint32_t tmem = *tmem_slot;
  const uint32_t s_col = p.qcols, l_col = s_col + BK;    // the queries, S, and the blocks of L^T
  bool ok = true;

  if (warp == 4) {
    // ---------------- TMA producer ----------------
    bool waited = false;
    int asked = 0;
    for (int base = 0; base < n_tiles; base += 32) {
      int page = -1;                                     // page numbers of up to 32 pages at a time, one per lane
      if (base + lane < n_tiles)
        page = kv.page_table[(size_t)slot * kv.table_width + iert_table_entry(kv, iert_walk_page(walk, t_lo + base + lane))];
      for (int k = 0; k < 32 && base + k < n_tiles; ++k) {
        const int it = base + k, st = it % p.stages;
        const int pgid = __shfl_sync(0xffffffffu, page, k);
        if (lane != 0 || !ok) continue;
        // the newest row, and the queries, are the work of the kernels in front
        if (!waited && (t_lo + it == walk.n - 1 || it >= p.stages - 1)) {
          pdl_wait();
          waited = true;
          mbar_expect_tx(q_full, p.nbox * QBOX);
          for (int x = 0; x < p.nbox; ++x) tma_load_2d(q_s + x * QBOX, &map_q, q_full, 64 * x, s * p.Hpad + rows0);
        }
        if (it == p.stages - 1 && !wait_bar(q_moved, 0, abort_flag)) { ok = false; continue; }
        if (it >= p.stages && !wait_bar(&c_empty[st], ((it / p.stages) - 1) & 1, abort_flag)) { ok = false; continue; }
        const bool page_ok = pgid >= 0 && pgid < kv.n_pages;
        if (!page_ok) atomicOr(p.err, IERT_ERR_PAGE_RANGE);      // (the softmax warps see the same and count no row of it)
        mbar_expect_tx(&c_full[st], p.nbox * BOX);
        for (int x = 0; x < p.nbox; ++x)
          tma_load_2d(c_s + (st * p.nbox + x) * BOX, &map_c, &c_full[st], 64 * x, (page_ok ? pgid : 0) * BK);
        asked = it + 1;
      }
    }
    if (lane == 0) {
      if (!waited) {
        pdl_wait();
        waited = true;
        mbar_expect_tx(q_full, p.nbox * QBOX);
        for (int x = 0; x < p.nbox; ++x) tma_load_2d(q_s + x * QBOX, &map_q, q_full, 64 * x, s * p.Hpad + rows0);
      }
      *armed = asked;
    }
  } else if (warp == 5) {
    // ---------------- MMA issuer (the whole warp, one lane of it acting) ----------------
    constexpr uint32_t IDESC_S = instr_desc_bf16(128, BK);
    constexpr uint32_t IDESC_L = instr_desc_bf16_a_mn(128, NH);
    const uint32_t leader = elect_leader();
    const uint32_t c_base = smem_addr(c_s), stage_bytes = p.nbox * BOX;
    auto scores = [&](int st) {                          // S = Qa C^T (the page in stage st has landed, the scores before are read)
      tc_fence_after();
      uint64_t cd = smem_desc_k128(c_base + st * stage_bytes);
      uint32_t qa = tmem;
      mma_ts(leader, tmem + s_col, qa, cd, IDESC_S, 0u);                           // columns beyond `width` are zeros
#pragma unroll
      for (int ks = 1; ks < 4; ++ks) mma_ts(leader, tmem + s_col, qa + ks * 8, cd + ks * 2, IDESC_S, 1u);
      for (int x = 1; x < p.nbox; ++x) {
        cd += BOX >> 4;
        qa += 32;
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) mma_ts(leader, tmem + s_col, qa + ks * 8, cd + ks * 2, IDESC_S, 1u);
      }
      mma_commit(leader, s_full);
    };
    // a wait of the whole warp: what one lane sees, all act on
    auto warp_wait = [&](uint64_t* bar, uint32_t parity) { return __all_sync(0xffffffffu, wait_bar(bar, parity, abort_flag)) != 0; };
    ok = warp_wait(q_moved, 0) && warp_wait(&c_full[0], 0);
    if (ok) scores(0);
    int st = 0, sn = 1 % p.stages;                       // the stages of page `it` and of the next one, and the next one's phase
    uint32_t ph = p.stages == 1 ? 1u : 0u;
    for (int it = 0; ok && it < n_tiles; ++it) {
      bool next_done = it + 1 >= n_tiles, ready = false;
      for (uint32_t i = 0; i < POLL_LIMIT && !ready; ++i) {
        if (!next_done && __all_sync(0xffffffffu, mbar_test(s_empty, it & 1) && mbar_test(&c_full[sn], ph))) {
          scores(sn);
          next_done = true;
        }
        ready = __all_sync(0xffffffffu, mbar_test(&p_ready[it & 1], (it >> 1) & 1));
        if ((i & 255u) == 255u && __any_sync(0xffffffffu, *abort_flag != 0)) break;
      }
      if (!ready) { ok = false; break; }
      tc_fence_after();
      uint64_t cd = smem_desc_mn128(c_base + st * stage_bytes, BOX);
      const uint64_t pd = smem_desc_k128(smem_addr(p_s) + (it & 1) * PBUF);
      const uint32_t again = it > 0 ? 1u : 0u;
      uint32_t d = tmem + l_col;
      for (int m = 0; m < p.mblocks; ++m) {
        mma_ss(leader, d, cd, pd, IDESC_L, again);
#pragma unroll
        for (int kk = 1; kk < BK / 16; ++kk) mma_ss(leader, d, cd + kk * (16 * 128 >> 4), pd + kk * 2, IDESC_L, 1u);
        cd += 2 * BOX >> 4;
        d += NH;
      }
      mma_commit(leader, &pv_done[it & 1]);
      mma_commit(leader, &c_empty[st]);
      if (!next_done) {
        if (!warp_wait(s_empty, it & 1) || !warp_wait(&c_full[sn], ph)) { ok = false; break; }
        scores(sn);
      }
      st = sn;
      if (++sn == p.stages) { sn = 0; ph ^= 1u; }
    }
    mma_commit(leader, drained);
  } else {
    // ---------------- softmax: lane = head (lane % NH), warp = 16 keys of the page ----------------
    pdl_wait();
    const uint32_t lane_bits = (uint32_t)(warp * 32) << 16;
    const int hl = lane % NH;
    if (!wait_bar(q_full, 0, abort_flag)) { ok = false; *abort_flag = 1; }
    for (int x = 0; x < p.nbox; ++x) {                   // 64 numbers of the head at a time: eight 16-byte chunks of its row
      uint32_t w[32];
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        const uint4 v = *reinterpret_cast<const uint4*>(q_s + x * QBOX + hl * 128 + ((c ^ (hl & 7)) << 4));
        w[4 * c] = v.x; w[4 * c + 1] = v.y; w[4 * c + 2] = v.z; w[4 * c + 3] = v.w;
      }
      tmem_st16_issue(tmem + lane_bits + x * 32, w);
      tmem_st16_issue(tmem + lane_bits + x * 32 + 16, w + 16);
    }
    tmem_st_wait();
    tc_fence_before();
    mbar_arrive(q_moved);
    float m_ref = -INFINITY, l = 0.f;                    // the head's reference maximum (base 2), alike in all warps; this thread's sum
    for (int it = 0; it < n_tiles; ++it) {
      const int pg = iert_walk_page(walk, t_lo + it), j0 = pg * BK;
      const int page = kv.page_table[(size_t)slot * kv.table_width + iert_table_entry(kv, pg)];
      const bool page_ok = page >= 0 && page < kv.n_pages;
      const bool partial = !page_ok || j0 + BK - 1 > pos || j0 < walk.j_min;      // some row of the page may not count
      auto counts = [&](int r) { return page_ok && j0 + r <= pos && (j0 + r >= walk.j_min || j0 + r < kv.keep); };
      if (!wait_bar(s_full, it & 1, abort_flag)) { ok = false; *abort_flag = 1; }
      tc_fence_after();
      float sc[16];
      tmem_ld16(tmem + lane_bits + s_col + 16 * warp, sc);
      tc_fence_before();
      mbar_arrive(s_empty);
#pragma unroll
      for (int c = 0; c < 16; ++c) sc[c] *= p.scale_log2e;
      if (partial) {
#pragma unroll
        for (int c = 0; c < 16; ++c) if (!counts(16 * warp + c)) sc[c] = -INFINITY;
        const int row = tid >> 1;
        if (!counts(row)) {                              // two threads a row, every other box each
          uint8_t* line = c_s + (it % p.stages) * p.nbox * BOX + row * 128;
          for (int x = tid & 1; x < p.nbox; x += 2)
#pragma unroll
            for (int c = 0; c < 8; ++c) *reinterpret_cast<uint4*>(line + x * BOX + c * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
      float top = sc[0];
#pragma unroll
      for (int c = 1; c < 16; ++c) top = fmaxf(top, sc[c]);
      float* wm = wmax + (it & 1) * 4 * 32;
      wm[warp * 32 + lane] = top;
      if (tid == 0) stop[it & 1] = *abort_flag;
      soft_sync();
      if (stop[it & 1]) { ok = false; break; }           // all four warps leave at the same barrier
      const float tm = fmaxf(fmaxf(wm[lane], wm[32 + lane]), fmaxf(wm[64 + lane], wm[96 + lane]));
      const bool grow = tm > m_ref + 8.0f || (m_ref == -INFINITY && tm != -INFINITY);
      if (__any_sync(0xffffffffu, grow)) {               // the same in all four warps
        const float m_new = grow ? tm : m_ref;
        const float alpha = !grow ? 1.f : (m_ref == -INFINITY ? 0.f : ex2(m_ref - m_new));
        m_ref = m_new;
        l *= alpha;
        if (it > 0) {
          if (!wait_bar(&pv_done[(it - 1) & 1], ((it - 1) >> 1) & 1, abort_flag)) { ok = false; *abort_flag = 1; }
          __syncwarp();
          tc_fence_after();
          for (int m = 0; m < p.mblocks; ++m)
#pragma unroll
            for (int c = 0; c < NH; c += 16) {
              float o[16];
              tmem_ld16(tmem + lane_bits + l_col + m * NH + c, o);
#pragma unroll
              for (int e = 0; e < 16; ++e) o[e] *= __shfl_sync(0xffffffffu, alpha, c + e);
              tmem_st16(tmem + lane_bits + l_col + m * NH + c, o);
            }
        }
      }
      // probabilities: head h is row h of the operand, the warp's keys are two 16-byte chunks of it; the buffer was last
      // read by the sum of page it - 2, which had finished before the scores of page `it` were committed
      const float neg = m_ref == -INFINITY ? 0.f : -m_ref;
      uint4 w2[2];
      __nv_bfloat162* wp = reinterpret_cast<__nv_bfloat162*>(w2);
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        const float pa = ex2(sc[2 * c] + neg), pb = ex2(sc[2 * c + 1] + neg);
        l += pa + pb;
        wp[c] = __floats2bfloat162_rn(pa, pb);
      }
      if (lane < NH) {
        uint8_t* pb = p_s + (it & 1) * PBUF + hl * 128;
        *reinterpret_cast<uint4*>(pb + (((2 * warp) ^ (hl & 7)) << 4)) = w2[0];
        *reinterpret_cast<uint4*>(pb + (((2 * warp + 1) ^ (hl & 7)) << 4)) = w2[1];
      }
      fence_proxy_async_smem();                          // the probabilities, and rows that were cleared, reach the tensor core
      tc_fence_before();
      mbar_arrive(&p_ready[it & 1]);
    }
    if (ok && !wait_bar(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1, abort_flag)) ok = false;
    if (!ok) *abort_flag = 1;
    wsum[warp * 32 + lane] = l;
    soft_sync();                                         // every warp has left the loop and said how
    if (tid == 0) stop[0] = *abort_flag;
    soft_sync();
    const bool good = stop[0] == 0;                      // an aborted run leaves an empty partial
    if (warp == 0 && lane < NH) {
      p.part_m[part_row0 + lane] = good && m_ref != -INFINITY ? m_ref * 0.6931471805599453f : -INFINITY;
      p.part_l[part_row0 + lane] = good ? (wsum[lane] + wsum[32 + lane]) + (wsum[64 + lane] + wsum[96 + lane]) : 0.f;
    }
    if (good) {
      tc_fence_after();
      for (int m = 0; m < p.mblocks; ++m) {
        const int r = m * 128 + tid;
        float* dst = p.part_acc + part_row0 * p.rank + r;
#pragma unroll
        for (int c = 0; c < NH; c += 16) {
          float o[16];
          tmem_ld16(tmem + lane_bits + l_col + m * NH + c, o);
#pragma unroll
          for (int e = 0; e < 16; ++e)
            if (r < p.rank && rows0 + c + e < p.H) dst[(size_t)(c + e) * p.rank] = o[e];
        }
      }
    }
  }
  if (!ok && lane == 0) {
    atomicOr(p.err, IERT_ERR_WAIT_EXPIRED);
    *abort_flag = 1;
  }
  tc_fence_before();
  __syncthreads();
  if (*abort_flag && tid == 0) {                         // copies and MMAs still on their way end before the memory is let go
    mbar_wait(drained, 0, WAIT_LIMIT);
    const int n = *armed;
    if (n >= 0) mbar_wait(q_full, 0, WAIT_LIMIT);
    for (int st = 0; st < p.stages; ++st)
      if (n > st) {
        const int last = ((n - 1 - st) / p.stages) * p.stages + st;
        mbar_wait(&c_full[st], (last / p.stages) & 1, WAIT_LIMIT);
      }
  }
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem, p.tmem_cols);
  }
}

size_t fixed_smem(int nh) {
  const size_t pbuf = (size_t)nh * 128;
  return (2 * pbuf > (size_t)BOX ? 2 * pbuf : (size_t)BOX) + 12 * 32 * sizeof(float) + (9 + 2 * MAX_STAGES) * sizeof(uint64_t) + 32;
}
int stages_for(int nh, int width) {
  const int nbox = (width + 63) / 64;
  const int n = (int)((227 * 1024 - fixed_smem(nh)) / ((size_t)nbox * BOX));
  return n > MAX_STAGES ? MAX_STAGES : n;
}

}  // namespace

// Heads per CTA (16 or 32) that the kernel runs at H heads, or 0 where it does not take the sizes.
int latent_umma_heads(int H, int rank, int R) {
  const int width = rank + R, nh = H > 16 ? 32 : 16;
  if (width % 8 || rank < 16 || rank > 512 || width > 640 || stages_for(nh, width) < 2) return 0;
  return nh;
}

// qa bf16 [T, Hpad, width]; part_m, part_l fp32 [T, splits, Hpad]; part_acc fp32 [T, splits, Hpad, rank] (rows of heads below
// H are written).  One token per sequence; a cache of bf16 rows `width` = rank + R wide, pages of 64.
int launch_latent_decode_umma(const void* qa, const IertBatchView* batch, const IertKvView* kv, int H, int Hpad, int R, float scale,
                              int splits, float* part_m, float* part_l, float* part_acc, int* err, cudaStream_t stream) {
  const int T = batch->n_tokens, width = kv->head_dim, rank = width - R;
  const int nh = latent_umma_heads(H, rank, R);
  if (!nh || Hpad % nh || ((uintptr_t)qa & 15) || ((uintptr_t)kv->k & 15)) return IERT_BAD_ARGUMENT;
  CUtensorMap map_c, map_q;
  if (!tma_host::tensor_map_2d(kv->k, (long long)kv->n_pages * BK, width, width, BK, &map_c) ||
      !tma_host::tensor_map_2d(qa, (long long)T * Hpad, width, width, nh, &map_q))
    return IERT_BAD_ARGUMENT;
  LatentUmmaParams p;
  p.Hpad = Hpad; p.H = H; p.rank = rank;
  p.nbox = (width + 63) / 64; p.qcols = p.nbox * 32; p.mblocks = (rank + 127) / 128;
  p.splits = splits; p.stages = stages_for(nh, width);
  const int cols = p.qcols + BK + p.mblocks * nh;       // at most 320 + 64 + 128
  p.tmem_cols = 32;
  while ((int)p.tmem_cols < cols) p.tmem_cols *= 2;
  p.scale_log2e = scale * 1.4426950408889634f;
  p.part_m = part_m; p.part_l = part_l; p.part_acc = part_acc; p.err = err;
  const size_t smem = fixed_smem(nh) + (size_t)p.stages * p.nbox * BOX;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(latent_decode_umma_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(latent_decode_umma_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) {
      cudaGetLastError();
      return IERT_CUDA_ERROR;
    }
    configured = true;
  }
  const dim3 grid(T, splits, Hpad / nh);
  if (nh == 16) launch_dep(latent_decode_umma_kernel<16>, grid, dim3(THREADS), smem, stream, map_c, map_q, p, *batch, *kv);
  else launch_dep(latent_decode_umma_kernel<32>, grid, dim3(THREADS), smem, stream, map_c, map_q, p, *batch, *kv);
  return cudaGetLastError() == cudaSuccess ? IERT_OK : IERT_CUDA_ERROR;
}
