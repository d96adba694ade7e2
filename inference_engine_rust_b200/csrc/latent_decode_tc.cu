// One-token steps of latent attention on the tensor cores (mma.sync m16n8k16, bf16 in, fp32 out),
// in the absorbed form: every head's query is first taken into the latent's coordinates,
// qa = W_uk[h]^T q (rank numbers), so that all heads of a sequence meet the same cached rows c_j:
//
//   S = Qa C^T   ([heads x rank] x [rank x keys]),   P = softmax with a sink,   L = P C  ([heads x keys] x [keys x rank])
//
// which is multi-query attention whose keys and values are the same rows.  W_uv is applied to L at the
// end, once per head.  Three kernels (the one in the middle is the one of latent_decode_umma.cu where that takes the sizes):
//   latent_absorb_q       qa [T, Hpad, rank] bf16 from q and W_uk (rows of padding heads are zero); q either in bf16 with
//                         its rotated part turned already, or the fp32 projection itself, turned on the way
//   latent_decode_tc      a CTA takes (sequence, a run of 64-key tiles, up to 32 heads): the tile of C comes
//                         into shared memory once (cp.async) and serves both products; warp w forms the
//                         scores of keys 16w..16w+15 of the tile for all the CTA's heads, the warps agree on
//                         row maxima and sums through shared memory, and warp w then owns a quarter of the
//                         rank columns of L (its accumulators).  Partial (max, sum, L) per run go to scratch.
//   latent_decode_merge   merges the runs in order, adds the sink's term exp(sink - M) to the denominator,
//                         and multiplies by W_uv: out [T, H*V].
// A window, a chunk or kept first positions of the cache view choose which pages are walked and which rows count.
// Sizes: rank a multiple of 32 (of 8 for the kernel of latent_decode_umma.cu) up to 512, pages of 64 positions, a bf16 cache.  Anything else is refused
// (IERT_BAD_ARGUMENT) and the caller runs the plain kernel.
#include "common.cuh"

#include <cstdlib>

using namespace iert;

namespace {

constexpr int BK = 64;            // keys per tile = positions per page
constexpr int THREADS = 128;
constexpr int MAX_NTW = 16;       // n-tiles of 8 rank columns per warp: rank <= 4 * 16 * 8 = 512
constexpr int PLD = BK + 8;       // row stride of the probabilities in shared memory (elements)

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ uint32_t lds32(const __nv_bfloat16* p) { return *reinterpret_cast<const uint32_t*>(p); }

// qa[t, h, :] = sum_d q[t, h, d] W_uk[h*D + d, :].  A block of 256 threads takes one head of TT tokens, so that the
// head's weights are read once for all of them: 64 threads across the rank (eight columns each, 16-byte loads of the
// weights) times four groups along d, added through shared memory in a fixed order.
constexpr int ABSORB_THREADS = 256;

// Asks for `bytes` bytes of weights to be brought into the L2 while the block still waits for the kernel in front.
__device__ __forceinline__ void fetch_ahead(const void* p, size_t bytes) {
  for (size_t i = (size_t)threadIdx.x * 128; i < bytes; i += (size_t)blockDim.x * 128)
    asm volatile("prefetch.global.L2 [%0];" ::"l"((const char*)p + i));
}

// TQ float: q is the projection as it stands, and the R last numbers of a head are turned here (inv_freq, rot_mul, pairing).
template <typename TQ, int TT>
__global__ void __launch_bounds__(ABSORB_THREADS)
latent_absorb_q_kernel(const TQ* __restrict__ q, long long ldq, const __nv_bfloat16* __restrict__ w_uk,
                       __nv_bfloat16* __restrict__ qa, int H, int Hpad, int D, int R, int rank, const float* __restrict__ inv_freq,
                       float rot_mul, int pairing, IertBatchView b) {
  extern __shared__ float sm_q[];
  float* q_s = sm_q;                    // [TT][D]
  float* part = sm_q + TT * D;          // [4][TT][rank]
  pdl_launch_dependents();
  const int t0 = blockIdx.x * TT, h = blockIdx.y, n_t = min(TT, b.n_tokens - t0);
  if (blockIdx.x == 0 && h < H) fetch_ahead(w_uk + (size_t)h * D * rank, (size_t)D * rank * 2);
  pdl_wait();
  if (h >= H) {                         // heads that only fill the MMA tile
    for (int i = threadIdx.x; i < n_t * (rank + R); i += blockDim.x)
      qa[((size_t)(t0 + i / (rank + R)) * Hpad + h) * (rank + R) + i % (rank + R)] = __float2bfloat16_rn(0.f);
    return;
  }
  for (int i = threadIdx.x; i < TT * D; i += blockDim.x) {
    const int t = i / D, d = i - t * D;
    q_s[i] = t < n_t ? to_f32(q[(size_t)(t0 + t) * ldq + (size_t)h * (D + R) + d]) : 0.f;
  }
  if (sizeof(TQ) == 4) {                // one token per sequence: token t is sequence t's
    const int half = R / 2;
    for (int i = threadIdx.x; i < n_t * half; i += blockDim.x) {
      const int t = t0 + i / half, k = i % half, pos = b.pos0[t];
      const TQ* v = q + (size_t)t * ldq + (size_t)h * (D + R) + D;
      __nv_bfloat16* dst = qa + ((size_t)t * Hpad + h) * (rank + R) + rank;
      const int i0 = pairing == IERT_PAIR_INTERLEAVED ? 2 * k : k, i1 = pairing == IERT_PAIR_INTERLEAVED ? 2 * k + 1 : k + half;
      const float x = to_f32(v[i0]), y = to_f32(v[i1]);
      float sn, co;
      sincosf((float)pos * inv_freq[k], &sn, &co);
      sn *= rot_mul;
      co *= rot_mul;
      dst[i0] = __float2bfloat16_rn(x * co - y * sn);
      dst[i1] = __float2bfloat16_rn(y * co + x * sn);
    }
  } else {
    for (int i = threadIdx.x; i < n_t * R; i += blockDim.x) {                        // turned already
      const int t = t0 + i / R, k = i % R;
      qa[((size_t)t * Hpad + h) * (rank + R) + rank + k] = __float2bfloat16_rn(to_f32(q[(size_t)t * ldq + (size_t)h * (D + R) + D + k]));
    }
  }
  __syncthreads();
  const int grp = threadIdx.x >> 6, lane64 = threadIdx.x & 63;
  const int d_lo = grp * ((D + 3) / 4), d_hi = min(D, d_lo + (D + 3) / 4);
  for (int r0 = lane64 * 8; r0 < rank; r0 += 64 * 8) {
    float a[TT][8];
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
      for (int e = 0; e < 8; ++e) a[t][e] = 0.f;
    const __nv_bfloat16* w = w_uk + (size_t)h * D * rank + r0;
#pragma unroll 8
    for (int d = d_lo; d < d_hi; ++d) {
      const uint4 v = *reinterpret_cast<const uint4*>(w + (size_t)d * rank);
      const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&v);
      float f[8];
#pragma unroll
      for (int e = 0; e < 4; ++e) { const float2 two = __bfloat1622float2(p[e]); f[2 * e] = two.x; f[2 * e + 1] = two.y; }
#pragma unroll
      for (int t = 0; t < TT; ++t) {
        const float qd = q_s[t * D + d];
#pragma unroll
        for (int e = 0; e < 8; ++e) a[t][e] = fmaf(qd, f[e], a[t][e]);
      }
    }
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
      for (int e = 0; e < 8; ++e) part[(grp * TT + t) * rank + r0 + e] = a[t][e];
  }
  __syncthreads();
  const int all = TT * rank;
  for (int i = threadIdx.x; i < n_t * rank; i += blockDim.x)
    qa[((size_t)(t0 + i / rank) * Hpad + h) * (rank + R) + i % rank] =
        __float2bfloat16_rn((part[i] + part[all + i]) + (part[2 * all + i] + part[3 * all + i]));
}

template <int MT>
__global__ void __launch_bounds__(THREADS)
latent_decode_tc_kernel(const __nv_bfloat16* __restrict__ qa, IertBatchView b, IertKvView kv, int Hpad, int R, float scale,
                        int splits, float* __restrict__ part_m, float* __restrict__ part_l,
                        float* __restrict__ part_acc, int* __restrict__ err) {
  extern __shared__ __align__(16) uint8_t smem[];
  // a cached row is `width` numbers: the latent (`rank`, which also serves as the value) and R rotated key numbers
  const int width = kv.head_dim, rank = width - R, ldc = width + 8;
  __nv_bfloat16* qa_s = reinterpret_cast<__nv_bfloat16*>(smem);     // [MT*16][ldc]
  __nv_bfloat16* c_s = qa_s + MT * 16 * ldc;                         // [BK][ldc]
  __nv_bfloat16* p_s = c_s + BK * ldc;                               // [MT*16][PLD]
  float* wmax = reinterpret_cast<float*>(p_s + MT * 16 * PLD);       // [4][MT*16]
  float* wsum = wmax + 4 * MT * 16;                                  // [4][MT*16]
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.x, split = blockIdx.y, rows0 = blockIdx.z * MT * 16;
  const int slot = b.slot_ids[s];
  if (slot < 0) return;
  const int pos = b.pos0[s];                         // one token per sequence: its own row is in the cache
  const IertPageWalk walk = iert_page_walk(kv, pos, BK);
  const int n_tiles = walk.n;
  const int t_lo = (int)((long long)split * n_tiles / splits), t_hi = (int)((long long)(split + 1) * n_tiles / splits);
  const size_t part_row0 = ((size_t)s * splits + split) * Hpad + rows0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  if (t_lo >= t_hi) {                                // an empty run: a partial that the merge skips
    if (tid < MT * 16) { part_m[part_row0 + tid] = -INFINITY; part_l[part_row0 + tid] = 0.f; }
    return;
  }
  const int chunks = width / 8;                      // 16-byte pieces per row
  for (int i = tid; i < MT * 16 * chunks; i += THREADS) {
    const int r = i / chunks, c = i - r * chunks;
    *reinterpret_cast<uint4*>(qa_s + r * ldc + c * 8) =
        *reinterpret_cast<const uint4*>(qa + ((size_t)s * Hpad + rows0 + r) * width + c * 8);
  }
  float m_run[MT][2], l_run[MT][2], acc[MT][MAX_NTW][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
    m_run[mt][0] = m_run[mt][1] = -INFINITY;
    l_run[mt][0] = l_run[mt][1] = 0.f;
#pragma unroll
    for (int nt = 0; nt < MAX_NTW; ++nt) acc[mt][nt][0] = acc[mt][nt][1] = acc[mt][nt][2] = acc[mt][nt][3] = 0.f;
  }
  const int ntw = rank / 32;                         // n-tiles of L that this warp owns
  const int col0 = warp * (rank / 4);

  for (int tile = t_lo; tile < t_hi; ++tile) {
    __syncthreads();                                 // the tile before is no longer read (and qa_s is written)
    const int pg = iert_walk_page(walk, tile);
    const int page = kv.page_table[(size_t)slot * kv.table_width + iert_table_entry(kv, pg)];
    const bool page_ok = page >= 0 && page < kv.n_pages;
    if (!page_ok && tid == 0) atomicOr(err, IERT_ERR_PAGE_RANGE);
    const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(kv.k) + (size_t)(page_ok ? page : 0) * BK * width;
    const int valid = page_ok ? min(BK, pos + 1 - pg * BK) : 0;      // rows beyond hold other sequences' leftovers
    const int first = walk.j_min - pg * BK, kept = kv.keep - pg * BK;   // rows in front of the window count if they are kept
    for (int i = tid; i < BK * chunks; i += THREADS) {
      const int r = i / chunks, c = i - r * chunks;
      __nv_bfloat16* dst = c_s + r * ldc + c * 8;
      if (r < valid && (r >= first || r < kept))
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src + (size_t)r * width + c * 8));
      else
        *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
    }
    asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
    __syncthreads();

    // ---- scores of this warp's 16 keys for all heads of the CTA
    float sc[MT][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) sc[mt][nt][0] = sc[mt][nt][1] = sc[mt][nt][2] = sc[mt][nt][3] = 0.f;
    for (int k0 = 0; k0 < width; k0 += 16) {
      uint32_t bf[2][2];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const __nv_bfloat16* row = c_s + (warp * 16 + nt * 8 + g) * ldc + k0 + 2 * t4;
        bf[nt][0] = lds32(row);
        bf[nt][1] = lds32(row + 8);
      }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        const __nv_bfloat16* row = qa_s + (mt * 16 + g) * ldc + k0 + 2 * t4;
        const uint32_t a[4] = {lds32(row), lds32(row + 8 * ldc), lds32(row + 8), lds32(row + 8 * ldc + 8)};
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) mma_bf16(sc[mt][nt], a, bf[nt][0], bf[nt][1]);
      }
    }
    // ---- scale, mask, row maxima over the whole tile
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float mx = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int j = warp * 16 + nt * 8 + 2 * t4 + e;
            const float v = (j < valid && (j >= first || j < kept)) ? sc[mt][nt][half * 2 + e] * scale : -INFINITY;
            sc[mt][nt][half * 2 + e] = v;
            mx = fmaxf(mx, v);
          }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        if (t4 == 0) wmax[warp * MT * 16 + mt * 16 + half * 8 + g] = mx;
      }
    __syncthreads();
    float alpha[MT][2];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = mt * 16 + half * 8 + g;
        float m_new = m_run[mt][half];
#pragma unroll
        for (int w = 0; w < 4; ++w) m_new = fmaxf(m_new, wmax[w * MT * 16 + row]);
        alpha[mt][half] = m_run[mt][half] == -INFINITY ? 0.f : expf(m_run[mt][half] - m_new);
        m_run[mt][half] = m_new;                     // finite: every page of the walk holds at least one visible key
        float sum = 0.f;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const float p0 = sc[mt][nt][half * 2] == -INFINITY ? 0.f : expf(sc[mt][nt][half * 2] - m_new);
          const float p1 = sc[mt][nt][half * 2 + 1] == -INFINITY ? 0.f : expf(sc[mt][nt][half * 2 + 1] - m_new);
          sum += p0 + p1;
          *reinterpret_cast<__nv_bfloat162*>(p_s + row * PLD + warp * 16 + nt * 8 + 2 * t4) = __floats2bfloat162_rn(p0, p1);
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if (t4 == 0) wsum[warp * MT * 16 + row] = sum;
      }
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = mt * 16 + half * 8 + g;
        l_run[mt][half] = l_run[mt][half] * alpha[mt][half] +
                          ((wsum[row] + wsum[MT * 16 + row]) + (wsum[2 * MT * 16 + row] + wsum[3 * MT * 16 + row]));
      }
    // ---- L += P C for this warp's rank columns
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < MAX_NTW; ++nt)
        if (nt < ntw) {
          acc[mt][nt][0] *= alpha[mt][0]; acc[mt][nt][1] *= alpha[mt][0];
          acc[mt][nt][2] *= alpha[mt][1]; acc[mt][nt][3] *= alpha[mt][1];
        }
#pragma unroll
    for (int ks = 0; ks < BK / 16; ++ks) {
      uint32_t a[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        const __nv_bfloat16* row = p_s + (mt * 16 + g) * PLD + ks * 16 + 2 * t4;
        a[mt][0] = lds32(row); a[mt][1] = lds32(row + 8 * PLD); a[mt][2] = lds32(row + 8); a[mt][3] = lds32(row + 8 * PLD + 8);
      }
      const __nv_bfloat16* krow = c_s + (ks * 16 + (lane & 15)) * ldc + col0;
#pragma unroll
      for (int nt = 0; nt < MAX_NTW; ++nt)
        if (nt < ntw) {
          uint32_t b0, b1;
          asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(b0), "=r"(b1) : "r"(smem_u32(krow + nt * 8)));
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) mma_bf16(acc[mt][nt], a[mt], b0, b1);
        }
    }
  }
  // ---- this run's partial result
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const size_t row = part_row0 + mt * 16 + half * 8 + g;
      if (warp == 0 && t4 == 0) { part_m[row] = m_run[mt][half]; part_l[row] = l_run[mt][half]; }
#pragma unroll
      for (int nt = 0; nt < MAX_NTW; ++nt)
        if (nt < ntw)
          *reinterpret_cast<float2*>(part_acc + row * rank + col0 + nt * 8 + 2 * t4) =
              make_float2(acc[mt][nt][half * 2], acc[mt][nt][half * 2 + 1]);
    }
}

constexpr int MERGE_THREADS = 256;

// A block merges the runs of one head of TT sequences and multiplies each by the head's W_uv, whose rows are read once for
// all of them.
template <typename T, int TT>
__global__ void __launch_bounds__(MERGE_THREADS)
latent_decode_merge_kernel(const float* __restrict__ part_m, const float* __restrict__ part_l,
                           const float* __restrict__ part_acc, int splits, int Hpad, int rank,
                           const float* __restrict__ sink, const float* __restrict__ gate, const T* __restrict__ w_uv,
                           T* __restrict__ out, IertBatchView b, int H, int V) {
  extern __shared__ float sm[];
  float* lat = sm;                 // [TT][rank]
  float* wgt = sm + TT * rank;     // [TT][64]
  pdl_launch_dependents();
  const int t0 = blockIdx.x * TT, h = blockIdx.y, n_t = min(TT, b.n_seqs - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // this block's rows of W_uv: several blocks share a head's (each merges the runs for itself)
  const int per_z = (V + gridDim.z - 1) / gridDim.z, e_lo = blockIdx.z * per_z, e_hi = min(V, e_lo + per_z);
  if (blockIdx.x == 0 && e_lo < e_hi) fetch_ahead(w_uv + ((size_t)h * V + e_lo) * rank, (size_t)(e_hi - e_lo) * rank * sizeof(T));
  pdl_wait();
  for (int t = warp; t < TT; t += MERGE_THREADS / 32) {          // splits <= 64: two runs per lane
    const bool live = t < n_t && b.slot_ids[t0 + t] >= 0;        // a padding sequence: weights of zero
    float mi[2], li[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int i = lane + 32 * k;
      const size_t row = ((size_t)(live ? t0 + t : 0) * splits + (i < splits ? i : 0)) * Hpad + h;
      mi[k] = live && i < splits ? part_m[row] : -INFINITY;
      li[k] = live && i < splits ? part_l[row] : 0.f;
    }
    const float snk = sink ? sink[h] : -INFINITY;
    const float M = fmaxf(warp_max(fmaxf(mi[0], mi[1])), snk);
    float w[2], part = 0.f;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      w[k] = mi[k] == -INFINITY ? 0.f : expf(mi[k] - M);
      part += w[k] * li[k];
    }
    const float L = warp_sum(part) + (sink ? expf(snk - M) : 0.f);
    const float inv = L > 0.f ? 1.0f / L : 0.f;
#pragma unroll
    for (int k = 0; k < 2; ++k) wgt[t * 64 + lane + 32 * k] = lane + 32 * k < splits ? w[k] * inv : 0.f;
  }
  __syncthreads();
  // the runs' partial sums, four numbers per thread, four runs' loads in flight; an empty run's row (weight 0) is never read
  const int r4 = rank >> 2;
  for (int j = threadIdx.x; j < TT * r4; j += MERGE_THREADS) {
    const int t = j / r4, r = 4 * (j - t * r4);
    const float* wt = wgt + t * 64;
    const float* src = part_acc + (((size_t)(t0 + t) * splits) * Hpad + h) * rank + r;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i0 = 0; i0 < splits; i0 += 4) {
      float4 v[4];
      float w[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        w[k] = wt[(i0 + k) & 63];                       // zero beyond the last run
        v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (w[k] != 0.f) v[k] = *reinterpret_cast<const float4*>(src + (size_t)(i0 + k) * Hpad * rank);
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        a.x = fmaf(w[k], v[k].x, a.x); a.y = fmaf(w[k], v[k].y, a.y);
        a.z = fmaf(w[k], v[k].z, a.z); a.w = fmaf(w[k], v[k].w, a.w);
      }
    }
    *reinterpret_cast<float4*>(lat + 4 * j) = a;
  }
  __syncthreads();
  // W_uv: rank is a multiple of 8, 16-byte loads of eight weights; the loads of ROWS rows are issued before the first is used
  constexpr int ROWS = TT > 2 ? 4 : 8;
  for (int e0 = e_lo + warp * ROWS; e0 < e_hi; e0 += (MERGE_THREADS / 32) * ROWS) {
    float a[ROWS][TT];
#pragma unroll
    for (int k = 0; k < ROWS; ++k)
#pragma unroll
      for (int t = 0; t < TT; ++t) a[k][t] = 0.f;
    for (int r = lane * 8; r < rank; r += 32 * 8) {
      uint4 v[ROWS];
#pragma unroll
      for (int k = 0; k < ROWS; ++k)
        v[k] = e0 + k < e_hi ? *reinterpret_cast<const uint4*>(w_uv + ((size_t)h * V + e0 + k) * rank + r) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
      for (int t = 0; t < TT; ++t) {
        float x[8];
#pragma unroll
        for (int c = 0; c < 8; ++c) x[c] = lat[t * rank + r + c];
#pragma unroll
        for (int k = 0; k < ROWS; ++k) {
          const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&v[k]);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float2 f = __bfloat1622float2(p[c]);
            a[k][t] = fmaf(f.x, x[2 * c], a[k][t]);
            a[k][t] = fmaf(f.y, x[2 * c + 1], a[k][t]);
          }
        }
      }
    }
#pragma unroll
    for (int k = 0; k < ROWS; ++k)
#pragma unroll
      for (int t = 0; t < TT; ++t) {
        const float sum = warp_sum(a[k][t]);
        if (lane == 0 && e0 + k < e_hi && t < n_t)
          out[((size_t)(t0 + t) * H + h) * V + e0 + k] = from_f32<T>(gate ? sum * gate[(size_t)(t0 + t) * H + h] : sum);
      }
  }
}

size_t decode_smem(int mt, int width) {
  return (size_t)(mt * 16 + BK) * (width + 8) * 2 + (size_t)mt * 16 * PLD * 2 + (size_t)8 * mt * 16 * 4;
}

bool umma_enabled() {
  static const bool on = [] { const char* e = getenv("IERT_LATENT_UMMA"); return !(e && e[0] == '0'); }();
  return on;
}

}  // namespace

// latent_decode_umma.cu
int latent_umma_heads(int H, int rank, int R);
int launch_latent_decode_umma(const void* qa, const IertBatchView* batch, const IertKvView* kv, int H, int Hpad, int R, float scale,
                              int splits, float* part_m, float* part_l, float* part_acc, int* err, cudaStream_t stream);

// Heads padded to whole MMA tiles (16, or 32 from 17 heads on), and how many runs of tiles a sequence is cut into.
// `table_width`: pages of the longest walk.
IERT_API int iert_latent_decode_tc_plan(int n_seqs, int H, int rank, int R, int table_width, int* Hpad, int* splits) {
  const int tiles = (H + 15) / 16, mt = tiles >= 2 ? 2 : 1;
  const int groups = (tiles + mt - 1) / mt;
  *Hpad = groups * mt * 16;
  if (umma_enabled() && latent_umma_heads(H, rank, R)) {
    // one CTA per SM: as many runs as end soonest, a run costing its pages and about two pages' worth of beginning and end
    const int slots = iert_sm_count_cached(), ctas = n_seqs * groups > 0 ? n_seqs * groups : 1;
    int best = 1;
    long long best_cost = -1;
    for (int k = 1; k <= 32; ++k) {
      const long long cost = (long long)((ctas * k + slots - 1) / slots) * ((table_width + k - 1) / k + 2);
      if (best_cost < 0 || cost < best_cost) { best = k; best_cost = cost; }
    }
    *splits = best;
    return IERT_OK;
  }
  int want = (2 * iert_sm_count_cached() + n_seqs * groups - 1) / (n_seqs * groups > 0 ? n_seqs * groups : 1);
  if (want > 32) want = 32;
  // a run's partial result (heads x rank floats) is as many bytes as 16 or more cached rows: runs of fewer than
  // four tiles of the longest sequence the cache can hold cost more than they spread
  if (want > (table_width + 3) / 4) want = (table_width + 3) / 4;
  if (want < 1) want = 1;
  *splits = want;
  return IERT_OK;
}

// q [T, ldq] (H*(D+R) per token, one token per sequence: per head D unrotated and R rotated numbers), bf16 with the rotated
// numbers turned already, or with q_f32 != 0 fp32 as projected (turned here by inv_freq, rot_mul and pairing); the cache's
// rows are rank + R wide (latent | rotated key part); w_uk [H*D, rank], w_uv [H*V, rank] bf16 row-major; gate: fp32 [T, H]
// or null.  qa: scratch bf16 [T, Hpad, rank + R]; part_m, part_l: fp32 [T, splits, Hpad]; part_acc: fp32 [T, splits, Hpad, rank];
// out bf16 [T, H*V].  Hpad and splits as iert_latent_decode_tc_plan gives them.
IERT_API int iert_latent_attention_decode_tc(const void* q, int q_f32, long long ldq, const float* inv_freq, float rot_mul, int pairing, const void* w_uk, const void* w_uv, void* out,
                                             const IertBatchView* batch, const IertKvView* kv, int H, int D, int R, int V,
                                             float scale, const float* sink, const float* gate, int Hpad, int splits,
                                             void* qa, float* part_m, float* part_l, float* part_acc, int* err,
                                             cudaStream_t stream) {
  const int T = batch->n_tokens, width = kv->head_dim, rank = width - R;
  if (T <= 0) return IERT_OK;
  const bool umma = umma_enabled() && latent_umma_heads(H, rank, R) && ((uintptr_t)qa & 15) == 0 && ((uintptr_t)kv->k & 15) == 0;
  if (!umma && (rank % 32 || R % 16 || rank < 32)) return IERT_BAD_ARGUMENT;
  if (T != batch->n_seqs || kv->dtype != IERT_BF16 || kv->kv_heads != 1 || kv->page_tokens != BK || rank % 8 || R < 0 ||
      width > 640 || rank < 8 || rank > MAX_NTW * 32 || H <= 0 || Hpad % 16 || Hpad < H || Hpad > 65535 || splits < 1 || splits > 64 ||
      D <= 0 || 4 * (D + 4 * rank) > 12000 || V <= 0 || (q_f32 && R > 0 && !inv_freq))
    return IERT_BAD_ARGUMENT;
  const int mt = Hpad % 32 == 0 ? 2 : 1;
  const size_t smem = decode_smem(mt, width);
  static bool configured = false;
  if (!configured) {
    const int most = (int)decode_smem(2, 640);
    if (cudaFuncSetAttribute(latent_decode_tc_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, most) != cudaSuccess ||
        cudaFuncSetAttribute(latent_decode_tc_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, most) != cudaSuccess) {
      cudaGetLastError();
      return IERT_CUDA_ERROR;
    }
    configured = true;
  }
  // tokens that share a head's weights in the kernels around: one when there are few, so that there are blocks enough
  const int tt = T <= 4 ? 1 : T <= 8 ? 2 : 4;
#define ABSORB(TQ, TT)                                                                                                             \
  launch_dep(latent_absorb_q_kernel<TQ, TT>, dim3((T + TT - 1) / TT, Hpad), dim3(ABSORB_THREADS), (size_t)TT * (D + 4 * rank) * sizeof(float), \
             stream, (const TQ*)q, ldq, (const __nv_bfloat16*)w_uk, (__nv_bfloat16*)qa, H, Hpad, D, R, rank, inv_freq, rot_mul, pairing, *batch)
  if (q_f32) { if (tt == 1) ABSORB(float, 1); else if (tt == 2) ABSORB(float, 2); else ABSORB(float, 4); }
  else { if (tt == 1) ABSORB(__nv_bfloat16, 1); else if (tt == 2) ABSORB(__nv_bfloat16, 2); else ABSORB(__nv_bfloat16, 4); }
#undef ABSORB
  dim3 grid(T, splits, Hpad / (mt * 16));
  if (umma) {
    const int st = launch_latent_decode_umma(qa, batch, kv, H, Hpad, R, scale, splits, part_m, part_l, part_acc, err, stream);
    if (st != IERT_OK) return IERT_CUDA_ERROR;       // (the sizes were checked above)
  } else if (mt == 2)
    launch_dep(latent_decode_tc_kernel<2>, grid, dim3(THREADS), smem, stream, (const __nv_bfloat16*)qa, *batch, *kv, Hpad, R,
               scale, splits, part_m, part_l, part_acc, err);
  else
    launch_dep(latent_decode_tc_kernel<1>, grid, dim3(THREADS), smem, stream, (const __nv_bfloat16*)qa, *batch, *kv, Hpad, R,
               scale, splits, part_m, part_l, part_acc, err);
#define MERGE(TT)                                                                                                                  \
  launch_dep(latent_decode_merge_kernel<__nv_bfloat16, TT>, dim3((T + TT - 1) / TT, H, V >= 64 && T <= 8 ? 2 : 1), dim3(MERGE_THREADS),                       \
             (size_t)TT * (rank + 64) * sizeof(float), stream, (const float*)part_m, (const float*)part_l, (const float*)part_acc, splits, \
             Hpad, rank, sink, gate, (const __nv_bfloat16*)w_uv, (__nv_bfloat16*)out, *batch, H, V)
  if (tt == 1) MERGE(1);
  else if (tt == 2) MERGE(2);
  else MERGE(4);
#undef MERGE
  return iert_check_launch("latent_attention_decode_tc");
}
