// Embedding with a second table indexed by a hash of the token and the token in front of it:
//
//   x[t] = table[id_t] * scale + pairs[row_t],   row_t = (id_(t-1) * mul_prev + id_t * mul_cur) mod buckets,
//   row_t = buckets (the table's last row) for a sequence's first token.
//
// The token in front of the first token that a step brings is part of the sequence's state: `last` [slots], one int32
// each, read where a sequence goes on and replaced by the last token of the step.  One block per token; the block of a
// sequence's first token of the step is the only one that reads or writes the state, so nothing races.
#include "common.cuh"

using namespace iert;

namespace {

// The pair row of token t (-1: padding, none), by one thread of its block; the block of a sequence's first token of the
// step also hands the step's last token on to the next.
__device__ __forceinline__ int pair_row(const int* ids, int t, int id, bool in_range, int buckets, long long mul_prev, long long mul_cur,
                                        int* last, long long last_stride, const IertBatchView& b, int* err) {
  if (!in_range) atomicOr(err, IERT_ERR_TOKEN_RANGE);
  const int s = sequence_of_token(b, t), slot = s >= 0 ? b.slot_ids[s] : -1;
  if (slot < 0) return -1;
  const int at = t - b.cu_q[s], pos = b.pos0[s] + at;
  int prev = 0;
  if (at > 0) prev = ids[t - 1];
  else if (pos > 0) prev = last[slot * last_stride];
  if (at == 0) last[slot * last_stride] = ids[b.cu_q[s + 1] - 1];
  if (pos == 0) return buckets;
  return (int)((unsigned long long)((long long)prev * mul_prev + (long long)id * mul_cur) % (unsigned long long)buckets);
}

template <typename TW, typename TP>
__global__ void embed_pairs_kernel(const TW* __restrict__ table, const TP* __restrict__ pairs, const int* __restrict__ ids,
                                   float* __restrict__ x, int hidden, int vocab, float scale, int buckets, long long mul_prev,
                                   long long mul_cur, int* __restrict__ last, long long last_stride, IertBatchView b,
                                   int* __restrict__ err) {
  __shared__ int row_s;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, id = ids[t];
  const bool in_range = id >= 0 && id < vocab;
  if (threadIdx.x == 0) row_s = pair_row(ids, t, id, in_range, buckets, mul_prev, mul_cur, last, last_stride, b, err);
  __syncthreads();
  const int row = row_s;
  const TW* src = table + (size_t)(in_range ? id : 0) * hidden;
  const TP* two = pairs + (size_t)(row >= 0 ? row : 0) * hidden;
  float* o = x + (size_t)t * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x)
    o[i] = (in_range ? to_f32(src[i]) * scale : 0.f) + (row >= 0 ? to_f32(two[i]) : 0.f);
}

// The same with 16-byte accesses for bf16 tables: eight numbers per thread and pass, the token's row on its way before
// the pair row is known.  hidden a multiple of 8, at most 8 * G * blockDim.x.
template <int G>
__global__ void embed_pairs_bf16x8_kernel(const __nv_bfloat16* __restrict__ table, const __nv_bfloat16* __restrict__ pairs,
                                          const int* __restrict__ ids, float* __restrict__ x, int hidden, int vocab, float scale,
                                          int buckets, long long mul_prev, long long mul_cur, int* __restrict__ last,
                                          long long last_stride, IertBatchView b, int* __restrict__ err) {
  __shared__ int row_s;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, id = ids[t];
  const bool in_range = id >= 0 && id < vocab;
  const __nv_bfloat16* src = table + (size_t)(in_range ? id : 0) * hidden;
  const uint4 none = make_uint4(0u, 0u, 0u, 0u);
  uint4 own[G];
#pragma unroll
  for (int k = 0; k < G; ++k) {
    const int i = 8 * (threadIdx.x + k * blockDim.x);
    own[k] = in_range && i < hidden ? *reinterpret_cast<const uint4*>(src + i) : none;
  }
  if (threadIdx.x == 0) row_s = pair_row(ids, t, id, in_range, buckets, mul_prev, mul_cur, last, last_stride, b, err);
  __syncthreads();
  const int row = row_s;
  const __nv_bfloat16* two = pairs + (size_t)(row >= 0 ? row : 0) * hidden;
  uint4 add[G];
#pragma unroll
  for (int k = 0; k < G; ++k) {
    const int i = 8 * (threadIdx.x + k * blockDim.x);
    add[k] = row >= 0 && i < hidden ? *reinterpret_cast<const uint4*>(two + i) : none;
  }
  float* o = x + (size_t)t * hidden;
#pragma unroll
  for (int k = 0; k < G; ++k) {
    const int i = 8 * (threadIdx.x + k * blockDim.x);
    if (i >= hidden) break;
    const __nv_bfloat162* pa = reinterpret_cast<const __nv_bfloat162*>(&own[k]);
    const __nv_bfloat162* pb = reinterpret_cast<const __nv_bfloat162*>(&add[k]);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float2 a0 = __bfloat1622float2(pa[2 * e]), a1 = __bfloat1622float2(pa[2 * e + 1]);
      const float2 b0 = __bfloat1622float2(pb[2 * e]), b1 = __bfloat1622float2(pb[2 * e + 1]);
      *reinterpret_cast<float4*>(o + i + 4 * e) =
          make_float4(a0.x * scale + b0.x, a0.y * scale + b0.y, a1.x * scale + b1.x, a1.y * scale + b1.y);
    }
  }
}

}  // namespace

// pairs: [buckets + 1, hidden]; last: int32, slot s at last[s * last_stride]; mul_prev, mul_cur >= 0.
IERT_API int iert_embed_pairs(const void* table, int table_dtype, const void* pairs, int pairs_dtype, const int* ids, float* x,
                              int n_tokens, int hidden, int vocab, float scale, int buckets, long long mul_prev, long long mul_cur,
                              int* last, long long last_stride, const IertBatchView* batch, int* err, cudaStream_t stream) {
  if (n_tokens <= 0) return IERT_OK;
  if (hidden <= 0 || vocab <= 0 || buckets <= 0 || mul_prev < 0 || mul_cur < 0 || n_tokens != batch->n_tokens) return IERT_BAD_ARGUMENT;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == IERT_BF16 && pairs_dtype == IERT_BF16 && hidden % 8 == 0 && hidden <= 8192 &&
      (((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)x) & 15) == 0) {
#define GO8(G, THREADS)                                                                                                      \
    launch_dep(embed_pairs_bf16x8_kernel<G>, dim3(n_tokens), dim3(THREADS), 0, stream, (const __nv_bfloat16*)table,          \
               (const __nv_bfloat16*)pairs, ids, x, hidden, vocab, scale, buckets, mul_prev, mul_cur, last, last_stride, *batch, err)
    if (hidden <= 1024) GO8(1, 128); else if (hidden <= 2048) GO8(1, 256); else if (hidden <= 4096) GO8(2, 256); else GO8(4, 256);
#undef GO8
    return iert_check_launch("embed_pairs");
  }
#define GO(A, C)                                                                                                             \
  launch_dep(embed_pairs_kernel<A, C>, dim3(n_tokens), dim3(threads), 0, stream, (const A*)table, (const C*)pairs, ids, x, hidden, \
             vocab, scale, buckets, mul_prev, mul_cur, last, last_stride, *batch, err)
  if (table_dtype == IERT_F32 && pairs_dtype == IERT_F32) GO(float, float);
  else if (table_dtype == IERT_BF16 && pairs_dtype == IERT_BF16) GO(__nv_bfloat16, __nv_bfloat16);
  else if (table_dtype == IERT_BF16 && pairs_dtype == IERT_F32) GO(__nv_bfloat16, float);
  else if (table_dtype == IERT_F32 && pairs_dtype == IERT_BF16) GO(float, __nv_bfloat16);
  else return IERT_BAD_ARGUMENT;
#undef GO
  return iert_check_launch("embed_pairs");
}
