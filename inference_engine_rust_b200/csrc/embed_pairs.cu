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
  if (threadIdx.x == 0) {
    if (!in_range) atomicOr(err, IERT_ERR_TOKEN_RANGE);
    const int s = sequence_of_token(b, t), slot = s >= 0 ? b.slot_ids[s] : -1;
    int row = -1;                               // padding: no pair row
    if (slot >= 0) {
      const int at = t - b.cu_q[s], pos = b.pos0[s] + at;
      int prev = -1;
      if (at > 0) prev = ids[t - 1];
      else if (pos > 0) prev = last[slot * last_stride];
      if (at == 0) last[slot * last_stride] = ids[b.cu_q[s + 1] - 1];
      row = pos == 0 ? buckets : (int)((unsigned long long)((long long)prev * mul_prev + (long long)id * mul_cur) % (unsigned long long)buckets);
    }
    row_s = row;
  }
  __syncthreads();
  const int row = row_s;
  const TW* src = table + (size_t)(in_range ? id : 0) * hidden;
  const TP* two = pairs + (size_t)(row >= 0 ? row : 0) * hidden;
  float* o = x + (size_t)t * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x)
    o[i] = (in_range ? to_f32(src[i]) * scale : 0.f) + (row >= 0 ? to_f32(two[i]) : 0.f);
}

}  // namespace

// pairs: [buckets + 1, hidden]; last: int32, slot s at last[s * last_stride]; mul_prev, mul_cur >= 0.
IERT_API int iert_embed_pairs(const void* table, int table_dtype, const void* pairs, int pairs_dtype, const int* ids, float* x,
                              int n_tokens, int hidden, int vocab, float scale, int buckets, long long mul_prev, long long mul_cur,
                              int* last, long long last_stride, const IertBatchView* batch, int* err, cudaStream_t stream) {
  if (n_tokens <= 0) return IERT_OK;
  if (hidden <= 0 || vocab <= 0 || buckets <= 0 || mul_prev < 0 || mul_cur < 0 || n_tokens != batch->n_tokens) return IERT_BAD_ARGUMENT;
  const int threads = hidden >= 1024 ? 256 : 128;
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
