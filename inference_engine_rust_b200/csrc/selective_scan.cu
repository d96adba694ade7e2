// The selective scan of a state-space mixer (Mamba: Gu and Dao, "Mamba: Linear-Time Sequence Modeling with Selective
// State Spaces").  With C channels, N states per channel and K convolution taps:
//
//   conv:   u[t, c] = silu(cb[c] + sum_j taps[c, K-1-j] x[t-j, c])         (causal, zeros before the start)
//   scan:   dt[t, c] = softplus(d[t, c] + db[c])
//           S[c, n] <- exp(dt[t, c] A[c, n]) S[c, n] + dt[t, c] u[t, c] B[t, n]
//           y[t, c] = sum_n S[c, n] C[t, n] + D[c] u[t, c];   out = y silu(z)
//
// The products d arrive in fp32; the step sizes, the state, the decays, the sums and the gate are fp32.  In
// bfloat16 runs A arrives as A log2(e) and a decay is one exponential to the base 2 of the special-function unit, whose
// relative error near 1 (2^-22) a state that hardly decays would gather over thousands of tokens; float32 runs take A as it
// is and form 1 + expm1(dt A).  A sequence's state is [S (C x N) | the last inputs of the convolution as a ring of K rows
// of C: the input of position p in row p % K] (see recurrent_prep.cu for why a ring needs no second launch).
//
// Prompts (selective_scan_kernel): a channel's state is spread over L neighbouring lanes, SPL = N / L states each in
// registers; a CTA of 128 threads owns 128 / L channels of one sequence and walks its tokens in chunks of 32.  While a
// chunk is computed, the next one's d, u, z, B and C are on their way into registers, which are then put into the other of
// two buffers in shared memory (as fp32, softplus applied): one barrier per chunk.  The lanes' partial sums of L tokens are added by a transposing reduction (L - 1 shuffles for
// L tokens), after which lane r holds token r's sum and applies D, the gate and the rounding.  A short last chunk is
// filled up with dt = 0, which changes no state.
// L is chosen at the launch: what bounds a prompt is the rate of exponentials (one per token, channel and state), so
// all that matters is enough warps per SM to keep that unit busy.
//
// One-token steps (selective_step_kernel): the same arithmetic, a thread per (channel, lane), no staging.
#include "common.cuh"

#include <stdlib.h>

using namespace iert;

namespace {

constexpr int MAX_TAPS = 16;
constexpr int THREADS = 128;
constexpr int CHUNK = 32;

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
// For results that are rounded to bfloat16.
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// softplus(v) = max(v, 0) + log(1 + e), e = exp(-|v|).  In bfloat16 runs without branches: the logarithm of the
// special-function unit where e is not small, else the first terms of the series of log(1 + e); relative error below 1e-5.
template <typename T>
__device__ __forceinline__ float softplus_of(float v) {
  if (sizeof(T) != 2) return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v)));
  const float e = __expf(-fabsf(v));
  const float series = e * fmaf(e, fmaf(e, fmaf(e, fmaf(e, 0.2f, -0.25f), 0.33333333f), -0.5f), 1.0f);
  return fmaxf(v, 0.f) + (e > 0.0625f ? __logf(1.0f + e) : series);
}

// The decay of a step: T the run's dtype (see above).
template <typename T>
__device__ __forceinline__ float decay_of(float dt, float A) {
  return sizeof(T) == 2 ? exp2_fast(dt * A) : 1.0f + expm1f(dt * A);
}

// Four consecutive numbers; `vec`: aligned, else one by one below `n` (zeros beyond).
__device__ __forceinline__ float4 load4(const float* p, bool vec, int n) {
  if (vec) return *reinterpret_cast<const float4*>(p);
  return make_float4(n > 0 ? p[0] : 0.f, n > 1 ? p[1] : 0.f, n > 2 ? p[2] : 0.f, n > 3 ? p[3] : 0.f);
}
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p, bool vec, int n) {
  if (vec) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
  }
  return make_float4(n > 0 ? to_f32(p[0]) : 0.f, n > 1 ? to_f32(p[1]) : 0.f, n > 2 ? to_f32(p[2]) : 0.f, n > 3 ? to_f32(p[3]) : 0.f);
}
// The same as stored, to be widened later: a load that nothing waits for.
template <typename T> struct Raw4;
template <> struct Raw4<float> { typedef float4 type; };
template <> struct Raw4<__nv_bfloat16> { typedef uint2 type; };
__device__ __forceinline__ float4 load_raw(const float* p, bool vec, int n) { return load4(p, vec, n); }
__device__ __forceinline__ uint2 load_raw(const __nv_bfloat16* p, bool vec, int n) {
  if (vec) return *reinterpret_cast<const uint2*>(p);
  const unsigned short* q = reinterpret_cast<const unsigned short*>(p);
  return make_uint2((n > 0 ? q[0] : 0u) | (n > 1 ? (uint32_t)q[1] << 16 : 0u), (n > 2 ? q[2] : 0u) | (n > 3 ? (uint32_t)q[3] << 16 : 0u));
}
__device__ __forceinline__ void zero_raw(float4& r) { r = make_float4(0.f, 0.f, 0.f, 0.f); }
__device__ __forceinline__ void zero_raw(uint2& r) { r = make_uint2(0u, 0u); }
__device__ __forceinline__ float4 widen(const float4& r) { return r; }
__device__ __forceinline__ float4 widen(const uint2& r) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, const float4& v, bool vec, int n) {
  if (vec) { *reinterpret_cast<float4*>(p) = v; return; }
  if (n > 0) p[0] = v.x;
  if (n > 1) p[1] = v.y;
  if (n > 2) p[2] = v.z;
  if (n > 3) p[3] = v.w;
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v, bool vec, int n) {
  if (vec) {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = raw;
    return;
  }
  if (n > 0) p[0] = __float2bfloat16_rn(v.x);
  if (n > 1) p[1] = __float2bfloat16_rn(v.y);
  if (n > 2) p[2] = __float2bfloat16_rn(v.z);
  if (n > 3) p[3] = __float2bfloat16_rn(v.w);
}

// ---------------------------------------------------------------------------------------
// convolution: four channels and PER consecutive tokens a thread

struct ConvArgs {
  const void* x;           // [T, ld] run dtype
  long long ld;
  const float* taps;       // fp32 [K, C] (transposed: one tap of all channels side by side)
  const float* bias;       // fp32 [C]
  float* state;            // per slot: ring [K, C] at ring_off
  long long state_stride, ring_off;
  void* u;                 // [T, C] run dtype
  int C, K, vec;
};

// KT > 0: K known, the last inputs stay in registers from token to token.  All inputs of a thread's run of tokens (neighbours
// in memory, whatever sequences they belong to) are asked for before the first is used.
template <typename T, int KT, int PER>
__global__ void __launch_bounds__(THREADS) selective_conv_kernel(ConvArgs a, IertBatchView b) {
  pdl_launch_dependents();
  const int K = KT > 0 ? KT : a.K;
  const int c = (blockIdx.y * THREADS + threadIdx.x) * 4;
  if (c >= a.C) return;
  const bool vec = a.vec;
  const int n = a.C - c, t0 = blockIdx.x * PER;
  constexpr int HELD = KT > 0 ? KT : 1;
  float4 w[HELD], hist[HELD];          // hist[j]: the input j tokens back
  if (KT > 0) {
#pragma unroll
    for (int j = 0; j < HELD; ++j) w[j] = load4(a.taps + (size_t)(K - 1 - j) * a.C + c, vec, n);
  }
  const float4 bias = load4(a.bias + c, vec, n);
  pdl_wait();
  const T* x = (const T*)a.x;
  typename Raw4<T>::type run[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i)
    if (t0 + i < b.n_tokens) run[i] = load_raw(x + (size_t)(t0 + i) * a.ld + c, vec, n);
  int seq = -2, slot = -1, q_begin = 0, q_end = 0, pos0 = 0;
  float* ring = nullptr;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int t = t0 + i;
    if (t >= b.n_tokens) break;
    bool fresh = false;
    if (seq < 0 || t >= q_end) {         // another sequence (or padding) from here on
      const int s = sequence_of_token(b, t);
      slot = s < 0 ? -1 : b.slot_ids[s];
      seq = slot < 0 ? -1 : s;
      if (slot >= 0) {
        q_begin = b.cu_q[s];
        q_end = b.cu_q[s + 1];
        pos0 = b.pos0[s];
        ring = a.state + (size_t)slot * a.state_stride + a.ring_off;
        fresh = true;
      }
    }
    if (slot < 0) continue;
    const int pos = pos0 + (t - q_begin);
    auto input = [&](int j) {            // j tokens back: from the step's rows, the ring, or zeros before the start
      if (t - j >= q_begin) return load4(x + (size_t)(t - j) * a.ld + c, vec, n);
      if (pos - j >= 0) return load4(ring + (size_t)((pos - j) % K) * a.C + c, vec, n);
      return make_float4(0.f, 0.f, 0.f, 0.f);
    };
    float4 acc = bias;
    const float4 now = widen(run[i]);
    if (KT > 0) {
      if (fresh) {
#pragma unroll
        for (int j = 1; j < HELD; ++j) hist[j] = input(j);
      }
      hist[0] = now;
#pragma unroll
      for (int j = HELD - 1; j >= 0; --j) {            // oldest first
        acc.x = fmaf(w[j].x, hist[j].x, acc.x); acc.y = fmaf(w[j].y, hist[j].y, acc.y);
        acc.z = fmaf(w[j].z, hist[j].z, acc.z); acc.w = fmaf(w[j].w, hist[j].w, acc.w);
      }
#pragma unroll
      for (int j = HELD - 1; j > 0; --j) hist[j] = hist[j - 1];
    } else {
      for (int j = K - 1; j >= 0; --j) {
        const float4 wv = load4(a.taps + (size_t)(K - 1 - j) * a.C + c, vec, n), xv = j == 0 ? now : input(j);
        acc.x = fmaf(wv.x, xv.x, acc.x); acc.y = fmaf(wv.y, xv.y, acc.y);
        acc.z = fmaf(wv.z, xv.z, acc.z); acc.w = fmaf(wv.w, xv.w, acc.w);
      }
    }
    store4((T*)a.u + (size_t)t * a.C + c,
           sizeof(T) == 2 ? make_float4(silu_fast(acc.x), silu_fast(acc.y), silu_fast(acc.z), silu_fast(acc.w))
                          : make_float4(silu_f(acc.x), silu_f(acc.y), silu_f(acc.z), silu_f(acc.w)), vec, n);
    if (t >= q_end - K) store4(ring + (size_t)(pos % K) * a.C + c, now, vec, n);      // a row no token of this launch reads
  }
}

// ---------------------------------------------------------------------------------------
// scan

struct ScanArgs {
  const void* u;           // [T, C] run dtype
  const float* dt;         // [T, C] fp32: the products, in front of bias and softplus
  const float* dt_bias;    // [C] fp32
  const void* bc;          // [T, ldp] run dtype: B [N] | C [N]
  long long ldp;
  const void* z;           // [T, ldz] run dtype
  long long ldz;
  const float* A2;         // [C, N] fp32: A log2(e) (float32 runs: A)
  const float* D;          // [C] fp32
  float* state;            // per slot: S [C, N] at s_off
  long long state_stride, s_off;
  void* out;               // [T, C] run dtype
  int C, N, vec, vec_bc;
};

constexpr size_t scan_smem_bytes(int L, int SPL) { return (size_t)2 * CHUNK * (4 * (THREADS / L) + 2 * L * SPL) * sizeof(float); }

template <typename T, int L, int SPL>
__global__ void __launch_bounds__(THREADS) selective_scan_kernel(ScanArgs a, IertBatchView b) {
  constexpr int CH = THREADS / L;                      // channels of the CTA
  constexpr int NP = L * SPL;                          // states, padded
  constexpr int Q = CH / 4;                            // runs of four channels in a row
  constexpr int ROWS_PT = CHUNK * Q / THREADS > 0 ? CHUNK * Q / THREADS : 1;      // such runs a thread fetches
  constexpr int BC_RUNS = CHUNK * 2 * NP / 4;          // runs of four numbers of B and C
  constexpr bool BC_AHEAD = NP <= 64;                  // small enough to fetch into registers ahead of time
  constexpr int BC_PT = BC_AHEAD ? (BC_RUNS + THREADS - 1) / THREADS : 1;
  extern __shared__ __align__(16) float sm[];          // scan_smem_bytes(L, SPL)
  // two buffers of [dt and dt u | u | z, then the results | B | C], each CHUNK rows
  constexpr int BUF = CHUNK * (4 * CH + 2 * NP);
  float2 (*d_s)[CH];
  float (*u_s)[CH], (*z_s)[CH], (*b_s)[NP], (*c_s)[NP];
  auto use = [&](int buf) {
    float* base = sm + buf * BUF;
    d_s = reinterpret_cast<float2 (*)[CH]>(base);
    u_s = reinterpret_cast<float (*)[CH]>(base + 2 * CHUNK * CH);
    z_s = reinterpret_cast<float (*)[CH]>(base + 3 * CHUNK * CH);
    b_s = reinterpret_cast<float (*)[NP]>(base + 4 * CHUNK * CH);
    c_s = reinterpret_cast<float (*)[NP]>(base + 4 * CHUNK * CH + CHUNK * NP);
  };
  pdl_launch_dependents();
  const int s = blockIdx.y;
  const int slot = b.slot_ids[s];
  const int t0 = b.cu_q[s], t1 = b.cu_q[s + 1];
  if (slot < 0 || t1 <= t0) return;
  const int tid = threadIdx.x, r = tid % L, ch = tid / L;
  const int c0 = blockIdx.x * CH, c = c0 + ch;
  const bool live = c < a.C;
  float A2[SPL], S[SPL];
#pragma unroll
  for (int i = 0; i < SPL; ++i) {
    const int n = r * SPL + i;
    A2[i] = live && n < a.N ? a.A2[(size_t)c * a.N + n] : 0.f;
  }
  const float Dc = live ? a.D[c] : 0.f;
  // the channels whose numbers this thread brings in are the same for all tokens
  static_assert(THREADS % Q == 0, "a thread's run of channels does not depend on the token");
  const int cq = c0 + 4 * (tid % Q);
  const float4 db = cq < a.C ? load4(a.dt_bias + cq, a.vec, a.C - cq) : make_float4(0.f, 0.f, 0.f, 0.f);
  pdl_wait();
  float* Sg = a.state + (size_t)slot * a.state_stride + a.s_off + (size_t)c * a.N;
#pragma unroll
  for (int i = 0; i < SPL; ++i) {
    const int n = r * SPL + i;
    S[i] = live && n < a.N ? Sg[n] : 0.f;
  }
  const T* u = (const T*)a.u;
  const T* z = (const T*)a.z;
  const T* bc = (const T*)a.bc;
  typedef typename Raw4<T>::type Raw;
  float4 dt_r[ROWS_PT];
  Raw u_r[ROWS_PT], z_r[ROWS_PT], bc_r[BC_PT];
  auto bc_run = [&](int x, int tc) {                   // run x of the chunk's [CHUNK][B NP | C NP]
    const int tt = x / (2 * NP / 4), q = x - tt * (2 * NP / 4);
    const bool is_c = q >= NP / 4;
    const int n = 4 * (is_c ? q - NP / 4 : q);
    Raw zero;
    zero_raw(zero);
    if (tc + tt >= t1 || n >= a.N) return zero;
    return load_raw(bc + (size_t)(tc + tt) * a.ldp + (is_c ? a.N : 0) + n, a.vec_bc, a.N - n);
  };
  auto fetch = [&](int tc) {
#pragma unroll
    for (int k = 0; k < ROWS_PT; ++k) {
      const int x = tid + k * THREADS;
      const int tt = x / Q, cc = c0 + 4 * (x % Q), t = tc + tt;
      dt_r[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      zero_raw(u_r[k]);
      zero_raw(z_r[k]);
      if (x < CHUNK * Q && t < t1 && cc < a.C) {
        const int n = a.C - cc;
        dt_r[k] = load4(a.dt + (size_t)t * a.C + cc, a.vec, n);
        u_r[k] = load_raw(u + (size_t)t * a.C + cc, a.vec, n);
        z_r[k] = load_raw(z + (size_t)t * a.ldz + cc, a.vec, n);
      }
    }
    if (BC_AHEAD) {
#pragma unroll
      for (int k = 0; k < BC_PT; ++k) {
        const int x = tid + k * THREADS;
        if (x < BC_RUNS) bc_r[k] = bc_run(x, tc);
      }
    }
  };
  auto put = [&](int tc) {
#pragma unroll
    for (int k = 0; k < ROWS_PT; ++k) {
      const int x = tid + k * THREADS;
      const int tt = x / Q, q = 4 * (x % Q);
      if (x < CHUNK * Q) {
        const float4 uv = widen(u_r[k]);
        float4 dv = make_float4(0.f, 0.f, 0.f, 0.f);       // a token beyond the sequence: no step
        if (tc + tt < t1)
          dv = make_float4(softplus_of<T>(dt_r[k].x + db.x), softplus_of<T>(dt_r[k].y + db.y), softplus_of<T>(dt_r[k].z + db.z),
                           softplus_of<T>(dt_r[k].w + db.w));
        *reinterpret_cast<float4*>(&d_s[tt][q]) = make_float4(dv.x, dv.x * uv.x, dv.y, dv.y * uv.y);
        *reinterpret_cast<float4*>(&d_s[tt][q + 2]) = make_float4(dv.z, dv.z * uv.z, dv.w, dv.w * uv.w);
        *reinterpret_cast<float4*>(&u_s[tt][q]) = uv;
        *reinterpret_cast<float4*>(&z_s[tt][q]) = widen(z_r[k]);
      }
    }
    auto put_bc = [&](int x, const Raw& raw) {
      const float4 v = widen(raw);
      const int tt = x / (2 * NP / 4), q = x - tt * (2 * NP / 4);
      if (q >= NP / 4) *reinterpret_cast<float4*>(&c_s[tt][4 * (q - NP / 4)]) = v;
      else *reinterpret_cast<float4*>(&b_s[tt][4 * q]) = v;
    };
    if (BC_AHEAD) {
#pragma unroll
      for (int k = 0; k < BC_PT; ++k) {
        const int x = tid + k * THREADS;
        if (x < BC_RUNS) put_bc(x, bc_r[k]);
      }
    } else {
      for (int x = tid; x < BC_RUNS; x += THREADS) put_bc(x, bc_run(x, tc));
    }
  };
  static_assert(NP % 4 == 0, "L is a multiple of 4");
  // What the chain of J tokens needs and no state enters: made one batch of tokens ahead of the chain, so that the shared
  // memory and the exponentials answer while the chain of the batch in front runs.
  constexpr int WANT = SPL >= 6 ? 2 : SPL >= 3 ? 4 : SPL == 2 ? 8 : 16;
  constexpr int J = WANT < L ? WANT : L;
  struct Ahead { float decay[J][SPL], in[J][SPL], out[J][SPL]; };
  auto prepare = [&](Ahead& x, int row) {
#pragma unroll
    for (int j = 0; j < J; ++j) {
      const float2 d = d_s[row + j][ch];
#pragma unroll
      for (int i = 0; i < SPL; ++i) {
        x.decay[j][i] = decay_of<T>(d.x, A2[i]);
        x.in[j][i] = d.y * b_s[row + j][r * SPL + i];
        x.out[j][i] = c_s[row + j][r * SPL + i];
      }
    }
  };
  T* out = (T*)a.out;
  auto store = [&](int tc) {                             // a chunk's results, by the threads that will overwrite them (put)
#pragma unroll
    for (int k = 0; k < ROWS_PT; ++k) {
      const int x = tid + k * THREADS;
      const int tt = x / Q, cc = c0 + 4 * (x % Q), t = tc + tt;
      if (x < CHUNK * Q && t < t1 && cc < a.C)
        store4(out + (size_t)t * a.C + cc, *reinterpret_cast<const float4*>(&z_s[tt][4 * (x % Q)]), a.vec, a.C - cc);
    }
  };
  int buf = 0;
  use(buf);
  fetch(t0);
  put(t0);
  for (int tc = t0; tc < t1; tc += CHUNK, buf ^= 1) {
    __syncthreads();                                     // this chunk is in place, the one in front is computed
    if (tc > t0) { use(buf ^ 1); store(tc - CHUNK); }
    if (tc + CHUNK < t1) fetch(tc + CHUNK);
    use(buf);
    Ahead cur;
    prepare(cur, 0);
#pragma unroll 2
    for (int g = 0; g < CHUNK; g += L) {
      float y[L];
#pragma unroll
      for (int h = 0; h < L; h += J) {
        Ahead nxt;
        prepare(nxt, min(g + h + J, CHUNK - J));       // (behind the chunk's last tokens: again those, for nothing)
#pragma unroll
        for (int j = 0; j < J; ++j) {
          float acc = 0.f;
#pragma unroll
          for (int i = 0; i < SPL; ++i) {
            S[i] = fmaf(cur.decay[j][i], S[i], cur.in[j][i]);
            acc = fmaf(S[i], cur.out[j][i], acc);
          }
          y[h + j] = acc;
        }
        cur = nxt;
      }
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) {
        const bool upper = r & o;
#pragma unroll
        for (int i = 0; i < o; ++i) {
          const float send = upper ? y[i] : y[i + o], mine = upper ? y[i + o] : y[i];
          y[i] = mine + __shfl_xor_sync(0xffffffffu, send, o);
        }
      }
      // lane r: token g + r
      const float uv = u_s[g + r][ch], zv = z_s[g + r][ch];
      z_s[g + r][ch] = fmaf(Dc, uv, y[0]) * (sizeof(T) == 2 ? silu_fast(zv) : silu_f(zv));
    }
    if (tc + CHUNK < t1) {
      use(buf ^ 1);
      put(tc + CHUNK);
    }
  }
  __syncthreads();
  use(buf ^ 1);
  store(t0 + (t1 - 1 - t0) / CHUNK * CHUNK);
  if (live) {
#pragma unroll
    for (int i = 0; i < SPL; ++i) {
      const int n = r * SPL + i;
      if (n < a.N) Sg[n] = S[i];
    }
  }
}

// One token per sequence: a thread per (channel, lane), `lanes` lanes a channel, ceil(N / lanes) states each.
template <typename T, int SPL>
__global__ void __launch_bounds__(THREADS) selective_step_kernel(ScanArgs a, int lanes, IertBatchView b) {
  pdl_launch_dependents();
  const int s = blockIdx.y;
  const int slot = b.slot_ids[s];
  const int c = blockIdx.x * (THREADS / lanes) + threadIdx.x / lanes, r = threadIdx.x % lanes;
  if (slot < 0 || b.cu_q[s + 1] <= b.cu_q[s]) return;
  const int t = b.cu_q[s];
  const bool live = c < a.C;
  float A2[SPL], S[SPL];
#pragma unroll
  for (int i = 0; i < SPL; ++i) {
    const int n = r * SPL + i;
    A2[i] = live && n < a.N ? a.A2[(size_t)c * a.N + n] : 0.f;
  }
  const float Dc = live ? a.D[c] : 0.f;
  float* Sg = a.state + (size_t)slot * a.state_stride + a.s_off + (size_t)c * a.N;
  pdl_wait();
#pragma unroll
  for (int i = 0; i < SPL; ++i) {
    const int n = r * SPL + i;
    S[i] = live && n < a.N ? Sg[n] : 0.f;
  }
  const float dt = live ? softplus_of<T>(a.dt[(size_t)t * a.C + c] + a.dt_bias[c]) : 0.f, uv = live ? to_f32(((const T*)a.u)[(size_t)t * a.C + c]) : 0.f;
  const float zv = live ? to_f32(((const T*)a.z)[(size_t)t * a.ldz + c]) : 0.f;
  const T* bc = (const T*)a.bc + (size_t)t * a.ldp;
  const float du = dt * uv;
  float acc = 0.f;
#pragma unroll
  for (int i = 0; i < SPL; ++i) {
    const int n = r * SPL + i;
    if (n < a.N) {
      S[i] = fmaf(decay_of<T>(dt, A2[i]), S[i], du * to_f32(bc[n]));
      acc = fmaf(S[i], to_f32(bc[a.N + n]), acc);
      if (live) Sg[n] = S[i];
    }
  }
  for (int o = lanes / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
  if (live && r == 0) ((T*)a.out)[(size_t)t * a.C + c] = from_f32<T>(fmaf(Dc, uv, acc) * silu_f(zv));
}

// States a lane holds: ceil(n) rounded up to one of the compiled sizes.
int states_per_lane(int N, int L) {
  const int need = (N + L - 1) / L;
  for (int s : {1, 2, 3, 4, 6, 8}) if (s >= need) return s;
  return 0;
}

template <typename T, int L, int SPL>
bool launch_scan_as(dim3 grid, cudaStream_t stream, const ScanArgs& a, const IertBatchView& b) {
  constexpr size_t smem = scan_smem_bytes(L, SPL);
  if (smem > 48 * 1024) {
    static bool configured = false;
    if (!configured && cudaFuncSetAttribute(selective_scan_kernel<T, L, SPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return false;
    configured = true;
  }
  launch_dep(selective_scan_kernel<T, L, SPL>, grid, dim3(THREADS), smem, stream, a, b);
  return true;
}

template <typename T, int L>
bool launch_scan(int spl, dim3 grid, cudaStream_t stream, const ScanArgs& a, const IertBatchView& b) {
  switch (spl) {
    case 1: return launch_scan_as<T, L, 1>(grid, stream, a, b);
    case 2: return launch_scan_as<T, L, 2>(grid, stream, a, b);
    case 3: return launch_scan_as<T, L, 3>(grid, stream, a, b);
    case 4: return launch_scan_as<T, L, 4>(grid, stream, a, b);
    case 6: return launch_scan_as<T, L, 6>(grid, stream, a, b);
    case 8: return launch_scan_as<T, L, 8>(grid, stream, a, b);
  }
  return false;
}

template <typename T>
bool launch_step(int spl, int lanes, dim3 grid, cudaStream_t stream, const ScanArgs& a, const IertBatchView& b) {
  switch (spl) {
    case 1: launch_dep(selective_step_kernel<T, 1>, grid, dim3(THREADS), 0, stream, a, lanes, b); return true;
    case 2: launch_dep(selective_step_kernel<T, 2>, grid, dim3(THREADS), 0, stream, a, lanes, b); return true;
    case 3: launch_dep(selective_step_kernel<T, 3>, grid, dim3(THREADS), 0, stream, a, lanes, b); return true;
    case 4: launch_dep(selective_step_kernel<T, 4>, grid, dim3(THREADS), 0, stream, a, lanes, b); return true;
    case 6: launch_dep(selective_step_kernel<T, 6>, grid, dim3(THREADS), 0, stream, a, lanes, b); return true;
    case 8: launch_dep(selective_step_kernel<T, 8>, grid, dim3(THREADS), 0, stream, a, lanes, b); return true;
  }
  return false;
}

template <typename T, int KT>
void launch_conv_as(cudaStream_t stream, const ConvArgs& a, const IertBatchView& b) {
  const int groups = (a.C + 4 * THREADS - 1) / (4 * THREADS);
  if (b.n_tokens >= 256)
    launch_dep(selective_conv_kernel<T, KT, 8>, dim3((b.n_tokens + 7) / 8, groups), dim3(THREADS), 0, stream, a, b);
  else
    launch_dep(selective_conv_kernel<T, KT, 1>, dim3(b.n_tokens, groups), dim3(THREADS), 0, stream, a, b);
}

template <typename T>
void launch_conv(cudaStream_t stream, const ConvArgs& a, const IertBatchView& b) {
  switch (a.K) {
    case 2: return launch_conv_as<T, 2>(stream, a, b);
    case 3: return launch_conv_as<T, 3>(stream, a, b);
    case 4: return launch_conv_as<T, 4>(stream, a, b);
    default: return launch_conv_as<T, 0>(stream, a, b);
  }
}

}  // namespace

// x: [T, ld] of `dtype` (C columns used); taps: fp32 [K, C]; bias: fp32 [C]; u: [T, C] of `dtype`; state: fp32 per slot, a ring of K
// rows of C at ring_off.
IERT_API int iert_selective_conv(const void* x, int dtype, long long ld, const float* taps, const float* bias, float* state,
                                 long long state_stride, long long ring_off, void* u, int C, int K, const IertBatchView* batch,
                                 cudaStream_t stream) {
  const int T = batch->n_tokens;
  if (T <= 0) return IERT_OK;
  if (C <= 0 || K < 1 || K > MAX_TAPS || (dtype != IERT_F32 && dtype != IERT_BF16)) return IERT_BAD_ARGUMENT;
  const int vec = C % 4 == 0 && ld % 4 == 0 && state_stride % 4 == 0 && ring_off % 4 == 0 &&
                  (((uintptr_t)x | (uintptr_t)taps | (uintptr_t)bias | (uintptr_t)state | (uintptr_t)u) & 15) == 0;
  const ConvArgs a = {x, ld, taps, bias, state, state_stride, ring_off, u, C, K, vec};
  if (dtype == IERT_F32) launch_conv<float>(stream, a, *batch);
  else launch_conv<__nv_bfloat16>(stream, a, *batch);
  return iert_check_launch("selective_conv");
}

// u, out: [T, C] of `dtype`; dt: fp32 [T, C], dt_bias: fp32 [C]; bc: [T, ldp] of `dtype`, B and C side by side; z: [T, ldz] of `dtype`; A2: fp32 [C, N] = A
// log2(e), or A itself where `dtype` is fp32; D: fp32 [C]; state: fp32 per slot, S [C, N] at s_off.  one_token: every sequence brings exactly one token.
IERT_API int iert_selective_scan(const void* u, int dtype, const float* dt, const float* dt_bias, const void* bc, long long ldp, const void* z, long long ldz,
                                 const float* A2, const float* D, float* state, long long state_stride, long long s_off, void* out,
                                 int C, int N, int one_token, const IertBatchView* batch, cudaStream_t stream) {
  if (batch->n_tokens <= 0 || batch->n_seqs <= 0) return IERT_OK;
  if (C <= 0 || N <= 0 || N > 256 || batch->n_seqs > 65535 || (dtype != IERT_F32 && dtype != IERT_BF16)) return IERT_BAD_ARGUMENT;
  const int vec = C % 4 == 0 && ldz % 4 == 0 &&
                  (((uintptr_t)u | (uintptr_t)dt | (uintptr_t)dt_bias | (uintptr_t)z | (uintptr_t)out) & 15) == 0;
  const int vec_bc = N % 4 == 0 && ldp % 4 == 0 && ((uintptr_t)bc & 15) == 0;
  const ScanArgs a = {u, dt, dt_bias, bc, ldp, z, ldz, A2, D, state, state_stride, s_off, out, C, N, vec, vec_bc};
  // lanes per channel: the fewest that hold all states (at most 8 each) and give about six warps per SM
  int L = 4;
  while (L < 32 && (!states_per_lane(N, L) || (long long)batch->n_seqs * C * L < 6LL * 32 * iert_sm_count_cached())) L *= 2;
  if (const char* forced = getenv("IERT_SCAN_LANES")) {            // for tests and measurements: 4, 8, 16 or 32
    const int f = atoi(forced);
    for (int l : {4, 8, 16, 32}) if (l == f && states_per_lane(N, l)) L = l;
  }
  const int spl = states_per_lane(N, L);
  if (!spl) return IERT_BAD_ARGUMENT;
  const dim3 grid((C + THREADS / L - 1) / (THREADS / L), batch->n_seqs);
  bool ok = false;
  if (one_token) {
    ok = dtype == IERT_F32 ? launch_step<float>(spl, L, grid, stream, a, *batch) : launch_step<__nv_bfloat16>(spl, L, grid, stream, a, *batch);
  } else {
#define GO(T) (L == 4 ? launch_scan<T, 4>(spl, grid, stream, a, *batch) : L == 8 ? launch_scan<T, 8>(spl, grid, stream, a, *batch) \
               : L == 16 ? launch_scan<T, 16>(spl, grid, stream, a, *batch) : launch_scan<T, 32>(spl, grid, stream, a, *batch))
    ok = dtype == IERT_F32 ? GO(float) : GO(__nv_bfloat16);
#undef GO
  }
  if (!ok) return IERT_BAD_ARGUMENT;
  return iert_check_launch("selective_scan");
}
