// LayerNorm of fp32 rows (the residual), one or two norms of the same row in one pass:
//
//   out[n] = (x - mean(x)) / sqrt(var(x) + eps) * w[n] + b[n],   var = mean((x - mean)^2),   n = 0 (, 1)
//
// Two norms that read the same row share its mean and its variance; only the weights differ.  The row is read once and
// stays in registers (16-byte accesses, four elements per group), the weights are fetched before the wait on the kernel
// in front, which they never depend on.  Everything fp32, sums in an order that depends on the sizes alone, one rounding
// at the store.
#include "common.cuh"

using namespace iert;

namespace {

struct LayerNormArgs {
  const float* x;            // [*, H]
  const int* rows_idx;       // output row i reads row rows_idx[i], or nullptr (i itself)
  int H;
  float eps;
  const float* w[2];
  const float* b[2];         // or nullptr
  void* out[2];              // [rows, H]; out[1] is nullptr when there is one norm
};

__device__ __forceinline__ void put4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, const float4& v) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = raw;
}

// G groups of four per thread; H a multiple of 4, at most 4 * G * blockDim.x.
template <typename T, int G, int N>
__global__ void layernorm_vec_kernel(LayerNormArgs a) {
  __shared__ float scratch[33];
  pdl_launch_dependents();
  const int n4 = a.H >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 w[N][G], b[N][G], x[G];
#pragma unroll
  for (int n = 0; n < N; ++n)
#pragma unroll
    for (int k = 0; k < G; ++k) {
      const int i = threadIdx.x + k * blockDim.x;
      w[n][k] = i < n4 ? *reinterpret_cast<const float4*>(a.w[n] + 4 * i) : zero;
      b[n][k] = i < n4 && a.b[n] ? *reinterpret_cast<const float4*>(a.b[n] + 4 * i) : zero;
    }
  pdl_wait();
  const int row = a.rows_idx ? a.rows_idx[blockIdx.x] : (int)blockIdx.x;
  const float* xr = a.x + (size_t)row * a.H;
  float sum = 0.f;
#pragma unroll
  for (int k = 0; k < G; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    x[k] = i < n4 ? *reinterpret_cast<const float4*>(xr + 4 * i) : zero;
    sum += (x[k].x + x[k].y) + (x[k].z + x[k].w);
  }
  const float mean = block_sum(sum, scratch) / (float)a.H;
  float dev = 0.f;
#pragma unroll
  for (int k = 0; k < G; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < n4) {
      x[k].x -= mean; x[k].y -= mean; x[k].z -= mean; x[k].w -= mean;
      dev += (x[k].x * x[k].x + x[k].y * x[k].y) + (x[k].z * x[k].z + x[k].w * x[k].w);
    }
  }
  const float r = 1.0f / sqrtf(block_sum(dev, scratch) / (float)a.H + a.eps);
#pragma unroll
  for (int n = 0; n < N; ++n) {
    T* o = (T*)a.out[n] + (size_t)blockIdx.x * a.H;
#pragma unroll
    for (int k = 0; k < G; ++k) {
      const int i = threadIdx.x + k * blockDim.x;
      if (i < n4)
        put4(o + 4 * i, make_float4(x[k].x * r * w[n][k].x + b[n][k].x, x[k].y * r * w[n][k].y + b[n][k].y,
                                    x[k].z * r * w[n][k].z + b[n][k].z, x[k].w * r * w[n][k].w + b[n][k].w));
    }
  }
}

// any row length: three passes over the row
template <typename T>
__global__ void layernorm_any_kernel(LayerNormArgs a) {
  __shared__ float scratch[33];
  pdl_launch_dependents();
  pdl_wait();
  const int row = a.rows_idx ? a.rows_idx[blockIdx.x] : (int)blockIdx.x;
  const float* xr = a.x + (size_t)row * a.H;
  float sum = 0.f;
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) sum += xr[i];
  const float mean = block_sum(sum, scratch) / (float)a.H;
  float dev = 0.f;
  for (int i = threadIdx.x; i < a.H; i += blockDim.x) { const float d = xr[i] - mean; dev = fmaf(d, d, dev); }
  const float r = 1.0f / sqrtf(block_sum(dev, scratch) / (float)a.H + a.eps);
  for (int n = 0; n < 2; ++n) {
    if (!a.out[n]) continue;
    T* o = (T*)a.out[n] + (size_t)blockIdx.x * a.H;
    for (int i = threadIdx.x; i < a.H; i += blockDim.x)
      o[i] = from_f32<T>((xr[i] - mean) * r * a.w[n][i] + (a.b[n] ? a.b[n][i] : 0.f));
  }
}

template <typename T, int N>
void launch_vec(const LayerNormArgs& a, int rows, cudaStream_t stream) {
  const int n4 = a.H >> 2;
  if (n4 <= 128) launch_dep(layernorm_vec_kernel<T, 1, N>, dim3(rows), dim3(128), 0, stream, a);
  else if (n4 <= 256) launch_dep(layernorm_vec_kernel<T, 1, N>, dim3(rows), dim3(256), 0, stream, a);
  else if (n4 <= 512) launch_dep(layernorm_vec_kernel<T, 2, N>, dim3(rows), dim3(256), 0, stream, a);
  else if (n4 <= 1024) launch_dep(layernorm_vec_kernel<T, 4, N>, dim3(rows), dim3(256), 0, stream, a);
  else launch_dep(layernorm_vec_kernel<T, 4, N>, dim3(rows), dim3(512), 0, stream, a);
}

}  // namespace

// x: fp32 rows of H; w0, b0 (and w1, b1 for a second norm of the same rows): fp32 [H], the b's optional; out0, out1 (or
// null): [rows, H] of out_dtype, apart from x.  rows_idx (optional) gathers rows of x.
IERT_API int iert_layernorm(const float* x, const int* rows_idx, int rows, int H, float eps, const float* w0, const float* b0,
                            void* out0, const float* w1, const float* b1, void* out1, int out_dtype, cudaStream_t stream) {
  if (rows <= 0) return IERT_OK;
  if (H <= 0 || !w0 || !out0 || (out1 && !w1) || (out_dtype != IERT_F32 && out_dtype != IERT_BF16)) return IERT_BAD_ARGUMENT;
  LayerNormArgs a = {x, rows_idx, H, eps, {w0, w1}, {b0, b1}, {out0, out1}};
  const uintptr_t all = (uintptr_t)x | (uintptr_t)w0 | (uintptr_t)b0 | (uintptr_t)out0 | (uintptr_t)w1 | (uintptr_t)b1 | (uintptr_t)out1;
  if (H % 4 == 0 && H <= 8192 && (all & 15) == 0) {
    if (out_dtype == IERT_F32) { if (out1) launch_vec<float, 2>(a, rows, stream); else launch_vec<float, 1>(a, rows, stream); }
    else { if (out1) launch_vec<__nv_bfloat16, 2>(a, rows, stream); else launch_vec<__nv_bfloat16, 1>(a, rows, stream); }
  } else if (out_dtype == IERT_F32) {
    launch_dep(layernorm_any_kernel<float>, dim3(rows), dim3(256), 0, stream, a);
  } else {
    launch_dep(layernorm_any_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, a);
  }
  return iert_check_launch("layernorm");
}
