// Layer norm (mean and variance, weight and bias) fused with the residual sum.  With d = sum_p delta[p] (+ bias), the pending
// branch output (float32 partial sums are added in index order), and
//     LN(v) = (v - mean) / sqrt(mean((v - mean)^2) + eps) * w + b
// there are two forms:
//   * before a branch:  x = residual + d;      out = LN(x);               residual <- x (when it is written back);
//   * after a branch:   x = residual + LN(d);  out = x, rounded;          residual <- x.
// The first also runs over gathered rows (the last norm of a model).  All arithmetic is float32; the variance is the mean
// of the squared deviations, taken from the values in registers, not from a sum of squares.
#include "common.cuh"

LSE_CHECK_DEFINE(lse_check_layer_norm)

namespace {
template <typename T> __device__ __forceinline__ void ln_load4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void ln_load4<float>(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <> __device__ __forceinline__ void ln_load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <typename T> __device__ __forceinline__ void ln_store4(T* p, const float (&v)[4]);
template <> __device__ __forceinline__ void ln_store4<float>(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void ln_store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[4]) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = raw;
}

// Four values of the sum of n_partials rows, eight loads in flight, added in index order from zero.
template <typename TD>
__device__ __forceinline__ void ln_sum4(const TD* del, int n_partials, long long stride, float (&sum)[4]) {
  int p = 0;
  for (; p + 8 <= n_partials; p += 8) {
    float a[8][4];
#pragma unroll
    for (int k = 0; k < 8; ++k) ln_load4<TD>(del + (size_t)(p + k) * stride, a[k]);
#pragma unroll
    for (int k = 0; k < 8; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) sum[e] += a[k][e];
  }
  for (; p + 4 <= n_partials; p += 4) {
    float a[4][4];
#pragma unroll
    for (int k = 0; k < 4; ++k) ln_load4<TD>(del + (size_t)(p + k) * stride, a[k]);
#pragma unroll
    for (int k = 0; k < 4; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) sum[e] += a[k][e];
  }
  for (; p < n_partials; ++p) {
    float a[4];
    ln_load4<TD>(del + (size_t)p * stride, a);
#pragma unroll
    for (int e = 0; e < 4; ++e) sum[e] += a[e];
  }
}

struct NormArgs {
  float* residual;
  int n_partials;
  long long partial_stride;
  const float* bias;
  const float* weight;
  const float* shift;
  const int* rows;
  int hidden, tokens, after, write_residual;
  float eps;
};

// Rows whose width is a multiple of 4 up to blockDim * 4 * C: the row stays in registers (a thread owns C float4 pieces).
template <typename TD, typename TO, int C>
__global__ void __launch_bounds__(256, C <= 4 ? 4 : 2)
layer_norm_regs_kernel(NormArgs a, const TD* __restrict__ delta, TO* __restrict__ out) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  const int pieces = a.hidden / 4;
  pdl_wait();
  const int t = a.rows ? LSE_CHECKED(a.rows[blockIdx.x], 0, a.tokens, 0, LSE_CHECK_ROW) : (int)blockIdx.x;
  float* res = a.residual + (size_t)t * a.hidden;
  const TD* del = delta ? delta + (size_t)t * a.hidden : nullptr;
  TO* dst = out ? out + (size_t)blockIdx.x * a.hidden : nullptr;
  float x[C][4], v[C][4];    // the residual's values; what is normed
  float total = 0.f;
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int piece = threadIdx.x + c * blockDim.x;
#pragma unroll
    for (int e = 0; e < 4; ++e) x[c][e] = v[c][e] = 0.f;
    if (piece < pieces) {
      const int i = piece * 4;
      ln_load4<float>(res + i, x[c]);
      if (del) ln_sum4<TD>(del + i, a.n_partials, a.partial_stride, v[c]);
      if (a.bias) {
        float b[4];
        ln_load4<float>(a.bias + i, b);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[c][e] += b[e];
      }
      if (!a.after) {
#pragma unroll
        for (int e = 0; e < 4; ++e) v[c][e] += x[c][e];
        if (a.write_residual) ln_store4<float>(res + i, v[c]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) total += v[c][e];
    }
  }
  const float mean = block_sum(total, scratch) / (float)a.hidden;
  float sq = 0.f;
#pragma unroll
  for (int c = 0; c < C; ++c)
    if ((int)(threadIdx.x + c * blockDim.x) < pieces) {
#pragma unroll
      for (int e = 0; e < 4; ++e) { v[c][e] -= mean; sq = fmaf(v[c][e], v[c][e], sq); }
    }
  const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)a.hidden + a.eps);
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int piece = threadIdx.x + c * blockDim.x;
    if (piece < pieces) {
      const int i = piece * 4;
      float w[4], b[4], y[4];
      ln_load4<float>(a.weight + i, w);
      ln_load4<float>(a.shift + i, b);
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = fmaf(v[c][e] * inv, w[e], b[e]);
      if (a.after) {
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] += x[c][e];
        ln_store4<float>(res + i, y);
      }
      if (dst) ln_store4<TO>(dst + i, y);
    }
  }
}

// Any width: what is normed waits in the output's place of the residual (before a branch) or is summed again.
template <typename TD, typename TO>
__global__ void __launch_bounds__(256)
layer_norm_any_kernel(NormArgs a, const TD* __restrict__ delta, TO* __restrict__ out) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = a.rows ? LSE_CHECKED(a.rows[blockIdx.x], 0, a.tokens, 0, LSE_CHECK_ROW) : (int)blockIdx.x;
  float* res = a.residual + (size_t)t * a.hidden;
  const TD* del = delta ? delta + (size_t)t * a.hidden : nullptr;
  TO* dst = out ? out + (size_t)blockIdx.x * a.hidden : nullptr;
  auto value = [&](int i) {
    float s = del ? sum_partials<TD>(del + i, a.n_partials, a.partial_stride) : 0.f;
    if (a.bias) s += a.bias[i];
    return a.after ? s : s + res[i];
  };
  float total = 0.f;
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) total += value(i);
  const float mean = block_sum(total, scratch) / (float)a.hidden;
  float sq = 0.f;
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) { const float d = value(i) - mean; sq = fmaf(d, d, sq); }
  const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)a.hidden + a.eps);
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) {
    const float v = value(i);
    float y = fmaf((v - mean) * inv, a.weight[i], a.shift[i]);
    if (a.after) { y += res[i]; res[i] = y; }
    else if (a.write_residual) res[i] = v;
    if (dst) dst[i] = from_f32<TO>(y);
  }
}
}  // namespace

// residual float32 [tokens, hidden]; delta [tokens, hidden] or n_partials partial sums partial_stride apart, or null;
// bias (of the pending output), weight, shift float32 [hidden] (bias may be null); after: see the top of the file;
// rows int32 [n_rows] or null (all rows in order; required with after); out [n_rows, hidden] or null.
extern "C" int lse_layer_norm(float* residual, const void* delta, int delta_dtype, int n_partials, long long partial_stride,
                              const float* bias, const float* weight, const float* shift, float eps, int after, void* out,
                              int out_dtype, const int* rows, int n_rows, int hidden, int tokens, int write_residual,
                              cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (hidden <= 0 || !residual || !weight || !shift || (delta && n_partials < 1) || (after && (rows || !delta)) ||
      (rows && write_residual) || (!after && !out))
    return LSE_ERR_BAD_ARGUMENT;
  const NormArgs args = {residual, n_partials, partial_stride, bias, weight, shift, rows, hidden, tokens, after, write_residual, eps};
  // narrow rows of many tokens: fewer threads a row, more rows an SM; float32 keeps one block size, hence one order of sums
  const int threads = (out_dtype == LSE_DTYPE_BF16 && n_rows > 256 && hidden <= 1024) ? 128 : 256;
  const bool aligned = (((uintptr_t)residual | (uintptr_t)delta | (uintptr_t)out | (uintptr_t)weight | (uintptr_t)shift | (uintptr_t)bias) & 15) == 0;
  const int pieces = aligned && hidden % 4 == 0 && partial_stride % 4 == 0 ? (hidden / 4 + threads - 1) / threads : 0;
#define LSE_LN_LAUNCH(K, TD, TO) lse_launch(K, n_rows, threads, 0, stream, args, (const TD*)delta, (TO*)out)
#define LSE_LN_CASE(TD, TO)                                                           \
  if (pieces == 1) LSE_LN_LAUNCH((layer_norm_regs_kernel<TD, TO, 1>), TD, TO);        \
  else if (pieces == 2) LSE_LN_LAUNCH((layer_norm_regs_kernel<TD, TO, 2>), TD, TO);   \
  else if (pieces == 3 || pieces == 4) LSE_LN_LAUNCH((layer_norm_regs_kernel<TD, TO, 4>), TD, TO); \
  else if (pieces >= 5 && pieces <= 8) LSE_LN_LAUNCH((layer_norm_regs_kernel<TD, TO, 8>), TD, TO); \
  else LSE_LN_LAUNCH((layer_norm_any_kernel<TD, TO>), TD, TO)
  if (delta_dtype == LSE_DTYPE_F32 && out_dtype == LSE_DTYPE_F32) { LSE_LN_CASE(float, float); }
  else if (delta_dtype == LSE_DTYPE_BF16 && out_dtype == LSE_DTYPE_BF16) { LSE_LN_CASE(__nv_bfloat16, __nv_bfloat16); }
  else if (delta_dtype == LSE_DTYPE_F32 && out_dtype == LSE_DTYPE_BF16) { LSE_LN_CASE(float, __nv_bfloat16); }
  else if (delta_dtype == LSE_DTYPE_BF16 && out_dtype == LSE_DTYPE_F32) { LSE_LN_CASE(__nv_bfloat16, float); }
  else return LSE_ERR_BAD_ARGUMENT;
#undef LSE_LN_CASE
#undef LSE_LN_LAUNCH
  LSE_LAUNCH_CHECK();
}
