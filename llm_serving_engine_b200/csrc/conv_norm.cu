// The residual sum, a layer's norm and a short convolution of the normed rows over time, in one pass; the forms of the
// sum and the norm without a convolution; and the small elementwise step of a token's own input.
//
//   x_t = residual_t + d_t,      d_t = delta_t (+ bias), or delta_t / rms(delta_t) * delta_weight
//   h_t = x_t / sqrt(mean(x_t^2) + eps) * weight
//   out_t = h_t + sum_j w[:, j] h_(t - taps + 1 + j)          (h = 0 before the request's first token)
//
// delta is a branch's pending output: rows of float32 or bfloat16, or a float32 stack of partial sums.  A request's last
// taps - 1 rows of h are kept, in float32, in its state slot ([slots, taps - 1, hidden], oldest first), so that a step
// can start anywhere.
//
//   lse_conv_norm:         the whole of it for 1 to 4 taps and widths that are multiples of four up to 8,192.  When every
//       request brings one token: one launch, a block per row, which moves its window on.  Else three: the sum with
//       the rows' factors 1 / rms, the norm with the convolution (x is read once more, from L2), the windows.
//   lse_delta_norm_rmsnorm: x and h without a convolution, any width, with gathered rows (a model's last norm) and as the
//       first half of convolutions that lse_conv_norm was not built for.
//   lse_residual_settle:   residual += d in place, and the sum rounded into the compute dtype.
//   lse_token_gate:        g[t, i] = gelu_tanh(z[t, i]) * table[id_t, offset + i], zero in the padding columns.
#include "common.cuh"

LSE_CHECK_DEFINE(lse_check_conv_norm)

namespace {
template <typename T> __device__ __forceinline__ void cn_load4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void cn_load4<float>(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <> __device__ __forceinline__ void cn_load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <typename T> __device__ __forceinline__ void cn_store4(T* p, const float (&v)[4]);
template <> __device__ __forceinline__ void cn_store4<float>(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void cn_store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[4]) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = raw;
}

// d and the sum: x (this thread's pieces threadIdx.x, threadIdx.x + blockDim.x, ... of four channels of one row) becomes
// residual + d; returns the sum of squares over the row.  Every load is issued before any is used.
template <typename TD, int C>
__device__ __forceinline__ float cn_sum_row(const float* __restrict__ res, const TD* __restrict__ del, int n_partials,
                                            long long partial_stride, const float* __restrict__ bias,
                                            const float* __restrict__ delta_weight, float delta_eps, int hidden,
                                            float* scratch, float (&x)[C][4]) {
  const int pieces = hidden / 4;
  float r[C][4], dw[C][4], sq = 0.f;
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int piece = threadIdx.x + c * blockDim.x;
#pragma unroll
    for (int e = 0; e < 4; ++e) x[c][e] = r[c][e] = dw[c][e] = 0.f;
    if (piece < pieces) {
      cn_load4<float>(res + piece * 4, r[c]);
      if (delta_weight) cn_load4<float>(delta_weight + piece * 4, dw[c]);
      if (del) {
        const TD* src = del + piece * 4;
        int p = 0;
        for (; p + 8 <= n_partials; p += 8) {     // eight loads in flight, added in index order
          float a[8][4];
#pragma unroll
          for (int k = 0; k < 8; ++k) cn_load4<TD>(src + (size_t)(p + k) * partial_stride, a[k]);
#pragma unroll
          for (int k = 0; k < 8; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) x[c][e] += a[k][e];
        }
        for (; p + 2 <= n_partials; p += 2) {
          float a[2][4];
#pragma unroll
          for (int k = 0; k < 2; ++k) cn_load4<TD>(src + (size_t)(p + k) * partial_stride, a[k]);
#pragma unroll
          for (int k = 0; k < 2; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) x[c][e] += a[k][e];
        }
        for (; p < n_partials; ++p) {
          float a[4];
          cn_load4<TD>(src + (size_t)p * partial_stride, a);
#pragma unroll
          for (int e = 0; e < 4; ++e) x[c][e] += a[e];
        }
        if (bias) {
          float b[4];
          cn_load4<float>(bias + piece * 4, b);
#pragma unroll
          for (int e = 0; e < 4; ++e) x[c][e] += b[e];
        }
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) sq = fmaf(x[c][e], x[c][e], sq);
  }
  if (delta_weight && del) {                      // the pending output passes a norm of its own
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)hidden + delta_eps);
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
      for (int e = 0; e < 4; ++e) x[c][e] = (x[c][e] * inv) * dw[c][e];
  }
  sq = 0.f;
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      x[c][e] += r[c][e];
      sq = fmaf(x[c][e], x[c][e], sq);
    }
  return block_sum(sq, scratch);
}

// Every request brings one row: a block per row, which finds its predecessors in the window and moves it on.
template <typename TD, typename TO, int TAPS, int C>
__global__ void __launch_bounds__(512)
conv_norm_single_kernel(float* __restrict__ residual, const TD* __restrict__ delta, int n_partials, long long partial_stride,
                        const float* __restrict__ bias, const float* __restrict__ delta_weight, float delta_eps,
                        const float* __restrict__ weight, float eps, const float* __restrict__ conv_weight,
                        float* __restrict__ state, const int* __restrict__ segment_of_token,
                        const int* __restrict__ segment_slot, TO* __restrict__ out, int hidden, int num_slots,
                        int num_segments) {
  constexpr int BACK = TAPS - 1, HELD = BACK > 0 ? BACK : 1;
  __shared__ float scratch[32];
  pdl_launch_dependents();
  const int pieces = hidden / 4;
  float nw[C][4], cw[C][4][TAPS];
#pragma unroll
  for (int c = 0; c < C; ++c) {      // the weights do not depend on earlier kernels
    const int piece = threadIdx.x + c * blockDim.x;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      nw[c][e] = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) cw[c][e][j] = 0.f;
    }
    if (piece < pieces) {
      cn_load4<float>(weight + piece * 4, nw[c]);
      float* flat = &cw[c][0][0];    // four channels' taps lie one after the other
#pragma unroll
      for (int k = 0; k < TAPS; ++k) {
        float a[4];
        cn_load4<float>(conv_weight + (size_t)piece * 4 * TAPS + 4 * k, a);
#pragma unroll
        for (int e = 0; e < 4; ++e) flat[4 * k + e] = a[e];
      }
    }
  }
  pdl_wait();
  const int row = blockIdx.x;
  int seg = segment_of_token[row];
  if (seg < 0) return;
  seg = LSE_CHECKED(seg, 0, num_segments, 0, LSE_CHECK_SEGMENT);
  float* window = BACK > 0 ? state + (size_t)LSE_CHECKED(segment_slot[seg], 0, num_slots, 0, LSE_CHECK_ROW) * BACK * hidden : nullptr;
  float before[HELD][C][4];
#pragma unroll
  for (int i = 0; i < BACK; ++i)
#pragma unroll
    for (int c = 0; c < C; ++c) {
      const int piece = threadIdx.x + c * blockDim.x;
#pragma unroll
      for (int e = 0; e < 4; ++e) before[i][c][e] = 0.f;
      if (piece < pieces) cn_load4<float>(window + (size_t)i * hidden + piece * 4, before[i][c]);
    }
  float* res = residual + (size_t)row * hidden;
  float x[C][4];
  const float sq = cn_sum_row<TD, C>(res, delta ? delta + (size_t)row * hidden : nullptr, n_partials, partial_stride, bias,
                                     delta_weight, delta_eps, hidden, scratch, x);
  const float inv = 1.0f / sqrtf(sq / (float)hidden + eps);
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int piece = threadIdx.x + c * blockDim.x;
    if (piece < pieces) {
      float h[4], y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        h[e] = (x[c][e] * inv) * nw[c][e];
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < BACK; ++j) sum = fmaf(cw[c][e][j], before[j][c][e], sum);
        y[e] = h[e] + fmaf(cw[c][e][TAPS - 1], h[e], sum);
      }
      cn_store4<TO>(out + (size_t)row * hidden + piece * 4, y);
      cn_store4<float>(res + piece * 4, x[c]);
#pragma unroll
      for (int i = 0; i + 1 < BACK; ++i) cn_store4<float>(window + (size_t)i * hidden + piece * 4, before[i + 1][c]);
      if (BACK > 0) cn_store4<float>(window + (size_t)(BACK - 1) * hidden + piece * 4, h);
    }
  }
}

// Many rows, first half: x in place, and every row's factor 1 / sqrt(mean(x^2) + eps).  A block per row.
template <typename TD, int C>
__global__ void __launch_bounds__(256)
conv_norm_rows_kernel(float* __restrict__ residual, const TD* __restrict__ delta, int n_partials, long long partial_stride,
                      const float* __restrict__ bias, const float* __restrict__ delta_weight, float delta_eps, float eps,
                      float* __restrict__ factor, int hidden) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, pieces = hidden / 4;
  float* res = residual + (size_t)row * hidden;
  float x[C][4];
  const float sq = cn_sum_row<TD, C>(res, delta ? delta + (size_t)row * hidden : nullptr, n_partials, partial_stride, bias,
                                     delta_weight, delta_eps, hidden, scratch, x);
  if (delta) {
#pragma unroll
    for (int c = 0; c < C; ++c) {
      const int piece = threadIdx.x + c * blockDim.x;
      if (piece < pieces) cn_store4<float>(res + piece * 4, x[c]);
    }
  }
  if (threadIdx.x == 0) factor[row] = 1.0f / sqrtf(sq / (float)hidden + eps);
}

// Second half: h = x * factor * weight and h + conv(h).  A thread owns four channels and walks CN_ROWS rows with the last
// taps - 1 rows of h in registers; the rows of x are fetched CN_AHEAD at a time.  grid (row tiles, channel tiles)
constexpr int CN_ROWS = 16, CN_AHEAD = 4;
template <typename TO, int TAPS>
__global__ void __launch_bounds__(128)
conv_norm_apply_kernel(const float* __restrict__ x, const float* __restrict__ factor, const float* __restrict__ weight,
                       const float* __restrict__ conv_weight, const float* __restrict__ state,
                       const int* __restrict__ segment_of_token, const int* __restrict__ segment_start,
                       const int* __restrict__ segment_slot, TO* __restrict__ out, int tokens, int hidden, int num_slots,
                       int num_segments) {
  constexpr int BACK = TAPS - 1, HELD = BACK > 0 ? BACK : 1;
  pdl_launch_dependents();
  const int piece = blockIdx.y * blockDim.x + threadIdx.x;
  if (piece * 4 >= hidden) return;
  float nw[4], cw[4][TAPS];
  cn_load4<float>(weight + piece * 4, nw);
  float* flat = &cw[0][0];
#pragma unroll
  for (int k = 0; k < TAPS; ++k) {
    float a[4];
    cn_load4<float>(conv_weight + (size_t)piece * 4 * TAPS + 4 * k, a);
#pragma unroll
    for (int e = 0; e < 4; ++e) flat[4 * k + e] = a[e];
  }
  pdl_wait();
  const int first = blockIdx.x * CN_ROWS, end = min(tokens, first + CN_ROWS);
  auto normed = [&](int row, float (&h)[4]) {
    float v[4];
    cn_load4<float>(x + (size_t)row * hidden + piece * 4, v);
    const float f = factor[row];
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = (v[e] * f) * nw[e];
  };
  float before[HELD][4];
  int held = -1;
  for (int base = first; base < end; base += CN_AHEAD) {
    float h[CN_AHEAD][4];
    int segs[CN_AHEAD];
#pragma unroll
    for (int g = 0; g < CN_AHEAD; ++g) {
      const int row = min(base + g, end - 1);
      segs[g] = segment_of_token[row];
      normed(row, h[g]);
    }
#pragma unroll
    for (int g = 0; g < CN_AHEAD; ++g) {
      const int row = base + g;
      if (row < end) {
        int seg = segs[g];
        if (seg < 0) {
          held = -1;
        } else {
          seg = LSE_CHECKED(seg, 0, num_segments, 0, LSE_CHECK_SEGMENT);
          if (BACK > 0 && seg != held) {        // the first row of a request in this tile
            const float* window = state + (size_t)LSE_CHECKED(segment_slot[seg], 0, num_slots, 0, LSE_CHECK_ROW) * BACK * hidden;
            const int l = row - segment_start[seg];
#pragma unroll
            for (int i = 0; i < BACK; ++i) {
              const int back = BACK - i;
              if (l - back >= 0) normed(row - back, before[i]);
              else cn_load4<float>(window + (size_t)(BACK + l - back) * hidden + piece * 4, before[i]);
            }
            held = seg;
          }
          float y[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < BACK; ++j) sum = fmaf(cw[e][j], before[j][e], sum);
            y[e] = h[g][e] + fmaf(cw[e][TAPS - 1], h[g][e], sum);
          }
          cn_store4<TO>(out + (size_t)row * hidden + piece * 4, y);
          if (BACK > 0) {
#pragma unroll
            for (int i = 0; i + 1 < BACK; ++i)
#pragma unroll
              for (int e = 0; e < 4; ++e) before[i][e] = before[i + 1][e];
#pragma unroll
            for (int e = 0; e < 4; ++e) before[HELD - 1][e] = h[g][e];
          }
        }
      }
    }
  }
}

// The windows after a step of many rows: entry i holds h at the request's row count - (taps - 1) + i of this step, or moves up
// from behind (in ascending order an entry only reads entries behind it).  grid (requests, channel tiles)
__global__ void __launch_bounds__(128)
conv_norm_state_kernel(const float* __restrict__ x, const float* __restrict__ factor, const float* __restrict__ weight,
                       float* __restrict__ state, const int* __restrict__ segment_start,
                       const int* __restrict__ segment_slot, int hidden, int taps, int num_slots) {
  pdl_launch_dependents();
  pdl_wait();
  const int seg = blockIdx.x;
  const int row0 = segment_start[seg], count = segment_start[seg + 1] - row0;
  const int piece = blockIdx.y * blockDim.x + threadIdx.x;
  if (count <= 0 || piece * 4 >= hidden) return;
  float* window = state + (size_t)LSE_CHECKED(segment_slot[seg], 0, num_slots, 0, LSE_CHECK_ROW) * (taps - 1) * hidden + piece * 4;
  float nw[4];
  cn_load4<float>(weight + piece * 4, nw);
#pragma unroll 4
  for (int i = 0; i < taps - 1; ++i) {
    const int l = count - (taps - 1) + i;
    float v[4];
    if (l < 0) {
      cn_load4<float>(window + (size_t)(i + count) * hidden, v);
    } else {
      cn_load4<float>(x + (size_t)(row0 + l) * hidden + piece * 4, v);
      const float f = factor[row0 + l];
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = (v[e] * f) * nw[e];
    }
    cn_store4<float>(window + (size_t)i * hidden, v);
  }
}

// A block per row; the row of x in shared memory.
template <typename TD, typename TO>
__global__ void __launch_bounds__(256)
delta_norm_rmsnorm_kernel(float* __restrict__ residual, const TD* __restrict__ delta, int n_partials,
                          long long partial_stride, const float* __restrict__ bias,
                          const float* __restrict__ delta_weight, float delta_eps, const float* __restrict__ weight,
                          float eps, TO* __restrict__ out, const int* __restrict__ rows, int hidden, int tokens,
                          int write_residual) {
  extern __shared__ float row_s[];
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = rows ? LSE_CHECKED(rows[blockIdx.x], 0, tokens, 0, LSE_CHECK_ROW) : blockIdx.x;
  float* res = residual + (size_t)t * hidden;
  const TD* del = delta ? delta + (size_t)t * hidden : nullptr;
  float sq = 0.f;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
    float v = del ? sum_partials<TD>(del + c, n_partials, partial_stride) : 0.f;
    if (del && bias) v += bias[c];
    row_s[c] = v;                    // read back by the same thread only
    sq = fmaf(v, v, sq);
  }
  const bool normed = delta_weight != nullptr && del != nullptr;
  const float inv_d = normed ? 1.0f / sqrtf(block_sum(sq, scratch) / (float)hidden + delta_eps) : 1.f;
  sq = 0.f;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
    const float x = res[c] + (normed ? (row_s[c] * inv_d) * delta_weight[c] : row_s[c]);
    if (write_residual) res[c] = x;
    row_s[c] = x;
    sq = fmaf(x, x, sq);
  }
  const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)hidden + eps);
  for (int c = threadIdx.x; c < hidden; c += blockDim.x)
    out[(size_t)blockIdx.x * hidden + c] = from_f32<TO>((row_s[c] * inv) * weight[c]);
}

// Four values a thread (by_four), else one.
template <typename TD, typename TO>
__global__ void __launch_bounds__(256)
residual_settle_kernel(float* __restrict__ residual, const TD* __restrict__ delta, int n_partials,
                       long long partial_stride, const float* __restrict__ bias, TO* __restrict__ copy, long long count,
                       int hidden, int by_four) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x;
  if (by_four) {
    if (i * 4 >= count) return;
    float x[4], sum[4] = {0.f, 0.f, 0.f, 0.f};
    cn_load4<float>(residual + i * 4, x);
    int p = 0;
    for (; p + 4 <= n_partials; p += 4) {
      float a[4][4];
#pragma unroll
      for (int k = 0; k < 4; ++k) cn_load4<TD>(delta + (size_t)(p + k) * partial_stride + i * 4, a[k]);
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int e = 0; e < 4; ++e) sum[e] += a[k][e];
    }
    for (; p < n_partials; ++p) {
      float a[4];
      cn_load4<TD>(delta + (size_t)p * partial_stride + i * 4, a);
#pragma unroll
      for (int e = 0; e < 4; ++e) sum[e] += a[e];
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] += sum[e] + (bias ? bias[(int)((i * 4 + e) % hidden)] : 0.f);
    cn_store4<float>(residual + i * 4, x);
    if (copy) cn_store4<TO>(copy + i * 4, x);
    return;
  }
  if (i >= count) return;
  const float x = residual[i] + (sum_partials<TD>(delta + i, n_partials, partial_stride) + (bias ? bias[(int)(i % hidden)] : 0.f));
  residual[i] = x;
  if (copy) copy[i] = from_f32<TO>(x);
}

template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
token_gate_kernel(const TI* __restrict__ z, int n_partials, long long partial_stride, long long ld,
                  const TO* __restrict__ table, long long table_ld, int offset, const int* __restrict__ ids, int vocab,
                  TO* __restrict__ out, int tokens, int dim, int out_ld) {
  pdl_launch_dependents();
  pdl_wait();
  const long long e = blockIdx.x * (long long)blockDim.x + threadIdx.x;
  if (e >= (long long)tokens * out_ld) return;
  const int t = (int)(e / out_ld), i = (int)(e % out_ld);
  float g = 0.f;
  if (i < dim) {
    const int id = LSE_CHECKED(ids[t], 0, vocab, 0, LSE_CHECK_TOKEN_ID);
    const float v = sum_partials<TI>(z + (size_t)t * ld + i, n_partials, partial_stride);
    const float inner = 0.7978845608028654f * fmaf(0.044715f * v * v, v, v);
    g = 0.5f * v * (1.0f + tanhf(inner)) * to_f32<TO>(table[(size_t)id * table_ld + offset + i]);
  }
  out[e] = from_f32<TO>(g);
}

}  // namespace

#define LSE_CN_TYPES(CASE)                                                                                   \
  if (delta_dtype == LSE_DTYPE_F32 && out_dtype == LSE_DTYPE_F32) { CASE(float, float) }                     \
  else if (delta_dtype == LSE_DTYPE_BF16 && out_dtype == LSE_DTYPE_BF16) { CASE(__nv_bfloat16, __nv_bfloat16) } \
  else if (delta_dtype == LSE_DTYPE_F32 && out_dtype == LSE_DTYPE_BF16) { CASE(float, __nv_bfloat16) }       \
  else if (delta_dtype == LSE_DTYPE_BF16 && out_dtype == LSE_DTYPE_F32) { CASE(__nv_bfloat16, float) }       \
  else return LSE_ERR_BAD_ARGUMENT;

// Whether lse_conv_norm takes this shape.
extern "C" int lse_conv_norm_supported(int hidden, int taps) {
  return hidden > 0 && hidden % 4 == 0 && hidden <= 8192 && taps >= 1 && taps <= 4;
}

// residual float32 [tokens, hidden], becomes x; delta [tokens, hidden] or a float32 stack, or null; bias float32 [hidden] or
// null (belongs to delta); delta_weight float32 [hidden] or null; conv_weight float32 [hidden, taps]; state float32 [slots,
// taps - 1, hidden], moved on; single: every request brings one token (one launch), else factor (float32 [tokens]) is
// scratch and three kernels run.
extern "C" int lse_conv_norm(float* residual, const void* delta, int delta_dtype, int n_partials, long long partial_stride,
                             const float* bias, const float* delta_weight, float delta_eps, const float* weight, float eps,
                             const float* conv_weight, float* state, const int* segment_of_token, const int* segment_start,
                             const int* segment_slot, void* out, int out_dtype, float* factor, int tokens, int hidden, int taps,
                             int single, int num_slots, int num_segments, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (!lse_conv_norm_supported(hidden, taps) || n_partials < 1 || partial_stride % 4 || (!single && !factor)) return LSE_ERR_BAD_ARGUMENT;
  const int pieces = hidden / 4;
  if (single) {
    const int threads = pieces <= 512 ? (pieces + 31) / 32 * 32 : 512;
#define LSE_CN_GO(TD, TO, TAPS, C)                                                                                     \
  lse_launch(conv_norm_single_kernel<TD, TO, TAPS, C>, tokens, threads, 0, stream, residual, (const TD*)delta, n_partials, \
             partial_stride, bias, delta_weight, delta_eps, weight, eps, conv_weight, state, segment_of_token,          \
             segment_slot, (TO*)out, hidden, num_slots, num_segments)
#define LSE_CN_TAPS(TD, TO, C)                     \
  switch (taps) {                                  \
    case 1: LSE_CN_GO(TD, TO, 1, C); break;        \
    case 2: LSE_CN_GO(TD, TO, 2, C); break;        \
    case 3: LSE_CN_GO(TD, TO, 3, C); break;        \
    default: LSE_CN_GO(TD, TO, 4, C); break;       \
  }
#define LSE_CN_CASE(TD, TO)                        \
  if (pieces <= 512) { LSE_CN_TAPS(TD, TO, 1) }    \
  else if (pieces <= 1024) { LSE_CN_TAPS(TD, TO, 2) } \
  else { LSE_CN_TAPS(TD, TO, 4) }
    if (delta_dtype == LSE_DTYPE_F32 && out_dtype == LSE_DTYPE_F32) { LSE_CN_CASE(float, float) }
    else if (delta_dtype == LSE_DTYPE_BF16 && out_dtype == LSE_DTYPE_BF16) { LSE_CN_CASE(__nv_bfloat16, __nv_bfloat16) }
    else if (delta_dtype == LSE_DTYPE_F32 && out_dtype == LSE_DTYPE_BF16) { LSE_CN_CASE(float, __nv_bfloat16) }
    else return LSE_ERR_BAD_ARGUMENT;
#undef LSE_CN_CASE
#undef LSE_CN_TAPS
#undef LSE_CN_GO
    LSE_LAUNCH_CHECK();
  }
#define LSE_CN_ROWS_GO(TD, C)                                                                                          \
  lse_launch(conv_norm_rows_kernel<TD, C>, tokens, threads, 0, stream, residual, (const TD*)delta, n_partials, partial_stride, \
             bias, delta_weight, delta_eps, eps, factor, hidden)
#define LSE_CN_ROWS_CASE(TD)                       \
  if (pieces <= 256) LSE_CN_ROWS_GO(TD, 1);        \
  else if (pieces <= 512) LSE_CN_ROWS_GO(TD, 2);   \
  else if (pieces <= 1024) LSE_CN_ROWS_GO(TD, 4);  \
  else LSE_CN_ROWS_GO(TD, 8)
  const int threads = pieces < 256 ? (pieces + 31) / 32 * 32 : 256;
  if (delta_dtype == LSE_DTYPE_F32) { LSE_CN_ROWS_CASE(float); }
  else if (delta_dtype == LSE_DTYPE_BF16) { LSE_CN_ROWS_CASE(__nv_bfloat16); }
  else return LSE_ERR_BAD_ARGUMENT;
#undef LSE_CN_ROWS_CASE
#undef LSE_CN_ROWS_GO
  const dim3 grid((tokens + CN_ROWS - 1) / CN_ROWS, (pieces + 127) / 128);
#define LSE_CN_APPLY(TO, TAPS)                                                                                         \
  lse_launch(conv_norm_apply_kernel<TO, TAPS>, grid, 128, 0, stream, (const float*)residual, (const float*)factor, weight, \
             conv_weight, (const float*)state, segment_of_token, segment_start, segment_slot, (TO*)out, tokens, hidden,   \
             num_slots, num_segments)
#define LSE_CN_APPLY_CASE(TO)                      \
  switch (taps) {                                  \
    case 1: LSE_CN_APPLY(TO, 1); break;            \
    case 2: LSE_CN_APPLY(TO, 2); break;            \
    case 3: LSE_CN_APPLY(TO, 3); break;            \
    default: LSE_CN_APPLY(TO, 4); break;           \
  }
  if (out_dtype == LSE_DTYPE_F32) { LSE_CN_APPLY_CASE(float) }
  else if (out_dtype == LSE_DTYPE_BF16) { LSE_CN_APPLY_CASE(__nv_bfloat16) }
  else return LSE_ERR_BAD_ARGUMENT;
#undef LSE_CN_APPLY_CASE
#undef LSE_CN_APPLY
  if (taps > 1)
    lse_launch(conv_norm_state_kernel, dim3(num_segments, (pieces + 127) / 128), 128, 0, stream, (const float*)residual,
               (const float*)factor, weight, state, segment_start, segment_slot, hidden, taps, num_slots);
  LSE_LAUNCH_CHECK();
}

// out [n_rows, hidden]; rows int32 [n_rows] into the tokens rows of residual, or null (n_rows = tokens).
extern "C" int lse_delta_norm_rmsnorm(float* residual, const void* delta, int delta_dtype, int n_partials,
                                      long long partial_stride, const float* bias, const float* delta_weight,
                                      float delta_eps, const float* weight, float eps, void* out, int out_dtype,
                                      const int* rows, int n_rows, int hidden, int tokens, int write_residual,
                                      cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (hidden <= 0 || n_partials < 1) return LSE_ERR_BAD_ARGUMENT;
  constexpr size_t MOST = 192 * 1024;
  const size_t smem = sizeof(float) * (size_t)hidden;
  if (smem > MOST) return LSE_ERR_TOO_LARGE;
#define LSE_CN_CASE(TD, TO)                                                                                            \
  if (smem > 40 * 1024) {                                                                                              \
    const cudaError_t err = cudaFuncSetAttribute(delta_norm_rmsnorm_kernel<TD, TO>,                                    \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MOST);              \
    if (err != cudaSuccess) return (int)err;                                                                           \
  }                                                                                                                    \
  lse_launch(delta_norm_rmsnorm_kernel<TD, TO>, n_rows, 256, smem, stream, residual, (const TD*)delta, n_partials,      \
             partial_stride, bias, delta_weight, delta_eps, weight, eps, (TO*)out, rows, hidden, tokens, write_residual);
  LSE_CN_TYPES(LSE_CN_CASE)
#undef LSE_CN_CASE
  LSE_LAUNCH_CHECK();
}

// copy [tokens, hidden] in the compute dtype, or null.
extern "C" int lse_residual_settle(float* residual, const void* delta, int delta_dtype, int n_partials,
                                   long long partial_stride, const float* bias, void* copy, int out_dtype, int tokens,
                                   int hidden, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (hidden <= 0 || n_partials < 1 || !delta) return LSE_ERR_BAD_ARGUMENT;
  const long long count = (long long)tokens * hidden;
  const int by_four = hidden % 4 == 0 && partial_stride % 4 == 0;
  const long long blocks = ((by_four ? count / 4 : count) + 255) / 256;
  if (blocks > 0x7fffffffLL) return LSE_ERR_TOO_LARGE;
#define LSE_CN_CASE(TD, TO)                                                                                            \
  lse_launch(residual_settle_kernel<TD, TO>, (unsigned)blocks, 256, 0, stream, residual, (const TD*)delta, n_partials,  \
             partial_stride, bias, (TO*)copy, count, hidden, by_four);
  LSE_CN_TYPES(LSE_CN_CASE)
#undef LSE_CN_CASE
  LSE_LAUNCH_CHECK();
}

// z: rows of ld values (float32 / bfloat16 / a float32 stack); table [vocab, table_ld] and out [tokens, out_ld] in the
// compute dtype; columns dim .. out_ld of out are zero.
extern "C" int lse_token_gate(const void* z, int z_dtype, int n_partials, long long partial_stride, long long ld,
                              const void* table, long long table_ld, int offset, const int* ids, int vocab, void* out,
                              int out_dtype, int tokens, int dim, int out_ld, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (dim <= 0 || out_ld < dim || n_partials < 1 || offset < 0 || offset + dim > table_ld) return LSE_ERR_BAD_ARGUMENT;
  const long long blocks = ((long long)tokens * out_ld + 255) / 256;
  if (blocks > 0x7fffffffLL) return LSE_ERR_TOO_LARGE;
  const int delta_dtype = z_dtype;
#define LSE_CN_CASE(TI, TO)                                                                                            \
  lse_launch(token_gate_kernel<TI, TO>, (unsigned)blocks, 256, 0, stream, (const TI*)z, n_partials, partial_stride, ld, \
             (const TO*)table, table_ld, offset, ids, vocab, (TO*)out, tokens, dim, out_ld);
  LSE_CN_TYPES(LSE_CN_CASE)
#undef LSE_CN_CASE
  LSE_LAUNCH_CHECK();
}
