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
//   lse_conv_norm:         the whole of it for 1 to 4 taps and widths that are multiples of four.  x goes to a residual
//       tensor of its own (residual_out): a block works its rows' predecessors out again from residual and delta,
//       so those must stay as they were.  A block walks a few rows with the last taps - 1 rows of h in registers.
//   lse_conv_norm_state:   moves the windows on after a step with portions (a block per request works the last
//       rows of h out from residual_out).  Steps of single tokens move them on inside lse_conv_norm.
//   lse_delta_norm_rmsnorm: x and h without a convolution, any width, with gathered rows (a model's last norm) and as the
//       first half of convolutions that lse_conv_norm was not built for.
//   lse_residual_settle:   residual += d in place, and the sum rounded into the compute dtype.
//   lse_token_gate:        g[t, i] = gelu_tanh(z[t, i]) * table[id_t, offset + i], zero in the padding columns.
#include "common.cuh"

LSE_CHECK_DEFINE(lse_check_conv_norm)

namespace {
constexpr int CN_GROUP = 4;       // rows whose sums of squares are reduced together

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

// N sums over the block at once (lanes by butterfly, then warps in index order); scratch holds N * 32 floats.
template <int N>
__device__ __forceinline__ void block_sums(float (&v)[N], float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int n = 0; n < N; ++n) v[n] = warp_sum(v[n]);
  __syncthreads();
  if (lane == 0) {
#pragma unroll
    for (int n = 0; n < N; ++n) scratch[n * 32 + warp] = v[n];
  }
  __syncthreads();
#pragma unroll
  for (int n = 0; n < N; ++n) {
    float total = 0.f;
    for (int w = 0; w < nwarps; ++w) total += scratch[n * 32 + w];
    v[n] = total;
  }
}

// A thread owns pieces threadIdx.x, threadIdx.x + blockDim.x, ... (C of them) of four neighbouring channels.
template <typename TD, typename TO, int TAPS, int C>
__global__ void __launch_bounds__(512)
conv_norm_kernel(const float* __restrict__ residual, float* __restrict__ residual_out, const TD* __restrict__ delta,
                 int n_partials, long long partial_stride, const float* __restrict__ bias,
                 const float* __restrict__ delta_weight, float delta_eps, const float* __restrict__ weight, float eps,
                 const float* __restrict__ conv_weight, float* __restrict__ state,
                 const int* __restrict__ segment_of_token, const int* __restrict__ segment_start,
                 const int* __restrict__ segment_slot, TO* __restrict__ out, int tokens, int rows_per_block, int hidden,
                 int move_windows, int num_slots, int num_segments) {
  constexpr int BACK = TAPS - 1, HELD = BACK > 0 ? BACK : 1;
  __shared__ float scratch[CN_GROUP * 32];
  pdl_launch_dependents();
  const int pieces = hidden / 4;
  float nw[C][4], cw[TAPS][C][4];
#pragma unroll
  for (int c = 0; c < C; ++c) {      // the weights do not depend on earlier kernels
    const int piece = threadIdx.x + c * blockDim.x;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      nw[c][e] = piece < pieces ? weight[piece * 4 + e] : 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) cw[j][c][e] = piece < pieces ? conv_weight[(size_t)(piece * 4 + e) * TAPS + j] : 0.f;
    }
  }
  pdl_wait();
  const int first = blockIdx.x * rows_per_block, end = min(tokens, first + rows_per_block);
  int start = first;
  if (BACK > 0) {                    // the rows before the block's own that belong to the same request
    const int seg = segment_of_token[first];
    if (seg >= 0) start = max(segment_start[LSE_CHECKED(seg, 0, num_segments, 0, LSE_CHECK_SEGMENT)], first - BACK);
  }
  float before[HELD][C][4];          // before[i]: h of the row BACK - i rows back
#pragma unroll
  for (int i = 0; i < HELD; ++i)
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
      for (int e = 0; e < 4; ++e) before[i][c][e] = 0.f;
  int held = -1;                     // the request that `before` belongs to
  for (int base = start; base < end; base += CN_GROUP) {
    float x[CN_GROUP][C][4], sums[CN_GROUP];
#pragma unroll
    for (int g = 0; g < CN_GROUP; ++g) {
      sums[g] = 0.f;
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const int piece = threadIdx.x + c * blockDim.x;
#pragma unroll
        for (int e = 0; e < 4; ++e) x[g][c][e] = 0.f;
        if (base + g < end && piece < pieces && delta) {
          const TD* src = delta + (size_t)(base + g) * hidden + piece * 4;
          int p = 0;
          for (; p + 4 <= n_partials; p += 4) {     // four loads in flight, added in index order
            float a[4][4];
#pragma unroll
            for (int k = 0; k < 4; ++k) cn_load4<TD>(src + (size_t)(p + k) * partial_stride, a[k]);
#pragma unroll
            for (int k = 0; k < 4; ++k)
#pragma unroll
              for (int e = 0; e < 4; ++e) x[g][c][e] += a[k][e];
          }
          for (; p < n_partials; ++p) {
            float a[4];
            cn_load4<TD>(src + (size_t)p * partial_stride, a);
#pragma unroll
            for (int e = 0; e < 4; ++e) x[g][c][e] += a[e];
          }
          if (bias) {
#pragma unroll
            for (int e = 0; e < 4; ++e) x[g][c][e] += bias[piece * 4 + e];
          }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) sums[g] = fmaf(x[g][c][e], x[g][c][e], sums[g]);
      }
    }
    if (delta_weight) {              // the pending output passes a norm of its own
      block_sums<CN_GROUP>(sums, scratch);
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const int piece = threadIdx.x + c * blockDim.x;
        float dw[4] = {0.f, 0.f, 0.f, 0.f};
        if (piece < pieces) cn_load4<float>(delta_weight + piece * 4, dw);
#pragma unroll
        for (int g = 0; g < CN_GROUP; ++g) {
          const float inv = 1.0f / sqrtf(sums[g] / (float)hidden + delta_eps);
#pragma unroll
          for (int e = 0; e < 4; ++e) x[g][c][e] = (x[g][c][e] * inv) * dw[e];
        }
      }
    }
#pragma unroll
    for (int g = 0; g < CN_GROUP; ++g) {
      sums[g] = 0.f;
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const int piece = threadIdx.x + c * blockDim.x;
        if (base + g < end && piece < pieces) {
          float r[4];
          cn_load4<float>(residual + (size_t)(base + g) * hidden + piece * 4, r);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            x[g][c][e] += r[e];
            sums[g] = fmaf(x[g][c][e], x[g][c][e], sums[g]);
          }
        }
      }
    }
    block_sums<CN_GROUP>(sums, scratch);
#pragma unroll
    for (int g = 0; g < CN_GROUP; ++g) {
      const int row = base + g;
      if (row < end) {
        int seg = segment_of_token[row];
        if (seg < 0) {
          held = -1;
        } else {
          seg = LSE_CHECKED(seg, 0, num_segments, 0, LSE_CHECK_SEGMENT);
          float* window = BACK > 0 ? state + (size_t)LSE_CHECKED(segment_slot[seg], 0, num_slots, 0, LSE_CHECK_ROW) * BACK * hidden : nullptr;
          if (BACK > 0 && seg != held) {
            if (row == segment_start[seg]) {    // else the block's first, predecessor, rows fill it
#pragma unroll
              for (int i = 0; i < BACK; ++i)
#pragma unroll
                for (int c = 0; c < C; ++c) {
                  const int piece = threadIdx.x + c * blockDim.x;
                  if (piece < pieces) cn_load4<float>(window + (size_t)i * hidden + piece * 4, before[i][c]);
                }
            }
            held = seg;
          }
          const float inv = 1.0f / sqrtf(sums[g] / (float)hidden + eps);
#pragma unroll
          for (int c = 0; c < C; ++c) {
            const int piece = threadIdx.x + c * blockDim.x;
            float h[4], y[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              h[e] = (x[g][c][e] * inv) * nw[c][e];
              float sum = 0.f;
#pragma unroll
              for (int j = 0; j < BACK; ++j) sum = fmaf(cw[j][c][e], before[j][c][e], sum);
              y[e] = h[e] + fmaf(cw[TAPS - 1][c][e], h[e], sum);
            }
            if (BACK > 0) {
#pragma unroll
              for (int i = 0; i + 1 < BACK; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) before[i][c][e] = before[i + 1][c][e];
#pragma unroll
              for (int e = 0; e < 4; ++e) before[HELD - 1][c][e] = h[e];
            }
            if (row >= first && piece < pieces) {
              cn_store4<float>(residual_out + (size_t)row * hidden + piece * 4, x[g][c]);
              cn_store4<TO>(out + (size_t)row * hidden + piece * 4, y);
              if (BACK > 0 && move_windows) {
#pragma unroll
                for (int i = 0; i < BACK; ++i) cn_store4<float>(window + (size_t)i * hidden + piece * 4, before[i][c]);
              }
            }
          }
        }
      }
    }
  }
}

// The windows after a step: entry i holds h at the request's row count - (taps - 1) + i of this step, or moves up from
// behind (in ascending order an entry only reads entries behind it).  A block per request; x: residual_out.
__global__ void __launch_bounds__(256)
conv_norm_state_kernel(const float* __restrict__ x, const float* __restrict__ weight, float eps, float* __restrict__ state,
                       const int* __restrict__ segment_start, const int* __restrict__ segment_slot, int hidden, int taps,
                       int num_slots) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int seg = blockIdx.x;
  const int row0 = segment_start[seg], count = segment_start[seg + 1] - row0;
  if (count <= 0) return;
  float* window = state + (size_t)LSE_CHECKED(segment_slot[seg], 0, num_slots, 0, LSE_CHECK_ROW) * (taps - 1) * hidden;
  for (int i = 0; i < taps - 1; ++i) {
    const int l = count - (taps - 1) + i;
    if (l < 0) {
      for (int c = threadIdx.x; c < hidden; c += blockDim.x)
        window[(size_t)i * hidden + c] = window[(size_t)(i + count) * hidden + c];
      continue;
    }
    const float* row = x + (size_t)(row0 + l) * hidden;
    float sq = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) sq = fmaf(row[c], row[c], sq);
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)hidden + eps);
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) window[(size_t)i * hidden + c] = (row[c] * inv) * weight[c];
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

template <typename TD, typename TO, int TAPS>
int launch_conv_norm(const float* residual, float* residual_out, const void* delta, int n_partials, long long partial_stride,
                     const float* bias, const float* delta_weight, float delta_eps, const float* weight, float eps,
                     const float* conv_weight, float* state, const int* segment_of_token, const int* segment_start,
                     const int* segment_slot, void* out, int tokens, int rows_per_block, int hidden, int move_windows,
                     int num_slots, int num_segments, cudaStream_t stream) {
  const dim3 grid((tokens + rows_per_block - 1) / rows_per_block);
  const int pieces = hidden / 4;
  const bool one = pieces <= 256;
  const int threads = ((one ? pieces : (pieces + 1) / 2) + 31) / 32 * 32;
#define LSE_CN_ARGS residual, residual_out, (const TD*)delta, n_partials, partial_stride, bias, delta_weight, delta_eps, \
  weight, eps, conv_weight, state, segment_of_token, segment_start, segment_slot, (TO*)out, tokens, rows_per_block,      \
  hidden, move_windows, num_slots, num_segments
  if (one) lse_launch(conv_norm_kernel<TD, TO, TAPS, 1>, grid, threads, 0, stream, LSE_CN_ARGS);
  else lse_launch(conv_norm_kernel<TD, TO, TAPS, 2>, grid, threads, 0, stream, LSE_CN_ARGS);
#undef LSE_CN_ARGS
  return (int)cudaGetLastError();
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
  return hidden > 0 && hidden % 4 == 0 && hidden <= 4096 && taps >= 1 && taps <= 4;
}

// residual, residual_out float32 [tokens, hidden] (different tensors); delta [tokens, hidden] or a float32 stack, or null;
// bias float32 [hidden] or null (belongs to delta); delta_weight float32 [hidden] or null; conv_weight float32 [hidden, taps];
// state float32 [slots, taps - 1, hidden]; move_windows: every request brings one token and its window moves on here.
extern "C" int lse_conv_norm(const float* residual, float* residual_out, const void* delta, int delta_dtype, int n_partials,
                             long long partial_stride, const float* bias, const float* delta_weight, float delta_eps,
                             const float* weight, float eps, const float* conv_weight, float* state,
                             const int* segment_of_token, const int* segment_start, const int* segment_slot, void* out,
                             int out_dtype, int tokens, int rows_per_block, int hidden, int taps, int move_windows,
                             int num_slots, int num_segments, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (!lse_conv_norm_supported(hidden, taps) || rows_per_block <= 0 || n_partials < 1 || partial_stride % 4 ||
      residual == residual_out || (move_windows && rows_per_block != 1))
    return LSE_ERR_BAD_ARGUMENT;
#define LSE_CN_TAPS(TD, TO, TAPS)                                                                                      \
  return launch_conv_norm<TD, TO, TAPS>(residual, residual_out, delta, n_partials, partial_stride, bias, delta_weight, \
                                        delta_eps, weight, eps, conv_weight, state, segment_of_token, segment_start,   \
                                        segment_slot, out, tokens, rows_per_block, hidden, move_windows, num_slots,    \
                                        num_segments, stream);
#define LSE_CN_CASE(TD, TO)                        \
  switch (taps) {                                  \
    case 1: LSE_CN_TAPS(TD, TO, 1)                 \
    case 2: LSE_CN_TAPS(TD, TO, 2)                 \
    case 3: LSE_CN_TAPS(TD, TO, 3)                 \
    default: LSE_CN_TAPS(TD, TO, 4)                \
  }
  if (out_dtype == LSE_DTYPE_F32 && delta_dtype != LSE_DTYPE_F32) return LSE_ERR_BAD_ARGUMENT;
  if (delta_dtype == LSE_DTYPE_F32 && out_dtype == LSE_DTYPE_F32) { LSE_CN_CASE(float, float) }
  if (delta_dtype == LSE_DTYPE_BF16 && out_dtype == LSE_DTYPE_BF16) { LSE_CN_CASE(__nv_bfloat16, __nv_bfloat16) }
  if (delta_dtype == LSE_DTYPE_F32 && out_dtype == LSE_DTYPE_BF16) { LSE_CN_CASE(float, __nv_bfloat16) }
  return LSE_ERR_BAD_ARGUMENT;
#undef LSE_CN_CASE
#undef LSE_CN_TAPS
}

extern "C" int lse_conv_norm_state(const float* x, const float* weight, float eps, float* state, const int* segment_start,
                                   const int* segment_slot, int max_segments, int hidden, int taps, int num_slots,
                                   cudaStream_t stream) {
  if (max_segments <= 0 || taps <= 1) return 0;
  if (hidden <= 0) return LSE_ERR_BAD_ARGUMENT;
  lse_launch(conv_norm_state_kernel, max_segments, 256, 0, stream, x, weight, eps, state, segment_start, segment_slot,
             hidden, taps, num_slots);
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
