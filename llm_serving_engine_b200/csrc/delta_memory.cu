// A matrix memory that decays per key channel and writes differences (the gated delta rule with a decay vector).  Per head,
// with unit vectors q (times a constant) and k of the head's group, v, a write strength beta and a keep factor per key
// channel, all float32:
//     S <- diag(keep_t) S;     u = beta_t (v_t - S^T k_t);     S <- S + k_t u^T;     o_t = S^T q_t        (S is [dim][vdim])
//
//   lse_delta_prepare: what stands between the stacked input projection and the recurrence.  q, k and v pass a short causal
//       convolution per channel and SiLU; each head of q and k becomes a unit vector (x / sqrt(sum x^2 + 1e-6)), q times
//       q_scale; beta = sigmoid of its column; the low-rank columns (inputs of the decays' and the gate's second product)
//       are rounded into the compute dtype.
//   lse_delta_scan:    the recurrence row by row over every request's rows, from and into its state slot (few rows, single
//       decoded tokens; delta_memory_chunks.cu has the form for many rows of a request); the keep
//       factors exp(-exp(a_log) softplus(z + dt_bias)) are worked out from the decays' product while a tile is staged.
#include "common.cuh"

LSE_CHECK_DEFINE(lse_check_delta_memory)

namespace {
constexpr int DM_SLOTS = 8;        // most values of a head (or of a piece of v) that a lane holds: up to 256 columns a warp
constexpr int DM_PIECE = 128;      // columns of v, and of the columns behind it, that one warp takes

template <typename T> __device__ __forceinline__ void dm_load4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void dm_load4<float>(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <> __device__ __forceinline__ void dm_load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}

// Column of a lane's slot: four neighbouring columns a lane when VEC (every operand aligned for it), else strided.
template <bool VEC> __device__ __forceinline__ int dm_column(int lane, int slot) {
  return VEC ? (lane + 32 * (slot / 4)) * 4 + slot % 4 : lane + 32 * slot;
}
template <typename TD, bool VEC, int NS>
__device__ __forceinline__ void dm_fetch(const TD* p, int n_partials, long long partial_stride, int lane, int width,
                                         float (&v)[NS]) {
#pragma unroll
  for (int s = 0; s < NS; ++s) v[s] = 0.f;
  if (VEC) {
#pragma unroll
    for (int k = 0; k < NS / 4; ++k) {
      const int c = (lane + 32 * k) * 4;
      if (c < width) {
        int q = 0;
        for (; q + 4 <= n_partials; q += 4) {
          float a[4][4];
#pragma unroll
          for (int i = 0; i < 4; ++i) dm_load4<TD>(p + (size_t)(q + i) * partial_stride + c, a[i]);
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) v[4 * k + e] += a[i][e];
        }
        for (; q < n_partials; ++q) {
          float a[4];
          dm_load4<TD>(p + (size_t)q * partial_stride + c, a);
#pragma unroll
          for (int e = 0; e < 4; ++e) v[4 * k + e] += a[e];
        }
      }
    }
  } else {
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      const int c = lane + 32 * s;
      if (c < width) v[s] = sum_partials<TD>(p + c, n_partials, partial_stride);
    }
  }
}
template <bool VEC, int NS>
__device__ __forceinline__ void dm_put(float* p, int lane, int width, const float (&v)[NS]) {
  if (VEC) {
#pragma unroll
    for (int k = 0; k < NS / 4; ++k) {
      const int c = (lane + 32 * k) * 4;
      if (c < width) *reinterpret_cast<float4*>(p + c) = make_float4(v[4 * k], v[4 * k + 1], v[4 * k + 2], v[4 * k + 3]);
    }
  } else {
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      const int c = lane + 32 * s;
      if (c < width) p[c] = v[s];
    }
  }
}

// Columns of proj: [q (groups * dim) | k (groups * dim) | v (heads * vdim) | beta (heads) | low (rank)].  A warp owns an item (a
// head of q, a head of k, a piece of v, a piece of the columns behind it) of rows_per_warp rows and walks them with the
// channels' last taps - 1 inputs in registers, DM_AHEAD rows fetched at a time (TAPS known; TAPS = 0: any number, fetched
// again for every row).  NS: values a lane holds (4 for items of up to 128 columns, 8 up to 256).
constexpr int DM_AHEAD = 4;
template <typename TD, typename TO, int TAPS, bool VEC, int NS>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const TD* __restrict__ proj, int n_partials, long long partial_stride, long long ld,
                     const float* __restrict__ conv_weight, float* __restrict__ state,
                     const int* __restrict__ segment_of_token, const int* __restrict__ segment_start,
                     const int* __restrict__ segment_slot, float* __restrict__ q_out, float* __restrict__ k_out,
                     float* __restrict__ v_out, float* __restrict__ beta_out, TO* __restrict__ low_out, int low_ld,
                     int tokens, int rows_per_warp, int groups, int heads, int dim, int vdim, int rank, int taps_rt,
                     float q_scale, int move_windows, int num_slots, int num_segments, int items) {
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const long long unit = (blockIdx.x * (long long)blockDim.x + threadIdx.x) >> 5;
  const int first = (int)(unit / items) * rows_per_warp, item = (int)(unit % items);
  if (first >= tokens) return;
  const int end = min(tokens, first + rows_per_warp);
  const int qk = groups * dim, value = heads * vdim, channels = 2 * qk + value;
  const int v_pieces = (value + DM_PIECE - 1) / DM_PIECE;
  if (item >= 2 * groups + v_pieces) {       // the columns behind v
    pdl_wait();
    const int lo = (item - 2 * groups - v_pieces) * DM_PIECE, hi = min(lo + DM_PIECE, heads + low_ld);
    for (int r = first; r < end; ++r) {
      if (segment_of_token[r] < 0) continue;
#pragma unroll
      for (int i = 0; i < DM_PIECE / 32; ++i) {
        const int c = lo + lane + 32 * i;
        if (c < hi) {
          const bool real = c < heads + rank;
          const float z = real ? sum_partials<TD>(proj + (size_t)r * ld + channels + c, n_partials, partial_stride) : 0.f;
          if (c < heads) beta_out[(size_t)r * heads + c] = 1.f / (1.f + expf(-z));
          else low_out[(size_t)r * low_ld + c - heads] = from_f32<TO>(z);
        }
      }
    }
    return;
  }
  int column, width, kind;                   // kind 0: q, 1: k, 2: v
  float* dst;
  size_t dst_ld;
  if (item < 2 * groups) {
    kind = item < groups ? 0 : 1;
    const int g = kind == 0 ? item : item - groups;
    column = item * dim; width = dim;
    dst = (kind == 0 ? q_out : k_out) + g * dim; dst_ld = qk;
  } else {
    kind = 2;
    const int lo = (item - 2 * groups) * DM_PIECE;
    column = 2 * qk + lo; width = min(DM_PIECE, value - lo);
    dst = v_out + lo; dst_ld = value;
  }
  constexpr int BACK = TAPS > 0 ? TAPS - 1 : 0, HELD = BACK > 0 ? BACK : 1;
  const int back_rt = TAPS > 0 ? BACK : taps_rt - 1;
  float w[TAPS > 0 ? TAPS : 1][NS];
  if (TAPS > 0) {                            // the weights do not depend on earlier kernels
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      const int c = dm_column<VEC>(lane, s);
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[j][s] = c < width ? conv_weight[(size_t)(column + c) * TAPS + j] : 0.f;
    }
  }
  pdl_wait();
  float before[HELD][NS];                    // before[i]: the input BACK - i rows back
  int held = -1;
  for (int base = first; base < end; base += DM_AHEAD) {
    float ahead[DM_AHEAD][NS];
    int segs[DM_AHEAD];
#pragma unroll
    for (int g = 0; g < DM_AHEAD; ++g) {
      segs[g] = -1;
      if (base + g < end) {
        segs[g] = segment_of_token[base + g];
        dm_fetch<TD, VEC, NS>(proj + (size_t)(base + g) * ld + column, n_partials, partial_stride, lane, width, ahead[g]);
      }
    }
#pragma unroll
    for (int g = 0; g < DM_AHEAD; ++g) {
      const int r = base + g;
      if (r >= end) break;
      int seg = segs[g];
      if (seg < 0) { held = -1; continue; }
      seg = LSE_CHECKED(seg, 0, num_segments, 0, LSE_CHECK_SEGMENT);
      float* window = back_rt > 0 ? state + (size_t)LSE_CHECKED(segment_slot[seg], 0, num_slots, 0, LSE_CHECK_ROW) * back_rt * channels + column : nullptr;
      float y[NS];
      if (TAPS > 0) {
        if (BACK > 0 && seg != held) {
          const int l = r - segment_start[seg];
#pragma unroll
          for (int i = 0; i < BACK; ++i) {
            const int back = BACK - i;
            if (l - back >= 0) dm_fetch<TD, VEC, NS>(proj + (size_t)(r - back) * ld + column, n_partials, partial_stride, lane, width, before[i]);
            else dm_fetch<float, VEC, NS>(window + (size_t)(BACK + l - back) * channels, 1, 0, lane, width, before[i]);
          }
          held = seg;
        }
#pragma unroll
        for (int s = 0; s < NS; ++s) {
          float sum = 0.f;
#pragma unroll
          for (int j = 0; j < BACK; ++j) sum = fmaf(w[j][s], before[j][s], sum);
          y[s] = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][s], ahead[g][s], sum);
        }
        if (BACK > 0) {
#pragma unroll
          for (int i = 0; i + 1 < BACK; ++i)
#pragma unroll
            for (int s = 0; s < NS; ++s) before[i][s] = before[i + 1][s];
#pragma unroll
          for (int s = 0; s < NS; ++s) before[HELD - 1][s] = ahead[g][s];
          if (move_windows)
#pragma unroll
            for (int i = 0; i < BACK; ++i) dm_put<VEC, NS>(window + (size_t)i * channels, lane, width, before[i]);
        }
      } else {
        const int l = r - segment_start[seg];
#pragma unroll
        for (int s = 0; s < NS; ++s) {
          const int c = dm_column<VEC>(lane, s);
          float sum = 0.f;
          if (c < width)
            for (int j = 0; j < taps_rt; ++j) {
              const int back = taps_rt - 1 - j;
              const float u = back == 0 ? ahead[g][s]
                  : l - back >= 0 ? sum_partials<TD>(proj + (size_t)(r - back) * ld + column + c, n_partials, partial_stride)
                                  : window[(size_t)(taps_rt - 1 + l - back) * channels + c];
              sum = fmaf(conv_weight[(size_t)(column + c) * taps_rt + j], u, sum);
            }
          y[s] = sum;
          if (move_windows && c < width) {
            for (int i = 0; i + 1 < back_rt; ++i) window[(size_t)i * channels + c] = window[(size_t)(i + 1) * channels + c];
            if (back_rt > 0) window[(size_t)(back_rt - 1) * channels + c] = ahead[g][s];
          }
        }
      }
      float sq = 0.f;
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        y[s] = y[s] / (1.f + expf(-y[s]));
        if (dm_column<VEC>(lane, s) >= width) y[s] = 0.f;
        sq = fmaf(y[s], y[s], sq);
      }
      if (kind < 2) {
        const float inv = (kind == 0 ? q_scale : 1.f) / sqrtf(warp_sum(sq) + 1e-6f);
#pragma unroll
        for (int s = 0; s < NS; ++s) y[s] *= inv;
      }
      dm_put<VEC, NS>(dst + (size_t)r * dst_ld, lane, width, y);
    }
  }
}

__device__ __forceinline__ float dm_keep(float z, float rate) {     // exp(-rate softplus(z))
  return expf(-rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
}

constexpr int DS_THREADS = 128;
constexpr int DS_ROWS = 32;        // rows of the state that a thread keeps

// A block owns (request, head, a tile of state columns); PARTS threads share a column (PARTS * 32 >= dim), a thread keeps
// 32 rows of it in registers.  Requests of more than max_rows rows (max_rows > 0) are left to the chunked form.
template <int PARTS>
__global__ void __launch_bounds__(DS_THREADS)
delta_scan_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v,
                  const float* __restrict__ beta, const float* __restrict__ z, int z_partials, long long z_stride,
                  long long z_ld, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                  float* __restrict__ state, const int* __restrict__ segment_start, const int* __restrict__ segment_slot,
                  float* __restrict__ out, int heads, int groups, int dim, int vdim, int num_slots, int max_rows) {
  constexpr int CW = 32 / PARTS, CB = 4 * CW;
  constexpr int PADDED = DS_ROWS + 4;                 // a part's rows, 16-byte aligned and four banks apart from the next part's
  constexpr int TS = PARTS * PADDED;
  constexpr int TT = PARTS <= 2 ? 16 : (PARTS == 4 ? 8 : 4);      // tokens staged at a time
  constexpr int LOADS = TT * PARTS * DS_ROWS / DS_THREADS;
  constexpr int V_LOADS = (TT * CB + DS_THREADS - 1) / DS_THREADS;
  __shared__ __align__(16) float q_s[TT * TS], k_s[TT * TS], g_s[TT * TS];
  __shared__ float v_s[TT * CB], beta_s[TT];
  const int seg = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * CB;
  const int group = h / (heads / groups);
  const float rate = expf(a_log[h]);
  pdl_launch_dependents();
  pdl_wait();
  const int row0 = segment_start[seg], row1 = segment_start[seg + 1];
  if (row1 <= row0 || (max_rows > 0 && row1 - row0 > max_rows)) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int part = lane / CW, cb = warp * CW + lane % CW, col = col0 + cb;
  float* st = state + ((size_t)LSE_CHECKED(segment_slot[seg], 0, num_slots, 0, LSE_CHECK_ROW) * heads + h) * dim * vdim;
  float s[DS_ROWS];
#pragma unroll
  for (int i = 0; i < DS_ROWS; ++i) {
    const int d = part * DS_ROWS + i;
    s[i] = d < dim && col < vdim ? st[(size_t)d * vdim + col] : 0.f;
  }
  float qv[LOADS], kv[LOADS], gv[LOADS], vv[V_LOADS], bv = 0.f;
  auto fetch = [&](int base) {         // a tile's rows into registers, all loads in flight together
    const int n = min(TT, row1 - base);
#pragma unroll
    for (int i = 0; i < LOADS; ++i) {
      const int e = threadIdx.x + i * DS_THREADS;
      const int t = e / (PARTS * DS_ROWS), d = e % (PARTS * DS_ROWS);
      qv[i] = kv[i] = gv[i] = 0.f;
      if (t < n && d < dim) {
        const size_t row = base + t;
        qv[i] = q[(row * groups + group) * dim + d];
        kv[i] = k[(row * groups + group) * dim + d];
        gv[i] = sum_partials<float>(z + row * z_ld + h * dim + d, z_partials, z_stride) + dt_bias[h * dim + d];
      }
    }
#pragma unroll
    for (int i = 0; i < V_LOADS; ++i) {
      const int e = threadIdx.x + i * DS_THREADS;
      const int t = e / CB, c = e % CB;
      vv[i] = e < TT * CB && t < n && col0 + c < vdim ? v[((size_t)(base + t) * heads + h) * vdim + col0 + c] : 0.f;
    }
    if (threadIdx.x < TT) bv = (int)threadIdx.x < n ? beta[(size_t)(base + threadIdx.x) * heads + h] : 0.f;
  };
  fetch(row0);
  for (int base = row0; base < row1; base += TT) {
    const int n = min(TT, row1 - base);
    __syncthreads();                   // the tile before has been used
#pragma unroll
    for (int i = 0; i < LOADS; ++i) {
      const int e = threadIdx.x + i * DS_THREADS;
      const int t = e / (PARTS * DS_ROWS), d = e % (PARTS * DS_ROWS);
      const int at = t * TS + (d / DS_ROWS) * PADDED + d % DS_ROWS;
      q_s[at] = qv[i];
      k_s[at] = kv[i];
      g_s[at] = dm_keep(gv[i], rate);
    }
#pragma unroll
    for (int i = 0; i < V_LOADS; ++i) {
      const int e = threadIdx.x + i * DS_THREADS;
      if (e < TT * CB) v_s[e] = vv[i];
    }
    if (threadIdx.x < TT) beta_s[threadIdx.x] = bv;
    __syncthreads();
    if (base + TT < row1) fetch(base + TT);
    for (int t = 0; t < n; ++t) {
      const float4* qr = reinterpret_cast<const float4*>(q_s + t * TS + part * PADDED);
      const float4* kr = reinterpret_cast<const float4*>(k_s + t * TS + part * PADDED);
      const float4* gr = reinterpret_cast<const float4*>(g_s + t * TS + part * PADDED);
      float dot[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < DS_ROWS / 4; ++i) {
        const float4 g = gr[i], kk = kr[i];
        s[4 * i + 0] *= g.x; s[4 * i + 1] *= g.y; s[4 * i + 2] *= g.z; s[4 * i + 3] *= g.w;
        dot[0] = fmaf(s[4 * i + 0], kk.x, dot[0]); dot[1] = fmaf(s[4 * i + 1], kk.y, dot[1]);
        dot[2] = fmaf(s[4 * i + 2], kk.z, dot[2]); dot[3] = fmaf(s[4 * i + 3], kk.w, dot[3]);
      }
      float held = (dot[0] + dot[1]) + (dot[2] + dot[3]);
#pragma unroll
      for (int off = CW; off < 32; off <<= 1) held += __shfl_xor_sync(0xffffffffu, held, off);
      const float u = beta_s[t] * (v_s[t * CB + cb] - held);
      float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < DS_ROWS / 4; ++i) {
        const float4 kk = kr[i], qq = qr[i];
        s[4 * i + 0] = fmaf(kk.x, u, s[4 * i + 0]); s[4 * i + 1] = fmaf(kk.y, u, s[4 * i + 1]);
        s[4 * i + 2] = fmaf(kk.z, u, s[4 * i + 2]); s[4 * i + 3] = fmaf(kk.w, u, s[4 * i + 3]);
        o[0] = fmaf(s[4 * i + 0], qq.x, o[0]); o[1] = fmaf(s[4 * i + 1], qq.y, o[1]);
        o[2] = fmaf(s[4 * i + 2], qq.z, o[2]); o[3] = fmaf(s[4 * i + 3], qq.w, o[3]);
      }
      float total = (o[0] + o[1]) + (o[2] + o[3]);
#pragma unroll
      for (int off = CW; off < 32; off <<= 1) total += __shfl_xor_sync(0xffffffffu, total, off);
      if (part == 0 && col < vdim) out[((size_t)(base + t) * heads + h) * vdim + col] = total;
    }
  }
#pragma unroll
  for (int i = 0; i < DS_ROWS; ++i) {
    const int d = part * DS_ROWS + i;
    if (d < dim && col < vdim) st[(size_t)d * vdim + col] = s[i];
  }
}
}  // namespace

// proj rows as above (float32 / bfloat16 / a float32 stack); conv_weight float32 [channels, taps]; state float32 [slots,
// taps - 1, channels]; q_out, k_out float32 [tokens, groups * dim], v_out [tokens, heads * vdim], beta_out [tokens, heads];
// low_out [tokens, low_ld] in the compute dtype, zero from column rank on; move_windows: every request brings one token
// and its window moves on here.
extern "C" int lse_delta_prepare(const void* proj, int proj_dtype, int n_partials, long long partial_stride, long long ld,
                                 const float* conv_weight, float* state, const int* segment_of_token,
                                 const int* segment_start, const int* segment_slot, float* q_out, float* k_out, float* v_out,
                                 float* beta_out, void* low_out, int low_dtype, int low_ld, int tokens, int groups, int heads,
                                 int dim, int vdim, int rank, int taps, float q_scale, int move_windows, int num_slots,
                                 int num_segments, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (groups <= 0 || heads <= 0 || heads % groups || dim <= 0 || dim > 32 * DM_SLOTS || vdim <= 0 || rank < 0 ||
      low_ld < rank || taps < 1 || n_partials < 1)
    return LSE_ERR_BAD_ARGUMENT;
  const int rows_per_warp = tokens >= 1024 && !move_windows ? 8 : 1;
  const int value = heads * vdim;
  const int items = 2 * groups + (value + DM_PIECE - 1) / DM_PIECE + (heads + low_ld + DM_PIECE - 1) / DM_PIECE;
  const long long warps = (long long)((tokens + rows_per_warp - 1) / rows_per_warp) * items;
  const long long blocks = (warps + 3) / 4;
  if (blocks > 0x7fffffffLL) return LSE_ERR_TOO_LARGE;
  const bool vec = dim % 4 == 0 && value % 4 == 0 && ld % 4 == 0 && partial_stride % 4 == 0 && (((uintptr_t)proj) & 15) == 0;
#define LSE_DM_NS(TD, TO, TAPS, VEC, NS)                                                                               \
  lse_launch(delta_prepare_kernel<TD, TO, TAPS, VEC, NS>, (unsigned)blocks, 128, 0, stream, (const TD*)proj, n_partials,    \
             partial_stride, ld, conv_weight, state, segment_of_token, segment_start, segment_slot, q_out, k_out, v_out, \
             beta_out, (TO*)low_out, low_ld, tokens, rows_per_warp, groups, heads, dim, vdim, rank, taps, q_scale,      \
             move_windows, num_slots, num_segments, items)
#define LSE_DM_GO(TD, TO, TAPS, VEC)                          \
  do {                                                        \
    if (dim <= 128) LSE_DM_NS(TD, TO, TAPS, VEC, 4);          \
    else LSE_DM_NS(TD, TO, TAPS, VEC, 8);                     \
  } while (0)
#define LSE_DM_TAPS(TD, TO, VEC)                              \
  do {                                                        \
    if (taps == 4) LSE_DM_GO(TD, TO, 4, VEC);                 \
    else if (taps == 3) LSE_DM_GO(TD, TO, 3, VEC);            \
    else LSE_DM_GO(TD, TO, 0, VEC);                           \
  } while (0)
#define LSE_DM_CASE(TD, TO)                   \
  do {                                        \
    if (vec) LSE_DM_TAPS(TD, TO, true);       \
    else LSE_DM_GO(TD, TO, 0, false);         \
  } while (0)
  if (proj_dtype == LSE_DTYPE_F32 && low_dtype == LSE_DTYPE_F32) LSE_DM_CASE(float, float);
  else if (proj_dtype == LSE_DTYPE_F32 && low_dtype == LSE_DTYPE_BF16) LSE_DM_CASE(float, __nv_bfloat16);
  else if (proj_dtype == LSE_DTYPE_BF16 && low_dtype == LSE_DTYPE_BF16) LSE_DM_CASE(__nv_bfloat16, __nv_bfloat16);
  else return LSE_ERR_BAD_ARGUMENT;
#undef LSE_DM_CASE
#undef LSE_DM_TAPS
#undef LSE_DM_GO
#undef LSE_DM_NS
  LSE_LAUNCH_CHECK();
}

// q, k float32 [tokens, groups, dim]; v float32 [tokens, heads, vdim]; beta float32 [tokens, heads]; z: the decays' product,
// float32 rows of z_ld values (or a stack of partial sums), head h's channels from column h * dim; dt_bias float32
// [heads * dim], a_log float32 [heads]; state float32 [slots, heads, dim, vdim]; out float32 [tokens, heads, vdim].
extern "C" int lse_delta_scan(const float* q, const float* k, const float* v, const float* beta, const float* z,
                              int z_partials, long long z_stride, long long z_ld, const float* dt_bias, const float* a_log,
                              float* state, const int* segment_start, const int* segment_slot, float* out,
                              int max_segments, int heads, int groups, int dim, int vdim, int num_slots, int max_rows,
                              cudaStream_t stream) {
  if (max_segments <= 0) return 0;
  if (heads <= 0 || groups <= 0 || heads % groups || heads > 65535 || dim <= 0 || dim > 8 * DS_ROWS || vdim <= 0 || z_partials < 1)
    return LSE_ERR_BAD_ARGUMENT;
#define LSE_DS_CASE(P)                                                                                                \
  lse_launch(delta_scan_kernel<P>, dim3(max_segments, heads, (vdim + 4 * (32 / P) - 1) / (4 * (32 / P))), DS_THREADS, 0, \
             stream, q, k, v, beta, z, z_partials, z_stride, z_ld, dt_bias, a_log, state, segment_start, segment_slot, out, \
             heads, groups, dim, vdim, num_slots, max_rows)
  if (dim <= DS_ROWS) LSE_DS_CASE(1);
  else if (dim <= 2 * DS_ROWS) LSE_DS_CASE(2);
  else if (dim <= 4 * DS_ROWS) LSE_DS_CASE(4);
  else LSE_DS_CASE(8);
#undef LSE_DS_CASE
  LSE_LAUNCH_CHECK();
}
