// The delta memory's recurrence (delta_memory.cu) for requests with many rows in a step: chunks of 16 rows, so that what one
// row hands to the next inside a chunk is worked out for all chunks side by side and only the state walks from chunk to
// chunk.  With P_t the product of the keep vectors of the chunk's rows up to t, and per row
//     u_t = beta_t (v_t - S_(t-1)^T (keep_t * k_t)),        S_(t-1) the state after row t - 1,
// a chunk that starts from the state S gives
//     u = Y - W S,        (I + A) [W | Y] = [diag(beta) (P * K) | diag(beta) V],
//     o = (P * Q) S + B u,        S' = diag(P_last) S + (E * K)^T u,
//     A[t, s] = beta_t sum_c k_t k_s (keep products of rows s + 1 .. t)_c   for s < t,
//     B[t, s] =        sum_c q_t k_s (the same)_c                            for s <= t,
//     E_t = keep products of rows t + 1 .. last.
// Products of keep factors are formed as products, never as quotients or differences of logarithms, so a factor that
// vanishes does no harm.  Everything is float32.
//
//   delta_chunk_prepare_kernel: a block per chunk and head works out W, P * Q (both stored by channel: [channel][32], rows of W
//       and then of P * Q), E * K, P_last, Y and B.
//   delta_chunk_scan_kernel:    a block per request, head and 16 columns of the state walks the request's chunks with the
//       state in shared memory; the next chunk's tiles travel (cp.async) while one is worked on.
// Rows beyond a request's last are rows with k = q = v = 0, beta = 0, keep = 1, which change nothing.
#include "common.cuh"

LSE_CHECK_DEFINE(lse_check_delta_memory_chunks)

namespace {
constexpr int DC = 16;             // rows of a chunk
constexpr int DCN = 16;            // columns of the state that a block of the scan owns
constexpr int DCS = 20;            // floats between the state's rows in shared memory: rows four apart lie half the banks apart

__device__ __forceinline__ float dc_keep(float z, float rate) {     // exp(-rate softplus(z))
  return expf(-rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
}
__device__ __forceinline__ int dc_chunks(int count, int min_rows) { return count > min_rows ? (count + DC - 1) / DC : 0; }

// floats of a chunk and head in the buffers
__host__ __device__ __forceinline__ long long dc_wq(int dp) { return (long long)dp * 2 * DC; }
__host__ __device__ __forceinline__ long long dc_k(int dp) { return (long long)dp * DC; }
__host__ __device__ __forceinline__ long long dc_all(int dp, int ep) { return dc_wq(dp) + dc_k(dp) + dp + DC * DC + (long long)DC * ep; }

// NJ: 32 * NJ channels (the head's, padded with zeros).  Threads: eight lanes share a row s, each with every eighth group
// of four channels; four rows a warp, so four warps.
template <int NJ>
__global__ void __launch_bounds__(128, 4)
delta_chunk_prepare_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v,
                           const float* __restrict__ beta, const float* __restrict__ z, int z_partials, long long z_stride,
                           long long z_ld, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                           const int* __restrict__ segment_start, float* __restrict__ buffer, int num_segments, int heads,
                           int groups, int dim, int vdim, int ep, int min_rows) {
  constexpr int DP = 32 * NJ, LD = DP;
  extern __shared__ __align__(16) float dc_smem[];
  float* q_s = dc_smem;                  // [16][DP]
  float* k_s = q_s + DC * LD;
  float* g_s = k_s + DC * LD;
  __shared__ __align__(16) float a_s[DC * DC], b_s[DC * DC];
  __shared__ float beta_s[DC];
  __shared__ int item[2];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, tid = threadIdx.x;
  if (tid < 32) {                        // which rows chunk blockIdx.x is: 32 requests at a time
    int before = 0, row = -1, rows = 0;
    for (int base = 0; base < num_segments && row < 0; base += 32) {
      const int s = base + tid;
      const int first = s < num_segments ? segment_start[s] : 0, count = s < num_segments ? segment_start[s + 1] - first : 0;
      const int mine = dc_chunks(count, min_rows);
      int incl = mine;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, incl, o);
        if (tid >= o) incl += up;
      }
      const int at = (int)blockIdx.x - before - (incl - mine);
      const unsigned vote = __ballot_sync(0xffffffffu, at >= 0 && at < mine);
      if (vote) {
        const int src = __ffs(vote) - 1;
        row = __shfl_sync(0xffffffffu, first + at * DC, src);
        rows = __shfl_sync(0xffffffffu, min(DC, count - at * DC), src);
      }
      before += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (tid == 0) { item[0] = row; item[1] = rows; }
  }
  __syncthreads();
  const int row0 = item[0], n = item[1];
  if (row0 < 0) return;
  const int group = h / (heads / groups);
  const float rate = expf(a_log[h]);
  float* mine = buffer + ((size_t)blockIdx.x * heads + h) * dc_all(DP, ep);
  float* wq_out = mine;                  // [DP][32]
  float* k_out = wq_out + dc_wq(DP);     // [16][DP]
  float* last_out = k_out + dc_k(DP);    // [DP]
  float* b_out = last_out + DP;          // [16][16], B by columns
  float* y_out = b_out + DC * DC;        // [16][ep]
  constexpr int AHEAD = 4 * NJ < 8 ? 4 * NJ : 8;      // of the 4 * NJ values a thread stages, so many loads of each kind in flight
#pragma unroll 1
  for (int e0 = tid; e0 < DC * DP; e0 += 128 * AHEAD) {
    float qq[AHEAD], kk[AHEAD], zz[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int e = e0 + 128 * i, t = e / DP, c = e % DP;
      qq[i] = kk[i] = zz[i] = 0.f;
      if (t < n && c < dim) {
        const size_t row = row0 + t;
        qq[i] = q[(row * groups + group) * dim + c];
        kk[i] = k[(row * groups + group) * dim + c];
        const float* src = z + row * z_ld + h * dim + c;
        zz[i] = z_partials == 1 ? *src : sum_partials<float>(src, z_partials, z_stride);
      }
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int e = e0 + 128 * i, t = e / DP, c = e % DP;
      const bool real = t < n && c < dim;
      q_s[t * LD + c] = qq[i]; k_s[t * LD + c] = kk[i];
      g_s[t * LD + c] = real ? dc_keep(zz[i] + dt_bias[h * dim + c], rate) : 1.f;
    }
  }
  if (tid < DC) beta_s[tid] = tid < n ? beta[(size_t)(row0 + tid) * heads + h] : 0.f;
  __syncthreads();
  {                                      // A and B: row s against every row t >= s, its products carried along
    const int lane8 = tid & 7, s = tid >> 3;
    float c[NJ][4];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const float4 kk = *reinterpret_cast<const float4*>(k_s + s * LD + (lane8 + 8 * j) * 4);
      c[j][0] = kk.x; c[j][1] = kk.y; c[j][2] = kk.z; c[j][3] = kk.w;
    }
    const int first = (tid >> 5) * 4;    // the warp's first row: all its lanes take the same steps
    for (int t = first; t < DC; ++t) {
      float kk_sum = 0.f, qk_sum = 0.f;
      if (t >= s) {
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const int at = t * LD + (lane8 + 8 * j) * 4;
          if (t > s) {
            const float4 g = *reinterpret_cast<const float4*>(g_s + at);
            c[j][0] *= g.x; c[j][1] *= g.y; c[j][2] *= g.z; c[j][3] *= g.w;
          }
          const float4 kt = *reinterpret_cast<const float4*>(k_s + at), qt = *reinterpret_cast<const float4*>(q_s + at);
          kk_sum = fmaf(kt.x, c[j][0], kk_sum); kk_sum = fmaf(kt.y, c[j][1], kk_sum);
          kk_sum = fmaf(kt.z, c[j][2], kk_sum); kk_sum = fmaf(kt.w, c[j][3], kk_sum);
          qk_sum = fmaf(qt.x, c[j][0], qk_sum); qk_sum = fmaf(qt.y, c[j][1], qk_sum);
          qk_sum = fmaf(qt.z, c[j][2], qk_sum); qk_sum = fmaf(qt.w, c[j][3], qk_sum);
        }
      }
#pragma unroll
      for (int o = 1; o < 8; o <<= 1) {
        kk_sum += __shfl_xor_sync(0xffffffffu, kk_sum, o);
        qk_sum += __shfl_xor_sync(0xffffffffu, qk_sum, o);
      }
      if (lane8 == 0) {
        a_s[t * DC + s] = t > s ? beta_s[t] * kk_sum : 0.f;
        b_s[s * DC + t] = t >= s ? qk_sum : 0.f;      // stored by column
      }
    }
    for (int t = 0; t < first; ++t)      // rows before the warp's rows: nothing
      if (lane8 == 0) a_s[t * DC + s] = b_s[s * DC + t] = 0.f;
  }
  __syncthreads();
  for (int e = tid; e < DC * DC; e += 128) b_out[e] = b_s[e];
  for (int col = tid; col < DP + ep; col += 128) {      // a column of W or of Y: forward substitution
    float x[DC];
    if (col < DP) {
      float product = 1.f, pq[DC];
#pragma unroll
      for (int t = 0; t < DC; ++t) {
        product *= g_s[t * LD + col];
        x[t] = beta_s[t] * (product * k_s[t * LD + col]);
        pq[t] = product * q_s[t * LD + col];
      }
      last_out[col] = product;
#pragma unroll
      for (int t = 0; t < DC; t += 4)
        *reinterpret_cast<float4*>(wq_out + (size_t)col * 2 * DC + DC + t) = make_float4(pq[t], pq[t + 1], pq[t + 2], pq[t + 3]);
      float after = 1.f;
#pragma unroll
      for (int t = DC - 1; t >= 0; --t) {
        k_out[(size_t)t * DP + col] = after * k_s[t * LD + col];
        after *= g_s[t * LD + col];
      }
    } else {
      const int c = col - DP;
#pragma unroll
      for (int t = 0; t < DC; ++t)
        x[t] = t < n && c < vdim ? beta_s[t] * v[((size_t)(row0 + t) * heads + h) * vdim + c] : 0.f;
    }
#pragma unroll
    for (int t = 1; t < DC; ++t) {
      float sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int s = 0; s < t; ++s) sum[s & 3] = fmaf(a_s[t * DC + s], x[s], sum[s & 3]);
      x[t] -= (sum[0] + sum[1]) + (sum[2] + sum[3]);
    }
    if (col < DP) {
#pragma unroll
      for (int t = 0; t < DC; t += 4)
        *reinterpret_cast<float4*>(wq_out + (size_t)col * 2 * DC + t) = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
    } else {
#pragma unroll
      for (int t = 0; t < DC; ++t) y_out[(size_t)t * ep + col - DP] = x[t];
    }
  }
}

__device__ __forceinline__ void dc_copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// Shared memory: the state [DP][20] (16 used), two stages of {WQ [DP][32], EK [16][DP], P_last [DP], B^T [16][16], Y [16][16]}, the
// warps' sums [8][128] float4, u [16][16].
template <int NJ>
__global__ void __launch_bounds__(256)
delta_chunk_scan_kernel(const float* __restrict__ buffer, float* __restrict__ state, const int* __restrict__ segment_start,
                        const int* __restrict__ segment_slot, float* __restrict__ out, int heads, int dim, int vdim, int ep,
                        int num_slots, int min_rows) {
  constexpr int DP = 32 * NJ;
  constexpr int STAGE = DP * 2 * DC + DP * DC + DP + 2 * DC * DC;
  constexpr int KW = DP / 8;             // channels of a warp's share of the product with the state
  extern __shared__ __align__(16) float dc_smem[];
  float* s_s = dc_smem;
  float* stage_s = s_s + DP * DCS;
  float4* red_s = reinterpret_cast<float4*>(stage_s + 2 * STAGE);
  float* u_s = reinterpret_cast<float*>(red_s + 8 * 128);
  __shared__ int base_s;
  pdl_launch_dependents();
  pdl_wait();
  const int seg = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * DCN, tid = threadIdx.x;
  const int row0 = segment_start[seg], count = segment_start[seg + 1] - row0;
  const int chunks = dc_chunks(count, min_rows);
  if (chunks == 0) return;
  const int lane = tid & 31, warp = tid >> 5;
  if (warp == 0) {                       // chunks of the requests before this one
    int before = 0;
    for (int s = lane; s < seg; s += 32) before += dc_chunks(segment_start[s + 1] - segment_start[s], min_rows);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
    if (lane == 0) base_s = before;
  }
  float* st = state + ((size_t)LSE_CHECKED(segment_slot[seg], 0, num_slots, 0, LSE_CHECK_ROW) * heads + h) * dim * vdim;
  for (int e = tid; e < DP * DCN; e += 256) {
    const int d = e / DCN, c = e % DCN;
    s_s[d * DCS + c] = d < dim && col0 + c < vdim ? st[(size_t)d * vdim + col0 + c] : 0.f;
  }
  __syncthreads();
  const long long per = dc_all(DP, ep);
  const float* first = buffer + ((size_t)base_s * heads + h) * per;
  constexpr int HEAD = DP * 2 * DC + DP * DC + DP + DC * DC;      // floats in front of Y, stored one after the other
  auto load = [&](int chunk, int stage) {
    const float* src = first + (size_t)chunk * heads * per;
    float* dst = stage_s + stage * STAGE;
    for (int e = tid; e < HEAD / 4; e += 256) dc_copy16(dst + e * 4, src + e * 4);
    if (tid < DC * DCN / 4) dc_copy16(dst + HEAD + tid * 4, src + HEAD + (size_t)(tid / 4) * ep + col0 + (tid % 4) * 4);
    asm volatile("cp.async.commit_group;\n" ::);
  };
  load(0, 0);
  const int rg = lane >> 2, cg = lane & 3;       // four rows of [W | P * Q], four columns
  for (int chunk = 0; chunk < chunks; ++chunk) {
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();                             // the chunk's tiles are there, the state is the last chunk's, its other stage is free
    if (chunk + 1 < chunks) load(chunk + 1, (chunk + 1) & 1);
    const float* wq = stage_s + (chunk & 1) * STAGE;
    const float* ek = wq + DP * 2 * DC;
    const float* last = ek + DP * DC;
    const float* bb = last + DP;
    const float* yy = bb + DC * DC;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll (KW < 16 ? KW : 16)
    for (int kk = 0; kk < KW; ++kk) {
      const int d = warp * KW + kk;
      const float4 a = *reinterpret_cast<const float4*>(wq + d * 2 * DC + rg * 4);
      const float4 b = *reinterpret_cast<const float4*>(s_s + d * DCS + cg * 4);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) red_s[warp * 128 + i * 32 + lane] = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    __syncthreads();
    float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
    const int row = rg * 4 + warp;               // of the 32 rows of [W | P * Q], for the first four warps
    if (warp < 4) {
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        const float4 p = red_s[w * 128 + tid];
        sum.x += p.x; sum.y += p.y; sum.z += p.z; sum.w += p.w;
      }
      if (row < DC) {
        const float4 y = *reinterpret_cast<const float4*>(yy + row * DCN + cg * 4);
        *reinterpret_cast<float4*>(u_s + row * DCN + cg * 4) = make_float4(y.x - sum.x, y.y - sum.y, y.z - sum.z, y.w - sum.w);
      }
    }
    __syncthreads();
    if (warp < 4 && row >= DC) {                 // o = (P * Q) S + B u
      const int t = row - DC, r = chunk * DC + t;
#pragma unroll
      for (int s = 0; s < DC; ++s) {
        const float b = bb[s * DC + t];
        const float4 u = *reinterpret_cast<const float4*>(u_s + s * DCN + cg * 4);
        sum.x = fmaf(b, u.x, sum.x); sum.y = fmaf(b, u.y, sum.y); sum.z = fmaf(b, u.z, sum.z); sum.w = fmaf(b, u.w, sum.w);
      }
      if (r < count) {
        float* dst = out + ((size_t)(row0 + r) * heads + h) * vdim + col0 + cg * 4;
        const int left = vdim - col0 - cg * 4;
        if (left >= 4 && vdim % 4 == 0) *reinterpret_cast<float4*>(dst) = sum;
        else {
          const float o[4] = {sum.x, sum.y, sum.z, sum.w};
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (j < left) dst[j] = o[j];
        }
      }
    }
    // S' = diag(P_last) S + (E * K)^T u: four rows and four columns a thread; the warps that had no outputs come first
    for (int tile = tid ^ 128; tile < DP; tile += 256) {
      const int d = (tile >> 2) * 4, c = (tile & 3) * 4;
      const float4 keep = *reinterpret_cast<const float4*>(last + d);
      const float kv[4] = {keep.x, keep.y, keep.z, keep.w};
      float s[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 old = *reinterpret_cast<const float4*>(s_s + (d + i) * DCS + c);
        s[i][0] = kv[i] * old.x; s[i][1] = kv[i] * old.y; s[i][2] = kv[i] * old.z; s[i][3] = kv[i] * old.w;
      }
#pragma unroll
      for (int t = 0; t < DC; ++t) {
        const float4 e = *reinterpret_cast<const float4*>(ek + t * DP + d);
        const float4 u = *reinterpret_cast<const float4*>(u_s + t * DCN + c);
        const float ev[4] = {e.x, e.y, e.z, e.w}, uv[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) s[i][j] = fmaf(ev[i], uv[j], s[i][j]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(s_s + (d + i) * DCS + c) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
    }
  }
  __syncthreads();
  for (int e = tid; e < DP * DCN; e += 256) {
    const int d = e / DCN, c = e % DCN;
    if (d < dim && col0 + c < vdim) st[(size_t)d * vdim + col0 + c] = s_s[d * DCS + c];
  }
}

template <int NJ>
int launch_delta_chunks(const float* q, const float* k, const float* v, const float* beta, const float* z, int z_partials,
                        long long z_stride, long long z_ld, const float* dt_bias, const float* a_log, float* state,
                        const int* segment_start, const int* segment_slot, float* out, float* buffer, int max_chunks,
                        int max_segments, int heads, int groups, int dim, int vdim, int num_slots, int min_rows,
                        cudaStream_t stream) {
  constexpr int DP = 32 * NJ;
  const int ep = (vdim + DCN - 1) / DCN * DCN;
  const size_t prepare_smem = sizeof(float) * 3 * DC * DP;
  const size_t scan_smem = sizeof(float) * (DP * DCS + 2 * (DP * 2 * DC + DP * DC + DP + 2 * DC * DC) + 8 * 512 + DC * DCN);
  static bool configured = false;
  if (!configured) {
    cudaError_t err = cudaFuncSetAttribute(delta_chunk_prepare_kernel<NJ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prepare_smem);
    if (err == cudaSuccess)
      err = cudaFuncSetAttribute(delta_chunk_scan_kernel<NJ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan_smem);
    if (err != cudaSuccess) return (int)err;
    configured = true;
  }
  lse_launch(delta_chunk_prepare_kernel<NJ>, dim3(max_chunks, heads), 128, prepare_smem, stream, q, k, v, beta, z, z_partials,
             z_stride, z_ld, dt_bias, a_log, segment_start, buffer, max_segments, heads, groups, dim, vdim, ep, min_rows);
  lse_launch(delta_chunk_scan_kernel<NJ>, dim3(max_segments, heads, ep / DCN), 256, scan_smem, stream, (const float*)buffer,
             state, segment_start, segment_slot, out, heads, dim, vdim, ep, num_slots, min_rows);
  return (int)cudaGetLastError();
}

int dc_channels(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
}  // namespace

extern "C" int lse_delta_chunk_rows(void) { return DC; }

// Floats of the buffer per chunk and head.
extern "C" int lse_delta_chunk_floats(int dim, int vdim) {
  return (int)dc_all(dc_channels(dim), (vdim + DCN - 1) / DCN * DCN);
}

// The arguments of lse_delta_scan, for the requests of more than min_rows rows: buffer holds max_chunks * heads *
// lse_delta_chunk_floats(dim, vdim) floats, and max_chunks bounds the chunks of all requests (tokens / 16 + requests).
extern "C" int lse_delta_chunk_scan(const float* q, const float* k, const float* v, const float* beta, const float* z,
                                    int z_partials, long long z_stride, long long z_ld, const float* dt_bias,
                                    const float* a_log, float* state, const int* segment_start, const int* segment_slot,
                                    float* out, float* buffer, int max_chunks, int max_segments, int heads, int groups, int dim,
                                    int vdim, int num_slots, int min_rows, cudaStream_t stream) {
  if (max_segments <= 0 || max_chunks <= 0) return 0;
  if (heads <= 0 || groups <= 0 || heads % groups || heads > 65535 || dim <= 0 || dim > 256 || vdim <= 0 || z_partials < 1 ||
      min_rows < 0 || (((uintptr_t)buffer) & 15))
    return LSE_ERR_BAD_ARGUMENT;
  if (vdim > 65535 * DCN) return LSE_ERR_TOO_LARGE;
#define LSE_DC_GO(NJ)                                                                                                  \
  return launch_delta_chunks<NJ>(q, k, v, beta, z, z_partials, z_stride, z_ld, dt_bias, a_log, state, segment_start,   \
                                 segment_slot, out, buffer, max_chunks, max_segments, heads, groups, dim, vdim, num_slots, \
                                 min_rows, stream)
  switch (dc_channels(dim)) {
    case 32: LSE_DC_GO(1);
    case 64: LSE_DC_GO(2);
    case 128: LSE_DC_GO(4);
    default: LSE_DC_GO(8);
  }
#undef LSE_DC_GO
}
