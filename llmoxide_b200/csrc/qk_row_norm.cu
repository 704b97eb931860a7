// RMS norm of a whole query (and key) projection, before it is split into heads, a temperature on the query, and the
// cache write of keys and values, in one pass over a token's row.
//
//   q = q / sqrt(mean(q^2) + eps) * q_gain * temp(p)        mean over all H*D values of the token's query row
//   k = k / sqrt(mean(k^2) + eps) * k_gain                  mean over all G*D values
//   temp(p) = 1 + coef * ln(floor((p + 1) / every) + 1)     p: the token's position; every 0: no temperature
//
// A row of the projection holds [ q (H*D) | k (G*D) | v (G*Dv) ], or q alone for a layer that borrows its keys and
// values.  One CTA per token; q and k are staged in shared memory as float32 (split partials are added in order while
// they are staged), both sums of squares are taken in one reduction, and everything is float32 until it is stored.
// A thread's share of the row and the reduction's order depend on the sizes alone.
#include "common.cuh"

__device__ __forceinline__ void qr_load4(const float* p, float* o) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  o[0] = x.x, o[1] = x.y, o[2] = x.z, o[3] = x.w;
}
__device__ __forceinline__ void qr_load4(const bf16* p, float* o) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  o[0] = a.x, o[1] = a.y, o[2] = b.x, o[3] = b.y;
}
__device__ __forceinline__ void qr_store4(float* p, const float* v) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void qr_store4(bf16* p, const float* v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 raw;
  raw.x = *reinterpret_cast<uint32_t*>(&a);
  raw.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}
// V consecutive values of the row, partials added in order
template <int V, typename TIN>
__device__ __forceinline__ void qr_value(const TIN* p, int n_split, size_t split_stride, float* o) {
  if (V == 4) qr_load4(p, o);
  else o[0] = to_f32(p[0]);
  for (int s = 1; s < n_split; ++s) {
    float t[4];
    if (V == 4) qr_load4(p + (size_t)s * split_stride, t);
    else t[0] = to_f32(p[(size_t)s * split_stride]);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] += t[e];
  }
}
template <int V, typename T>
__device__ __forceinline__ void qr_put(T* p, const float* v) {
  if (V == 4) qr_store4(p, v);
  else p[0] = from_f32<T>(v[0]);
}
template <int V>
__device__ __forceinline__ void qr_get(const float* p, float* v) {
  if (V == 4) qr_load4(p, v);
  else v[0] = p[0];
}

template <typename TIN, typename TA, typename TC, int V>
__global__ void __launch_bounds__(512)
qk_row_norm_kernel(const TIN* __restrict__ proj, int n_split, size_t split_stride, size_t row_stride,
                   TA* __restrict__ q_out, TC* __restrict__ k_cache, TC* __restrict__ v_cache,
                   const int* __restrict__ block_table, int table_width, const int* __restrict__ token_seq,
                   const int* __restrict__ token_pos, const float* __restrict__ q_gain,
                   const float* __restrict__ k_gain, float eps, float temp_coef, int temp_every, int H, int G, int D,
                   int Dv, int has_kv, int n_seqs, int n_pages) {
  extern __shared__ __align__(16) float qr_row[];       // [H*D | G*D]
  __shared__ float red[2][32];
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  const int nq = H * D, nk = has_kv ? G * D : 0, nv = has_kv ? G * Dv : 0;
  const int pos = token_pos[t];
  int page = 0;
  if (has_kv) {
    const int b = token_seq[t];
    bool bad = b < 0 || b >= n_seqs || pos < 0 || pos / LLMX_PAGE >= table_width;
    if (!bad) {
      page = block_table[(size_t)b * table_width + pos / LLMX_PAGE];
      bad = page < 0 || page >= n_pages;
    }
    if (bad) {                                          // uniform over the CTA
      if (threadIdx.x == 0) llmx_report(1);
      return;
    }
  }
  pdl_wait();
  const TIN* row = proj + (size_t)t * row_stride;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x * V; i < nq + nk; i += blockDim.x * V) {
    float x[V];
    qr_value<V>(row + i, n_split, split_stride, x);
    qr_put<V>(qr_row + i, x);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s += x[e] * x[e];
    if (i < nq) sq += s; else sk += s;                  // (nq is a multiple of V)
  }
  // the values need no norm: straight into the cache
  for (int i = threadIdx.x * V; i < nv; i += blockDim.x * V) {
    float x[V];
    qr_value<V>(row + nq + nk + i, n_split, split_stride, x);
    const int g = i / Dv;
    qr_put<V>(v_cache + cache_row_offset(page, g, pos % LLMX_PAGE, G, Dv) + (i - g * Dv), x);
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) red[0][warp] = sq, red[1][warp] = sk;
  __syncthreads();
  sq = warp_sum(lane < n_warps ? red[0][lane] : 0.f);
  sk = warp_sum(lane < n_warps ? red[1][lane] : 0.f);
  float rq = 1.0f / sqrtf(sq / (float)nq + eps);
  const float rk = has_kv ? 1.0f / sqrtf(sk / (float)nk + eps) : 0.f;
  float temp = 1.0f;
  if (temp_every > 0) temp = 1.0f + temp_coef * logf((float)((pos + 1) / temp_every) + 1.0f);
  // every thread takes the values it staged itself: no barrier between the two uses of the row
  for (int i = threadIdx.x * V; i < nq + nk; i += blockDim.x * V) {
    float x[V], gn[V];
    qr_get<V>(qr_row + i, x);
    if (i < nq) {
      qr_get<V>(q_gain + i, gn);
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] = (x[e] * rq) * gn[e] * temp;
      qr_put<V>(q_out + (size_t)t * nq + i, x);
    } else {
      const int j = i - nq, g = j / D;
      qr_get<V>(k_gain + j, gn);
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] = (x[e] * rk) * gn[e];
      qr_put<V>(k_cache + cache_row_offset(page, g, pos % LLMX_PAGE, G, D) + (j - g * D), x);
    }
  }
}

// proj [T, row_stride] (or n_split float32 partials split_stride elements apart); q_out [T, H*D]; the caches
// [pages, G, PAGE, D] and [pages, G, PAGE, Dv]; has_kv 0: the row is q alone and neither cache nor block table is
// read or written.  temp_every 0: no temperature.
LLMX_API int llmx_qk_row_norm(const void* proj, int in_dtype, int n_split, long long split_stride, long long row_stride,
                              void* q_out, int act_dtype, void* k_cache, void* v_cache, int cache_dtype,
                              const int* block_table, int table_width, const int* token_seq, const int* token_pos,
                              const float* q_gain, const float* k_gain, float eps, float temp_coef, int temp_every,
                              int n_tokens, int H, int G, int D, int Dv, int has_kv, int n_seqs, long long n_pages,
                              cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || D <= 0 || n_split < 1 || temp_every < 0 || (has_kv && (G <= 0 || Dv <= 0))) return LLMX_REFUSED(1);
  if (row_stride < (long long)H * D + (has_kv ? (long long)G * (D + Dv) : 0)) return LLMX_REFUSED(1);
  if (!q_gain || (has_kv && (!k_gain || !k_cache || !v_cache || !block_table || !token_seq))) return LLMX_REFUSED(4);
  const int n = H * D + (has_kv ? G * D : 0);
  const size_t smem = (size_t)n * sizeof(float);
  if (smem > 200 * 1024) return LLMX_REFUSED(3);
  const uintptr_t addrs = (uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)q_gain |
                          (has_kv ? ((uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)k_gain) : 0);
  const bool vec = D % 4 == 0 && (!has_kv || Dv % 4 == 0) && row_stride % 4 == 0 && split_stride % 4 == 0 && !(addrs & 15);
  int threads = ((n + 3) / 4 + 31) / 32 * 32;
  threads = threads < 64 ? 64 : threads > 512 ? 512 : threads;
#define GO(TIN, TA, TC, V)                                                                                               \
  do {                                                                                                                   \
    if (smem > 48 * 1024) {                                                                                              \
      cudaError_t e = cudaFuncSetAttribute(qk_row_norm_kernel<TIN, TA, TC, V>,                                           \
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                      \
      if (e != cudaSuccess) return (int)e;                                                                               \
    }                                                                                                                    \
    launch_pdl(qk_row_norm_kernel<TIN, TA, TC, V>, dim3(n_tokens), dim3(threads), smem, stream, (const TIN*)proj,        \
               n_split, (size_t)split_stride, (size_t)row_stride, (TA*)q_out, (TC*)k_cache, (TC*)v_cache, block_table,   \
               table_width, token_seq, token_pos, q_gain, k_gain, eps, temp_coef, temp_every, H, G, D, Dv, has_kv,       \
               n_seqs, (int)n_pages);                                                                                    \
  } while (0)
#define CASE(TIN, TA, TC)          \
  do {                             \
    if (vec) GO(TIN, TA, TC, 4);   \
    else GO(TIN, TA, TC, 1);       \
  } while (0)
  switch (in_dtype * 4 + act_dtype * 2 + cache_dtype) {
    case 0: CASE(float, float, float); break;
    case 3: CASE(float, bf16, bf16); break;
    case 7: CASE(bf16, bf16, bf16); break;
    default: return LLMX_REFUSED(2);
  }
#undef CASE
#undef GO
  return LLMX_LAUNCH_STATUS();
}
