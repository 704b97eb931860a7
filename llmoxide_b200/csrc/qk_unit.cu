// Attention whose keys are its values: what lies between the fused projection and the scores, and the output's gate.
//
// qk_unit_rope_cache   a projected row holds q heads, then k heads (D dims each), then columns it does not read.  Per head:
//                      x = row + bias; a key head's x goes into the value store as it is; q and k are rotated (pairs
//                      (i, i + n_rot/2) of the first n_rot dims, float32 tables), divided by their root mean square over
//                      the head's D dims (no weight) and go to q_out and the key store.
// gate_rows            out[t, c] *= sigmoid(z[t, c]), z columns of the projection (partials added in order).
//
// One warp per head; a step of many tokens gives a warp four heads of its token, so that the token's indices and
// rotation rows are fetched once.  Everything is float32 until it is stored.
#include "common.cuh"

#define QU_WARPS 4
#define QU_MAX_D 256

__device__ __forceinline__ void qu_load4(const float* p, float* o) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  o[0] = x.x, o[1] = x.y, o[2] = x.z, o[3] = x.w;
}
__device__ __forceinline__ void qu_load4(const bf16* p, float* o) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  o[0] = a.x, o[1] = a.y, o[2] = b.x, o[3] = b.y;
}
__device__ __forceinline__ void qu_store4(float* p, const float* v) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void qu_store4(bf16* p, const float* v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 raw;
  raw.x = *reinterpret_cast<uint32_t*>(&a);
  raw.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}

// V: dims a lane takes at a time (4 where sizes and addresses allow, else 1); SPW: heads per warp.
template <typename TIN, typename TC, int V, int SPW>
__global__ void __launch_bounds__(QU_WARPS * 32)
qk_unit_rope_cache_kernel(const TIN* __restrict__ proj, int n_split, size_t split_stride, size_t row_stride,
                          const float* __restrict__ bias, TC* __restrict__ q_out, TC* __restrict__ k_cache,
                          TC* __restrict__ v_cache, const int* __restrict__ block_table, int table_width,
                          const int* __restrict__ token_seq, const int* __restrict__ token_pos, float eps,
                          const float* __restrict__ cos_t, const float* __restrict__ sin_t, int n_rot, int H, int G, int D,
                          int n_seqs, int n_pages) {
  constexpr int NV = QU_MAX_D / (32 * V);               // a lane's vectors of a head
  __shared__ __align__(16) float head_buf[QU_WARPS][QU_MAX_D];
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x;
  const int slot0 = (blockIdx.y * QU_WARPS + warp) * SPW;
  if (slot0 >= H + G) return;
  const int b = token_seq[t], pos = token_pos[t];
  if (b < 0 || b >= n_seqs || pos < 0 || pos / LLMX_PAGE >= table_width) {
    if (lane == 0) llmx_report(1);
    return;
  }
  int page = 0;
  if (slot0 + SPW > H) page = block_table[(size_t)b * table_width + pos / LLMX_PAGE];
  if (page < 0 || page >= n_pages) {
    if (lane == 0) llmx_report(1);
    return;
  }
  float* buf = head_buf[warp];
  const int half = n_rot >> 1;
  const float* cs = n_rot ? cos_t + (size_t)pos * half : nullptr;
  const float* sn = n_rot ? sin_t + (size_t)pos * half : nullptr;
  pdl_wait();
  const TIN* row = proj + (size_t)t * row_stride;
  float x[SPW][NV][V];
#pragma unroll
  for (int j = 0; j < SPW; ++j) {                       // the warp's heads are asked for together
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (k * 32 + lane) * V;
#pragma unroll
      for (int e = 0; e < V; ++e) x[j][k][e] = 0.f;
      if (slot0 + j < H + G && i < D) {
        const size_t c = (size_t)(slot0 + j) * D + i;
        if (V == 4) {
          qu_load4(row + c, x[j][k]);
          for (int s = 1; s < n_split; ++s) {
            float y[4];
            qu_load4(row + (size_t)s * split_stride + c, y);
#pragma unroll
            for (int e = 0; e < V; ++e) x[j][k][e] += y[e];
          }
          if (bias) {
            float y[4];
            qu_load4(bias + c, y);
#pragma unroll
            for (int e = 0; e < V; ++e) x[j][k][e] += y[e];
          }
        } else {
          x[j][k][0] = split_value(row, c, n_split, split_stride) + (bias ? bias[c] : 0.f);
        }
      }
    }
  }
#pragma unroll
  for (int j = 0; j < SPW; ++j) {
    const int slot = slot0 + j;
    if (slot >= H + G) break;
    const bool is_q = slot < H;
    TC* dst = q_out + (size_t)t * H * D + (size_t)slot * D;
    if (!is_q) {
      const size_t off = cache_row_offset(page, slot - H, pos % LLMX_PAGE, G, D);
      dst = k_cache + off;
#pragma unroll
      for (int k = 0; k < NV; ++k) {                    // the value: the key as projected
        const int i = (k * 32 + lane) * V;
        if (i < D) {
          if (V == 4) qu_store4(v_cache + off + i, x[j][k]);
          else v_cache[off + i] = from_f32<TC>(x[j][k][0]);
        }
      }
    }
    if (n_rot) {
#pragma unroll
      for (int k = 0; k < NV; ++k) {
        const int i = (k * 32 + lane) * V;
        if (i < n_rot) {
#pragma unroll
          for (int e = 0; e < V; ++e) buf[i + e] = x[j][k][e];
        }
      }
      __syncwarp();
#pragma unroll
      for (int k = 0; k < NV; ++k) {
        const int i = (k * 32 + lane) * V;              // (V = 4: the rotation's borders are multiples of four)
        if (i < n_rot) {
          const bool low = i < half;
          const int at = low ? i : i - half, other = low ? i + half : i - half;
#pragma unroll
          for (int e = 0; e < V; ++e) {
            const float c = cs[at + e], s = sn[at + e], o = buf[other + e];
            x[j][k][e] = low ? x[j][k][e] * c - o * s : x[j][k][e] * c + o * s;
          }
        }
      }
      __syncwarp();                                     // buf is filled again for the warp's next head
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k)
#pragma unroll
      for (int e = 0; e < V; ++e) ss += x[j][k][e] * x[j][k][e];
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)D + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (k * 32 + lane) * V;
      if (i < D) {
        float y[V];
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = x[j][k][e] * r;
        if (V == 4) qu_store4(dst + i, y);
        else dst[i] = from_f32<TC>(y[0]);
      }
    }
  }
}

// proj [T, row_stride] (or n_split partials of it) with q heads from column 0 and k heads behind them; bias: null or
// float32 [(H + G) * D]; q_out [T, H*D] and the cache entry [n_pages, G, 64, D] of one dtype; n_rot 0: no rotation.
LLMX_API int llmx_qk_unit_rope_cache(const void* proj, int in_dtype, int n_split, long long split_stride,
                                     long long row_stride, const float* bias, void* q_out, void* k_cache, void* v_cache,
                                     int cache_dtype, const int* block_table, int table_width, const int* token_seq,
                                     const int* token_pos, float eps, const float* cos_t, const float* sin_t, int n_rot,
                                     int n_tokens, int H, int G, int D, int n_seqs, long long n_pages,
                                     cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || D <= 0 || D > QU_MAX_D || n_rot < 0 || n_rot > D || (n_rot & 1) || n_split < 1 ||
      row_stride < (long long)(H + G) * D)
    return LLMX_REFUSED(1);
  if (n_rot > 0 && (!cos_t || !sin_t)) return LLMX_REFUSED(4);
  const int spw = n_tokens > 64 ? 4 : 1;
  const bool vec = D % 4 == 0 && n_rot % 8 == 0 && row_stride % 4 == 0 && split_stride % 4 == 0 &&
                   !(((uintptr_t)proj | (uintptr_t)bias | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15);
  const dim3 grid(n_tokens, (H + G + QU_WARPS * spw - 1) / (QU_WARPS * spw));
#define GO2(TIN, TC, V, SPW)                                                                                            \
  launch_pdl(qk_unit_rope_cache_kernel<TIN, TC, V, SPW>, grid, dim3(QU_WARPS * 32), 0, stream, (const TIN*)proj, n_split, \
             (size_t)split_stride, (size_t)row_stride, bias, (TC*)q_out, (TC*)k_cache, (TC*)v_cache, block_table,       \
             table_width, token_seq, token_pos, eps, cos_t, sin_t, n_rot, H, G, D, n_seqs, (int)n_pages)
#define GO(TIN, TC)                                    \
  do {                                                 \
    if (vec && spw == 4) GO2(TIN, TC, 4, 4);           \
    else if (vec) GO2(TIN, TC, 4, 1);                  \
    else if (spw == 4) GO2(TIN, TC, 1, 4);             \
    else GO2(TIN, TC, 1, 1);                           \
  } while (0)
  if (in_dtype == LLMX_F32 && cache_dtype == LLMX_F32) GO(float, float);
  else if (in_dtype == LLMX_F32 && cache_dtype == LLMX_BF16) GO(float, bf16);
  else if (in_dtype == LLMX_BF16 && cache_dtype == LLMX_BF16) GO(bf16, bf16);
  else return LLMX_REFUSED(2);
#undef GO
#undef GO2
  return LLMX_LAUNCH_STATUS();
}

// V consecutive columns a thread (8 where sizes and addresses allow).
template <typename TO, typename TZ, int V>
__global__ void __launch_bounds__(256)
gate_rows_kernel(TO* __restrict__ out, const TZ* __restrict__ z, int n_split, size_t split_stride, size_t row_stride,
                 size_t n, int width) {
  pdl_launch_dependents();
  pdl_wait();
  for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V; i < n; i += (size_t)gridDim.x * blockDim.x * V) {
    const size_t t = i / width, c = i - t * width;
    const TZ* zp = z + t * row_stride + c;
    if (V == 1) {
      out[i] = from_f32<TO>(to_f32(out[i]) / (1.0f + expf(-split_value(zp, 0, n_split, split_stride))));
      continue;
    }
    float zs[8], o[8];
#pragma unroll
    for (int e = 0; e < 8; e += 4) {
      qu_load4(zp + e, zs + e);
      qu_load4(out + i + e, o + e);
    }
    for (int s = 1; s < n_split; ++s) {
      float y[8];
#pragma unroll
      for (int e = 0; e < 8; e += 4) qu_load4(zp + (size_t)s * split_stride + e, y + e);
#pragma unroll
      for (int e = 0; e < 8; ++e) zs[e] += y[e];
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = o[e] / (1.0f + expf(-zs[e]));
#pragma unroll
    for (int e = 0; e < 8; e += 4) qu_store4(out + i + e, o + e);
  }
}

// out [T, width] contiguous; z: [T, row_stride] from its first gate column on (or n_split partials of it).
LLMX_API int llmx_gate_rows(void* out, int out_dtype, const void* z, int z_dtype, int n_split, long long split_stride,
                            long long row_stride, int n_tokens, int width, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (width <= 0 || n_split < 1 || row_stride < width) return LLMX_REFUSED(1);
  const size_t n = (size_t)n_tokens * width;
  const bool vec = width % 8 == 0 && row_stride % 4 == 0 && split_stride % 4 == 0 && !((uintptr_t)out & 15) &&
                   !((uintptr_t)z & 15);
  const size_t units = vec ? n / 8 : n;
  const int blocks = (int)((units + 255) / 256 < 148 * 16 ? (units + 255) / 256 : 148 * 16);
#define GO(TO, TZ)                                                                                                     \
  do {                                                                                                                 \
    if (vec) launch_pdl(gate_rows_kernel<TO, TZ, 8>, dim3(blocks), dim3(256), 0, stream, (TO*)out, (const TZ*)z, n_split, \
                        (size_t)split_stride, (size_t)row_stride, n, width);                                           \
    else launch_pdl(gate_rows_kernel<TO, TZ, 1>, dim3(blocks), dim3(256), 0, stream, (TO*)out, (const TZ*)z, n_split,  \
                    (size_t)split_stride, (size_t)row_stride, n, width);                                               \
  } while (0)
  if (out_dtype == LLMX_F32 && z_dtype == LLMX_F32) GO(float, float);
  else if (out_dtype == LLMX_BF16 && z_dtype == LLMX_F32) GO(bf16, float);
  else if (out_dtype == LLMX_BF16 && z_dtype == LLMX_BF16) GO(bf16, bf16);
  else return LLMX_REFUSED(2);
#undef GO
  return LLMX_LAUNCH_STATUS();
}
