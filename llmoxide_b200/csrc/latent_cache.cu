// Attention over a cache of latents: a position's cached row is [ c (rank) | rotated key part (R) ], one for all heads.
//
//   k_h = [ rot part | W_uk,h c ],  v_h = W_uv,h c,   score = (q_rot . rot part + q_plain . W_uk,h c) * scale
//
// so a head's score is (q_rot . rot part + (W_uk,h^T q_plain) . c) * scale and its output W_uv,h (sum_j w_j c_j): with the
// query taken through W_uk^T first ("absorbed") the cached rows serve as keys and values of every head as they are.
// `sinks` (float32 [H] or null): exp(sinks[h]) joins head h's denominator, a score without key and value, not scaled.
//
//   latent_prep      the latent's RMS norm, the rotations, the cache row, the query in the layout its attention takes
//   head_product     y[t, h] = W_h x[t, h] for every head (the query into the latent space, the output out of it)
//   latent_decode    absorbed attention on the tensor cores (mma.sync), every token on its own: 16 heads a CTA, the
//                    cached rows cut into shares, partial results merged by latent_combine
//   latent_paged     absorbed attention in float32 arithmetic, one warp per (token, head): every size, both dtypes
//   latent_gather, latent_assemble   prompts: the latents of the step's sequences out of their pages, and, behind the
//                    product [W_uk; W_uv] c over them, every head's keys and values in pages of their own, which the
//                    tiled prompt attention kernels read like any cache
//
// Scores, statistics, rotations and norms are float32; bfloat16 is rounded to only where something is stored or is an
// operand of a tensor-core product.
#include "tc_ptx.cuh"

#define LC_TILE 32           // cached rows per tile of latent_decode
#define LC_HEADS 16          // heads per CTA
#define LC_WARPS 4
#define LC_PREP_HEADS 4      // query heads per CTA of latent_prep
#define LC_MAX_CHUNKS 128    // shares of one token's rows
#define LC_MAX_RANK 512      // latent_decode; latent_paged takes up to LC_MAX_RANK_GENERAL
#define LC_MAX_RANK_GENERAL 1024

template <typename T>
__device__ __forceinline__ float lc_value(const T* p, int n_split, size_t split_stride) {
  return split_value(p, 0, n_split, split_stride);
}

// Where token t lives: false (and a report) when the step's arrays do not fit the launch.
__device__ __forceinline__ bool lc_page(const int* block_table, int table_width, int b, int pos, int n_seqs, int n_pages,
                                        int* page) {
  if (b < 0 || b >= n_seqs || pos < 0 || pos / LLMX_PAGE >= table_width) return false;
  *page = block_table[(size_t)b * table_width + pos / LLMX_PAGE];
  return *page >= 0 && *page < n_pages;
}

// ---------------------------------------------------------------------------
// CTA (t, 0) does the token's latent and its cache row, CTA (t, y > 0) LC_PREP_HEADS query heads.  down: [T, down_stride] with the latent at column 0 and the shared key part at column rank (float32
// or float32 partials); q: [T, q_stride], every head [ R rotated | D plain ].  Pairs (i, i + R/2) turn by the
// position's angles.  q goes to rot_out[(t H + h) rot_ld + 0..R-1] and plain_out[(t H + h) plain_ld + 0..D-1].
// ---------------------------------------------------------------------------
template <typename TIN, typename TQ, typename TR, typename TP, typename TC>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const TIN* __restrict__ down, int n_split, size_t split_stride, size_t down_stride,
                   const TQ* __restrict__ q, int q_split, size_t q_split_stride, size_t q_stride,
                   const float* __restrict__ gain, float eps, TC* __restrict__ cache, TR* __restrict__ rot_out,
                   size_t rot_ld, TP* __restrict__ plain_out, size_t plain_ld, const int* __restrict__ block_table,
                   int table_width, const int* __restrict__ token_seq, const int* __restrict__ token_pos,
                   const float* __restrict__ cos_t, const float* __restrict__ sin_t, int H, int D, int R, int rank,
                   int n_seqs, int n_pages) {
  extern __shared__ __align__(16) float lc_row[];       // [rank]
  __shared__ float red[32];
  pdl_launch_dependents();
  const int t = blockIdx.x, b = token_seq[t], pos = token_pos[t], half = R >> 1;
  int page = 0;
  if (!lc_page(block_table, table_width, b, pos, n_seqs, n_pages, &page)) {        // uniform over the CTA
    if (threadIdx.x == 0) llmx_report(1);
    return;
  }
  const float* cs = cos_t + (size_t)pos * half;
  const float* sn = sin_t + (size_t)pos * half;
  pdl_wait();
  const TIN* row = down + (size_t)t * down_stride;
  if (blockIdx.y > 0) {
    const TQ* qrow = q + (size_t)t * q_stride;
    const int h_lo = (blockIdx.y - 1) * LC_PREP_HEADS, n_h = min(LC_PREP_HEADS, H - h_lo), E = R + D;
    for (int e = threadIdx.x; e < n_h * half; e += blockDim.x) {
      const int h = h_lo + e / half, i = e % half;
      const float c = cs[i], s = sn[i];
      const float x = lc_value(qrow + (size_t)h * E + i, q_split, q_split_stride);
      const float y = lc_value(qrow + (size_t)h * E + i + half, q_split, q_split_stride);
      TR* dst = rot_out + ((size_t)t * H + h) * rot_ld + i;
      dst[0] = from_f32<TR>(x * c - y * s);
      dst[half] = from_f32<TR>(y * c + x * s);
    }
    for (int e = threadIdx.x; e < n_h * D; e += blockDim.x) {
      const int h = h_lo + e / D, i = e % D;
      plain_out[((size_t)t * H + h) * plain_ld + i] = from_f32<TP>(lc_value(qrow + (size_t)h * E + R + i, q_split, q_split_stride));
    }
    return;
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < rank; i += blockDim.x) {
    const float v = lc_value(row + i, n_split, split_stride);
    lc_row[i] = v;
    ss += v * v;
  }
  const float rstd = 1.0f / sqrtf(block_sum(ss, red) / (float)rank + eps);
  TC* dst = cache + cache_row_offset(page, 0, pos % LLMX_PAGE, 1, rank + R);
  for (int i = threadIdx.x; i < rank; i += blockDim.x) dst[i] = from_f32<TC>((lc_row[i] * rstd) * gain[i]);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float c = cs[i], s = sn[i];
    const float x = lc_value(row + rank + i, n_split, split_stride), y = lc_value(row + rank + i + half, n_split, split_stride);
    dst[rank + i] = from_f32<TC>(x * c - y * s);
    dst[rank + i + half] = from_f32<TC>(y * c + x * s);
  }
}

LLMX_API int llmx_latent_prep(const void* down, int in_dtype, int n_split, long long split_stride, long long down_stride,
                              const void* q, int q_dtype, int q_split, long long q_split_stride, long long q_stride,
                              const float* gain, float eps, void* cache, int cache_dtype, void* rot_out, long long rot_ld,
                              void* plain_out, long long plain_ld, int out_dtype, const int* block_table, int table_width,
                              const int* token_seq, const int* token_pos, const float* cos_t, const float* sin_t,
                              int n_tokens, int H, int D, int R, int rank, int n_seqs, long long n_pages,
                              cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || D <= 0 || R <= 0 || (R & 1) || rank <= 0 || n_split < 1 || q_split < 1 || down_stride < rank + R ||
      q_stride < (long long)H * (R + D) || rot_ld < R || plain_ld < D)
    return LLMX_REFUSED(1);
  if (!cos_t || !sin_t || !gain) return LLMX_REFUSED(4);
  const size_t smem = (size_t)rank * sizeof(float);
  if (smem > 48 * 1024) return LLMX_REFUSED(3);
  const dim3 prep_grid(n_tokens, 1 + (H + LC_PREP_HEADS - 1) / LC_PREP_HEADS);
#define CASE(TQ, TO, TC)                                                                                                 \
  launch_pdl(latent_prep_kernel<float, TQ, TO, TO, TC>, prep_grid, dim3(256), smem, stream, (const float*)down,            \
             n_split, (size_t)split_stride, (size_t)down_stride, (const TQ*)q, q_split, (size_t)q_split_stride,          \
             (size_t)q_stride, gain, eps, (TC*)cache, (TO*)rot_out, (size_t)rot_ld, (TO*)plain_out, (size_t)plain_ld,    \
             block_table, table_width, token_seq, token_pos, cos_t, sin_t, H, D, R, rank, n_seqs, (int)n_pages)
  if (in_dtype != LLMX_F32) return LLMX_REFUSED(2);
  switch (q_dtype * 4 + out_dtype * 2 + cache_dtype) {
    case 0: CASE(float, float, float); break;
    case 1: CASE(float, float, bf16); break;
    case 3: CASE(float, bf16, bf16); break;
    case 5: CASE(bf16, float, bf16); break;
    case 7: CASE(bf16, bf16, bf16); break;
    default: return LLMX_REFUSED(2);
  }
#undef CASE
  return LLMX_LAUNCH_STATUS();
}

// ---------------------------------------------------------------------------
// y[t, h, 0..N-1] = W[h] x[t, h, 0..K-1], W [H, N, K].  x rows x_ld apart per (t, h), y rows y_ld apart.
// ---------------------------------------------------------------------------
__device__ __forceinline__ void lc_mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                       uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// bfloat16 on the tensor cores: a warp owns 16 rows of W_h (the M axis) and 8 TN tokens.  A lane reads 16 bytes of a row
// at a time, eight neighbouring k; the two products of a 32-wide block of k take the lane's words in the same order from
// W and from x, so which k meets which is the same on both sides and the sum does not notice the order.
template <int TN>
__global__ void __launch_bounds__(128)
head_product_mma_kernel(const bf16* __restrict__ x, size_t x_ld, const bf16* __restrict__ w, bf16* __restrict__ y,
                        size_t y_ld, int T, int H, int N, int K) {
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gq = lane >> 2, tq = lane & 3;
  const int h = blockIdx.y, n0 = (blockIdx.x * (blockDim.x >> 5) + warp) * 16, t0 = blockIdx.z * 8 * TN;
  if (n0 >= N) return;
  const bf16* wlo = w + ((size_t)h * N + n0 + gq) * K;
  const bf16* whi = wlo + (size_t)8 * K;
  const bool lo_live = n0 + gq < N, hi_live = n0 + gq + 8 < N;
  float acc[TN][4];
#pragma unroll
  for (int j = 0; j < TN; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const bf16* xr[TN];
  bool x_live[TN];
#pragma unroll
  for (int j = 0; j < TN; ++j) {
    const int t = t0 + 8 * j + gq;
    x_live[j] = t < T;
    xr[j] = x + ((size_t)(x_live[j] ? t : 0) * H + h) * x_ld;
  }
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  pdl_wait();
#pragma unroll(TN == 1 ? 8 : 4)
  for (int k0 = 0; k0 < K; k0 += 32) {
    const int k = k0 + 8 * tq;
    const bool in = k < K;                               // K is a multiple of 8
    const uint4 a = in && lo_live ? *reinterpret_cast<const uint4*>(wlo + k) : zero;
    const uint4 c = in && hi_live ? *reinterpret_cast<const uint4*>(whi + k) : zero;
#pragma unroll
    for (int j = 0; j < TN; ++j) {
      const uint4 v = in && x_live[j] ? *reinterpret_cast<const uint4*>(xr[j] + k) : zero;
      lc_mma(acc[j], a.x, c.x, a.y, c.y, v.x, v.y);
      lc_mma(acc[j], a.z, c.z, a.w, c.w, v.z, v.w);
    }
  }
#pragma unroll
  for (int j = 0; j < TN; ++j) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {                        // rows n0 + gq (+8), tokens 2 tq (+1)
      const int n = n0 + gq + 8 * (e >> 1), t = t0 + 8 * j + 2 * tq + (e & 1);
      if (n < N && t < T) y[((size_t)t * H + h) * y_ld + n] = from_f32<bf16>(acc[j][e]);
    }
  }
}

// Any size and dtype, float32 sums: one warp per output, lanes over k.
template <typename TX, typename TW, typename TY>
__global__ void __launch_bounds__(256)
head_product_kernel(const TX* __restrict__ x, size_t x_ld, const TW* __restrict__ w, TY* __restrict__ y, size_t y_ld, int H,
                    int N, int K) {
  extern __shared__ __align__(16) float lc_row[];       // [K]
  pdl_launch_dependents();
  const int t = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  const TX* xr = x + ((size_t)t * H + h) * x_ld;
  for (int k = threadIdx.x; k < K; k += blockDim.x) lc_row[k] = to_f32(xr[k]);
  __syncthreads();
  for (int n = warp; n < N; n += 8) {
    const TW* wr = w + ((size_t)h * N + n) * K;
    float s = 0.f;
    for (int k = lane; k < K; k += 32) s = fmaf(to_f32(wr[k]), lc_row[k], s);
    s = warp_sum(s);
    if (lane == 0) y[((size_t)t * H + h) * y_ld + n] = from_f32<TY>(s);
  }
}

LLMX_API int llmx_head_product(const void* x, int x_dtype, long long x_ld, const void* w, int w_dtype, void* y, int y_dtype,
                               long long y_ld, int n_tokens, int H, int N, int K, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || N <= 0 || K <= 0 || x_ld < K || y_ld < N || H > 65535) return LLMX_REFUSED(1);
  if (x_dtype == LLMX_BF16 && w_dtype == LLMX_BF16 && y_dtype == LLMX_BF16 && K % 8 == 0 && x_ld % 8 == 0 &&
      !(((uintptr_t)x | (uintptr_t)w) & 15)) {
    const int tn = n_tokens <= 8 ? 1 : n_tokens <= 16 ? 2 : 4;
    // warps per CTA: one while four would leave SMs without a CTA
    const int warps = (long long)((N + 63) / 64) * H * ((n_tokens + 8 * tn - 1) / (8 * tn)) < 148 ? 1 : 4;
    const dim3 grid((N + 16 * warps - 1) / (16 * warps), H, (n_tokens + 8 * tn - 1) / (8 * tn));
    if (grid.z > 65535) return LLMX_REFUSED(3);
#define GO(TN)                                                                                                          \
  launch_pdl(head_product_mma_kernel<TN>, grid, dim3(32 * warps), 0, stream, (const bf16*)x, (size_t)x_ld, (const bf16*)w,     \
             (bf16*)y, (size_t)y_ld, n_tokens, H, N, K)
    if (tn == 1) GO(1); else if (tn == 2) GO(2); else GO(4);
#undef GO
    return LLMX_LAUNCH_STATUS();
  }
  const size_t smem = (size_t)K * sizeof(float);
  if (smem > 48 * 1024) return LLMX_REFUSED(3);
#define CASE(TX, TW, TY)                                                                                                \
  launch_pdl(head_product_kernel<TX, TW, TY>, dim3(n_tokens, H), dim3(256), smem, stream, (const TX*)x, (size_t)x_ld,   \
             (const TW*)w, (TY*)y, (size_t)y_ld, H, N, K)
  switch (x_dtype * 4 + w_dtype * 2 + y_dtype) {
    case 0: CASE(float, float, float); break;
    case 1: CASE(float, float, bf16); break;
    case 2: CASE(float, bf16, float); break;
    case 3: CASE(float, bf16, bf16); break;
    case 7: CASE(bf16, bf16, bf16); break;
    default: return LLMX_REFUSED(2);
  }
#undef CASE
  return LLMX_LAUNCH_STATUS();
}

// ---------------------------------------------------------------------------
// Absorbed attention, one warp per (token, head), float32: q float32 [T, H, rank + R] = [ absorbed | rotated ]; lat
// float32 [T, H, rank].  Rows 32 at a time from position 0: lane j scores row base + j, then the lanes own dims
// (lane, lane + 32, ..) of the sum.  The order depends on the position alone.
// ---------------------------------------------------------------------------
template <typename TC, int OWN>
__global__ void __launch_bounds__(128)
latent_paged_kernel(const float* __restrict__ q, float* __restrict__ lat, const TC* __restrict__ cache,
                    const int* __restrict__ block_table, int table_width, const int* __restrict__ token_seq,
                    const int* __restrict__ token_pos, const float* __restrict__ sinks, float scale, int H, int rank,
                    int R) {
  extern __shared__ __align__(16) float lc_row[];       // [4 warps][rank + R]
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x, h = blockIdx.y * 4 + warp, E = rank + R;
  if (h >= H) return;
  const int p = token_pos[t];
  const int* pages = block_table + (size_t)token_seq[t] * table_width;
  float* qs = lc_row + warp * E;
  const float* qrow = q + ((size_t)t * H + h) * E;
  for (int i = lane; i < E; i += 32) qs[i] = qrow[i];
  __syncwarp();
  float acc[OWN];
#pragma unroll
  for (int i = 0; i < OWN; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int base = 0; base <= p; base += 32) {
    const int j = base + lane;
    float s = -INFINITY;
    if (j <= p) {
      const TC* row = cache + cache_row_offset(pages[j / LLMX_PAGE], 0, j % LLMX_PAGE, 1, E);
      float dot = 0.f;
      for (int i = 0; i < E; ++i) dot += qs[i] * to_f32(row[i]);
      s = dot * scale;
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float corr = expf(m - m_new);
    const float e = j <= p ? expf(s - m_new) : 0.f;
    l = l * corr + warp_sum(e);
#pragma unroll
    for (int i = 0; i < OWN; ++i) acc[i] *= corr;
    const int n = min(32, p - base + 1);
    for (int jj = 0; jj < n; ++jj) {
      const float w = __shfl_sync(0xffffffffu, e, jj);
      const int key = base + jj;
      const TC* row = cache + cache_row_offset(pages[key / LLMX_PAGE], 0, key % LLMX_PAGE, 1, E);
#pragma unroll
      for (int i = 0; i < OWN; ++i) {
        const int d = lane + 32 * i;
        if (d < rank) acc[i] += w * to_f32(row[d]);
      }
    }
    m = m_new;
  }
  if (sinks) l += expf(sinks[h] - m);
  const float inv = 1.0f / l;
  float* o = lat + ((size_t)t * H + h) * rank;
#pragma unroll
  for (int i = 0; i < OWN; ++i) {
    const int d = lane + 32 * i;
    if (d < rank) o[d] = acc[i] * inv;
  }
}

LLMX_API int llmx_latent_paged(const float* q, float* lat, const void* cache, int cache_dtype, const int* block_table,
                               int table_width, const int* token_seq, const int* token_pos, const float* sinks, float scale,
                               int n_tokens, int H, int rank, int R, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || rank <= 0 || rank > LC_MAX_RANK_GENERAL || R < 0) return LLMX_REFUSED(1);
  const size_t smem = (size_t)4 * (rank + R) * sizeof(float);
  if (smem > 48 * 1024) return LLMX_REFUSED(3);
  const dim3 grid(n_tokens, (H + 3) / 4);
#define GO(TC, OWN)                                                                                                     \
  launch_pdl(latent_paged_kernel<TC, OWN>, grid, dim3(128), smem, stream, q, lat, (const TC*)cache, block_table,        \
             table_width, token_seq, token_pos, sinks, scale, H, rank, R)
#define CASE(TC)                        \
  do {                                  \
    if (rank <= 128) GO(TC, 4);         \
    else if (rank <= 256) GO(TC, 8);    \
    else if (rank <= 512) GO(TC, 16);   \
    else GO(TC, 32);                    \
  } while (0)
  if (cache_dtype == LLMX_F32) CASE(float);
  else if (cache_dtype == LLMX_BF16) CASE(bf16);
  else return LLMX_REFUSED(2);
#undef CASE
#undef GO
  return LLMX_LAUNCH_STATUS();
}

// ---------------------------------------------------------------------------
// Absorbed attention on the tensor cores.  grid (shares, ceil(H / 16), tokens), 4 warps and one that copies.  A CTA owns one token, 16 heads
// (the 16-wide M axis of mma.sync m16n8k16) and one share of the token's cached rows, which it walks in tiles of 32
// through a ring of shared-memory stages; a tile comes as one bulk copy per row, asked for by the fifth warp's lanes
// (rows padded by 16 bytes in shared memory: ldmatrix without conflicts; asking takes half as long as multiplying, so it
// is nobody else's work).
//   S = Q C^T     warp w: rows 8 w .. 8 w + 7 of the tile, all rank + R dims
//   O += P C      the warps share the latent's 16-dim blocks (block i belongs to warp i % 4), all 32 rows
// Maximum and probabilities pass between the warps through shared memory.
// ---------------------------------------------------------------------------
__device__ __forceinline__ void lc_bulk_copy(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst),
               "l"(src), "r"(bytes), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void lc_ldmatrix_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}
__device__ __forceinline__ void lc_ldmatrix_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void lc_ldmatrix_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2,
                                                     uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}

// A barrier of the four warps that multiply.
__device__ __forceinline__ void lc_sync_warps() { asm volatile("bar.sync 1, %0;" ::"n"(LC_WARPS * 32) : "memory"); }

#define LC_P_ROW (LC_TILE * 2 + 16)      // bytes of a row of probabilities

// NB: 16-dim blocks of the latent per warp, at most; STAGES: tiles in shared memory
template <int NB, int STAGES>
__global__ void __launch_bounds__(LC_WARPS * 32 + 32, 2)
latent_decode_kernel(const bf16* __restrict__ q, const bf16* __restrict__ cache, const int* __restrict__ block_table,
                     int table_width, const int* __restrict__ token_seq, const int* __restrict__ token_pos,
                     const int* __restrict__ seq_past, const float* __restrict__ sinks, float scale_log2, int H, int rank,
                     int R, int n_chunks, float* __restrict__ part_o, float* __restrict__ part_ml, bf16* __restrict__ lat,
                     int n_seqs, int n_pages) {
  extern __shared__ __align__(128) uint8_t lc_smem[];
  __shared__ float s_max[LC_WARPS][LC_HEADS], s_sum[LC_WARPS][LC_HEADS];
  __shared__ __align__(8) uint64_t lc_bars[STAGES + 1];              // one a stage, then the query's
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, tq = lane & 3;
  const int chunk = blockIdx.x, h0 = blockIdx.y * LC_HEADS, t = blockIdx.z;
  const int n_heads = min(LC_HEADS, H - h0), E = rank + R, pieces = E / 8;
  const int row_bytes = E * 2 + 16, tile_bytes = LC_TILE * row_bytes;
  const int b = token_seq[t], p = token_pos[t];
  if (b < 0 || b >= n_seqs || p < 0 || p / LLMX_PAGE >= table_width) {
    if (tid == 0) llmx_report(2);
    return;
  }
  const int* pages = block_table + (size_t)b * table_width;
  const int past = seq_past[b];
  const uint32_t sQ = (uint32_t)__cvta_generic_to_shared(lc_smem), sP = sQ + LC_HEADS * row_bytes;
  const uint32_t sT = sP + LC_HEADS * LC_P_ROW;
  uint8_t* pT = lc_smem + LC_HEADS * (row_bytes + LC_P_ROW);
  const int n_all = p / LC_TILE + 1, per = (n_all + n_chunks - 1) / n_chunks;
  const int lo = chunk * per, n_tiles = min(per, n_all - lo);           // <= 0: nothing to do
  const uint32_t bars = smem_u32(lc_bars), copy_bytes = (uint32_t)E * 2u;
  if (tid == 0) {
    for (int i = 0; i <= STAGES; ++i) mbar_init(bars + 8 * i, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  int next_page = 0;                                   // of the tile that load_tile is called for next
  if (warp == LC_WARPS && n_tiles > 0) next_page = pages[lo * LC_TILE / LLMX_PAGE];
  auto load_tile = [&](int i) {                        // the copying warp
    const int key0 = (lo + i) * LC_TILE, st = i % STAGES, valid = min(LC_TILE, p - key0 + 1);
    if (llmx_withhold && i == 0 && (blockIdx.x | blockIdx.y | blockIdx.z) == 0) return;      // (tests: never asked for)
    int page = next_page;                              // (a tile lies within one page)
    if (i + 1 < n_tiles) next_page = pages[(key0 + LC_TILE) / LLMX_PAGE];
    if (page < 0 || page >= n_pages) {
      if (lane == 0) llmx_report(2);
      page = 0;
    }
    const bf16* src = cache + cache_row_offset(page, 0, key0 % LLMX_PAGE, 1, E);
    if (lane == 0) mbar_expect_tx(bars + 8 * st, (uint32_t)valid * copy_bytes);
    __syncwarp();
    if (lane < valid)
      lc_bulk_copy(sT + (uint32_t)(st * tile_bytes + lane * row_bytes), src + (size_t)lane * E, copy_bytes, bars + 8 * st);
    // rows past the token's own were never written by it (or belong to nobody): weight 0, but 0 * NaN is NaN
    for (int r = valid; r < LC_TILE; ++r)
      for (int c = lane; c < pieces; c += 32)
        *reinterpret_cast<uint4*>(pT + st * tile_bytes + r * row_bytes + c * 16) = make_uint4(0u, 0u, 0u, 0u);
  };
  // Tiles wholly of earlier steps are complete: they start before the kernel ahead has ended.
  if (warp == LC_WARPS) {
    int issued = 0;
    for (; issued < STAGES - 1 && issued < n_tiles && (lo + issued + 1) * LC_TILE <= past; ++issued) load_tile(issued);
    pdl_wait();
    if (n_tiles > 0) {                 // the query tile; rows of missing heads hold anything and are not stored
      if (lane == 0) mbar_expect_tx(bars + 8 * STAGES, (uint32_t)n_heads * copy_bytes);
      __syncwarp();
      if (lane < n_heads)
        lc_bulk_copy(sQ + (uint32_t)(lane * row_bytes), q + ((size_t)t * H + h0 + lane) * E, copy_bytes, bars + 8 * STAGES);
    }
    for (; issued < STAGES - 1 && issued < n_tiles; ++issued) load_tile(issued);
    for (int i = 0; i < n_tiles; ++i) {
      if (!__syncthreads_and(1)) return;               // the tile before is done with: its stage takes the next one
      if (i + STAGES - 1 < n_tiles) load_tile(i + STAGES - 1);
    }
    return;
  }
  pdl_wait();

  const int n_blocks = rank / 16;
  float o[NB][2][4];
#pragma unroll
  for (int i = 0; i < NB; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;          // heads gq and gq + 8; l over this warp's rows
  const int ksteps = E / 16;
  const uint32_t q_addr = sQ + (uint32_t)((lane & 15) * row_bytes + (lane >> 4) * 16);
  for (int i = 0; i < n_tiles; ++i) {
    // the tile has landed (and, first, the query); everyone has left the tile before, whose stage the next copy fills
    bool ok = i > 0 || mbar_wait(bars + 8 * STAGES, 0);
    ok = ok && mbar_wait(bars + 8 * (i % STAGES), (i / STAGES) & 1);
    if (!__syncthreads_and(ok)) {
      if (tid == 0) llmx_report(4);
      return;
    }
    const uint32_t tile = sT + (uint32_t)((i % STAGES) * tile_bytes);
    const int key0 = (lo + i) * LC_TILE;
    // ---- scores of this warp's 8 rows: four chains of 16-dim steps
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f}, s3[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t k_addr = tile + (uint32_t)((warp * 8 + (lane & 7)) * row_bytes + (lane >> 3) * 16);
    // four steps' operands at a time, the next four asked for before these are multiplied
    uint32_t kb[2][8], qa[2][16];
    auto fetch = [&](int at, uint32_t* kf, uint32_t* qf) {
      lc_ldmatrix_x4(k_addr + at * 32, kf[0], kf[1], kf[2], kf[3]);
      lc_ldmatrix_x4(k_addr + at * 32 + 64, kf[4], kf[5], kf[6], kf[7]);
#pragma unroll
      for (int x = 0; x < 4; ++x)
        lc_ldmatrix_x4(q_addr + (at + x) * 32, qf[4 * x], qf[4 * x + 1], qf[4 * x + 2], qf[4 * x + 3]);
    };
    auto multiply = [&](const uint32_t* kf, const uint32_t* qf) {
      lc_mma(s0, qf[0], qf[1], qf[2], qf[3], kf[0], kf[1]);
      lc_mma(s1, qf[4], qf[5], qf[6], qf[7], kf[2], kf[3]);
      lc_mma(s2, qf[8], qf[9], qf[10], qf[11], kf[4], kf[5]);
      lc_mma(s3, qf[12], qf[13], qf[14], qf[15], kf[6], kf[7]);
    };
    const int quads = ksteps >> 2;
    if (quads > 0) fetch(0, kb[0], qa[0]);
    int g4 = 0;
    for (; g4 + 2 <= quads; g4 += 2) {
      fetch(4 * g4 + 4, kb[1], qa[1]);
      multiply(kb[0], qa[0]);
      if (g4 + 2 < quads) fetch(4 * g4 + 8, kb[0], qa[0]);
      multiply(kb[1], qa[1]);
    }
    if (g4 < quads) multiply(kb[0], qa[0]);
    for (int ks = quads * 4; ks < ksteps; ++ks) {
      uint32_t b0, b1, a0, a1, a2, a3;
      lc_ldmatrix_x2(tile + (uint32_t)((warp * 8 + (lane & 7)) * row_bytes + ((lane >> 3) & 1) * 16) + ks * 32, b0, b1);
      lc_ldmatrix_x4(q_addr + ks * 32, a0, a1, a2, a3);
      lc_mma(s0, a0, a1, a2, a3, b0, b1);
    }
    // the first block's latents for the second product, ahead of the probabilities
    uint32_t vb[2][8];
    auto fetch_v = [&](int blk, uint32_t* vf) {
      // transposed: (rows 0-7, dims lo), (rows 8-15, dims lo), (rows 0-7, dims hi), (rows 8-15, dims hi)
#pragma unroll
      for (int kk = 0; kk < 2; ++kk)
        lc_ldmatrix_x4_trans(tile + (uint32_t)((kk * 16 + (lane & 15)) * row_bytes + blk * 32 + (lane >> 4) * 16), vf[4 * kk],
                             vf[4 * kk + 1], vf[4 * kk + 2], vf[4 * kk + 3]);
    };
    if (warp < n_blocks) fetch_v(warp, vb[0]);
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool vis = key0 + warp * 8 + 2 * tq + e <= p;
      s0[e] = vis ? ((s0[e] + s1[e]) + (s2[e] + s3[e])) * scale_log2 : -INFINITY;
      s0[2 + e] = vis ? ((s0[2 + e] + s1[2 + e]) + (s2[2 + e] + s3[2 + e])) * scale_log2 : -INFINITY;
      mx0 = fmaxf(mx0, s0[e]);
      mx1 = fmaxf(mx1, s0[2 + e]);
    }
#pragma unroll
    for (int sh = 1; sh < 4; sh <<= 1) {
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, sh));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, sh));
    }
    if (tq == 0) s_max[warp][gq] = mx0, s_max[warp][gq + 8] = mx1;
    lc_sync_warps();
#pragma unroll
    for (int w = 0; w < LC_WARPS; ++w) mx0 = fmaxf(mx0, s_max[w][gq]), mx1 = fmaxf(mx1, s_max[w][gq + 8]);
    mx0 = fmaxf(mx0, m0);                              // a tile's first row is always seen
    mx1 = fmaxf(mx1, m1);
    const float c0 = ex2_approx(m0 - mx0), c1 = ex2_approx(m1 - mx1);
    const bool rescale = __any_sync(0xffffffffu, mx0 != m0 || mx1 != m1);      // some maximum has grown
    m0 = mx0;
    m1 = mx1;
    {
      const float e0 = ex2_approx(s0[0] - mx0), e1 = ex2_approx(s0[1] - mx0);
      const float e2 = ex2_approx(s0[2] - mx1), e3 = ex2_approx(s0[3] - mx1);
      l0 = l0 * c0 + (e0 + e1);
      l1 = l1 * c1 + (e2 + e3);
      __nv_bfloat162 pa = __floats2bfloat162_rn(e0, e1), pb = __floats2bfloat162_rn(e2, e3);
      uint8_t* prow = lc_smem + LC_HEADS * row_bytes + (warp * 8 + 2 * tq) * 2;
      *reinterpret_cast<__nv_bfloat162*>(prow + gq * LC_P_ROW) = pa;
      *reinterpret_cast<__nv_bfloat162*>(prow + (gq + 8) * LC_P_ROW) = pb;
    }
    lc_sync_warps();
    // ---- O = c O + P C
    uint32_t pf[2][4];
#pragma unroll
    for (int kk = 0; kk < 2; ++kk)
      lc_ldmatrix_x4(sP + (uint32_t)((lane & 15) * LC_P_ROW + kk * 32 + (lane >> 4) * 16), pf[kk][0], pf[kk][1], pf[kk][2],
                     pf[kk][3]);
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
      const int blk = warp + LC_WARPS * nb;
      if (blk < n_blocks) {
        if (nb + 1 < NB && blk + LC_WARPS < n_blocks) fetch_v(blk + LC_WARPS, vb[(nb + 1) & 1]);
        const uint32_t* vf = vb[nb & 1];
        if (rescale) {
#pragma unroll
          for (int j = 0; j < 2; ++j) o[nb][j][0] *= c0, o[nb][j][1] *= c0, o[nb][j][2] *= c1, o[nb][j][3] *= c1;
        }
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
          lc_mma(o[nb][0], pf[kk][0], pf[kk][1], pf[kk][2], pf[kk][3], vf[4 * kk], vf[4 * kk + 1]);
          lc_mma(o[nb][1], pf[kk][0], pf[kk][1], pf[kk][2], pf[kk][3], vf[4 * kk + 2], vf[4 * kk + 3]);
        }
      }
    }
  }
  lc_sync_warps();
  // ---- the sums of the four warps' rows
#pragma unroll
  for (int sh = 1; sh < 4; sh <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, sh);
    l1 += __shfl_xor_sync(0xffffffffu, l1, sh);
  }
  if (tq == 0) s_sum[warp][gq] = l0, s_sum[warp][gq + 8] = l1;
  lc_sync_warps();
  l0 = (s_sum[0][gq] + s_sum[1][gq]) + (s_sum[2][gq] + s_sum[3][gq]);
  l1 = (s_sum[0][gq + 8] + s_sum[1][gq + 8]) + (s_sum[2][gq + 8] + s_sum[3][gq + 8]);
  const bool live0 = gq < n_heads, live1 = gq + 8 < n_heads;
  if (n_chunks == 1) {
    if (sinks) {
      if (live0) l0 += exp2f(sinks[h0 + gq] * 1.4426950408889634f - m0);
      if (live1) l1 += exp2f(sinks[h0 + gq + 8] * 1.4426950408889634f - m1);
    }
    const float i0 = 1.0f / l0, i1 = 1.0f / l1;
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
      const int blk = warp + LC_WARPS * nb;
      if (blk >= n_blocks) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int d = blk * 16 + j * 8 + 2 * tq;
        if (live0)
          *reinterpret_cast<__nv_bfloat162*>(lat + ((size_t)t * H + h0 + gq) * rank + d) =
              __floats2bfloat162_rn(o[nb][j][0] * i0, o[nb][j][1] * i0);
        if (live1)
          *reinterpret_cast<__nv_bfloat162*>(lat + ((size_t)t * H + h0 + gq + 8) * rank + d) =
              __floats2bfloat162_rn(o[nb][j][2] * i1, o[nb][j][3] * i1);
      }
    }
    return;
  }
  const size_t u0 = ((size_t)t * H + h0 + gq) * n_chunks + chunk, u1 = ((size_t)t * H + h0 + gq + 8) * n_chunks + chunk;
  if (warp == 0 && tq == 0) {                          // (a share without rows: maximum -inf, sum 0, sums of latents 0)
    if (live0) part_ml[2 * u0] = m0, part_ml[2 * u0 + 1] = l0;
    if (live1) part_ml[2 * u1] = m1, part_ml[2 * u1 + 1] = l1;
  }
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) {
    const int blk = warp + LC_WARPS * nb;
    if (blk >= n_blocks) continue;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int d = blk * 16 + j * 8 + 2 * tq;
      if (live0) *reinterpret_cast<float2*>(part_o + u0 * rank + d) = make_float2(o[nb][j][0], o[nb][j][1]);
      if (live1) *reinterpret_cast<float2*>(part_o + u1 * rank + d) = make_float2(o[nb][j][2], o[nb][j][3]);
    }
  }
}

// out = sum_c 2^(m_c - m) O_c / (sum_c 2^(m_c - m) l_c + 2^(sink - m)), shares in order.  One CTA per (head, token).
__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                      const float* __restrict__ sinks, bf16* __restrict__ lat, int H, int rank, int n_chunks) {
  __shared__ float fac[LC_MAX_CHUNKS];
  __shared__ float inv;
  pdl_launch_dependents();
  const int h = blockIdx.x, t = blockIdx.y;
  const size_t u = ((size_t)t * H + h) * n_chunks;
  pdl_wait();
  if (threadIdx.x < 32) {
    float mx = -INFINITY, l = 0.f;
    for (int c = threadIdx.x; c < n_chunks; c += 32) mx = fmaxf(mx, part_ml[2 * (u + c)]);
    mx = warp_max(mx);
    for (int c = threadIdx.x; c < n_chunks; c += 32) {
      const float m = part_ml[2 * (u + c)], f = m == -INFINITY ? 0.f : exp2f(m - mx);
      fac[c] = f;
      l += f * part_ml[2 * (u + c) + 1];
    }
    l = warp_sum(l);
    if (sinks) l += exp2f(sinks[h] * 1.4426950408889634f - mx);
    if (threadIdx.x == 0) inv = 1.0f / l;
  }
  __syncthreads();
  for (int d = threadIdx.x * 4; d < rank; d += 512) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    const float* src = part_o + u * rank + d;
#pragma unroll 8
    for (int c = 0; c < n_chunks; ++c) {
      const float f = fac[c];
      const float4 v = *reinterpret_cast<const float4*>(src + (size_t)c * rank);
      a.x = fmaf(f, v.x, a.x);
      a.y = fmaf(f, v.y, a.y);
      a.z = fmaf(f, v.z, a.z);
      a.w = fmaf(f, v.w, a.w);
    }
    __nv_bfloat162 lo = __floats2bfloat162_rn(a.x * inv, a.y * inv), hi = __floats2bfloat162_rn(a.z * inv, a.w * inv);
    *reinterpret_cast<uint2*>(lat + ((size_t)t * H + h) * rank + d) =
        make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  }
}

// q bf16 [T, H, rank + R] = [ absorbed | rotated ], cache bf16 [pages, 64, rank + R], lat bf16 [T, H, rank]; every token
// t reads its sequence's rows 0 .. token_pos[t].  rank and R multiples of 16, rank <= 512.  n_chunks <= LC_MAX_CHUNKS shares;
// more than one: part_o float32 [T, H, n_chunks, rank], part_ml float32 [T, H, n_chunks, 2].
LLMX_API int llmx_latent_decode(const void* q, const void* cache, const int* block_table, int table_width,
                                const int* token_seq, const int* token_pos, const int* seq_past, const float* sinks,
                                float scale, int n_tokens, int H, int rank, int R, int n_chunks, float* part_o,
                                float* part_ml, void* lat, int n_seqs, long long n_pages, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || rank <= 0 || rank % 16 || rank > LC_MAX_RANK || R < 0 || R % 16 || n_chunks < 1 || n_chunks > LC_MAX_CHUNKS ||
      n_pages <= 0)
    return LLMX_REFUSED(1);
  if (n_chunks > 1 && (!part_o || !part_ml)) return LLMX_REFUSED(4);
  if (((uintptr_t)q | (uintptr_t)cache | (uintptr_t)lat | (uintptr_t)part_o) & 15) return LLMX_REFUSED(1);
  if (n_tokens > 65535) return LLMX_REFUSED(3);
  const int row_bytes = (rank + R) * 2 + 16;
  const size_t fixed = (size_t)LC_HEADS * (row_bytes + LC_P_ROW), tile = (size_t)LC_TILE * row_bytes;
  const int stages = fixed + 3 * tile <= 112 * 1024 ? 3 : 2;
  const size_t smem = fixed + stages * tile;
  if (smem > 220 * 1024) return LLMX_REFUSED(3);
  const dim3 grid(n_chunks, (H + LC_HEADS - 1) / LC_HEADS, n_tokens);
#define GO(NB, ST)                                                                                                       \
  do {                                                                                                                   \
    static bool attr_set = false;                                                                                        \
    if (!attr_set && smem > 48 * 1024) {                                                                                 \
      cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<NB, ST>, cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                           220 * 1024);                                                                  \
      if (e != cudaSuccess) return (int)e;                                                                               \
      attr_set = true;                                                                                                   \
    }                                                                                                                    \
    launch_pdl(latent_decode_kernel<NB, ST>, grid, dim3(LC_WARPS * 32 + 32), smem, stream, (const bf16*)q, (const bf16*)cache, \
               block_table, table_width, token_seq, token_pos, seq_past, sinks, scale * 1.4426950408889634f, H, rank, R, \
               n_chunks, part_o, part_ml, (bf16*)lat, n_seqs, (int)n_pages);                                             \
  } while (0)
#define GO_S(NB)               \
  do {                         \
    if (stages == 3) GO(NB, 3); \
    else GO(NB, 2);            \
  } while (0)
  if (rank <= 128) GO_S(2);
  else if (rank <= 256) GO_S(4);
  else GO_S(8);
#undef GO_S
#undef GO
  if (n_chunks > 1) {
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return (int)e;
    launch_pdl(latent_combine_kernel, dim3(H, n_tokens), dim3(128), 0, stream, (const float*)part_o, (const float*)part_ml,
               sinks, (bf16*)lat, H, rank, n_chunks);
  }
  return LLMX_LAUNCH_STATUS();
}

// ---------------------------------------------------------------------------
// Prompts: the step's sequences in scratch pages, sequence after sequence, each from a page's start.
// ---------------------------------------------------------------------------
// The sequence and its page that scratch page `slot` stands for; len: the sequence's positions after the step.
__device__ __forceinline__ bool lc_scratch_page(int slot, const int* seq_start, const int* seq_past, int n_seqs, int* seq,
                                                int* index, int* len) {
  int left = slot;
  for (int b = 0; b < n_seqs; ++b) {
    const int n = seq_past[b] + (seq_start[b + 1] - seq_start[b]), pages = (n + LLMX_PAGE - 1) / LLMX_PAGE;
    if (left < pages) {
      *seq = b, *index = left, *len = n;
      return true;
    }
    left -= pages;
  }
  return false;
}

// One CTA per scratch page: writes the page's entry of the scratch block table and copies its latents (without the
// rotated part) to rows 64 slot .. 64 slot + 63 of c_out [rows, rank]; rows past the sequence's end are zero.
template <bool VEC>
__global__ void __launch_bounds__(256)
latent_gather_kernel(const bf16* __restrict__ cache, const int* __restrict__ block_table, int table_width,
                     const int* __restrict__ seq_start, const int* __restrict__ seq_past, int n_seqs,
                     int* __restrict__ scratch_table, bf16* __restrict__ c_out, int rank, int R, int n_pages) {
  pdl_launch_dependents();
  const int slot = blockIdx.x;
  int b, index, len;
  if (!lc_scratch_page(slot, seq_start, seq_past, n_seqs, &b, &index, &len) || index >= table_width) {
    if (threadIdx.x == 0) llmx_report(3);
    return;
  }
  int page = block_table[(size_t)b * table_width + index];
  if (page < 0 || page >= n_pages) {
    if (threadIdx.x == 0) llmx_report(3);
    page = 0;
  }
  pdl_wait();
  if (threadIdx.x == 0) scratch_table[(size_t)b * table_width + index] = slot;
  const int E = rank + R, rows = min(LLMX_PAGE, len - index * LLMX_PAGE);
  const bf16* src = cache + (size_t)page * LLMX_PAGE * E;
  bf16* dst = c_out + (size_t)slot * LLMX_PAGE * rank;
  if (VEC) {
    const int pieces = rank / 8;
    for (int e = threadIdx.x; e < LLMX_PAGE * pieces; e += blockDim.x) {
      const int r = e / pieces, c = (e - r * pieces) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < rows) v = *reinterpret_cast<const uint4*>(src + (size_t)r * E + c);
      *reinterpret_cast<uint4*>(dst + (size_t)r * rank + c) = v;
    }
  } else {
    for (int e = threadIdx.x; e < LLMX_PAGE * rank; e += blockDim.x) {
      const int r = e / rank, c = e - r * rank;
      dst[e] = r < rows ? src[(size_t)r * E + c] : from_f32<bf16>(0.f);
    }
  }
}

// One CTA per (scratch page, head): k_out [pages, H, 64, R + D] = [ rotated part of the cached row | W_uk c ],
// v_out [pages, H, 64, Dv], out of kv [rows, H D + H Dv] (keys of every head, then values).
template <int V>
__global__ void __launch_bounds__(256)
latent_assemble_kernel(const bf16* __restrict__ kv, const bf16* __restrict__ cache, const int* __restrict__ block_table,
                       int table_width, const int* __restrict__ seq_start, const int* __restrict__ seq_past, int n_seqs,
                       bf16* __restrict__ k_out, bf16* __restrict__ v_out, int H, int D, int R, int Dv, int rank,
                       int n_pages) {
  pdl_launch_dependents();
  const int slot = blockIdx.x, h = blockIdx.y;
  int b, index, len;
  if (!lc_scratch_page(slot, seq_start, seq_past, n_seqs, &b, &index, &len) || index >= table_width) {
    if (threadIdx.x == 0) llmx_report(3);
    return;
  }
  int page = block_table[(size_t)b * table_width + index];
  if (page < 0 || page >= n_pages) {
    if (threadIdx.x == 0) llmx_report(3);
    page = 0;
  }
  pdl_wait();
  const int E = R + D, ld = rank + R, rows = min(LLMX_PAGE, len - index * LLMX_PAGE);
  const size_t kv_ld = (size_t)H * (D + Dv);
  const bf16* src = cache + (size_t)page * LLMX_PAGE * ld + rank;
  const bf16* kvr = kv + (size_t)slot * LLMX_PAGE * kv_ld;
  bf16* kd = k_out + ((size_t)slot * H + h) * LLMX_PAGE * E;
  bf16* vd = v_out + ((size_t)slot * H + h) * LLMX_PAGE * Dv;
  auto copy = [&](bf16* dst, const bf16* from, bool live) {
    if (V == 8) {
      uint4 x = make_uint4(0u, 0u, 0u, 0u);
      if (live) x = *reinterpret_cast<const uint4*>(from);
      *reinterpret_cast<uint4*>(dst) = x;
    } else {
      dst[0] = live ? from[0] : from_f32<bf16>(0.f);
    }
  };
  const int ek = E / V, ev = Dv / V;
  for (int e = threadIdx.x; e < LLMX_PAGE * ek; e += blockDim.x) {
    const int r = e / ek, c = (e - r * ek) * V;
    copy(kd + (size_t)r * E + c, c < R ? src + (size_t)r * ld + c : kvr + (size_t)r * kv_ld + (size_t)h * D + (c - R),
         r < rows);
  }
  for (int e = threadIdx.x; e < LLMX_PAGE * ev; e += blockDim.x) {
    const int r = e / ev, c = (e - r * ev) * V;
    copy(vd + (size_t)r * Dv + c, kvr + (size_t)r * kv_ld + (size_t)H * D + (size_t)h * Dv + c, r < rows);
  }
}

// n_scratch: pages of all the step's sequences together, each sequence's positions rounded up to whole pages.
LLMX_API int llmx_latent_gather(const void* cache, const int* block_table, int table_width, const int* seq_start,
                                const int* seq_past, int n_seqs, int n_scratch, int* scratch_table, void* c_out, int rank,
                                int R, long long n_pages, cudaStream_t stream) {
  if (n_scratch <= 0) return 0;
  if (rank <= 0 || R < 0 || n_seqs <= 0 || n_pages <= 0) return LLMX_REFUSED(1);
  const bool vec = rank % 8 == 0 && R % 8 == 0 && !(((uintptr_t)cache | (uintptr_t)c_out) & 15);
  if (vec)
    launch_pdl(latent_gather_kernel<true>, dim3(n_scratch), dim3(256), 0, stream, (const bf16*)cache, block_table,
               table_width, seq_start, seq_past, n_seqs, scratch_table, (bf16*)c_out, rank, R, (int)n_pages);
  else
    launch_pdl(latent_gather_kernel<false>, dim3(n_scratch), dim3(256), 0, stream, (const bf16*)cache, block_table,
               table_width, seq_start, seq_past, n_seqs, scratch_table, (bf16*)c_out, rank, R, (int)n_pages);
  return LLMX_LAUNCH_STATUS();
}

LLMX_API int llmx_latent_assemble(const void* kv, const void* cache, const int* block_table, int table_width,
                                  const int* seq_start, const int* seq_past, int n_seqs, int n_scratch, void* k_out,
                                  void* v_out, int H, int D, int R, int Dv, int rank, long long n_pages,
                                  cudaStream_t stream) {
  if (n_scratch <= 0) return 0;
  if (H <= 0 || H > 65535 || D <= 0 || R < 0 || Dv <= 0 || rank <= 0 || n_seqs <= 0 || n_pages <= 0) return LLMX_REFUSED(1);
  const bool vec = D % 8 == 0 && R % 8 == 0 && Dv % 8 == 0 && rank % 8 == 0 &&
                   !(((uintptr_t)kv | (uintptr_t)cache | (uintptr_t)k_out | (uintptr_t)v_out) & 15);
#define GO(V)                                                                                                           \
  launch_pdl(latent_assemble_kernel<V>, dim3(n_scratch, H), dim3(256), 0, stream, (const bf16*)kv, (const bf16*)cache,  \
             block_table, table_width, seq_start, seq_past, n_seqs, (bf16*)k_out, (bf16*)v_out, H, D, R, Dv, rank,      \
             (int)n_pages)
  if (vec) GO(8); else GO(1);
#undef GO
  return LLMX_LAUNCH_STATUS();
}
