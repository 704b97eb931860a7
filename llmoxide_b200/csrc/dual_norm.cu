// The residual add of a block whose two sublayers read the same stream, and the two norms of the next such block, in
// one pass over a row:
//
//   v = h[t,:] + sum_s a[s][t,:] + sum_s b[s][t,:] (+ bias)       the partials of each sublayer's result, in order
//   h[t,:] = v when write_h
//   n = v / sqrt(mean(v^2) + eps);  out0[r,:] = n * gain0;  out1[r,:] = n * gain1
//
// for output row r, t = rows ? rows[r] : r.  One root mean square serves both norms.  Either group of partials, the
// bias and the second output may be missing.  One CTA per row; a row of up to 8192 aligned floats stays in registers,
// any other is staged in shared memory.  Thread count and each thread's columns depend on d (and the pointers'
// alignment) alone, so a row's sums do not depend on the batch.  Everything is float32.
#include "common.cuh"

struct DnGroup {
  const void* p;          // null: no such group
  int n_split, is_bf16;
  size_t stride;
};

__device__ __forceinline__ float4 dn_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 dn_load4(const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void dn_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void dn_store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<uint32_t*>(&a);
  raw.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ void dn_add4(float4& v, const float4 y) { v.x += y.x, v.y += y.y, v.z += y.z, v.w += y.w; }

// v[c] += the group's partials in order, J partials of every vector of the thread in flight together
template <int NC, int J, typename TD>
__device__ __forceinline__ void dn_add_group(float4 (&v)[NC], const TD* p, int n_split, size_t stride, const int (&col)[NC],
                                             int d) {
  for (int s0 = 0; s0 < n_split; s0 += J) {
    float4 y[NC][J];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int j = 0; j < J; ++j)
        if (col[c] < d && s0 + j < n_split) y[c][j] = dn_load4(p + (size_t)(s0 + j) * stride + col[c]);
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int j = 0; j < J; ++j)
        if (col[c] < d && s0 + j < n_split) dn_add4(v[c], y[c][j]);
  }
}

// DEEP: a step of few rows and many partials (a decode step): their loads are batched and the gains fetched ahead of the
// wait; otherwise few registers, so that several rows share an SM.
template <typename TO, int NC, bool DEEP>
__global__ void __launch_bounds__(512)
dual_norm_kernel(float* __restrict__ h, const DnGroup ga, const DnGroup gb, const float* __restrict__ bias,
                 const int* __restrict__ rows, const float* __restrict__ gain0, const float* __restrict__ gain1, float eps,
                 TO* __restrict__ out0, TO* __restrict__ out1, int d, int write_h) {
  __shared__ float red[32];
  pdl_launch_dependents();
  const int r = blockIdx.x;
  const int t = rows ? rows[r] : r;                     // a step input, not a result of the kernel before
  float* hrow = h + (size_t)t * d;
  constexpr int J = !DEEP ? (NC == 1 ? 2 : 1) : NC == 1 ? 8 : NC == 2 ? 4 : 2;
  float4 v[NC], g0[NC], g1[NC];
  int col[NC];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    col[c] = (c * blockDim.x + threadIdx.x) * 4;
    const bool live = DEEP && col[c] < d;
    g0[c] = live && out0 ? dn_load4(gain0 + col[c]) : make_float4(0.f, 0.f, 0.f, 0.f);       // weights: ahead of the wait
    g1[c] = live && out1 ? dn_load4(gain1 + col[c]) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
#pragma unroll
  for (int c = 0; c < NC; ++c) v[c] = col[c] < d ? dn_load4(hrow + col[c]) : make_float4(0.f, 0.f, 0.f, 0.f);
  const size_t at = (size_t)t * d;
  auto add = [&](const DnGroup& g) {
    if (!g.p) return;
    if (g.is_bf16) dn_add_group<NC, J>(v, (const bf16*)g.p + at, g.n_split, g.stride, col, d);
    else dn_add_group<NC, J>(v, (const float*)g.p + at, g.n_split, g.stride, col, d);
  };
  add(ga);
  add(gb);
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    if (col[c] < d) {
      if (bias) dn_add4(v[c], dn_load4(bias + col[c]));
      if (write_h) dn_store4(hrow + col[c], v[c]);
    }
    ss += v[c].x * v[c].x;                              // (dead vectors are zero)
    ss += v[c].y * v[c].y;
    ss += v[c].z * v[c].z;
    ss += v[c].w * v[c].w;
  }
  if (!out0) return;                                    // only the sum was asked for (uniform)
  const float rs = 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps);
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    if (col[c] >= d) continue;
    if (!DEEP) {
      g0[c] = dn_load4(gain0 + col[c]);
      if (out1) g1[c] = dn_load4(gain1 + col[c]);
    }
    const float4 n = make_float4(v[c].x * rs, v[c].y * rs, v[c].z * rs, v[c].w * rs);
    dn_store4(out0 + (size_t)r * d + col[c], make_float4(n.x * g0[c].x, n.y * g0[c].y, n.z * g0[c].z, n.w * g0[c].w));
    if (out1) dn_store4(out1 + (size_t)r * d + col[c], make_float4(n.x * g1[c].x, n.y * g1[c].y, n.z * g1[c].z, n.w * g1[c].w));
  }
}

// Any width and alignment: one column a thread and step, the row staged in shared memory.
template <typename TO>
__global__ void __launch_bounds__(512)
dual_norm_any_kernel(float* __restrict__ h, const DnGroup ga, const DnGroup gb, const float* __restrict__ bias,
                     const int* __restrict__ rows, const float* __restrict__ gain0, const float* __restrict__ gain1,
                     float eps, TO* __restrict__ out0, TO* __restrict__ out1, int d, int write_h) {
  extern __shared__ float dn_row[];                     // [d]
  __shared__ float red[32];
  pdl_launch_dependents();
  const int r = blockIdx.x;
  const int t = rows ? rows[r] : r;
  float* hrow = h + (size_t)t * d;
  pdl_wait();
  float ss = 0.f;
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    float v = hrow[i];
    auto add = [&](const DnGroup& g) {
      if (!g.p) return;
      for (int s = 0; s < g.n_split; ++s) {
        const size_t at = (size_t)s * g.stride + (size_t)t * d + i;
        v += g.is_bf16 ? to_f32(((const bf16*)g.p)[at]) : ((const float*)g.p)[at];
      }
    };
    add(ga);
    add(gb);
    if (bias) v += bias[i];
    if (write_h) hrow[i] = v;
    dn_row[i] = v;
    ss += v * v;
  }
  if (!out0) return;
  const float rs = 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps);
  for (int i = threadIdx.x; i < d; i += blockDim.x) {   // (every thread takes the columns it staged itself)
    const float n = dn_row[i] * rs;
    out0[(size_t)r * d + i] = from_f32<TO>(n * gain0[i]);
    if (out1) out1[(size_t)r * d + i] = from_f32<TO>(n * gain1[i]);
  }
}

// h float32 [T, d]; a, b: null, or n_split partials [T, d] stride elements apart; bias: null or float32 [d]; rows:
// int32 [n_rows] or null (every row of h); out0 (with gain0), out1 (with gain1): [n_rows, d] or null, out1 only beside
// out0.
LLMX_API int llmx_dual_norm(float* h, const void* a, int dtype_a, int n_a, long long stride_a, const void* b, int dtype_b,
                            int n_b, long long stride_b, const float* bias, const int* rows, int n_rows,
                            const float* gain0, const float* gain1, float eps, void* out0, void* out1, int out_dtype, int d,
                            int write_h, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (d <= 0 || (a && n_a < 1) || (b && n_b < 1) || (out0 && !gain0) || (out1 && (!gain1 || !out0))) return LLMX_REFUSED(1);
  if ((a && dtype_a != LLMX_F32 && dtype_a != LLMX_BF16) || (b && dtype_b != LLMX_F32 && dtype_b != LLMX_BF16) ||
      (out0 && out_dtype != LLMX_F32 && out_dtype != LLMX_BF16))
    return LLMX_REFUSED(2);
  const DnGroup ga = {a, n_a, dtype_a == LLMX_BF16, (size_t)stride_a}, gb = {b, n_b, dtype_b == LLMX_BF16, (size_t)stride_b};
  auto aligned = [](const DnGroup& g) { return !g.p || (!((uintptr_t)g.p & (g.is_bf16 ? 7 : 15)) && g.stride % 4 == 0); };
  const uintptr_t outs = (uintptr_t)out0 | (uintptr_t)out1;
  const int vecs = d / 4;
  const bool vec = d % 4 == 0 && vecs <= 4 * 512 && aligned(ga) && aligned(gb) &&
                   !(((uintptr_t)h | (uintptr_t)bias | (uintptr_t)gain0 | (uintptr_t)gain1) & 15) &&
                   !(outs & (out_dtype == LLMX_F32 ? 15 : 7));
  const bool out_bf16 = out0 && out_dtype == LLMX_BF16;
#define ARGS(TO) h, ga, gb, bias, rows, gain0, gain1, eps, (TO*)out0, (TO*)out1, d, write_h
  if (vec) {
    const int nc = vecs <= 512 ? 1 : vecs <= 1024 ? 2 : 4;
    int threads = ((vecs + nc - 1) / nc + 31) / 32 * 32;
    if (threads < 64) threads = 64;
#define GO(TO, NC)                                                                                                \
  do {                                                                                                            \
    if (n_rows <= 64) launch_pdl(dual_norm_kernel<TO, NC, true>, dim3(n_rows), dim3(threads), 0, stream, ARGS(TO)); \
    else launch_pdl(dual_norm_kernel<TO, NC, false>, dim3(n_rows), dim3(threads), 0, stream, ARGS(TO));           \
  } while (0)
    if (out_bf16) {
      if (nc == 1) GO(bf16, 1); else if (nc == 2) GO(bf16, 2); else GO(bf16, 4);
    } else {
      if (nc == 1) GO(float, 1); else if (nc == 2) GO(float, 2); else GO(float, 4);
    }
#undef GO
    return LLMX_LAUNCH_STATUS();
  }
  const size_t smem = (size_t)d * sizeof(float);
  if (smem > 200 * 1024) return LLMX_REFUSED(3);
#define GO(TO)                                                                                                     \
  do {                                                                                                             \
    if (smem > 48 * 1024) {                                                                                        \
      cudaError_t e = cudaFuncSetAttribute(dual_norm_any_kernel<TO>, cudaFuncAttributeMaxDynamicSharedMemorySize,  \
                                           (int)smem);                                                             \
      if (e != cudaSuccess) return (int)e;                                                                         \
    }                                                                                                              \
    launch_pdl(dual_norm_any_kernel<TO>, dim3(n_rows), dim3(256), smem, stream, ARGS(TO));                         \
  } while (0)
  if (out_bf16) GO(bf16); else GO(float);
#undef GO
#undef ARGS
  return LLMX_LAUNCH_STATUS();
}
