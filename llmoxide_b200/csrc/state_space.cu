// The state-space recurrence of a Mamba-2 layer (T. Dao and A. Gu, "Transformers are SSMs: Generalized Models and
// Efficient Algorithms Through Structured State Space Duality"), with the short convolution in front of it and the gated
// norm behind it.
//
// A projected row holds [z: inner | x: inner | B: G N | C: G N | dt: H], inner = H P.  Per token, head h, group h / (H/G):
//   x, B, C = silu(conv(x, B, C) + conv_bias)        causal convolution over time per channel, zeros before the start
//   dt = softplus(dt + dt_bias),  a = exp(-exp(A_log) dt)
//   S <- a S + dt B x^T,   y = S^T C + D x           S [N, P] per head, starts at zero
//   y <- y silu(z);  out = y / sqrt(mean(y^2) + eps) * gain, the mean over each of `parts` equal runs of columns
//
// State of a sequence (float32): S of every head [H, N, P], then the convolution's rows as a ring of `taps` rows of
// C = inner + 2 G N channels: position p's projected row lies at row p % taps.  A token reads the taps - 1 rows before it
// and never the row it will occupy, so in a step of single tokens every CTA may write the new row at once.
//
// Prompts.  Chunks of 64 tokens, counted from a sequence's first token of the step.  With E the state a chunk starts
// from, gamma_i = a_0 .. a_i and L_ij = a_(j+1) .. a_i (L_ii = 1),
//   y_i = gamma_i (E^T C_i) + sum_(j<=i) L_ij (C_i . B_j) dt_j x_j + D x_i
//   E'  = gamma_63 E + sum_j L_63,j dt_j B_j x_j^T
// which is the recurrence written out as products of small matrices.  The decays enter as products of a, never as
// differences of logarithms, so a decay that underflows or is one loses nothing.
//   ss_prep    convolution, SiLU, dt and a, into float32 rows per head and group
//   ss_chunk   per (chunk, head): the chunk's own part of E'; per (chunk, group): the 64 x 64 products C_i . B_j
//   ss_pass    walks a sequence's chunks in order: leaves every chunk its E and the sequence its new state; moves the ring
//   ss_out     per (chunk, head): the outputs, times silu(z)
//   ss_norm    the norm
// The products run on the FMA units from tiles in shared memory, 8 x 8 results a thread: the recurrence is float32 by the
// design, which the tensor cores' formats are not.  Single tokens: ss_decode, one CTA per (sequence, head), S read and
// written once; then ss_norm.
//
// Everything is float32.  A prompt's sums are ordered by its chunks, so a position's result may differ in rounding between
// cuttings.
#include "common.cuh"

#define SS_CHUNK 64
#define SS_RUN 16                // tokens a thread of ss_prep walks
#define SS_MAX_TAPS 16
#define SS_LDM 68                // row stride of the masked 64 x 64 matrix in shared memory: 16-byte stores meet no bank twice

__device__ __forceinline__ float ss_silu(float x) { return __fdividef(x, 1.0f + expf(-x)); }   // (quotient within 2 ulp)
__device__ __forceinline__ float ss_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float4 ss_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void ss_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }

struct SsDims {
  int H, G, N, P, taps;
  __host__ __device__ int inner() const { return H * P; }
  __host__ __device__ int channels() const { return H * P + 2 * G * N; }
  __host__ __device__ int Np() const { return (N + 3) & ~3; }      // prepared rows are padded to four floats (zeros)
  __host__ __device__ int Pp() const { return (P + 3) & ~3; }
};
struct SsProj {                  // the projection: float32, n_split partials added in order
  const float* p;
  int n_split;
  size_t split_stride, row_stride;
  __device__ __forceinline__ float at(size_t t, int c) const {
    return split_value(p + t * row_stride, c, n_split, split_stride);
  }
};

// Slots of sequence b in units of `unit` tokens start at seq_start[b] / unit + b: the last b whose first slot is <= slot.
__device__ __forceinline__ int ss_find_seq(const int* seq_start, int n_seqs, int slot, int unit) {
  int lo = 0, hi = n_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (seq_start[mid] / unit + mid <= slot) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// ---------------------------------------------------------------------------
// One thread per channel and run of SS_RUN tokens of one sequence.  xs [T][H][Pp], bs and cs [T][G][Np], da [H][T] (a, dt).
// TAPS > 0: compiled for that many taps, the run's rows asked for together; 0: any number.  SPLIT: the projection comes as
// partials.
// ---------------------------------------------------------------------------
template <int TAPS, bool SPLIT>
__global__ void __launch_bounds__(128)
ss_prep_kernel(const SsProj proj, const SsDims dm, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
               const float* __restrict__ a_log, const float* __restrict__ dt_bias, const float* __restrict__ state,
               size_t slot_stride, size_t ring_off, float* __restrict__ xs, float* __restrict__ bs, float* __restrict__ cs,
               float2* __restrict__ da, const int* __restrict__ seq_start, const int* __restrict__ seq_past,
               const int* __restrict__ seq_slot, int n_seqs, int n_tokens, int n_slots) {
  pdl_launch_dependents();
  const int slot = blockIdx.x, C = dm.channels();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  const int b = ss_find_seq(seq_start, n_seqs, slot, SS_RUN);
  const int row0 = seq_start[b], n_new = seq_start[b + 1] - row0, p0 = seq_past[b], sl = seq_slot[b];
  const int first = (slot - (row0 / SS_RUN + b)) * SS_RUN;           // the run's first token within the sequence
  if (first >= n_new) return;                                        // (uniform) a slot no sequence fills
  if (first < 0 || row0 < 0 || row0 + n_new > n_tokens || p0 < 0 || sl < 0 || sl >= n_slots) {
    if (c == 0) llmx_report(1);
    return;
  }
  const int n = min(SS_RUN, n_new - first);
  auto proj_at = [&](int t, int c) { return SPLIT ? proj.at(t, c) : proj.p[(size_t)t * proj.row_stride + c]; };
  const int taps = TAPS > 0 ? TAPS : dm.taps;
  pdl_wait();
  if (c >= C + dm.H) return;
  if (c >= C) {                                                       // a head's step size and decay
    const int h = c - C;
    const float bias = dt_bias[h], rate = expf(a_log[h]);
    const int col = dm.inner() + C + h;
    float z[SS_RUN];
#pragma unroll
    for (int i = 0; i < SS_RUN; ++i) z[i] = i < n ? proj_at(row0 + first + i, col) : 0.f;
#pragma unroll
    for (int i = 0; i < SS_RUN; ++i)
      if (i < n) {
        const float dt = ss_softplus(z[i] + bias);
        da[(size_t)h * n_tokens + row0 + first + i] = make_float2(expf(-rate * dt), dt);
      }
    return;
  }
  const float* ring = state + (size_t)sl * slot_stride + ring_off;
  const int col = dm.inner() + c;
  auto u_at = [&](int i) {                                            // the projected row i tokens into the sequence's new ones
    if (i >= 0) return proj_at(row0 + i, col);
    return p0 + i >= 0 ? ring[(size_t)((p0 + i) % taps) * C + c] : 0.f;
  };
  float y[SS_RUN];
  const float bias = conv_b ? conv_b[c] : 0.f;
  if (TAPS > 0) {
    constexpr int NT = TAPS > 0 ? TAPS : 1;
    float u[SS_RUN + NT - 1];
#pragma unroll
    for (int r = 0; r < SS_RUN + NT - 1; ++r) u[r] = r - (NT - 1) < n ? u_at(first + r - (NT - 1)) : 0.f;
#pragma unroll
    for (int i = 0; i < SS_RUN; ++i) y[i] = bias;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const float w = conv_w[(size_t)j * C + c];
#pragma unroll
      for (int i = 0; i < SS_RUN; ++i) y[i] = fmaf(w, u[i + j], y[i]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < SS_RUN; ++i) {
      y[i] = bias;
      if (i < n)
        for (int j = 0; j < taps; ++j) y[i] = fmaf(conv_w[(size_t)j * C + c], u_at(first + i - taps + 1 + j), y[i]);
    }
  }
  // where the channel's values go: a head's x, or a group's B or C; the last of a row writes its padding too
  float* dst;
  size_t step;
  int at, size, padded;
  if (c < dm.inner()) {
    const int h = c / dm.P;
    at = c - h * dm.P, size = dm.P, padded = dm.Pp(), step = (size_t)dm.H * padded, dst = xs + (size_t)h * padded;
  } else {
    const int e = c - dm.inner(), gn = dm.G * dm.N, is_c = e >= gn, f = is_c ? e - gn : e, g = f / dm.N;
    at = f - g * dm.N, size = dm.N, padded = dm.Np(), step = (size_t)dm.G * padded;
    dst = (is_c ? cs : bs) + (size_t)g * padded;
  }
  dst += (size_t)(row0 + first) * step;
#pragma unroll
  for (int i = 0; i < SS_RUN; ++i)
    if (i < n) {
      dst[(size_t)i * step + at] = ss_silu(y[i]);
      if (at == size - 1)
        for (int e = size; e < padded; ++e) dst[(size_t)i * step + e] = 0.f;
    }
}

// ---------------------------------------------------------------------------
// acc[r][c] += sum_k A[k][row r] B[k][col c]: K rows of 64 results in shared memory, 64 threads, 8 x 8 results each, so that
// the four 16-byte reads a thread makes per k (512 bytes a warp each, 128 a cycle) last as long as its 64 multiply-adds.
// A thread's rows are i0 .. i0+3 and i0+32 .. i0+35, its columns j0 .. j0+3 and j0+32 .. j0+35: neighbouring lanes read
// neighbouring 16 bytes.
// ---------------------------------------------------------------------------
#define SS_THREADS 64
__device__ __forceinline__ int ss_row0() { return (threadIdx.x >> 3) * 4; }
__device__ __forceinline__ int ss_col0() { return (threadIdx.x & 7) * 4; }
// Two multiply-adds in one instruction, each rounded like fmaf: (d.x, d.y) += a * (b.x, b.y).
__device__ __forceinline__ void ss_fma2(float& dx, float& dy, float a, float bx, float by) {
  asm("{\n.reg .b64 va, vb, vd;\nmov.b64 va, {%2, %2};\nmov.b64 vb, {%3, %4};\nmov.b64 vd, {%0, %1};\n"
      "fma.rn.f32x2 vd, va, vb, vd;\nmov.b64 {%0, %1}, vd;\n}"
      : "+f"(dx), "+f"(dy)
      : "f"(a), "f"(bx), "f"(by));
}
// LOW false: only the rows from 32 on (a triangle's lower half has nothing above).
template <int UNROLL, bool LOW = true>
__device__ __forceinline__ void ss_product(float (&acc)[8][8], const float* A, int lda, const float* B, int ldb, int K) {
  const float* ap = A + ss_row0();
  const float* bp = B + ss_col0();
#pragma unroll UNROLL
  for (int k = 0; k < K; ++k) {
    const float4 a0 = LOW ? ss_load4(ap + k * lda) : make_float4(0.f, 0.f, 0.f, 0.f), a1 = ss_load4(ap + k * lda + 32);
    const float4 b0 = ss_load4(bp + k * ldb), b1 = ss_load4(bp + k * ldb + 32);
    const float av[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
    const float bv[8] = {b0.x, b0.y, b0.z, b0.w, b1.x, b1.y, b1.z, b1.w};
#pragma unroll
    for (int r = LOW ? 0 : 4; r < 8; ++r)
#pragma unroll
      for (int c = 0; c < 8; c += 2) ss_fma2(acc[r][c], acc[r][c + 1], av[r], bv[c], bv[c + 1]);
  }
}
__device__ __forceinline__ int ss_row(int i0, int r) { return i0 + (r & 3) + ((r & 4) << 3); }   // the r-th of a thread's rows
__device__ __forceinline__ void ss_copy16(float* dst, const float* src, bool live) {             // 16 bytes, or zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src),
               "r"(live ? 16 : 0)
               : "memory");
}
__device__ __forceinline__ void ss_copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ss_copy_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// The chunk of a slot: its sequence, first token, number of tokens (0: none) and number within the sequence.
struct SsChunk {
  int b, t0, n, index;
};
__device__ __forceinline__ SsChunk ss_chunk_of(const int* seq_start, int n_seqs, int n_tokens, int slot) {
  SsChunk k;
  k.b = ss_find_seq(seq_start, n_seqs, slot, SS_CHUNK);
  const int row0 = seq_start[k.b], n_new = seq_start[k.b + 1] - row0;
  k.index = slot - (row0 / SS_CHUNK + k.b);
  k.t0 = row0 + k.index * SS_CHUNK;
  k.n = min(SS_CHUNK, n_new - k.index * SS_CHUNK);
  if (k.index < 0 || row0 < 0 || row0 + n_new > n_tokens) k.n = 0;    // (ss_prep has reported it)
  return k;
}

// st [slots][H][N][Pp]: the chunk's own part of its last state; at [slots][H]: gamma of its last token; cb [slots][G][64][64]:
// C_i . B_j at row j, column i.
__global__ void __launch_bounds__(SS_THREADS)
ss_chunk_kernel(const float* __restrict__ xs, const float* __restrict__ bs, const float* __restrict__ cs,
                const float2* __restrict__ da, float* __restrict__ st, float* __restrict__ at, float* __restrict__ cb,
                const int* __restrict__ seq_start, int n_seqs, int n_tokens, const SsDims dm) {
  __shared__ __align__(16) float As[64 * 64];
  __shared__ __align__(16) float Bs[64 * 64];
  __shared__ float ws[SS_CHUNK];
  pdl_launch_dependents();
  const int tid = threadIdx.x, slot = blockIdx.x;
  const SsChunk ck = ss_chunk_of(seq_start, n_seqs, n_tokens, slot);
  if (ck.n <= 0) return;                               // (uniform)
  const int Np = dm.Np(), Pp = dm.Pp();
  const int p_tiles = (Pp + 63) >> 6, tiles = ((dm.N + 63) >> 6) * p_tiles;
  float acc[8][8];
#pragma unroll
  for (int r = 0; r < 8; ++r)
#pragma unroll
    for (int c = 0; c < 8; ++c) acc[r][c] = 0.f;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const int i0 = ss_row0(), j0 = ss_col0();
  pdl_wait();
  if ((int)blockIdx.y < dm.H * tiles) {
    const int h = blockIdx.y / tiles, tl = blockIdx.y - h * tiles;
    const int n0 = (tl / p_tiles) * 64, c0 = (tl % p_tiles) * 64;
    const int g = h / (dm.H / dm.G);
    // 16 lanes a row: x goes straight to shared memory, B through registers, where it takes its token's weight
    const int lr = tid >> 4, lc = (tid & 15) * 4;
    const float* brow = bs + ((size_t)ck.t0 * dm.G + g) * Np + n0 + lc;
    const float* xrow = xs + ((size_t)ck.t0 * dm.H + h) * Pp + c0 + lc;
    const bool b_live = n0 + lc < Np, x_live = c0 + lc < Pp;
#pragma unroll
    for (int m = 0; m < 16; ++m) {
      const int j = lr + 4 * m;
      const bool live = x_live && j < ck.n;
      ss_copy16(Bs + j * 64 + lc, live ? xrow + (size_t)j * dm.H * Pp : xs, live);
    }
    ss_copy_commit();
    float4 bv[16];
#pragma unroll
    for (int m = 0; m < 16; ++m) {
      const int j = lr + 4 * m;
      bv[m] = b_live && j < ck.n ? ss_load4(brow + (size_t)j * dm.G * Np) : zero;
    }
    if (tid < 32) {
      // w_j = (a_(j+1) .. a_last) dt_j, two tokens a lane, by a suffix product over the warp
      const float2* dp = da + (size_t)h * n_tokens + ck.t0;
      const float2 e0 = 2 * tid < ck.n ? dp[2 * tid] : make_float2(1.f, 0.f);
      const float2 e1 = 2 * tid + 1 < ck.n ? dp[2 * tid + 1] : make_float2(1.f, 0.f);
      float v = e0.x * e1.x;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_down_sync(0xffffffffu, v, o);
        if (tid + o < 32) v *= y;
      }
      float after = __shfl_down_sync(0xffffffffu, v, 1);
      if (tid == 31) after = 1.f;
      ws[2 * tid + 1] = after * e1.y;
      ws[2 * tid] = after * e1.x * e0.y;
      if (tid == 0 && tl == 0) at[(size_t)slot * dm.H + h] = v;
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < 16; ++m) {
      const int j = lr + 4 * m;
      const float w = ws[j];
      ss_store4(As + j * 64 + lc, make_float4(bv[m].x * w, bv[m].y * w, bv[m].z * w, bv[m].w * w));
    }
    ss_copy_wait<0>();
    __syncthreads();
    ss_product<4>(acc, As, 64, Bs, 64, (ck.n + 3) & ~3);   // (rows past the chunk's tokens are zero)
    float* dst = st + ((size_t)slot * dm.H + h) * dm.N * Pp + c0 + j0;
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const int n = n0 + ss_row(i0, r);
      if (n >= dm.N) continue;
      if (c0 + j0 < Pp) ss_store4(dst + (size_t)n * Pp, make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]));
      if (c0 + j0 + 32 < Pp) ss_store4(dst + (size_t)n * Pp + 32, make_float4(acc[r][4], acc[r][5], acc[r][6], acc[r][7]));
    }
    return;
  }
  // ---- C_i . B_j of a group: both operands are turned so that a row of shared memory holds one dim of all tokens
  const int g = blockIdx.y - dm.H * tiles;
  const float* crow = cs + ((size_t)(ck.t0 + tid) * dm.G + g) * Np;
  const float* brow = bs + ((size_t)(ck.t0 + tid) * dm.G + g) * Np;
  const bool live = tid < ck.n;
  for (int kb = 0; kb < Np; kb += 32) {
    float4 cv[8], bv[8];
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      cv[m] = live && kb + 4 * m < Np ? ss_load4(crow + kb + 4 * m) : zero;
      bv[m] = live && kb + 4 * m < Np ? ss_load4(brow + kb + 4 * m) : zero;
    }
    __syncthreads();                                   // (the tiles of the block before have been read)
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      float* ap = As + 4 * m * 64 + tid;
      float* bp = Bs + 4 * m * 64 + tid;
      ap[0] = cv[m].x, ap[64] = cv[m].y, ap[128] = cv[m].z, ap[192] = cv[m].w;
      bp[0] = bv[m].x, bp[64] = bv[m].y, bp[128] = bv[m].z, bp[192] = bv[m].w;
    }
    __syncthreads();
    ss_product<4>(acc, As, 64, Bs, 64, min(32, Np - kb));
  }
  float* dst = cb + ((size_t)slot * dm.G + g) * 4096;
#pragma unroll
  for (int c = 0; c < 8; ++c) {
    float* row = dst + ss_row(j0, c) * 64 + i0;
    ss_store4(row, make_float4(acc[0][c], acc[1][c], acc[2][c], acc[3][c]));
    ss_store4(row + 32, make_float4(acc[4][c], acc[5][c], acc[6][c], acc[7][c]));
  }
}

// Every four elements of a sequence's state, one thread: E_0 is the stored state, E_(c+1) = at_c E_c + st_c; st_c becomes
// E_c, the stored state the last E.  CTAs behind those move the convolution's ring on, a channel a thread.
__global__ void __launch_bounds__(256)
ss_pass_kernel(const SsProj proj, const SsDims dm, float* __restrict__ st, const float* __restrict__ at,
               float* __restrict__ state, size_t slot_stride, size_t ring_off, const int* __restrict__ seq_start,
               const int* __restrict__ seq_past, const int* __restrict__ seq_slot, int n_tokens, int n_slots,
               int state_blocks) {
  pdl_launch_dependents();
  const int b = blockIdx.y;
  const int row0 = seq_start[b], n_new = seq_start[b + 1] - row0, p0 = seq_past[b], sl = seq_slot[b];
  if (row0 < 0 || n_new <= 0 || row0 + n_new > n_tokens || p0 < 0 || sl < 0 || sl >= n_slots) {
    if (threadIdx.x == 0) llmx_report(2);
    return;
  }
  pdl_wait();
  float* base = state + (size_t)sl * slot_stride;
  if ((int)blockIdx.x >= state_blocks) {
    const int c = (blockIdx.x - state_blocks) * 256 + threadIdx.x, C = dm.channels();
    if (c >= C) return;
    float* ring = base + ring_off;
    for (int i = max(0, n_new - dm.taps); i < n_new; ++i)
      ring[(size_t)((p0 + i) % dm.taps) * C + c] = proj.at(row0 + i, dm.inner() + c);
    return;
  }
  const int Pp = dm.Pp(), p4 = Pp >> 2;
  const size_t per_head = (size_t)dm.N * p4;
  const size_t idx = (size_t)blockIdx.x * 256 + threadIdx.x;
  if (idx >= per_head * dm.H) return;
  const int h = (int)(idx / per_head), n = (int)((idx - h * per_head) / p4), p = (int)(idx % p4) * 4;
  const int chunks = (n_new + SS_CHUNK - 1) / SS_CHUNK, slot0 = row0 / SS_CHUNK + b;
  float* sp = base + ((size_t)h * dm.N + n) * dm.P + p;
  const bool vec = (dm.P & 3) == 0;
  float4 e;
  if (vec) e = ss_load4(sp);
  else e = make_float4(sp[0], p + 1 < dm.P ? sp[1] : 0.f, p + 2 < dm.P ? sp[2] : 0.f, p + 3 < dm.P ? sp[3] : 0.f);
  const size_t step = (size_t)dm.H * dm.N * Pp;
  float* cp = st + (size_t)slot0 * step + ((size_t)h * dm.N + n) * Pp + p;
  const float* ap = at + (size_t)slot0 * dm.H + h;
  for (int c0 = 0; c0 < chunks; c0 += 4) {              // four chunks' parts in flight
    float4 s[4];
    float a[4];
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (c0 + u < chunks) s[u] = ss_load4(cp + (size_t)(c0 + u) * step), a[u] = ap[(size_t)(c0 + u) * dm.H];
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (c0 + u < chunks) {
        ss_store4(cp + (size_t)(c0 + u) * step, e);
        e = make_float4(fmaf(a[u], e.x, s[u].x), fmaf(a[u], e.y, s[u].y), fmaf(a[u], e.z, s[u].z), fmaf(a[u], e.w, s[u].w));
      }
  }
  if (vec) {
    ss_store4(sp, e);
  } else {
    sp[0] = e.x;
    if (p + 1 < dm.P) sp[1] = e.y;
    if (p + 2 < dm.P) sp[2] = e.z;
    if (p + 3 < dm.P) sp[3] = e.w;
  }
}

// y [T][inner] = (recurrence's output + D x) silu(z), 64 tokens x 64 columns of a head per CTA.
__global__ void __launch_bounds__(SS_THREADS)
ss_out_kernel(const SsProj proj, const SsDims dm, const float* __restrict__ xs, const float* __restrict__ cs,
              const float2* __restrict__ da, const float* __restrict__ st, const float* __restrict__ cb,
              const float* __restrict__ skip, float* __restrict__ y, const int* __restrict__ seq_start, int n_seqs,
              int n_tokens) {
  __shared__ __align__(16) float Ms[64 * SS_LDM];      // row j: L_ij (C_i . B_j) dt_j over i; before that the turned C
  __shared__ __align__(16) float Bs[2][32 * 64];       // rows of E, then of x
  __shared__ float a_s[SS_CHUNK], gamma[SS_CHUNK];
  pdl_launch_dependents();
  const int tid = threadIdx.x, slot = blockIdx.x;
  const SsChunk ck = ss_chunk_of(seq_start, n_seqs, n_tokens, slot);
  if (ck.n <= 0) return;                               // (uniform)
  const int Np = dm.Np(), Pp = dm.Pp(), p_tiles = (Pp + 63) >> 6;
  const int h = blockIdx.y / p_tiles, c0 = (blockIdx.y - h * p_tiles) * 64;
  const int g = h / (dm.H / dm.G);
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  pdl_wait();
  const int lr = tid >> 4, lc = (tid & 15) * 4;        // a row of E or x: 16 lanes
  const bool col_live = c0 + lc < Pp;
  const float* e_base = st + ((size_t)slot * dm.H + h) * dm.N * Pp + c0 + lc;
  const float* x_base = xs + ((size_t)ck.t0 * dm.H + h) * Pp + c0 + lc;
  const float* crow = cs + ((size_t)(ck.t0 + tid) * dm.G + g) * Np;
  const int e_steps = (dm.N + 31) >> 5, steps = e_steps + ((ck.n + 31) >> 5);
  auto copy_rows = [&](int step) {                      // 32 rows of E, then of x, into one of two buffers
    float* dst = Bs[step & 1] + lc;
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      const int r = lr + 4 * m, k = (step < e_steps ? step : step - e_steps) * 32 + r;
      const bool live = col_live && (step < e_steps ? k < dm.N : k < ck.n);
      const float* src = step < e_steps ? e_base + (size_t)k * Pp : x_base + (size_t)k * dm.H * Pp;
      ss_copy16(dst + r * 64, live ? src : xs, live);
    }
    ss_copy_commit();
  };
  float4 cv[8];
  auto fetch_c = [&](int kb) {
#pragma unroll
    for (int m = 0; m < 8; ++m) cv[m] = tid < ck.n && kb + 4 * m < Np ? ss_load4(crow + kb + 4 * m) : zero;
  };
  copy_rows(0);
  fetch_c(0);
  const float2 own = tid < ck.n ? da[(size_t)h * n_tokens + ck.t0 + tid] : make_float2(1.f, 0.f);    // this token's a and dt
  a_s[tid] = own.x;
  float acc[8][8];
#pragma unroll
  for (int r = 0; r < 8; ++r)
#pragma unroll
    for (int c = 0; c < 8; ++c) acc[r][c] = 0.f;
  const int i0 = ss_row0(), j0 = ss_col0();
  // ---- E^T C_i
  for (int s = 0; s < e_steps; ++s) {
    float* As = Ms + (s & 1) * 32 * 64;
#pragma unroll
    for (int m = 0; m < 8; ++m) {                      // C turned: a row of shared memory holds one dim of all tokens
      float* ap = As + 4 * m * 64 + tid;
      ap[0] = cv[m].x, ap[64] = cv[m].y, ap[128] = cv[m].z, ap[192] = cv[m].w;
    }
    ss_copy_wait<0>();
    __syncthreads();                                   // (and every thread is done with the tiles of the step before)
    copy_rows(s + 1);
    if (s + 1 < e_steps) fetch_c((s + 1) * 32);
    ss_product<2>(acc, As, 64, Bs[s & 1], 64, min(32, Np - s * 32));
  }
  __syncthreads();                                     // the turned C has been read: its place takes the masked matrix
  if (tid < 32) {                                      // gamma, two tokens a lane, by a prefix product over the warp
    const float a0 = a_s[2 * tid], a1 = a_s[2 * tid + 1];
    float v = a0 * a1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float u = __shfl_up_sync(0xffffffffu, v, o);
      if (tid >= o) v *= u;
    }
    float before = __shfl_up_sync(0xffffffffu, v, 1);
    if (tid == 0) before = 1.f;
    gamma[2 * tid] = before * a0;
    gamma[2 * tid + 1] = before * a0 * a1;
  }
  {
    // L_ij by multiplying a along i, a thread a column j; what lies above the diagonal is zero
    const float* cbj = cb + (((size_t)slot * dm.G + g) * 64 + tid) * 64;
    float L = own.y;                                   // (dt_j rides on it)
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      float4 d[4];
#pragma unroll
      for (int m = 0; m < 4; ++m) d[m] = 16 * q + 15 >= tid ? ss_load4(cbj + 16 * q + 4 * m) : zero;
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        float o[4] = {d[m].x, d[m].y, d[m].z, d[m].w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = 16 * q + 4 * m + e;
          if (i > tid) L *= a_s[i];
          o[e] = i >= tid ? o[e] * L : 0.f;
        }
        ss_store4(Ms + tid * SS_LDM + 16 * q + 4 * m, make_float4(o[0], o[1], o[2], o[3]));
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    const float ga = gamma[ss_row(i0, r)];
#pragma unroll
    for (int c = 0; c < 8; ++c) acc[r][c] *= ga;
  }
  // ---- + sum over the chunk's own tokens
  for (int s = e_steps; s < steps; ++s) {
    ss_copy_wait<0>();
    __syncthreads();
    if (s + 1 < steps) copy_rows(s + 1);
    const int jb = (s - e_steps) * 32;
    if (jb == 0) ss_product<2>(acc, Ms, SS_LDM, Bs[s & 1], 64, min(32, ck.n));
    else ss_product<2, false>(acc, Ms + jb * SS_LDM, SS_LDM, Bs[s & 1], 64, ck.n - jb);      // (they reach rows 32.. only)
  }
  // ---- + D x, times silu(z)
  const int inner = dm.inner();
  const float dsk = skip[h];
  const bool vec = (dm.P & 3) == 0 && (proj.row_stride & 3) == 0 && (proj.split_stride & 3) == 0;
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    const int i = ss_row(i0, r);
    if (i >= ck.n) continue;
    const size_t t = (size_t)(ck.t0 + i);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int p = c0 + j0 + 32 * half;
      if (p >= dm.P) continue;
      const float4 x = ss_load4(xs + (t * dm.H + h) * Pp + p);
      const float* ar = acc[r] + 4 * half;
      float v[4] = {fmaf(dsk, x.x, ar[0]), fmaf(dsk, x.y, ar[1]), fmaf(dsk, x.z, ar[2]), fmaf(dsk, x.w, ar[3])};
      float* dst = y + t * inner + (size_t)h * dm.P + p;
      if (vec) {
        const float* zp = proj.p + t * proj.row_stride + h * dm.P + p;
        float4 z = ss_load4(zp);
        for (int q = 1; q < proj.n_split; ++q) {
          const float4 u = ss_load4(zp + (size_t)q * proj.split_stride);
          z.x += u.x, z.y += u.y, z.z += u.z, z.w += u.w;
        }
        ss_store4(dst, make_float4(v[0] * ss_silu(z.x), v[1] * ss_silu(z.y), v[2] * ss_silu(z.z), v[3] * ss_silu(z.w)));
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (p + c < dm.P) dst[c] = v[c] * ss_silu(proj.at(t, h * dm.P + p + c));
      }
    }
  }
}

// out[t] = y[t] / sqrt(mean(y^2) + eps) * gain over every one of `parts` equal runs of the row; a CTA per (token, run).
template <typename TO>
__global__ void __launch_bounds__(256)
ss_norm_kernel(const float* __restrict__ y, const float* __restrict__ gain, float eps, TO* __restrict__ out, int width,
               int parts) {
  __shared__ float red[32];
  pdl_launch_dependents();
  const size_t at = ((size_t)blockIdx.x * parts + blockIdx.y) * width;
  const float* yp = y + at;
  const float* gp = gain + (size_t)blockIdx.y * width;
  TO* op = out + at;
  pdl_wait();
  const bool vec = (width & 3) == 0;                    // (then every run starts on a 16-byte boundary)
  float ss = 0.f;
  if (vec) {
    for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
      const float4 v = ss_load4(yp + i);
      ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) ss += yp[i] * yp[i];
  }
  const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
  if (vec) {
    for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
      const float4 v = ss_load4(yp + i), g = ss_load4(gp + i);
      const float o[4] = {(v.x * r) * g.x, (v.y * r) * g.y, (v.z * r) * g.z, (v.w * r) * g.w};
      if constexpr (sizeof(TO) == 4) {
        ss_store4(op + i, make_float4(o[0], o[1], o[2], o[3]));
      } else {
        __nv_bfloat162 a = __floats2bfloat162_rn(o[0], o[1]), b = __floats2bfloat162_rn(o[2], o[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&a);
        raw.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(op + i) = raw;
      }
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) op[i] = from_f32<TO>((yp[i] * r) * gp[i]);
  }
}

// ---------------------------------------------------------------------------
// One token of a sequence, one CTA per (head, sequence).  A thread owns V columns of S and every R-th of its rows; the
// first eight of those are asked for before anything else.  y [B][inner] as ss_out leaves it.
// ---------------------------------------------------------------------------
template <int V>
__device__ __forceinline__ void ss_loadv(const float* p, float (&o)[V]) {
  if constexpr (V == 4) {
    const float4 v = ss_load4(p);
    o[0] = v.x, o[1] = v.y, o[2] = v.z, o[3] = v.w;
  } else {
    o[0] = p[0];
  }
}

template <int V>
__global__ void __launch_bounds__(256, 4)
ss_decode_kernel(const SsProj proj, const SsDims dm, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                 const float* __restrict__ a_log, const float* __restrict__ dt_bias, const float* __restrict__ skip,
                 float* __restrict__ state, size_t slot_stride, size_t ring_off, float* __restrict__ y,
                 const int* __restrict__ seq_past, const int* __restrict__ seq_slot, int n_slots) {
  extern __shared__ __align__(16) float ss_smem[];
  constexpr int U = 8;
  pdl_launch_dependents();
  const int tid = threadIdx.x, h = blockIdx.x, b = blockIdx.y;
  const int N = dm.N, P = dm.P, Pp = dm.Pp(), C = dm.channels(), inner = dm.inner(), taps = dm.taps;
  const int per_group = dm.H / dm.G, g = h / per_group;
  float* x_s = ss_smem;                                 // [Pp]
  float* b_s = x_s + Pp;                                // [N]
  float* c_s = b_s + N;                                 // [N]
  float* red = c_s + N + (-(2 * N) & 3);                // [R][Pp]
  const int pos = seq_past[b], sl = seq_slot[b];
  if (pos < 0 || sl < 0 || sl >= n_slots) {
    if (tid == 0) llmx_report(3);
    return;
  }
  const int cols = P / V, R = 256 / cols;               // (cols <= 256)
  const int nr = tid / cols, pc = (tid - nr * cols) * V;
  const bool live = nr < R;
  float* base = state + (size_t)sl * slot_stride;
  float* S = base + (size_t)h * N * P + pc;
  float* ring = base + ring_off;
  pdl_wait();
  float s[U][V];
#pragma unroll
  for (int u = 0; u < U; ++u)
    if (live && nr + u * R < N) ss_loadv<V>(S + (size_t)(nr + u * R) * P, s[u]);
  for (int idx = tid; idx < P + 2 * N; idx += 256) {    // the head's x, its group's B and C
    const int c = idx < P ? h * P + idx : idx < P + N ? inner + g * N + idx - P : inner + dm.G * N + g * N + idx - P - N;
    const float u = proj.at(b, inner + c);
    float v = conv_b ? conv_b[c] : 0.f;
    for (int j = 0; j < taps - 1; ++j) {
      const int p = pos - taps + 1 + j;
      if (p >= 0) v = fmaf(conv_w[(size_t)j * C + c], ring[(size_t)(p % taps) * C + c], v);
    }
    v = fmaf(conv_w[(size_t)(taps - 1) * C + c], u, v);
    if (idx < P || h % per_group == 0) ring[(size_t)(pos % taps) * C + c] = u;
    v = ss_silu(v);
    if (idx < P) x_s[idx] = v;
    else if (idx < P + N) b_s[idx - P] = v;
    else c_s[idx - P - N] = v;
  }
  const float dt = ss_softplus(proj.at(b, inner + C + h) + dt_bias[h]);
  const float a = expf(-expf(a_log[h]) * dt);
  __syncthreads();
  if (live) {
    float xd[V], acc[V];
#pragma unroll
    for (int e = 0; e < V; ++e) xd[e] = x_s[pc + e] * dt, acc[e] = 0.f;
    for (int n0 = nr; n0 < N; n0 += U * R) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int n = n0 + u * R;
        if (n < N) {
          if (n0 > nr) ss_loadv<V>(S + (size_t)n * P, s[u]);
          const float bn = b_s[n], cn = c_s[n];
#pragma unroll
          for (int e = 0; e < V; ++e) {
            s[u][e] = fmaf(a, s[u][e], bn * xd[e]);
            acc[e] = fmaf(cn, s[u][e], acc[e]);
          }
          if constexpr (V == 4) ss_store4(S + (size_t)n * P, make_float4(s[u][0], s[u][1], s[u][2], s[u][3]));
          else S[(size_t)n * P] = s[u][0];
        }
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) red[nr * Pp + pc + e] = acc[e];
  }
  __syncthreads();
  for (int p = tid; p < P; p += 256) {
    float v = 0.f;
    for (int r = 0; r < R; ++r) v += red[r * Pp + p];
    v = fmaf(skip[h], x_s[p], v);
    y[(size_t)b * inner + (size_t)h * P + p] = v * ss_silu(proj.at(b, h * P + p));
  }
}

// ---------------------------------------------------------------------------
static int ss_check(const SsDims& dm, long long row_stride, int n_split, long long slot_stride, long long ring_off,
                    const float* state, int n_seqs) {
  if (dm.H <= 0 || dm.G <= 0 || dm.H % dm.G || dm.N <= 0 || dm.P <= 0 || dm.P > 256 || dm.N > 1024 || n_split < 1)
    return LLMX_REFUSED(1);
  if (dm.taps < 1 || dm.taps > SS_MAX_TAPS || row_stride < dm.inner() + dm.channels() + dm.H) return LLMX_REFUSED(1);
  if (ring_off < (long long)dm.H * dm.N * dm.P || slot_stride < ring_off + (long long)dm.taps * dm.channels() ||
      (slot_stride & 3) || ((uintptr_t)state & 15) || n_seqs > 65535)
    return LLMX_REFUSED(1);
  return 0;
}

// proj float32 [T, row_stride] (or n_split partials); conv_w [taps, C] tap-major, conv_b [C] or null; a_log, dt_bias, skip
// [H]; state [slots, slot_stride] with the ring from ring_off.  Scratch, float32, 16-byte aligned: xs [T, H, Pp], bs and cs
// [T, G, Np], da [H, T, 2], st [T/64 + n_seqs, H, N, Pp], at [T/64 + n_seqs, H], cb [T/64 + n_seqs, G, 64, 64].  y [T, inner].
LLMX_API int llmx_ss_prompt(const float* proj, int n_split, long long split_stride, long long row_stride, const float* conv_w,
                            const float* conv_b, int taps, const float* a_log, const float* dt_bias, const float* skip,
                            float* state, long long slot_stride, long long ring_off, int n_slots, float* xs, float* bs,
                            float* cs, float* da, float* st, float* at, float* cb, float* y, const int* seq_start,
                            const int* seq_past, const int* seq_slot, int n_tokens, int n_seqs, int H, int G, int N, int P,
                            cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  const SsDims dm = {H, G, N, P, taps};
  if (const int bad = ss_check(dm, row_stride, n_split, slot_stride, ring_off, state, n_seqs)) return bad;
  if (((uintptr_t)xs | (uintptr_t)bs | (uintptr_t)cs | (uintptr_t)da | (uintptr_t)st | (uintptr_t)cb | (uintptr_t)y) & 15)
    return LLMX_REFUSED(1);
  const SsProj pr = {proj, n_split, (size_t)split_stride, (size_t)row_stride};
  const int C = dm.channels(), p_tiles = (dm.Pp() + 63) / 64, n_tiles = (N + 63) / 64;
  const int runs = n_tokens / SS_RUN + n_seqs, chunks = n_tokens / SS_CHUNK + n_seqs;
  if ((long long)H * p_tiles * n_tiles + G > 65535) return LLMX_REFUSED(3);
  const dim3 pgrid(runs, (C + H + 127) / 128);
#define PREP(TAPS)                       \
  do {                                    \
    if (n_split > 1) PREP2(TAPS, true);   \
    else PREP2(TAPS, false);              \
  } while (0)
#define PREP2(TAPS, SPLIT)                                                                                               \
  launch_pdl(ss_prep_kernel<TAPS, SPLIT>, pgrid, dim3(128), 0, stream, pr, dm, conv_w, conv_b, a_log, dt_bias, (const float*)state, \
             (size_t)slot_stride, (size_t)ring_off, xs, bs, cs, (float2*)da, seq_start, seq_past, seq_slot, n_seqs,      \
             n_tokens, n_slots)
  switch (taps) {
    case 2: PREP(2); break;
    case 3: PREP(3); break;
    case 4: PREP(4); break;
    default: PREP(0); break;
  }
#undef PREP
#undef PREP2
  launch_pdl(ss_chunk_kernel, dim3(chunks, H * p_tiles * n_tiles + G), dim3(SS_THREADS), 0, stream, (const float*)xs,
             (const float*)bs, (const float*)cs, (const float2*)da, st, at, cb, seq_start, n_seqs, n_tokens, dm);
  const long long quads = (long long)H * N * (dm.Pp() / 4);
  const int state_blocks = (int)((quads + 255) / 256), ring_blocks = taps > 1 ? (C + 255) / 256 : 0;
  launch_pdl(ss_pass_kernel, dim3(state_blocks + ring_blocks, n_seqs), dim3(256), 0, stream, pr, dm, st, (const float*)at,
             state, (size_t)slot_stride, (size_t)ring_off, seq_start, seq_past, seq_slot, n_tokens, n_slots, state_blocks);
  launch_pdl(ss_out_kernel, dim3(chunks, H * p_tiles), dim3(SS_THREADS), 0, stream, pr, dm, (const float*)xs, (const float*)cs,
             (const float2*)da, (const float*)st, (const float*)cb, skip, y, seq_start, n_seqs, n_tokens);
  return LLMX_LAUNCH_STATUS();
}

LLMX_API int llmx_ss_decode(const float* proj, int n_split, long long split_stride, long long row_stride, const float* conv_w,
                            const float* conv_b, int taps, const float* a_log, const float* dt_bias, const float* skip,
                            float* state, long long slot_stride, long long ring_off, int n_slots, float* y,
                            const int* seq_past, const int* seq_slot, int n_seqs, int H, int G, int N, int P,
                            cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  const SsDims dm = {H, G, N, P, taps};
  if (const int bad = ss_check(dm, row_stride, n_split, slot_stride, ring_off, state, n_seqs)) return bad;
  const SsProj pr = {proj, n_split, (size_t)split_stride, (size_t)row_stride};
  const bool vec = P % 4 == 0;
  const int cols = vec ? P / 4 : P, R = 256 / cols;
  const size_t smem = ((size_t)dm.Pp() + 2 * N + 3 + (size_t)R * dm.Pp()) * sizeof(float);
  if (smem > 48 * 1024) return LLMX_REFUSED(3);
#define GO(V)                                                                                                             \
  launch_pdl(ss_decode_kernel<V>, dim3(H, n_seqs), dim3(256), smem, stream, pr, dm, conv_w, conv_b, a_log, dt_bias, skip, \
             state, (size_t)slot_stride, (size_t)ring_off, y, seq_past, seq_slot, n_slots)
  if (vec) GO(4); else GO(1);
#undef GO
  return LLMX_LAUNCH_STATUS();
}

// y float32 [T, parts * width], gain float32 [parts * width], out of the same shape.
LLMX_API int llmx_ss_norm(const float* y, const float* gain, float eps, void* out, int out_dtype, int n_tokens, int width,
                          int parts, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (width <= 0 || parts <= 0 || parts > 65535 || (((uintptr_t)y | (uintptr_t)gain | (uintptr_t)out) & 15))
    return LLMX_REFUSED(1);
  const int need = width % 4 == 0 ? width / 4 : width;
  const int threads = need >= 256 ? 256 : (need + 31) / 32 * 32;
  if (out_dtype == LLMX_F32)
    launch_pdl(ss_norm_kernel<float>, dim3(n_tokens, parts), dim3(threads), 0, stream, y, gain, eps, (float*)out, width, parts);
  else if (out_dtype == LLMX_BF16)
    launch_pdl(ss_norm_kernel<bf16>, dim3(n_tokens, parts), dim3(threads), 0, stream, y, gain, eps, (bf16*)out, width, parts);
  else
    return LLMX_REFUSED(2);
  return LLMX_LAUNCH_STATUS();
}
