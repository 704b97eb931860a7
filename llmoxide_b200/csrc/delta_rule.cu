// The gated delta rule: a recurrence over a per-sequence state that corrects what the state already holds for a key
// before it writes, with a short convolution, an activation and unit norms on the way in.
//
// Per token and key/query head (D dims), value head h (Dv dims, sharing key head h / (H/G)):
//   q, k, v = silu(conv(projection))            causal convolution over time per channel, zeros before the start
//   q = q / sqrt(sum q^2 + unit_eps) * q_scale,  k = k / sqrt(sum k^2 + unit_eps)
//   beta = sigmoid(b),  g = exp(-exp(A_log) * softplus(a + dt_bias))                       per value head
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q                           S [D, Dv], starts at zero
//
// State of a sequence (float32): S of every value head [H, D, Dv], then the convolution's rows as a ring of `taps`
// rows of C = 2 G D + H Dv channels: position p's projected row lies at row p % taps.  A token reads the taps - 1 rows
// before it and never the row it will occupy, so in a step of single tokens every CTA may write the new row at once.
//
// Prompts.  The recurrence is walked in chunks of 8 tokens, counted from a sequence's first token of the step.  With S
// the state a chunk starts from, gamma_i = g_0 .. g_i and R_ij = g_(j+1) .. g_i,
//   u_i = beta_i v_i - beta_i gamma_i (S^T k_i) - sum_(j<i) beta_i R_ij (k_i . k_j) u_j
//   o_i = gamma_i (S^T q_i) + sum_(j<=i) R_ij (q_i . k_j) u_j
//   S'  = gamma_7 S + sum_j R_7j k_j u_j^T
// which is the recurrence above written out: the eight products S^T k_i and the eight S^T q_i do not wait for one
// another, and the chain from token to token is one multiply-add per earlier token and column.  The decays enter as
// products of g, never as differences of logarithms.  A chunk of fewer tokens is filled up with tokens of
// k = q = v = 0, beta = 0, g = 1, which change nothing.
//   delta_prep   one CTA per (chunk, key head): convolution, activation, unit norms, the two 8 x 8 matrices of dot
//                products, and per value head the gates and the coefficients above
//   delta_scan   a group of lanes (32, 16 or 8: D / 4) owns four columns of S, four dims a lane and the columns in
//                registers; partial products are added up by a transposing reduction.  It also moves the ring on.
// Single tokens: delta_decode, one CTA per (sequence, value head), does all of it and the norm and gate behind the
// recurrence (y = o / sqrt(mean o^2 + eps) * gain * silu(gate)), reading and writing S once.
//
// Everything is float32.  A decode step's sums and a prompt's are ordered differently, so a position's result may
// differ in rounding between cuttings.
#include "common.cuh"

#define DR_CHUNK 8
#define DR_STAGES 3
#define DR_MAX_D 256
#define DR_MAX_TAPS 16
#define DR_A 0                   // coefficients of a (chunk, value head): A [8][8] (column j < i: beta_i R_ij k_i.k_j)
#define DR_B 64                  // B [8][8] (column j <= i: R_ij q_i.k_j)
#define DR_BG 128                // beta_i gamma_i [8]
#define DR_G 136                 // gamma_i [8]
#define DR_W 144                 // R_7j [8]
#define DR_GL 152                // gamma_7, then padding
#define DR_COEF 156              // floats

__device__ __forceinline__ float dr_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float dr_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float dr_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// value of column c of a row: one tensor, or split partials added in order
template <typename TIN>
__device__ __forceinline__ float dr_value(const TIN* row, int c, int n_split, size_t split_stride) {
  float v = to_f32(row[c]);
  for (int s = 1; s < n_split; ++s) v += to_f32(row[s * split_stride + c]);
  return v;
}

struct DeltaIn {
  int n_split;
  size_t split_stride, row_stride;
  int q_off, k_off, v_off, b_off, a_off, g_off;      // columns of the projection
  const float* conv_w;                               // [taps][C], tap-major; channels q | k | v
  const float* a_log;                                // [H]
  const float* dt_bias;                              // [H]
  int taps, H, G, D, Dv;
  float q_scale, unit_eps;
  size_t slot_stride, ring_off;                      // floats: a slot's state; where its ring starts
};

// Column of the projection that channel c of the convolution reads.
__device__ __forceinline__ int dr_column(const DeltaIn& in, int c) {
  const int nq = in.G * in.D;
  return c < nq ? in.q_off + c : c < 2 * nq ? in.k_off + (c - nq) : in.v_off + (c - 2 * nq);
}

// The sequence a chunk belongs to: chunk slots of sequence b start at seq_start[b] / 8 + b.  Returns -1 for none.
__device__ __forceinline__ int dr_find_seq(const int* seq_start, int n_seqs, int slot) {
  int lo = 0, hi = n_seqs - 1;
  while (lo < hi) {                                  // the last b whose first slot is <= slot
    const int mid = (lo + hi + 1) >> 1;
    if (seq_start[mid] / DR_CHUNK + mid <= slot) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// The convolution of one channel for the chunk's tokens (positions pos0 .. pos0 + 7, the first n live), then SiLU.
// TAPS > 0: compiled for that many taps; 0: any number.
template <int TAPS, typename TIN>
__device__ __forceinline__ void dr_conv8(const DeltaIn& in, const TIN* proj, const float* ring, int C, int c, int row0,
                                         int p0, int pos0, int n, float* y) {
  const int taps = TAPS > 0 ? TAPS : in.taps;
  const int col = dr_column(in, c);
  auto u_at = [&](int p) {                            // the projected row of position p (p < pos0 + n)
    if (p >= p0) return dr_value(proj + (size_t)(row0 + p - p0) * in.row_stride, col, in.n_split, in.split_stride);
    return p >= 0 ? ring[(size_t)(p % taps) * C + c] : 0.f;
  };
  if (TAPS > 0) {
    float u[DR_CHUNK + (TAPS > 0 ? TAPS : 1) - 1];
#pragma unroll
    for (int r = 0; r < DR_CHUNK + TAPS - 1; ++r) u[r] = r - (TAPS - 1) < n ? u_at(pos0 - (TAPS - 1) + r) : 0.f;
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) y[i] = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const float w = in.conv_w[(size_t)j * C + c];
#pragma unroll
      for (int i = 0; i < DR_CHUNK; ++i) y[i] = fmaf(w, u[i + j], y[i]);
    }
  } else {
    for (int i = 0; i < DR_CHUNK; ++i) {
      y[i] = 0.f;
      if (i < n)
        for (int j = 0; j < taps; ++j) y[i] = fmaf(in.conv_w[(size_t)j * C + c], u_at(pos0 + i - taps + 1 + j), y[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < DR_CHUNK; ++i) y[i] = i < n ? dr_silu(y[i]) : 0.f;
}

// prep buffers: qk [slots][G][2][8][Dp] (keys, then queries), vv [slots][H][8][Dvp] (beta_i v_i), co [slots][H][DR_COEF]
template <typename TIN, int TAPS>
__global__ void __launch_bounds__(256)
delta_prep_kernel(const TIN* __restrict__ proj, const DeltaIn in, const float* __restrict__ state,
                  float* __restrict__ qk, float* __restrict__ vv, float* __restrict__ co,
                  const int* __restrict__ seq_start, const int* __restrict__ seq_past,
                  const int* __restrict__ seq_slot, int n_seqs, int n_tokens, int n_slots) {
  extern __shared__ __align__(16) float dr_smem[];
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slot = blockIdx.x, j = blockIdx.y;        // chunk slot, key/query head
  const int H = in.H, G = in.G, D = in.D, Dv = in.Dv, R = H / G, C = 2 * G * D + H * Dv;
  const int Dp = (D + 3) & ~3, Dvp = (Dv + 3) & ~3, ld = Dp + 4;
  const int b = dr_find_seq(seq_start, n_seqs, slot);
  const int row0 = seq_start[b], n_new = seq_start[b + 1] - row0, p0 = seq_past[b], sl = seq_slot[b];
  const int chunk = slot - (row0 / DR_CHUNK + b);
  if (chunk * DR_CHUNK >= n_new) return;              // (uniform) a slot no sequence fills
  if (row0 < 0 || row0 + n_new > n_tokens || p0 < 0 || sl < 0 || sl >= n_slots || chunk < 0) {
    if (tid == 0) llmx_report(1);
    return;
  }
  const int n = min(DR_CHUNK, n_new - chunk * DR_CHUNK), pos0 = p0 + chunk * DR_CHUNK, t0 = row0 + chunk * DR_CHUNK;
  const float* ring = state + (size_t)sl * in.slot_stride + in.ring_off;
  float* sk = dr_smem;                                // [8][ld]
  float* sq = sk + DR_CHUNK * ld;                     // [8][ld]
  float* dots = sq + DR_CHUNK * ld;                   // [2][8][8]: k_i . k_j, q_i . k_j
  float* gates = dots + 128;                          // [R][2][8]: beta, g
  pdl_wait();
  // ---- q and k of this head: convolution and activation, one channel a thread
  for (int e = tid; e < 2 * Dp; e += blockDim.x) {
    const bool is_k = e >= Dp;
    const int d = is_k ? e - Dp : e;
    float y[DR_CHUNK];
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) y[i] = 0.f;
    if (d < D) dr_conv8<TAPS>(in, proj, ring, C, (is_k ? G * D : 0) + j * D + d, row0, p0, pos0, n, y);
    float* dst = (is_k ? sk : sq) + d;
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) dst[i * ld] = y[i];
  }
  // ---- gates of the head's value heads
  for (int e = tid; e < R * DR_CHUNK; e += blockDim.x) {
    const int hr = e / DR_CHUNK, i = e - hr * DR_CHUNK, h = j * R + hr;
    float beta = 0.f, g = 1.f;
    if (i < n) {
      const TIN* row = proj + (size_t)(t0 + i) * in.row_stride;
      beta = dr_sigmoid(dr_value(row, in.b_off + h, in.n_split, in.split_stride));
      const float a = dr_value(row, in.a_off + h, in.n_split, in.split_stride);
      g = expf(-expf(in.a_log[h]) * dr_softplus(a + in.dt_bias[h]));
    }
    gates[hr * 16 + i] = beta;
    gates[hr * 16 + 8 + i] = g;
  }
  __syncthreads();
  // ---- unit norms: one warp per row
  for (int r = warp; r < 2 * DR_CHUNK; r += blockDim.x >> 5) {
    const bool is_q = r >= DR_CHUNK;
    float* row = is_q ? sq + (r - DR_CHUNK) * ld : sk + r * ld;
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss += row[d] * row[d];
    const float scale = (is_q ? in.q_scale : 1.f) / sqrtf(warp_sum(ss) + in.unit_eps);
    float* out = qk + (((size_t)slot * G + j) * 2 + (is_q ? 1 : 0)) * DR_CHUNK * Dp + (size_t)(r & 7) * Dp;
    for (int d = lane; d < Dp; d += 32) {
      const float x = row[d] * scale;
      row[d] = x;
      out[d] = x;
    }
  }
  __syncthreads();
  // ---- the dot products, four lanes each
  for (int e = tid; e < 128 * 4; e += blockDim.x) {   // (a warp's 32 threads take part together: 512 is a multiple)
    const int pair = e >> 2, part = e & 3, which = pair >> 6, i = (pair >> 3) & 7, jj = pair & 7;
    const float* x = (which ? sq : sk) + i * ld;
    const float* y = sk + jj * ld;
    float s = 0.f;
    if (which ? jj <= i : jj < i)
      for (int d = part; d < D; d += 4) s = fmaf(x[d], y[d], s);
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    s += __shfl_xor_sync(0xffffffffu, s, 2);
    if (part == 0) dots[pair] = s;
  }
  __syncthreads();
  // ---- coefficients of every value head
  for (int e = tid; e < R * 64; e += blockDim.x) {
    const int hr = e >> 6, i = (e >> 3) & 7, jj = e & 7;
    const float* beta = gates + hr * 16;
    const float* g = beta + 8;
    float* c = co + ((size_t)slot * H + j * R + hr) * DR_COEF;
    float rij = 1.f;
    for (int m = jj + 1; m <= i; ++m) rij *= g[m];
    c[DR_A + i * 8 + jj] = jj < i ? beta[i] * rij * dots[i * 8 + jj] : 0.f;
    c[DR_B + i * 8 + jj] = jj <= i ? rij * dots[64 + i * 8 + jj] : 0.f;
    if (i == 7) c[DR_W + jj] = rij;
    if (jj == 0) {
      const float gam = g[0] * rij;                   // rij is g_1 .. g_i here
      c[DR_G + i] = gam;
      c[DR_BG + i] = beta[i] * gam;
      if (i == 7) c[DR_GL] = gam, c[DR_GL + 1] = c[DR_GL + 2] = c[DR_GL + 3] = 0.f;
    }
  }
  // ---- values
  for (int e = tid; e < R * Dvp; e += blockDim.x) {
    const int hr = e / Dvp, d = e - hr * Dvp, h = j * R + hr;
    float y[DR_CHUNK];
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) y[i] = 0.f;
    if (d < Dv) dr_conv8<TAPS>(in, proj, ring, C, 2 * G * D + h * Dv + d, row0, p0, pos0, n, y);
    float* out = vv + ((size_t)slot * H + h) * DR_CHUNK * Dvp + d;
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) out[(size_t)i * Dvp] = y[i] * gates[hr * 16 + i];
  }
}

__device__ __forceinline__ void dr_cp_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src)
               : "memory");
}

// Adds N values over LANES neighbouring lanes; afterwards lane r (of the group) holds the sums of the values
// r * (N / LANES) .. + N / LANES - 1 in v[0 ..].  Halving: at every step a lane hands half of its values to its partner.
template <int N, int LANES>
__device__ __forceinline__ void dr_reduce(float* v, int r) {
  int n = N;
#pragma unroll
  for (int bit = LANES / 2; bit > 0; bit >>= 1) {
    n >>= 1;
    const bool up = (r & bit) != 0;
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
      if (i < n) {
        const float mine = up ? v[n + i] : v[i], give = up ? v[i] : v[n + i];
        v[i] = mine + __shfl_xor_sync(0xffffffffu, give, bit);
      }
    }
  }
}

#define DR_WARPS 4

// Four columns of S per group of LANES lanes; lane r of a group owns dims 4 (r + LANES i) + 0..3, i < NI.
template <int LANES, int NI>
__global__ void __launch_bounds__(DR_WARPS * 32)
delta_scan_kernel(const float* __restrict__ qk, const float* __restrict__ vv, const float* __restrict__ co,
                  float* __restrict__ out, float* __restrict__ state, size_t slot_stride,
                  const int* __restrict__ seq_start, const int* __restrict__ seq_slot, int H, int G, int D, int Dv,
                  int n_slots) {
  extern __shared__ __align__(16) float dr_smem[];
  constexpr int GROUPS = 32 / LANES, COLS = DR_WARPS * GROUPS * 4;     // columns of a CTA
  const int Dp = (D + 3) & ~3, Dvp = (Dv + 3) & ~3;
  const int stage_len = 2 * DR_CHUNK * Dp + DR_CHUNK * COLS + DR_COEF;
  float* work = dr_smem + DR_STAGES * stage_len;       // [DR_WARPS][GROUPS][64 sums | 32 weighted u]
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, grp = lane / LANES, r = lane % LANES;
  const int b = blockIdx.z, h = blockIdx.y, c_cta = blockIdx.x * COLS;
  const int c_loc = (warp * GROUPS + grp) * 4, c0 = c_cta + c_loc;     // this group's first column
  const int row0 = seq_start[b], n_new = seq_start[b + 1] - row0, sl = seq_slot[b];
  if (n_new <= 0) return;
  if (sl < 0 || sl >= n_slots) {
    if (tid == 0) llmx_report(2);
    return;
  }
  float* S = state + (size_t)sl * slot_stride + (size_t)h * D * Dv;
  const int slot0 = row0 / DR_CHUNK + b, n_chunks = (n_new + DR_CHUNK - 1) / DR_CHUNK;
  const int j = h / (H / G);
  float* wsum = work + (warp * GROUPS + grp) * 96;
  float* wu = wsum + 64;
  pdl_wait();

  float s[NI][4][4];                                   // [dims block][dim][column]
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int d = 0; d < 4; ++d)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int dim = 4 * (r + LANES * i) + d;
        s[i][d][c] = (dim < D && c0 + c < Dv) ? S[(size_t)dim * Dv + c0 + c] : 0.f;
      }

  const int qk_pieces = 2 * DR_CHUNK * Dp / 4, v_pieces = DR_CHUNK * COLS / 4, co_pieces = DR_COEF / 4;
  auto load_chunk = [&](int ch) {
    float* buf = dr_smem + (ch % DR_STAGES) * stage_len;
    const float* qsrc = qk + ((size_t)(slot0 + ch) * G + j) * 2 * DR_CHUNK * Dp;
    for (int e = tid; e < qk_pieces; e += DR_WARPS * 32) dr_cp_async16(buf + 4 * e, qsrc + 4 * e);
    const float* vsrc = vv + ((size_t)(slot0 + ch) * H + h) * DR_CHUNK * Dvp;
    float* vbuf = buf + 2 * DR_CHUNK * Dp;
    for (int e = tid; e < v_pieces; e += DR_WARPS * 32) {
      const int i = e / (COLS / 4), c = (e - i * (COLS / 4)) * 4;
      if (c_cta + c < Dvp) dr_cp_async16(vbuf + i * COLS + c, vsrc + (size_t)i * Dvp + c_cta + c);
    }
    const float* csrc = co + ((size_t)(slot0 + ch) * H + h) * DR_COEF;
    float* cbuf = vbuf + DR_CHUNK * COLS;
    for (int e = tid; e < co_pieces; e += DR_WARPS * 32) dr_cp_async16(cbuf + 4 * e, csrc + 4 * e);
  };
  for (int c = 0; c < DR_STAGES - 1; ++c) {
    if (c < n_chunks) load_chunk(c);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  const int col = lane & 3, c_of_lane = c_loc + col;   // (LANES is a multiple of 4)
  const bool live = c0 + col < Dv;
  float* out_col = out + (size_t)row0 * H * Dv + (size_t)h * Dv + c0 + col;
  for (int ch = 0; ch < n_chunks; ++ch) {
    if (ch + DR_STAGES - 1 < n_chunks) load_chunk(ch + DR_STAGES - 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group %0;" ::"n"(DR_STAGES - 1) : "memory");
    __syncthreads();
    const float* buf = dr_smem + (ch % DR_STAGES) * stage_len;
    const float* kbuf = buf;
    const float* qbuf = buf + DR_CHUNK * Dp;
    const float* vbuf = buf + 2 * DR_CHUNK * Dp;
    const float* cbuf = vbuf + DR_CHUNK * COLS;
    // ---- S^T k_i and S^T q_i: this lane's dims, then the sum over the group
    // value index of a sum: column * 8 + token
    float acc[32];
    auto products = [&](const float* rows) {
#pragma unroll
      for (int i = 0; i < DR_CHUNK; ++i) {
        float p[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int ni = 0; ni < NI; ++ni) {
          const int d = 4 * (r + LANES * ni);
          if (d < Dp) {
            const float4 x = *reinterpret_cast<const float4*>(rows + i * Dp + d);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              p[c] = fmaf(x.x, s[ni][0][c], p[c]);
              p[c] = fmaf(x.y, s[ni][1][c], p[c]);
              p[c] = fmaf(x.z, s[ni][2][c], p[c]);
              p[c] = fmaf(x.w, s[ni][3][c], p[c]);
            }
          }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[c * 8 + i] = p[c];
      }
      dr_reduce<32, LANES>(acc, r);
    };
    products(kbuf);
#pragma unroll
    for (int i = 0; i < 32 / LANES; ++i) wsum[r * (32 / LANES) + i] = acc[i];
    products(qbuf);
#pragma unroll
    for (int i = 0; i < 32 / LANES; ++i) wsum[32 + r * (32 / LANES) + i] = acc[i];
    __syncwarp();
    // ---- the chain from token to token, for this lane's column (every lane of a column alike)
    float u[DR_CHUNK];
    {
      const float4 k0 = *reinterpret_cast<const float4*>(wsum + col * 8), k1 = *reinterpret_cast<const float4*>(wsum + col * 8 + 4);
      const float ks[DR_CHUNK] = {k0.x, k0.y, k0.z, k0.w, k1.x, k1.y, k1.z, k1.w};
#pragma unroll
      for (int i = 0; i < DR_CHUNK; ++i) u[i] = fmaf(-cbuf[DR_BG + i], ks[i], vbuf[i * COLS + c_of_lane]);
#pragma unroll
      for (int i = 0; i < DR_CHUNK; ++i)
#pragma unroll
        for (int m = i + 1; m < DR_CHUNK; ++m) u[m] = fmaf(-cbuf[DR_A + m * 8 + i], u[i], u[m]);
    }
    // ---- outputs: the lanes of a column share its eight tokens
    const int n_tok = min(DR_CHUNK, n_new - ch * DR_CHUNK);
#pragma unroll
    for (int e = 0; e < DR_CHUNK * 4 / LANES; ++e) {
      const int i = (r >> 2) + e * (LANES / 4);
      float o = cbuf[DR_G + i] * wsum[32 + col * 8 + i];
      const float4 b0 = *reinterpret_cast<const float4*>(cbuf + DR_B + i * 8), b1 = *reinterpret_cast<const float4*>(cbuf + DR_B + i * 8 + 4);
      o = fmaf(b0.x, u[0], o);
      o = fmaf(b0.y, u[1], o);
      o = fmaf(b0.z, u[2], o);
      o = fmaf(b0.w, u[3], o);
      o = fmaf(b1.x, u[4], o);
      o = fmaf(b1.y, u[5], o);
      o = fmaf(b1.z, u[6], o);
      o = fmaf(b1.w, u[7], o);
      if (live && i < n_tok) out_col[(size_t)(ch * DR_CHUNK + i) * H * Dv] = o;
    }
    // ---- the state: every lane needs all four columns' u, weighted
    if (r < 4) {
#pragma unroll
      for (int i = 0; i < DR_CHUNK; ++i) wu[i * 4 + col] = cbuf[DR_W + i] * u[i];
    }
    __syncwarp();
    const float gl = cbuf[DR_GL];
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int d = 0; d < 4; ++d)
#pragma unroll
        for (int c = 0; c < 4; ++c) s[i][d][c] *= gl;
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) {
      const float4 w = *reinterpret_cast<const float4*>(wu + i * 4);
#pragma unroll
      for (int ni = 0; ni < NI; ++ni) {
        const int d = 4 * (r + LANES * ni);
        if (d < Dp) {
          const float4 x = *reinterpret_cast<const float4*>(kbuf + i * Dp + d);
          const float xs[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
          for (int dd = 0; dd < 4; ++dd) {
            s[ni][dd][0] = fmaf(xs[dd], w.x, s[ni][dd][0]);
            s[ni][dd][1] = fmaf(xs[dd], w.y, s[ni][dd][1]);
            s[ni][dd][2] = fmaf(xs[dd], w.z, s[ni][dd][2]);
            s[ni][dd][3] = fmaf(xs[dd], w.w, s[ni][dd][3]);
          }
        }
      }
    }
    __syncthreads();                                   // the buffer is refilled by the next round's copies
  }
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int d = 0; d < 4; ++d)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int dim = 4 * (r + LANES * i) + d;
        if (dim < D && c0 + c < Dv) S[(size_t)dim * Dv + c0 + c] = s[i][d][c];
      }
}

// The ring after a prompt step: the projected rows of the last taps - 1 tokens of every sequence (rows of earlier
// positions that are still wanted stay where they are).  One thread per (sequence, channel).
template <typename TIN>
__global__ void delta_ring_kernel(const TIN* __restrict__ proj, const DeltaIn in, float* __restrict__ state,
                                  const int* __restrict__ seq_start, const int* __restrict__ seq_past,
                                  const int* __restrict__ seq_slot, int n_tokens, int n_slots) {
  pdl_launch_dependents();
  const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int C = 2 * in.G * in.D + in.H * in.Dv;
  const int row0 = seq_start[b], n_new = seq_start[b + 1] - row0, p0 = seq_past[b], sl = seq_slot[b];
  if (row0 < 0 || row0 + n_new > n_tokens || p0 < 0 || sl < 0 || sl >= n_slots) {
    if (c == 0) llmx_report(3);
    return;
  }
  pdl_wait();
  if (c >= C) return;
  float* ring = state + (size_t)sl * in.slot_stride + in.ring_off;
  const int col = dr_column(in, c);
  for (int i = max(0, n_new - (in.taps - 1)); i < n_new; ++i)
    ring[(size_t)((p0 + i) % in.taps) * C + c] = dr_value(proj + (size_t)(row0 + i) * in.row_stride, col, in.n_split, in.split_stride);
}

// One new token per sequence.  256 threads: warp w owns dims w, w + 8, .. of S, a lane V neighbouring columns of a tile
// of 32 V; DPT: dims per warp.
template <typename TIN, typename TO, int DPT, int V>
__global__ void __launch_bounds__(256)
delta_decode_kernel(const TIN* __restrict__ proj, const DeltaIn in, float* __restrict__ state,
                    const float* __restrict__ gain, float eps, TO* __restrict__ y, const int* __restrict__ seq_past,
                    const int* __restrict__ seq_slot, int n_slots) {
  extern __shared__ __align__(16) float dr_smem[];
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x, b = blockIdx.y;
  const int H = in.H, G = in.G, D = in.D, Dv = in.Dv, taps = in.taps, C = 2 * G * D + H * Dv, j = h / (H / G);
  const int p = seq_past[b], sl = seq_slot[b];
  if (p < 0 || sl < 0 || sl >= n_slots) {
    if (tid == 0) llmx_report(4);
    return;
  }
  float* base = state + (size_t)sl * in.slot_stride;
  float* S = base + (size_t)h * D * Dv;
  float* ring = base + in.ring_off;
  float* sq = dr_smem;                                  // [D]
  float* sk = sq + DR_MAX_D;                            // [D]
  float* sums = sk + DR_MAX_D;                          // q.q, k.k, q.k, beta, g
  float* part = sums + 8;                               // [8 warps][2][32 V]
  float* so = part + 8 * 2 * 32 * V;                    // [Dv] the head's output
  float* sv = so + ((Dv + 3) & ~3);                     // [Dv]
  __shared__ float red[32];
  pdl_wait();
  const TIN* row = proj + (size_t)b * in.row_stride;
  // the first tile of S is asked for before anything else
  float s[DPT][V];
  auto load_tile = [&](int c0) {
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      const int d = warp + 8 * i;
#pragma unroll
      for (int e = 0; e < V; ++e) s[i][e] = 0.f;
      if (d < D && c0 < Dv) {
        if (V == 4) {
          const float4 x = *reinterpret_cast<const float4*>(S + (size_t)d * Dv + c0);
          s[i][0] = x.x;
          if (V == 4) s[i][1 % V] = x.y, s[i][2 % V] = x.z, s[i][3 % V] = x.w;
        } else {
          s[i][0] = S[(size_t)d * Dv + c0];
        }
      }
    }
  };
  load_tile(lane * V);
  // ---- convolution, activation; the token's projected row joins the ring
  for (int e = tid; e < 2 * D + Dv; e += 256) {
    const int c = e < D ? j * D + e : e < 2 * D ? G * D + j * D + (e - D) : 2 * G * D + h * Dv + (e - 2 * D);
    const float own = dr_value(row, dr_column(in, c), in.n_split, in.split_stride);
    float acc = 0.f;
    for (int m = 0; m < taps; ++m) {
      const int pp = p - taps + 1 + m;
      const float u = m == taps - 1 ? own : pp >= 0 ? ring[(size_t)(pp % taps) * C + c] : 0.f;
      acc = fmaf(in.conv_w[(size_t)m * C + c], u, acc);
    }
    if (taps > 1) ring[(size_t)(p % taps) * C + c] = own;      // (heads that share a key head write the same number)
    acc = dr_silu(acc);
    if (e < D) sq[e] = acc;
    else if (e < 2 * D) sk[e - D] = acc;
    else sv[e - 2 * D] = acc;
  }
  __syncthreads();
  if (warp < 3) {
    const float* x = warp == 1 ? sk : sq;
    const float* z = warp == 0 ? sq : sk;
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss += x[d] * z[d];
    ss = warp_sum(ss);
    if (lane == 0) sums[warp] = ss;
  } else if (warp == 3 && lane == 0) {
    sums[3] = dr_sigmoid(dr_value(row, in.b_off + h, in.n_split, in.split_stride));
    const float a = dr_value(row, in.a_off + h, in.n_split, in.split_stride);
    sums[4] = expf(-expf(in.a_log[h]) * dr_softplus(a + in.dt_bias[h]));
  }
  __syncthreads();
  const float fq = in.q_scale / sqrtf(sums[0] + in.unit_eps), fk = 1.f / sqrtf(sums[1] + in.unit_eps);
  const float qk = sums[2] * fq * fk, beta = sums[3], g = sums[4];
  float ss_o = 0.f;
  for (int tile = 0; tile < Dv; tile += 32 * V) {
    const int c0 = tile + lane * V;
    if (tile > 0) load_tile(c0);
    // ---- S^T k and S^T q of the old state
    float pk[V], pq[V];
#pragma unroll
    for (int e = 0; e < V; ++e) pk[e] = pq[e] = 0.f;
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      const int d = warp + 8 * i;
      if (d < D) {
        const float kd = sk[d], qd = sq[d];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          pk[e] = fmaf(kd, s[i][e], pk[e]);
          pq[e] = fmaf(qd, s[i][e], pq[e]);
        }
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      part[(warp * 2) * 32 * V + lane * V + e] = pk[e];
      part[(warp * 2 + 1) * 32 * V + lane * V + e] = pq[e];
    }
    __syncthreads();
    float u[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      float ks = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) ks += part[(w * 2) * 32 * V + lane * V + e];
      u[e] = c0 + e < Dv ? beta * (sv[c0 + e] - g * (ks * fk)) : 0.f;
    }
    if (warp == 0) {
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float qs = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) qs += part[(w * 2 + 1) * 32 * V + lane * V + e];
        // o = (g S + k u^T)^T q = g S^T q + (k . q) u
        const float o = fmaf(qk, u[e], g * (qs * fq));
        if (c0 + e < Dv) {
          so[c0 + e] = o;
          ss_o += o * o;
        }
      }
    }
    // ---- S <- g S + k u^T
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      const int d = warp + 8 * i;
      if (d < D && c0 < Dv) {
        const float kd = sk[d] * fk;
        if (V == 4) {
          float4 x;
          x.x = fmaf(kd, u[0], g * s[i][0]);
          x.y = fmaf(kd, u[1 % V], g * s[i][1 % V]);
          x.z = fmaf(kd, u[2 % V], g * s[i][2 % V]);
          x.w = fmaf(kd, u[3 % V], g * s[i][3 % V]);
          *reinterpret_cast<float4*>(S + (size_t)d * Dv + c0) = x;
        } else {
          S[(size_t)d * Dv + c0] = fmaf(kd, u[0], g * s[i][0]);
        }
      }
    }
    __syncthreads();                                    // part is written again by the next tile
  }
  // ---- the head's norm and gate
  const float rstd = 1.0f / sqrtf(block_sum(ss_o, red) / (float)Dv + eps);
  for (int c = tid; c < Dv; c += 256) {
    const float z = dr_value(row, in.g_off + h * Dv + c, in.n_split, in.split_stride);
    y[((size_t)b * H + h) * Dv + c] = from_f32<TO>(((so[c] * rstd) * gain[c]) * dr_silu(z));
  }
}

static int dr_check(const DeltaIn& in, long long row_stride) {
  if (in.H <= 0 || in.G <= 0 || in.H % in.G || in.D <= 0 || in.D > DR_MAX_D || in.Dv <= 0 || in.taps < 1 ||
      in.taps > DR_MAX_TAPS || in.n_split < 1)
    return LLMX_REFUSED(1);
  const long long nq = (long long)in.G * in.D, nv = (long long)in.H * in.Dv;
  if (in.q_off < 0 || in.q_off + nq > row_stride || in.k_off < 0 || in.k_off + nq > row_stride || in.v_off < 0 ||
      in.v_off + nv > row_stride || in.b_off < 0 || in.b_off + in.H > row_stride || in.a_off < 0 ||
      in.a_off + in.H > row_stride || in.g_off < 0 || in.g_off + nv > row_stride)
    return LLMX_REFUSED(1);
  const size_t C = 2 * nq + nv;
  if (in.ring_off < (size_t)nv * in.D || in.slot_stride < in.ring_off + C * in.taps || (in.slot_stride & 3))
    return LLMX_REFUSED(1);
  if (!in.conv_w || !in.a_log || !in.dt_bias) return LLMX_REFUSED(4);
  return 0;
}

// proj: [T, row_stride] float32 or bfloat16, or n_split float32 partials; state: float32 [n_slots, slot_stride].
// Prompts: qk, vv, co are float32 scratch, 16-byte aligned, for T / 8 + n_seqs chunks:
// [chunks, G, 16, Dp], [chunks, H, 8, Dvp], [chunks, H, 156]; out float32 [T, H*Dv].
LLMX_API int llmx_delta_prompt(const void* proj, int in_dtype, int n_split, long long split_stride, long long row_stride,
                               int q_off, int k_off, int v_off, int b_off, int a_off, int g_off, const float* conv_w,
                               int taps, const float* a_log, const float* dt_bias, float q_scale, float unit_eps,
                               float* state, long long slot_stride, long long ring_off, int n_slots, float* qk, float* vv,
                               float* co, float* out, const int* seq_start, const int* seq_past, const int* seq_slot,
                               int n_tokens, int n_seqs, int H, int G, int D, int Dv, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  const DeltaIn in = {n_split, (size_t)split_stride, (size_t)row_stride, q_off, k_off, v_off, b_off, a_off, g_off,
                      conv_w, a_log, dt_bias, taps, H, G, D, Dv, q_scale, unit_eps, (size_t)slot_stride, (size_t)ring_off};
  const int bad = dr_check(in, row_stride);
  if (bad) return bad;
  if (n_seqs > 65535 || H > 65535 || (((uintptr_t)qk | (uintptr_t)vv | (uintptr_t)co | (uintptr_t)state) & 15)) return LLMX_REFUSED(3);
  if (in_dtype != LLMX_F32 && in_dtype != LLMX_BF16) return LLMX_REFUSED(2);
  const int Dp = (D + 3) & ~3, R = H / G;
  const size_t psmem = (size_t)(2 * DR_CHUNK * (Dp + 4) + 128 + R * 16) * sizeof(float);
  if (psmem > 48 * 1024) return LLMX_REFUSED(3);
  const dim3 pgrid(n_tokens / DR_CHUNK + n_seqs, G);
#define PREP(TIN, TAPS)                                                                                                 \
  launch_pdl(delta_prep_kernel<TIN, TAPS>, pgrid, dim3(256), psmem, stream, (const TIN*)proj, in, (const float*)state,  \
             qk, vv, co, seq_start, seq_past, seq_slot, n_seqs, n_tokens, n_slots)
#define PREP_T(TIN)                       \
  do {                                    \
    if (taps == 4) PREP(TIN, 4);          \
    else if (taps == 3) PREP(TIN, 3);     \
    else if (taps == 2) PREP(TIN, 2);     \
    else if (taps == 1) PREP(TIN, 1);     \
    else PREP(TIN, 0);                    \
  } while (0)
  if (in_dtype == LLMX_F32) PREP_T(float); else PREP_T(bf16);
#undef PREP_T
#undef PREP
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
#define SCAN(LANES, NI)                                                                                                 \
  do {                                                                                                                  \
    const int cols = DR_WARPS * (32 / LANES) * 4;                                                                       \
    const size_t smem = (size_t)(DR_STAGES * (2 * DR_CHUNK * Dp + DR_CHUNK * cols + DR_COEF) +                          \
                                 DR_WARPS * (32 / LANES) * 96) * sizeof(float);                                         \
    static bool attr_set = false;                                                                                       \
    if (!attr_set && smem > 48 * 1024) {                                                                                \
      e = cudaFuncSetAttribute(delta_scan_kernel<LANES, NI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);  \
      if (e != cudaSuccess) return (int)e;                                                                              \
      attr_set = true;                                                                                                  \
    }                                                                                                                   \
    launch_pdl(delta_scan_kernel<LANES, NI>, dim3((Dv + cols - 1) / cols, H, n_seqs), dim3(DR_WARPS * 32), smem, stream, \
               (const float*)qk, (const float*)vv, (const float*)co, out, state, (size_t)slot_stride, seq_start,        \
               seq_slot, H, G, D, Dv, n_slots);                                                                         \
  } while (0)
  if (Dp <= 32) SCAN(8, 1);
  else if (Dp <= 64) SCAN(16, 1);
  else if (Dp <= 128) SCAN(32, 1);
  else SCAN(32, 2);
#undef SCAN
  e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
  if (taps > 1) {
    const int C = 2 * G * D + H * Dv;
    const dim3 rgrid((C + 127) / 128, n_seqs);
    if (in_dtype == LLMX_F32)
      launch_pdl(delta_ring_kernel<float>, rgrid, dim3(128), 0, stream, (const float*)proj, in, state, seq_start, seq_past,
                 seq_slot, n_tokens, n_slots);
    else
      launch_pdl(delta_ring_kernel<bf16>, rgrid, dim3(128), 0, stream, (const bf16*)proj, in, state, seq_start, seq_past,
                 seq_slot, n_tokens, n_slots);
  }
  return LLMX_LAUNCH_STATUS();
}

// One token per sequence: y [n_seqs, H*Dv] = o / sqrt(mean o^2 + eps) * gain * silu(gate) per head; gain float32 [Dv].
LLMX_API int llmx_delta_decode(const void* proj, int in_dtype, int n_split, long long split_stride, long long row_stride,
                               int q_off, int k_off, int v_off, int b_off, int a_off, int g_off, const float* conv_w,
                               int taps, const float* a_log, const float* dt_bias, float q_scale, float unit_eps,
                               float* state, long long slot_stride, long long ring_off, int n_slots, const float* gain,
                               float eps, void* y, int out_dtype, const int* seq_past, const int* seq_slot, int n_seqs,
                               int H, int G, int D, int Dv, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  const DeltaIn in = {n_split, (size_t)split_stride, (size_t)row_stride, q_off, k_off, v_off, b_off, a_off, g_off,
                      conv_w, a_log, dt_bias, taps, H, G, D, Dv, q_scale, unit_eps, (size_t)slot_stride, (size_t)ring_off};
  const int bad = dr_check(in, row_stride);
  if (bad) return bad;
  if (!gain) return LLMX_REFUSED(4);
  if (n_seqs > 65535 || ((uintptr_t)state & 15)) return LLMX_REFUSED(3);
  const bool vec = Dv % 4 == 0;
  const size_t smem = (size_t)(2 * DR_MAX_D + 8 + 8 * 2 * 32 * (vec ? 4 : 1) + 2 * ((Dv + 3) & ~3)) * sizeof(float);
  if (smem > 48 * 1024) return LLMX_REFUSED(3);
#define GO(TIN, TO, DPT, V)                                                                                           \
  launch_pdl(delta_decode_kernel<TIN, TO, DPT, V>, dim3(H, n_seqs), dim3(256), smem, stream, (const TIN*)proj, in,    \
             state, gain, eps, (TO*)y, seq_past, seq_slot, n_slots)
#define GO_D(TIN, TO, V)                        \
  do {                                          \
    if (D <= 32) GO(TIN, TO, 4, V);             \
    else if (D <= 64) GO(TIN, TO, 8, V);        \
    else if (D <= 128) GO(TIN, TO, 16, V);      \
    else GO(TIN, TO, 32, V);                    \
  } while (0)
#define GO_V(TIN, TO)                \
  do {                               \
    if (vec) GO_D(TIN, TO, 4);       \
    else GO_D(TIN, TO, 1);           \
  } while (0)
  switch (in_dtype * 2 + out_dtype) {
    case 0: GO_V(float, float); break;
    case 1: GO_V(float, bf16); break;
    case 3: GO_V(bf16, bf16); break;
    default: return LLMX_REFUSED(2);
  }
#undef GO_V
#undef GO_D
#undef GO
  return LLMX_LAUNCH_STATUS();
}
