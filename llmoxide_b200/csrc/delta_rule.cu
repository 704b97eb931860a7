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
//   delta_scan   a group of lanes (32, 16 or 8: D / 4) owns two or four columns of S, four dims a lane and column in
//                registers; the partial products of a chunk's eight tokens are added up by a halving reduction that
//                leaves every lane the sums of its own token and column
//   delta_ring   moves the ring on
// Single tokens: delta_decode, one CTA per (sequence, value head), does all of it and the norm and gate behind the
// recurrence (y = o / sqrt(mean o^2 + eps) * gain * silu(gate)), reading and writing S once.
//
// Everything is float32.  A decode step's sums and a prompt's are ordered differently, so a position's result may
// differ in rounding between cuttings.
#include "tc_ptx.cuh"

#define DR_CHUNK 8
#define DR_STAGES 3
#define DR_MAX_D 256
#define DR_MAX_TAPS 16
// coefficients of a (chunk, value head), floats
#define DR_A 0                   // A, rows 1..7 of a strictly lower triangle: row i at i (i - 1) / 2, beta_i R_ij k_i.k_j
#define DR_BG 28                 // beta_i gamma_i [8]
#define DR_W 36                  // R_7j [8]
#define DR_G 44                  // gamma_i [8]
#define DR_GL 52                 // gamma_7, three unused
#define DR_B 56                  // B [8][8] (column j <= i: R_ij q_i.k_j)
#define DR_COEF 120
#define DR_PAD 16                // floats between the rows of q and k in delta_prep: its 16-byte reads meet no bank twice

__device__ __forceinline__ float dr_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float dr_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float dr_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// value of column c of a row: one tensor, or split partials added in order
template <typename TIN>
__device__ __forceinline__ float dr_value(const TIN* row, int c, int n_split, size_t split_stride) {
  return split_value(row, c, n_split, split_stride);
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

// prep buffers: qk [slots][G][2][8][DL] (keys, then queries; DL: the staged row of delta_scan, zeros beyond D), vv [slots][H][Dvp][8] (beta_i v_i, a column's tokens
// together), co [slots][H][DR_COEF]
template <typename TIN, int TAPS>
__global__ void __launch_bounds__(256, 3)
delta_prep_kernel(const TIN* __restrict__ proj, const DeltaIn in, const float* __restrict__ state,
                  float* __restrict__ qk, float* __restrict__ vv, float* __restrict__ co,
                  const int* __restrict__ seq_start, const int* __restrict__ seq_past,
                  const int* __restrict__ seq_slot, int n_seqs, int n_tokens, int n_slots, int DL) {
  extern __shared__ __align__(128) float dr_smem[];
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slot = blockIdx.x, j = blockIdx.y;        // chunk slot, key/query head
  const int H = in.H, G = in.G, D = in.D, Dv = in.Dv, R = H / G, C = 2 * G * D + H * Dv;
  const int Dp = (D + 3) & ~3, Dvp = (Dv + 3) & ~3, ld = Dp + DR_PAD;
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
  // ---- values of the head's value heads, a channel a thread; the first ones wait in registers for their beta, so that
  // their loads are in flight together with those of q and k
  auto value = [&](int e, float* y) {
    const int hr = e / Dvp, d = e - hr * Dvp;
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) y[i] = 0.f;
    if (d < Dv) dr_conv8<TAPS>(in, proj, ring, C, 2 * G * D + (j * R + hr) * Dv + d, row0, p0, pos0, n, y);
  };
  auto put_value = [&](int e, const float* y) {
    const int hr = e / Dvp, d = e - hr * Dvp;
    const float* beta = gates + hr * 16;
    float4* out = reinterpret_cast<float4*>(vv + (((size_t)slot * H + j * R + hr) * Dvp + d) * DR_CHUNK);
    out[0] = make_float4(y[0] * beta[0], y[1] * beta[1], y[2] * beta[2], y[3] * beta[3]);
    out[1] = make_float4(y[4] * beta[4], y[5] * beta[5], y[6] * beta[6], y[7] * beta[7]);
  };
  float y_first[DR_CHUNK];
  if (tid < R * Dvp) value(tid, y_first);
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
  // ---- gates
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
  if (tid < R * Dvp) put_value(tid, y_first);
  // ---- unit norms: one warp per row
  for (int r = warp; r < 2 * DR_CHUNK; r += blockDim.x >> 5) {
    const bool is_q = r >= DR_CHUNK;
    float* row = is_q ? sq + (r - DR_CHUNK) * ld : sk + r * ld;
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss += row[d] * row[d];
    const float scale = (is_q ? in.q_scale : 1.f) / sqrtf(warp_sum(ss) + in.unit_eps);
    float* out = qk + (((size_t)slot * G + j) * 2 + (is_q ? 1 : 0)) * DR_CHUNK * DL + (size_t)(r & 7) * DL;
    for (int d = lane; d < DL; d += 32) {
      const float x = d < Dp ? row[d] * scale : 0.f;
      if (d < Dp) row[d] = x;
      out[d] = x;
    }
  }
  __syncthreads();
  // ---- the dot products, four lanes each (rows of 4-float pieces, a lane every fourth piece)
  for (int e = tid; e < 128 * 4; e += blockDim.x) {   // (a warp's 32 threads take part together: 512 is a multiple)
    const int pair = e >> 2, part = e & 3, which = pair >> 6, i = (pair >> 3) & 7, jj = pair & 7;
    const float* x = (which ? sq : sk) + i * ld;
    const float* y = sk + jj * ld;
    float s = 0.f;
    if (which ? jj <= i : jj < i)
      for (int d = 4 * part; d < Dp; d += 16) {
        const float4 xa = *reinterpret_cast<const float4*>(x + d), ya = *reinterpret_cast<const float4*>(y + d);
        s = fmaf(xa.x, ya.x, s);
        s = fmaf(xa.y, ya.y, s);
        s = fmaf(xa.z, ya.z, s);
        s = fmaf(xa.w, ya.w, s);
      }
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
    if (jj < i) c[DR_A + i * (i - 1) / 2 + jj] = beta[i] * rij * dots[i * 8 + jj];
    c[DR_B + i * 8 + jj] = jj <= i ? rij * dots[64 + i * 8 + jj] : 0.f;
    if (i == 7) c[DR_W + jj] = rij;
    if (jj == 0) {
      const float gam = g[0] * rij;                   // rij is g_1 .. g_i here
      c[DR_G + i] = gam;
      c[DR_BG + i] = beta[i] * gam;
      if (i == 7) c[DR_GL] = gam, c[DR_GL + 1] = c[DR_GL + 2] = c[DR_GL + 3] = 0.f;
    }
  }
  for (int e = tid + blockDim.x; e < R * Dvp; e += blockDim.x) {        // the value channels beyond a thread's first
    float y[DR_CHUNK];
    value(e, y);
    put_value(e, y);
  }
}

__host__ __device__ constexpr int dr_log2(int n) { return n <= 1 ? 0 : 1 + dr_log2(n / 2); }

__device__ __forceinline__ void dr_bulk_copy(uint32_t dst, const float* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst),
               "l"(src), "r"(bytes), "r"(bar)
               : "memory");
}
// Eight neighbouring floats of shared memory, 16-byte aligned.
__device__ __forceinline__ void dr_load8(const float* p, float* x) {
  const float4 a = *reinterpret_cast<const float4*>(p), c = *reinterpret_cast<const float4*>(p + 4);
  x[0] = a.x, x[1] = a.y, x[2] = a.z, x[3] = a.w, x[4] = c.x, x[5] = c.y, x[6] = c.z, x[7] = c.w;
}

// CPG columns of S per group of LANES lanes; lane r of a group owns dims 4 (r + LANES i) + 0..3, i < NI, of each.
// Chunks come into a ring of shared-memory stages by bulk copies of one thread, two chunks ahead.
//
// How a chunk's partial products are added up.  A lane's bits say, from the top, which tokens, which column and which
// copy of them it ends up with: TB token bits (a lane ends with NT = 8 >> TB neighbouring tokens), CB column bits, the
// rest copies.  A lane takes the rows of k or q in the order i ^ (its token bits) and keeps column p ^ (its column) at
// place p of its registers, so that at every halving what it keeps lies in the lower half of its array and what its
// partner is owed in the upper half: one shuffle and one addition a value, no selects.  The same order gives every lane
// the other columns' u with one shuffle each.
template <int LANES, int NI, int CPG>
__global__ void __launch_bounds__(128)
delta_scan_kernel(const float* __restrict__ qk, const float* __restrict__ vv, const float* __restrict__ co,
                  float* __restrict__ out, float* __restrict__ state, size_t slot_stride,
                  const int* __restrict__ seq_start, const int* __restrict__ seq_slot, int H, int G, int D, int Dv,
                  int n_slots) {
  extern __shared__ __align__(128) float dr_smem[];
  __shared__ __align__(8) uint64_t dr_bars[DR_STAGES];
  constexpr int GROUPS = 32 / LANES, CB = dr_log2(CPG), LB = dr_log2(LANES);
  constexpr int TB = LB - CB < 3 ? LB - CB : 3, DUP = LB - CB - TB, NT = 8 >> TB;
  constexpr int DL = 4 * LANES * NI;                   // dims of a staged row (beyond D: zeros)
  const int cols = (blockDim.x >> 5) * GROUPS * CPG;   // columns of the CTA
  const int Dvp = (Dv + 3) & ~3;
  const int stage_len = 2 * DR_CHUNK * DL + DR_COEF + DR_CHUNK * cols;
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, grp = lane / LANES, r = lane % LANES;
  const int b = blockIdx.z, h = blockIdx.y, c_cta = blockIdx.x * cols;
  const int c_loc = (warp * GROUPS + grp) * CPG, c0 = c_cta + c_loc;   // this group's first column
  const int tl = r >> (CB + DUP), cl = (r >> DUP) & (CPG - 1), flip = tl << (3 - TB);
  const int row0 = seq_start[b], n_new = seq_start[b + 1] - row0, sl = seq_slot[b];
  if (n_new <= 0) return;
  if (sl < 0 || sl >= n_slots) {
    if (tid == 0) llmx_report(2);
    return;
  }
  float* S = state + (size_t)sl * slot_stride + (size_t)h * D * Dv;
  const int slot0 = row0 / DR_CHUNK + b, n_chunks = (n_new + DR_CHUNK - 1) / DR_CHUNK;
  const int j = h / (H / G);
  const uint32_t bars = smem_u32(dr_bars), ring = smem_u32(dr_smem);
  if (tid == 0) {
    for (int i = 0; i < DR_STAGES; ++i) mbar_init(bars + 8 * i, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  const uint32_t v_bytes = (uint32_t)(DR_CHUNK * min(cols, Dvp - c_cta)) * 4u;
  auto load_chunk = [&](int ch) {                      // one thread
    if (llmx_withhold && ch == 0 && (blockIdx.x | blockIdx.y | blockIdx.z) == 0) return;     // (tests: never asked for)
    const int st = ch % DR_STAGES;
    const uint32_t dst = ring + (uint32_t)(st * stage_len) * 4u, bar = bars + 8 * st;
    mbar_expect_tx(bar, 2u * DR_CHUNK * DL * 4u + DR_COEF * 4u + v_bytes);
    dr_bulk_copy(dst, qk + ((size_t)(slot0 + ch) * G + j) * 2 * DR_CHUNK * DL, 2u * DR_CHUNK * DL * 4u, bar);
    dr_bulk_copy(dst + 2u * DR_CHUNK * DL * 4u, co + ((size_t)(slot0 + ch) * H + h) * DR_COEF, DR_COEF * 4u, bar);
    dr_bulk_copy(dst + (2u * DR_CHUNK * DL + DR_COEF) * 4u, vv + (((size_t)(slot0 + ch) * H + h) * Dvp + c_cta) * DR_CHUNK,
                 v_bytes, bar);
  };
  __syncthreads();
  pdl_wait();
  if (tid == 0)
    for (int c = 0; c < DR_STAGES - 1 && c < n_chunks; ++c) load_chunk(c);

  float s[NI][4][CPG];                                 // [dims block][dim][column c0 + (place ^ cl)]
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int d = 0; d < 4; ++d)
#pragma unroll
      for (int c = 0; c < CPG; ++c) {
        const int dim = 4 * (r + LANES * i) + d, col = c0 + (c ^ cl);
        s[i][d][c] = (dim < D && col < Dv) ? S[(size_t)dim * Dv + col] : 0.f;
      }
  const bool writes = c0 + cl < Dv && (r & ((1 << DUP) - 1)) == 0;
  const size_t out_stride = (size_t)H * Dv;
  float* out_col = out + ((size_t)row0 + tl * NT) * out_stride + (size_t)h * Dv + c0 + cl;    // its first token of a chunk
  for (int ch = 0; ch < n_chunks; ++ch) {
    // this chunk has landed; everyone has left the one before, whose stage the next copy fills
    const bool ok = mbar_wait(bars + 8 * (ch % DR_STAGES), (ch / DR_STAGES) & 1);
    if (!__syncthreads_and(ok)) {
      if (tid == 0) llmx_report(5);
      break;
    }
    if (tid == 0 && ch + DR_STAGES - 1 < n_chunks) load_chunk(ch + DR_STAGES - 1);
    const float* kbuf = dr_smem + (ch % DR_STAGES) * stage_len;
    const float* qbuf = kbuf + DR_CHUNK * DL;
    const float* cbuf = qbuf + DR_CHUNK * DL;
    const float* vbuf = cbuf + DR_COEF;
    // ---- rows . S over this lane's dims, then over the group: afterwards res[e] belongs to token tl NT + e, column cl
    auto products = [&](const float* rows, float* res) {
      float acc[DR_CHUNK][CPG];
#pragma unroll
      for (int i = 0; i < DR_CHUNK; ++i) {
#pragma unroll
        for (int c = 0; c < CPG; ++c) acc[i][c] = 0.f;
        const float* row = rows + (i ^ flip) * DL + 4 * r;
#pragma unroll
        for (int ni = 0; ni < NI; ++ni) {
          const float4 x = *reinterpret_cast<const float4*>(row + 4 * LANES * ni);
#pragma unroll
          for (int c = 0; c < CPG; ++c) {
            acc[i][c] = fmaf(x.x, s[ni][0][c], acc[i][c]);
            acc[i][c] = fmaf(x.y, s[ni][1][c], acc[i][c]);
            acc[i][c] = fmaf(x.z, s[ni][2][c], acc[i][c]);
            acc[i][c] = fmaf(x.w, s[ni][3][c], acc[i][c]);
          }
        }
      }
#pragma unroll
      for (int t = 0; t < TB; ++t) {
        const int half = 4 >> t;
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (i < half)
#pragma unroll
            for (int c = 0; c < CPG; ++c) acc[i][c] += __shfl_xor_sync(0xffffffffu, acc[i + half][c], LANES >> (t + 1));
      }
#pragma unroll
      for (int t = 0; t < CB; ++t) {
        const int half = CPG >> (t + 1);
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
          for (int c = 0; c < CPG / 2; ++c)
            if (c < half) acc[i][c] += __shfl_xor_sync(0xffffffffu, acc[i][c + half], half << DUP);
      }
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        res[i] = acc[i][0];
#pragma unroll
        for (int t = 0; t < DUP; ++t) res[i] += __shfl_xor_sync(0xffffffffu, res[i], 1 << t);
      }
    };
    float ks_own[NT], qs[NT], u[DR_CHUNK], w[DR_CHUNK];
    products(kbuf, ks_own);
    products(qbuf, qs);
    // ---- the chain from token to token, for this lane's column (every lane of a column alike)
    {
      float bg[DR_CHUNK], a[28];
      dr_load8(vbuf + (c_loc + cl) * 8, u);
      dr_load8(cbuf + DR_BG, bg);
#pragma unroll
      for (int i = 0; i < 28; i += 4) {
        const float4 x = *reinterpret_cast<const float4*>(cbuf + DR_A + i);
        a[i] = x.x, a[i + 1] = x.y, a[i + 2] = x.z, a[i + 3] = x.w;
      }
      const int base = lane & ~((LANES - 1) & ~((1 << (CB + DUP)) - 1));      // token bits cleared
#pragma unroll
      for (int i = 0; i < DR_CHUNK; ++i) {
        const float ks = __shfl_sync(0xffffffffu, ks_own[i % NT], base | ((i / NT) << (CB + DUP)));
        u[i] = fmaf(-bg[i], ks, u[i]);
      }
#pragma unroll
      for (int i = 1; i < DR_CHUNK; ++i)
#pragma unroll
        for (int m = 0; m < i; ++m) u[i] = fmaf(-a[i * (i - 1) / 2 + m], u[m], u[i]);
    }
    dr_load8(cbuf + DR_W, w);
    const float gl = cbuf[DR_GL];
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) w[i] *= u[i];
#pragma unroll
    for (int ni = 0; ni < NI; ++ni)
#pragma unroll
      for (int d = 0; d < 4; ++d)
#pragma unroll
        for (int c = 0; c < CPG; ++c) s[ni][d][c] *= gl;
#pragma unroll
    for (int i = 0; i < DR_CHUNK; ++i) {
      float wc[CPG];
      wc[0] = w[i];
#pragma unroll
      for (int c = 1; c < CPG; ++c) wc[c] = __shfl_xor_sync(0xffffffffu, w[i], c << DUP);
#pragma unroll
      for (int ni = 0; ni < NI; ++ni) {
        const float4 x = *reinterpret_cast<const float4*>(kbuf + i * DL + 4 * (r + LANES * ni));
#pragma unroll
        for (int c = 0; c < CPG; ++c) {
          s[ni][0][c] = fmaf(x.x, wc[c], s[ni][0][c]);
          s[ni][1][c] = fmaf(x.y, wc[c], s[ni][1][c]);
          s[ni][2][c] = fmaf(x.z, wc[c], s[ni][2][c]);
          s[ni][3][c] = fmaf(x.w, wc[c], s[ni][3][c]);
        }
      }
    }
    // ---- outputs
    const int n_tok = n_new - ch * DR_CHUNK;
#pragma unroll
    for (int e = 0; e < NT; ++e) {
      const int i = tl * NT + e;
      float bi[DR_CHUNK];
      dr_load8(cbuf + DR_B + i * 8, bi);
      float o = cbuf[DR_G + i] * qs[e];
#pragma unroll
      for (int m = 0; m < DR_CHUNK; ++m) o = fmaf(bi[m], u[m], o);
      if (writes && i < n_tok) out_col[e * out_stride] = o;
    }
    out_col += DR_CHUNK * out_stride;
  }
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int d = 0; d < 4; ++d)
#pragma unroll
      for (int c = 0; c < CPG; ++c) {
        const int dim = 4 * (r + LANES * i) + d, col = c0 + (c ^ cl);
        if (dim < D && col < Dv) S[(size_t)dim * Dv + col] = s[i][d][c];
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
  extern __shared__ __align__(128) float dr_smem[];
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
  // ... then what the end needs of the projection, and the head's gates
  float z_own = 0.f;
  if (tid < Dv) z_own = dr_value(row, in.g_off + h * Dv + tid, in.n_split, in.split_stride);
  if (tid == 255) {
    sums[3] = dr_sigmoid(dr_value(row, in.b_off + h, in.n_split, in.split_stride));
    const float a = dr_value(row, in.a_off + h, in.n_split, in.split_stride);
    sums[4] = expf(-expf(in.a_log[h]) * dr_softplus(a + in.dt_bias[h]));
  }
  // ---- convolution, activation; the token's projected row joins the ring
  const int p_place = p % taps;
  for (int e = tid; e < 2 * D + Dv; e += 256) {
    const int c = e < D ? j * D + e : e < 2 * D ? G * D + j * D + (e - D) : 2 * G * D + h * Dv + (e - 2 * D);
    const float own = dr_value(row, dr_column(in, c), in.n_split, in.split_stride);
    float acc = 0.f;
    int place = p_place;                                  // the row of position p - taps + 1: the one behind p's
#pragma unroll 4
    for (int m = 0; m < taps; ++m) {
      place = place + 1 == taps ? 0 : place + 1;
      const float u = m == taps - 1 ? own : p - taps + 1 + m >= 0 ? ring[(size_t)place * C + c] : 0.f;
      acc = fmaf(in.conv_w[(size_t)m * C + c], u, acc);
    }
    if (taps > 1) ring[(size_t)p_place * C + c] = own;      // (heads that share a key head write the same number)
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
    const float z = c == tid ? z_own : dr_value(row, in.g_off + h * Dv + c, in.n_split, in.split_stride);
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
// [chunks, G, 16, DL] (DL: D rounded up to 32, 64, 128 or 256), [chunks, H, Dvp, 8], [chunks, H, 120]; out float32 [T, H*Dv].
LLMX_API int llmx_delta_prompt(const void* proj, int in_dtype, int n_split, long long split_stride, long long row_stride,
                               int q_off, int k_off, int v_off, int b_off, int a_off, int g_off, const float* conv_w,
                               int taps, const float* a_log, const float* dt_bias, float q_scale, float unit_eps,
                               float* state, long long slot_stride, long long ring_off, int n_slots, float* qk, float* vv,
                               float* co, float* out, const int* seq_start, const int* seq_past, const int* seq_slot,
                               int n_tokens, int n_seqs, int H, int G, int D, int Dv, int n_sm, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  const DeltaIn in = {n_split, (size_t)split_stride, (size_t)row_stride, q_off, k_off, v_off, b_off, a_off, g_off,
                      conv_w, a_log, dt_bias, taps, H, G, D, Dv, q_scale, unit_eps, (size_t)slot_stride, (size_t)ring_off};
  const int bad = dr_check(in, row_stride);
  if (bad) return bad;
  if (n_seqs > 65535 || H > 65535 || (((uintptr_t)qk | (uintptr_t)vv | (uintptr_t)co | (uintptr_t)state) & 15)) return LLMX_REFUSED(3);
  if (in_dtype != LLMX_F32 && in_dtype != LLMX_BF16) return LLMX_REFUSED(2);
  const int Dp = (D + 3) & ~3, R = H / G, DL = Dp <= 32 ? 32 : Dp <= 64 ? 64 : Dp <= 128 ? 128 : 256;
  const size_t psmem = (size_t)(2 * DR_CHUNK * (Dp + DR_PAD) + 128 + R * 16) * sizeof(float);
  if (psmem > 48 * 1024) return LLMX_REFUSED(3);
  const dim3 pgrid(n_tokens / DR_CHUNK + n_seqs, G);
#define PREP(TIN, TAPS)                                                                                                 \
  launch_pdl(delta_prep_kernel<TIN, TAPS>, pgrid, dim3(256), psmem, stream, (const TIN*)proj, in, (const float*)state,  \
             qk, vv, co, seq_start, seq_past, seq_slot, n_seqs, n_tokens, n_slots, DL)
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
  // Launched in order, never beside the preparation: its CTAs all run at once for the whole prompt, and those placed
  // while another kernel still fills part of the GPU would stay crowded on the SMs that had room (measured: twice the
  // time).
  // Two columns a group while that leaves the GPU less than two warps a scheduler, else four; fewer warps a CTA while
  // there are fewer CTAs than SMs.
  const int groups = Dp <= 32 ? 4 : Dp <= 64 ? 2 : 1;                   // lane groups per warp
  const long long heads = (long long)n_seqs * H;
  const int cpg = heads * ((Dv + 4 * groups - 1) / (4 * groups)) < 8LL * n_sm ? 2 : 4;
  int warps = 4;
  while (warps > 1 && heads * ((Dv + warps * groups * cpg - 1) / (warps * groups * cpg)) < n_sm) warps >>= 1;
  const int cols = warps * groups * cpg;
  const size_t smem = (size_t)DR_STAGES * (2 * DR_CHUNK * DL + DR_COEF + DR_CHUNK * cols) * sizeof(float);
#define SCAN2(LANES, NI, CPG)                                                                                           \
  do {                                                                                                                  \
    static bool attr_set = false;                                                                                       \
    if (!attr_set && smem > 48 * 1024) {                                                                                \
      e = cudaFuncSetAttribute(delta_scan_kernel<LANES, NI, CPG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024); \
      if (e != cudaSuccess) return (int)e;                                                                              \
      attr_set = true;                                                                                                  \
    }                                                                                                                   \
    delta_scan_kernel<LANES, NI, CPG><<<dim3((Dv + cols - 1) / cols, H, n_seqs), warps * 32, smem, stream>>>(           \
        qk, vv, co, out, state, (size_t)slot_stride, seq_start, seq_slot, H, G, D, Dv, n_slots);                        \
  } while (0)
#define SCAN(LANES, NI)               \
  do {                                \
    if (cpg == 2) SCAN2(LANES, NI, 2); \
    else SCAN2(LANES, NI, 4);         \
  } while (0)
  if (Dp <= 32) SCAN(8, 1);
  else if (Dp <= 64) SCAN(16, 1);
  else if (Dp <= 128) SCAN(32, 1);
  else SCAN(32, 2);
#undef SCAN2
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
