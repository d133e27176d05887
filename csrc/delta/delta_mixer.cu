// K16d: gated delta rule over ragged portions of sequences, with what surrounds it in the layer.  Per token, head h of H and
// the query / key head g = h / (H / G):
//
//   q, k, v = silu(causal depthwise convolution over time of the projected rows)
//   q = q / sqrt(sum q^2 + 1e-6) / sqrt(dk),  k = k / sqrt(sum k^2 + 1e-6)
//   beta = sigmoid(b),  decay = exp(-exp(a_log) * softplus(a + dt_bias))
//   S <- decay * S,  u = beta * (v - S^T k),  S <- S + k u^T,  o = S^T q                  S [dk, dv]
//   out = o / sqrt(mean(o^2) + eps) * w * silu(gate)
//
// (or sigmoid(gate)).  With one decay per key channel, decay = exp(-exp(a_log) * softplus(raw + dt_bias)) is a vector over the rows
// of S, raw and dt_bias have a value per head and channel.
//
// Everything between the loads and `out` is fp32; the projected rows and `out` have the element type of the matrix products.
// A portion reads its sequence's state rows (none: zero) and leaves the new state in other rows, so every CTA of a launch may
// read the old ones whenever it runs.  Rows of heads are padded to multiples of 8 with zeros, which stay zero.
//
// One token per sequence (delta_step): a CTA per head and sequence; the state passes through registers once.
//
// Portions: delta_prep makes q, k and v of blocks of 16 tokens, delta_solve two triangular matrices per block and head; delta_scan
// carries the state through the blocks; delta_finish normalises and gates.  Within a block, with the running sum c of the log
// decays, the definition above is
//
//   u_i + beta_i sum_(j < i) e^(c_i - c_j) (k_i . k_j) u_j = beta_i (v_i - e^(c_i) S^T k_i)
//   o_i = e^(c_i) S^T q_i + sum_(j <= i) e^(c_i - c_j) (q_i . k_j) u_j
//   S  <- e^(c_end) S + sum_j e^(c_end - c_j) k_j u_j^T
//
// with the S that enters the block.  So with x_j = v_j - e^(c_j) S^T k_j and the inverse T of the unit triangular system (times
// beta), u = T x and o = e^c S^T q + W x, W = (decayed q k^T) T: T and W hold no column of S, are made once per block and head,
// and the scan is left with products.  Entries of T are at most one (products of contractions), exponents never positive.
// Columns of S do not meet: a warp owns a few of them.
//
// Decays per channel put vectors in the place of e^c: with D(i, j) the diagonal of the products of the decays of tokens j + 1 .. i,
// the pair products are k_i^T D(i, j) k_j and q_i^T D(i, j) k_j, made per value head by walking i upwards with the running product
// (delta_prep_channel): no exponential, nothing is divided by a decay, all factors are at most one.  What the scan reads are then
// D(i, -1) k_i and D(i, -1) q_i in front of S and D(end, j) k_j behind it.
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace delta {

constexpr int BT = 16;        // tokens per block

__device__ __forceinline__ float silu(float v) { return __fdividef(v, 1.f + __expf(-v)); }
__device__ __forceinline__ float softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float log_decay(const UbDeltaArgs& a, float x, int h) { return -expf(a.a_log[h]) * softplus(x + a.dt_bias[h]); }

__device__ __forceinline__ float channel_decay(const UbDeltaArgs& a, long long row, int h, int d, float rate /* exp(a_log) */) {
  return expf(-rate * softplus(a.decay[row * a.ld_decay + (long long)h * a.dk + d] + a.dt_bias[(long long)h * a.dk + d]));
}
__device__ __forceinline__ float out_gate(const UbDeltaArgs& a, float v) {
  const float s = __fdividef(1.f, 1.f + __expf(-v));
  return a.gate_act == 1 ? s : v * s;
}

__device__ __forceinline__ int state_row(const UbDeltaArgs& a, const int* rows, int seq) {
  const int r = rows != nullptr ? rows[seq] : -1;
  if (r >= a.state_rows) {
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, seq);
    return -1;
  }
  return r;
}

// ------------------------------------------------------------------------------------------------------------------------
// one token per sequence
// ------------------------------------------------------------------------------------------------------------------------
// NT threads; ROWS: rows of S that a thread holds (four columns each); 0: S is read twice instead (heads too large for registers).
template <typename T, int NT, int ROWS, bool CH>
__global__ void __launch_bounds__(NT, ROWS <= 8 ? 768 / NT : ROWS <= 16 ? 512 / NT : 1) delta_step_kernel(const UbDeltaArgs a, const int cl /* threads across the columns */) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int HELD = ROWS > 0 ? ROWS : 1;
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.x, seq = blockIdx.y, dk = a.dk, dv = a.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nrg = NT / cl, rg = tid / cl, col = (tid % cl) * 4;
  float* qkv = sm;                               // [2 dk + dv] after the convolutions
  float* part = qkv + 2 * dk + dv;               // [8][2][dv] partial products with the old state
  float* u_s = part + 8 * 2 * dv;            // [dv]
  float* o_s = u_s + dv;                         // [dv]
  float* sc = o_s + dv;                          // scalars: 1 / |q|, 1 / |k|, q . k, beta, decay; then eight sums
  float* dec = sc + 16;                          // [dk] decays of the rows (CH)
  const int group = a.H / a.G, g = h / group, m = a.taps - 1, C = 2 * a.G * dk + a.H * dv;
  const long long row = a.row0 + seq;
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  const bool on = col < dv;
  const float* src = a.state + ((long long)max(si, 0) * a.H + h) * dk * dv + col;
  float* dst = a.state + ((long long)max(so, 0) * a.H + h) * dk * dv + col;

  float4 S[HELD];
#pragma unroll
  for (int i = 0; i < HELD; ++i) S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  if (ROWS > 0 && si >= 0 && on) {
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
      const int r = rg + i * nrg;
      if (r < dk) S[i] = __ldcs(reinterpret_cast<const float4*>(src + (long long)r * dv));
    }
  }
  // convolutions of this head's channels; the oldest input leaves, the current one joins.  Four taps (of two
  // channels, where a thread holds little of S) are requested together.
  constexpr int CU = NT == 128 ? 2 : 1;
  for (int c0 = tid; c0 < 2 * dk + dv; c0 += CU * NT) {
    float acc[CU], cur[CU];
    int ch[CU];
    bool in[CU], keep[CU];
#pragma unroll
    for (int u = 0; u < CU; ++u) {
      const int c = c0 + u * NT;
      acc[u] = 0.f;
      in[u] = c < 2 * dk + dv;
      ch[u] = !in[u] ? 0 : c < dk ? g * dk + c : c < 2 * dk ? a.G * dk + g * dk + (c - dk) : 2 * a.G * dk + h * dv + (c - 2 * dk);
      keep[u] = in[u] && so >= 0 && (c >= 2 * dk || h % group == 0);
      cur[u] = (float)reinterpret_cast<const T*>(a.qkv)[row * a.ld + ch[u]];
    }
    const T* w = reinterpret_cast<const T*>(a.conv);
    for (int j0 = 0; j0 < a.taps; j0 += 4) {
      float v[CU][4], k[CU][4];
#pragma unroll
      for (int u = 0; u < CU; ++u)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = j0 + j;
          k[u][j] = r < a.taps ? (float)w[(long long)r * C + ch[u]] : 0.f;
          v[u][j] = r < m ? (si >= 0 ? a.conv_state[((long long)si * m + r) * C + ch[u]] : 0.f) : cur[u];
        }
#pragma unroll
      for (int u = 0; u < CU; ++u)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = j0 + j;
          if (r >= a.taps) break;
          acc[u] = fmaf(k[u][j], v[u][j], acc[u]);
          if (keep[u] && r > 0) a.conv_state[((long long)so * m + r - 1) * C + ch[u]] = v[u][j];
        }
    }
#pragma unroll
    for (int u = 0; u < CU; ++u)
      if (in[u]) qkv[c0 + u * NT] = silu(acc[u]);
  }
  float gate = 0.f, nw = 0.f;                    // dv <= NT (launch_step)
  if (tid < dv) {
    gate = (float)reinterpret_cast<const T*>(a.gate)[row * a.ld_gate + (long long)h * dv + tid];
    nw = a.norm_w[tid];
  }
  if (CH) {
    const float rate = expf(a.a_log[h]);
    for (int d = tid; d < dk; d += NT) dec[d] = channel_decay(a, row, h, d, rate);
  }
  if (tid == 0) {
    sc[3] = 1.f / (1.f + expf(-(float)reinterpret_cast<const T*>(a.b)[row * a.ld + h]));
    sc[4] = CH ? 1.f : expf(log_decay(a, (float)reinterpret_cast<const T*>(a.a)[row * a.ld + h], h));
  }
  __syncthreads();
  if (warp < 3) {                                // |q|^2, |k|^2, q . k
    const float *x = warp == 1 ? qkv + dk : qkv, *y = warp == 0 ? qkv : qkv + dk;
    float s = 0.f;
    for (int i = lane; i < dk; i += 32) s = fmaf(x[i], y[i], s);
    s = warp_sum(s);
    if (lane == 0) sc[warp] = warp < 2 ? 1.f / sqrtf(s + 1e-6f) : s;
  }
  float4 P = make_float4(0.f, 0.f, 0.f, 0.f), R = P;          // S^T k and S^T q, up to the factors of k and q
  auto meet = [&](const float4 s, int r) {
    float kk = qkv[dk + r], qq = qkv[r];
    if (CH) { kk *= dec[r]; qq *= dec[r]; }
    P.x = fmaf(s.x, kk, P.x); P.y = fmaf(s.y, kk, P.y); P.z = fmaf(s.z, kk, P.z); P.w = fmaf(s.w, kk, P.w);
    R.x = fmaf(s.x, qq, R.x); R.y = fmaf(s.y, qq, R.y); R.z = fmaf(s.z, qq, R.z); R.w = fmaf(s.w, qq, R.w);
  };
  if (si >= 0 && on) {
    if (ROWS > 0) {
#pragma unroll
      for (int i = 0; i < HELD; ++i)
        if (rg + i * nrg < dk) meet(S[i], rg + i * nrg);
    } else {
      for (int r = rg; r < dk; r += nrg) meet(*reinterpret_cast<const float4*>(src + (long long)r * dv), r);
    }
  }
  // row groups inside a warp first (cl < 32), then the partial sums of all warps through shared memory
  for (int o = cl; o < 32; o <<= 1) {
    P.x += __shfl_xor_sync(0xffffffffu, P.x, o); P.y += __shfl_xor_sync(0xffffffffu, P.y, o);
    P.z += __shfl_xor_sync(0xffffffffu, P.z, o); P.w += __shfl_xor_sync(0xffffffffu, P.w, o);
    R.x += __shfl_xor_sync(0xffffffffu, R.x, o); R.y += __shfl_xor_sync(0xffffffffu, R.y, o);
    R.z += __shfl_xor_sync(0xffffffffu, R.z, o); R.w += __shfl_xor_sync(0xffffffffu, R.w, o);
  }
  const int slot = cl >= 32 ? rg : warp, nslots = cl >= 32 ? nrg : NT / 32;
  if (on && (cl >= 32 || lane < cl)) {
    *reinterpret_cast<float4*>(part + (slot * 2) * dv + col) = P;
    *reinterpret_cast<float4*>(part + (slot * 2 + 1) * dv + col) = R;
  }
  __syncthreads();
  const float rk = sc[1], rq = sc[0] * (1.f / sqrtf((float)a.dk_real)), beta = sc[3], decay = sc[4];
  float o = 0.f;
  if (tid < dv) {
    float p = 0.f, r = 0.f;
    for (int s = 0; s < nslots; ++s) { p += part[(s * 2) * dv + tid]; r += part[(s * 2 + 1) * dv + tid]; }
    const float u = beta * (qkv[2 * dk + tid] - decay * rk * p);
    o = fmaf(sc[2] * rq * rk, u, decay * rq * r);
    u_s[tid] = u;
  }
  const float sq = warp_sum(o * o);
  if (lane == 0) sc[8 + warp] = sq;
  __syncthreads();
  if (tid < dv) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < NT / 32; ++w) s += sc[8 + w];
    reinterpret_cast<T*>(a.out)[row * a.ld_out + (long long)h * dv + tid] = T(o * (1.f / sqrtf(s / a.dv_real + a.eps)) * nw * out_gate(a, gate));
  }
  if (so >= 0 && on) {
    const float4 u = *reinterpret_cast<const float4*>(u_s + col);
    auto write = [&](float4 s, int r) {
      const float kk = qkv[dk + r] * rk, g = CH ? dec[r] : decay;
      s.x = fmaf(kk, u.x, g * s.x); s.y = fmaf(kk, u.y, g * s.y);
      s.z = fmaf(kk, u.z, g * s.z); s.w = fmaf(kk, u.w, g * s.w);
      __stcs(reinterpret_cast<float4*>(dst + (long long)r * dv), s);
    };
    if (ROWS > 0) {
#pragma unroll
      for (int i = 0; i < HELD; ++i)
        if (rg + i * nrg < dk) write(S[i], rg + i * nrg);
    } else {
      for (int r = rg; r < dk; r += nrg)
        write(si >= 0 ? *reinterpret_cast<const float4*>(src + (long long)r * dv) : make_float4(0.f, 0.f, 0.f, 0.f), r);
    }
  }
}

template <typename T, bool CH>
static cudaError_t launch_step(const UbDeltaArgs& a, cudaStream_t st) {
  int cl = 2;
  while (cl * 4 < a.dv) cl <<= 1;                // <= 64
  const int nt = a.dv <= 128 && a.dk * a.dv <= 64 * 64 ? 128 : 256;          // small states: more CTAs per SM
  const int nrg = nt / cl, need = (a.dk + nrg - 1) / nrg;
  const size_t smem = sizeof(float) * (2 * a.dk + a.dv + 16 * a.dv + 2 * a.dv + 16 + (CH ? a.dk : 0));
  const dim3 grid(a.H, a.num_seqs), block(nt);
  auto go = [&](auto kern) { return launch_pdl(kern, grid, block, smem, st, a, cl); };
  if (nt == 128) {
    if (need <= 2) return go(delta_step_kernel<T, 128, 2, CH>);
    if (need <= 8) return go(delta_step_kernel<T, 128, 8, CH>);
    if (need <= 32) return go(delta_step_kernel<T, 128, 32, CH>);
    return go(delta_step_kernel<T, 128, 0, CH>);
  }
  if (need <= 8) return go(delta_step_kernel<T, 256, 8, CH>);
  if (need <= 16) return go(delta_step_kernel<T, 256, 16, CH>);
  if (need <= 32) return go(delta_step_kernel<T, 256, 32, CH>);
  return go(delta_step_kernel<T, 256, 0, CH>);
}

// ------------------------------------------------------------------------------------------------------------------------
// portions: what the scan reads
// ------------------------------------------------------------------------------------------------------------------------
// workspace, per row of the launch: q and k [2 G dk], v (later o) [H dv], the row's entries of T and W [H][2][16], (-e^c, e^c,
// e^(c_end - c), 0) [H][4], k.k and q.k with the tokens of the row's block [G][2][16].  With decays per channel: decayed q, decayed k
// and k decayed to the block's end [3 H dk], the products per value head [H][2][16], and behind them, per block and head, the
// products of the block's decays [dk].
__device__ __forceinline__ int qk_row(const UbDeltaArgs& a) { return a.decay != nullptr ? 3 * a.H * a.dk : 2 * a.G * a.dk; }
__device__ __forceinline__ float* ws_qk(const UbDeltaArgs& a) { return a.ws; }
__device__ __forceinline__ float* ws_v(const UbDeltaArgs& a) { return a.ws + (long long)a.rows * qk_row(a); }
__device__ __forceinline__ float* ws_tw(const UbDeltaArgs& a) { return ws_v(a) + (long long)a.rows * a.H * a.dv; }
__device__ __forceinline__ float* ws_gl(const UbDeltaArgs& a) { return ws_tw(a) + (long long)a.rows * a.H * 2 * BT; }
__device__ __forceinline__ float* ws_gram(const UbDeltaArgs& a) { return ws_gl(a) + (long long)a.rows * a.H * 4; }

__device__ __forceinline__ float* ws_end(const UbDeltaArgs& a) { return ws_gram(a) + (long long)a.rows * a.H * 2 * BT; }
// number of a sequence's first block among those of the launch: the gaps between sequences are harmless
__device__ __forceinline__ long long first_block(int qs, int seq) { return qs / BT + seq; }

constexpr int PREP_T = 256;
constexpr int LDM = BT + 1;                      // row of a 16 x 16 matrix in shared memory
constexpr int LDH = 2 * BT * LDM + BT;           // two of them per value head, half the banks apart from the next head's

// Two tokens of eight neighbouring channels behind convolution and silu: channel `ch` of the rows, c8 on their own axis.
template <typename T>
__device__ __forceinline__ void conv_pair(const UbDeltaArgs& a, long long row, int t, int q_len, int si, int ch, int C, float (&y)[2][8]) {
  const int m = a.taps - 1;
#pragma unroll
  for (int e = 0; e < 8; ++e) y[0][e] = y[1][e] = 0.f;
  const T* w = reinterpret_cast<const T*>(a.conv) + ch;
  auto input = [&](int tt, float (&v)[8]) {
    if (tt >= 0 && tt < q_len) {
      load8(reinterpret_cast<const T*>(a.qkv) + (row + tt) * a.ld + ch, v);
    } else if (tt < 0 && si >= 0) {
      load8(a.conv_state + ((long long)si * m + m + tt) * C + ch, v);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = 0.f;
    }
  };
  // input t - m + j meets tap j of token t and tap j - 1 of token t + 1
  float before[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) before[e] = 0.f;
#pragma unroll 4
  for (int j = 0; j <= m; ++j) {
    float v[8], k[8];
    input(t - m + j, v);
    load8(w + (long long)j * C, k);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      y[0][e] = fmaf(k[e], v[e], y[0][e]);
      y[1][e] = fmaf(before[e], v[e], y[1][e]);
      before[e] = k[e];
    }
  }
  float v[8];
  input(t + 1, v);
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    y[0][e] = silu(y[0][e]);
    y[1][e] = silu(fmaf(before[e], v[e], y[1][e]));
  }
}

// The last taps - 1 inputs of a portion are the sequence's state: eight channels of them.
template <typename T>
__device__ __forceinline__ void keep_inputs(const UbDeltaArgs& a, long long row, int q_len, int si, int so, int ch, int C) {
  const int m = a.taps - 1;
  for (int r = 0; r < m; ++r) {
    const int t = q_len - m + r;
    float v[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = 0.f;
    if (t >= 0) load8(reinterpret_cast<const T*>(a.qkv) + (row + t) * a.ld + ch, v);
    else if (si >= 0) load8(a.conv_state + ((long long)si * m + m + t) * C + ch, v);
    store8(a.conv_state + ((long long)so * m + r) * C + ch, v);
  }
}

// Sixteen tokens of 256 value channels.
template <typename T>
__device__ __forceinline__ void prep_values(const UbDeltaArgs& a, int unit, long long row, long long wrow, int t0, int q_len, int si, int so, bool last) {
  const int tid = threadIdx.x, C = 2 * a.G * a.dk + a.H * a.dv;
  const int c = unit * PREP_T + (tid % 32) * 8, t = t0 + (tid / 32) * 2;
  if (c >= a.H * a.dv) return;
  const int ch = 2 * a.G * a.dk + c;
  float y[2][8];
  if (t < q_len) {
    conv_pair<T>(a, row, t, q_len, si, ch, C, y);
    store8(ws_v(a) + (wrow + t) * a.H * a.dv + c, y[0]);
    if (t + 1 < q_len) store8(ws_v(a) + (wrow + t + 1) * a.H * a.dv + c, y[1]);
  }
  if (last && tid < 32) keep_inputs<T>(a, row, q_len, si, so, ch, C);
}

// One block of 16 tokens of one query / key head, or (units G ..) of 256 value channels.
template <typename T>
__global__ void __launch_bounds__(PREP_T) delta_prep_kernel(const UbDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int unit = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int qs = a.q_start[seq], q_len = a.q_start[seq + 1] - qs, t0 = blockIdx.x * BT;
  if (t0 >= q_len) return;
  const int n = min(BT, q_len - t0), dk = a.dk, C = 2 * a.G * dk + a.H * a.dv;
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  const bool last = so >= 0 && t0 + n == q_len;
  const long long row = a.row0 + qs, wrow = qs;  // rows of the step / of the workspace
  float y[2][8];
  if (unit >= a.G) {
    prep_values<T>(a, unit - a.G, row, wrow, t0, q_len, si, so, last);
    return;
  }
  const int ldy = dk + 4;
  float* qk_s = sm;                              // [2][16][dk + 4] q, then k
  // lanes of one (q or k, two tokens) row pair lie side by side
  const int nch = dk / 8;
  int L = 1;
  while (L < nch) L <<= 1;                       // <= 32
  for (int task = tid / L; task < BT; task += PREP_T / L) {      // q of tokens 0, 1 | k of tokens 0, 1 | q of tokens 2, 3 | ..
    const int part = task & 1, r = (task >> 1) * 2, c = (tid % L) * 8, t = t0 + r;
    const bool on = c < dk && t < q_len;
    const int ch = part * a.G * dk + unit * dk + c;
#pragma unroll
    for (int e = 0; e < 8; ++e) y[0][e] = y[1][e] = 0.f;
    if (on) conv_pair<T>(a, row, t, q_len, si, ch, C, y);
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) { s0 = fmaf(y[0][e], y[0][e], s0); s1 = fmaf(y[1][e], y[1][e], s1); }
    for (int o = L / 2; o > 0; o >>= 1) { s0 += __shfl_xor_sync(0xffffffffu, s0, o); s1 += __shfl_xor_sync(0xffffffffu, s1, o); }
    const float f = part == 0 ? 1.f / sqrtf((float)a.dk_real) : 1.f;
    const float f0 = f / sqrtf(s0 + 1e-6f), f1 = f / sqrtf(s1 + 1e-6f);
    if (c < dk) {
#pragma unroll
      for (int e = 0; e < 8; ++e) { y[0][e] *= f0; y[1][e] = t + 1 < q_len ? y[1][e] * f1 : 0.f; }
      store8(qk_s + (part * BT + r) * ldy + c, y[0]);
      store8(qk_s + (part * BT + r + 1) * ldy + c, y[1]);
      float* dst = ws_qk(a) + (wrow + t) * 2 * a.G * dk + (long long)part * a.G * dk + (long long)unit * dk + c;
      if (t < q_len) store8(dst, y[0]);
      if (t + 1 < q_len) store8(dst + 2LL * a.G * dk, y[1]);
    }
    if (last && on && r == 0) keep_inputs<T>(a, row, q_len, si, so, ch, C);
  }
  __syncthreads();
  {
    const int i = tid / BT, j = tid % BT;        // PREP_T = 16 * 16 pairs
    float kk = 0.f, qk = 0.f;
    if (j <= i) {
      const float *qi = qk_s + i * ldy, *ki = qk_s + (BT + i) * ldy, *kj = qk_s + (BT + j) * ldy;
#pragma unroll 4
      for (int c = 0; c < dk; c += 4) {
        const float4 x = *reinterpret_cast<const float4*>(ki + c), q = *reinterpret_cast<const float4*>(qi + c);
        const float4 z = *reinterpret_cast<const float4*>(kj + c);
        kk = fmaf(x.x, z.x, fmaf(x.y, z.y, fmaf(x.z, z.z, fmaf(x.w, z.w, kk))));
        qk = fmaf(q.x, z.x, fmaf(q.y, z.y, fmaf(q.z, z.z, fmaf(q.w, z.w, qk))));
      }
    }
    if (i < n) {
      float* dst = ws_gram(a) + ((wrow + t0 + i) * a.G + unit) * 2 * BT;
      dst[j] = j < i ? kk : 0.f;
      dst[BT + j] = qk;
    }
  }
}

// The same with decays per channel: one block of 16 tokens of one VALUE head, or (units H ..) of 256 value channels.
template <typename T>
__global__ void __launch_bounds__(PREP_T, 4) delta_prep_channel_kernel(const UbDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int unit = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int qs = a.q_start[seq], q_len = a.q_start[seq + 1] - qs, t0 = blockIdx.x * BT;
  if (t0 >= q_len) return;
  const int n = min(BT, q_len - t0), dk = a.dk, C = 2 * a.G * dk + a.H * a.dv;
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  const bool last = so >= 0 && t0 + n == q_len;
  const long long row = a.row0 + qs, wrow = qs;
  if (unit >= a.H) {
    prep_values<T>(a, unit - a.H, row, wrow, t0, q_len, si, so, last);
    return;
  }
  const int h = unit, group = a.H / a.G, g = h / group, ldy = dk + 4;
  float *q_s = sm, *k_s = sm + BT * ldy, *d_s = sm + 2 * BT * ldy;           // [16][dk + 4] each
  // the decays of four channels of a token per item; the loads are under way while the convolutions run
  constexpr int DI = BT * 256 / 4 / PREP_T;
  const int quads = dk / 4;
  float4 raw[DI];
#pragma unroll
  for (int u = 0; u < DI; ++u) {
    const int i = tid + u * PREP_T, t = i / quads;
    raw[u] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t < n) raw[u] = *reinterpret_cast<const float4*>(a.decay + (row + t0 + t) * a.ld_decay + (long long)h * dk + (i - t * quads) * 4);
  }
  const int nch = dk / 8;
  int L = 1;
  while (L < nch) L <<= 1;                       // <= 32
  for (int task = tid / L; task < BT; task += PREP_T / L) {
    const int part = task & 1, r = (task >> 1) * 2, c = (tid % L) * 8, t = t0 + r;
    const bool on = c < dk && t < q_len;
    const int ch = part * a.G * dk + g * dk + c;
    float y[2][8];
#pragma unroll
    for (int e = 0; e < 8; ++e) y[0][e] = y[1][e] = 0.f;
    if (on) conv_pair<T>(a, row, t, q_len, si, ch, C, y);
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) { s0 = fmaf(y[0][e], y[0][e], s0); s1 = fmaf(y[1][e], y[1][e], s1); }
    for (int o = L / 2; o > 0; o >>= 1) { s0 += __shfl_xor_sync(0xffffffffu, s0, o); s1 += __shfl_xor_sync(0xffffffffu, s1, o); }
    const float f = part == 0 ? 1.f / sqrtf((float)a.dk_real) : 1.f;
    const float f0 = f / sqrtf(s0 + 1e-6f), f1 = f / sqrtf(s1 + 1e-6f);
    if (c < dk) {
#pragma unroll
      for (int e = 0; e < 8; ++e) { y[0][e] *= f0; y[1][e] = t + 1 < q_len ? y[1][e] * f1 : 0.f; }
      store8((part == 0 ? q_s : k_s) + r * ldy + c, y[0]);
      store8((part == 0 ? q_s : k_s) + (r + 1) * ldy + c, y[1]);
    }
    if (last && on && r == 0 && h % group == 0) keep_inputs<T>(a, row, q_len, si, so, ch, C);
  }
  const float rate = -expf(a.a_log[h]);
#pragma unroll
  for (int u = 0; u < DI; ++u) {
    const int i = tid + u * PREP_T, t = i / quads, d = (i - t * quads) * 4;
    if (t >= BT) continue;
    float4 g = make_float4(1.f, 1.f, 1.f, 1.f);               // tokens past the end: no decay
    if (t < n) {
      const float4 b = *reinterpret_cast<const float4*>(a.dt_bias + (long long)h * dk + d);
      g = make_float4(expf(rate * softplus(raw[u].x + b.x)), expf(rate * softplus(raw[u].y + b.y)), expf(rate * softplus(raw[u].z + b.z)),
                      expf(rate * softplus(raw[u].w + b.w)));
    }
    *reinterpret_cast<float4*>(d_s + t * ldy + d) = g;
  }
  __syncthreads();
  // products of the decays from the block's start and to its end; a thread owns a channel
  const long long HK = (long long)a.H * dk;
  float* dst = ws_qk(a) + (wrow + t0) * 3 * HK + (long long)h * dk;
  for (int i = tid; i < 2 * dk; i += PREP_T) {
    const int d = i < dk ? i : i - dk;
    float p = 1.f;
    if (i < dk) {
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        p *= d_s[t * ldy + d];
        if (t < n) {
          dst[t * 3 * HK + d] = q_s[t * ldy + d] * p;
          dst[t * 3 * HK + HK + d] = k_s[t * ldy + d] * p;
        }
      }
      ws_end(a)[((first_block(qs, seq) + blockIdx.x) * a.H + h) * dk + d] = p;
    } else {
#pragma unroll
      for (int t = BT - 1; t >= 0; --t) {
        if (t < n) dst[t * 3 * HK + 2 * HK + d] = k_s[t * ldy + d] * p;
        p *= d_s[t * ldy + d];
      }
    }
  }
  // k_j with the decayed keys and queries of the tokens behind it: sixteen lanes share a j and split the channels
  const int j = tid / BT, l = tid % BT;
  float kk[BT], qk[BT];
#pragma unroll
  for (int i = 0; i < BT; ++i) kk[i] = qk[i] = 0.f;
  for (int c = l * 4; c < dk; c += 4 * BT) {
    float4 w = *reinterpret_cast<const float4*>(k_s + j * ldy + c);
#pragma unroll
    for (int i = 0; i < BT; ++i) {
      if (i < j) continue;
      const float4 q = *reinterpret_cast<const float4*>(q_s + i * ldy + c);
      if (i > j) {
        const float4 f = *reinterpret_cast<const float4*>(d_s + i * ldy + c), k = *reinterpret_cast<const float4*>(k_s + i * ldy + c);
        w.x *= f.x; w.y *= f.y; w.z *= f.z; w.w *= f.w;
        kk[i] = fmaf(k.x, w.x, fmaf(k.y, w.y, fmaf(k.z, w.z, fmaf(k.w, w.w, kk[i]))));
      }
      qk[i] = fmaf(q.x, w.x, fmaf(q.y, w.y, fmaf(q.z, w.z, fmaf(q.w, w.w, qk[i]))));
    }
  }
  // sums over the sixteen lanes; lane i is left with those of token i
#pragma unroll
  for (int o = BT / 2; o > 0; o >>= 1) {
    const bool up = l & o;
#pragma unroll
    for (int m = 0; m < o; ++m) {
      const float k0 = __shfl_xor_sync(0xffffffffu, up ? kk[m] : kk[m + o], o), q0 = __shfl_xor_sync(0xffffffffu, up ? qk[m] : qk[m + o], o);
      kk[m] = (up ? kk[m + o] : kk[m]) + k0;
      qk[m] = (up ? qk[m + o] : qk[m]) + q0;
    }
  }
  if (l < n) {
    float* gr = ws_gram(a) + ((wrow + t0 + l) * a.H + h) * 2 * BT + j;
    gr[0] = kk[0];
    gr[BT] = qk[0];
  }
}

constexpr int SOLVE_T = 128;                     // eight (block, head) pairs per CTA

// T and W of a block and head: sixteen lanes, lane j makes column j of both.
template <typename T, bool CH>
__global__ void __launch_bounds__(SOLVE_T) delta_solve_kernel(const UbDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sm[SOLVE_T / BT][LDH];
  const int seq = blockIdx.z, unit = threadIdx.x / BT, j = threadIdx.x % BT;
  const int qs = a.q_start[seq], q_len = a.q_start[seq + 1] - qs, t0 = blockIdx.x * BT;
  if (t0 >= q_len) return;
  const int n = min(BT, q_len - t0), h_ = blockIdx.y * (SOLVE_T / BT) + unit, h = min(h_, a.H - 1), g = h / (a.H / a.G);
  const bool on = h_ < a.H, tok = j < n;
  const long long row = a.row0 + qs, wrow = qs;
  float* sys = sm[unit];
  const long long at = (row + t0 + min(j, n - 1)) * a.ld + h;
  // tokens past the end: no decay; decays per channel are in the products already
  float c = tok && !CH ? log_decay(a, (float)reinterpret_cast<const T*>(a.a)[at], h) : 0.f;
  const float beta = tok ? 1.f / (1.f + expf(-(float)reinterpret_cast<const T*>(a.b)[at])) : 0.f;
#pragma unroll
  for (int o = 1; o < BT; o <<= 1) {
    const float v = __shfl_up_sync(0xffffffffu, c, o, BT);
    if (j >= o) c += v;
  }
  const float c_end = __shfl_sync(0xffffffffu, c, BT - 1, BT);
  const int units = CH ? a.H : a.G;              // heads that have products of their own
  const float* gram = ws_gram(a) + ((wrow + t0) * units + (CH ? h : g)) * 2 * BT + j;
#pragma unroll
  for (int i = 0; i < BT; ++i) {
    const float ci = __shfl_sync(0xffffffffu, c, i, BT), bi = __shfl_sync(0xffffffffu, beta, i, BT);
    const float e = j <= i && i < n ? expf(ci - c) : 0.f;
    const float* p = gram + (long long)min(i, n - 1) * units * 2 * BT;
    sys[i * LDM + j] = bi * e * p[0];
    sys[(BT + i) * LDM + j] = e * p[BT];
  }
  __syncwarp();
  float x[BT];                                   // column j of the inverse, then of T
#pragma unroll
  for (int i = 0; i < BT; ++i) {
    float v = i == j ? 1.f : 0.f;
#pragma unroll
    for (int k = 0; k < i; ++k) v = fmaf(-sys[i * LDM + k], x[k], v);
    x[i] = v;
  }
#pragma unroll
  for (int i = 0; i < BT; ++i) x[i] *= beta;
  float* dst = ws_tw(a) + ((wrow + t0) * a.H + h) * 2 * BT + j;
#pragma unroll
  for (int i = 0; i < BT; ++i) {
    float w = 0.f;
#pragma unroll
    for (int k = 0; k <= i; ++k) w = fmaf(sys[(BT + i) * LDM + k], x[k], w);
    if (on && i < n) {
      dst[(long long)i * a.H * 2 * BT] = x[i];
      dst[(long long)i * a.H * 2 * BT + BT] = w;
    }
  }
  if (on && tok) {
    const float e = expf(c);
    *reinterpret_cast<float4*>(ws_gl(a) + ((wrow + t0 + j) * a.H + h) * 4) = make_float4(-e, e, expf(c_end - c), 0.f);
  }
}

// ------------------------------------------------------------------------------------------------------------------------
// portions: the scan
// ------------------------------------------------------------------------------------------------------------------------
constexpr int SCAN_W = 4;     // warps per CTA

__device__ __forceinline__ void cp16(float* dst, const float* src, bool ok) {
  const int sz = ok ? 16 : 0;                    // 0 source bytes: the destination is zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(sz) : "memory");
}

// RPL rows and four columns of S per lane, LPG lanes per column group.
//
// Sums over the lanes of a group are taken by halving: a lane hands over what its partner keeps.  So that this needs no
// selection, lanes hold things in the order in which they give them away: the first operand of an odd half-group's lane is q
// where the others' is k, the LPG / 8 lanes that share a column take LPG / 8 tokens at a time and number them from their own one
// (slot s holds token s ^ own), and likewise the four columns.  In the end a lane has one number for every LPG / 8th token.
template <int RPL, int LPG, bool CH>
struct Scan {
  static constexpr int DK = RPL * LPG;           // rows that fit
  static constexpr int CPW = 4 * (32 / LPG);     // columns per warp
  static constexpr int COLS = CPW * SCAN_W;      // ... per CTA
  static constexpr int REPS = LPG / 8;           // lanes per column and kind of product
  static constexpr int OWN = BT / REPS;          // tokens a lane ends up with: q * REPS + rep
  static constexpr int GT = RPL >= 16 ? (REPS > 2 ? REPS : 2) : 4;             // tokens whose products with S are under way together
  struct Stage {
    float kq[CH ? 3 : 2][BT][DK], v[2][BT][COLS], tw[BT][2 * BT], gl[BT][4];          // v[1] stays zero
    float end[CH ? DK : 4];                      // decays of the rows over the block
  };
  struct Smem {
    Stage st[2];
    float2 u[SCAN_W][2][BT][CPW];                // u e^(c_end - c), twice each; in the second copy neighbouring columns change places
  };
};

template <int RPL, int LPG, bool CH>
__global__ void __launch_bounds__(SCAN_W * 32) delta_scan_kernel(const UbDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  using C = Scan<RPL, LPG, CH>;
  extern __shared__ __align__(16) uint8_t raw[];
  typename C::Smem& s = *reinterpret_cast<typename C::Smem*>(raw);
  const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qs = a.q_start[seq], q_len = a.q_start[seq + 1] - qs;
  if (q_len <= 0) return;
  const int grp = lane / LPG, l = lane % LPG, g = h / (a.H / a.G), dk = a.dk, dv = a.dv;
  const int cta_col = blockIdx.x * C::COLS, wcol = warp * C::CPW + grp * 4, col = cta_col + wcol;
  const bool on = col < dv;
  // after the reduction a lane holds one number per token: of S^T k (even half of the group) or S^T q, for its own column
  const int type = l / (LPG / 2), mycol = (l / (LPG / 8)) & 3, rep = l % (LPG / 8);
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  auto first_row = [&](int p) { return 4 * (l + LPG * (p >> 1)) + 2 * (p & 1); };     // of pair p
  auto turn = [&](const float4 f) {              // columns 0 .. 3 <-> slots 0 .. 3
    const float4 h2 = mycol & 2 ? make_float4(f.z, f.w, f.x, f.y) : f;
    return mycol & 1 ? make_float4(h2.y, h2.x, h2.w, h2.z) : h2;
  };

  uint64_t S[RPL / 2][4];
  {
    const float* src = a.state + ((long long)max(si, 0) * a.H + h) * dk * dv + col;
#pragma unroll
    for (int p = 0; p < RPL / 2; ++p) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
      const int r = first_row(p);
      if (si >= 0 && on && r < dk) {
        x = turn(*reinterpret_cast<const float4*>(src + (long long)r * dv));
        y = turn(*reinterpret_cast<const float4*>(src + (long long)(r + 1) * dv));
      }
      S[p][0] = pack_f32x2(x.x, y.x); S[p][1] = pack_f32x2(x.y, y.y); S[p][2] = pack_f32x2(x.z, y.z); S[p][3] = pack_f32x2(x.w, y.w);
    }
  }
  for (int i = tid; i < 2 * BT * C::COLS; i += SCAN_W * 32) s.st[i / (BT * C::COLS)].v[1][0][i % (BT * C::COLS)] = 0.f;
  const float *qk = ws_qk(a), *tw = ws_tw(a), *gl = ws_gl(a);
  float* vo = ws_v(a);
  const int blocks = (q_len + BT - 1) / BT;
  // this thread's share of the copies: chunk (row, column) of k and q, of v, of the matrices, and of the decays
  constexpr int KC = C::DK / 4, KR = SCAN_W * 32 / KC, VC = C::COLS / 4, VR = SCAN_W * 32 / VC;
  static_assert(SCAN_W * 32 % KC == 0 && BT % KR == 0, "whole rows of k per pass");
  const int kr = tid / KC, kc = tid % KC * 4, vr = tid / VC, vc = tid % VC * 4;
  auto fetch = [&](int b) {
    if (b < blocks) {
      typename C::Stage& st = s.st[b & 1];
      const int t0 = b * BT, n = min(BT, q_len - t0);
      const long long row = (long long)qs + t0;
      {
        const long long ld = qk_row(a), next = (long long)(CH ? a.H : a.G) * dk;         // next: q to k, k to the k behind S
        const float* p = qk + (row + kr) * ld + (long long)(CH ? h : g) * dk + kc;
#pragma unroll
        for (int i = 0; i < BT / KR; ++i, p += KR * ld) {
          const bool ok = kr + i * KR < n && kc < dk;
          cp16(&st.kq[1][kr + i * KR][kc], ok ? p : qk, ok);
          cp16(&st.kq[0][kr + i * KR][kc], ok ? p + next : qk, ok);
          if (CH) cp16(&st.kq[CH ? 2 : 0][kr + i * KR][kc], ok ? p + 2 * next : qk, ok);
        }
        if (CH && tid < C::DK / 4)
          cp16(&st.end[CH ? 4 * tid : 0], ws_end(a) + ((first_block(qs, seq) + b) * a.H + h) * dk + (4 * tid < dk ? 4 * tid : 0), 4 * tid < dk);
      }
      for (int t = vr; t < BT; t += VR) {
        const bool ok = t < n && cta_col + vc < dv;
        cp16(&st.v[0][t][vc], vo + (ok ? (row + t) * a.H * dv + (long long)h * dv + cta_col + vc : 0), ok);
      }
      {
        const int t = tid / 8, c = tid % 8 * 4;  // 128 threads: 16 rows of 32
        cp16(&st.tw[t][c], tw + (t < n ? ((row + t) * a.H + h) * 2 * BT + c : 0), t < n);
      }
      // tokens past the end repeat the last one's decay; their k, v and matrix rows are zero, so they write nothing
      if (tid < BT) cp16(&st.gl[tid][0], gl + ((row + min(tid, n - 1)) * a.H + h) * 4, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);
  for (int b = 0; b < blocks; ++b) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                             // block b has landed; everyone is done with the one before
    fetch(b + 1);
    const typename C::Stage& st = s.st[b & 1];
    const int t0 = b * BT, n = min(BT, q_len - t0);
    const float *mine = &st.kq[type][0][4 * l], *theirs = &st.kq[type ^ 1][0][4 * l];

    // products of all tokens with the entering state: x (of the tokens' k) or e^c S^T q
    float f[C::OWN][4];
#pragma unroll
    for (int tg = 0; tg < BT; tg += C::GT) {
      uint64_t P[C::GT][4], R[C::GT][4];
#pragma unroll
      for (int t = 0; t < C::GT; ++t)
#pragma unroll
        for (int c = 0; c < 4; ++c) P[t][c] = R[t][c] = 0ull;
#pragma unroll
      for (int x = 0; x < RPL / 4; ++x) {
        ulonglong2 k[C::GT], q[C::GT];
#pragma unroll
        for (int t = 0; t < C::GT; ++t) {
          const int at = (C::REPS == 1 ? tg + t : (tg + t) ^ rep) * C::DK + 4 * LPG * x;
          k[t] = *reinterpret_cast<const ulonglong2*>(mine + at);
          q[t] = *reinterpret_cast<const ulonglong2*>(theirs + at);
        }
#pragma unroll
        for (int t = 0; t < C::GT; ++t)
#pragma unroll
          for (int c = 0; c < 4; ++c) { P[t][c] = fma_f32x2(k[t].x, S[2 * x][c], P[t][c]); R[t][c] = fma_f32x2(q[t].x, S[2 * x][c], R[t][c]); }
#pragma unroll
        for (int t = 0; t < C::GT; ++t)
#pragma unroll
          for (int c = 0; c < 4; ++c) { P[t][c] = fma_f32x2(k[t].y, S[2 * x + 1][c], P[t][c]); R[t][c] = fma_f32x2(q[t].y, S[2 * x + 1][c], R[t][c]); }
      }
      float w[C::GT][4];
#pragma unroll
      for (int t = 0; t < C::GT; ++t)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          float p0, p1, r0, r1;
          unpack_f32x2(P[t][c], p0, p1);
          unpack_f32x2(R[t][c], r0, r1);
          w[t][c] = p0 + p1 + __shfl_xor_sync(0xffffffffu, r0 + r1, LPG / 2);
        }
      // the tokens that share lanes
#pragma unroll
      for (int o = C::REPS / 2; o > 0; o >>= 1)
#pragma unroll
        for (int t = 0; t < C::GT; ++t)
          if (t % (2 * o) < o && t % C::REPS < 2 * o) {
#pragma unroll
            for (int c = 0; c < 4; ++c) w[t][c] += __shfl_xor_sync(0xffffffffu, w[t + o][c], o);
          }
#pragma unroll
      for (int t = 0; t < C::GT; t += C::REPS)
#pragma unroll
        for (int c = 0; c < 4; ++c) f[(tg + t) / C::REPS][c] = w[t][c];
    }
    float val[C::OWN];
#pragma unroll
    for (int q = 0; q < C::OWN; ++q) {
      f[q][0] += __shfl_xor_sync(0xffffffffu, f[q][2], LPG / 4);
      f[q][1] += __shfl_xor_sync(0xffffffffu, f[q][3], LPG / 4);
    }
#pragma unroll
    for (int q = 0; q < C::OWN; ++q) val[q] = f[q][0] + __shfl_xor_sync(0xffffffffu, f[q][1], LPG / 8);
#pragma unroll
    for (int q = 0; q < C::OWN; ++q) {
      const int t = q * C::REPS + rep;
      val[q] = fmaf(val[q], st.gl[t][type], st.v[type][t][wcol + mycol]);
    }
    // u = T x in the lanes that hold x, o = e^c S^T q + W x in the others
    float x[BT];
#pragma unroll
    for (int j = 0; j < BT; ++j) x[j] = __shfl_sync(0xffffffffu, val[j / C::REPS], (lane & ~(LPG / 2 | (C::REPS - 1))) + j % C::REPS);
    if (type == 0) {
#pragma unroll
      for (int q = 0; q < C::OWN; ++q) val[q] = 0.f;
    }
#pragma unroll
    for (int j4 = 0; j4 < BT / 4; ++j4)
#pragma unroll
      for (int q = 4 * j4 / C::REPS; q < C::OWN; ++q) {          // beyond the diagonal the rows hold zeros
        const float4 m = *reinterpret_cast<const float4*>(&st.tw[q * C::REPS + rep][type * BT + 4 * j4]);
        val[q] = fmaf(m.x, x[4 * j4], fmaf(m.y, x[4 * j4 + 1], fmaf(m.z, x[4 * j4 + 2], fmaf(m.w, x[4 * j4 + 3], val[q]))));
      }
    if (type == 0) {
#pragma unroll
      for (int q = 0; q < C::OWN; ++q) {
        const int t = q * C::REPS + rep;
        const float u = val[q] * st.gl[t][2];
        s.u[warp][0][t][grp * 4 + mycol] = make_float2(u, u);
        s.u[warp][1][t][grp * 4 + (mycol ^ 1)] = make_float2(u, u);
      }
    } else if (on) {
      float* dst = vo + ((long long)qs + t0 + rep) * a.H * dv + (long long)h * dv + col + mycol;
#pragma unroll
      for (int q = 0; q < C::OWN; ++q, dst += (long long)C::REPS * a.H * dv)
        if (q * C::REPS + rep < n) *dst = val[q];
    }
    __syncwarp();
    // the state behind the block
    const float end = st.gl[BT - 1][1];
    const uint64_t fade = pack_f32x2(end, end);
    const float* kk = &st.kq[CH ? 2 : 0][0][4 * l];
    const float2 *ua = &s.u[warp][mycol & 1][0][grp * 4 + (mycol & 2)], *ub = &s.u[warp][mycol & 1][0][grp * 4 + ((mycol & 2) ^ 2)];
    if (CH) {
#pragma unroll
      for (int x2 = 0; x2 < RPL / 4; ++x2) {
        const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(&st.end[CH ? 4 * l + 4 * LPG * x2 : 0]);
#pragma unroll
        for (int c = 0; c < 4; ++c) { S[2 * x2][c] = mul_f32x2(S[2 * x2][c], f.x); S[2 * x2 + 1][c] = mul_f32x2(S[2 * x2 + 1][c], f.y); }
      }
    } else {
#pragma unroll
      for (int p = 0; p < RPL / 2; ++p)
#pragma unroll
        for (int c = 0; c < 4; ++c) S[p][c] = mul_f32x2(S[p][c], fade);
    }
#pragma unroll
    for (int j = 0; j < BT; ++j) {
      const ulonglong2 u01 = *reinterpret_cast<const ulonglong2*>(ua + j * C::CPW), u23 = *reinterpret_cast<const ulonglong2*>(ub + j * C::CPW);
      const uint64_t u[4] = {u01.x, u01.y, u23.x, u23.y};
#pragma unroll
      for (int x2 = 0; x2 < RPL / 4; ++x2) {
        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(kk + j * C::DK + 4 * LPG * x2);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          S[2 * x2][c] = fma_f32x2(k.x, u[c], S[2 * x2][c]);
          S[2 * x2 + 1][c] = fma_f32x2(k.y, u[c], S[2 * x2 + 1][c]);
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  if (so >= 0 && on) {
    float* dst = a.state + ((long long)so * a.H + h) * dk * dv + col;
#pragma unroll
    for (int p = 0; p < RPL / 2; ++p) {
      const int r = first_row(p);
      if (r >= dk) continue;
      float4 x, y;
      unpack_f32x2(S[p][0], x.x, y.x); unpack_f32x2(S[p][1], x.y, y.y); unpack_f32x2(S[p][2], x.z, y.z); unpack_f32x2(S[p][3], x.w, y.w);
      *reinterpret_cast<float4*>(dst + (long long)r * dv) = turn(x);
      *reinterpret_cast<float4*>(dst + (long long)(r + 1) * dv) = turn(y);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------------
// portions: norm and gate of the outputs, eight columns per lane
// ------------------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) delta_finish_kernel(const UbDeltaArgs a, const int L /* lanes per row and head */) {
  pdl_launch_dependents();
  pdl_wait();
  const int dv = a.dv, c = (threadIdx.x % L) * 8;
  const long long i = (long long)blockIdx.x * (256 / L) + threadIdx.x / L;
  const bool on = i < (long long)a.rows * a.H && c < dv;
  const long long t = i / a.H;
  const int h = int(i % a.H);
  float o[8], g[8], w[8], sq = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) o[e] = 0.f;
  if (on) {
    load8(ws_v(a) + t * a.H * dv + (long long)h * dv + c, o);
    load8(reinterpret_cast<const T*>(a.gate) + (a.row0 + t) * a.ld_gate + (long long)h * dv + c, g);
    load8(a.norm_w + c, w);
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) sq = fmaf(o[e], o[e], sq);
  for (int x = L / 2; x > 0; x >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, x);
  if (!on) return;
  const float r = 1.f / sqrtf(sq / a.dv_real + a.eps);
#pragma unroll
  for (int e = 0; e < 8; ++e) o[e] *= r * w[e] * out_gate(a, g[e]);
  store8(reinterpret_cast<T*>(a.out) + (a.row0 + t) * a.ld_out + (long long)h * dv + c, o);
}

template <int RPL, int LPG, bool CH>
static cudaError_t launch_scan(const UbDeltaArgs& a, cudaStream_t st) {
  using C = Scan<RPL, LPG, CH>;
  constexpr size_t smem = sizeof(typename C::Smem);
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<RPL, LPG, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(delta_scan_kernel<RPL, LPG, CH>, dim3((a.dv + C::COLS - 1) / C::COLS, a.H, a.num_seqs), dim3(SCAN_W * 32), smem, st, a);
}

template <typename T, bool CH>
static cudaError_t launch_portions(const UbDeltaArgs& a, cudaStream_t st) {
  const size_t smem = sizeof(float) * (CH ? 3 : 2) * BT * (a.dk + 4);
  const int blocks = (a.max_q + BT - 1) / BT;
  const dim3 grid(blocks, (CH ? a.H : a.G) + (a.H * a.dv + PREP_T - 1) / PREP_T, a.num_seqs);
  cudaError_t e = cudaSuccess;
  if constexpr (CH) {
    if (smem > 48 * 1024) e = cudaFuncSetAttribute(delta_prep_channel_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess) e = launch_pdl(delta_prep_channel_kernel<T>, grid, dim3(PREP_T), smem, st, a);
  } else {
    e = launch_pdl(delta_prep_kernel<T>, grid, dim3(PREP_T), smem, st, a);
  }
  if (e != cudaSuccess) return e;
  e = launch_pdl(delta_solve_kernel<T, CH>, dim3(blocks, (a.H + SOLVE_T / BT - 1) / (SOLVE_T / BT), a.num_seqs), dim3(SOLVE_T), (size_t)0, st, a);
  if (e != cudaSuccess) return e;
  // few lanes per column keep the reductions short, many of them spread a small launch over the device
  const long long cols = (long long)a.num_seqs * a.H * a.dv;
  int lanes = a.lanes;
  if (lanes == 0) lanes = cols / 16 >= 888 ? 8 : cols / 8 >= 400 ? 16 : 32;
  if (a.dk > 128 && lanes < 16) lanes = 16;
  if (a.dk <= 32) e = launch_scan<4, 8, CH>(a, st);
  else if (a.dk <= 64) e = lanes <= 8 ? launch_scan<8, 8, CH>(a, st) : launch_scan<4, 16, CH>(a, st);
  else if (a.dk <= 128) e = lanes <= 8 ? launch_scan<16, 8, CH>(a, st) : lanes <= 16 ? launch_scan<8, 16, CH>(a, st) : launch_scan<4, 32, CH>(a, st);
  else e = lanes <= 16 ? launch_scan<16, 16, CH>(a, st) : launch_scan<8, 32, CH>(a, st);
  if (e != cudaSuccess) return e;
  int L = 1;
  while (L * 8 < a.dv) L <<= 1;
  const long long per = 256 / L;
  return launch_pdl(delta_finish_kernel<T>, dim3((unsigned)(((long long)a.rows * a.H + per - 1) / per)), dim3(256), (size_t)0, st, a, L);
}

}  // namespace delta
}  // namespace ub

extern "C" long long ub_delta_workspace_floats(int rows, int num_seqs, int H, int G, int dk, int dv, int channel_decay) {
  constexpr int BT = ub::delta::BT;
  const long long qk = channel_decay ? 3LL * H * dk : 2LL * G * dk, units = channel_decay ? H : G;
  const long long end = channel_decay ? (rows / BT + num_seqs + 1LL) * H * dk : 0;
  return (long long)rows * (qk + (long long)H * dv + 2LL * BT * (H + units) + 4LL * H) + end;
}

extern "C" int ub_delta_mixer(const UbDeltaArgs* args, void* stream) {
  using namespace ub;
  UbDeltaArgs full = *args;
  if (full.ld_gate <= 0) full.ld_gate = full.ld;
  const UbDeltaArgs* a = &full;
  const bool ch = a->decay != nullptr;
  if (a->num_seqs <= 0 || a->max_q <= 0 || a->rows <= 0) return 0;
  if (a->H <= 0 || a->G <= 0 || a->H % a->G != 0 || a->H > 65535 || a->num_seqs > 65535) return -2;
  if (a->dk % 8 != 0 || a->dv % 8 != 0 || a->dk <= 0 || a->dv <= 0 || a->dk > 256 || a->dv > 256) return -3;
  if (a->dk_real <= 0 || a->dk_real > a->dk || a->dv_real <= 0 || a->dv_real > a->dv) return -3;
  if (a->taps < 1 || a->taps > 16 || a->ld % 8 != 0 || a->ld_out % 8 != 0 || a->ld_gate % 8 != 0 || (ch && a->ld_decay % 4 != 0)) return -4;
  if (a->qkv == nullptr || a->gate == nullptr || a->b == nullptr || (a->a == nullptr && !ch) || a->conv == nullptr || a->state == nullptr ||
      a->out == nullptr || a->norm_w == nullptr || a->a_log == nullptr || a->dt_bias == nullptr)
    return -5;
  if (a->taps > 1 && a->conv_state == nullptr) return -5;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (a->q_start == nullptr) {
    if (a->rows != a->num_seqs) return -6;
    if (ch) e = a->f32 ? delta::launch_step<float, true>(*a, st) : delta::launch_step<__nv_bfloat16, true>(*a, st);
    else e = a->f32 ? delta::launch_step<float, false>(*a, st) : delta::launch_step<__nv_bfloat16, false>(*a, st);
  } else {
    if (a->ws == nullptr || (ch ? a->H : a->G) + a->H * a->dv / 256 + 1 > 65535) return -6;
    if (ch) e = a->f32 ? delta::launch_portions<float, true>(*a, st) : delta::launch_portions<__nv_bfloat16, true>(*a, st);
    else e = a->f32 ? delta::launch_portions<float, false>(*a, st) : delta::launch_portions<__nv_bfloat16, false>(*a, st);
  }
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
