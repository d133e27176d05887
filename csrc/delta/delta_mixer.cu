// K16d: gated delta rule over ragged portions of sequences, with what surrounds it in the layer.  Per token, head h of H and
// the query / key head g = h / (H / G):
//
//   q, k, v = silu(causal depthwise convolution over time of the projected rows)
//   q = q / sqrt(sum q^2 + 1e-6) / sqrt(dk),  k = k / sqrt(sum k^2 + 1e-6)
//   beta = sigmoid(b),  decay = exp(-exp(a_log) * softplus(a + dt_bias))
//   S <- decay * S,  u = beta * (v - S^T k),  S <- S + k u^T,  o = S^T q                  S [dk, dv]
//   out = o / sqrt(mean(o^2) + eps) * w * silu(gate)
//
// Everything between the loads and `out` is fp32; the projected rows and `out` have the element type of the matrix products.
// A portion reads its sequence's state rows (none: zero) and leaves the new state in other rows, so every CTA of a launch may
// read the old ones whenever it runs.  Rows of heads are padded to multiples of 8 with zeros, which stay zero.
//
// One token per sequence (delta_step): a CTA per head and sequence; the state passes through registers once.
//
// Portions: delta_prep makes q, k and v of 16 tokens, their products k.k and q.k among themselves, and running sums of the
// log decays; delta_scan carries the state through blocks of 16 tokens; delta_finish normalises and gates.  Within a block
// with the log decays' running sum c,
//
//   u_i = beta_i (v_i - e^(c_i) S^T k_i - sum_(j < i) e^(c_i - c_j) (k_i . k_j) u_j)
//   o_i = e^(c_i) S^T q_i + sum_(j <= i) e^(c_i - c_j) (q_i . k_j) u_j
//   S  <- e^(c_end) S + sum_j e^(c_end - c_j) k_j u_j^T
//
// so the products with S of all 16 tokens are independent, and what is left of the recurrence is a triangular solve of 16
// scalars per column.  Exponents are never positive.  Columns of S do not meet: a warp owns a few of them.
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace delta {

constexpr int BT = 16;        // tokens per block

__device__ __forceinline__ float silu(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float log_decay(const UbDeltaArgs& a, float x, int h) { return -expf(a.a_log[h]) * softplus(x + a.dt_bias[h]); }

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
constexpr int STEP_T = 256;

// ROWS: rows of S that a thread holds (four columns each); 0: S is read twice instead (heads too large for registers).
template <typename T, int ROWS>
__global__ void __launch_bounds__(STEP_T) delta_step_kernel(const UbDeltaArgs a, const int cl /* threads across the columns */) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int HELD = ROWS > 0 ? ROWS : 1;
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.x, seq = blockIdx.y, dk = a.dk, dv = a.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nrg = STEP_T / cl, rg = tid / cl, col = (tid % cl) * 4;
  float* qkv = sm;                               // [2 dk + dv] after the convolutions
  float* part = qkv + 2 * dk + dv;               // [8][2][dv] partial products with the old state
  float* u_s = part + 8 * 2 * dv;            // [dv]
  float* o_s = u_s + dv;                         // [dv]
  float* sc = o_s + dv;                          // scalars: 1 / |q|, 1 / |k|, q . k, beta, decay; then eight sums
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
  // convolutions of this head's channels; the oldest input leaves, the current one joins
  for (int c = tid; c < 2 * dk + dv; c += STEP_T) {
    const int ch = c < dk ? g * dk + c : c < 2 * dk ? a.G * dk + g * dk + (c - dk) : 2 * a.G * dk + h * dv + (c - 2 * dk);
    const bool keep = so >= 0 && (c >= 2 * dk || h % group == 0);
    const T* w = reinterpret_cast<const T*>(a.conv) + ch;
    const float cur = (float)reinterpret_cast<const T*>(a.qkv)[row * a.ld + ch];
    float acc = 0.f;
    for (int j = 0; j < m; ++j) {
      const float v = si >= 0 ? a.conv_state[((long long)si * m + j) * C + ch] : 0.f;
      acc = fmaf((float)w[(long long)j * C], v, acc);
      if (keep && j > 0) a.conv_state[((long long)so * m + j - 1) * C + ch] = v;
    }
    if (keep && m > 0) a.conv_state[((long long)so * m + m - 1) * C + ch] = cur;
    qkv[c] = silu(fmaf((float)w[(long long)m * C], cur, acc));
  }
  float gate = 0.f, nw = 0.f;                    // dv <= STEP_T (host check)
  if (tid < dv) {
    gate = (float)reinterpret_cast<const T*>(a.gate)[row * a.ld + (long long)h * dv + tid];
    nw = a.norm_w[tid];
  }
  if (tid == 0) {
    sc[3] = 1.f / (1.f + expf(-(float)reinterpret_cast<const T*>(a.b)[row * a.ld + h]));
    sc[4] = expf(log_decay(a, (float)reinterpret_cast<const T*>(a.a)[row * a.ld + h], h));
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
    const float kk = qkv[dk + r], qq = qkv[r];
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
  const int slot = cl >= 32 ? rg : warp, nslots = cl >= 32 ? nrg : STEP_T / 32;
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
    for (int w = 0; w < STEP_T / 32; ++w) s += sc[8 + w];
    reinterpret_cast<T*>(a.out)[row * a.ld_out + (long long)h * dv + tid] = T(o * (1.f / sqrtf(s / a.dv_real + a.eps)) * nw * silu(gate));
  }
  if (so >= 0 && on) {
    const float4 u = *reinterpret_cast<const float4*>(u_s + col);
    auto write = [&](float4 s, int r) {
      const float kk = qkv[dk + r] * rk;
      s.x = fmaf(kk, u.x, decay * s.x); s.y = fmaf(kk, u.y, decay * s.y);
      s.z = fmaf(kk, u.z, decay * s.z); s.w = fmaf(kk, u.w, decay * s.w);
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

template <typename T>
static cudaError_t launch_step(const UbDeltaArgs& a, cudaStream_t st) {
  int cl = 2;
  while (cl * 4 < a.dv) cl <<= 1;                // <= 64
  const int nrg = STEP_T / cl, need = (a.dk + nrg - 1) / nrg;
  const size_t smem = sizeof(float) * (2 * a.dk + a.dv + 16 * a.dv + 2 * a.dv + 16);
  const dim3 grid(a.H, a.num_seqs), block(STEP_T);
  auto go = [&](auto kern) { return launch_pdl(kern, grid, block, smem, st, a, cl); };
  if (need <= 1) return go(delta_step_kernel<T, 1>);
  if (need <= 4) return go(delta_step_kernel<T, 4>);
  if (need <= 8) return go(delta_step_kernel<T, 8>);
  if (need <= 16) return go(delta_step_kernel<T, 16>);
  if (need <= 32) return go(delta_step_kernel<T, 32>);
  return go(delta_step_kernel<T, 0>);
}

// ------------------------------------------------------------------------------------------------------------------------
// portions: what the scan reads
// ------------------------------------------------------------------------------------------------------------------------
// workspace, per row of the launch: q and k [2 G dk], v (later o) [H dv], k.k and q.k with the tokens of the row's block
// [G][2][16], running log decay and beta [H][2]
__device__ __forceinline__ float* ws_qk(const UbDeltaArgs& a) { return a.ws; }
__device__ __forceinline__ float* ws_v(const UbDeltaArgs& a) { return a.ws + (long long)a.rows * 2 * a.G * a.dk; }
__device__ __forceinline__ float* ws_gram(const UbDeltaArgs& a) { return ws_v(a) + (long long)a.rows * a.H * a.dv; }
__device__ __forceinline__ float* ws_cb(const UbDeltaArgs& a) { return ws_gram(a) + (long long)a.rows * a.G * 2 * BT; }

constexpr int PREP_T = 256;

// One block of 16 tokens of one query / key head, or of one value head (units G ..).
template <typename T>
__global__ void __launch_bounds__(PREP_T) delta_prep_kernel(const UbDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int unit = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qs = a.q_start[seq], q_len = a.q_start[seq + 1] - qs, t0 = blockIdx.x * BT;
  if (t0 >= q_len) return;
  const int n = min(BT, q_len - t0), m = a.taps - 1, dk = a.dk, dv = a.dv;
  const bool is_qk = unit < a.G;
  const int h = unit - a.G, C = 2 * a.G * dk + a.H * dv;
  const int width = is_qk ? 2 * dk : dv;         // channels of this unit
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  auto channel = [&](int c) { return is_qk ? (c < dk ? unit * dk + c : a.G * dk + unit * dk + (c - dk)) : 2 * a.G * dk + h * dv + c; };
  float* in = sm;                                // [16 + m][width] inputs
  float* y = in + (BT + m) * width;              // [16][width + 4]
  const int ldy = width + 4;
  const long long row = a.row0 + qs, wrow = qs;  // rows of the step / of the workspace
  for (int i = tid; i < (n + m) * (width / 8); i += PREP_T) {
    const int r = i / (width / 8), c = i % (width / 8) * 8, t = t0 - m + r, ch = channel(c);
    float v[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = 0.f;
    if (t >= 0) load8(reinterpret_cast<const T*>(a.qkv) + (row + t) * a.ld + ch, v);
    else if (si >= 0) load8(a.conv_state + ((long long)si * m + m + t) * C + ch, v);
    store8(in + r * width + c, v);
  }
  __syncthreads();
  if (so >= 0 && t0 + n == q_len) {              // the last inputs are the sequence's state
    for (int i = tid; i < m * width; i += PREP_T) {
      const int r = i / width, c = i % width;
      a.conv_state[((long long)so * m + r) * C + channel(c)] = in[(n + r) * width + c];
    }
  }
  for (int c = tid; c < width; c += PREP_T) {
    const T* w = reinterpret_cast<const T*>(a.conv) + channel(c);
    float acc[BT];
#pragma unroll
    for (int r = 0; r < BT; ++r) acc[r] = 0.f;
    for (int j = 0; j <= m; ++j) {
      const float wj = (float)w[(long long)j * C];
#pragma unroll
      for (int r = 0; r < BT; ++r)
        if (r < n) acc[r] = fmaf(wj, in[(r + j) * width + c], acc[r]);
    }
#pragma unroll
    for (int r = 0; r < BT; ++r) {
      if (r >= n) break;
      const float s = silu(acc[r]);
      if (is_qk) y[r * ldy + c] = s;
      else ws_v(a)[(wrow + t0 + r) * a.H * dv + (long long)h * dv + c] = s;
    }
  }
  if (!is_qk) {
    if (warp == 0) {
      const bool ok = lane < n;
      const long long at = (row + t0 + lane) * a.ld + h;
      float c = ok ? log_decay(a, (float)reinterpret_cast<const T*>(a.a)[at], h) : 0.f;
#pragma unroll
      for (int o = 1; o < BT; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, c, o);
        if (lane >= o) c += v;
      }
      if (ok) {
        const float beta = 1.f / (1.f + expf(-(float)reinterpret_cast<const T*>(a.b)[at]));
        *reinterpret_cast<float2*>(ws_cb(a) + ((wrow + t0 + lane) * a.H + h) * 2) = make_float2(c, beta);
      }
    }
    return;
  }
  __syncthreads();
  const float qs_ = 1.f / sqrtf((float)a.dk_real);
  for (int i = warp; i < 2 * n; i += PREP_T / 32) {             // unit vectors: q rows, then k rows
    const int r = i >> 1, part = i & 1;
    float* p = y + r * ldy + part * dk;
    float s = 0.f;
    for (int c = lane; c < dk; c += 32) s = fmaf(p[c], p[c], s);
    s = 1.f / sqrtf(warp_sum(s) + 1e-6f);
    if (part == 0) s *= qs_;
    float* dst = ws_qk(a) + (wrow + t0 + r) * 2 * a.G * dk + (long long)part * a.G * dk + (long long)unit * dk;
    for (int c = lane; c < dk; c += 32) {
      const float v = p[c] * s;
      p[c] = v;
      dst[c] = v;
    }
  }
  __syncthreads();
  const int i = tid / BT, j = tid % BT;          // PREP_T = 16 * 16 pairs
  if (i < n) {
    float kk = 0.f, qk = 0.f;
    if (j <= i) {
      const float *ki = y + i * ldy + dk, *qi = y + i * ldy, *kj = y + j * ldy + dk;
      for (int c = 0; c < dk; c += 4) {
        const float4 x = *reinterpret_cast<const float4*>(ki + c), q = *reinterpret_cast<const float4*>(qi + c);
        const float4 z = *reinterpret_cast<const float4*>(kj + c);
        kk = fmaf(x.x, z.x, fmaf(x.y, z.y, fmaf(x.z, z.z, fmaf(x.w, z.w, kk))));
        qk = fmaf(q.x, z.x, fmaf(q.y, z.y, fmaf(q.z, z.z, fmaf(q.w, z.w, qk))));
      }
    }
    float* dst = ws_gram(a) + ((wrow + t0 + i) * a.G + unit) * 2 * BT;
    dst[j] = j < i ? kk : 0.f;
    dst[BT + j] = qk;
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
template <int RPL, int LPG>
struct Scan {
  static constexpr int DK = RPL * LPG;           // rows that fit
  static constexpr int CPW = 4 * (32 / LPG);     // columns per warp
  static constexpr int COLS = CPW * SCAN_W;      // ... per CTA
  struct Stage {
    float k[BT][DK], q[BT][DK], v[BT][COLS], gram[BT][2 * BT + 4], cb[BT][2];
  };
  struct Smem {
    Stage st[2];
    float mat[2][BT][BT];                        // by column j: -e^(c_i - c_j) k_i.k_j (i > j), e^(c_i - c_j) q_i.k_j (i >= j)
    float grow[BT], left[BT];                    // e^(c_i), e^(c_end - c_j)
    float u[SCAN_W][BT][CPW];
  };
};

template <int RPL, int LPG>
__global__ void __launch_bounds__(SCAN_W * 32) delta_scan_kernel(const UbDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  using C = Scan<RPL, LPG>;
  extern __shared__ __align__(16) uint8_t raw[];
  typename C::Smem& s = *reinterpret_cast<typename C::Smem*>(raw);
  const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qs = a.q_start[seq], q_len = a.q_start[seq + 1] - qs;
  if (q_len <= 0) return;
  const int grp = lane / LPG, l = lane % LPG, g = h / (a.H / a.G), dk = a.dk, dv = a.dv;
  const int cta_col = blockIdx.x * C::COLS, wcol = warp * C::CPW + grp * 4, col = cta_col + wcol;
  const bool on = col < dv;
  // after the reduction a lane holds one number per token: of S^T k (even half of the group) or S^T q, for one column
  const int type = l / (LPG / 2), mycol = (l / (LPG / 8)) & 3, rep = l % (LPG / 8);
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  auto first_row = [&](int p) { return 4 * (l + LPG * (p >> 1)) + 2 * (p & 1); };     // of pair p

  uint64_t S[RPL / 2][4];
  {
    const float* src = a.state + ((long long)max(si, 0) * a.H + h) * dk * dv + col;
#pragma unroll
    for (int p = 0; p < RPL / 2; ++p) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
      const int r = first_row(p);
      if (si >= 0 && on && r < dk) {
        x = *reinterpret_cast<const float4*>(src + (long long)r * dv);
        y = *reinterpret_cast<const float4*>(src + (long long)(r + 1) * dv);
      }
      S[p][0] = pack_f32x2(x.x, y.x); S[p][1] = pack_f32x2(x.y, y.y); S[p][2] = pack_f32x2(x.z, y.z); S[p][3] = pack_f32x2(x.w, y.w);
    }
  }
  const float *qk = ws_qk(a), *gram = ws_gram(a), *cbp = ws_cb(a);
  float* vo = ws_v(a);
  const int blocks = (q_len + BT - 1) / BT;
  auto fetch = [&](int b) {
    if (b < blocks) {
      typename C::Stage& st = s.st[b & 1];
      const int t0 = b * BT, n = min(BT, q_len - t0);
      const long long row = (long long)qs + t0;
      for (int i = tid; i < BT * (C::DK / 4); i += SCAN_W * 32) {
        const int t = i / (C::DK / 4), c = i % (C::DK / 4) * 4;
        const bool ok = t < n && c < dk;
        const float* p = qk + (ok ? (row + t) * 2 * a.G * dk + (long long)g * dk + c : 0);
        cp16(&st.q[t][c], p, ok);
        cp16(&st.k[t][c], ok ? p + (long long)a.G * dk : p, ok);
      }
      for (int i = tid; i < BT * (C::COLS / 4); i += SCAN_W * 32) {
        const int t = i / (C::COLS / 4), c = i % (C::COLS / 4) * 4;
        const bool ok = t < n && cta_col + c < dv;
        cp16(&st.v[t][c], vo + (ok ? (row + t) * a.H * dv + (long long)h * dv + cta_col + c : 0), ok);
      }
      for (int i = tid; i < BT * (2 * BT / 4); i += SCAN_W * 32) {
        const int t = i / (2 * BT / 4), c = i % (2 * BT / 4) * 4;
        cp16(&st.gram[t][c], gram + (t < n ? ((row + t) * a.G + g) * 2 * BT + c : 0), t < n);
      }
      // tokens past the end repeat the last one's decay; their k and v are zero, so they write nothing
      if (tid < BT) {
        const float* p = cbp + ((row + min(tid, n - 1)) * a.H + h) * 2;
        asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(smem_u32(&st.cb[tid][0])), "l"(p) : "memory");
      }
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
    const float c_end = st.cb[BT - 1][0];
    for (int i = tid; i < BT * BT; i += SCAN_W * 32) {
      const int r = i % BT, j = i / BT;
      const float e = j <= r ? expf(st.cb[r][0] - st.cb[j][0]) : 0.f;
      s.mat[0][j][r] = j < r ? -e * st.gram[r][j] : 0.f;
      s.mat[1][j][r] = j <= r ? e * st.gram[r][BT + j] : 0.f;
    }
    if (tid < BT) s.grow[tid] = expf(st.cb[tid][0]);
    else if (tid < 2 * BT) s.left[tid - BT] = expf(c_end - st.cb[tid - BT][0]);
    __syncthreads();

    // products of all tokens with the entering state
    float val[BT];
#pragma unroll
    for (int t = 0; t < BT; ++t) {
      uint64_t P[4] = {0ull, 0ull, 0ull, 0ull}, R[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
      for (int x = 0; x < RPL / 4; ++x) {
        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(&st.k[t][4 * (l + LPG * x)]);
        const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(&st.q[t][4 * (l + LPG * x)]);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          P[c] = fma_f32x2(k.x, S[2 * x][c], P[c]);
          R[c] = fma_f32x2(q.x, S[2 * x][c], R[c]);
          P[c] = fma_f32x2(k.y, S[2 * x + 1][c], P[c]);
          R[c] = fma_f32x2(q.y, S[2 * x + 1][c], R[c]);
        }
      }
      float p[4], r[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float lo, hi;
        unpack_f32x2(P[c], lo, hi);
        p[c] = lo + hi;
        unpack_f32x2(R[c], lo, hi);
        r[c] = lo + hi;
      }
      // each step halves what a lane still carries: 4 + 2 + 1 shuffles, then whole sums over lanes that hold the same
      float f[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const float mine = type ? r[c] : p[c], other = type ? p[c] : r[c];
        f[c] = mine + __shfl_xor_sync(0xffffffffu, other, LPG / 2);
      }
      const bool b1 = mycol & 2, b0 = mycol & 1;
      float f0 = b1 ? f[2] : f[0], f1 = b1 ? f[3] : f[1];
      f0 += __shfl_xor_sync(0xffffffffu, b1 ? f[0] : f[2], LPG / 4);
      f1 += __shfl_xor_sync(0xffffffffu, b1 ? f[1] : f[3], LPG / 4);
      float z = b0 ? f1 : f0;
      z += __shfl_xor_sync(0xffffffffu, b0 ? f0 : f1, LPG / 8);
#pragma unroll
      for (int o = LPG / 16; o > 0; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
      z *= s.grow[t];
      val[t] = type ? z : st.v[t][wcol + mycol] - z;
    }
    // the triangular solve: u_j is final when its turn comes
    const int from = lane & ~(LPG / 2);          // the lane of this column that solves
#pragma unroll
    for (int j = 0; j < BT; ++j) {
      const float u = __shfl_sync(0xffffffffu, val[j] * st.cb[j][1], from);
      if (type == 0 && rep == 0) s.u[warp][j][grp * 4 + mycol] = u * s.left[j];
#pragma unroll
      for (int x = j / 4; x < BT / 4; ++x) {
        const float4 m = *reinterpret_cast<const float4*>(&s.mat[type][j][4 * x]);
        if (4 * x >= j) val[4 * x] = fmaf(m.x, u, val[4 * x]);
        if (4 * x + 1 >= j) val[4 * x + 1] = fmaf(m.y, u, val[4 * x + 1]);
        if (4 * x + 2 >= j) val[4 * x + 2] = fmaf(m.z, u, val[4 * x + 2]);
        if (4 * x + 3 >= j) val[4 * x + 3] = fmaf(m.w, u, val[4 * x + 3]);
      }
    }
    if (type == 1 && rep == 0 && on) {
      float* dst = vo + ((long long)qs + t0) * a.H * dv + (long long)h * dv + col + mycol;
#pragma unroll
      for (int t = 0; t < BT; ++t)
        if (t < n) dst[(long long)t * a.H * dv] = val[t];
    }
    __syncwarp();
    // the state behind the block
    const uint64_t fade = pack_f32x2(s.grow[BT - 1], s.grow[BT - 1]);
#pragma unroll
    for (int p = 0; p < RPL / 2; ++p)
#pragma unroll
      for (int c = 0; c < 4; ++c) S[p][c] = mul_f32x2(S[p][c], fade);
#pragma unroll
    for (int j = 0; j < BT; ++j) {
      const float4 u4 = *reinterpret_cast<const float4*>(&s.u[warp][j][grp * 4]);
      const uint64_t u[4] = {pack_f32x2(u4.x, u4.x), pack_f32x2(u4.y, u4.y), pack_f32x2(u4.z, u4.z), pack_f32x2(u4.w, u4.w)};
#pragma unroll
      for (int x = 0; x < RPL / 4; ++x) {
        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(&st.k[j][4 * (l + LPG * x)]);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          S[2 * x][c] = fma_f32x2(k.x, u[c], S[2 * x][c]);
          S[2 * x + 1][c] = fma_f32x2(k.y, u[c], S[2 * x + 1][c]);
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
      *reinterpret_cast<float4*>(dst + (long long)r * dv) = x;
      *reinterpret_cast<float4*>(dst + (long long)(r + 1) * dv) = y;
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------------
// portions: norm and gate of the outputs, a warp per row and head
// ------------------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) delta_finish_kernel(const UbDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = blockIdx.x * 8LL + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, dv = a.dv;
  if (i >= (long long)a.rows * a.H) return;
  const long long t = i / a.H;
  const int h = int(i % a.H), c = lane * 8;
  float o[8], g[8], w[8], sq = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) o[e] = 0.f;
  if (c < dv) {
    load8(ws_v(a) + t * a.H * dv + (long long)h * dv + c, o);
    load8(reinterpret_cast<const T*>(a.gate) + (a.row0 + t) * a.ld + (long long)h * dv + c, g);
    load8(a.norm_w + c, w);
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) sq = fmaf(o[e], o[e], sq);
  sq = warp_sum(sq);
  if (c >= dv) return;
  const float r = 1.f / sqrtf(sq / a.dv_real + a.eps);
#pragma unroll
  for (int e = 0; e < 8; ++e) o[e] *= r * w[e] * silu(g[e]);
  store8(reinterpret_cast<T*>(a.out) + (a.row0 + t) * a.ld_out + (long long)h * dv + c, o);
}

template <int RPL, int LPG>
static cudaError_t launch_scan(const UbDeltaArgs& a, cudaStream_t st) {
  using C = Scan<RPL, LPG>;
  constexpr size_t smem = sizeof(typename C::Smem);
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<RPL, LPG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(delta_scan_kernel<RPL, LPG>, dim3((a.dv + C::COLS - 1) / C::COLS, a.H, a.num_seqs), dim3(SCAN_W * 32), smem, st, a);
}

template <typename T>
static cudaError_t launch_portions(const UbDeltaArgs& a, cudaStream_t st) {
  const int width = 2 * a.dk > a.dv ? 2 * a.dk : a.dv;
  const size_t smem = sizeof(float) * ((size_t)(BT + a.taps - 1) * width + (size_t)BT * (2 * a.dk + 4));
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(delta_prep_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  cudaError_t e = launch_pdl(delta_prep_kernel<T>, dim3((a.max_q + BT - 1) / BT, a.G + a.H, a.num_seqs), dim3(PREP_T), smem, st, a);
  if (e != cudaSuccess) return e;
  // few lanes per column keep the reductions short, many of them spread a small launch over the device
  const long long cols = (long long)a.num_seqs * a.H * a.dv;
  int lanes = a.lanes;
  if (lanes == 0) lanes = cols / 16 >= 2 * 592 ? 8 : cols / 8 >= 592 ? 16 : 32;
  if (a.dk > 128 && lanes < 16) lanes = 16;
  if (a.dk <= 32) e = launch_scan<4, 8>(a, st);
  else if (a.dk <= 64) e = lanes <= 8 ? launch_scan<8, 8>(a, st) : launch_scan<4, 16>(a, st);
  else if (a.dk <= 128) e = lanes <= 8 ? launch_scan<16, 8>(a, st) : lanes <= 16 ? launch_scan<8, 16>(a, st) : launch_scan<4, 32>(a, st);
  else e = lanes <= 16 ? launch_scan<16, 16>(a, st) : launch_scan<8, 32>(a, st);
  if (e != cudaSuccess) return e;
  return launch_pdl(delta_finish_kernel<T>, dim3((unsigned)(((long long)a.rows * a.H + 7) / 8)), dim3(256), (size_t)0, st, a);
}

}  // namespace delta
}  // namespace ub

extern "C" long long ub_delta_workspace_floats(int rows, int H, int G, int dk, int dv) {
  return (long long)rows * (2LL * G * dk + (long long)H * dv + 2LL * ub::delta::BT * G + 2LL * H);
}

extern "C" int ub_delta_mixer(const UbDeltaArgs* a, void* stream) {
  using namespace ub;
  if (a->num_seqs <= 0 || a->max_q <= 0 || a->rows <= 0) return 0;
  if (a->H <= 0 || a->G <= 0 || a->H % a->G != 0 || a->H > 65535 || a->num_seqs > 65535) return -2;
  if (a->dk % 8 != 0 || a->dv % 8 != 0 || a->dk <= 0 || a->dv <= 0 || a->dk > 256 || a->dv > 256) return -3;
  if (a->dk_real <= 0 || a->dk_real > a->dk || a->dv_real <= 0 || a->dv_real > a->dv) return -3;
  if (a->taps < 1 || a->taps > 16 || a->ld % 8 != 0 || a->ld_out % 8 != 0) return -4;
  if (a->qkv == nullptr || a->gate == nullptr || a->b == nullptr || a->a == nullptr || a->conv == nullptr || a->state == nullptr ||
      a->out == nullptr || a->norm_w == nullptr || a->a_log == nullptr || a->dt_bias == nullptr)
    return -5;
  if (a->taps > 1 && a->conv_state == nullptr) return -5;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (a->q_start == nullptr) {
    if (a->rows != a->num_seqs) return -6;
    e = a->f32 ? delta::launch_step<float>(*a, st) : delta::launch_step<__nv_bfloat16>(*a, st);
  } else {
    if (a->ws == nullptr || a->G + a->H > 65535) return -6;
    e = a->f32 ? delta::launch_portions<float>(*a, st) : delta::launch_portions<__nv_bfloat16>(*a, st);
  }
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
