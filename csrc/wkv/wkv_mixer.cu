// K16c: the matrix-state recurrence of RWKV-6 style layers over ragged portions of sequences, with what follows it in the
// layer: per head and token
//
//   o[j]   = sum_i r[i] * (S[i][j] + u[i] k[i] v[j])          S[i][j] <- d[i] S[i][j] + k[i] v[j],  d = exp(-exp(ww))
//   out[j] = o[j] / sqrt(mean(o^2) + eps) * w[j] * silu(g[j])
//
// State, decays and everything between the loads and `out` are fp32; r, k, v, g and out have the element type of the matrix
// products.  A portion reads its sequence's state row (none: zero) and leaves the new state in another row.
//
// Four columns and D / RG rows of S live in the registers of a thread, as pairs of neighbouring rows: the row factors r, k and
// d come as pairs from shared memory and two multiply-adds are one instruction.  RG = 8 neighbouring lanes hold the row
// groups of the same columns, so a token's output needs four shuffles.  Tokens come in tiles of 16 through shared memory; the bonus term
// is one scalar per token, sum_i r u k, times v.
//
// Long prompts (wkv_chunk / wkv_carry / wkv_out): chunks of CL tokens run in parallel from a zero state and leave their
// outputs, r * (product of the decays before the token), their end state and their total decay; the carry walks the chunks
// and replaces end states by entering states; the last pass adds (r * product) S_entering to every output and finishes it.
// Products of decays are at most one, so nothing is ever divided by a decay.
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace wkv {

constexpr int TB = 16;      // tokens per shared-memory tile
constexpr int RG = 8;       // row groups (lanes of a warp that share columns)

__device__ __forceinline__ float silu(float v) { return v / (1.f + expf(-v)); }

template <int DP>
struct Tile {
  float r[TB][DP], k[TB][DP], d[TB][DP], v[TB][DP], y[TB][DP];
  float bonus[TB];
};

// tokens [t, t + n) of one head, converted to fp32 (decays evaluated); columns beyond D are zero (decay one)
template <typename T, int DP>
__device__ __forceinline__ void load_tile(const UbWkvArgs& a, Tile<DP>& s, long long row, int n, int h) {
  const int D = a.D, cpr = DP / 8;
  for (int i = threadIdx.x; i < n * cpr; i += blockDim.x) {
    const int t = i / cpr, c = (i % cpr) * 8;
    float r[8], k[8], v[8], w[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) { r[e] = k[e] = v[e] = 0.f; w[e] = 1.f; }
    if (c < D) {
      const long long off = (row + t) * a.ld + (long long)h * D + c;
      load8(reinterpret_cast<const T*>(a.r) + off, r);
      load8(reinterpret_cast<const T*>(a.k) + off, k);
      load8(reinterpret_cast<const T*>(a.v) + off, v);
      load8(a.ww + off, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) w[e] = expf(-expf(w[e]));
    }
    store8(&s.r[t][c], r);
    store8(&s.k[t][c], k);
    store8(&s.v[t][c], v);
    store8(&s.d[t][c], w);
  }
}

template <int DP>
__device__ __forceinline__ void bonus_terms(const UbWkvArgs& a, Tile<DP>& s, int n, int h) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  for (int t = warp; t < n; t += nw) {
    float b = 0.f;
    for (int i = lane; i < a.D; i += 32) b = fmaf(s.r[t][i] * a.u[h * a.D + i], s.k[t][i], b);
    b = warp_sum(b);
    if (lane == 0) s.bonus[t] = b;
  }
}

// One thread's share of the state and the walk over a tile.
template <int DP>
struct State {
  static constexpr int RPT = DP / RG;            // rows per thread
  uint64_t S[RPT / 2][4];                        // [pair of rows][column]
  int rg, cg;

  __device__ __forceinline__ State() {
    const int lane = threadIdx.x & 31;
    rg = lane & 7;
    cg = (threadIdx.x >> 5) * 4 + (lane >> 3);
  }
  // first row of pair p: groups of four rows, RG groups apart
  __device__ __forceinline__ int row(int p) const { return 4 * (rg + RG * (p >> 1)) + 2 * (p & 1); }

  __device__ __forceinline__ void load(const float* st, int D) {
#pragma unroll
    for (int p = 0; p < RPT / 2; ++p) {
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f), g = f;
      if (st != nullptr && row(p) < D && cg * 4 < D) {
        f = *reinterpret_cast<const float4*>(st + (long long)row(p) * D + cg * 4);
        g = *reinterpret_cast<const float4*>(st + (long long)(row(p) + 1) * D + cg * 4);
      }
      S[p][0] = pack_f32x2(f.x, g.x); S[p][1] = pack_f32x2(f.y, g.y); S[p][2] = pack_f32x2(f.z, g.z); S[p][3] = pack_f32x2(f.w, g.w);
    }
  }
  __device__ __forceinline__ void store(float* st, int D) const {
#pragma unroll
    for (int p = 0; p < RPT / 2; ++p) {
      if (row(p) >= D || cg * 4 >= D) continue;
      float4 f, g;
      unpack_f32x2(S[p][0], f.x, g.x); unpack_f32x2(S[p][1], f.y, g.y); unpack_f32x2(S[p][2], f.z, g.z); unpack_f32x2(S[p][3], f.w, g.w);
      *reinterpret_cast<float4*>(st + (long long)row(p) * D + cg * 4) = f;
      *reinterpret_cast<float4*>(st + (long long)(row(p) + 1) * D + cg * 4) = g;
    }
  }
  __device__ __forceinline__ void walk(Tile<DP>& s, int n) {
    for (int t = 0; t < n; ++t) {
      const float4 v4 = *reinterpret_cast<const float4*>(&s.v[t][cg * 4]);
      const uint64_t v[4] = {pack_f32x2(v4.x, v4.x), pack_f32x2(v4.y, v4.y), pack_f32x2(v4.z, v4.z), pack_f32x2(v4.w, v4.w)};
      uint64_t y2[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
      for (int q = 0; q < RPT / 4; ++q) {
        const int i = 4 * (rg + RG * q);
        const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(&s.r[t][i]);
        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(&s.k[t][i]);
        const ulonglong2 d = *reinterpret_cast<const ulonglong2*>(&s.d[t][i]);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          y2[c] = fma_f32x2(r.x, S[2 * q][c], y2[c]);
          S[2 * q][c] = fma_f32x2(d.x, S[2 * q][c], mul_f32x2(k.x, v[c]));
          y2[c] = fma_f32x2(r.y, S[2 * q + 1][c], y2[c]);
          S[2 * q + 1][c] = fma_f32x2(d.y, S[2 * q + 1][c], mul_f32x2(k.y, v[c]));
        }
      }
      float y[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float lo, hi;
        unpack_f32x2(y2[c], lo, hi);
        y[c] = lo + hi;
      }
      // sum over the eight row groups, each step halving what a lane still carries: four shuffles for four columns
      const bool b2 = rg & 4, b1 = rg & 2;
      float a0 = b2 ? y[2] : y[0], a1 = b2 ? y[3] : y[1];
      a0 += __shfl_xor_sync(0xffffffffu, b2 ? y[0] : y[2], 4);
      a1 += __shfl_xor_sync(0xffffffffu, b2 ? y[1] : y[3], 4);
      float c = b1 ? a1 : a0;
      c += __shfl_xor_sync(0xffffffffu, b1 ? a0 : a1, 2);
      c += __shfl_xor_sync(0xffffffffu, c, 1);
      if ((rg & 1) == 0) s.y[t][cg * 4 + (b2 ? 2 : 0) + (b1 ? 1 : 0)] = c;
    }
  }
};

// head norm, weight and gate of the tokens warp, warp + nw, ... < n; o(t, c) is the recurrence's output of token t in column
// c.  Four tokens of a warp go together, so that their gates are under way at the same time.
template <typename T, int DP, typename F>
__device__ __forceinline__ void finish_tokens(const UbWkvArgs& a, long long row, int n, int h, F o) {
  constexpr int CPL = DP / 32, U = 4;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const T* gp = reinterpret_cast<const T*>(a.g);
  T* out = reinterpret_cast<T*>(a.out);
  float w[CPL];
#pragma unroll
  for (int j = 0; j < CPL; ++j) w[j] = lane + 32 * j < a.D ? a.norm_w[h * a.D + lane + 32 * j] : 0.f;
  for (int t0 = warp; t0 < n; t0 += U * nw) {
    float v[U][CPL], g[U][CPL], sq[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int t = t0 + u * nw;
      sq[u] = 0.f;
#pragma unroll
      for (int j = 0; j < CPL; ++j) {
        const int c = lane + 32 * j;
        const bool ok = t < n && c < a.D;
        g[u][j] = ok ? float(gp[(row + t) * a.ld + (long long)h * a.D + c]) : 0.f;
        v[u][j] = ok ? o(t, c) : 0.f;
        sq[u] = fmaf(v[u][j], v[u][j], sq[u]);
      }
    }
#pragma unroll
    for (int x = 16; x > 0; x >>= 1)
#pragma unroll
      for (int u = 0; u < U; ++u) sq[u] += __shfl_xor_sync(0xffffffffu, sq[u], x);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int t = t0 + u * nw;
      if (t >= n) continue;
      const float r = 1.f / sqrtf(sq[u] / a.norm_dim + a.eps);
#pragma unroll
      for (int j = 0; j < CPL; ++j) {
        const int c = lane + 32 * j;
        if (c < a.D) out[(row + t) * a.ld + (long long)h * a.D + c] = T(v[u][j] * r * w[j] * silu(g[u][j]));
      }
    }
  }
}

__device__ __forceinline__ void seq_rows(const UbWkvArgs& a, int seq, int& qs, int& q_len) {
  qs = a.q_start != nullptr ? a.q_start[seq] : seq;
  q_len = a.q_start != nullptr ? a.q_start[seq + 1] - qs : 1;
}

__device__ __forceinline__ int state_row(const UbWkvArgs& a, const int* rows, int seq) {
  const int r = rows != nullptr ? rows[seq] : -1;
  if (r >= a.state_rows) {
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, seq);
    return -1;
  }
  return r;
}

template <typename T, int DP>
__global__ void __launch_bounds__(DP * 2) wkv_seq_kernel(const UbWkvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t raw[];
  Tile<DP>& s = *reinterpret_cast<Tile<DP>*>(raw);
  const int h = blockIdx.x, seq = blockIdx.y;
  int qs, q_len;
  seq_rows(a, seq, qs, q_len);
  if (q_len <= 0) return;
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  const long long per = (long long)a.D * a.D, row0 = a.row0 + qs;
  State<DP> st;
  st.load(si >= 0 ? a.state + ((long long)si * a.H + h) * per : nullptr, a.D);
  for (int t0 = 0; t0 < q_len; t0 += TB) {
    const int n = min(TB, q_len - t0);
    __syncthreads();
    load_tile<T, DP>(a, s, row0 + t0, n, h);
    __syncthreads();
    bonus_terms<DP>(a, s, n, h);
    st.walk(s, n);
    if (so >= 0 && t0 + n == q_len) st.store(a.state + ((long long)so * a.H + h) * per, a.D);
    __syncthreads();
    finish_tokens<T, DP>(a, row0 + t0, n, h, [&](int t, int c) { return fmaf(s.bonus[t], s.v[t][c], s.y[t][c]); });
  }
}

// One token of every sequence: a read and a write of the state.  Everything else that the CTA needs is requested in front of
// the state, so that its latency runs under the state's.
template <typename T, int DP>
__global__ void __launch_bounds__(DP * 2, DP <= 64 ? 1024 / (DP * 2) : 2) wkv_step_kernel(const UbWkvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ __align__(16) float r_s[DP], k_s[DP], d_s[DP], v_s[DP], y_s[DP];
  __shared__ float red[DP / 32 > 0 ? DP / 32 : 1], red2[DP / 32 > 0 ? DP / 32 : 1];
  const int h = blockIdx.x, seq = blockIdx.y, i = threadIdx.x, D = a.D, warp = i >> 5, lane = i & 31;
  const long long off = (a.row0 + seq) * a.ld + (long long)h * D + i;
  const bool mine = i < D;
  float r = 0.f, k = 0.f, v = 0.f, g = 0.f, ww = 0.f, u = 0.f, nw = 0.f;
  if (mine) {
    r = float(reinterpret_cast<const T*>(a.r)[off]);
    k = float(reinterpret_cast<const T*>(a.k)[off]);
    v = float(reinterpret_cast<const T*>(a.v)[off]);
    g = float(reinterpret_cast<const T*>(a.g)[off]);
    ww = a.ww[off];
    u = a.u[h * D + i];
    nw = a.norm_w[h * D + i];
  }
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  const long long per = (long long)D * D;
  State<DP> st;
  // four columns of a thread, its rows in pairs: the layout of State, loaded row by row
  float4 f[State<DP>::RPT];
  const float* src = a.state + ((long long)max(si, 0) * a.H + h) * per;
#pragma unroll
  for (int p = 0; p < State<DP>::RPT; ++p) {
    const int row = st.row(p >> 1) + (p & 1);
    f[p] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (si >= 0 && row < D && st.cg * 4 < D) f[p] = __ldcs(reinterpret_cast<const float4*>(src + (long long)row * D + st.cg * 4));
  }
  if (i < DP) {
    r_s[i] = r;
    k_s[i] = k;
    v_s[i] = v;
    d_s[i] = mine ? expf(-expf(ww)) : 1.f;
    const float b = warp_sum(r * u * k);
    if (lane == 0) red[warp] = b;
  }
  __syncthreads();
  float bonus = 0.f;
#pragma unroll
  for (int w = 0; w < DP / 32; ++w) bonus += red[w];
  float y[4] = {0.f, 0.f, 0.f, 0.f};
  const float4 v4 = *reinterpret_cast<const float4*>(&v_s[st.cg * 4]);
  float* dst = a.state + ((long long)max(so, 0) * a.H + h) * per;
#pragma unroll
  for (int p = 0; p < State<DP>::RPT; ++p) {
    const int row = st.row(p >> 1) + (p & 1);
    const float rr = r_s[row], kk = k_s[row], dd = d_s[row];
    y[0] = fmaf(rr, f[p].x, y[0]); y[1] = fmaf(rr, f[p].y, y[1]); y[2] = fmaf(rr, f[p].z, y[2]); y[3] = fmaf(rr, f[p].w, y[3]);
    f[p].x = fmaf(dd, f[p].x, kk * v4.x); f[p].y = fmaf(dd, f[p].y, kk * v4.y);
    f[p].z = fmaf(dd, f[p].z, kk * v4.z); f[p].w = fmaf(dd, f[p].w, kk * v4.w);
    if (so >= 0 && row < D && st.cg * 4 < D) __stcs(reinterpret_cast<float4*>(dst + (long long)row * D + st.cg * 4), f[p]);
  }
#pragma unroll
  for (int o = 4; o > 0; o >>= 1)
#pragma unroll
    for (int c = 0; c < 4; ++c) y[c] += __shfl_xor_sync(0xffffffffu, y[c], o);
  if (st.rg == 0) *reinterpret_cast<float4*>(&y_s[st.cg * 4]) = make_float4(y[0], y[1], y[2], y[3]);
  __syncthreads();
  const float o = mine ? fmaf(bonus, v, y_s[i]) : 0.f;
  if (i < DP) {
    const float sq = warp_sum(o * o);
    if (lane == 0) red2[warp] = sq;
  }
  __syncthreads();
  if (!mine) return;
  float sq = 0.f;
#pragma unroll
  for (int w = 0; w < DP / 32; ++w) sq += red2[w];
  reinterpret_cast<T*>(a.out)[off] = T(o * (1.f / sqrtf(sq / a.norm_dim + a.eps)) * nw * silu(g));
}

// (sequence, chunk inside it) of a chunk index of the launch; false past the last one
__device__ __forceinline__ bool find_chunk(const UbWkvArgs& a, int idx, int& seq, int& t0, int& t1, int& qs) {
  int base = 0;
  for (seq = 0; seq < a.num_seqs; ++seq) {
    qs = a.q_start[seq];
    const int q_len = a.q_start[seq + 1] - qs, n = (q_len + a.chunk - 1) / a.chunk;
    if (idx < base + n) {
      t0 = (idx - base) * a.chunk;
      t1 = min(t0 + a.chunk, q_len);
      return true;
    }
    base += n;
  }
  return false;
}

// workspace: local outputs and r * product [rows][ld] each, then per chunk and head the end (later: entering) state and the
// chunk's decays
__device__ __forceinline__ float* ws_y(const UbWkvArgs& a) { return a.ws; }
__device__ __forceinline__ float* ws_rp(const UbWkvArgs& a) { return a.ws + (long long)a.rows * a.ld; }
__device__ __forceinline__ float* ws_q(const UbWkvArgs& a, int chunk, int h) {
  return a.ws + 2LL * a.rows * a.ld + ((long long)chunk * a.H + h) * a.D * a.D;
}
__device__ __forceinline__ float* ws_p(const UbWkvArgs& a, int chunk, int h) {
  return a.ws + 2LL * a.rows * a.ld + (long long)a.max_chunks * a.H * a.D * a.D + ((long long)chunk * a.H + h) * a.D;
}

template <typename T, int DP>
__global__ void __launch_bounds__(DP * 2) wkv_chunk_kernel(const UbWkvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t raw[];
  Tile<DP>& s = *reinterpret_cast<Tile<DP>*>(raw);
  const int h = blockIdx.x, chunk = blockIdx.y;
  int seq, c0, c1, qs;
  if (!find_chunk(a, chunk, seq, c0, c1, qs)) return;
  State<DP> st;
  st.load(nullptr, a.D);
  float prod = 1.f;                              // thread i < D: product of row i's decays so far
  for (int t0 = c0; t0 < c1; t0 += TB) {
    const int n = min(TB, c1 - t0);
    __syncthreads();
    load_tile<T, DP>(a, s, a.row0 + qs + t0, n, h);
    __syncthreads();
    bonus_terms<DP>(a, s, n, h);
    st.walk(s, n);
    __syncthreads();
    const long long off = (long long)(qs + t0) * a.ld + (long long)h * a.D;
    for (int i = threadIdx.x; i < n * (DP / 4); i += blockDim.x) {
      const int t = i / (DP / 4), c = i % (DP / 4) * 4;
      if (c >= a.D) continue;
      const float b = s.bonus[t];
      const float4 v = *reinterpret_cast<const float4*>(&s.v[t][c]), y = *reinterpret_cast<const float4*>(&s.y[t][c]);
      *reinterpret_cast<float4*>(ws_y(a) + off + (long long)t * a.ld + c) = make_float4(fmaf(b, v.x, y.x), fmaf(b, v.y, y.y), fmaf(b, v.z, y.z), fmaf(b, v.w, y.w));
    }
    if (threadIdx.x < a.D) {
      for (int t = 0; t < n; ++t) {
        ws_rp(a)[off + (long long)t * a.ld + threadIdx.x] = s.r[t][threadIdx.x] * prod;
        prod *= s.d[t][threadIdx.x];
      }
    }
  }
  st.store(ws_q(a, chunk, h), a.D);
  if (threadIdx.x < a.D) ws_p(a, chunk, h)[threadIdx.x] = prod;
}

__global__ void __launch_bounds__(256) wkv_carry_kernel(const UbWkvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, seq = blockIdx.y, per = a.D * a.D;
  int base = 0;
  for (int i = 0; i < seq; ++i) base += (a.q_start[i + 1] - a.q_start[i] + a.chunk - 1) / a.chunk;
  const int q_len = a.q_start[seq + 1] - a.q_start[seq], n = (q_len + a.chunk - 1) / a.chunk;
  if (n <= 0) return;
  const int si = state_row(a, a.state_in, seq), so = state_row(a, a.state_out, seq);
  const int e = (blockIdx.z * 256 + threadIdx.x) * 4;             // four columns of one row (D is a multiple of 8)
  if (e >= per) return;
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (si >= 0) S = *reinterpret_cast<const float4*>(a.state + ((long long)si * a.H + h) * per + e);
  // eight chunks are requested before the first of them is used
  constexpr int U = 8;
  const int row = e / a.D;
  for (int c0 = 0; c0 < n; c0 += U) {
    float4 v[U];
    float p[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (c0 + u < n) {
        v[u] = __ldcs(reinterpret_cast<const float4*>(ws_q(a, base + c0 + u, h) + e));
        p[u] = __ldg(ws_p(a, base + c0 + u, h) + row);
      }
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (c0 + u < n) {
        *reinterpret_cast<float4*>(ws_q(a, base + c0 + u, h) + e) = S;
        S = make_float4(fmaf(p[u], S.x, v[u].x), fmaf(p[u], S.y, v[u].y), fmaf(p[u], S.z, v[u].z), fmaf(p[u], S.w, v[u].w));
      }
  }
  if (so >= 0) *reinterpret_cast<float4*>(a.state + ((long long)so * a.H + h) * per + e) = S;
}

// 64 tokens of a chunk per CTA: y += (r * product) S_entering, then norm, weight and gate
constexpr int OT = 64, OG = OT / 8;      // tokens per CTA, per thread

template <typename T, int DP>
__global__ void __launch_bounds__(DP * 2) wkv_out_kernel(const UbWkvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t raw[];
  float(*S)[DP] = reinterpret_cast<float(*)[DP]>(raw);
  float(*rp)[DP + 4] = reinterpret_cast<float(*)[DP + 4]>(raw + sizeof(float) * DP * DP);
  const int h = blockIdx.x, chunk = blockIdx.y;
  int seq, c0, c1, qs;
  if (!find_chunk(a, chunk, seq, c0, c1, qs)) return;
  const int t0 = c0 + blockIdx.z * OT, n = min(OT, c1 - t0), D = a.D;
  if (n <= 0) return;
  const float* q = ws_q(a, chunk, h);
  for (int i = threadIdx.x; i < DP * DP / 4; i += blockDim.x) {
    const int r = i / (DP / 4), c = (i % (DP / 4)) * 4;
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r < D && c < D) f = *reinterpret_cast<const float4*>(q + r * D + c);
    *reinterpret_cast<float4*>(&S[r][c]) = f;
  }
  const long long off = (long long)(qs + t0) * a.ld + (long long)h * D;
  for (int i = threadIdx.x; i < OT * DP / 4; i += blockDim.x) {
    const int t = i / (DP / 4), c = (i % (DP / 4)) * 4;
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t < n && c < D) f = *reinterpret_cast<const float4*>(ws_rp(a) + off + (long long)t * a.ld + c);
    *reinterpret_cast<float4*>(&rp[t][c]) = f;
  }
  __syncthreads();
  // DP / 4 column groups x 8 token groups
  const int cg = threadIdx.x % (DP / 4), tg = threadIdx.x / (DP / 4);
  float acc[OG][4];
#pragma unroll
  for (int t = 0; t < OG; ++t)
#pragma unroll
    for (int c = 0; c < 4; ++c) acc[t][c] = 0.f;
  for (int i = 0; i < D; i += 4) {
    float4 s4[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) s4[e] = *reinterpret_cast<const float4*>(&S[i + e][cg * 4]);
#pragma unroll
    for (int t = 0; t < OG; ++t) {
      const float4 p4 = *reinterpret_cast<const float4*>(&rp[tg * OG + t][i]);
      const float p[4] = {p4.x, p4.y, p4.z, p4.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        acc[t][0] = fmaf(p[e], s4[e].x, acc[t][0]); acc[t][1] = fmaf(p[e], s4[e].y, acc[t][1]);
        acc[t][2] = fmaf(p[e], s4[e].z, acc[t][2]); acc[t][3] = fmaf(p[e], s4[e].w, acc[t][3]);
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int t = 0; t < OG; ++t) {
    const int tt = tg * OG + t;
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (tt < n && cg * 4 < D) f = *reinterpret_cast<const float4*>(ws_y(a) + off + (long long)tt * a.ld + cg * 4);
    *reinterpret_cast<float4*>(&rp[tt][cg * 4]) = make_float4(acc[t][0] + f.x, acc[t][1] + f.y, acc[t][2] + f.z, acc[t][3] + f.w);
  }
  __syncthreads();
  finish_tokens<T, DP>(a, a.row0 + qs + t0, n, h, [&](int t, int c) { return rp[t][c]; });
}

template <typename K>
static cudaError_t allow_smem(K kern, size_t smem) {
  return smem > 48 * 1024 ? cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : cudaSuccess;
}

template <typename T, int DP>
static cudaError_t launch(const UbWkvArgs& a, cudaStream_t st) {
  const dim3 block(DP * 2);
  const size_t tile = sizeof(Tile<DP>), out = sizeof(float) * (DP * DP + OT * (DP + 4));
  cudaError_t e;
  if (a.q_start == nullptr) return launch_pdl(wkv_step_kernel<T, DP>, dim3(a.H, a.num_seqs), block, (size_t)0, st, a);
  if (a.chunk <= 0) {
    if ((e = allow_smem(wkv_seq_kernel<T, DP>, tile)) != cudaSuccess) return e;
    return launch_pdl(wkv_seq_kernel<T, DP>, dim3(a.H, a.num_seqs), block, tile, st, a);
  }
  if ((e = allow_smem(wkv_chunk_kernel<T, DP>, tile)) != cudaSuccess) return e;
  if ((e = allow_smem(wkv_out_kernel<T, DP>, out)) != cudaSuccess) return e;
  if ((e = launch_pdl(wkv_chunk_kernel<T, DP>, dim3(a.H, a.max_chunks), block, tile, st, a)) != cudaSuccess) return e;
  if ((e = launch_pdl(wkv_carry_kernel, dim3(a.H, a.num_seqs, (a.D * a.D / 4 + 255) / 256), dim3(256), (size_t)0, st, a)) != cudaSuccess)
    return e;
  return launch_pdl(wkv_out_kernel<T, DP>, dim3(a.H, a.max_chunks, (a.chunk + OT - 1) / OT), block, out, st, a);
}

template <typename T>
static cudaError_t launch_sized(const UbWkvArgs& a, cudaStream_t st) {
  if (a.D <= 32) return launch<T, 32>(a, st);
  if (a.D <= 64) return launch<T, 64>(a, st);
  return launch<T, 128>(a, st);
}

}  // namespace wkv
}  // namespace ub

extern "C" long long ub_wkv_workspace_floats(int rows, int ld, int H, int D, int max_chunks) {
  return 2LL * rows * ld + (long long)max_chunks * H * ((long long)D * D + D);
}

extern "C" int ub_wkv_mixer(const UbWkvArgs* a, void* stream) {
  using namespace ub;
  if (a->num_seqs <= 0 || a->H <= 0) return 0;
  if (a->D <= 0 || a->D % 8 != 0 || a->D > 128 || a->ld != a->H * a->D || a->norm_dim <= 0) return -2;
  if (a->state == nullptr || a->num_seqs > 65535) return -3;
  if (a->chunk > 0 && (a->q_start == nullptr || a->ws == nullptr || a->max_chunks <= 0 || a->max_chunks > 65535)) return -4;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = a->f32 ? wkv::launch_sized<float>(*a, st) : wkv::launch_sized<__nv_bfloat16>(*a, st);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
