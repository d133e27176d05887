// K5s: what a sublayer reads, for designs that normalise both sides of a sublayer and put a short convolution in front of it.
// One pass over the token rows does, all in 32 bits:
//
//   x' = x + norm_y(y)            (y: the previous sublayer's rows; absent at the first sublayer)
//   n  = norm(x')
//   h_t = n_t + sum_j conv[j] * n_(t - taps + 1 + j)                                   (causal, per channel)
//   out = h_t, or for every token-shift mix m:  out_m = h_t + (h_(t-1) - h_t) * mu_m   (recurrent mixers)
//
// norm(v) = v / sqrt(mean(v^2) + eps) * (w_off + w).  Sequences are ragged portions; what lies in front of a portion comes
// from the sequence's state rows (the last taps - 1 values of n, the last h), and the portion leaves its own behind in
// OTHER rows, so every CTA of the launch may read the old ones whenever it runs.
//
// Without convolution and mixes a row depends on nothing but itself: sublayer_alone_kernel, one CTA per row, in which y may
// also be a mixture-of-experts result that is summed here, with a gate on its always-on part.
//
// One token per sequence (decoding) has a kernel of its own: what the state contributes does not depend on the norms, so all
// loads are under way before the first sum.  Longer portions: a CTA takes `tile` consecutive tokens of one sequence and recomputes the few rows of n in front of them (x and y are read
// again, x' goes to a buffer of its own), so tiles are independent.  The last taps - 1 rows of n stay in shared memory; a
// thread touches only its own columns there.
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace subin {

constexpr int MIXES = 5;      // token-shift mixes of a recurrent mixer

// eight weights as they lie in memory, widened when they are used
template <typename T>
struct Raw8;
template <>
struct Raw8<__nv_bfloat16> {
  uint4 v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) { f[2 * e] = bf16_lo(u[e]); f[2 * e + 1] = bf16_hi(u[e]); }
  }
};
template <>
struct Raw8<float> {
  float v[8];
  __device__ __forceinline__ void load(const float* p) { load8(p, v); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = v[e];
  }
};

// one barrier per sum: the two halves of `red` alternate
template <int NW>
__device__ __forceinline__ float block_sum(float v, float (*red)[NW], int& flip) {
  v = warp_sum(v);
  const int nw = blockDim.x >> 5;
  if ((threadIdx.x & 31) == 0) red[flip][threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int w = 0; w < nw; ++w) s += red[flip][w];
  flip ^= 1;
  return s;
}

template <typename T, int CH>
__global__ void __launch_bounds__(256) sublayer_in_kernel(const UbSublayerInArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float hist[];       // [taps - 1][2][nch][4]: rows of n, halves of a chunk apart
  __shared__ float red[2][8];
  const int seq = blockIdx.y, nch = a.Hp / 8, m = a.taps > 0 ? a.taps - 1 : 0;
  const int qs = a.q_start != nullptr ? a.q_start[seq] : seq;
  const int q_len = a.q_start != nullptr ? a.q_start[seq + 1] - qs : 1;
  const int t0 = blockIdx.x * a.tile, t1 = min(t0 + a.tile, q_len);
  if (t0 >= t1) return;
  int si = a.state_in != nullptr ? a.state_in[seq] : -1, so = a.state_out != nullptr ? a.state_out[seq] : -1;
  if (si >= a.state_rows || so >= a.state_rows) {
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, seq);
    si = so = -1;
  }
  const bool mix = a.n_mix > 0;
  const int s0 = max(0, t0 - m - (mix ? 1 : 0));      // first token whose n is needed
  const T* y = reinterpret_cast<const T*>(a.y);
  const long long row0 = a.row0 + qs;
  int flip = 0;
  const int wrap = m > 0 ? m : 1;
  auto slot = [&](int idx) { return (idx + wrap * ((m + wrap - 1) / wrap)) % wrap; };     // idx >= -m
  auto hrow = [&](int s, int half, int ch) { return reinterpret_cast<float4*>(hist + ((s * 2 + half) * nch + ch) * 4); };

  if (s0 == 0 && m > 0) {
    for (int r = 0; r < m; ++r) {
      const int s = slot(r - m);
      for (int ch = threadIdx.x; ch < nch; ch += blockDim.x) {
        float4 lo = make_float4(0.f, 0.f, 0.f, 0.f), hi = lo;
        if (si >= 0) {
          const float4* p = reinterpret_cast<const float4*>(a.conv_state + ((long long)si * m + r) * a.Hp + ch * 8);
          lo = p[0];
          hi = p[1];
        }
        *hrow(s, 0, ch) = lo;
        *hrow(s, 1, ch) = hi;
      }
    }
  }
  float prev[CH][8];
  float xc[CH][8], yc[CH][8];
#pragma unroll
  for (int c = 0; c < CH; ++c)
#pragma unroll
    for (int e = 0; e < 8; ++e) prev[c][e] = xc[c][e] = yc[c][e] = 0.f;
  if (mix && s0 == 0 && si >= 0) {
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch < nch) load8(a.shift_state + (long long)si * a.Hp + ch * 8, prev[c]);
    }
  }
  auto fetch = [&](int t) {
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nch) continue;
      load8(a.x + (row0 + t) * a.Hp + ch * 8, xc[c]);
      if (y != nullptr) load8(y + (row0 + t) * a.Hp + ch * 8, yc[c]);
    }
  };
  fetch(s0);
  for (int t = s0; t < t1; ++t) {
    float n[CH][8];
    if (y != nullptr) {
      float sq = 0.f;
#pragma unroll
      for (int c = 0; c < CH; ++c)
#pragma unroll
        for (int e = 0; e < 8; ++e) sq += yc[c][e] * yc[c][e];            // pad columns are zero
      const float r = 1.f / sqrtf(block_sum(sq, red, flip) / a.H + a.eps);
#pragma unroll
      for (int c = 0; c < CH; ++c) {
        const int ch = threadIdx.x + c * blockDim.x;
        if (ch >= nch) continue;
        float w[8];
        load8(reinterpret_cast<const T*>(a.wy) + ch * 8, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) xc[c][e] += yc[c][e] * r * (a.w_off + w[e]);
        if (t >= t0) store8(a.x_out + (row0 + t) * a.Hp + ch * 8, xc[c]);
      }
    }
    float sq = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c)
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        n[c][e] = xc[c][e];
        sq += n[c][e] * n[c][e];
      }
    if (t + 1 < t1) fetch(t + 1);
    const float r = 1.f / sqrtf(block_sum(sq, red, flip) / a.H + a.eps);
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nch) continue;
      float w[8], h[8];
      load8(reinterpret_cast<const T*>(a.wn) + ch * 8, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        n[c][e] *= r * (a.w_off + w[e]);
        h[e] = n[c][e];
      }
      if (a.taps > 0 && (t >= t0 || (mix && t == t0 - 1))) {
        for (int j = 0; j < m; ++j) {
          const int s = slot(t - m + j);
          const float4 lo = *hrow(s, 0, ch), hi = *hrow(s, 1, ch);
          float k[8];
          load8(reinterpret_cast<const T*>(a.conv) + (long long)j * a.Hp + ch * 8, k);
          h[0] = fmaf(k[0], lo.x, h[0]); h[1] = fmaf(k[1], lo.y, h[1]); h[2] = fmaf(k[2], lo.z, h[2]); h[3] = fmaf(k[3], lo.w, h[3]);
          h[4] = fmaf(k[4], hi.x, h[4]); h[5] = fmaf(k[5], hi.y, h[5]); h[6] = fmaf(k[6], hi.z, h[6]); h[7] = fmaf(k[7], hi.w, h[7]);
        }
        float k[8];
        load8(reinterpret_cast<const T*>(a.conv) + (long long)m * a.Hp + ch * 8, k);
#pragma unroll
        for (int e = 0; e < 8; ++e) h[e] = fmaf(k[e], n[c][e], h[e]);
      }
      if (m > 0) {
        const int s = slot(t);
        *hrow(s, 0, ch) = make_float4(n[c][0], n[c][1], n[c][2], n[c][3]);
        *hrow(s, 1, ch) = make_float4(n[c][4], n[c][5], n[c][6], n[c][7]);
      }
      if (t >= t0) {
        T* out = reinterpret_cast<T*>(a.out) + (row0 + t) * a.Hp + ch * 8;
        if (!mix) store8(out, h);
        for (int i = 0; i < a.n_mix; ++i) {
          float mu[8], o[8];
          load8(reinterpret_cast<const T*>(a.mu) + (long long)i * a.Hp + ch * 8, mu);
#pragma unroll
          for (int e = 0; e < 8; ++e) o[e] = h[e] + (prev[c][e] - h[e]) * mu[e];
          store8(out + (long long)i * a.out_mix_stride, o);
        }
      }
      if (mix) {
#pragma unroll
        for (int e = 0; e < 8; ++e) prev[c][e] = h[e];
      }
      if (t == q_len - 1 && so >= 0) {                // the end of the portion: its last rows are the sequence's state
        for (int r2 = 0; r2 < m; ++r2) {
          const int s = slot(q_len - m + r2);
          float4* p = reinterpret_cast<float4*>(a.conv_state + ((long long)so * m + r2) * a.Hp + ch * 8);
          p[0] = *hrow(s, 0, ch);
          p[1] = *hrow(s, 1, ch);
        }
        if (mix) store8(a.shift_state + (long long)so * a.Hp + ch * 8, h);
      }
    }
  }
}

// Portions at up to 4096 columns and four taps: a thread owns one chunk, and the weights, the last rows of n and the
// prefetched next token all stay in registers.
template <typename T, int TAPS, bool MIX>
__global__ void __launch_bounds__(512) sublayer_rows_kernel(const UbSublayerInArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int M = TAPS - 1;
  __shared__ float red[2][16];
  const int seq = blockIdx.y, ch = threadIdx.x;
  const int qs = a.q_start[seq], q_len = a.q_start[seq + 1] - qs;
  const int t0 = blockIdx.x * a.tile, t1 = min(t0 + a.tile, q_len);
  if (t0 >= t1) return;
  int si = a.state_in != nullptr ? a.state_in[seq] : -1, so = a.state_out != nullptr ? a.state_out[seq] : -1;
  if (si >= a.state_rows || so >= a.state_rows) {
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, seq);
    si = so = -1;
  }
  const bool on = ch < a.Hp / 8;
  const int s0 = max(0, t0 - M - (MIX ? 1 : 0));
  const T* y = reinterpret_cast<const T*>(a.y);
  const long long base = (a.row0 + qs) * a.Hp + ch * 8;
  Raw8<T> wy8, wn8, k8[TAPS], mu8[MIX ? MIXES : 1];
  float hist[M > 0 ? M : 1][8], prev[8], x[8], yv[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    prev[e] = x[e] = yv[e] = 0.f;
#pragma unroll
    for (int r = 0; r < M; ++r) hist[r][e] = 0.f;
  }
  auto fetch = [&](int t) {
    load8(a.x + base + (long long)t * a.Hp, x);
    if (y != nullptr) load8(y + base + (long long)t * a.Hp, yv);
  };
  if (on) {
    fetch(s0);
    if (y != nullptr) wy8.load(reinterpret_cast<const T*>(a.wy) + ch * 8);
    wn8.load(reinterpret_cast<const T*>(a.wn) + ch * 8);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) k8[j].load(reinterpret_cast<const T*>(a.conv) + (long long)j * a.Hp + ch * 8);
    if (MIX) {
#pragma unroll
      for (int i = 0; i < MIXES; ++i) mu8[i].load(reinterpret_cast<const T*>(a.mu) + (long long)i * a.Hp + ch * 8);
    }
    if (s0 == 0 && si >= 0) {
#pragma unroll
      for (int r = 0; r < M; ++r) load8(a.conv_state + ((long long)si * M + r) * a.Hp + ch * 8, hist[r]);
      if (MIX) load8(a.shift_state + (long long)si * a.Hp + ch * 8, prev);
    }
  }
  int flip = 0;
  for (int t = s0; t < t1; ++t) {
    if (y != nullptr) {
      float sq = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) sq += yv[e] * yv[e];
      const float r = 1.f / sqrtf(block_sum(sq, red, flip) / a.H + a.eps);
      if (on) {
        float w[8];
        wy8.get(w);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] += yv[e] * r * (a.w_off + w[e]);
        if (t >= t0) store8(a.x_out + base + (long long)t * a.Hp, x);
      }
    }
    float n[8], sq = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      n[e] = x[e];
      sq += n[e] * n[e];
    }
    if (on && t + 1 < t1) fetch(t + 1);
    const float r = 1.f / sqrtf(block_sum(sq, red, flip) / a.H + a.eps);
    if (!on) continue;
    float w[8], h[8];
    wn8.get(w);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      n[e] *= r * (a.w_off + w[e]);
      h[e] = n[e];
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      float k[8];
      k8[j].get(k);
#pragma unroll
      for (int e = 0; e < 8; ++e) h[e] = fmaf(k[e], j < M ? hist[j < M ? j : 0][e] : n[e], h[e]);
    }
#pragma unroll
    for (int r2 = 0; r2 < M; ++r2)
#pragma unroll
      for (int e = 0; e < 8; ++e) hist[r2][e] = r2 + 1 < M ? hist[r2 + 1 < M ? r2 + 1 : 0][e] : n[e];
    if (t >= t0) {
      T* out = reinterpret_cast<T*>(a.out) + base + (long long)t * a.Hp;
      if (!MIX) {
        store8(out, h);
      } else {
#pragma unroll
        for (int i = 0; i < MIXES; ++i) {
          float mu[8], o[8];
          mu8[i].get(mu);
#pragma unroll
          for (int e = 0; e < 8; ++e) o[e] = h[e] + (prev[e] - h[e]) * mu[e];
          store8(out + (long long)i * a.out_mix_stride, o);
        }
      }
    }
    if (MIX) {
#pragma unroll
      for (int e = 0; e < 8; ++e) prev[e] = h[e];
    }
    if (t == q_len - 1 && so >= 0) {
#pragma unroll
      for (int r2 = 0; r2 < M; ++r2) store8(a.conv_state + ((long long)so * M + r2) * a.Hp + ch * 8, hist[r2]);
      if (MIX) store8(a.shift_state + (long long)so * a.Hp + ch * 8, h);
    }
  }
}

template <typename T, int TAPS>
static cudaError_t launch_rows(const UbSublayerInArgs& a, cudaStream_t st) {
  const dim3 grid((a.max_q + a.tile - 1) / a.tile, a.num_seqs), block((a.Hp / 8 + 31) / 32 * 32);
  return a.n_mix > 0 ? launch_pdl(sublayer_rows_kernel<T, TAPS, true>, grid, block, (size_t)0, st, a)
                     : launch_pdl(sublayer_rows_kernel<T, TAPS, false>, grid, block, (size_t)0, st, a);
}

// One token of every sequence.
template <typename T, int CH>
__global__ void __launch_bounds__(512) sublayer_step_kernel(const UbSublayerInArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[2][16];
  const int seq = blockIdx.x, nch = a.Hp / 8, m = a.taps > 0 ? a.taps - 1 : 0;
  const long long row = a.row0 + seq;
  const bool mix = a.n_mix > 0;
  const T* y = reinterpret_cast<const T*>(a.y);
  float x[CH][8], yv[CH][8], old[CH][8], prev[CH][8];
  float sq = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
#pragma unroll
    for (int e = 0; e < 8; ++e) x[c][e] = yv[c][e] = old[c][e] = prev[c][e] = 0.f;
    if (ch >= nch) continue;
    load8(a.x + row * a.Hp + ch * 8, x[c]);
    if (y != nullptr) load8(y + row * a.Hp + ch * 8, yv[c]);
#pragma unroll
    for (int e = 0; e < 8; ++e) sq += yv[c][e] * yv[c][e];
  }
  int si = a.state_in != nullptr ? a.state_in[seq] : -1, so = a.state_out != nullptr ? a.state_out[seq] : -1;
  if (si >= a.state_rows || so >= a.state_rows) {
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, seq);
    si = so = -1;
  }
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (ch >= nch) continue;
    if (mix && si >= 0) load8(a.shift_state + (long long)si * a.Hp + ch * 8, prev[c]);
#pragma unroll 3
    for (int j = 0; j < m; ++j) {                     // the taps in front of the token; its predecessors move up one row
      float v[8], k[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = 0.f;
      if (si >= 0) load8(a.conv_state + ((long long)si * m + j) * a.Hp + ch * 8, v);
      load8(reinterpret_cast<const T*>(a.conv) + (long long)j * a.Hp + ch * 8, k);
#pragma unroll
      for (int e = 0; e < 8; ++e) old[c][e] = fmaf(k[e], v[e], old[c][e]);
      if (so >= 0 && j > 0) store8(a.conv_state + ((long long)so * m + j - 1) * a.Hp + ch * 8, v);
    }
  }
  Raw8<T> wy8[CH], wn8[CH], k8[CH], mu8[CH][MIXES];
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (ch >= nch) continue;
    if (y != nullptr) wy8[c].load(reinterpret_cast<const T*>(a.wy) + ch * 8);
    wn8[c].load(reinterpret_cast<const T*>(a.wn) + ch * 8);
    if (a.taps > 0) k8[c].load(reinterpret_cast<const T*>(a.conv) + (long long)m * a.Hp + ch * 8);
    if (mix) {
#pragma unroll
      for (int i = 0; i < MIXES; ++i) mu8[c][i].load(reinterpret_cast<const T*>(a.mu) + (long long)i * a.Hp + ch * 8);
    }
  }
  int flip = 0;
  if (y != nullptr) {
    const float r = 1.f / sqrtf(block_sum(sq, red, flip) / a.H + a.eps);
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nch) continue;
      float w[8];
      wy8[c].get(w);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[c][e] += yv[c][e] * r * (a.w_off + w[e]);
      store8(a.x_out + row * a.Hp + ch * 8, x[c]);
    }
  }
  sq = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c)
#pragma unroll
    for (int e = 0; e < 8; ++e) sq += x[c][e] * x[c][e];
  const float r = 1.f / sqrtf(block_sum(sq, red, flip) / a.H + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (ch >= nch) continue;
    float w[8], k[8], n[8], h[8];
    wn8[c].get(w);
#pragma unroll
    for (int e = 0; e < 8; ++e) k[e] = 0.f;
    if (a.taps > 0) k8[c].get(k);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      n[e] = x[c][e] * r * (a.w_off + w[e]);
      h[e] = fmaf(k[e], n[e], n[e] + old[c][e]);
    }
    T* out = reinterpret_cast<T*>(a.out) + row * a.Hp + ch * 8;
    if (!mix) {
      store8(out, h);
    } else {
#pragma unroll
      for (int i = 0; i < MIXES; ++i) {
        float mu[8], o[8];
        mu8[c][i].get(mu);
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = h[e] + (prev[c][e] - h[e]) * mu[e];
        store8(out + (long long)i * a.out_mix_stride, o);
      }
    }
    if (so >= 0) {
      if (m > 0) store8(a.conv_state + ((long long)so * m + m - 1) * a.Hp + ch * 8, n);
      if (mix) store8(a.shift_state + (long long)so * a.Hp + ch * 8, h);
    }
  }
}

// Rows that depend on nothing but themselves.
template <typename T, int CH>
__global__ void __launch_bounds__(CH == 1 ? 512 : 256, CH == 1 ? 2 : 1) sublayer_alone_kernel(const UbSublayerInArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[2][16];
  const int nch = a.Hp / 8;
  long long src = blockIdx.x;
  if (a.rows != nullptr) {
    src = a.rows[blockIdx.x];
    if (src < 0 || src >= a.x_rows) {
      if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, blockIdx.x);
      src = 0;
    }
  }
  const T* y = reinterpret_cast<const T*>(a.y);
  const T* yx = reinterpret_cast<const T*>(a.yx);
  const float gate = a.y_gate != nullptr ? a.y_gate[src] : 1.f;
  float x[CH][8], f[CH][8];
  float sq = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
#pragma unroll
    for (int e = 0; e < 8; ++e) x[c][e] = f[c][e] = 0.f;
    if (ch >= nch) continue;
    load8(a.x + src * a.Hp + ch * 8, x[c]);
    if (y == nullptr && yx == nullptr) continue;
    if (y != nullptr) {
      load8(y + src * a.Hp + ch * 8, f[c]);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[c][e] *= gate;
    }
    for (int k0 = 0; yx != nullptr && k0 < a.K; k0 += 4) {         // four experts' rows are under way at a time
      Raw8<T> g[4];
      float w[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        w[j] = 0.f;
        const int slot = k0 + j < a.K ? __ldg(a.row_slot + src * a.K + k0 + j) : -1;
        if (slot >= a.slots) {
          set_err(a.err, ERR_BOUNDS, blockIdx.x);
        } else if (slot >= 0) {
          w[j] = __ldg(a.topk_w + src * a.K + k0 + j);
          g[j].load(yx + (long long)slot * a.Hp + ch * 8);
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (w[j] == 0.f) continue;               // uniform
        float v[8];
        g[j].get(v);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[c][e] = fmaf(w[j], v[e], f[c][e]);
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) sq += f[c][e] * f[c][e];           // pad columns are zero
  }
  int flip = 0;
  if (y != nullptr || yx != nullptr) {
    const float r = 1.f / sqrtf(block_sum(sq, red, flip) / a.H + a.eps);
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nch) continue;
      float w[8];
      load8(reinterpret_cast<const T*>(a.wy) + ch * 8, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[c][e] += f[c][e] * r * (a.w_off + w[e]);
      if (a.x_out != nullptr) store8(a.x_out + (long long)blockIdx.x * a.Hp + ch * 8, x[c]);
    }
  }
  sq = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c)
#pragma unroll
    for (int e = 0; e < 8; ++e) sq += x[c][e] * x[c][e];
  const float r = 1.f / sqrtf(block_sum(sq, red, flip) / a.H + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (ch >= nch) continue;
    float w[8];
    load8(reinterpret_cast<const T*>(a.wn) + ch * 8, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[c][e] *= r * (a.w_off + w[e]);
    store8(reinterpret_cast<T*>(a.out) + (long long)blockIdx.x * a.Hp + ch * 8, x[c]);
  }
}

template <typename T>
static cudaError_t launch_alone(const UbSublayerInArgs& a, cudaStream_t st) {
  const int nch = a.Hp / 8;
  const dim3 grid(a.n_rows);
  if (nch <= 512) return launch_pdl(sublayer_alone_kernel<T, 1>, grid, dim3((nch + 31) / 32 * 32), (size_t)0, st, a);
  if (nch <= 1024) return launch_pdl(sublayer_alone_kernel<T, 4>, grid, dim3(256), (size_t)0, st, a);
  return launch_pdl(sublayer_alone_kernel<T, 8>, grid, dim3(256), (size_t)0, st, a);
}

template <typename T>
static cudaError_t launch_step(const UbSublayerInArgs& a, cudaStream_t st) {
  const int nch = a.Hp / 8;
  const int threads = nch >= 512 ? 512 : (nch + 31) / 32 * 32;
  const int ch = (nch + threads - 1) / threads;
  const dim3 grid(a.num_seqs), block(threads);
  if (ch <= 1) return launch_pdl(sublayer_step_kernel<T, 1>, grid, block, (size_t)0, st, a);
  if (ch <= 2) return launch_pdl(sublayer_step_kernel<T, 2>, grid, block, (size_t)0, st, a);
  return launch_pdl(sublayer_step_kernel<T, 4>, grid, block, (size_t)0, st, a);
}

template <typename T>
static cudaError_t launch(const UbSublayerInArgs& a, cudaStream_t st) {
  if (a.q_start == nullptr) return launch_step<T>(a, st);
  if (a.Hp <= 4096 && a.taps >= 1 && a.taps <= 4) {
    if (a.taps == 1) return launch_rows<T, 1>(a, st);
    if (a.taps == 2) return launch_rows<T, 2>(a, st);
    if (a.taps == 3) return launch_rows<T, 3>(a, st);
    return launch_rows<T, 4>(a, st);
  }
  const int nch = a.Hp / 8;
  const int threads = nch >= 256 ? 256 : (nch + 31) / 32 * 32;
  const int ch = (nch + threads - 1) / threads;
  const size_t smem = (size_t)(a.taps > 1 ? a.taps - 1 : 0) * a.Hp * sizeof(float);
  const dim3 grid((a.max_q + a.tile - 1) / a.tile, a.num_seqs), block(threads);
  auto go = [&](auto kern) {
    if (smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return e;
    }
    return launch_pdl(kern, grid, block, smem, st, a);
  };
  if (ch <= 1) return go(sublayer_in_kernel<T, 1>);
  if (ch <= 2) return go(sublayer_in_kernel<T, 2>);
  if (ch <= 4) return go(sublayer_in_kernel<T, 4>);
  return go(sublayer_in_kernel<T, 8>);
}

}  // namespace subin
}  // namespace ub

extern "C" int ub_sublayer_in(const UbSublayerInArgs* a, void* stream) {
  using namespace ub;
  if (a->n_rows > 0) {
    if (a->H <= 0 || a->Hp % 8 != 0 || a->Hp < a->H || a->Hp > 16384) return -2;
    if (a->x == nullptr || a->wn == nullptr || a->out == nullptr || a->taps != 0 || a->n_mix != 0) return -3;
    if ((a->y != nullptr || a->yx != nullptr) && a->wy == nullptr) return -4;
    if (a->yx != nullptr && (a->row_slot == nullptr || a->topk_w == nullptr || a->K <= 0)) return -4;
    if (a->rows != nullptr && a->x_out != nullptr) return -4;
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
    cudaError_t e = a->f32 ? subin::launch_alone<float>(*a, s) : subin::launch_alone<__nv_bfloat16>(*a, s);
    if (e == cudaSuccess) e = cudaGetLastError();
    return e == cudaSuccess ? 0 : -(int)e;
  }
  if (a->num_seqs <= 0 || a->max_q <= 0) return 0;
  if (a->yx != nullptr || a->y_gate != nullptr || a->rows != nullptr) return -4;
  if (a->H <= 0 || a->Hp % 8 != 0 || a->Hp < a->H || a->Hp > 16384) return -2;
  if (a->x == nullptr || a->wn == nullptr || a->out == nullptr || a->tile <= 0 || a->num_seqs > 65535) return -3;
  if (a->y != nullptr && (a->wy == nullptr || a->x_out == nullptr || a->x_out == a->x)) return -4;
  if (a->taps > 0 && a->conv == nullptr) return -5;
  if (a->taps > 1 && (a->conv_state == nullptr || (long long)(a->taps - 1) * a->Hp * 4 > 220 * 1024)) return -5;
  if (a->n_mix != 0 && (a->n_mix != subin::MIXES || a->mu == nullptr || a->shift_state == nullptr)) return -6;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = a->f32 ? subin::launch<float>(*a, st) : subin::launch<__nv_bfloat16>(*a, st);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
