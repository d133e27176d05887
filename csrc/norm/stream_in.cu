// K5t: what a sublayer reads, for designs whose norm needs no statistics (Dynamic Tanh, "Transformers without Normalization", Zhu
// et al.) around a 32-bit residual stream.  One pass over the token rows does, all in 32 bits:
//
//   x' = x + scale * y                            (y: the previous sublayer's rows; absent at the first sublayer)
//   s  = sum_j mix[j] * X_j + mix[n] * x'         (average over depth: X_j are the rows of n earlier layers; absent: s = x')
//   h  = tanh(alpha * s) * w + b
//   out_t = h_t + (h_(t-1) - h_t) * shift         (absent: out = h)
//
// x may be the embedding rows of token ids, gathered here.  x' (to be one of the X_j of later layers) and s (the stream that goes
// on) are written where they are asked for.
//
// Columns never meet, so a thread owns eight of them and walks over the tokens of a tile without a barrier.  With a token shift the
// rows are portions of sequences: what lies in front of a portion is the sequence's state row, the portion leaves its last h in
// ANOTHER row, and the row in front of a tile is computed again from x, y and X (so s goes to a buffer of its own).
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace streamin {

constexpr int THREADS = 128;

template <typename T, bool SHIFT>
__global__ void __launch_bounds__(THREADS) stream_in_kernel(const UbStreamInArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * THREADS + threadIdx.x) * 8;
  const int seq = SHIFT ? blockIdx.z : 0;
  int qs = 0, q_len = a.n_rows;
  if (SHIFT) {
    qs = a.q_start != nullptr ? a.q_start[seq] : seq;
    q_len = a.q_start != nullptr ? a.q_start[seq + 1] - qs : 1;
  }
  const int t0 = blockIdx.y * a.tile, t1 = min(t0 + a.tile, q_len);
  if (c >= a.Hp || t0 >= t1) return;               // no barriers below
  const long long Hp = a.Hp, row0 = SHIFT ? a.row0 + qs : 0;
  float w[8], b[8], prev[8], mu[8];
  load8(reinterpret_cast<const T*>(a.w) + c, w);
  load8(reinterpret_cast<const T*>(a.b) + c, b);
#pragma unroll
  for (int e = 0; e < 8; ++e) prev[e] = mu[e] = 0.f;
  const float m_own = a.mix != nullptr ? a.mix[a.n_hist] : 1.f;

  // h of one row; `dst` >= 0: x' and s are kept there
  auto value = [&](long long src, long long dst, float (&h)[8]) {
    float x[8];
    if (a.ids != nullptr) {
      int id = a.ids[src];
      if (id < 0 || id >= a.vocab) {
        if (c == 0) set_err(a.err, ERR_BOUNDS, (int)src);
        id = 0;
      }
      load8(reinterpret_cast<const T*>(a.table) + id * Hp + c, x);
    } else {
      load8(a.x + src * Hp + c, x);
    }
    if (a.y != nullptr) {
      float y[8];
      load8(reinterpret_cast<const T*>(a.y) + src * Hp + c, y);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = fmaf(a.scale, y[e], x[e]);
    }
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
    if (a.mix != nullptr) {                        // all loads of a row are under way before the first store
      const float* p = a.hist + src * Hp + c;
#pragma unroll 4
      for (int j = 0; j < a.n_hist; ++j, p += a.hist_stride) {
        float v[8];
        load8(p, v);
        const float m = __ldg(a.mix + j);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = fmaf(m, v[e], acc[e]);
      }
    }
    if (dst >= 0 && a.x_res != nullptr) store8(a.x_res + dst * Hp + c, x);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = fmaf(m_own, x[e], acc[e]);              // without an average 1 * x + 0
    if (dst >= 0 && a.x_out != nullptr) store8(a.x_out + dst * Hp + c, x);
#pragma unroll
    for (int e = 0; e < 8; ++e) h[e] = fmaf(tanhf(a.alpha * x[e]), w[e], b[e]);
  };

  if (!SHIFT) {
    for (int t = t0; t < t1; ++t) {
      long long src = t;
      if (a.rows != nullptr) {
        src = a.rows[t];
        if (src < 0 || src >= a.x_rows) {
          if (c == 0) set_err(a.err, ERR_BOUNDS, t);
          src = 0;
        }
      }
      float h[8];
      value(src, t, h);
      store8(reinterpret_cast<T*>(a.out) + t * Hp + c, h);
    }
    return;
  }
  int si = a.state_in != nullptr ? a.state_in[seq] : -1, so = a.state_out != nullptr ? a.state_out[seq] : -1;
  if (si >= a.state_rows || so >= a.state_rows) {
    if (c == 0) set_err(a.err, ERR_BOUNDS, seq);
    si = so = -1;
  }
  load8(reinterpret_cast<const T*>(a.shift) + c, mu);
  if (t0 > 0) value(row0 + t0 - 1, -1, prev);
  else if (si >= 0) load8(a.shift_state + si * Hp + c, prev);
  for (int t = t0; t < t1; ++t) {
    float h[8], o[8];
    value(row0 + t, row0 + t, h);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      o[e] = fmaf(prev[e] - h[e], mu[e], h[e]);
      prev[e] = h[e];
    }
    store8(reinterpret_cast<T*>(a.out) + (row0 + t) * Hp + c, o);
  }
  if (t1 == q_len && so >= 0) store8(a.shift_state + so * Hp + c, prev);
}

template <typename T>
static cudaError_t launch(const UbStreamInArgs& a, cudaStream_t st) {
  const int cols = (a.Hp / 8 + THREADS - 1) / THREADS;
  if (a.shift != nullptr)
    return launch_pdl(stream_in_kernel<T, true>, dim3(cols, (a.max_q + a.tile - 1) / a.tile, a.num_seqs), dim3(THREADS), (size_t)0, st, a);
  return launch_pdl(stream_in_kernel<T, false>, dim3(cols, (a.n_rows + a.tile - 1) / a.tile), dim3(THREADS), (size_t)0, st, a);
}

}  // namespace streamin
}  // namespace ub

extern "C" int ub_stream_in(const UbStreamInArgs* a, void* stream) {
  using namespace ub;
  const bool shift = a->shift != nullptr;
  if (shift ? (a->num_seqs <= 0 || a->max_q <= 0) : a->n_rows <= 0) return 0;
  if (a->Hp <= 0 || a->Hp % 8 != 0 || a->tile <= 0) return -2;
  if ((a->x == nullptr) == (a->ids == nullptr) || a->w == nullptr || a->b == nullptr || a->out == nullptr) return -3;
  if (a->ids != nullptr && (a->table == nullptr || a->vocab <= 0)) return -3;
  if (a->mix != nullptr && (a->n_hist < 0 || (a->n_hist > 0 && a->hist == nullptr))) return -4;
  if (shift && (a->num_seqs > 65535 || a->rows != nullptr || (a->x != nullptr && (a->x_out == a->x || a->x_res == a->x)))) return -5;
  if (shift && (a->state_in != nullptr || a->state_out != nullptr) && a->shift_state == nullptr) return -5;
  if (a->rows != nullptr && (a->x_out != nullptr || a->x_res != nullptr)) return -5;
  const long long tiles = ((shift ? a->max_q : a->n_rows) + (long long)a->tile - 1) / a->tile;
  if (tiles > 65535) return -6;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = a->f32 ? streamin::launch<float>(*a, st) : streamin::launch<__nv_bfloat16>(*a, st);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
