// K3o: what stands between an attention's outputs and its output projection, per token and head, in 32 bits:
//
//   maps = 2:   o = a1 - lambda * a2,   o = o / sqrt(mean(o^2) + eps) * factor      (a1, a2: the outputs of heads 2 h and 2 h + 1)
//   rotation:   pair (u, v) = (o_i, o_(i + half)) becomes (u cos + v sin, v cos - u sin), angle = position * freq_i
//               (values that were rotated by their own position are turned back by the query's)
//   gate:       o *= sigmoid(g_head), or o_e *= sigmoid(g_(head, e))
//
// One CTA per token; LPH lanes (a power of two, LPH * 8 >= dv) own a head, eight elements each.  A lane meets the same angles in
// every head, so they stay in registers.
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace fin {

enum { TURN_NONE = 0, TURN_CHUNKS = 1, TURN_ODD = 2 /* halves that are no whole chunks */ };

__device__ __forceinline__ float sigmoid(float v) { return 1.f / (1.f + __expf(-v)); }

template <typename T, int LPH, int TURN>
__global__ void __launch_bounds__(128) attn_finish_kernel(const UbAttnFinishArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float cs[];                   // cos [half] then sin [half]
  constexpr int ngrp = 128 / LPH;
  const int t = blockIdx.x, grp = threadIdx.x / LPH, c = (threadIdx.x % LPH) * 8, dv = a.dv, half = a.dv_real / 2;
  float co[8], si[8];
  if (TURN != TURN_NONE) {
    const float pos = (float)a.positions[t];
    for (int i = threadIdx.x; i < half; i += 128) {
      float s, k;
      sincosf(pos * a.inv_freq[i], &s, &k);
      cs[i] = k;
      cs[half + i] = s;
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const int i = c + e;
      co[e] = 1.f;
      si[e] = 0.f;
      if (i < half) { co[e] = cs[i]; si[e] = cs[half + i]; }
      else if (i < 2 * half) { co[e] = cs[i - half]; si[e] = -cs[i]; }
    }
  }
  const int hc = half / 8, ch = c / 8, partner = ch < hc ? ch + hc : (ch < 2 * hc ? ch - hc : ch);
  const T* att = reinterpret_cast<const T*>(a.att) + (long long)t * a.ld_att;
  const T* gate = reinterpret_cast<const T*>(a.gate) + (long long)t * a.ld_gate;
  T* out = reinterpret_cast<T*>(a.out) + (long long)t * a.ld_out;
  for (int h0 = 0; h0 < a.H; h0 += ngrp) {
    const int h = h0 + grp;
    const bool on = h < a.H && c < dv;
    float o[8], g[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = g[e] = 0.f;
    if (on) {
      load8(att + (long long)h * a.maps * dv + c, o);
      if (a.gate_kind == 2) load8(gate + (long long)h * dv + c, g);
      else if (a.gate_kind == 1) g[0] = (float)gate[h];
    }
    if (a.maps == 2) {
      float b[8], sq = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) b[e] = 0.f;
      if (on) load8(att + ((long long)h * 2 + 1) * dv + c, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        o[e] = fmaf(-a.lambda, b[e], o[e]);
        sq = fmaf(o[e], o[e], sq);                // pad elements are zero
      }
#pragma unroll
      for (int x = LPH / 2; x > 0; x >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, x);
      const float r = a.factor / sqrtf(sq / a.dv_real + a.eps);
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] *= r;
    }
    if (TURN == TURN_CHUNKS) {
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] = fmaf(__shfl_sync(0xffffffffu, o[e], partner, LPH), si[e], o[e] * co[e]);
    }
    if (!on) continue;
    if (TURN == TURN_ODD) {                       // one map: the other half of a pair is read again
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int i = c + e;
        if (i < 2 * half) o[e] = fmaf((float)att[(long long)h * dv + (i < half ? i + half : i - half)], si[e], o[e] * co[e]);
      }
    }
    if (a.gate_kind == 2) {
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] *= sigmoid(g[e]);
    } else if (a.gate_kind == 1) {
      const float s = sigmoid(g[0]);
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] *= s;
    }
    store8(out + (long long)h * dv + c, o);
  }
}

template <typename T, int LPH>
static cudaError_t launch(const UbAttnFinishArgs& a, cudaStream_t st) {
  const dim3 grid(a.T), block(128);
  if (a.inv_freq == nullptr) return launch_pdl(attn_finish_kernel<T, LPH, TURN_NONE>, grid, block, (size_t)0, st, a);
  const size_t smem = sizeof(float) * (a.dv_real > 0 ? a.dv_real : 1);
  return a.dv_real % 16 == 0 ? launch_pdl(attn_finish_kernel<T, LPH, TURN_CHUNKS>, grid, block, smem, st, a)
                             : launch_pdl(attn_finish_kernel<T, LPH, TURN_ODD>, grid, block, smem, st, a);
}

template <typename T>
static cudaError_t launch(const UbAttnFinishArgs& a, cudaStream_t st) {
  if (a.dv <= 32) return launch<T, 4>(a, st);
  if (a.dv <= 64) return launch<T, 8>(a, st);
  if (a.dv <= 128) return launch<T, 16>(a, st);
  return launch<T, 32>(a, st);
}

}  // namespace fin
}  // namespace ub

extern "C" int ub_attn_finish(const UbAttnFinishArgs* a, void* stream) {
  using namespace ub;
  if (a->T <= 0) return 0;
  if (a->H <= 0 || a->dv % 8 != 0 || a->dv <= 0 || a->dv > 256 || a->dv_real <= 0 || a->dv_real > a->dv) return -2;
  if (a->maps != 1 && a->maps != 2) return -2;
  if (a->ld_att % 8 != 0 || a->ld_out % 8 != 0 || (a->gate_kind == 2 && a->ld_gate % 8 != 0)) return -3;
  if (a->att == nullptr || a->out == nullptr || (a->gate_kind != 0 && a->gate == nullptr)) return -3;
  if (a->inv_freq != nullptr && (a->positions == nullptr || a->dv_real % 2 != 0 || (a->maps == 2 && a->dv_real % 16 != 0))) return -4;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = a->f32 ? fin::launch<float>(*a, st) : fin::launch<__nv_bfloat16>(*a, st);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
