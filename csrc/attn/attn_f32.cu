// K3f / K4f: paged attention in true 32-bit arithmetic over fp32 caches, prompt portions and decoded tokens alike.
//
// One warp per (query token, query head).  Keys are taken 32 at a time: lane j forms the whole score of key j (so a
// score's bits do not depend on where its key sits in the batch of 32), the batch joins an online softmax, and the lanes
// then split the value columns.  Masks (causal, window, kv_start), ALiBi and softmax sinks as in the bf16 kernels.  It
// serves models that are run in 32-bit for accuracy; speed comes second.
#include <math_constants.h>

#include "../common/ptx.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace af32 {

constexpr int WARPS = 4;

template <int MAX_D>
__global__ void __launch_bounds__(WARPS * 32) attn_f32_kernel(const UbAttnArgs a, const int Dv) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float q_s[WARPS][MAX_D];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.z, h = blockIdx.y;
  const int qs = a.q_start != nullptr ? a.q_start[seq] : seq;
  const int q_len = a.q_start != nullptr ? a.q_start[seq + 1] - qs : 1;
  const int qi = blockIdx.x * WARPS + warp;
  if (qi >= q_len) return;                       // warp-uniform; the block has no barrier
  const int kv_len = a.seq_lens[seq];
  const int qpos = kv_len - q_len + qi;
  const int kvh = h / (a.Hq / a.Hkv);
  const int D = a.D;
  const float* q = reinterpret_cast<const float*>(a.q) + (long long)(qs + qi) * a.q_stride + (long long)h * D;
  for (int d = lane; d < D; d += 32) q_s[warp][d] = q[d];
  __syncwarp();
  const float* kc = reinterpret_cast<const float*>(a.k_cache);
  const float* vc = reinterpret_cast<const float*>(a.kv_shared ? a.k_cache : a.v_cache);
  const int v_ld = a.kv_shared ? D : Dv;         // shared rows: the value is the front of the key row
  const int* bt = a.block_tables + (long long)seq * a.max_blocks_per_seq;
  const int hi = a.causal || a.q_start == nullptr ? min(kv_len, qpos + 1) : kv_len;
  int lo = max(a.kv_start, 0);
  if (a.window > 0) lo = max(lo, qpos - a.window + 1);
  if (a.chunk > 0) lo = max(lo, qpos / a.chunk * a.chunk);
  const float slope = a.alibi_slopes != nullptr ? a.alibi_slopes[h] : 0.f;
  float m = -CUDART_INF_F, l = 0.f, acc[MAX_D / 32];
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) acc[i] = 0.f;
  for (int k0 = lo; k0 < hi; k0 += 32) {
    const int pos = k0 + lane;
    long long row = -1;                          // (block, head, offset) row of the caches
    if (pos < hi) {
      const int bi = pos / a.block_size;
      const int blk = bi < a.max_blocks_per_seq ? bt[bi] : -1;
      if (blk < 0 || blk >= a.num_blocks) set_err(a.err, ERR_BOUNDS, seq);
      else row = ((long long)blk * a.Hkv + kvh) * a.block_size + pos % a.block_size;
    }
    float s = -CUDART_INF_F;
    if (row >= 0) {
      const float* kr = kc + row * D;
      float d0 = 0.f;
      for (int d = 0; d < D; d += 4) {
        const float4 kv = *reinterpret_cast<const float4*>(kr + d);
        d0 = fmaf(q_s[warp][d], kv.x, d0);
        d0 = fmaf(q_s[warp][d + 1], kv.y, d0);
        d0 = fmaf(q_s[warp][d + 2], kv.z, d0);
        d0 = fmaf(q_s[warp][d + 3], kv.w, d0);
      }
      d0 *= a.scale;
      if (a.softcap > 0.f) d0 = a.softcap * tanhf(d0 / a.softcap);
      s = d0 + slope * (float)(pos - qpos);
    }
    const float mx = fmaxf(m, warp_max(s));
    if (mx == -CUDART_INF_F) continue;
    const float al = expf(m - mx);               // m = -inf: 0
    const float p = s == -CUDART_INF_F ? 0.f : expf(s - mx);
    l = l * al + warp_sum(p);
    m = mx;
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) acc[i] *= al;
    const int n = min(32, hi - k0);
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const long long rj = __shfl_sync(0xffffffffu, row, j);
      if (rj < 0) continue;
      const float* vr = vc + rj * v_ld;
#pragma unroll
      for (int i = 0; i < MAX_D / 32; ++i)
        if (i * 32 + lane < Dv) acc[i] = fmaf(pj, vr[i * 32 + lane], acc[i]);
    }
  }
  float lse = l > 0.f ? m + logf(l) : -CUDART_INF_F;
  if (a.sinks != nullptr) {
    const float sk = a.sinks[h];
    const float mx = fmaxf(m, sk);
    const float al = expf(m - mx);
    l = l * al + expf(sk - mx);
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) acc[i] *= al;
    lse = mx + logf(l);
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  float* out = reinterpret_cast<float*>(a.out) + (long long)(qs + qi) * a.o_stride + (long long)h * Dv;
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i)
    if (i * 32 + lane < Dv) out[i * 32 + lane] = acc[i] * inv;
  if (lane == 0 && a.lse != nullptr) a.lse[(long long)(qs + qi) * a.Hq + h] = lse;
}

}  // namespace af32
}  // namespace ub

extern "C" int ub_attn_f32(const UbAttnArgs* a, void* stream) {
  using namespace ub::af32;
  const int Dv = a->Dv > 0 ? a->Dv : a->D;
  if (a->num_seqs <= 0) return 0;
  if (a->q_start != nullptr && a->max_q_len <= 0) return 0;
  if (a->Hkv <= 0 || a->Hq % a->Hkv != 0) return -2;
  const int top = a->D > Dv ? a->D : Dv;
  if (top > 640 || (a->kv_shared && Dv > a->D) || a->D % 4 != 0 || (reinterpret_cast<uintptr_t>(a->k_cache) & 15)) return -4;
  if (a->merge_o != nullptr || a->splits > 1) return -7;
  const int mq = a->q_start != nullptr ? a->max_q_len : 1;
  const dim3 grid((mq + WARPS - 1) / WARPS, a->Hq, a->num_seqs), block(WARPS * 32);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = top <= 256 ? ub::launch_pdl(attn_f32_kernel<256>, grid, block, (size_t)0, st, *a, Dv)
                             : ub::launch_pdl(attn_f32_kernel<640>, grid, block, (size_t)0, st, *a, Dv);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
