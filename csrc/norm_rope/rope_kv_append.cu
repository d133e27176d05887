// K6: per-head RMSNorm (optional, QK-norm models) + rotary embedding of q and k + append of the
// rotated k and of v into the paged KV cache, in one pass over the QKV GEMM output.
// Cache layout: [num_blocks, Hkv, block_size, D] bf16 for K and for V, so one (block, head) page
// is a contiguous block_size x D tile that attention kernels can fetch with bulk copies.
// One CTA per token, one warp per head (round-robin).  cos/sin are computed on the fly from the
// position (no table in HBM); partial rotary, linear position scaling and Llama-3 frequency
// scaling are parameters (or a table of frequencies).  Heads with a norm, interleaved pairs or a value size of its own go
// through a second kernel in which a few lanes own a head, eight elements each; it also has a 32-bit form, and one norm over
// all query (key) elements of a token instead of one per head.
// Slots are bounds-checked: a bad slot sets the error word and is skipped.
//
// Replaces in the reference: apply_rope / apply_rope_with_offset (crates/runtime/src/models_v2/
// llama.rs:761-883), LayerKVCache::append (crates/runtime/src/kv_cache.rs:91-134) and the scalar /
// NEON apply_rope (crates/runtime/src/simd/arch/scalar.rs:112-153).
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {

__device__ __forceinline__ float rope_inv_freq(int i, const UbRopeArgs& a) {
  // i = pair index in [0, rd/2)
  float inv = exp2f(-(2.f * i / a.rotary_dim) * log2f(a.theta));
  if (a.l3_factor > 0.f) {
    const float two_pi = 6.283185307179586f;
    const float wavelen = two_pi / inv;
    const float low_wl = a.l3_orig_ctx / a.l3_low_freq_factor;
    const float high_wl = a.l3_orig_ctx / a.l3_high_freq_factor;
    if (wavelen > low_wl) {
      inv = inv / a.l3_factor;
    } else if (wavelen >= high_wl) {
      const float smooth = (a.l3_orig_ctx / wavelen - a.l3_low_freq_factor) /
                           (a.l3_high_freq_factor - a.l3_low_freq_factor);
      inv = (1.f - smooth) * inv / a.l3_factor + smooth * inv;
    }
  }
  return inv;
}

__global__ void __launch_bounds__(128) rope_kv_append_kernel(const UbRopeArgs a) {
  pdl_launch_dependents();
  pdl_wait();          // no global access before the previous kernel has completed
  extern __shared__ float sm[];  // [4 warps][D] staging (QK-norm / interleaved path), then [rotary_dim] cos | sin
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int D = a.D;
  float* hv = sm + warp * D;
  const int nheads = a.Hq + 2 * a.Hkv;
  __nv_bfloat16* base = reinterpret_cast<__nv_bfloat16*>(a.qkv) + (long long)t * nheads * D;
  const float pos = (float)a.positions[t] * a.pos_scale;
  const long long slot = a.slot_mapping != nullptr ? (long long)a.slot_mapping[t] : -1;
  bool slot_ok = slot >= 0;
  if (slot >= a.num_slots) {
    slot_ok = false;
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, t);
  }
  const int half = a.rotary_dim / 2;
  // the angles depend on the token and the pair only: once per CTA, shared by all heads
  float* cs = sm + 4 * D;           // cos [half] then sin [half]
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(pos * rope_inv_freq(i, a), &s, &c);
    cs[i] = c;
    cs[half + i] = s;
  }
  __syncthreads();
  const long long blk = slot_ok ? slot / a.block_size : 0, off = slot_ok ? slot % a.block_size : 0;
  const bool fast = !a.interleaved && a.q_norm_w == nullptr && a.k_norm_w == nullptr && (half % 2 == 0) && (D % 8 == 0);

  if (fast) {
    // Flat over (head, two adjacent pairs): consecutive threads touch consecutive 4-byte words of a head, and a thread's
    // loads of several items are issued before the first of them is used.
    constexpr int U = 4;
    const int ppl = half / 2;                       // items per rotated head
    const int nrot = a.Hq + a.Hkv;
    const int items = nrot * ppl;
    __nv_bfloat16* kc = reinterpret_cast<__nv_bfloat16*>(a.k_cache) + ((blk * a.Hkv) * a.block_size + off) * D;
    const long long khead = (long long)a.block_size * D;      // cache stride between KV heads of one block
    for (int it0 = threadIdx.x; it0 < items; it0 += U * blockDim.x) {
      uint32_t lo[U], hi[U];
      int hh[U], ii[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int it = it0 + u * blockDim.x;
        hh[u] = -1;
        if (it < items) {
          hh[u] = it / ppl;
          ii[u] = 2 * (it - hh[u] * ppl);
          const __nv_bfloat16* src = base + (long long)hh[u] * D;
          lo[u] = *reinterpret_cast<const uint32_t*>(src + ii[u]);
          hi[u] = *reinterpret_cast<const uint32_t*>(src + ii[u] + half);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (hh[u] < 0) continue;
        const int i = ii[u];
        const float c0 = cs[i], c1 = cs[i + 1], s0 = cs[half + i], s1 = cs[half + i + 1];
        const float x0 = bf16_lo(lo[u]), x1 = bf16_hi(lo[u]), y0 = bf16_lo(hi[u]), y1 = bf16_hi(hi[u]);
        const uint32_t olo = pack_bf16x2(x0 * c0 - y0 * s0, x1 * c1 - y1 * s1);
        const uint32_t ohi = pack_bf16x2(y0 * c0 + x0 * s0, y1 * c1 + x1 * s1);
        __nv_bfloat16* src = base + (long long)hh[u] * D;
        *reinterpret_cast<uint32_t*>(src + i) = olo;
        *reinterpret_cast<uint32_t*>(src + i + half) = ohi;
        if (hh[u] >= a.Hq && slot_ok) {
          __nv_bfloat16* kd = kc + (hh[u] - a.Hq) * khead;
          *reinterpret_cast<uint32_t*>(kd + i) = olo;
          *reinterpret_cast<uint32_t*>(kd + i + half) = ohi;
        }
      }
    }
    if (slot_ok) {
      // partial rotary: the unrotated tail of every K head goes to the cache as it is
      const int tail = (D - a.rotary_dim) / 2;
      for (int it = threadIdx.x; it < a.Hkv * tail; it += blockDim.x) {
        const int hk = it / tail, i = a.rotary_dim + 2 * (it - hk * tail);
        *reinterpret_cast<uint32_t*>(kc + hk * khead + i) =
            *reinterpret_cast<const uint32_t*>(base + (long long)(a.Hq + hk) * D + i);
      }
      // V heads: straight 16-byte copies
      __nv_bfloat16* vcd = reinterpret_cast<__nv_bfloat16*>(a.v_cache) + ((blk * a.Hkv) * a.block_size + off) * D;
      const int cpr = D / 8;
      for (int it = threadIdx.x; it < a.Hkv * cpr; it += blockDim.x) {
        const int hk = it / cpr, c = it - hk * cpr;
        reinterpret_cast<uint4*>(vcd + hk * khead)[c] =
            reinterpret_cast<const uint4*>(base + (long long)(a.Hq + a.Hkv + hk) * D)[c];
      }
    }
    return;
  }

  for (int h = warp; h < nheads; h += 4) {
    const bool is_q = h < a.Hq;
    const bool is_k = !is_q && h < a.Hq + a.Hkv;
    __nv_bfloat16* src = base + (long long)h * D;
    if (!is_q && !is_k) {
      // V head: straight copy into the cache
      if (slot_ok) {
        const int hk = h - a.Hq - a.Hkv;
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(a.v_cache) + ((blk * a.Hkv + hk) * a.block_size + off) * D;
        if (D % 8 == 0) {
          for (int i = lane; i < D / 8; i += 32) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
        } else {
          for (int i = lane; i < D; i += 32) dst[i] = src[i];
        }
      }
      continue;
    }
    __nv_bfloat16* kdst = nullptr;
    if (is_k && slot_ok) {
      const int hk = h - a.Hq;
      kdst = reinterpret_cast<__nv_bfloat16*>(a.k_cache) + ((blk * a.Hkv + hk) * a.block_size + off) * D;
    }
    float ss = 0.f;
    for (int i = lane; i < D; i += 32) {
      const float v = __bfloat162float(src[i]);
      hv[i] = v;
      ss += v * v;
    }
    const __nv_bfloat16* nw = is_q ? reinterpret_cast<const __nv_bfloat16*>(a.q_norm_w)
                                   : reinterpret_cast<const __nv_bfloat16*>(a.k_norm_w);
    if (nw != nullptr) {
      ss = warp_sum(ss);
      const float rstd = rsqrtf(ss / D + a.norm_eps);
      __syncwarp();
      for (int i = lane; i < D; i += 32) hv[i] = hv[i] * rstd * __bfloat162float(nw[i]);
    }
    __syncwarp();
    if (half > 0) {
      for (int i = lane; i < half; i += 32) {
        const float c = cs[i], s = cs[half + i];
        const int i0 = a.interleaved ? 2 * i : i;
        const int i1 = a.interleaved ? 2 * i + 1 : i + half;
        const float x0 = hv[i0], x1 = hv[i1];
        hv[i0] = x0 * c - x1 * s;
        hv[i1] = x1 * c + x0 * s;
      }
      __syncwarp();
    }
    for (int i = lane; i < D; i += 32) {
      const __nv_bfloat16 b = __float2bfloat16(hv[i]);
      src[i] = b;
      if (kdst != nullptr) kdst[i] = b;
    }
    __syncwarp();
  }
}

// LPH lanes per head (a power of two, LPH * 8 >= D), eight consecutive elements of the head per lane: the norm is a shuffle
// reduction among the lanes of the head, interleaved pairs are lane-local, half-split pairs come from the lane that holds
// the other half.  K goes to the cache and, unless k_cache_only, back into the row; V is copied to the cache.  A thread
// requests its chunks of U heads (and its share of V) before it works out the angles; a lane meets the same angles in every
// head, so they stay in registers.
enum { PAIR_HALVES = 0, PAIR_NEIGHBOURS = 1, PAIR_ODD = 2 /* halves that are no whole chunks */ };

// VTURN: values are cached turned by their position.
template <typename T, int LPH, int PAIR, bool VTURN>
__global__ void __launch_bounds__(128, 8) head_norm_rope_kernel(const UbRopeArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int U = 2;
  extern __shared__ float cs[];                   // cos [half] then sin [half], the same for the values
  __shared__ float red[2][4];
  const int t = blockIdx.x, D = a.D, Dv = a.Dv, half = a.rotary_dim / 2;
  constexpr int ngrp = 128 / LPH, batch = U * ngrp;
  const int grp = threadIdx.x / LPH, c = threadIdx.x % LPH;
  const int nrot = a.Hq + a.Hkv;
  const bool have = c * 8 < D;                    // the last lanes of a group may own nothing
  T* row = reinterpret_cast<T*>(a.qkv) + (long long)t * a.ld;
  float v[U][8];
  auto load = [&](int h0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int h = h0 + u * ngrp + grp;
#pragma unroll
      for (int e = 0; e < 8; ++e) v[u][e] = 0.f;
      if (h < nrot && have) load8(row + h * D + c * 8, v[u]);
    }
  };
  load(0);
  const long long slot = a.slot_mapping != nullptr ? (long long)a.slot_mapping[t] : -1;
  bool slot_ok = slot >= 0;
  if (slot >= a.num_slots) {
    slot_ok = false;
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, t);
  }
  const long long blk = slot_ok ? slot / a.block_size : 0, off = slot_ok ? slot % a.block_size : 0;
  const float pos = (float)a.positions[t] * a.pos_scale;
  const int vh = VTURN ? a.v_rot / 2 : 0;
  // the first chunk of V that this thread turns, and its partners
  float vx[8], vo[8];
  auto load_v = [&](int it) {
    const int cpr = Dv / 8, hk = it / cpr, i0 = (it - hk * cpr) * 8;
    const T* head = row + nrot * D + hk * Dv;
    load8(head + i0, vx);
    if (vh % 8 == 0) {
      if (i0 < 2 * vh) load8(head + (i0 < vh ? i0 + vh : i0 - vh), vo);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) vo[e] = i0 + e < 2 * vh ? (float)head[i0 + e < vh ? i0 + e + vh : i0 + e - vh] : 0.f;
    }
  };
  const bool turn_v = VTURN && slot_ok && a.v_cache != nullptr;
  if (turn_v && threadIdx.x < a.Hkv * (Dv / 8)) load_v(threadIdx.x);
  float* vcs = cs + 2 * half;
  for (int i = threadIdx.x; i < half + vh; i += 128) {
    const bool v_angle = VTURN && i >= half;
    const float f = v_angle ? a.v_inv_freq[i - half] : a.inv_freq != nullptr ? a.inv_freq[i] : rope_inv_freq(i, a);
    float s, co;
    sincosf(pos * f, &s, &co);
    if (v_angle) {
      vcs[i - half] = co;
      vcs[vh + i - half] = s;
    } else {
      cs[i] = co * a.gain;
      cs[half + i] = s * a.gain;
    }
  }
  if (slot_ok && a.v_cache != nullptr && !VTURN) {
    const int cpr = Dv / 8;
    const T* vr = row + nrot * D;
    T* vd = reinterpret_cast<T*>(a.v_cache) + (blk * a.Hkv * a.block_size + off) * Dv;
    for (int it = threadIdx.x; it < a.Hkv * cpr; it += 128) {
      const int hk = it / cpr, ch = it - hk * cpr;
      float w[8];
      load8(vr + it * 8, w);
      store8(vd + (long long)hk * a.block_size * Dv + ch * 8, w);
    }
  }
  if (a.row_norm) {
    float sq = 0.f, sk = 0.f;
    for (int h0 = 0; h0 < nrot; h0 += batch) {
      if (h0 > 0) load(h0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += v[u][e] * v[u][e];
        if (h0 + u * ngrp + grp < a.Hq) sq += ss; else sk += ss;
      }
    }
    if (batch < nrot) load(0);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sk; }
  }
  __syncthreads();                                // angles and sums complete; nobody has written to the row yet
  if (turn_v) {                    // turned values go to the cache only, the row stays
    const int cpr = Dv / 8;
    T* vd = reinterpret_cast<T*>(a.v_cache) + (blk * a.Hkv * a.block_size + off) * Dv;
    for (int it = threadIdx.x; it < a.Hkv * cpr; it += 128) {
      const int hk = it / cpr, i0 = (it - hk * cpr) * 8;
      if (it >= 128) load_v(it);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int i = i0 + e;
        if (i < vh) vx[e] = vx[e] * vcs[i] - vo[e] * vcs[vh + i];
        else if (i < 2 * vh) vx[e] = vx[e] * vcs[i - vh] + vo[e] * vcs[i];
      }
      store8(vd + (long long)hk * a.block_size * Dv + i0, vx);
    }
  }
  float rq = 1.f, rk = 1.f;                       // row norms: one factor for all queries, one for all keys
  if (a.row_norm) {
    rq = 1.f / sqrtf((red[0][0] + red[0][1] + red[0][2] + red[0][3]) / (float)(a.Hq * a.norm_dim) + a.norm_eps);
    if (a.Hkv > 0) rk = 1.f / sqrtf((red[1][0] + red[1][1] + red[1][2] + red[1][3]) / (float)(a.Hkv * a.norm_dim) + a.norm_eps);
  }
  const bool normed = a.q_norm_w != nullptr || a.k_norm_w != nullptr;
  // element e of this lane's chunk becomes x * co[e] + other * si[e]
  constexpr int NA = PAIR == PAIR_NEIGHBOURS ? 4 : 8;
  float co[NA], si[NA];
  int partner = c;
#pragma unroll
  for (int e = 0; e < NA; ++e) {
    co[e] = 1.f;
    si[e] = 0.f;
    if (PAIR == PAIR_NEIGHBOURS) {
      const int i = c * 4 + e;
      if (i < half) { co[e] = cs[i]; si[e] = cs[half + i]; }
    } else {
      const int i = c * 8 + e;
      if (i < half) { co[e] = cs[i]; si[e] = -cs[half + i]; }
      else if (i < 2 * half) { co[e] = cs[i - half]; si[e] = cs[i]; }
    }
  }
  if (PAIR == PAIR_HALVES) {
    const int hc = half / 8;                      // chunks per half
    partner = c < hc ? c + hc : (c < 2 * hc ? c - hc : c);
  }
  T* kd = reinterpret_cast<T*>(a.k_cache) + (blk * a.Hkv * a.block_size + off) * D + c * 8;
  for (int h0 = 0; h0 < nrot; h0 += batch) {
    if (h0 > 0) load(h0);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int h = h0 + u * ngrp + grp;
      if (h0 + u * ngrp >= nrot) break;           // uniform
      const bool ok = h < nrot && have;
      float (&x)[8] = v[u];
      const T* nw = reinterpret_cast<const T*>(h < a.Hq ? a.q_norm_w : a.k_norm_w);
      float r = 1.f;
      if (normed) {
        if (a.row_norm) {
          r = h < a.Hq ? rq : rk;
          nw += (h < a.Hq ? h : h - a.Hq) * D;
        } else {
          float ss = 0.f;
#pragma unroll
          for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
#pragma unroll
          for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
          if (nw != nullptr) r = 1.f / sqrtf(ss / (float)a.norm_dim + a.norm_eps);
        }
        if (ok && nw != nullptr) {
          float w[8];
          load8(nw + c * 8, w);
#pragma unroll
          for (int e = 0; e < 8; ++e) x[e] = x[e] * r * w[e];
        }
      }
      if (half > 0) {
        if (PAIR == PAIR_NEIGHBOURS) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float x0 = x[2 * e], x1 = x[2 * e + 1];
            x[2 * e] = x0 * co[e] - x1 * si[e];
            x[2 * e + 1] = x1 * co[e] + x0 * si[e];
          }
        } else if (PAIR == PAIR_ODD) {            // the other half of a pair lies across chunks: fetched element by element
          float o[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const int i = c * 8 + e, j = i < half ? i + half : i - half;
            o[e] = 0.f;
            if (ok && i < 2 * half) o[e] = (float)row[h * D + j] * r * (nw != nullptr ? (float)nw[j] : 1.f);
          }
          __syncwarp();                           // a head's lanes have read it before one of them writes
#pragma unroll
          for (int e = 0; e < 8; ++e) x[e] = x[e] * co[e % NA] + o[e] * si[e % NA];
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) x[e] = x[e] * co[e % NA] + __shfl_sync(0xffffffffu, x[e], partner, LPH) * si[e % NA];
        }
      }
      if (!ok) continue;
      if (h < a.Hq || !a.k_cache_only || !slot_ok) store8(row + h * D + c * 8, x);
      if (h >= a.Hq && slot_ok && a.k_cache != nullptr) store8(kd + (long long)(h - a.Hq) * a.block_size * D, x);
    }
  }
}

template <typename T, int PAIR, bool VTURN>
static cudaError_t launch_head_norm_rope(const UbRopeArgs& a, cudaStream_t st) {
  const size_t smem = (size_t)(a.rotary_dim + (a.v_inv_freq != nullptr ? a.v_rot : 0) + 1) * sizeof(float);
  const dim3 grid(a.T), block(128);
  if (a.D <= 32) return launch_pdl(head_norm_rope_kernel<T, 4, PAIR, VTURN>, grid, block, smem, st, a);
  if (a.D <= 64) return launch_pdl(head_norm_rope_kernel<T, 8, PAIR, VTURN>, grid, block, smem, st, a);
  if (a.D <= 128) return launch_pdl(head_norm_rope_kernel<T, 16, PAIR, VTURN>, grid, block, smem, st, a);
  return launch_pdl(head_norm_rope_kernel<T, 32, PAIR, VTURN>, grid, block, smem, st, a);
}

template <typename T, int PAIR>
static cudaError_t launch_head_norm_rope(const UbRopeArgs& a, cudaStream_t st) {
  return a.v_inv_freq != nullptr ? launch_head_norm_rope<T, PAIR, true>(a, st) : launch_head_norm_rope<T, PAIR, false>(a, st);
}

template <typename T>
static cudaError_t launch_head_norm_rope(const UbRopeArgs& a, cudaStream_t st) {
  if (a.interleaved) return launch_head_norm_rope<T, PAIR_NEIGHBOURS>(a, st);
  return a.rotary_dim % 16 != 0 ? launch_head_norm_rope<T, PAIR_ODD>(a, st) : launch_head_norm_rope<T, PAIR_HALVES>(a, st);
}

}  // namespace ub

extern "C" int ub_rope_kv_append(const UbRopeArgs* a, void* stream_v) {
  if (a->T <= 0) return 0;
  if (a->D > 512 || (a->rotary_dim & 1) || a->rotary_dim > a->D) return -2;
  const int Dv = a->Dv > 0 ? a->Dv : a->D;
  const long long dense = (long long)(a->Hq + a->Hkv) * a->D + (long long)a->Hkv * Dv;
  const long long ld = a->ld > 0 ? a->ld : dense;
  if (a->v_inv_freq != nullptr && ((a->v_rot & 1) || a->v_rot <= 0 || a->v_rot > Dv)) return -2;
  const bool general = a->f32 || a->v_inv_freq != nullptr || Dv != a->D || a->inv_freq != nullptr || (a->norm_dim > 0 && a->norm_dim != a->D) || a->row_norm || ld != dense;
  const bool wide_ok = a->D % 8 == 0 && Dv % 8 == 0 && a->D <= 256 && ld % 8 == 0 && ld >= dense;
  if (a->row_norm && (a->q_norm_w == nullptr || (a->Hkv > 0 && a->k_norm_w == nullptr))) return -5;
  if (general && !wide_ok) return -4;
  if (wide_ok && (general || a->interleaved || a->q_norm_w != nullptr || a->k_norm_w != nullptr)) {
    UbRopeArgs b = *a;
    b.Dv = Dv;
    b.ld = ld;
    if (b.norm_dim <= 0) b.norm_dim = b.D;
    if (b.gain <= 0.f) b.gain = 1.f;
    cudaError_t e = b.f32 ? ub::launch_head_norm_rope<float>(b, (cudaStream_t)stream_v)
                          : ub::launch_head_norm_rope<__nv_bfloat16>(b, (cudaStream_t)stream_v);
    if (e == cudaSuccess) e = cudaGetLastError();
    return e == cudaSuccess ? 0 : -(int)e;
  }
  ub::launch_pdl(ub::rope_kv_append_kernel, dim3(a->T), dim3(128), (4 * a->D + a->rotary_dim) * sizeof(float), (cudaStream_t)stream_v, *a);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
