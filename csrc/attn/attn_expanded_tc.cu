// K3m: prompt attention of multi-head latent attention on the 5th-generation tensor cores, over latents that have been
// expanded to keys and values of every head.
//
// Inputs lie in plain rows, no pages: q [T, H, dim + rot]; kv [R, H, dim + vdim] (unrotated key and value of every head, the
// product of the gathered latents with the key and value matrices) and lat [R, kv_rank + rot], whose tail is the rotated key
// part that all heads share.  The rows of a sequence are consecutive from a multiple of 16 on.
//
// Work unit: 128 query tokens of one (sequence, head).  Per tile of 128 keys:
//   S = Q K^T           tcgen05.mma, K in 64-wide column blocks: up to two of the head's own, one of the shared part
//   P = exp2(S - m)     two softmax warpgroups, 64 keys each, one query row per thread; P goes back into the S columns
//   O_h += P_h V        tcgen05.mma with P from tensor memory and V MN-major, one accumulator per key half in TMEM
// The halves are independent flash-attention streams (own exponent reference, moved lazily, own row sum), merged once at
// the end, where the softmax sink joins the denominator.  All operands come by TMA (128-byte swizzle), K two stages, V two.
//
// Sizes: dim and vdim multiples of 16 up to 128, rot a multiple of 8 up to 64.  The block of the shared part is 64 wide
// whatever rot is: columns behind the row's end are filled with zeros by the copy, so what Q holds there does not matter.
#include <cuda.h>
#include <math_constants.h>

#include "../common/ptx.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace xtc {

constexpr int BM = 128, BN = 128, THREADS = 320;
constexpr int BLOCK_BYTES = 128 * 128;              // 128 rows of 64 bf16
constexpr int SMEM_Q = 0;                           // 3 column blocks
constexpr int SMEM_K = SMEM_Q + 3 * BLOCK_BYTES;    // 2 stages of 3 column blocks
constexpr int SMEM_V = SMEM_K + 6 * BLOCK_BYTES;    // 2 stages of 2 column blocks
constexpr int SMEM_BAR = SMEM_V + 4 * BLOCK_BYTES;  // 208 KB of tiles
constexpr int SMEM_XCH = SMEM_BAR + 256;
constexpr int SMEM_TOTAL = SMEM_XCH + 2048 + 1024;  // + alignment slack
constexpr float LOG2E = 1.4426950408889634f;

struct Params {
  __nv_bfloat16* out;
  const int *seq_lens, *q_start, *page_start;
  const float* sinks;
  int* err;
  int H, dim, rot, vdim, kv_rank;
  long long o_stride;
  float scale_log2;
};

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__global__ void __launch_bounds__(THREADS, 1)
attn_expanded_tc_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv,
                        const __grid_constant__ CUtensorMap tmap_lat, const Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + SMEM_BAR);
  uint64_t* q_full = bars + 0;
  uint64_t* k_full = bars + 1;    // [2]
  uint64_t* k_empty = bars + 3;   // [2]
  uint64_t* v_full = bars + 5;    // [2]
  uint64_t* v_empty = bars + 7;   // [2]
  uint64_t* s_full = bars + 9;    // [2]
  uint64_t* p_full = bars + 11;   // [2] one per key half
  uint64_t* o_full = bars + 13;   // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.z, head = blockIdx.y;
  const int q_begin = p.q_start[seq], q_end = p.q_start[seq + 1], q_len = q_end - q_begin;
  const int t0 = q_begin + (int(gridDim.x) - 1 - int(blockIdx.x)) * BM;      // the longest tiles start first
  if (t0 >= q_end) return;                                                   // whole CTA, nothing allocated yet
  const int kv_len = p.seq_lens[seq];
  const int row0 = p.page_start[seq] * 16;                                   // first expanded row of the sequence
  const int t_last = min(t0 + BM, q_end) - 1;
  const int kv_hi = max(0, min(kv_len, kv_len - q_len + (t_last - q_begin) + 1));
  const int n_tiles = (kv_hi + BN - 1) / BN;
  const int kb = (p.dim + 63) / 64, vb = (p.vdim + 63) / 64;                 // column blocks of a key / value

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 128); mbar_init(&o_full[i], 1);
    }
    fence_mbar_init();
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_kv);
    tma_prefetch_desc(&tmap_lat);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 256;

  if (warp == 0) {
    // ------------------------------ TMA producer ------------------------------
    if (lane == 0 && n_tiles > 0) {
      const int qx = head * (p.dim + p.rot), kx = head * (p.dim + p.vdim);
      mbar_arrive_expect_tx(q_full, (kb + 1) * BLOCK_BYTES);
      for (int c = 0; c < kb; ++c) tma_load_2d(smem + SMEM_Q + c * BLOCK_BYTES, &tmap_q, q_full, qx + c * 64, t0);
      tma_load_2d(smem + SMEM_Q + 2 * BLOCK_BYTES, &tmap_q, q_full, qx + p.dim, t0);
      auto load_k = [&](int j) {
        const int st = j & 1, r = row0 + j * BN;
        if (!mbar_wait(&k_empty[st], ((j >> 1) & 1) ^ 1, abort_flag, p.err, 600 + st)) return false;
        mbar_arrive_expect_tx(&k_full[st], (kb + 1) * BLOCK_BYTES);
        uint8_t* dst = smem + SMEM_K + st * 3 * BLOCK_BYTES;
        for (int c = 0; c < kb; ++c) tma_load_2d(dst + c * BLOCK_BYTES, &tmap_kv, &k_full[st], kx + c * 64, r);
        tma_load_2d(dst + 2 * BLOCK_BYTES, &tmap_lat, &k_full[st], p.kv_rank, r);
        return true;
      };
      auto load_v = [&](int j) {
        const int st = j & 1, r = row0 + j * BN;
        if (!mbar_wait(&v_empty[st], ((j >> 1) & 1) ^ 1, abort_flag, p.err, 610 + st)) return false;
        mbar_arrive_expect_tx(&v_full[st], vb * BLOCK_BYTES);
        uint8_t* dst = smem + SMEM_V + st * 2 * BLOCK_BYTES;
        for (int c = 0; c < vb; ++c) tma_load_2d(dst + c * BLOCK_BYTES, &tmap_kv, &v_full[st], kx + p.dim + c * 64, r);
        return true;
      };
      bool ok = load_k(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (j + 1 < n_tiles) ok = load_k(j + 1);
        if (ok) ok = load_v(j);
      }
    }
  } else if (warp == 1) {
    // ------------------------------ MMA issuer ------------------------------
    if (lane == 0 && n_tiles > 0) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(BM, BN, 0, 0);
      const uint32_t idesc_pv = make_idesc_bf16(BM, p.vdim, 0, 1);           // B = V is MN-major ([key][d], d contiguous)
      const uint64_t q_desc = make_smem_desc_sw128(smem_u32(smem + SMEM_Q), 16, 1024);
      const uint64_t k_desc0 = make_smem_desc_sw128(smem_u32(smem + SMEM_K), 16, 1024);
      const uint64_t v_desc0 = make_smem_desc_sw128(smem_u32(smem + SMEM_V), BLOCK_BYTES, 1024);
      const int ks_own = p.dim / 16, ks_all = ks_own + (p.rot + 15) / 16;
      auto issue_qk = [&](int j) {
        const uint64_t k_desc = smem_desc_advance(k_desc0, (j & 1) * 3 * BLOCK_BYTES);
        const uint32_t d = tmem_s + (j & 1) * BN;
        for (int k = 0; k < ks_all; ++k) {
          const int blk = k < ks_own ? k >> 2 : 2, in = k < ks_own ? k & 3 : k - ks_own;
          const uint32_t off = blk * BLOCK_BYTES + in * 32;
          umma_bf16_ss(d, smem_desc_advance(q_desc, off), smem_desc_advance(k_desc, off), idesc_qk, k != 0);
        }
      };
      bool ok = mbar_wait(q_full, 0, abort_flag, p.err, 620) && mbar_wait(&k_full[0], 0, abort_flag, p.err, 621);
      if (ok) {
        tc_fence_after();
        issue_qk(0);
        umma_commit(&s_full[0]);
        umma_commit(&k_empty[0]);
      }
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (j + 1 < n_tiles) {
          const int jn = j + 1, sn = jn & 1;
          if (!mbar_wait(&k_full[sn], (jn >> 1) & 1, abort_flag, p.err, 622)) { ok = false; break; }
          // S buffer sn: last read by P V of tile j - 1, which this thread issued before (MMAs run in issue order)
          tc_fence_after();
          issue_qk(jn);
          umma_commit(&s_full[sn]);
          umma_commit(&k_empty[sn]);
        }
        const int s = j & 1;
        if (!mbar_wait(&v_full[s], (j >> 1) & 1, abort_flag, p.err, 625)) { ok = false; break; }
        const uint64_t v_desc = smem_desc_advance(v_desc0, s * 2 * BLOCK_BYTES);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          if (!mbar_wait(&p_full[h], j & 1, abort_flag, p.err, 624 + 10 * h)) { ok = false; break; }
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < 4; ++k)                                        // 16 keys = two 8-key groups of 1024 B
            umma_bf16_ts(tmem_o + h * 128, tmem_s + s * BN + h * 64 + k * 8, smem_desc_advance(v_desc, (h * 4 + k) * 2048),
                         idesc_pv, (j > 0 || k != 0) ? 1u : 0u);
          umma_commit(&o_full[h]);
        }
        if (!ok) break;
        umma_commit(&v_empty[s]);
      }
    }
  } else {
    // ------------------------------ softmax + output (warps 2..9) ------------------------------
    const int half = (warp - 2) >> 2, qd = warp & 3, row = qd * 32 + lane;
    const uint32_t lane_off = uint32_t(qd * 32) << 16;
    const int tok = t0 + row;
    const bool row_valid = tok < q_end;
    int limit = row_valid ? min(kv_len, kv_len - q_len + (tok - q_begin) + 1) : 0;
    if (limit < 0) limit = 0;
    float m = -CUDART_INF_F, l = 0.f;           // exponent reference (log2 domain, moves lazily by steps above 8), row sum
    const uint32_t o_mine = tmem_o + half * 128 + lane_off, o_other = tmem_o + (half ^ 1) * 128 + lane_off;
    const int ocols = (p.vdim + 31) / 32;       // 32-column groups of an accumulator
    auto wait_all = [&](uint64_t* bar, uint32_t parity, int code) {
      return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, p.err, code)) != 0;
    };
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      const int b = j & 1;
      ok = ok && wait_all(&s_full[b], (j >> 1) & 1, 630);
      tc_fence_after();
      const uint32_t s_addr = tmem_s + b * BN + half * 64 + lane_off;
      const int key0 = j * BN + half * 64;
      const bool full = key0 + 64 <= limit;
      uint32_t sv[2][32];
      tmem_ld_32x32(s_addr, sv[0]);
      tmem_ld_32x32(s_addr + 32, sv[1]);
      tmem_ld_wait();
      float mx4[4] = {-CUDART_INF_F, -CUDART_INF_F, -CUDART_INF_F, -CUDART_INF_F};
      if (full) {
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 32; i += 2)
            mx4[(i >> 1) & 3] = max3(mx4[(i >> 1) & 3], __uint_as_float(sv[c][i]), __uint_as_float(sv[c][i + 1]));
      } else {
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (key0 + c * 32 + i < limit) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sv[c][i]));
      }
      const float m_tile = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2;
      float alpha = 1.f;
      if (m_tile > m + 8.f) {
        alpha = (m == -CUDART_INF_F) ? 0.f : ex2_approx(m - m_tile);
        m = m_tile;
      }
      const float m_use = (m == -CUDART_INF_F) ? 0.f : m;
      uint64_t ps2[2] = {0ull, 0ull};
      const uint64_t sc2 = pack_f32x2(p.scale_log2, p.scale_log2), nm2 = pack_f32x2(-m_use, -m_use);
      uint32_t packed[32];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float x0, x1;
          unpack_f32x2(fma_f32x2(pack_f32x2(__uint_as_float(sv[c][2 * i]), __uint_as_float(sv[c][2 * i + 1])), sc2, nm2), x0, x1);
          float p0 = ex2_approx(x0), p1 = ex2_approx(x1);
          if (!full) {
            const int k0 = key0 + c * 32 + 2 * i;
            if (k0 >= limit) p0 = 0.f;
            if (k0 + 1 >= limit) p1 = 0.f;
          }
          ps2[i & 1] = add_f32x2(ps2[i & 1], pack_f32x2(p0, p1));
          packed[c * 16 + i] = pack_bf16x2(p0, p1);
        }
      }
      float ps4[4];
      unpack_f32x2(ps2[0], ps4[0], ps4[1]);
      unpack_f32x2(ps2[1], ps4[2], ps4[3]);
      tmem_st_32x32(s_addr, packed);            // 64 keys = 32 packed columns over the head of this half's S columns
      if (j > 0) ok = ok && wait_all(&o_full[half], (j - 1) & 1, 631);
      l = l * alpha + ((ps4[0] + ps4[1]) + (ps4[2] + ps4[3]));
      if (j > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
        tc_fence_after();
        for (int c = 0; c < ocols; ++c) {
          uint32_t r[32];
          tmem_ld_32x32(o_mine + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
          tmem_st_32x32(o_mine + c * 32, r);
        }
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_full[half]);
    }
    if (n_tiles > 0) {
      ok = ok && wait_all(&o_full[half], (n_tiles - 1) & 1, 632);
      ok = ok && wait_all(&o_full[half ^ 1], (n_tiles - 1) & 1, 633);
    }
    tc_fence_after();
    float* xch = reinterpret_cast<float*>(smem + SMEM_XCH);                  // [2 halves][128 rows][m, l]
    xch[(half * 128 + row) * 2] = m;
    xch[(half * 128 + row) * 2 + 1] = l;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const float m_o = xch[((half ^ 1) * 128 + row) * 2], l_o = xch[((half ^ 1) * 128 + row) * 2 + 1];
    const float sink = p.sinks != nullptr ? p.sinks[head] * LOG2E : -CUDART_INF_F;
    const float mm = fmaxf(fmaxf(m, m_o), sink);
    const float w_mine = (m == -CUDART_INF_F) ? 0.f : exp2f(m - mm);
    const float w_other = (m_o == -CUDART_INF_F) ? 0.f : exp2f(m_o - mm);
    const float lt = l * w_mine + l_o * w_other + (sink == -CUDART_INF_F ? 0.f : exp2f(sink - mm));
    if (ok) {
      const float inv = lt > 0.f ? 1.f / lt : 0.f;
      const float c_mine = l > 0.f ? inv * w_mine : 0.f, c_other = l_o > 0.f ? inv * w_other : 0.f;
      __nv_bfloat16* dst = p.out + (long long)tok * p.o_stride + (long long)head * p.vdim;
      // the column groups alternate between the two halves
      for (int c = half; c < ocols; c += 2) {
        uint32_t r[32], r2[32];
        tmem_ld_32x32(o_mine + c * 32, r);
        tmem_ld_32x32(o_other + c * 32, r2);
        tmem_ld_wait();
        if (row_valid) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c * 32 + i >= p.vdim) continue;
            float o[8];
#pragma unroll
            for (int e = 0; e < 8; ++e)
              o[e] = (c_mine != 0.f ? __uint_as_float(r[i + e]) * c_mine : 0.f) + (c_other != 0.f ? __uint_as_float(r2[i + e]) * c_other : 0.f);
            *reinterpret_cast<uint4*>(dst + c * 32 + i) =
                make_uint4(pack_bf16x2(o[0], o[1]), pack_bf16x2(o[2], o[3]), pack_bf16x2(o[4], o[5]), pack_bf16x2(o[6], o[7]));
          }
        }
        __syncwarp();
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    for (int i = 0; i < 64; ++i) __nanosleep(20000);   // let bulk copies in flight land before smem is reused
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// a row-major matrix read in blocks of 128 rows x 64 columns
static int encode(CUtensorMap* out, const void* base, long long rows, long long cols, long long ld) {
  static EncodeTiledFn fn = nullptr;
  if (fn == nullptr) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
      return -1;
    fn = reinterpret_cast<EncodeTiledFn>(ptr);
  }
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
  cuuint32_t box[2] = {64, 128}, estr[2] = {1, 1};
  const CUresult r = fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -(int)r - 1000;
}

// 16 rows of a sequence per CTA: the cache page, or zeros behind the sequence's end (and behind the last sequence)
__global__ void __launch_bounds__(128) gather_kernel(const UbExpandArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int page = blockIdx.x, chunks = a.row / 8;
  int seq = 0;
  while (seq < a.num_seqs && page >= a.page_start[seq + 1]) ++seq;
  const uint4* src = nullptr;
  int valid = 0;
  if (seq < a.num_seqs) {
    const int pi = page - a.page_start[seq];
    valid = min(16, a.seq_lens[seq] - pi * 16);
    const int blk = pi < a.max_blocks_per_seq ? a.block_tables[(long long)seq * a.max_blocks_per_seq + pi] : -1;
    if (valid > 0 && (blk < 0 || blk >= a.num_blocks)) {
      if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, seq);
      valid = 0;
    }
    src = reinterpret_cast<const uint4*>(a.cache) + (long long)max(blk, 0) * 16 * chunks;
  }
  uint4* dst = reinterpret_cast<uint4*>(a.lat) + (long long)page * 16 * chunks;
  for (int i = threadIdx.x; i < 16 * chunks; i += 128) dst[i] = i / chunks < valid ? src[i] : make_uint4(0, 0, 0, 0);
}

}  // namespace xtc
}  // namespace ub

extern "C" int ub_latent_gather(const UbExpandArgs* a, void* stream) {
  using namespace ub;
  if (a->rows <= 0) return 0;
  if (a->rows % 16 != 0 || a->row % 8 != 0 || a->block_size != 16 || a->page_start == nullptr) return -2;
  cudaError_t e = launch_pdl(xtc::gather_kernel, dim3(a->rows / 16), dim3(128), (size_t)0, reinterpret_cast<cudaStream_t>(stream), *a);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

extern "C" int ub_attn_expanded_supported(int dim, int rot, int vdim) {
  return dim % 16 == 0 && dim >= 16 && dim <= 128 && vdim % 16 == 0 && vdim >= 16 && vdim <= 128 && rot % 8 == 0 && rot >= 8 && rot <= 64;
}

extern "C" int ub_attn_expanded(const UbExpandArgs* a, void* stream_v) {
  using namespace ub;
  using namespace ub::xtc;
  if (a->num_seqs <= 0 || a->max_q <= 0 || a->T <= 0) return 0;
  if (!ub_attn_expanded_supported(a->dim, a->rot, a->vdim) || a->num_seqs > 65535 || a->H > 65535) return -4;
  if (a->q_stride % 8 != 0 || a->o_stride % 8 != 0 || a->kv_rank % 8 != 0 || a->row != a->kv_rank + a->rot) return -3;
  if ((reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->kv) | reinterpret_cast<uintptr_t>(a->lat) |
       reinterpret_cast<uintptr_t>(a->out)) & 15)
    return -3;
  CUtensorMap tq, tkv, tl;
  const long long kv_cols = (long long)a->H * (a->dim + a->vdim);
  int rc = encode(&tq, a->q, a->T, (long long)a->H * (a->dim + a->rot), a->q_stride);
  if (rc == 0) rc = encode(&tkv, a->kv, a->rows, kv_cols, kv_cols);
  if (rc == 0) rc = encode(&tl, a->lat, a->rows, a->row, a->row);
  if (rc != 0) return rc;
  Params p;
  p.out = reinterpret_cast<__nv_bfloat16*>(a->out);
  p.seq_lens = a->seq_lens;
  p.q_start = a->q_start;
  p.page_start = a->page_start;
  p.sinks = a->sinks;
  p.err = a->err;
  p.H = a->H; p.dim = a->dim; p.rot = a->rot; p.vdim = a->vdim; p.kv_rank = a->kv_rank;
  p.o_stride = a->o_stride;
  p.scale_log2 = a->scale * LOG2E;
  static bool attr_set[UB_MAX_DEVICES] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < UB_MAX_DEVICES && !attr_set[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(attn_expanded_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_TOTAL);
    if (e != cudaSuccess) return -(int)e;
    attr_set[dev] = true;
  }
  const dim3 grid((a->max_q + BM - 1) / BM, a->H, a->num_seqs);
  cudaError_t e = launch_pdl(attn_expanded_tc_kernel, grid, dim3(THREADS), (size_t)SMEM_TOTAL, reinterpret_cast<cudaStream_t>(stream_v), tq,
                             tkv, tl, p);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
