// K4m: attention of many query heads over one cached latent row per token (multi-head latent attention with the key and
// value matrices taken to the query and output side).  A cache row is [latent (Dv) | rotated key part (D - Dv)]: the whole
// row is the key of every head, its first Dv elements are the value.  Paged like the other caches, one row per position.
//
// A CTA takes 16 * MT rows -- a row is (query token, head) -- of one sequence and one range of its keys; with one query per
// sequence these are the heads, so a tile of cache rows fetched once serves all of them, as key and as value.
//
// Four warps fetch: tiles of 64 positions by cp.async into a ring of two or three stages whose rows are padded by 16 bytes
// (ldmatrix without bank conflicts), the block table read once, ahead.  The fill of a tile is bound by the path from L2 into
// shared memory and takes about as long as the tile's arithmetic, so it has warps of its own.  Eight warps compute: the
// scores in four groups of 16 positions times two halves of the row, the online softmax in fp32 on the summed halves, then
// the value columns among them.  Causal by position; softmax sinks join in the epilogue, or for split ranges in the merge,
// once.
#include <math_constants.h>

#include "../common/ptx.cuh"
#include "../include/unillm_b200.h"

extern "C" int ub_attn_split_merge(const UbAttnArgs* a, void* stream);

namespace ub {
namespace latent {

constexpr int KT = 64, THREADS = 256, LOADERS = 128;   // computing and fetching threads
constexpr float LOG2E = 1.4426950408889634f, LN2 = 0.6931471805599453f;

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool pred) {
  const int sz = pred ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(sz));
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

constexpr int S_PITCH = KT + 4;            // floats
constexpr int P_PITCH = KT * 2 + 16;       // bytes

constexpr int BT_MAX = 512;                // block-table entries held in shared memory

struct Layout {
  int pitch, q, kv, s, p, row, bt, total;  // byte offsets
  __host__ __device__ Layout(int D, int mt, int stages) {
    pitch = (D + 15) / 16 * 32 + 16;
    q = 0;
    kv = 16 * mt * pitch;
    s = kv + stages * KT * pitch;
    p = s + 2 * 16 * mt * S_PITCH * 4;
    row = p + 16 * mt * P_PITCH;
    bt = row + 16 * mt * 3 * 4;            // behind alpha, max, sum per row
    total = bt + BT_MAX * 4;
  }
};

// Narrow rows: two CTAs on an SM, so that one computes while the other one's warps meet at a barrier.
template <int MT, int VP>
struct Residency { static constexpr int CTAS = MT == 1 && VP <= 2 ? 2 : 0; };     // 0: left to the compiler

template <int MT, int VP>
__global__ void __launch_bounds__(THREADS + LOADERS, (Residency<MT, VP>::CTAS)) attn_latent_kernel(const UbAttnArgs a, const int stages) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int ROWS = 16 * MT, TPR = THREADS / ROWS, CPT = KT / TPR;
  extern __shared__ __align__(128) uint8_t sm[];
  __shared__ uint64_t full[3], empty[3];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  const Layout L(a.D, MT, stages);
  const int D = a.D, Dv = a.Dv, nch = D / 8, nck = (D + 15) / 16 * 2;
  float* s_sm = reinterpret_cast<float*>(sm + L.s);
  float* alpha_sm = reinterpret_cast<float*>(sm + L.row);
  float* m_sm = alpha_sm + ROWS;
  float* l_sm = m_sm + ROWS;
  const int seq = blockIdx.z, split = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qs = a.q_start != nullptr ? a.q_start[seq] : seq;
  const int q_len = a.q_start != nullptr ? a.q_start[seq + 1] - qs : 1;
  const int rows_total = q_len * a.Hq, row0 = blockIdx.x * ROWS;
  if (row0 >= rows_total) return;
  const int kv_len = a.seq_lens[seq];
  const int q0 = kv_len - q_len;                          // position of the portion's first query
  const int visible = min(kv_len, q0 + (min(row0 + ROWS, rows_total) - 1) / a.Hq + 1);
  int per = (visible + a.splits - 1) / a.splits;
  per = (per + a.block_size - 1) / a.block_size * a.block_size;
  const int kv_lo = split * per, kv_hi = min(visible, kv_lo + per);
  const int n_tiles = kv_hi > kv_lo ? (kv_hi - kv_lo + KT - 1) / KT : 0;
  const int* bt = a.block_tables + (long long)seq * a.max_blocks_per_seq;
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(a.k_cache);
  const __nv_bfloat16* qg = reinterpret_cast<const __nv_bfloat16*>(a.q);
  const uint32_t q_u = smem_u32(sm + L.q), kv_u = smem_u32(sm + L.kv), p_u = smem_u32(sm + L.p);

  for (int i = threadIdx.x; i < ROWS * nck; i += THREADS + LOADERS) {
    const int r = i / nck, c = i % nck, row = row0 + r;
    const bool ok = row < rows_total && c < nch;
    const int tok = ok ? row / a.Hq : 0, h = ok ? row % a.Hq : 0;
    cp_async16(q_u + r * L.pitch + c * 16, qg + (ok ? (long long)(qs + tok) * a.q_stride + (long long)h * D + c * 8 : 0), ok);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  int* bt_sm = reinterpret_cast<int*>(sm + L.bt);
  const int page0 = kv_lo / a.block_size, pages = n_tiles > 0 ? (kv_hi - 1) / a.block_size - page0 + 1 : 0;
  for (int i = threadIdx.x; i < min(pages, BT_MAX); i += THREADS + LOADERS) bt_sm[i] = page0 + i < a.max_blocks_per_seq ? bt[page0 + i] : -1;
  if (threadIdx.x == 0) {
    abort_word = 0;
    for (int i = 0; i < stages; ++i) {
      mbar_init(&full[i], LOADERS);
      mbar_init(&empty[i], THREADS);
    }
    fence_mbar_init();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();

  // A wait that gives up has set the error word and the abort flag; the later ones then return at once, and every thread
  // goes on to its end in step with the others.
  if (warp >= THREADS / 32) {
    // ------------------------------ fetching warps ------------------------------
    const int bs_shift = 31 - __clz(a.block_size);         // a power of two (host check)
    const int w = warp - THREADS / 32;
    constexpr int RPW = KT / (LOADERS / 32), CPR = 3;      // rows per warp, chunks per lane and row (D <= 640, with padding)
    int st = 0, ph = 1;
    for (int t = 0; t < n_tiles; ++t) {
      const int base = kv_lo + t * KT;
      // lane r looks row r's page up; nothing but the shuffled offset then stands between the copies
      long long src = -1;
      if (lane < RPW) {
        const int pos = base + w * RPW + lane;
        if (pos < kv_hi) {
          const int bi = pos >> bs_shift;
          const int blk = bi - page0 < BT_MAX ? bt_sm[bi - page0] : (bi < a.max_blocks_per_seq ? bt[bi] : -1);
          if (blk < 0 || blk >= a.num_blocks) set_err(a.err, ERR_BOUNDS, seq);
          else src = (((long long)blk << bs_shift) + (pos & (a.block_size - 1))) * D;
        }
      }
      const bool ok = __all_sync(0xffffffffu, mbar_wait(&empty[st], ph, abort_flag, a.err, 710 + st));
      if (ok) {
        const uint32_t dst = kv_u + (st * KT + w * RPW) * L.pitch + lane * 16;
#pragma unroll
        for (int r = 0; r < RPW; ++r) {
          const long long off = __shfl_sync(0xffffffffu, src, r);
          const __nv_bfloat16* g = cache + (off >= 0 ? off : 0) + lane * 8;
#pragma unroll
          for (int k = 0; k < CPR; ++k) {
            const int c = lane + 32 * k;
            const bool in = off >= 0 && c < nch;
            if (c < nck) cp_async16(dst + r * L.pitch + k * 512, in ? g + k * 256 : cache, in);
          }
        }
      }
      asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];" ::"r"(smem_u32(&full[st])) : "memory");
      if (++st == stages) { st = 0; ph ^= 1; }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    return;
  }
  // ------------------------------ computing warps ------------------------------
  auto sync = [] { asm volatile("bar.sync 1, 256;" ::: "memory"); };

  float o[MT][VP * 2][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int j = 0; j < VP * 2; ++j) o[mt][j][0] = o[mt][j][1] = o[mt][j][2] = o[mt][j][3] = 0.f;
  const int my_row = threadIdx.x / TPR, part = threadIdx.x % TPR;       // softmax: TPR neighbouring lanes per row
  const int my_pos = q0 + min(row0 + my_row, rows_total - 1) / a.Hq;
  float m_run = -CUDART_INF_F, l_run = 0.f;
  const float sc = a.scale * LOG2E;
  const int tg = warp & 3, kh = warp >> 2, nks = nck / 2, half = (nks + 1) / 2;
  const int ks0 = kh * half, ks1 = min(nks, ks0 + half);

  int st = 0, ph = 0;
  for (int t = 0; t < n_tiles; ++t) {
    mbar_wait(&full[st], ph, abort_flag, a.err, 700 + st);
    const uint32_t kb = kv_u + st * KT * L.pitch;
    {
      float s[MT][2][4], s2[MT][2][4];                     // even and odd steps: two chains of dependent MMAs
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[mt][j][e] = s2[mt][j][e] = 0.f;
      const int mi = lane >> 3;
      const uint32_t baddr = kb + (tg * 16 + (mi >> 1) * 8 + (lane & 7)) * L.pitch + (mi & 1) * 16;
      const uint32_t aaddr = q_u + ((lane & 7) + ((lane >> 3) & 1) * 8) * L.pitch + (lane >> 4) * 16;
      auto step = [&](int ks, float (&acc)[MT][2][4]) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4(baddr + ks * 32, b0, b1, b2, b3);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          uint32_t af[4];
          ldsm_x4(aaddr + mt * 16 * L.pitch + ks * 32, af[0], af[1], af[2], af[3]);
          mma_bf16(acc[mt][0], af, b0, b1);
          mma_bf16(acc[mt][1], af, b2, b3);
        }
      };
      int ks = ks0;
#pragma unroll 3
      for (; ks + 1 < ks1; ks += 2) {
        step(ks, s);
        step(ks + 1, s2);
      }
      if (ks < ks1) step(ks, s);
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          float* d = s_sm + (kh * ROWS + mt * 16 + (lane >> 2)) * S_PITCH + tg * 16 + j * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(d) = make_float2(s[mt][j][0] + s2[mt][j][0], s[mt][j][1] + s2[mt][j][1]);
          *reinterpret_cast<float2*>(d + 8 * S_PITCH) = make_float2(s[mt][j][2] + s2[mt][j][2], s[mt][j][3] + s2[mt][j][3]);
        }
    }
    sync();
    {
      const float* s0 = s_sm + my_row * S_PITCH;
      const float* s1 = s0 + ROWS * S_PITCH;
      const int base = kv_lo + t * KT;
      float v[CPT], mx = m_run;
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        const int col = part + TPR * c, pos = base + col;
        v[c] = pos < kv_hi && pos <= my_pos ? (s0[col] + s1[col]) * sc : -CUDART_INF_F;
        mx = fmaxf(mx, v[c]);
      }
#pragma unroll
      for (int w = TPR / 2; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      const float al = mx == -CUDART_INF_F ? 1.f : exp2f(m_run - mx);
      float sum = 0.f;
      __nv_bfloat16* p = reinterpret_cast<__nv_bfloat16*>(sm + L.p + my_row * P_PITCH);
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        const float e = v[c] == -CUDART_INF_F ? 0.f : exp2f(v[c] - mx);
        sum += e;
        p[part + TPR * c] = __float2bfloat16(e);
      }
#pragma unroll
      for (int w = TPR / 2; w > 0; w >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
      m_run = mx;
      l_run = l_run * al + sum;
      if (part == 0) alpha_sm[my_row] = al;
    }
    sync();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float al_a = alpha_sm[mt * 16 + (lane >> 2)], al_b = alpha_sm[mt * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int j = 0; j < VP * 2; ++j) { o[mt][j][0] *= al_a; o[mt][j][1] *= al_a; o[mt][j][2] *= al_b; o[mt][j][3] *= al_b; }
    }
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        ldsm_x4(p_u + (mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * P_PITCH + (kk * 2 + (lane >> 4)) * 16, pf[mt][0], pf[mt][1],
                pf[mt][2], pf[mt][3]);
#pragma unroll
      for (int i = 0; i < VP; ++i) {
        const int dp = warp * VP + i;
        if (dp * 16 >= Dv) continue;                       // warp-uniform
        const int mi = lane >> 3;
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(kb + (kk * 16 + (mi & 1) * 8 + (lane & 7)) * L.pitch + (dp * 2 + (mi >> 1)) * 16, b0, b1, b2, b3);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(o[mt][i * 2], pf[mt], b0, b1);
          mma_bf16(o[mt][i * 2 + 1], pf[mt], b2, b3);
        }
      }
    }
    mbar_arrive(&empty[st]);
    if (++st == stages) { st = 0; ph ^= 1; }
  }
  if (part == 0) {
    m_sm[my_row] = m_run;
    l_sm[my_row] = l_run;
  }
  sync();
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int r = mt * 16 + (lane >> 2) + hf * 8, row = row0 + r;
      if (row >= rows_total) continue;
      const int tok = row / a.Hq, h = row % a.Hq;
      float m = m_sm[r], l = l_sm[r], f = 1.f;
      if (a.sinks != nullptr && a.splits == 1) {
        const float sk = a.sinks[h] * LOG2E, m2 = fmaxf(m, sk);
        f = m == -CUDART_INF_F ? 0.f : exp2f(m - m2);
        l = l * f + exp2f(sk - m2);
        m = m2;
      }
      const float inv = l > 0.f ? f / l : 0.f;
      const float lse = l > 0.f ? (m + log2f(l)) * LN2 : -CUDART_INF_F;
      float* sp = a.scratch + (((long long)(qs + tok) * a.Hq + h) * a.splits + split) * (Dv + 2);
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(a.out) + (long long)(qs + tok) * a.o_stride + (long long)h * Dv;
#pragma unroll
      for (int j = 0; j < VP * 2; ++j) {
        const int d = (warp * VP * 2 + j) * 8 + (lane & 3) * 2;
        if (d >= Dv) continue;
        const float v0 = o[mt][j][hf * 2] * inv, v1 = o[mt][j][hf * 2 + 1] * inv;
        if (a.splits == 1) {
          *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16x2(v0, v1);
        } else {
          sp[d] = v0;
          sp[d + 1] = v1;
        }
      }
      if (warp == 0 && (lane & 3) == 0) {
        if (a.splits > 1) sp[Dv] = lse;
        else if (a.lse != nullptr) a.lse[(long long)(qs + tok) * a.Hq + h] = lse;
      }
    }
}

template <int MT, int VP>
static int launch(const UbAttnArgs& a, int mq, cudaStream_t st) {
  // two stages where that lets a second CTA onto the SM, else as many as fit
  const bool pair = Residency<MT, VP>::CTAS == 2 && Layout(a.D, MT, 2).total <= 112 * 1024;
  const int stages = !pair && Layout(a.D, MT, 3).total <= 225 * 1024 ? 3 : 2;
  const Layout L(a.D, MT, stages);
  static int allowed[UB_MAX_DEVICES] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < UB_MAX_DEVICES && allowed[dev] < L.total) {
    const cudaError_t e = cudaFuncSetAttribute(attn_latent_kernel<MT, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total);
    if (e != cudaSuccess) return -(int)e;
    allowed[dev] = L.total;
  }
  const dim3 grid((mq * a.Hq + 16 * MT - 1) / (16 * MT), a.splits, a.num_seqs);
  cudaError_t e = launch_pdl(attn_latent_kernel<MT, VP>, grid, dim3(THREADS + LOADERS), (size_t)L.total, st, a, stages);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

template <int MT>
static int launch_sized(const UbAttnArgs& a, int mq, cudaStream_t st) {
  if (a.Dv <= 128) return launch<MT, 1>(a, mq, st);
  if (a.Dv <= 256) return launch<MT, 2>(a, mq, st);
  return launch<MT, 4>(a, mq, st);
}

}  // namespace latent
}  // namespace ub

// Prompt portions (q_start) or one query per sequence; splits > 1 only for the latter.
extern "C" int ub_attn_latent(const UbAttnArgs* a, void* stream) {
  using namespace ub;
  if (a->num_seqs <= 0) return 0;
  if (a->q_start != nullptr && a->max_q_len <= 0) return 0;
  const int mq = a->q_start != nullptr ? a->max_q_len : 1;
  if (a->D % 8 != 0 || a->Dv % 8 != 0 || a->Dv <= 0 || a->Dv >= a->D || a->Dv > 512 || a->D > 640 || a->Hq <= 0) return -2;
  if (a->q_stride % 8 != 0 || a->o_stride % 2 != 0 || a->splits < 1 || a->num_seqs > 65535) return -3;
  if (a->splits > 1 && (a->q_start != nullptr || a->scratch == nullptr)) return -3;
  if (a->block_size <= 0 || (a->block_size & (a->block_size - 1))) return -5;
  if (a->window > 0 || a->alibi_slopes != nullptr || a->merge_o != nullptr || a->kv_start > 0) return -7;
  if ((reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->k_cache) | reinterpret_cast<uintptr_t>(a->out)) & 15) return -4;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const int rc = (long long)mq * a->Hq <= 16 ? latent::launch_sized<1>(*a, mq, st) : latent::launch_sized<2>(*a, mq, st);
  if (rc != 0 || a->splits == 1) return rc;
  return ub_attn_split_merge(a, stream);
}
