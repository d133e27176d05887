// K1h: one small matrix per attention head,  out[t, h, :] = x[t, h, :] @ w[h]^T,  w[h] stored [N, K]: the key and value
// matrices of multi-head latent attention, taken to the query and output side of the attention.  Rows of x and out may lie
// anywhere (token and head strides), so the fused projections are read and written in place.
//
// bf16: warp MMAs over 64-column tiles, 16 or 64 tokens per CTA, K in steps of 64 through a three-stage cp.async ring; the
// work is a read of the matrices at decode sizes.  fp32: FMA, one output per thread, for models run in 32-bit.
#include "../common/ptx.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace hgemm {

constexpr int BN = 64, BKH = 64, STAGES = 3;

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool pred) {
  const int sz = pred ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 128-byte rows, 16-byte chunks XOR-swizzled by the row
__device__ __forceinline__ uint32_t off(int row, int chunk) { return (uint32_t)(row * 128 + ((chunk ^ (row & 7)) << 4)); }

// WIDE: 64 tokens per CTA, a warp has 16 of them and all 64 columns; else 16 tokens, a warp has 16 columns.
template <bool WIDE>
__global__ void __launch_bounds__(128) gemm_heads_kernel(const UbHeadGemmArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int BM = WIDE ? 64 : 16, NT = WIDE ? 8 : 2, STAGE = (BM + BN) * 128;
  __shared__ __align__(128) uint8_t sm[STAGES * STAGE];
  const int n0 = blockIdx.x * BN, h = blockIdx.y, m0 = blockIdx.z * BM, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.x) + (long long)h * a.x_head;
  const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.w) + (long long)h * a.N * a.K;
  const int nk = (a.K + BKH - 1) / BKH;
  auto issue = [&](int kb) {
    if (kb < nk) {
      const uint32_t st = smem_u32(sm + (kb % STAGES) * STAGE);
      for (int i = threadIdx.x; i < (BM + BN) * 8; i += 128) {
        const int r = i >> 3, c = i & 7, k = kb * BKH + c * 8;
        const bool isx = r < BM;
        const int row = isx ? m0 + r : n0 + r - BM;
        const bool ok = k < a.K && row < (isx ? a.M : a.N);
        const __nv_bfloat16* src = isx ? x + (ok ? row * a.x_stride + k : 0) : w + (ok ? (long long)row * a.K + k : 0);
        cp_async16(st + (isx ? off(r, c) : BM * 128 + off(r - BM, c)), src, ok);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  for (int s = 0; s < STAGES - 1; ++s) issue(s);
  const int mr = WIDE ? warp * 16 : 0, nc = WIDE ? 0 : warp * 16;
  for (int kb = 0; kb < nk; ++kb) {
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    __syncthreads();
    issue(kb + STAGES - 1);
    const uint32_t xs = smem_u32(sm + (kb % STAGES) * STAGE), ws = xs + BM * 128;
#pragma unroll
    for (int ks = 0; ks < BKH / 16; ++ks) {
      uint32_t af[4];
      ldsm_x4(xs + off(mr + (lane & 7) + ((lane >> 3) & 1) * 8, ks * 2 + (lane >> 4)), af[0], af[1], af[2], af[3]);
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) {
        const int mi = lane >> 3;
        uint32_t b0, b1, b2, b3;
        ldsm_x4(ws + off(nc + j * 16 + (mi >> 1) * 8 + (lane & 7), ks * 2 + (mi & 1)), b0, b1, b2, b3);
        mma_bf16(acc[j * 2], af, b0, b1);
        mma_bf16(acc[j * 2 + 1], af, b2, b3);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (long long)h * a.out_head;
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int n = n0 + nc + j * 8 + (lane & 3) * 2;
    if (n >= a.N) continue;                                 // N is even
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int m = m0 + mr + (lane >> 2) + half * 8;
      if (m < a.M) *reinterpret_cast<uint32_t*>(out + m * a.out_stride + n) = pack_bf16x2(acc[j][half * 2], acc[j][half * 2 + 1]);
    }
  }
}

__global__ void __launch_bounds__(128) gemm_heads_f32_kernel(const UbHeadGemmArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int n = blockIdx.x * 128 + threadIdx.x, h = blockIdx.y, m = blockIdx.z;
  if (n >= a.N) return;
  const float* x = reinterpret_cast<const float*>(a.x) + m * a.x_stride + (long long)h * a.x_head;
  const float* w = reinterpret_cast<const float*>(a.w) + ((long long)h * a.N + n) * a.K;
  float s = 0.f;
  for (int k = 0; k < a.K; k += 4) {
    const float4 p = *reinterpret_cast<const float4*>(x + k), q = *reinterpret_cast<const float4*>(w + k);
    s = fmaf(p.x, q.x, s);
    s = fmaf(p.y, q.y, s);
    s = fmaf(p.z, q.z, s);
    s = fmaf(p.w, q.w, s);
  }
  reinterpret_cast<float*>(a.out)[m * a.out_stride + (long long)h * a.out_head + n] = s;
}

}  // namespace hgemm
}  // namespace ub

extern "C" int ub_gemm_heads(const UbHeadGemmArgs* a, void* stream) {
  using namespace ub;
  if (a->M <= 0 || a->N <= 0 || a->K <= 0 || a->H <= 0) return 0;
  if (a->N % 8 != 0 || a->K % 8 != 0 || (a->x_stride | a->x_head | a->out_stride | a->out_head) % 8 != 0) return -2;
  if ((reinterpret_cast<uintptr_t>(a->x) | reinterpret_cast<uintptr_t>(a->w) | reinterpret_cast<uintptr_t>(a->out)) & 15) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const bool wide = a->M > 32;
  const int bm = a->f32 ? 1 : wide ? 64 : 16, gz = (a->M + bm - 1) / bm;
  if (gz > 65535 || a->H > 65535) return -4;
  cudaError_t e;
  if (a->f32) e = launch_pdl(hgemm::gemm_heads_f32_kernel, dim3((a->N + 127) / 128, a->H, gz), dim3(128), (size_t)0, st, *a);
  else if (wide) e = launch_pdl(hgemm::gemm_heads_kernel<true>, dim3((a->N + 63) / 64, a->H, gz), dim3(128), (size_t)0, st, *a);
  else e = launch_pdl(hgemm::gemm_heads_kernel<false>, dim3((a->N + 63) / 64, a->H, gz), dim3(128), (size_t)0, st, *a);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
