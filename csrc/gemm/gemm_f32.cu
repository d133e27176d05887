// K1f: the GEMM in true 32-bit arithmetic,  out[M, N] = epilogue(x[M, K] @ w[N, K]^T)  with fp32 operands on the FMA
// pipe (no reduced-precision tensor mode).  It serves models that are run in 32-bit for accuracy; speed comes second.
//
// Same argument block and epilogue as ub_gemm_tn: scale, bias, activation, gated form (act(gate) * up), residual, and the
// grouped (mixture-of-experts) mode driven by the device-built tile table.  x, w, bias, residual and out are all fp32.
// One CTA of 256 threads per 64 x 64 output tile, K in steps of 16 through shared memory, 4 x 4 outputs per thread; a
// tile's sum runs over k in order, so a row's bits do not depend on the other rows of the launch.
#include "../common/ptx.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace gf32 {

constexpr int BM = 64, BN = 64, BKF = 16;

__device__ __forceinline__ float act_apply(float v, const UbGemmArgs& a) {
  switch (a.act) {
    case UB_ACT_SILU: return v / (1.f + expf(-v));
    case UB_ACT_GELU: return 0.5f * v * (1.f + erff(v * 0.70710678118654752f));
    case UB_ACT_GELU_TANH: return 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    case UB_ACT_RELU: return fmaxf(v, 0.f);
    case UB_ACT_RELU2: { const float r = fmaxf(v, 0.f); return r * r; }
    case UB_ACT_QUICK_GELU: return v / (1.f + expf(-1.702f * v));
    case UB_ACT_SIGMOID: return 1.f / (1.f + expf(-v));
    case UB_ACT_TANH: return tanhf(v);
    case UB_ACT_SOFTPLUS: return v > 20.f ? v : log1pf(expf(v));
    case UB_ACT_XIELU: return fmaf(0.5f, v, v > 0.f ? a.act_a * v * v : a.act_b * (expm1f(v) - v));
    default: return v;
  }
}

template <bool DUAL>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const UbGemmArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int NT = DUAL ? 2 : 1;
  __shared__ float xs[BKF][BM + 4];
  __shared__ float ws[NT][BKF][BN + 4];
  const float* x = reinterpret_cast<const float*>(a.x);
  const float* w = reinterpret_cast<const float*>(a.w);
  const int n0 = blockIdx.x * BN;
  int m0, m_end;
  long long wrow0 = 0;
  if (a.grp_tiles != nullptr) {
    // token tile y / subs of the table, 64-row slice y % subs of it
    const int subs = (a.tile_tokens + BM - 1) / BM;
    const int4 t = reinterpret_cast<const int4*>(a.grp_tiles)[blockIdx.y / subs];
    if (t.x < 0) return;
    m0 = t.y + (blockIdx.y % subs) * BM;
    m_end = min(t.z, t.y + a.tile_tokens);
    wrow0 = (long long)t.x * a.grp_w_rows;
    if (m0 < 0 || m_end > a.M || wrow0 + a.grp_w_rows > a.w_rows_total) {
      if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, blockIdx.y);
      return;
    }
  } else {
    m0 = blockIdx.y * BM;
    m_end = a.M;
  }
  if (m0 >= m_end) return;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;     // 4 columns tx * 4.., 4 rows ty * 4..
  float acc[NT][4][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[n][i][j] = 0.f;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // loader: row lr, four k
  for (int k0 = 0; k0 < a.K; k0 += BKF) {
    const int k = k0 + lk;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int kk = k + j;
      xs[lk + j][lr] = (m0 + lr < m_end && kk < a.K) ? x[(long long)(m0 + lr) * a.ldx + kk] : 0.f;
#pragma unroll
      for (int n = 0; n < NT; ++n)
        ws[n][lk + j][lr] = (n0 + lr < a.N && kk < a.K) ? w[(wrow0 + n0 + lr + (long long)n * a.up_row_off) * a.ldw + kk] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < BKF; ++kk) {
      float xv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) xv[i] = xs[kk][ty * 4 + i];
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float wv = ws[n][kk][tx * 4 + j];
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[n][i][j] = fmaf(xv[i], wv, acc[n][i][j]);
        }
    }
    __syncthreads();
  }
  const float sc = a.out_scale != 0.f ? a.out_scale : 1.f;
  float* out = reinterpret_cast<float*>(a.out);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= m_end) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= a.N) continue;
      float v = acc[0][i][j] * sc;
      if (DUAL) {
        v = act_apply(v, a) * (acc[NT - 1][i][j] * sc);
      } else {
        if (a.bias != nullptr) v += reinterpret_cast<const float*>(a.bias)[n];
        v = act_apply(v, a);
      }
      if (a.residual != nullptr) v += reinterpret_cast<const float*>(a.residual)[(long long)m * a.ldr + n];
      out[(long long)m * a.ldo + n] = v;
    }
  }
}

}  // namespace gf32
}  // namespace ub

extern "C" int ub_gemm_f32(const UbGemmArgs* a, void* stream) {
  using namespace ub::gf32;
  if (a->M <= 0 || a->N <= 0 || a->K <= 0) return 0;
  if (a->rs_world > 0 || a->ag_world > 0) return -6;       // no fused collectives in 32-bit
  int ny = (a->M + BM - 1) / BM;
  if (a->grp_tiles != nullptr) {
    if (a->tile_tokens <= 0 || a->grp_max_tiles <= 0 || a->grp_w_rows <= 0 || a->bias != nullptr) return -6;
    ny = a->grp_max_tiles * ((a->tile_tokens + BM - 1) / BM);
  }
  if (ny > 65535) return -7;
  const dim3 grid((a->N + BN - 1) / BN, ny);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = a->dual ? ub::launch_pdl(gemm_f32_kernel<true>, grid, dim3(256), (size_t)0, st, *a)
                          : ub::launch_pdl(gemm_f32_kernel<false>, grid, dim3(256), (size_t)0, st, *a);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
