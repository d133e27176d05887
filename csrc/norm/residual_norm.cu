// K5r: norms around a residual stream that is kept in 32 bits.
//
//  * residual_norm: x[t] += norm(f[t]) for a design that normalises the OUTPUT of its sublayers.  f is the sublayer's
//    row, or a mixture-of-experts result that is summed here instead of in a combine kernel of its own:
//    f = base + sum_k w[t, k] * y[row_slot[t, k]].  The new x is written back in fp32 and once more in the element
//    type of the matrix products, which is what the next sublayer reads.
//  * row_norm: norm(x[rows[t]]) of the stream itself (final norm with the gather of the sampled rows, or the first norm
//    of a design that normalises its inputs).
//  * embed: the stream's first value, in both forms.
//
// One CTA per token row; a row's 8-element chunks stay in registers between the passes (mean, then the mean of the
// squared deviations).  Rows are `Hp` elements apart (H rounded up to 8); the weights of the pad columns are zero, so the
// pad stays zero.
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace rnorm {

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int w = 0; w < nw; ++w) s += red[w];
  return s;
}

template <typename T, int CH>
__global__ void __launch_bounds__(256) residual_norm_kernel(const UbResidualNormArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[8];
  const int t = blockIdx.x, nch = a.Hp / 8;
  const T* base = reinterpret_cast<const T*>(a.y);
  const T* yx = reinterpret_cast<const T*>(a.yx);
  float f[CH][8];
  float sum = 0.f, sq = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
#pragma unroll
    for (int e = 0; e < 8; ++e) f[c][e] = 0.f;
    if (ch >= nch) continue;
    if (base != nullptr) load8(base + (long long)t * a.Hp + ch * 8, f[c]);
    if (yx != nullptr) {
      // four experts' rows are requested before the first is used
      for (int k0 = 0; k0 < a.K; k0 += 4) {
        float g[4][8], w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          w[j] = 0.f;
#pragma unroll
          for (int e = 0; e < 8; ++e) g[j][e] = 0.f;
          if (k0 + j < a.K) {
            const int slot = __ldg(a.row_slot + (long long)t * a.K + k0 + j);
            if (slot >= 0 && slot < a.slots) {
              w[j] = __ldg(a.topk_w + (long long)t * a.K + k0 + j);
              load8(yx + (long long)slot * a.Hp + ch * 8, g[j]);
            } else if (slot >= a.slots) {
              set_err(a.err, ERR_BOUNDS, t);
            }
          }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int e = 0; e < 8; ++e) f[c][e] = fmaf(w[j], g[j][e], f[c][e]);
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e)
      if (ch * 8 + e < a.H) { sum += f[c][e]; sq += f[c][e] * f[c][e]; }
  }
  float mean = 0.f, var;
  if (a.kind == 1) {
    mean = block_sum(sum, red) / a.H;
    float d2 = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nch) continue;
#pragma unroll
      for (int e = 0; e < 8; ++e)
        if (ch * 8 + e < a.H) { const float d = f[c][e] - mean; d2 += d * d; }
    }
    var = block_sum(d2, red) / a.H;
  } else {
    var = block_sum(sq, red) / a.H;
  }
  const float rstd = 1.f / sqrtf(var + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (ch >= nch) continue;
    float w[8], b[8], x[8];
    load8(reinterpret_cast<const T*>(a.weight) + ch * 8, w);
    if (a.bias != nullptr) {
      load8(reinterpret_cast<const T*>(a.bias) + ch * 8, b);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) b[e] = 0.f;
    }
    float* xr = a.x + (long long)t * a.Hp + ch * 8;
    load8(xr, x);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] += (f[c][e] - mean) * rstd * (a.w_off + w[e]) + b[e];
    store8(xr, x);
    store8(reinterpret_cast<T*>(a.out) + (long long)t * a.Hp + ch * 8, x);
  }
}

template <typename T, int CH>
__global__ void __launch_bounds__(256) row_norm_kernel(const UbResidualNormArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[8];
  const int t = blockIdx.x, nch = a.Hp / 8;
  int src = a.rows != nullptr ? a.rows[t] : t;
  if (src < 0 || src >= a.x_rows) {
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, t);
    src = 0;
  }
  float f[CH][8];
  float sum = 0.f, sq = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (ch >= nch) continue;
    load8(a.x + (long long)src * a.Hp + ch * 8, f[c]);
#pragma unroll
    for (int e = 0; e < 8; ++e)
      if (ch * 8 + e < a.H) { sum += f[c][e]; sq += f[c][e] * f[c][e]; }
  }
  float mean = 0.f, var;
  if (a.kind == 1) {
    mean = block_sum(sum, red) / a.H;
    float d2 = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      const int ch = threadIdx.x + c * blockDim.x;
      if (ch >= nch) continue;
#pragma unroll
      for (int e = 0; e < 8; ++e)
        if (ch * 8 + e < a.H) { const float d = f[c][e] - mean; d2 += d * d; }
    }
    var = block_sum(d2, red) / a.H;
  } else {
    var = block_sum(sq, red) / a.H;
  }
  const float rstd = 1.f / sqrtf(var + a.eps);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int ch = threadIdx.x + c * blockDim.x;
    if (ch >= nch) continue;
    float w[8], b[8];
    load8(reinterpret_cast<const T*>(a.weight) + ch * 8, w);
    if (a.bias != nullptr) {
      load8(reinterpret_cast<const T*>(a.bias) + ch * 8, b);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) b[e] = 0.f;
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) f[c][e] = (f[c][e] - mean) * rstd * (a.w_off + w[e]) + b[e];
    store8(reinterpret_cast<T*>(a.out) + (long long)t * a.Hp + ch * 8, f[c]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) embed_residual_kernel(const int* __restrict__ ids, const T* __restrict__ table,
                                                             float* __restrict__ x, T* __restrict__ out, int rows, int Hp, int V,
                                                             float scale, int* err) {
  pdl_launch_dependents();
  pdl_wait();
  const int nch = Hp / 8;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < (long long)rows * nch;
       i += (long long)gridDim.x * blockDim.x) {
    const int t = int(i / nch), ch = int(i % nch);
    int id = ids[t];
    if (id < 0 || id >= V) {
      if (ch == 0) set_err(err, ERR_BOUNDS, t);
      id = 0;
    }
    float f[8];
    load8(table + (long long)id * Hp + ch * 8, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= scale;
    store8(x + (long long)t * Hp + ch * 8, f);
    store8(out + (long long)t * Hp + ch * 8, f);
  }
}

template <typename T>
static cudaError_t launch(const UbResidualNormArgs& a, bool residual, cudaStream_t st) {
  const int nch = a.Hp / 8;
  const int threads = nch >= 256 ? 256 : (nch + 31) / 32 * 32;
  const int ch = (nch + threads - 1) / threads;
  const dim3 grid(a.T), block(threads);
#define UB_RN(C)                                                                                        \
  return residual ? launch_pdl(residual_norm_kernel<T, C>, grid, block, (size_t)0, st, a)               \
                  : launch_pdl(row_norm_kernel<T, C>, grid, block, (size_t)0, st, a)
  if (ch <= 1) { UB_RN(1); }
  if (ch <= 2) { UB_RN(2); }
  if (ch <= 4) { UB_RN(4); }
  UB_RN(8);
#undef UB_RN
}

static int run(const UbResidualNormArgs* a, bool residual, void* stream) {
  if (a->T <= 0) return 0;
  if (a->H <= 0 || a->Hp % 8 != 0 || a->Hp < a->H || a->Hp > 16384) return -2;
  if (a->x == nullptr || a->out == nullptr || a->weight == nullptr) return -3;
  if (a->yx != nullptr && (a->row_slot == nullptr || a->topk_w == nullptr || a->K <= 0)) return -4;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = a->f32 ? launch<float>(*a, residual, st) : launch<__nv_bfloat16>(*a, residual, st);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

}  // namespace rnorm
}  // namespace ub

extern "C" int ub_residual_norm(const UbResidualNormArgs* a, void* stream) {
  if (a->y == nullptr && a->yx == nullptr) return -5;
  return ub::rnorm::run(a, true, stream);
}

extern "C" int ub_row_norm(const UbResidualNormArgs* a, void* stream) { return ub::rnorm::run(a, false, stream); }

extern "C" int ub_embed_residual(const int* ids, const void* table, float* x, void* out, int rows, int Hp, int V, float scale,
                                 int f32, int* err, void* stream) {
  using namespace ub;
  if (rows <= 0) return 0;
  if (Hp % 8 != 0 || V <= 0) return -2;
  const long long work = (long long)rows * (Hp / 8);
  const int grid = (int)(work + 255 < 148LL * 8 * 256 ? (work + 255) / 256 : 148 * 8);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = f32 ? launch_pdl(rnorm::embed_residual_kernel<float>, dim3(grid), dim3(256), (size_t)0, st, ids,
                                   reinterpret_cast<const float*>(table), x, reinterpret_cast<float*>(out), rows, Hp, V, scale, err)
                      : launch_pdl(rnorm::embed_residual_kernel<__nv_bfloat16>, dim3(grid), dim3(256), (size_t)0, st, ids,
                                   reinterpret_cast<const __nv_bfloat16*>(table), x, reinterpret_cast<__nv_bfloat16*>(out), rows, Hp,
                                   V, scale, err);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
