// K6m: between the projections of multi-head latent attention.
//
//  * latent_rows: of a token's down-projections [q latent | kv latent | rotated key part], the q latent is RMS-normed into
//    the input of the query projection, the kv latent is RMS-normed and, with the rotated key part behind it, becomes the
//    token's cache row.
//  * latent_rotate: the rotated part of every head's query, in place.
//
// Pairs are adjacent elements; frequencies come from the host, cosine and sine carry a common gain.  Segments are padded to
// multiples of 8 elements (zero weights keep the pads zero).  Norms and angles are fp32.
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {
namespace latrow {

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int nw = blockDim.x >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int w = 0; w < nw; ++w) s += red[w];
  return s;
}

// eight elements (pairs first / 2 ..) turned by pos * freq
__device__ __forceinline__ void rotate8(float (&v)[8], int first, int dims, float pos, const float* freq, float gain) {
#pragma unroll
  for (int e = 0; e < 8; e += 2) {
    if (first + e >= dims) break;
    float s, c;
    sincosf(pos * freq[(first + e) / 2], &s, &c);
    s *= gain;
    c *= gain;
    const float x0 = v[e], x1 = v[e + 1];
    v[e] = x0 * c - x1 * s;
    v[e + 1] = x1 * c + x0 * s;
  }
}

template <typename T>
__device__ __forceinline__ void norm_segment(const T* src, const T* w, T* dst, int n, int real, float eps, float* red) {
  float sq = 0.f;
  for (int c = threadIdx.x; c < n / 8; c += blockDim.x) {
    float v[8];
    load8(src + c * 8, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) sq += v[e] * v[e];
  }
  const float r = 1.f / sqrtf(block_sum(sq, red) / real + eps);
  if (dst == nullptr) return;
  for (int c = threadIdx.x; c < n / 8; c += blockDim.x) {
    float v[8], g[8];
    load8(src + c * 8, v);
    load8(w + c * 8, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = v[e] * r * g[e];
    store8(dst + c * 8, v);
  }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_rows_kernel(const UbLatentArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[4];
  const int t = blockIdx.x;
  const T* src = reinterpret_cast<const T*>(a.down) + (long long)t * (a.q_rank + a.kv_rank + a.rot);
  norm_segment<T>(src, reinterpret_cast<const T*>(a.q_norm_w), reinterpret_cast<T*>(a.q_latent) + (long long)t * a.q_rank, a.q_rank,
                  a.q_real, a.eps, red);
  long long slot = a.slot_mapping[t];
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, t);
    slot = -1;
  }
  T* row = slot >= 0 ? reinterpret_cast<T*>(a.cache) + slot * (a.kv_rank + a.rot) : nullptr;
  norm_segment<T>(src + a.q_rank, reinterpret_cast<const T*>(a.kv_norm_w), row, a.kv_rank, a.kv_real, a.eps, red);
  if (row == nullptr) return;
  const float pos = (float)a.positions[t];
  for (int c = threadIdx.x; c < a.rot / 8; c += blockDim.x) {
    float v[8];
    load8(src + a.q_rank + a.kv_rank + c * 8, v);
    rotate8(v, c * 8, a.rot_dims, pos, a.inv_freq, a.gain);
    store8(row + a.kv_rank + c * 8, v);
  }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_rotate_kernel(const UbLatentArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, rc = a.rot / 8;
  const float pos = (float)a.positions[t];
  const T* src = reinterpret_cast<const T*>(a.q) + (long long)t * a.q_stride + a.q_off;
  T* dst = reinterpret_cast<T*>(a.q_out) + (long long)t * a.qo_stride + a.qo_off;
  for (int i = threadIdx.x; i < a.H * rc; i += blockDim.x) {
    const int h = i / rc, c = (i % rc) * 8;
    float v[8];
    load8(src + (long long)h * a.q_head + c, v);
    rotate8(v, c, a.rot_dims, pos, a.inv_freq, a.gain);
    store8(dst + (long long)h * a.qo_head + c, v);
  }
}

static bool bad(const UbLatentArgs& a) { return a.rot % 8 != 0 || a.rot_dims > a.rot || a.rot_dims % 2 != 0 || a.inv_freq == nullptr; }

}  // namespace latrow
}  // namespace ub

extern "C" int ub_latent_rows(const UbLatentArgs* a, void* stream) {
  using namespace ub;
  if (a->T <= 0) return 0;
  if (latrow::bad(*a) || a->q_rank % 8 != 0 || a->kv_rank % 8 != 0 || a->q_real <= 0 || a->kv_real <= 0) return -2;
  if (a->down == nullptr || a->q_latent == nullptr || a->cache == nullptr || a->slot_mapping == nullptr) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = a->f32 ? launch_pdl(latrow::latent_rows_kernel<float>, dim3(a->T), dim3(128), (size_t)0, st, *a)
                         : launch_pdl(latrow::latent_rows_kernel<__nv_bfloat16>, dim3(a->T), dim3(128), (size_t)0, st, *a);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}

extern "C" int ub_latent_rotate(const UbLatentArgs* a, void* stream) {
  using namespace ub;
  if (a->T <= 0) return 0;
  if (latrow::bad(*a) || a->H <= 0) return -2;
  if (a->q == nullptr || a->q_out == nullptr || (a->q_off | a->qo_off | a->q_head | a->qo_head) % 8 != 0 || a->q_stride % 8 != 0 ||
      a->qo_stride % 8 != 0)
    return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e = a->f32 ? launch_pdl(latrow::latent_rotate_kernel<float>, dim3(a->T), dim3(128), (size_t)0, st, *a)
                         : launch_pdl(latrow::latent_rotate_kernel<__nv_bfloat16>, dim3(a->T), dim3(128), (size_t)0, st, *a);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
