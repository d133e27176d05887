// K6d: rows of a differential attention for kernels that know one map per head.  A head has two queries and two keys (one pair per
// softmax map) over one value; cached as one key row [key of map 1 | key of map 2], it becomes an attention of twice as many query
// heads, in which the query of a map is zero where the other map's key lies:
//
//   q_out[t, 2 h + m] = [0 .. | q[t, h, m] at m * dim | .. 0]                        [T, heads * maps, maps * dim]
//   k_cache[slot(t), g] = [k[t, g, 0] | k[t, g, 1]],  v_cache[slot(t), g] = v[t, g]
//
// so a cached row is read once for both maps.  Rows hold [Q | K | V] (or Q alone, for layers that read another layer's cache).
// One CTA per token, 16-byte accesses; slots are bounds-checked.
#include "../common/elem.cuh"
#include "../include/unillm_b200.h"

namespace ub {

template <typename V>
__global__ void __launch_bounds__(128) map_rows_kernel(const UbMapRowsArgs a, const int per /* elements per access */) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, cd = a.dim / per, cv = a.dv / per, M = a.maps;
  const V* row = reinterpret_cast<const V*>(a.src) + (long long)t * (a.ld / per);
  V* q = reinterpret_cast<V*>(a.q_out) + (long long)t * a.H * M * M * cd;
  for (int i = threadIdx.x; i < a.H * M * M * cd; i += 128) {
    const int c = i % cd, part = (i / cd) % M, head = i / (cd * M);        // head of the kernel: 2 h + m
    V v{};
    if (part == head % M) v = row[head * cd + c];
    q[i] = v;
  }
  if (a.slot_mapping == nullptr) return;
  const long long slot = a.slot_mapping[t];
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0) set_err(a.err, ERR_BOUNDS, t);
    return;
  }
  if (slot < 0) return;
  const long long blk = slot / a.block_size, off = slot % a.block_size;
  const int ck = M * cd;
  const V *k = row + a.H * ck, *v = k + a.G * ck;
  V* kd = reinterpret_cast<V*>(a.k_cache) + (blk * a.G * a.block_size + off) * ck;
  V* vd = reinterpret_cast<V*>(a.v_cache) + (blk * a.G * a.block_size + off) * cv;
  for (int i = threadIdx.x; i < a.G * ck; i += 128) kd[(long long)(i / ck) * a.block_size * ck + i % ck] = k[i];
  for (int i = threadIdx.x; i < a.G * cv; i += 128) vd[(long long)(i / cv) * a.block_size * cv + i % cv] = v[i];
}

}  // namespace ub

extern "C" int ub_map_rows(const UbMapRowsArgs* a, void* stream) {
  using namespace ub;
  if (a->T <= 0) return 0;
  const int per = a->f32 ? 4 : 8;
  if (a->H <= 0 || a->maps <= 0 || a->dim % 8 != 0 || a->ld % per != 0 || a->src == nullptr || a->q_out == nullptr) return -2;
  if (a->slot_mapping != nullptr && (a->k_cache == nullptr || a->v_cache == nullptr || a->G <= 0 || a->dv % 8 != 0 || a->block_size <= 0)) return -3;
  cudaError_t e = launch_pdl(map_rows_kernel<uint4>, dim3(a->T), dim3(128), (size_t)0, reinterpret_cast<cudaStream_t>(stream), *a, per);
  if (e == cudaSuccess) e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -(int)e;
}
