// Shared by the kernels that attend to cached latents directly.
#pragma once

#include "dz_elem.cuh"

namespace dz {

struct LatentParams {
  const void* q;                         // [rows, heads, rank + rot]
  const void* cache;                     // [slots, rank + rot]
  const int* tables;
  int table_width, block_size;
  const int* q_starts;
  const int* ctx_lens;
  int num_seqs, rows, heads, rank, rot;
  float scale;
  const float* sink;
  void* out;                             // [rows, heads, rank]
  int splits;
  float* partial;                        // [rows, heads, splits, rank + 2]
  int* tickets;                          // [rows, head groups]
  int64_t cache_rows;
  int* status;                           // first error a kernel met (sticky until read)
};

// Keys of a split, whole tiles of 64; the last splits of a short sequence may have none.
__device__ __forceinline__ int keys_per_split(int n, int splits) { return ((n + splits - 1) / splits + 63) / 64 * 64; }

// Called by every thread of a CTA after it has written its split's sums, maximum (log2 units) and
// denominator to p.partial: the last CTA of a (row, head group) to arrive at its ticket merges the
// splits.  Nothing waits.  Grid (head groups, rows, splits).
template <typename T>
__device__ __forceinline__ void merge_splits(const LatentParams& p, int row, int h0, int live, int* s_last) {
  const int lane = threadIdx.x & 31, warps = blockDim.x >> 5, w = p.rank + 2;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    int* tk = p.tickets + (size_t)row * gridDim.x + blockIdx.x;
    *s_last = atomicAdd(tk, 1) == p.splits - 1;
    if (*s_last) *tk = 0;                                            // ready for the next launch
  }
  __syncthreads();
  if (!*s_last) return;
  __threadfence();
  for (int h = threadIdx.x >> 5; h < live; h += warps) {             // a warp merges a head
    const size_t at = (size_t)row * p.heads + h0 + h;
    const float* pp = p.partial + at * p.splits * w;
    const float sk2 = p.sink ? p.sink[h0 + h] * 1.4426950408889634f : -INFINITY;
    float top = sk2;
    for (int s = 0; s < p.splits; ++s) top = fmaxf(top, __ldcg(pp + s * w + p.rank));
    float den = p.sink ? exp2f(sk2 - top) : 0.f;
    for (int s = 0; s < p.splits; ++s) den += __ldcg(pp + s * w + p.rank + 1) * exp2f(__ldcg(pp + s * w + p.rank) - top);
    const float inv = 1.f / den;
    for (int c = lane * 2; c < p.rank; c += 64) {                    // rank is a multiple of eight
      float x = 0.f, y = 0.f;
      for (int s = 0; s < p.splits; ++s) {
        const float f = exp2f(__ldcg(pp + s * w + p.rank) - top);
        const float2 v = __ldcg(reinterpret_cast<const float2*>(pp + s * w + c));
        x += v.x * f;
        y += v.y * f;
      }
      *reinterpret_cast<uint32_t*>((T*)p.out + at * p.rank + c) = Cvt<T>::down(x * inv, y * inv);
    }
  }
}

// dz_latent_tc.cu
bool latent_tc_supported(const LatentParams& p, int dtype);
int latent_tc_groups(int heads);
int launch_latent_tc(const LatentParams& p, int dtype, cudaStream_t st);

}  // namespace dz
