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
  float* partial;                        // [rows, heads, splits, partial_row(rank)]
  int* tickets;                          // [rows, head groups]
  int64_t cache_rows;
  int* status;                           // first error a kernel met (sticky until read)
};

// Keys of a split, whole tiles of 64; the last splits of a short sequence may have none.
__device__ __forceinline__ int keys_per_split(int n, int splits) { return ((n + splits - 1) / splits + 63) / 64 * 64; }

// A split's sums, then its maximum (log2 units) and its denominator; padded to whole float4.
__host__ __device__ constexpr int partial_row(int rank) { return rank + 4; }

// Called by every thread of a CTA after it has written its split's part of p.partial: the last CTA of a
// (row, head group) to arrive at its ticket merges the splits.  Nothing waits.  Grid (head groups, rows,
// splits); `factors`: shared memory for 2 * live * splits floats that nothing uses any more.
template <typename T>
__device__ __forceinline__ void merge_splits(const LatentParams& p, int row, int h0, int live, int* s_last, float* factors) {
  const int w = partial_row(p.rank);
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
  const float* base = p.partial + ((size_t)row * p.heads + h0) * p.splits * w;
  // a thread per (head, split), the splits of a head next to each other
  for (int i = threadIdx.x; i < live * p.splits; i += blockDim.x)
    reinterpret_cast<float2*>(factors)[i] = __ldcg(reinterpret_cast<const float2*>(base + (size_t)i * w + p.rank));
  __syncthreads();
  for (int h = threadIdx.x; h < live; h += blockDim.x) {
    float2* f = reinterpret_cast<float2*>(factors) + h * p.splits;
    const float sk2 = p.sink ? p.sink[h0 + h] * 1.4426950408889634f : -INFINITY;
    float top = sk2;
    for (int s = 0; s < p.splits; ++s) top = fmaxf(top, f[s].x);
    float den = p.sink ? exp2f(sk2 - top) : 0.f;
    for (int s = 0; s < p.splits; ++s) {
      f[s].x = exp2f(f[s].x - top);
      den += f[s].y * f[s].x;
    }
    for (int s = 0; s < p.splits; ++s) f[s].x /= den;
  }
  __syncthreads();
  const int quads = p.rank / 4;                                      // rank is a multiple of eight
#pragma unroll 4
  for (int i = threadIdx.x; i < live * quads; i += blockDim.x) {
    const int h = i / quads, c = (i - h * quads) * 4;
    const float* pp = base + (size_t)h * p.splits * w + c;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 2
    for (int s = 0; s < p.splits; ++s) {
      const float f = factors[2 * (h * p.splits + s)];
      const float4 v = __ldcg(reinterpret_cast<const float4*>(pp + (size_t)s * w));
      a.x += v.x * f; a.y += v.y * f; a.z += v.z * f; a.w += v.w * f;
    }
    *reinterpret_cast<uint2*>((T*)p.out + ((size_t)row * p.heads + h0 + h) * p.rank + c) =
        make_uint2(Cvt<T>::down(a.x, a.y), Cvt<T>::down(a.z, a.w));
  }
}

// dz_latent_tc.cu
bool latent_tc_supported(const LatentParams& p, int dtype);
int latent_tc_groups(int heads);
int launch_latent_tc(const LatentParams& p, int dtype, cudaStream_t st);

}  // namespace dz
