// Shared by the sliding-window attention kernels.
#pragma once

#include "dz_elem.cuh"

namespace dz {

struct AttnParams {
  const void* qkv;
  int64_t row_stride;                    // elements
  int k_off, v_off;                      // columns where the key / value parts start
  void* out;                             // [rows, heads * vdim]
  const void* k_cache;                   // [slots, kv_heads, dim]
  const void* v_cache;                   // [slots, kv_heads, vdim]
  const int* block_tables;               // [sequences, ring_blocks]
  int ring_blocks, block_size;
  const int* q_starts;                   // [sequences + 1] first row of every sequence
  const int* ctx_lens;                   // [sequences] tokens already in the cache
  int heads, kv_heads, dim, vdim;
  float scale;
  int window;
  const float* bias;                     // [heads, bias_len] or nullptr
  int bias_len;
  int rows;                              // of qkv
  int* status;                           // first error a kernel met (sticky until read)
};

__device__ __forceinline__ size_t ring_slot(const AttnParams& p, const int* table, int t) {
  const int b = t / p.block_size;
  return (size_t)table[b % p.ring_blocks] * p.block_size + (t - b * p.block_size);
}

constexpr float kLog2e = 1.4426950408889634f;

// dz_window_attention_tc.cu: prompt portions on tcgen05
bool window_prefill_tc_supported(const AttnParams& p, int dtype);
int launch_window_prefill_tc(const AttnParams& p, int num_seqs, int max_q, int dtype, cudaStream_t st);

}  // namespace dz
