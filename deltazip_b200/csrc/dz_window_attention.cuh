// Shared by the sliding-window attention kernels.
#pragma once

#include "dz_elem.cuh"

namespace dz {

// Where a sequence's keys are.
enum KeySource {
  kKeysSplit = 0,                        // positions before ctx in the cache, the others in the rows themselves
  kKeysCached = 1,                       // all in the cache
  kKeysRows = 2                          // all in rows of their own, from kv_starts[sequence] on
};

struct AttnParams {
  const void* qkv;
  int64_t row_stride;                    // elements
  int k_off, v_off;                      // columns of `kv` where the key / value parts start
  void* out;                             // [rows, heads * vdim]
  const void* k_cache;                   // [slots, kv_heads, dim]
  const void* v_cache;                   // [slots, kv_heads, vdim]; any-size kernel: the first vdim of every v_row
  int v_row;
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
  const float* sink;                     // [heads] one more score per row without a key or value, or nullptr
  int source;                            // KeySource
  const void* kv;                        // rows with keys and values: qkv, or rows of their own
  int64_t kv_stride;
  const int* kv_starts;                  // [sequences + 1], kKeysRows
  int kv_rows;                           // of kv
  int* status;                           // first error a kernel met (sticky until read)
};

__device__ __forceinline__ size_t ring_slot(const AttnParams& p, const int* table, int t) {
  const int b = t / p.block_size;
  return (size_t)table[b % p.ring_blocks] * p.block_size + (t - b * p.block_size);
}

// The first position of a sequence whose key lies in `kv`, and the row it lies in.
struct KeyRows {
  int first, row;
  __device__ __forceinline__ KeyRows(const AttnParams& p, int seq, int q0, int ctx) {
    first = p.source == kKeysSplit ? ctx : p.source == kKeysRows ? 0 : 0x7fffffff;
    row = p.source == kKeysRows ? p.kv_starts[seq] : q0;
  }
};

constexpr float kLog2e = 1.4426950408889634f;

// dz_window_attention.cu: any type, any sizes, one CTA per (row, head)
int launch_attention_any(const AttnParams& p, int num_seqs, int dtype, cudaStream_t st);

// dz_window_attention_tc.cu: prompt portions on tcgen05
bool window_prefill_tc_supported(const AttnParams& p, int dtype);
int launch_window_prefill_tc(const AttnParams& p, int num_seqs, int max_q, int dtype, cudaStream_t st);

}  // namespace dz
