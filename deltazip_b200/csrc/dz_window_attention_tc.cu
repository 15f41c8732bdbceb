// Sliding-window attention for prompt portions on the 5th-generation tensor cores.
//
// A CTA takes 256 query rows of one (sequence, head) as two tiles of 128 (the MMA's M, one row per
// TMEM lane) and walks the keys in tiles of 64 that both read.  Roles of its twelve warps:
//   0-3, 4-7  softmax of query tile 0 / 1: a thread owns a row -- scores from TMEM into registers,
//             scale + bias + mask, running maximum, exponentials, weights back to TMEM
//   8-9       copies into 128-byte-swizzled shared memory, three or four stages: TMA where a tile lies in the
//             projection rows, 16-byte asynchronous copies where it comes from the cache ring or ends
//             with the sequence
//   10, 11    MMA issue for query tile 0 / 1: S = Q K^T (both operands in shared memory), O += P V
//             (P in TMEM, V read as it lies, keys along K and value columns contiguous)
// The two query tiles are independent chains, and each has two score buffers, so the scores of the
// next key tile are computed under the softmax of this one.
//
// TMEM: S0 (2 x 64) | S1 (2 x 64) | O0 (128) | O1 (128 columns).  The weights take the place of the
// scores they came from: 32 columns of 16-bit pairs (hi) and 32 with what the rounding left (lo); two
// products with v keep the weights at about 32-bit accuracy.
//
// The running maximum is only moved when it has grown by more than 8 (log2 units): weights then stay
// below 2^8, sums stay exact, and most tiles need no pass over O.
#include <algorithm>
#include <type_traits>

#include "dz_tc.cuh"
#include "dz_window_attention.cuh"

namespace dz {
namespace {

constexpr int kTileM = 128, kTileKeys = 64, kMaxStages = 4;
constexpr int kMaxDim = 192;                            // then the shared memory holds three stages of keys
constexpr int kThreadsTc = 384, kCopyThreads = 64;
constexpr int kSlabQ = kTileM * 128, kSlab = kTileKeys * 128;   // rows of 64 16-bit elements
constexpr int kBiasTc = 4096;
constexpr int kBiasPad = kTileM + kTileKeys - 2;        // distances from -kBiasPad up are in the table
constexpr float kMaxGrowth = 8.f;

// Pairs of 32-bit operations in one instruction.
struct Pair {
  unsigned long long v;
  __device__ __forceinline__ Pair() {}
  __device__ __forceinline__ Pair(float a, float b) {
    asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(a), "f"(b));
  }
  __device__ __forceinline__ void get(float& a, float& b) const {
    asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
  }
};
__device__ __forceinline__ Pair fma2(Pair a, Pair b, Pair c) {
  Pair d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d.v) : "l"(a.v), "l"(b.v), "l"(c.v));
  return d;
}
__device__ __forceinline__ Pair add2(Pair a, Pair b) {
  Pair d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d.v) : "l"(a.v), "l"(b.v));
  return d;
}

// Two weights as hi + lo pairs.  bf16: hi is the upper half of the float as it stands, lo the rounded rest.
template <typename T> __device__ __forceinline__ void split_weights(float a, float b, uint32_t& hi, uint32_t& lo) {
  if constexpr (std::is_same<T, __nv_bfloat16>::value) {
    const uint32_t ua = __float_as_uint(a), ub = __float_as_uint(b);
    hi = __byte_perm(ua, ub, 0x7632);
    float ra, rb;
    fma2(Pair(__uint_as_float(ua & 0xffff0000u), __uint_as_float(ub & 0xffff0000u)), Pair(-1.f, -1.f), Pair(a, b)).get(ra, rb);
    lo = Cvt<T>::down(ra, rb);
  } else {
    split_pair<T>(a, b, hi, lo);
  }
}

__device__ __forceinline__ void cp_async16_u32(uint32_t dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}

// As warp_umma_ss, with the first operand in tensor memory.
__device__ __forceinline__ void warp_umma_ts(uint32_t d, uint32_t a, uint32_t b_lo, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p, e;\n\t.reg .b64 db;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "setp.ne.b32 p, %5, 0;\n\t"
      "mov.b64 db, {%2, %3};\n\t"
      "@e tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], db, %4, p;\n\t}" ::"r"(d),
      "r"(a), "r"(b_lo), "r"(kDescHi), "r"(idesc), "r"(acc)
      : "memory");
}

template <typename T, int kStages>
__global__ void __launch_bounds__(kThreadsTc, 1)
window_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                         const AttnParams p) {
  constexpr int DT = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
  extern __shared__ uint8_t smem_dyn[];
  __shared__ uint64_t b_full[kStages], b_empty[kStages], b_s[2][2], b_p[2][2], b_pv[2], b_o[2], b_q;
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort;
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;
  const int seq = blockIdx.z, head = blockIdx.y % p.heads, v0 = (blockIdx.y / p.heads) * 128;
  pdl_wait();
  pdl_launch();
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0, ctx = p.ctx_lens[seq];
  const int m0 = (gridDim.x - 1 - blockIdx.x) * 2 * kTileM;     // long rows first: an even end
  if (m0 >= qn) return;
  const int kvh = head / (p.heads / p.kv_heads);
  const int vcols = min(128, p.vdim - v0);
  const int ks = (p.dim + 63) / 64, vs = (vcols + 63) / 64;      // slabs
  const uint32_t s_base = (smem_u32(smem_dyn) + 1023u) & ~1023u;
  const uint32_t s_q = s_base, s_k = s_q + 2 * ks * kSlabQ, s_v = s_k + kStages * ks * kSlab;
  float* s_bias = reinterpret_cast<float*>(smem_dyn + (s_v + kStages * vs * kSlab - smem_u32(smem_dyn)));
  volatile int* abort_flag = &s_abort;
  const T* qkv = (const T*)p.qkv;
  const T* kv = (const T*)p.kv;
  const int* table = p.block_tables + (size_t)seq * p.ring_blocks;
  const KeyRows kr(p, seq, q0, ctx);

  // key tiles: all of the CTA's, and of those the range [ta, tb) with keys a query tile may see
  const int first = p.window > 0 ? max(0, ctx + m0 - p.window + 1) : 0;
  const int end = ctx + min(m0 + 2 * kTileM, qn);
  const int tiles = (end - first + kTileKeys - 1) / kTileKeys;
  const int g = warp < 8 ? warp >> 2 : warp - 10;                // query tile of this warp (copy warps: unused)
  const int w0 = ctx + m0 + g * kTileM;                          // position of the tile's first row
  const int rows = min(kTileM, qn - m0 - g * kTileM);
  const int lo = p.window > 0 ? max(0, w0 - p.window + 1) : 0;
  const int ta = rows > 0 ? (lo - first) / kTileKeys : 0;
  const int tb = rows > 0 ? (w0 + rows - first + kTileKeys - 1) / kTileKeys : 0;

  if (tid == 0) {
    for (int i = 0; i < kStages; ++i) {
      mbar_init(smem_u32(&b_full[i]), kCopyThreads);
      mbar_init(smem_u32(&b_empty[i]), 2);
    }
    for (int i = 0; i < 2; ++i) {
      for (int k = 0; k < 2; ++k) {
        mbar_init(smem_u32(&b_s[i][k]), 1);
        mbar_init(smem_u32(&b_p[i][k]), kTileM / 32);
      }
      mbar_init(smem_u32(&b_pv[i]), 1);
      mbar_init(smem_u32(&b_o[i]), 1);
    }
    mbar_init(smem_u32(&b_q), 9);                                // eight softmax warps, one copy thread
    s_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    fence_proxy_async();
  }
  if (warp == 10) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "n"(512)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (p.dim % 16) {                                              // columns up to the MMA's K read as zero
    for (uint32_t i = tid * 16; i < (uint32_t)(2 * ks * kSlabQ + kStages * ks * kSlab); i += kThreadsTc * 16)
      sts128(s_q + i, make_uint4(0, 0, 0, 0));
    __syncthreads();
  }
  const int blen = p.bias ? p.bias_len : 1;
  fence_proxy_async();                                           // zeroed columns, for the MMAs
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // queries come by TMA where the 256 rows and their columns are all the sequence's and head's own
  const bool q_tma = p.dim % 16 == 0 && m0 + 2 * kTileM <= qn;
  const uint32_t tmem = s_tmem;

  if (warp >= 10) {
    // ---- MMA issue ----
    const uint32_t id_s = make_idesc<DT>(kTileKeys, false);
    const uint32_t id_o = make_idesc<DT>(vs * 64, false) | (1u << 16);       // B transposed
    const uint32_t t_s = tmem + g * 128, t_o = tmem + 256 + g * 128, s_qg = s_q + g * ks * kSlabQ;
    const int rest = (p.dim % 64 + 15) / 16;                                 // MMAs of the last slab, 0: a whole one
    auto scores = [&](int j) {
      const int st = j % kStages, buf = (j - ta) & 1;
      bar_wait(&b_full[st], (j / kStages) & 1, abort_flag, p.status);
      __syncwarp();
      tc_fence_after();
      const uint32_t a = desc_lo(s_qg), b = desc_lo(s_k + st * ks * kSlab), d = t_s + buf * 64;
      for (int c = 0; c < ks; ++c) {
        const uint32_t ac = a + c * (kSlabQ >> 4), bc = b + c * (kSlab >> 4);
        if (c + 1 < ks || rest == 0) {
#pragma unroll
          for (int k = 0; k < 4; ++k) warp_umma_ss(d, ac + 2 * k, bc + 2 * k, id_s, c + k > 0);
        } else {
          for (int k = 0; k < rest; ++k) warp_umma_ss(d, ac + 2 * k, bc + 2 * k, id_s, c + k > 0);
        }
      }
      warp_umma_commit(smem_u32(&b_s[g][buf]));
    };
    bar_wait(&b_q, 0, abort_flag, p.status);
    for (int j = 0; j < tiles; ++j) {
      const int st = j % kStages;
      if (j < ta || j >= tb) {
        bar_wait(&b_full[st], (j / kStages) & 1, abort_flag, p.status);
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(&b_empty[st]));
        continue;
      }
      if (j == ta) {
        scores(j);
        if (j + 1 < tb) scores(j + 1);
      }
      const int n = j - ta, buf = n & 1;
      bar_wait(&b_p[g][buf], (n >> 1) & 1, abort_flag, p.status);
      __syncwarp();
      tc_fence_after();
      const uint32_t b = desc_lo_mn(s_v + st * vs * kSlab, kSlab), pw = t_s + buf * 64;
#pragma unroll
      for (int k = 0; k < kTileKeys / 16; ++k) {                              // 16 keys: 2048 bytes of v
        warp_umma_ts(t_o, pw + k * 8, b + k * 128, id_o, (n > 0 || k > 0) ? 1u : 0u);
        warp_umma_ts(t_o, pw + 32 + k * 8, b + k * 128, id_o, 1u);
      }
      warp_umma_commit(smem_u32(&b_empty[st]));
      warp_umma_commit(smem_u32(&b_pv[g]));
      if (j + 2 < tb) scores(j + 2);               // behind the product that reads these columns' weights
      if (j + 1 == tb) warp_umma_commit(smem_u32(&b_o[g]));
    }
  } else if (warp >= 8) {
    // ---- copies ----
    const int t = tid - 256, c = t & 15;
    if (t == 0) {
      const uint32_t bar = smem_u32(&b_q);
      if (q_tma) {
        mbar_expect_tx(bar, 2 * ks * kSlabQ);
        for (int i = 0; i < 2 * ks; ++i)                          // two boxes of 64 rows fill a slab
          for (int half = 0; half < 2; ++half)
            tma_load_2d(s_q + i * kSlabQ + half * (kSlabQ / 2), &map_q, head * p.dim + (i % ks) * 64,
                        q0 + m0 + (i / ks) * kTileM + half * 64, bar);
      } else {
        mbar_arrive(bar);
      }
    }
    for (int j = 0; j < tiles; ++j) {
      const int st = j % kStages, key0 = first + j * kTileKeys;
      bar_wait(&b_empty[st], ((j / kStages) & 1) ^ 1, abort_flag, p.status);
      const uint32_t dk = s_k + st * ks * kSlab, dv = s_v + st * vs * kSlab, full = smem_u32(&b_full[st]);
      if (key0 >= kr.first && key0 + kTileKeys <= end) {
        if (t == 0) {
          const int row = kr.row + key0 - kr.first;
          mbar_expect_tx(full, (ks + vs) * kSlab);
          for (int i = 0; i < ks; ++i) tma_load_2d(dk + i * kSlab, &map_kv, p.k_off + kvh * p.dim + i * 64, row, full);
          for (int i = 0; i < vs; ++i) tma_load_2d(dv + i * kSlab, &map_kv, p.v_off + kvh * p.vdim + v0 + i * 64, row, full);
        } else {
          mbar_arrive(full);
        }
        continue;
      }
#pragma unroll 4
      for (int r = t >> 4; r < kTileKeys; r += kCopyThreads / 16) {
        const int key = key0 + r;
        const bool ok = key < end;
        const T *kp, *vp;
        if (!ok || key >= kr.first) {
          const T* row = kv + (size_t)(ok ? kr.row + key - kr.first : 0) * p.kv_stride;
          kp = row + p.k_off + (size_t)kvh * p.dim;
          vp = row + p.v_off + (size_t)kvh * p.vdim;
        } else {
          const size_t slot = ring_slot(p, table, key) * p.kv_heads + kvh;
          kp = (const T*)p.k_cache + slot * p.dim;
          vp = (const T*)p.v_cache + slot * p.vdim;
        }
        for (int e = c; e < p.dim / 8; e += 16) cp_async16_u32(dk + swizzled(r, e, kSlab), kp + e * 8, ok);
        if (c < vcols / 8) cp_async16_u32(dv + swizzled(r, c, kSlab), vp + v0 + c * 8, ok);
      }
      cp_async_commit();
      cp_async_wait<0>();
      fence_proxy_async();
      mbar_arrive(full);
    }
  } else {
    // ---- softmax ----
    if (!q_tma) {
      for (int c = tid & 15; c < p.dim / 8; c += 16) {
        for (int i = tid >> 4; i < 2 * kTileM; i += 16) {
          const bool ok = m0 + i < qn;
          const T* src = qkv + (size_t)(q0 + (ok ? m0 + i : 0)) * p.row_stride + (size_t)head * p.dim + c * 8;
          cp_async16_u32(s_q + (i >> 7) * ks * kSlabQ + swizzled(i & 127, c, kSlabQ), src, ok);
        }
      }
      cp_async_commit();
      cp_async_wait<0>();
      fence_proxy_async();
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(smem_u32(&b_q));
    for (int i = tid; i < blen + 2 * kBiasPad; i += 256) {
      const int d = i - kBiasPad;
      s_bias[i] = d < 0 ? -INFINITY : p.bias ? p.bias[(size_t)head * p.bias_len + min(d, blen - 1)] * kLog2e : 0.f;
    }
    named_bar_sync(1, 256);
    const int r = (warp & 3) * 32 + lane, pos = w0 + r;
    const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t t_o = tmem + 256 + g * 128 + lane_addr;
    const float scale2 = p.scale * kLog2e, far_bias = s_bias[kBiasPad + blen - 1];
    float m = p.sink ? p.sink[head] * kLog2e : -INFINITY, l = p.sink ? 1.f : 0.f;
    for (int j = ta; j < tb; ++j) {
      const int n = j - ta, buf = n & 1;
      const uint32_t t_s = tmem + g * 128 + buf * 64 + lane_addr;
      bar_wait(&b_s[g][buf], (n >> 1) & 1, abort_flag, p.status);
      tc_fence_after();
      float s[kTileKeys];
#pragma unroll
      for (int c = 0; c < kTileKeys; c += 32) tmem_ld32(t_s + c, s + c);
      tmem_wait_ld();
      const int t0 = first + j * kTileKeys;
      const bool cut = p.window > 0 && w0 + kTileM - 1 - t0 >= p.window;
      float mul = 1.f, add = 0.f;                    // what is still to be applied to s
      if (w0 - (t0 + kTileKeys - 1) >= blen - 1 && !cut && scale2 > 0.f) {
        mul = scale2;                                // every distance is in the last column, all keys visible
        add = far_bias;
      } else {                                       // the table holds minus infinity at negative distances
        if (w0 - (t0 + kTileKeys - 1) >= blen - 1) {
#pragma unroll
          for (int c = 0; c < kTileKeys; ++c) s[c] = fmaf(s[c], scale2, far_bias);
        } else {
          const float* tab = s_bias + kBiasPad + (pos - t0);
#pragma unroll
          for (int c = 0; c < kTileKeys; ++c) s[c] = fmaf(s[c], scale2, tab[-c]);
        }
        if (cut) {
          const int out = pos - p.window - t0;       // keys up to here have left the window
#pragma unroll
          for (int c = 0; c < kTileKeys; ++c) s[c] = c <= out ? -INFINITY : s[c];
        }
      }
      float mx[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int c = 4; c < kTileKeys; ++c) mx[c & 3] = fmaxf(mx[c & 3], s[c]);
      const float top = fmaf(fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])), mul, add);
      float f = 1.f;
      if (m == -INFINITY) {
        m = top;                                     // nothing summed so far
      } else if (top > m + kMaxGrowth) {
        f = ex2(m - top);
        m = top;
        l *= f;
      }
      const bool rescale = __any_sync(0xffffffffu, f != 1.f);
      add -= m == -INFINITY ? 0.f : m;
      const Pair mul2(mul, mul), add2v(add, add);
      Pair sum[2] = {Pair(0.f, 0.f), Pair(0.f, 0.f)};
#pragma unroll
      for (int c = 0; c < kTileKeys; c += 32) {
        uint32_t hi[16], low[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float a, b;
          fma2(Pair(s[c + 2 * i], s[c + 2 * i + 1]), mul2, add2v).get(a, b);
          a = ex2(a);
          b = ex2(b);
          sum[i & 1] = add2(sum[i & 1], Pair(a, b));
          split_weights<T>(a, b, hi[i], low[i]);
        }
        tmem_st16(t_s + c / 2, hi);
        tmem_st16(t_s + 32 + c / 2, low);
      }
      float la, lb;
      add2(sum[0], sum[1]).get(la, lb);
      l += la + lb;
      if (rescale) {
        if (n > 0) bar_wait(&b_pv[g], (n - 1) & 1, abort_flag, p.status);   // O holds the products so far
        tc_fence_after();
        for (int c = 0; c < vs * 64; c += 32) {
          float o[32];
          tmem_ld32(t_o + c, o);
          tmem_wait_ld();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] *= f;
          tmem_st16(t_o + c, reinterpret_cast<const uint32_t*>(o));
          tmem_st16(t_o + c + 16, reinterpret_cast<const uint32_t*>(o + 16));
        }
      }
      tmem_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&b_p[g][buf]));
    }
    if (tb > ta) bar_wait(&b_o[g], 0, abort_flag, p.status);
    tc_fence_after();
    const float inv = 1.f / l;
    T* op = (T*)p.out + (size_t)(q0 + m0 + g * kTileM + r) * p.heads * p.vdim + (size_t)head * p.vdim + v0;
    for (int c = 0; c < vcols; c += 32) {
      float o[32];
      tmem_ld32(t_o + c, o);
      tmem_wait_ld();
      if (r < rows) {
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          if (c + i < vcols) {
            float v[8];
#pragma unroll
            for (int q = 0; q < 8; ++q) v[q] = o[i + q] * inv;
            store8<T>(op + c + i, v);
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (s_abort) {                                                  // let copies and MMAs under way end
    const unsigned long long t0 = globaltimer();
    while (globaltimer() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 10) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(512) : "memory");
  }
}

int tc_stages(const AttnParams& p) { return p.dim <= 128 ? kMaxStages : kMaxStages - 1; }

size_t tc_smem(const AttnParams& p) {
  const int kStages = tc_stages(p), ks = (p.dim + 63) / 64, vs = (std::min(128, p.vdim) + 63) / 64;
  const int blen = p.bias ? p.bias_len : 1;
  return (size_t)2 * ks * kSlabQ + (size_t)kStages * (ks + vs) * kSlab + (size_t)(blen + 2 * kBiasPad) * 4 + 1024;
}

template <typename T>
int run(const AttnParams& p, int num_seqs, int max_q, cudaStream_t st) {
  const size_t smem = tc_smem(p);
  constexpr int kDt = std::is_same<T, __nv_bfloat16>::value;
  CUtensorMap map_q, map_kv;
  int rc = make_map(&map_q, p.qkv, p.rows, (int)p.row_stride, kTileKeys, kDt);
  if (!rc) rc = make_map(&map_kv, p.kv, p.kv_rows, (int)p.kv_stride, kTileKeys, kDt);
  if (rc) return rc;
  const dim3 grid((max_q + 2 * kTileM - 1) / (2 * kTileM), p.heads * ((p.vdim + 127) / 128), num_seqs);
  auto kern = tc_stages(p) == kMaxStages ? window_prefill_tc_kernel<T, kMaxStages> : window_prefill_tc_kernel<T, kMaxStages - 1>;
  DZ_CUDA_OK(allow_smem(kern, smem));
  DZ_CUDA_OK(launch_ex(kern, grid, dim3(kThreadsTc), smem, 1, st, map_q, map_kv, p));
  return DZ_OK;
}

}  // namespace

bool window_prefill_tc_supported(const AttnParams& p, int dtype) {
  return (dtype == DZ_DTYPE_F16 || dtype == DZ_DTYPE_BF16) && p.dim <= kMaxDim && p.dim % 8 == 0 &&
         p.row_stride < (1ll << 31) && p.kv_stride < (1ll << 31) && tc_smem(p) <= kMaxDynSmem && p.vdim % 8 == 0 &&
         (!p.bias || p.bias_len <= kBiasTc) && p.heads * ((p.vdim + 127) / 128) <= 65535;
}

int launch_window_prefill_tc(const AttnParams& p, int num_seqs, int max_q, int dtype, cudaStream_t st) {
  return dtype == DZ_DTYPE_BF16 ? run<__nv_bfloat16>(p, num_seqs, max_q, st) : run<__half>(p, num_seqs, max_q, st);
}

}  // namespace dz
