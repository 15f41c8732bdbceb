// Causal attention with a sliding window and a learned additive bias per distance, over rows of a
// fused projection [q | k | v] and a paged cache used as a ring.
//
//   score(i, j) = (q_i . k_j) * scale + bias[head][min(i - j, bias_len - 1)],  visible when
//   0 <= i - j < window (window <= 0: all earlier keys),  softmax, times v.
//
// q, k share the head size `dim`, v has its own `vdim`; query head h reads key/value head
// h / (heads / kv_heads).  Position t of a sequence lives in cache slot
//   table[(t / block_size) % ring_blocks] * block_size + t % block_size,
// so a sequence that only looks back `window` tokens needs ceil(window / block_size) blocks however
// long it gets.  A portion of a prompt reads its own keys and values from the projection rows and
// earlier ones from the cache, and is appended to the cache afterwards (`dz_kv_append`): the ring
// never has to hold more than a window.  A decoded token is appended before attention, inside the
// query / key norm.
//
// Keys and values may also lie in rows of their own (`kv`, all positions of a sequence from
// kv_starts[sequence] on), and a row may have a sink: one more score in the softmax's denominator,
// not scaled, without a key or a value.
//
// Scores, softmax weights and sums are 32-bit.  In the tensor-core kernel a weight enters its
// product with v as a hi + lo pair of 16-bit numbers.
#include "dz_window_attention.cuh"

namespace dz {
namespace {

// -------------------------------------------------------------------------------------------------
// RMS norm of the whole query row and of the whole key row (all heads at once), in place, and the
// optional append of the normed key and of the value to the cache.
// -------------------------------------------------------------------------------------------------
template <typename T, int VEC>
__device__ __forceinline__ void norm_part(T* p, int n, const float* w, float eps, float* part, T* cache) {
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
    if constexpr (VEC == 8) {
      float f[8];
      load8<T>(p + i, f);
#pragma unroll
      for (int q = 0; q < 8; ++q) ss += f[q] * f[q];
    } else {
      const float f = Cvt<T>::one(p[i]);
      ss += f * f;
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, part) / (float)n + eps);
  for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
    if constexpr (VEC == 8) {
      float f[8], g[8];
      load8<T>(p + i, f);
      load8<float>(w + i, g);
#pragma unroll
      for (int q = 0; q < 8; ++q) f[q] = f[q] * inv * g[q];
      store8<T>(p + i, f);
      if (cache) store8<T>(cache + i, f);
    } else {
      const T v = Cvt<T>::from(Cvt<T>::one(p[i]) * inv * w[i]);
      p[i] = v;
      if (cache) cache[i] = v;
    }
  }
}

template <typename T, int VEC>
__device__ __forceinline__ void copy_part(const T* src, T* dst, int n) {
  for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
    if constexpr (VEC == 8 && sizeof(T) == 2) {
      *reinterpret_cast<uint4*>(dst + i) = *reinterpret_cast<const uint4*>(src + i);
    } else if constexpr (VEC == 8) {
      reinterpret_cast<float4*>(dst + i)[0] = reinterpret_cast<const float4*>(src + i)[0];
      reinterpret_cast<float4*>(dst + i)[1] = reinterpret_cast<const float4*>(src + i)[1];
    } else {
      dst[i] = src[i];
    }
  }
}

// grid (rows, 2): y = 0 the query part, y = 1 the key part and the cache append
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
qk_norm_kernel(T* __restrict__ qkv, int64_t row_stride, int qn, int kn, int vn, const float* __restrict__ wq,
               const float* __restrict__ wk, float eps, T* __restrict__ k_cache, T* __restrict__ v_cache,
               const long long* __restrict__ slot_mapping) {
  __shared__ float s_part[8];
  pdl_wait();
  pdl_launch();
  T* row = qkv + (size_t)blockIdx.x * row_stride;
  if (blockIdx.y == 0) {
    norm_part<T, VEC>(row, qn, wq, eps, s_part, nullptr);
    return;
  }
  const long long slot = slot_mapping ? slot_mapping[blockIdx.x] : -1;
  norm_part<T, VEC>(row + qn, kn, wk, eps, s_part, slot >= 0 ? k_cache + (size_t)slot * kn : nullptr);
  if (slot >= 0) copy_part<T, VEC>(row + qn + kn, v_cache + (size_t)slot * vn, vn);
}

template <typename T, int VEC>
__global__ void __launch_bounds__(128)
kv_append_kernel(const T* __restrict__ qkv, int64_t row_stride, int k_off, int kn, int vn, T* __restrict__ k_cache,
                 T* __restrict__ v_cache, const long long* __restrict__ slot_mapping) {
  pdl_wait();
  pdl_launch();
  const long long slot = slot_mapping[blockIdx.x];
  if (slot < 0) return;
  const T* row = qkv + (size_t)blockIdx.x * row_stride + k_off;
  copy_part<T, VEC>(row, k_cache + (size_t)slot * kn, kn);
  copy_part<T, VEC>(row + kn, v_cache + (size_t)slot * vn, vn);
}

// -------------------------------------------------------------------------------------------------
// Any type, any sizes: one CTA per (row, head), 128 keys at a time.  The 32-bit path, and the
// 16-bit one for sizes the kernels below do not take.
// -------------------------------------------------------------------------------------------------
constexpr int kAnyThreads = 128, kAnyMaxV = 8;       // vdim <= 8 * 128

template <typename T>
__global__ void __launch_bounds__(kAnyThreads)
attention_any_kernel(AttnParams p, int num_seqs) {
  __shared__ float s_w[kAnyThreads];
  __shared__ size_t s_v[kAnyThreads];                // value row of every key of the tile
  __shared__ float s_part[kAnyThreads / 32];
  __shared__ int s_seq;
  extern __shared__ float s_q[];
  pdl_wait();
  pdl_launch();
  const int row = blockIdx.x, head = blockIdx.y, kvh = head / (p.heads / p.kv_heads);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int s = threadIdx.x; s < num_seqs; s += kAnyThreads)
    if (row >= p.q_starts[s] && row < p.q_starts[s + 1]) s_seq = s;
  const T* qkv = (const T*)p.qkv;
  for (int d = threadIdx.x; d < p.dim; d += kAnyThreads)
    s_q[d] = Cvt<T>::one(qkv[(size_t)row * p.row_stride + (size_t)head * p.dim + d]);
  __syncthreads();
  const int seq = s_seq, q0 = p.q_starts[seq], ctx = p.ctx_lens[seq], pos = ctx + row - q0;
  const int* table = p.block_tables + (size_t)seq * p.ring_blocks;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const KeyRows kr(p, seq, q0, ctx);
  const T* kv = (const T*)p.kv;
  float m = p.sink ? p.sink[head] : -INFINITY, l = p.sink ? 1.f : 0.f, acc[kAnyMaxV];
#pragma unroll
  for (int c = 0; c < kAnyMaxV; ++c) acc[c] = 0.f;
  for (int t0 = lo; t0 <= pos; t0 += kAnyThreads) {
    const int n = min(kAnyThreads, pos + 1 - t0);
    for (int k = warp; k < n; k += kAnyThreads / 32) {
      const int t = t0 + k;
      const T* kp;
      if (t >= kr.first) {
        kp = kv + (size_t)(kr.row + t - kr.first) * p.kv_stride + p.k_off + (size_t)kvh * p.dim;
      } else {
        kp = (const T*)p.k_cache + (ring_slot(p, table, t) * p.kv_heads + kvh) * p.dim;
      }
      float s = 0.f;
      for (int d = lane; d < p.dim; d += 32) s += s_q[d] * Cvt<T>::one(kp[d]);
      s = warp_sum(s);
      if (lane == 0) {
        s = s * p.scale;
        if (p.bias) s += p.bias[(size_t)head * p.bias_len + min(pos - t, p.bias_len - 1)];
        s_w[k] = s;
        s_v[k] = t >= kr.first ? (size_t)(kr.row + t - kr.first) * p.kv_stride + p.v_off + (size_t)kvh * p.vdim
                               : (ring_slot(p, table, t) * p.kv_heads + kvh) * p.v_row;
      }
    }
    __syncthreads();
    const float sv = (int)threadIdx.x < n ? s_w[threadIdx.x] : -INFINITY;
    float mx = warp_max(sv);
    if (lane == 0) s_part[warp] = mx;
    __syncthreads();
    for (int w = 0; w < kAnyThreads / 32; ++w) mx = fmaxf(mx, s_part[w]);
    const float mn = fmaxf(m, mx), c = expf(m - mn);
    const float e = (int)threadIdx.x < n ? expf(sv - mn) : 0.f;
    l = l * c + block_sum(e, s_part);
    s_w[threadIdx.x] = e;
    __syncthreads();
#pragma unroll
    for (int v = 0; v < kAnyMaxV; ++v) {
      const int d = threadIdx.x + v * kAnyThreads;
      if (d < p.vdim) {
        float a = acc[v] * c;
        for (int k = 0; k < n; ++k)
          a += s_w[k] * Cvt<T>::one((t0 + k >= kr.first ? kv : (const T*)p.v_cache)[s_v[k] + d]);
        acc[v] = a;
      }
    }
    m = mn;
    __syncthreads();
  }
#pragma unroll
  for (int v = 0; v < kAnyMaxV; ++v) {
    const int d = threadIdx.x + v * kAnyThreads;
    if (d < p.vdim)
      ((T*)p.out)[(size_t)row * p.heads * p.vdim + (size_t)head * p.vdim + d] = Cvt<T>::from(acc[v] / l);
  }
}

// -------------------------------------------------------------------------------------------------
// Decode: one query row per sequence, all keys in the cache.  Grid (kv heads x groups of G query
// heads, sequences, splits).  A half-warp owns a key/value row (16 lanes x 16 bytes, NK / NV such
// loads), a warp two pairs of rows per step; each half-warp keeps a running (max, sum, accumulator),
// merged by shuffles, then through shared memory, then -- with splits -- by the last CTA of a
// (sequence, head group) to arrive at its ticket.  Nothing waits on anything.
// -------------------------------------------------------------------------------------------------
// CTAs an SM is to hold where the compiler would take registers for fewer; 0: as it likes.
__host__ __device__ constexpr int decode_ctas(int g, int nk, int nv) {
  return g != 2 ? 0 : nk + nv == 2 ? 3 : nk + nv == 4 ? 2 : 0;
}
template <typename T, int G, int NK, int NV>
__global__ void __launch_bounds__(256, decode_ctas(G, NK, NV))
window_decode_kernel(AttnParams p, int splits, float* __restrict__ partial, int* __restrict__ tickets) {
  constexpr int kWarps = 8, VW = NV * 128;
  __shared__ float s_m[kWarps][G], s_l[kWarps][G];
  __shared__ float s_acc[kWarps][G][VW];
  __shared__ int s_last;
  const int seq = blockIdx.y, split = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = lane >> 4, hl = lane & 15;
  const int ratio = p.heads / p.kv_heads, chunks = (ratio + G - 1) / G;
  const int kvh = blockIdx.x / chunks, g0 = (blockIdx.x % chunks) * G;
  pdl_wait();
  pdl_launch();
  const int pos = p.ctx_lens[seq];                  // the query's position; its key is in the cache
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, n = pos + 1 - lo;
  const int per = (n + splits - 1) / splits;
  const int t0 = lo + split * per, t1 = min(pos + 1, t0 + per);
  const int* table = p.block_tables + (size_t)seq * p.ring_blocks;
  const T* kc = (const T*)p.k_cache;
  const T* vc = (const T*)p.v_cache;
  float q[G][NK][8], m[G], l[G], acc[G][NV][8];
  const float* bias[G];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int head = kvh * ratio + min(g0 + g, ratio - 1);      // a surplus lane repeats the last head
    bias[g] = p.bias ? p.bias + (size_t)head * p.bias_len : nullptr;
    // one half-warp of one split starts with the sink in its sum
    const bool sink = p.sink && split == 0 && threadIdx.x < 16;
    m[g] = sink ? p.sink[head] : -INFINITY;
    l[g] = sink ? 1.f : 0.f;
#pragma unroll
    for (int c = 0; c < NK; ++c) {
      const int d = (c * 16 + hl) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) q[g][c][j] = 0.f;
      if (d < p.dim) {
        load8<T>((const T*)p.qkv + (size_t)seq * p.row_stride + (size_t)head * p.dim + d, q[g][c]);
#pragma unroll
        for (int j = 0; j < 8; ++j) q[g][c][j] *= p.scale;
      }
    }
#pragma unroll
    for (int c = 0; c < NV; ++c)
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[g][c][j] = 0.f;
  }
  for (int base = t0 + 2 * warp; base < t1; base += 4 * kWarps) {
    const int ta = base + half, tb = ta + 2 * kWarps;
    const bool a_ok = ta < t1, b_ok = tb < t1;
    const int tac = min(ta, t1 - 1), tbc = min(tb, t1 - 1);     // rows read for absent keys
    const size_t ra = ring_slot(p, table, tac) * p.kv_heads + kvh;
    const size_t rb = ring_slot(p, table, tbc) * p.kv_heads + kvh;
    uint4 ka[NK], kb[NK], va[NV], vb[NV];
#pragma unroll
    for (int c = 0; c < NK; ++c) {
      const int d = (c * 16 + hl) * 8;
      ka[c] = kb[c] = make_uint4(0, 0, 0, 0);
      if (d < p.dim) {
        ka[c] = *reinterpret_cast<const uint4*>(kc + ra * p.dim + d);
        kb[c] = *reinterpret_cast<const uint4*>(kc + rb * p.dim + d);
      }
    }
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int d = (c * 16 + hl) * 8;
      va[c] = vb[c] = make_uint4(0, 0, 0, 0);
      if (d < p.vdim) {
        va[c] = *reinterpret_cast<const uint4*>(vc + ra * p.vdim + d);
        vb[c] = *reinterpret_cast<const uint4*>(vc + rb * p.vdim + d);
      }
    }
    float pa[G], pb[G];
    {
      float sa[G], sb[G];
#pragma unroll
      for (int g = 0; g < G; ++g) sa[g] = sb[g] = 0.f;
#pragma unroll
      for (int c = 0; c < NK; ++c) {
        const uint32_t wa[4] = {ka[c].x, ka[c].y, ka[c].z, ka[c].w}, wb[4] = {kb[c].x, kb[c].y, kb[c].z, kb[c].w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 fa = Cvt<T>::up(wa[j]), fb = Cvt<T>::up(wb[j]);
#pragma unroll
          for (int g = 0; g < G; ++g) {
            sa[g] += q[g][c][2 * j] * fa.x + q[g][c][2 * j + 1] * fa.y;
            sb[g] += q[g][c][2 * j] * fb.x + q[g][c][2 * j + 1] * fb.y;
          }
        }
      }
#pragma unroll
      for (int g = 0; g < G; ++g) {
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) {                        // within the half-warp
          sa[g] += __shfl_xor_sync(0xffffffffu, sa[g], o);
          sb[g] += __shfl_xor_sync(0xffffffffu, sb[g], o);
        }
        if (bias[g]) {
          sa[g] += bias[g][min(pos - tac, p.bias_len - 1)];
          sb[g] += bias[g][min(pos - tbc, p.bias_len - 1)];
        }
        if (!a_ok) sa[g] = -INFINITY;
        if (!b_ok) sb[g] = -INFINITY;                            // b_ok implies a_ok
        const float mn = fmaxf(m[g], fmaxf(sa[g], sb[g]));
        const float ms = mn == -INFINITY ? 0.f : mn;
        const float c = __expf(m[g] - ms);
        pa[g] = __expf(sa[g] - ms);
        pb[g] = __expf(sb[g] - ms);
        l[g] = l[g] * c + pa[g] + pb[g];
        m[g] = mn;
#pragma unroll
        for (int v = 0; v < NV; ++v)
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[g][v][j] *= c;
      }
    }
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const uint32_t wa[4] = {va[c].x, va[c].y, va[c].z, va[c].w}, wb[4] = {vb[c].x, vb[c].y, vb[c].z, vb[c].w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 fa = Cvt<T>::up(wa[j]), fb = Cvt<T>::up(wb[j]);
#pragma unroll
        for (int g = 0; g < G; ++g) {
          acc[g][c][2 * j] += pa[g] * fa.x + pb[g] * fb.x;
          acc[g][c][2 * j + 1] += pa[g] * fa.y + pb[g] * fb.y;
        }
      }
    }
  }
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const float mo = __shfl_xor_sync(0xffffffffu, m[g], 16);
    const float lo_ = __shfl_xor_sync(0xffffffffu, l[g], 16);
    const float mm = fmaxf(m[g], mo);
    const float c0 = m[g] == -INFINITY ? 0.f : __expf(m[g] - mm);
    const float c1 = mo == -INFINITY ? 0.f : __expf(mo - mm);
    if (lane == 0) {
      s_m[warp][g] = mm;
      s_l[warp][g] = l[g] * c0 + lo_ * c1;
    }
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float ao = __shfl_xor_sync(0xffffffffu, acc[g][v][j], 16);
        if (half == 0) s_acc[warp][g][(v * 16 + hl) * 8 + j] = acc[g][v][j] * c0 + ao * c1;
      }
  }
  __syncthreads();
  const int live = min(G, ratio - g0);
  for (int i = threadIdx.x; i < live * p.vdim; i += 256) {
    const int g = i / p.vdim, d = i % p.vdim;
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) mm = fmaxf(mm, s_m[w][g]);
    float ll = 0.f, a = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float c = s_m[w][g] == -INFINITY ? 0.f : __expf(s_m[w][g] - mm);
      ll += s_l[w][g] * c;
      a += s_acc[w][g][d] * c;
    }
    const int head = kvh * ratio + g0 + g;
    if (splits == 1) {
      ((T*)p.out)[((size_t)seq * p.heads + head) * p.vdim + d] = Cvt<T>::from(a / ll);
    } else {
      float* pp = partial + (((size_t)seq * p.heads + head) * splits + split) * (p.vdim + 2);
      pp[d] = a;
      if (d == 0) { pp[p.vdim] = mm; pp[p.vdim + 1] = ll; }
    }
  }
  if (splits == 1) return;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    int* tk = tickets + (size_t)seq * gridDim.x + blockIdx.x;
    s_last = atomicAdd(tk, 1) == splits - 1;
    if (s_last) *tk = 0;                              // ready for the next launch
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int i = threadIdx.x; i < live * p.vdim; i += 256) {
    const int g = i / p.vdim, d = i % p.vdim, head = kvh * ratio + g0 + g, w = p.vdim + 2;
    const float* pp = partial + ((size_t)seq * p.heads + head) * splits * w;
    float mm = -INFINITY;
    for (int s = 0; s < splits; ++s) mm = fmaxf(mm, __ldcg(pp + s * w + p.vdim));
    float ll = 0.f, a = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = __ldcg(pp + s * w + p.vdim);
      const float c = ms == -INFINITY ? 0.f : __expf(ms - mm);
      ll += __ldcg(pp + s * w + p.vdim + 1) * c;
      a += __ldcg(pp + s * w + d) * c;
    }
    ((T*)p.out)[((size_t)seq * p.heads + head) * p.vdim + d] = Cvt<T>::from(a / ll);
  }
}

// -------------------------------------------------------------------------------------------------
// Short prompt portions, and sizes the tcgen05 kernel (dz_window_attention_tc.cu) does not take, on
// warp-level MMAs: 64 query rows of one (sequence, head) per CTA, 16 per warp,
// 64 keys per step, double-buffered through cp.async.  Grid (row tiles, heads x tiles of DVP value
// columns, sequences).
// -------------------------------------------------------------------------------------------------
constexpr int kBM = 64, kBN = 64, kBiasSmem = 4096;

template <typename T, int DVP>
__global__ void __launch_bounds__(128)
window_prefill_kernel(AttnParams p, int dimp) {
  constexpr int NT = DVP / 8;
  extern __shared__ uint4 smem_raw[];
  const int seq = blockIdx.z, head = blockIdx.y % p.heads, v0 = (blockIdx.y / p.heads) * DVP;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_wait();
  pdl_launch();
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0, ctx = p.ctx_lens[seq];
  const int m0 = blockIdx.x * kBM;
  if (m0 >= qn) return;
  const int kvh = head / (p.heads / p.kv_heads);
  const int ldk = dimp + 8, ldv = DVP + 8;
  T* sq = reinterpret_cast<T*>(smem_raw);
  T* sk = sq + kBM * ldk;
  T* sv = sk + 2 * kBN * ldk;
  float* sb = reinterpret_cast<float*>(sv + 2 * kBN * ldv);
  const int vcols = min(DVP, p.vdim - v0);
  const int* table = p.block_tables + (size_t)seq * p.ring_blocks;
  const T* qkv = (const T*)p.qkv;
  const T* kv = (const T*)p.kv;
  const KeyRows kr(p, seq, q0, ctx);
  const int blen = p.bias ? p.bias_len : 0;
  const bool bias_in_smem = blen <= kBiasSmem;
  const float* gbias = p.bias ? p.bias + (size_t)head * p.bias_len : nullptr;

  if (p.dim < dimp || vcols < DVP) {                // padding columns read as zero
    const int words = (kBM * ldk + 2 * kBN * ldk + 2 * kBN * ldv) / 8;
    for (int i = tid; i < words; i += 128) smem_raw[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();
  }
  if (bias_in_smem)
    for (int i = tid; i < blen; i += 128) sb[i] = gbias[i] * kLog2e;

  const int r = tid >> 1, c0 = tid & 1;             // a pair of threads copies a row
  {
    const bool ok = m0 + r < qn;
    const T* src = qkv + (size_t)(q0 + (ok ? m0 + r : 0)) * p.row_stride + (size_t)head * p.dim;
    for (int c = c0; c < p.dim / 8; c += 2) cp_async16(sq + r * ldk + c * 8, src + c * 8, ok);
  }
  const int end = ctx + min(m0 + kBM, qn);          // keys [first, end)
  const int first = p.window > 0 ? max(0, ctx + m0 - p.window + 1) : 0;
  const int tiles = (end - first + kBN - 1) / kBN;

  auto load = [&](int buf, int t0) {
    const int t = t0 + r;
    const bool ok = t < end;
    const T *ks, *vs;
    if (!ok || t >= kr.first) {
      const T* row = kv + (size_t)(ok ? kr.row + t - kr.first : 0) * p.kv_stride;
      ks = row + p.k_off + (size_t)kvh * p.dim;
      vs = row + p.v_off + (size_t)kvh * p.vdim;
    } else {
      const size_t s = ring_slot(p, table, t) * p.kv_heads + kvh;
      ks = (const T*)p.k_cache + s * p.dim;
      vs = (const T*)p.v_cache + s * p.vdim;
    }
    T* dk = sk + (buf * kBN + r) * ldk;
    T* dv = sv + (buf * kBN + r) * ldv;
    for (int c = c0; c < p.dim / 8; c += 2) cp_async16(dk + c * 8, ks + c * 8, ok);
    for (int c = c0; c < vcols / 8; c += 2) cp_async16(dv + c * 8, vs + v0 + c * 8, ok);
  };

  float o[NT][4], mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
  if (p.sink) {
    mrow[0] = mrow[1] = p.sink[head] * kLog2e;
    lrow[0] = lrow[1] = (lane & 3) == 0 ? 1.f : 0.f;
  }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
  const int w0 = ctx + m0 + warp * 16;              // position of the warp's first row
  const int i0 = w0 + (lane >> 2), i1 = i0 + 8;
  const float scale2 = p.scale * kLog2e;

  load(0, first);
  cp_async_commit();
  for (int it = 0; it < tiles; ++it) {
    const int t0 = first + it * kBN, buf = it & 1;
    if (it + 1 < tiles) {
      load(buf ^ 1, t0 + kBN);
      cp_async_commit();
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    // keys no row of this warp may see: nothing to do (later rows of the tile, or an older window)
    const bool any = t0 <= w0 + 15 && (p.window <= 0 || t0 + kBN - 1 > w0 - p.window);
    if (any) {
      float s[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
      const T* aq = sq + (warp * 16 + (lane & 15)) * ldk + (lane >> 4) * 8;
      const T* bk = sk + (buf * kBN + (lane & 7) + ((lane >> 4) & 1) * 8) * ldk + ((lane >> 3) & 1) * 8;
      for (int kk = 0; kk < dimp; kk += 16) {
        uint32_t a[4];
        ldsm4(a, aq + kk);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t b[4];
          ldsm4(b, bk + j * 16 * ldk + kk);
          mma16816<T>(s[2 * j], a, b[0], b[1]);
          mma16816<T>(s[2 * j + 1], a, b[2], b[3]);
        }
      }
      // scale + bias, in units of log2
      const int near = w0 - (t0 + kBN - 1);         // smallest distance in the tile
      if (blen == 0 || near >= blen - 1) {
        const float c = blen == 0 ? 0.f : gbias[blen - 1] * kLog2e;
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) s[i][j] = fmaf(s[i][j], scale2, c);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int t = t0 + i * 8 + (lane & 3) * 2 + (j & 1);
            const int d = min(max((j < 2 ? i0 : i1) - t, 0), blen - 1);
            s[i][j] = fmaf(s[i][j], scale2, bias_in_smem ? sb[d] : gbias[d] * kLog2e);
          }
      }
      if (near < 0 || (p.window > 0 && w0 + 15 - t0 >= p.window)) {
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int t = t0 + i * 8 + (lane & 3) * 2 + (j & 1), d = (j < 2 ? i0 : i1) - t;
            if (d < 0 || (p.window > 0 && d >= p.window)) s[i][j] = -INFINITY;
          }
      }
      float corr[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < 8; ++i) mx = fmaxf(mx, fmaxf(s[i][2 * h], s[i][2 * h + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float mn = fmaxf(mrow[h], mx), ms = mn == -INFINITY ? 0.f : mn;
        corr[h] = exp2f(mrow[h] - ms);
        mrow[h] = mn;
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          s[i][2 * h] = exp2f(s[i][2 * h] - ms);
          s[i][2 * h + 1] = exp2f(s[i][2 * h + 1] - ms);
          sum += s[i][2 * h] + s[i][2 * h + 1];
        }
        lrow[h] = lrow[h] * corr[h] + sum;           // this lane's columns; lanes are summed at the end
      }
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        o[i][0] *= corr[0];
        o[i][1] *= corr[0];
        o[i][2] *= corr[1];
        o[i][3] *= corr[1];
      }
      const T* bv = sv + (buf * kBN + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + ((lane >> 4) & 1) * 8;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t hi[4], lo[4];
        split_pair<T>(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
        split_pair<T>(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
        split_pair<T>(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
        split_pair<T>(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int i = 0; i < NT; i += 2) {
          uint32_t b[4];
          ldsm4_t(b, bv + kk * 16 * ldv + i * 8);
          mma16816<T>(o[i], hi, b[0], b[1]);
          mma16816<T>(o[i + 1], hi, b[2], b[3]);
          mma16816<T>(o[i], lo, b[0], b[1]);
          mma16816<T>(o[i + 1], lo, b[2], b[3]);
        }
      }
    }
    __syncthreads();                                // the buffer is loaded again two steps on
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    float l = lrow[h];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    const float inv = 1.f / l;
    const int row = m0 + warp * 16 + (lane >> 2) + 8 * h;
    if (row < qn) {
      T* op = (T*)p.out + (size_t)(q0 + row) * p.heads * p.vdim + (size_t)head * p.vdim + v0;
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int c = i * 8 + (lane & 3) * 2;
        if (c < vcols) *reinterpret_cast<uint32_t*>(op + c) = Cvt<T>::down(o[i][2 * h] * inv, o[i][2 * h + 1] * inv);
      }
    }
  }
}

template <typename T, int DVP>
int run_prefill(const AttnParams& p, int num_seqs, int max_q, int dimp, size_t smem, cudaStream_t st) {
  const dim3 grid((max_q + kBM - 1) / kBM, p.heads * ((p.vdim + DVP - 1) / DVP), num_seqs);
  DZ_CUDA_OK(allow_smem(window_prefill_kernel<T, DVP>, smem));
  DZ_CUDA_OK(launch_ex(window_prefill_kernel<T, DVP>, grid, dim3(128), smem, 1, st, p, dimp));
  return DZ_OK;
}

template <typename T, int G>
int run_decode_g(const AttnParams& p, dim3 grid, int splits, float* partial, int* tickets, cudaStream_t st) {
  const int nk = (p.dim + 127) / 128, nv = (p.vdim + 127) / 128;
  if (nk == 1 && nv == 1)
    DZ_CUDA_OK(launch_pdl(window_decode_kernel<T, G, 1, 1>, grid, dim3(256), st, p, splits, partial, tickets));
  else if (nk == 1)
    DZ_CUDA_OK(launch_pdl(window_decode_kernel<T, G, 1, 2>, grid, dim3(256), st, p, splits, partial, tickets));
  else if (nv == 1)
    DZ_CUDA_OK(launch_pdl(window_decode_kernel<T, G, 2, 1>, grid, dim3(256), st, p, splits, partial, tickets));
  else
    DZ_CUDA_OK(launch_pdl(window_decode_kernel<T, G, 2, 2>, grid, dim3(256), st, p, splits, partial, tickets));
  return DZ_OK;
}

constexpr int kTcMinRows = 64;                 // portions up to this many rows stay off the 256-row kernel
constexpr size_t kAttnStatusBytes = 256;        // workspace: [status word | tickets | partials]

int decode_group(int heads, int kv_heads) {
  const int r = heads / kv_heads;
  return r == 1 ? 1 : r == 2 ? 2 : 4;
}
int decode_grid_x(int heads, int kv_heads) {
  const int r = heads / kv_heads, g = decode_group(heads, kv_heads);
  return kv_heads * ((r + g - 1) / g);
}

// The 16-byte copies of the fast kernels need 8-element rows everywhere.
bool fast_shapes(const AttnParams& p, int dtype) {
  return dtype != DZ_DTYPE_F32 && p.dim % 8 == 0 && p.vdim % 8 == 0 && p.row_stride % 8 == 0 && p.k_off % 8 == 0 &&
         p.v_off % 8 == 0 && p.v_row % 8 == 0 && p.kv_stride % 8 == 0 && aligned16(p.qkv) && aligned16(p.out) &&
         aligned16(p.k_cache) && aligned16(p.v_cache) && aligned16(p.kv);
}

}  // namespace

int launch_attention_any(const AttnParams& p, int num_seqs, int dtype, cudaStream_t st) {
  if (p.vdim > kAnyMaxV * kAnyThreads || p.dim > 8192 || p.heads > 65535) return DZ_ERR_SHAPE;
  DZ_DISPATCH(dtype, DZ_CUDA_OK(launch_ex(attention_any_kernel<T>, dim3(p.rows, p.heads), dim3(kAnyThreads),
                                          (size_t)p.dim * 4, 1, st, p, num_seqs)));
  return DZ_OK;
}

}  // namespace dz

using namespace dz;

extern "C" {

int dz_qk_norm(void* qkv, int64_t row_stride, int q_width, int k_width, int v_width, const float* wq, const float* wk,
               float eps, void* k_cache, void* v_cache, const int64_t* slot_mapping, int M, int dtype, void* stream) {
  if (!qkv || !wq || !wk || M < 0 || q_width <= 0 || k_width <= 0 || v_width <= 0 ||
      row_stride < (int64_t)q_width + k_width + v_width || (slot_mapping && (!k_cache || !v_cache)))
    return DZ_ERR_INVALID_ARG;
  if (M == 0) return DZ_OK;
  const bool vec = q_width % 8 == 0 && k_width % 8 == 0 && v_width % 8 == 0 && row_stride % 8 == 0 &&
                   aligned16(qkv) && aligned16(wq) && aligned16(wk) && aligned16(k_cache) && aligned16(v_cache);
  DZ_DISPATCH(dtype, DZ_CUDA_OK(launch_pdl(vec ? qk_norm_kernel<T, 8> : qk_norm_kernel<T, 1>, dim3(M, 2), dim3(256),
                                           (cudaStream_t)stream, (T*)qkv, row_stride, q_width, k_width, v_width, wq,
                                           wk, eps, (T*)k_cache, (T*)v_cache, (const long long*)slot_mapping)));
  return DZ_OK;
}

int dz_kv_append(const void* qkv, int64_t row_stride, int k_off, int k_width, int v_width, void* k_cache,
                 void* v_cache, const int64_t* slot_mapping, int M, int dtype, void* stream) {
  if (!qkv || !k_cache || !v_cache || !slot_mapping || M < 0 || k_width <= 0 || v_width <= 0 || k_off < 0 ||
      row_stride < (int64_t)k_off + k_width + v_width)
    return DZ_ERR_INVALID_ARG;
  if (M == 0) return DZ_OK;
  const bool vec = k_off % 8 == 0 && k_width % 8 == 0 && v_width % 8 == 0 && row_stride % 8 == 0 && aligned16(qkv) &&
                   aligned16(k_cache) && aligned16(v_cache);
  DZ_DISPATCH(dtype, DZ_CUDA_OK(launch_pdl(vec ? kv_append_kernel<T, 8> : kv_append_kernel<T, 1>, dim3(M), dim3(128),
                                           (cudaStream_t)stream, (const T*)qkv, row_stride, k_off, k_width, v_width,
                                           (T*)k_cache, (T*)v_cache, (const long long*)slot_mapping)));
  return DZ_OK;
}

size_t dz_window_attention_workspace_bytes(int num_seqs, int heads, int kv_heads, int vdim, int splits) {
  if (num_seqs <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || vdim <= 0) return 0;
  if (splits <= 1) return kAttnStatusBytes;
  return kAttnStatusBytes + kTicketBytes + (size_t)num_seqs * heads * splits * (vdim + 2) * 4;
}

int dz_window_attention(const dz_window_attention_args* a, void* stream) {
  const bool own = a && a->kv;                     // keys and values in rows of their own
  if (!a || !a->qkv || !a->out || !a->q_starts || !a->ctx_lens) return DZ_ERR_INVALID_ARG;
  if (own ? (!a->kv_starts || a->kv_rows <= 0 || a->decode) : (!a->k_cache || !a->v_cache || !a->block_tables))
    return DZ_ERR_INVALID_ARG;
  if (a->num_seqs < 0 || a->rows < 0 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 ||
      a->vdim <= 0 || (!own && (a->ring_blocks <= 0 || a->block_size <= 0)) || a->splits < 1 || a->splits > 64 ||
      (a->bias && a->bias_len <= 0) || !is_float_dtype(a->dtype))
    return DZ_ERR_INVALID_ARG;
  const int64_t kv_stride = own ? a->kv_stride : a->row_stride;
  if (a->k_off < 0 || a->v_off < 0 || kv_stride < (int64_t)a->v_off + (int64_t)a->kv_heads * a->vdim ||
      kv_stride < (int64_t)a->k_off + (int64_t)a->kv_heads * a->dim ||
      a->row_stride < (int64_t)a->heads * a->dim)
    return DZ_ERR_INVALID_ARG;
  if (a->num_seqs == 0 || a->rows == 0) return DZ_OK;
  if (a->num_seqs > 65535 || (a->decode && a->rows != a->num_seqs)) return DZ_ERR_INVALID_ARG;
  AttnParams p = {a->qkv, a->row_stride, a->k_off, a->v_off, a->out, a->k_cache, a->v_cache, a->vdim, a->block_tables,
                  a->ring_blocks, a->block_size, a->q_starts, a->ctx_lens, a->heads, a->kv_heads, a->dim, a->vdim,
                  a->scale, a->window, a->bias, a->bias_len, a->rows, a->sink, own ? kKeysRows : kKeysSplit,
                  own ? a->kv : a->qkv, kv_stride, a->kv_starts, own ? a->kv_rows : a->rows, nullptr};
  if (a->workspace && a->workspace_bytes >= kAttnStatusBytes) p.status = (int*)a->workspace;
  cudaStream_t st = (cudaStream_t)stream;
  if (!fast_shapes(p, a->dtype)) return launch_attention_any(p, a->num_seqs, a->dtype, st);
  if (a->decode && a->dim <= 256 && a->vdim <= 256) {
    float* partial = nullptr;
    int* tickets = nullptr;
    if (a->splits > 1) {
      if (!a->workspace || a->workspace_bytes < dz_window_attention_workspace_bytes(a->num_seqs, a->heads, a->kv_heads,
                                                                                    a->vdim, a->splits))
        return DZ_ERR_WORKSPACE;
      tickets = (int*)((uint8_t*)a->workspace + kAttnStatusBytes);
      partial = (float*)((uint8_t*)tickets + kTicketBytes);
      if ((int64_t)a->num_seqs * decode_grid_x(a->heads, a->kv_heads) > kMaxTickets) return DZ_ERR_TOO_LARGE;
    }
    const dim3 grid(decode_grid_x(a->heads, a->kv_heads), a->num_seqs, a->splits);
    const int g = decode_group(a->heads, a->kv_heads);
    DZ_DISPATCH16(a->dtype, return g == 1   ? run_decode_g<T, 1>(p, grid, a->splits, partial, tickets, st)
                                   : g == 2 ? run_decode_g<T, 2>(p, grid, a->splits, partial, tickets, st)
                                            : run_decode_g<T, 4>(p, grid, a->splits, partial, tickets, st));
  }
  const int max_q = a->max_q > 0 ? a->max_q : a->rows;
  if (max_q > kTcMinRows && window_prefill_tc_supported(p, a->dtype))
    return launch_window_prefill_tc(p, a->num_seqs, max_q, a->dtype, st);
  const int dimp = (a->dim + 15) / 16 * 16;
  const int dvp = a->vdim <= 64 ? 64 : a->vdim <= 96 ? 96 : a->vdim <= 128 ? 128 : a->vdim <= 192 ? 192 : 256;
  const size_t bias_bytes = a->bias && a->bias_len <= kBiasSmem ? (size_t)a->bias_len * 4 : 0;
  const size_t smem = ((size_t)(kBM + 2 * kBN) * (dimp + 8) + (size_t)2 * kBN * (dvp + 8)) * 2 + bias_bytes;
  if (smem > kMaxDynSmem || (int64_t)a->heads * ((a->vdim + dvp - 1) / dvp) > 65535)
    return launch_attention_any(p, a->num_seqs, a->dtype, st);
  DZ_DISPATCH16(a->dtype, switch (dvp) {
    case 64: return run_prefill<T, 64>(p, a->num_seqs, max_q, dimp, smem, st);
    case 96: return run_prefill<T, 96>(p, a->num_seqs, max_q, dimp, smem, st);
    case 128: return run_prefill<T, 128>(p, a->num_seqs, max_q, dimp, smem, st);
    case 192: return run_prefill<T, 192>(p, a->num_seqs, max_q, dimp, smem, st);
    default: return run_prefill<T, 256>(p, a->num_seqs, max_q, dimp, smem, st);
  });
  return DZ_OK;
}

}  // extern "C"
