// Linear attention with a constant decay per head ("Lightning Attention-2: A Free Lunch for Handling
// Unlimited Sequence Lengths in Large Language Models", Qin et al.).  Per head, with decay w:
//
//   S_t = w S_(t-1) + k_t v_t^T      o_t = S_t^T q_t      q, k, v = SiLU of the projection rows
//
// and after it, over all heads of a token together, out = RMS norm(o) * weight * sigmoid(g).  S [dim, vdim]
// lives in a 32-bit pool, one slot per sequence; a sequence without context starts from zero without its
// slot being read.
//
// Two kernels.  The recurrent one streams the state once per token; it serves decoding, where its last
// CTA of a sequence also does the norm and the gate, and the 32-bit type.  The chunkwise one takes 64
// tokens at a time on the tensor cores for prompt portions.
#include "dz_elem.cuh"

namespace dz {
namespace {

constexpr int kL = 64, kPowers = kL + 1;

struct LightningParams {
  const void* x;                         // rows [q (heads*dim) | k (heads*dim) | v | g (heads*vdim)]
  int64_t row_stride;
  int k_off, v_off, g_off;
  const float* powers;                   // [heads, kPowers] w^0 ... w^64
  const float* norm_w;                   // [heads * vdim]
  float eps;
  void* out;                             // [rows, heads * vdim]
  float* o;                              // [rows, heads * vdim] recurrent kernel: the output before the norm
  float* S;
  const int* slots;
  const int* q_starts;
  const int* ctx_lens;
  int heads, dim, vdim;
  int* tickets;                          // [sequences], or nullptr: the norm is another launch's
};

__device__ __forceinline__ float silu_exact(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }

// out = o / sqrt(mean(o^2) + eps) * w * sigmoid(g) over the n columns of one row, by one CTA
template <typename T, typename I, int VEC>
__device__ __forceinline__ void norm_gate_row(const I* o, const T* g, const float* w, float eps, T* out, int n, float* part) {
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < n; c += blockDim.x * VEC) {
    if constexpr (VEC == 8) {
      float f[8];
      load8<I>(o + c, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
    } else {
      const float f = Cvt<I>::one(o[c]);
      ss += f * f;
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, part) / (float)n + eps);
  for (int c = threadIdx.x * VEC; c < n; c += blockDim.x * VEC) {
    if constexpr (VEC == 8) {
      float f[8], e[8], v[8];
      load8<I>(o + c, f);
      load8<T>(g + c, e);
      load8<float>(w + c, v);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = f[j] * inv * v[j] / (1.f + (sizeof(T) == 4 ? expf(-e[j]) : __expf(-e[j])));
      store8<T>(out + c, f);
    } else {
      out[c] = Cvt<T>::from(Cvt<I>::one(o[c]) * inv * w[c] / (1.f + expf(-Cvt<T>::one(g[c]))));
    }
  }
}

template <typename T, typename I, int VEC>
__global__ void __launch_bounds__(256)
row_norm_gate_kernel(const I* o, const T* __restrict__ g, int64_t g_stride, const float* __restrict__ w, float eps, T* out,
                     int n) {
  __shared__ float s_part[8];
  pdl_wait();
  pdl_launch();
  const size_t row = blockIdx.x;
  norm_gate_row<T, I, VEC>(o + row * n, g + row * g_stride, w, eps, out + row * n, n, s_part);
}

// -------------------------------------------------------------------------------------------------
// Recurrent form.  A CTA owns columns [x vt, (x + 1) vt) of S of one (head, sequence), streamed from and
// to the pool.  Grid (column slices, heads, sequences).
// -------------------------------------------------------------------------------------------------
constexpr int kRecThreads = 256, kRowsInFlight = 8;

template <typename T, int VEC>
__global__ void __launch_bounds__(kRecThreads, 3)
lightning_recurrent_kernel(LightningParams p, int vt) {
  extern __shared__ float sm[];
  __shared__ float s_part[kRecThreads / 32];
  __shared__ int s_last;
  const int head = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  float* sq = sm;
  float* sk = sq + p.dim;
  float* sv = sk + p.dim;
  float* so = sv + vt;                              // [row groups, vt]
  const int v0 = blockIdx.x * vt, nv = max(0, min(vt, p.vdim - v0));
  const int cg_n = vt / VEC, rg_n = kRecThreads / cg_n;         // column groups, row groups
  const int cgi = tid % cg_n, rgi = tid / cg_n;
  const bool mine = rgi < rg_n && cgi * VEC < nv;
  pdl_wait();
  pdl_launch();
  const int q0 = p.q_starts[seq], tn = p.q_starts[seq + 1] - q0, ctx = p.ctx_lens[seq], slot = p.slots[seq];
  const int n = p.heads * p.vdim;
  const float keep = p.powers[(size_t)head * kPowers + 1];
  float* S = p.S + ((size_t)slot * p.heads + head) * p.dim * p.vdim + v0;

  // rows d0, d0 + rg_n, ... of this thread's columns of S (zero where there are none)
  float s[kRowsInFlight][VEC];
  auto load_rows = [&](int d0, bool zero) {
#pragma unroll
    for (int u = 0; u < kRowsInFlight; ++u) {
      const int d = d0 + u * rg_n;
#pragma unroll
      for (int j = 0; j < VEC; ++j) s[u][j] = 0.f;
      if (mine && d < p.dim && !zero) {
        const float* src = S + (size_t)d * p.vdim + cgi * VEC;
        if constexpr (VEC == 4) {
          const float4 x = *reinterpret_cast<const float4*>(src);
          s[u][0] = x.x; s[u][1] = x.y; s[u][2] = x.z; s[u][3] = x.w;
        } else {
          s[u][0] = *src;
        }
      }
    }
  };

  for (int t = 0; t < tn; ++t) {
    const T* row = (const T*)p.x + (size_t)(q0 + t) * p.row_stride;
    const bool zero = ctx == 0 && t == 0;           // the state before this token is zero
    load_rows(rgi, zero);                           // on their way while q, k and v are read
    for (int d = tid; d < p.dim; d += kRecThreads) {
      sq[d] = silu_exact(Cvt<T>::one(row[(size_t)head * p.dim + d]));
      sk[d] = silu_exact(Cvt<T>::one(row[p.k_off + (size_t)head * p.dim + d]));
    }
    for (int c = tid; c < nv; c += kRecThreads)
      sv[c] = silu_exact(Cvt<T>::one(row[p.v_off + (size_t)head * p.vdim + v0 + c]));
    __syncthreads();
    float o[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = 0.f;
    if (mine) {
      float v[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = sv[cgi * VEC + j];
      for (int d0 = rgi; d0 < p.dim; d0 += rg_n * kRowsInFlight) {
        if (d0 != rgi) load_rows(d0, zero);
#pragma unroll
        for (int u = 0; u < kRowsInFlight; ++u) {
          const int d = d0 + u * rg_n;
          if (d < p.dim) {
            const float kd = sk[d], qd = sq[d];
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
              s[u][j] = s[u][j] * keep + kd * v[j];
              o[j] += s[u][j] * qd;
            }
            float* dst = S + (size_t)d * p.vdim + cgi * VEC;
            if constexpr (VEC == 4) *reinterpret_cast<float4*>(dst) = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
            else *dst = s[u][0];
          }
        }
      }
    }
    if (rgi < rg_n) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) so[rgi * vt + cgi * VEC + j] = o[j];
    }
    __syncthreads();
    float* dst = p.o + (size_t)(q0 + t) * n + (size_t)head * p.vdim + v0;
    for (int c = tid; c < nv; c += kRecThreads) {
      float a = 0.f;
      for (int g = 0; g < rg_n; ++g) a += so[g * vt + c];
      dst[c] = a;
    }
    __syncthreads();
  }
  if (!p.tickets) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    s_last = atomicAdd(p.tickets + seq, 1) == (int)(gridDim.x * gridDim.y) - 1;
    if (s_last) p.tickets[seq] = 0;                 // ready for the next launch
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int t = 0; t < tn; ++t) {
    const float* o = p.o + (size_t)(q0 + t) * n;
    const T* g = (const T*)p.x + (size_t)(q0 + t) * p.row_stride + p.g_off;
    T* out = (T*)p.out + (size_t)(q0 + t) * n;
    if (VEC == 4 && n % 8 == 0 && p.g_off % 8 == 0 && p.row_stride % 8 == 0) {
      norm_gate_row<T, float, 8>(o, g, p.norm_w, p.eps, out, n, s_part);
    } else {
      norm_gate_row<T, float, 1>(o, g, p.norm_w, p.eps, out, n, s_part);
    }
  }
}

// -------------------------------------------------------------------------------------------------
// Chunkwise form, 16-bit activations.  Inside a chunk of L tokens, t = 0 ... L - 1,
//   o_t = sum_{s <= t} w^(t-s) (q_t.k_s) v_s + w^(t+1) q_t S_start
//   S_end = w^L S_start + sum_s w^(L-1-s) k_s v_s^T.
// A CTA owns VT value columns of one (head, sequence) and walks the chunks.  Eight warps bring a chunk in
// while the one before is worked on: rows from memory, SiLU, rounded to 16 bits, v also times its power
// of w.  Eight others multiply; their slice of S stays in registers in 32 bits as accumulators of the
// update.  32-bit operands (S, weighted scores, weighted v) enter the MMAs as hi + lo pairs.  A warp owns
// NTW groups of eight of k's columns (64 NTW >= dim).  Writes o before the norm.  Grid (tiles of VT
// columns, heads, sequences).
// -------------------------------------------------------------------------------------------------
constexpr int kMmaThreads = 256, kLoadThreads = 256, kChunkThreads = kMmaThreads + kLoadThreads;

__device__ __forceinline__ void bar_sync(int id, int count) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(count) : "memory"); }
__device__ __forceinline__ void bar_arrive(int id, int count) {
  __threadfence_block();
  asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(count) : "memory");
}

template <int VT> __host__ __device__ constexpr int chunk_ldv() { return VT + 8; }
template <int VT> __host__ __device__ inline int stage_elems(int dimp) { return kL * (2 * (dimp + 8) + 3 * chunk_ldv<VT>()); }

template <typename T> __device__ __forceinline__ uint4 silu8(const uint4& v) {
  uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = Cvt<T>::up(w[j]);
    w[j] = Cvt<T>::down(silu_fast(f.x), silu_fast(f.y));
  }
  return make_uint4(w[0], w[1], w[2], w[3]);
}

template <typename T, int VT, int NTW>
__global__ void __launch_bounds__(kChunkThreads, 1)
lightning_chunk_kernel(LightningParams p, int dimp, int stages) {
  constexpr int NT = VT / 16, MT = VT / 16, LDV = chunk_ldv<VT>();      // output: a warp has 16 rows, half of the columns
  extern __shared__ uint4 smem_raw[];
  __shared__ float s_pw[kPowers];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int head = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * VT;
  pdl_wait();
  pdl_launch();
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0;
  if (qn <= 0) return;
  const int ctx = p.ctx_lens[seq], slot = p.slots[seq];
  const int vcols = min(VT, p.vdim - v0);
  const int ldk = dimp + 8, lds = dimp + 8, stage = stage_elems<VT>(dimp);
  T* base_s = reinterpret_cast<T*>(smem_raw);
  T* sh = base_s + stages * stage;                                // S transposed, hi and lo: [VT][lds]
  T* sl = sh + VT * lds;
  const int words = (stages * stage + 2 * VT * lds) / 8;
  for (int i = tid; i < words; i += kChunkThreads) smem_raw[i] = make_uint4(0, 0, 0, 0);
  for (int i = tid; i < kPowers; i += kChunkThreads) s_pw[i] = p.powers[(size_t)head * kPowers + i];
  __syncthreads();
  const int chunks = (qn + kL - 1) / kL;
  const T* x = (const T*)p.x;

  if (warp >= kMmaThreads / 32) {
    // ---- copies ----
    const int lt = tid - kMmaThreads, nv = p.dim / 8, nw = vcols / 8;
    for (int it = 0; it < chunks; ++it) {
      const int st = stages == 2 ? it & 1 : 0, base = it * kL, len = min(kL, qn - base);
      T* sq = base_s + st * stage;
      T* sk = sq + kL * ldk;
      T* sv = sk + kL * ldk;
      T* wh = sv + kL * LDV;
      T* wl = wh + kL * LDV;
      const T* rows = x + (size_t)(q0 + base) * p.row_stride;
      if (it >= stages) bar_sync(4 + st, kChunkThreads);
      constexpr int U = 4;                                         // loads of each kind in flight
      for (int i0 = lt; i0 < kL * nv; i0 += U * kLoadThreads) {
        uint4 a[U], b[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int i = i0 + u * kLoadThreads, r = i / nv, c = i - r * nv;
          a[u] = b[u] = make_uint4(0, 0, 0, 0);
          if (r < len) {                                           // absent tokens are zero
            const T* src = rows + (size_t)r * p.row_stride + (size_t)head * p.dim + c * 8;
            a[u] = *reinterpret_cast<const uint4*>(src);
            b[u] = *reinterpret_cast<const uint4*>(src + p.k_off);
          }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int i = i0 + u * kLoadThreads, r = i / nv, c = i - r * nv;
          if (r < kL) {
            *reinterpret_cast<uint4*>(sq + r * ldk + c * 8) = silu8<T>(a[u]);
            *reinterpret_cast<uint4*>(sk + r * ldk + c * 8) = silu8<T>(b[u]);
          }
        }
      }
      for (int i = lt; i < kL * nw; i += kLoadThreads) {
        const int r = i / nw, c = i - r * nw;
        uint4 a = make_uint4(0, 0, 0, 0);
        if (r < len)
          a = silu8<T>(*reinterpret_cast<const uint4*>(rows + (size_t)r * p.row_stride + p.v_off + (size_t)head * p.vdim +
                                                       v0 + c * 8));
        const float w = r < len ? s_pw[len - 1 - r] : 0.f;
        const uint32_t in[4] = {a.x, a.y, a.z, a.w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = Cvt<T>::up(in[j]);
          split_pair<T>(f.x * w, f.y * w, hi[j], lo[j]);
        }
        *reinterpret_cast<uint4*>(sv + r * LDV + c * 8) = a;
        *reinterpret_cast<uint4*>(wh + r * LDV + c * 8) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(wl + r * LDV + c * 8) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      bar_arrive(2 + st, kChunkThreads);
    }
    return;
  }

  // ---- products ----
  const int rw = warp & 3, cw = (warp >> 2) * (VT / 2);
  float* S = p.S + ((size_t)slot * p.heads + head) * p.dim * p.vdim + v0;
  // The state: rows mt * 16 + lane / 4 (+ 8), columns nt * 8 + 2 (lane % 4) (+ 1) of the transposed slice,
  // nt = warp + 8 i.
  float acc[MT][NTW][4];
  const int col0 = warp * 8 + (lane & 3) * 2;
  auto each = [&](auto&& fn) {                       // fn(value, dim index, value column)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = col0 + i * 64 + (e & 1), v = mt * 16 + (lane >> 2) + (e >> 1) * 8;
          if (d < p.dim && v < vcols) fn(acc[mt][i][e], d, v);
        }
  };
  auto publish = [&]() {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int i = 0; i < NTW; ++i)
        if (warp + 8 * i < dimp / 8) {
#pragma unroll
          for (int e = 0; e < 4; e += 2) {
            const int at = (mt * 16 + (lane >> 2) + e * 4) * lds + col0 + i * 64;
            split_pair<T>(acc[mt][i][e], acc[mt][i][e + 1], *reinterpret_cast<uint32_t*>(sh + at),
                          *reinterpret_cast<uint32_t*>(sl + at));
          }
        }
  };
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[mt][i][e] = 0.f;
  bool have_state = ctx > 0;
  if (have_state) {
    each([&](float& a, int d, int v) { a = S[(size_t)d * p.vdim + v]; });
    publish();
    bar_sync(1, kMmaThreads);
  }
  for (int it = 0; it < chunks; ++it) {
    const int st = stages == 2 ? it & 1 : 0, base = it * kL, len = min(kL, qn - base);
    const T* sq = base_s + st * stage;
    const T* sk = sq + kL * ldk;
    const T* sv = sk + kL * ldk;
    const T* wh = sv + kL * LDV;
    const T* wl = wh + kL * LDV;
    bar_sync(2 + st, kChunkThreads);
    const int r0 = rw * 16 + (lane >> 2), r1 = r0 + 8;
    if (rw * 16 < len) {
      float o[NT][4];
#pragma unroll
      for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
      float s[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
      const T* aq = sq + (rw * 16 + (lane & 15)) * ldk + (lane >> 4) * 8;
      const T* bk = sk + ((lane & 7) + ((lane >> 4) & 1) * 8) * ldk + ((lane >> 3) & 1) * 8;
      for (int kk = 0; kk < dimp; kk += 16) {
        uint32_t a[4];
        ldsm4(a, aq + kk);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (j <= rw) {                             // keys up to the warp's last row
            uint32_t b[4];
            ldsm4(b, bk + j * 16 * ldk + kk);
            mma16816<T>(s[2 * j], a, b[0], b[1]);
            mma16816<T>(s[2 * j + 1], a, b[2], b[3]);
          }
        }
        if (have_state) {
          uint32_t bh[NT / 2][4], bl[NT / 2][4];
#pragma unroll
          for (int i = 0; i < NT / 2; ++i) {
            const int at = (cw + i * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * lds + ((lane >> 3) & 1) * 8 + kk;
            ldsm4(bh[i], sh + at);
            ldsm4(bl[i], sl + at);
          }
#pragma unroll
          for (int i = 0; i < NT; ++i) mma16816<T>(o[i], a, bh[i / 2][2 * (i & 1)], bh[i / 2][2 * (i & 1) + 1]);
#pragma unroll
          for (int i = 0; i < NT; ++i) mma16816<T>(o[i], a, bl[i / 2][2 * (i & 1)], bl[i / 2][2 * (i & 1) + 1]);
        }
      }
      const float in0 = s_pw[r0 + 1], in1 = s_pw[r1 + 1];
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        o[i][0] *= in0;
        o[i][1] *= in0;
        o[i][2] *= in1;
        o[i][3] *= in1;
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int n = (j < 2 ? r0 : r1) - (i * 8 + (lane & 3) * 2 + (j & 1));
          s[i][j] *= n >= 0 ? s_pw[n] : 0.f;
        }
      const T* bv = sv + ((lane & 7) + ((lane >> 3) & 1) * 8) * LDV + ((lane >> 4) & 1) * 8;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        if (kk <= rw) {
          uint32_t hi[4], lo[4];
          split_pair<T>(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
          split_pair<T>(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
          split_pair<T>(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
          split_pair<T>(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
          for (int i = 0; i < NT; i += 2) {
            uint32_t b[4];
            ldsm4_t(b, bv + kk * 16 * LDV + cw + i * 8);
            mma16816<T>(o[i], hi, b[0], b[1]);
            mma16816<T>(o[i + 1], hi, b[2], b[3]);
            mma16816<T>(o[i], lo, b[0], b[1]);
            mma16816<T>(o[i + 1], lo, b[2], b[3]);
          }
        }
      }
      T* op = (T*)p.out + (size_t)(q0 + base) * p.heads * p.vdim + (size_t)head * p.vdim + v0;
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int c = cw + i * 8 + (lane & 3) * 2;
        if (c < vcols) {
          if (r0 < len) *reinterpret_cast<uint32_t*>(op + (size_t)r0 * p.heads * p.vdim + c) = Cvt<T>::down(o[i][0], o[i][1]);
          if (r1 < len) *reinterpret_cast<uint32_t*>(op + (size_t)r1 * p.heads * p.vdim + c) = Cvt<T>::down(o[i][2], o[i][3]);
        }
      }
    }
    const float decay = s_pw[len];
    uint32_t kb[NTW][8];                             // this warp's columns of k, all 64 tokens
#pragma unroll
    for (int i = 0; i < NTW; ++i)
      if (warp + 8 * i < dimp / 8) {
        uint32_t b[4];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          ldsm4_t(b, sk + (j * 32 + lane) * ldk + (warp + 8 * i) * 8);
#pragma unroll
          for (int e = 0; e < 4; ++e) kb[i][4 * j + e] = b[e];
        }
      }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {                // 16 value columns
#pragma unroll
      for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[mt][i][e] *= decay;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t hi[4], lo[4];
        const int at = (kk * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * LDV + mt * 16 + ((lane >> 3) & 1) * 8;
        ldsm4_t(hi, wh + at);
        ldsm4_t(lo, wl + at);
#pragma unroll
        for (int i = 0; i < NTW; ++i)
          if (warp + 8 * i < dimp / 8) mma16816<T>(acc[mt][i], hi, kb[i][2 * kk], kb[i][2 * kk + 1]);
#pragma unroll
        for (int i = 0; i < NTW; ++i)
          if (warp + 8 * i < dimp / 8) mma16816<T>(acc[mt][i], lo, kb[i][2 * kk], kb[i][2 * kk + 1]);
      }
    }
    if (it + stages < chunks) bar_arrive(4 + st, kChunkThreads);
    if (it + 1 < chunks) {
      bar_sync(1, kMmaThreads);                      // the old state has been read
      publish();
      bar_sync(1, kMmaThreads);
    }
    have_state = true;
  }
  each([&](float& a, int d, int v) { S[(size_t)d * p.vdim + v] = a; });
}

template <int VT> size_t chunk_smem(int dimp, int stages) {
  return ((size_t)stages * stage_elems<VT>(dimp) + 2 * VT * (dimp + 8)) * 2;
}

template <typename T, int VT, int NTW>
int run_chunk_n(const LightningParams& p, int num_seqs, int dimp, cudaStream_t st) {
  const int stages = chunk_smem<VT>(dimp, 2) <= kMaxDynSmem ? 2 : 1;
  const size_t smem = chunk_smem<VT>(dimp, stages);
  DZ_CUDA_OK(allow_smem(lightning_chunk_kernel<T, VT, NTW>, smem));
  DZ_CUDA_OK(launch_ex(lightning_chunk_kernel<T, VT, NTW>, dim3((p.vdim + VT - 1) / VT, p.heads, num_seqs),
                       dim3(kChunkThreads), smem, 1, st, p, dimp, stages));
  return DZ_OK;
}
template <typename T>
int run_chunk(const LightningParams& p, int num_seqs, int dimp, cudaStream_t st) {
  const bool wide = p.vdim > 32;
  if (dimp <= 64) return wide ? run_chunk_n<T, 64, 1>(p, num_seqs, dimp, st) : run_chunk_n<T, 32, 1>(p, num_seqs, dimp, st);
  if (dimp <= 128) return wide ? run_chunk_n<T, 64, 2>(p, num_seqs, dimp, st) : run_chunk_n<T, 32, 2>(p, num_seqs, dimp, st);
  if (dimp <= 256) return run_chunk_n<T, 32, 4>(p, num_seqs, dimp, st);
  return run_chunk_n<T, 32, 8>(p, num_seqs, dimp, st);
}

template <typename T>
int run_recurrent(const LightningParams& p, int num_seqs, cudaStream_t st) {
  const bool vec = p.vdim % 4 == 0 && aligned16(p.S) && aligned16(p.x) && aligned16(p.out) && aligned16(p.norm_w);
  const int v = vec ? 4 : 1;
  // columns per CTA: a slice of S of at most 64 KB, and no more column groups than threads
  int c = 1;
  while (p.vdim > c * v && ((size_t)p.dim * ((p.vdim + c - 1) / c) * 4 > 64 * 1024 || (p.vdim + c - 1) / c > v * kRecThreads))
    c *= 2;
  const int vt = ((p.vdim + c - 1) / c + v - 1) / v * v, rg = kRecThreads / (vt / v);
  const size_t smem = ((size_t)2 * p.dim + vt + (size_t)rg * vt) * 4;
  if (smem > kMaxDynSmem) return DZ_ERR_SHAPE;
  const dim3 grid((p.vdim + vt - 1) / vt, p.heads, num_seqs);
  auto kern = vec ? lightning_recurrent_kernel<T, 4> : lightning_recurrent_kernel<T, 1>;
  DZ_CUDA_OK(allow_smem(kern, smem));
  DZ_CUDA_OK(launch_ex(kern, grid, dim3(kRecThreads), smem, 1, st, p, vt));
  return DZ_OK;
}

template <typename T, typename I>
int run_norm(const LightningParams& p, const I* o, int rows, cudaStream_t st) {
  const int n = p.heads * p.vdim;
  const bool vec = n % 8 == 0 && p.g_off % 8 == 0 && p.row_stride % 8 == 0 && aligned16(p.x) && aligned16(p.out) &&
                   aligned16(p.norm_w) && aligned16(o);
  DZ_CUDA_OK(launch_pdl(vec ? row_norm_gate_kernel<T, I, 8> : row_norm_gate_kernel<T, I, 1>, dim3(rows), dim3(256), st, o,
                        (const T*)p.x + p.g_off, p.row_stride, p.norm_w, p.eps, (T*)p.out, n));
  return DZ_OK;
}

}  // namespace
}  // namespace dz

using namespace dz;

extern "C" {

int dz_lightning_chunk_supported(int dim, int vdim, int dtype) {
  if (dtype != DZ_DTYPE_F16 && dtype != DZ_DTYPE_BF16) return 0;
  if (dim <= 0 || vdim <= 0 || dim % 8 || vdim % 8) return 0;
  const int dimp = (dim + 15) / 16 * 16;
  return dimp <= 512 && chunk_smem<32>(dimp, 1) <= kMaxDynSmem;
}

size_t dz_lightning_workspace_bytes(int rows, int num_seqs, int heads, int vdim, int chunkwise) {
  if (rows <= 0 || num_seqs <= 0 || heads <= 0 || vdim <= 0 || chunkwise) return 0;
  return kTicketBytes + (size_t)rows * heads * vdim * 4;
}

int dz_lightning(const dz_lightning_args* a, void* stream) {
  if (!a || !a->x || !a->powers || !a->norm_weight || !a->out || !a->S || !a->slots || !a->q_starts || !a->ctx_lens)
    return DZ_ERR_INVALID_ARG;
  if (a->num_seqs < 0 || a->num_seqs > 65535 || a->rows < 0 || a->heads <= 0 || a->heads > 65535 || a->dim <= 0 ||
      a->vdim <= 0 || !is_float_dtype(a->dtype))
    return DZ_ERR_INVALID_ARG;
  const int64_t qk = (int64_t)a->heads * a->dim, vv = (int64_t)a->heads * a->vdim;
  if (a->k_off < 0 || a->v_off < 0 || a->g_off < 0 || a->row_stride < qk || a->row_stride < a->k_off + qk ||
      a->row_stride < a->v_off + vv || a->row_stride < a->g_off + vv)
    return DZ_ERR_INVALID_ARG;
  if (a->num_seqs == 0 || a->rows == 0) return DZ_OK;
  LightningParams p = {a->x, a->row_stride, a->k_off, a->v_off, a->g_off, a->powers, a->norm_weight, a->eps, a->out, nullptr,
                       a->S, a->slots, a->q_starts, a->ctx_lens, a->heads, a->dim, a->vdim, nullptr};
  cudaStream_t st = (cudaStream_t)stream;
  if (!a->chunkwise) {
    if (!a->workspace || a->workspace_bytes < dz_lightning_workspace_bytes(a->rows, a->num_seqs, a->heads, a->vdim, 0))
      return DZ_ERR_WORKSPACE;
    const bool fused = a->rows == a->num_seqs;     // one token each: the norm rides on the last CTA of a row
    if (fused) p.tickets = (int*)a->workspace;
    p.o = (float*)((uint8_t*)a->workspace + kTicketBytes);
    int rc = DZ_OK;
    DZ_DISPATCH(a->dtype, rc = run_recurrent<T>(p, a->num_seqs, st));
    if (rc || fused) return rc;
    DZ_DISPATCH(a->dtype, return (run_norm<T, float>(p, p.o, a->rows, st)));
    return DZ_OK;
  }
  if (!dz_lightning_chunk_supported(a->dim, a->vdim, a->dtype)) return DZ_ERR_UNSUPPORTED;
  if (a->row_stride % 8 || a->k_off % 8 || a->v_off % 8 || !aligned16(a->x) || !aligned16(a->out)) return DZ_ERR_ALIGNMENT;
  int rc = DZ_OK;
  DZ_DISPATCH16(a->dtype, rc = run_chunk<T>(p, a->num_seqs, (a->dim + 15) / 16 * 16, st));
  if (rc) return rc;
  DZ_DISPATCH16(a->dtype, return (run_norm<T, T>(p, (const T*)p.out, a->rows, st)));
  return DZ_OK;
}

}  // extern "C"
