// Matrix-memory recurrence with exponential gates (the mLSTM cell of "xLSTM: Extended Long
// Short-Term Memory", Beck et al.).  Per head, with log gates i and f <= 0 and a running maximum m:
//
//   m' = max(f + m, i)      S' = e^(f + m - m') S + e^(i - m') k v^T      n' likewise with k alone
//   o  = S'^T q / (max(|n'.q|, e^-m') + 1e-6)
//
// i = cap tanh((w_i.h + b_i) / cap),  f = logsigmoid(cap tanh((w_f.h + b_f) / cap)),  q scaled by
// `scale`.  S [dim, vdim], n [dim] and m live in 32-bit pools, one slot per sequence; m and the state
// start at zero, which a sequence without context gets without its slot being read.
//
// Two kernels.  The recurrent one streams the state once per token and also does what follows the
// cell (per-head RMS norm, weight, sigmoid output gate); it serves decoding and the 32-bit type.  The
// chunkwise one takes 64 tokens at a time on the tensor cores for prompt portions.
#include <cooperative_groups.h>

#include "dz_elem.cuh"

namespace cg = cooperative_groups;

namespace dz {
namespace {

constexpr float kDenEps = 1e-6f;

struct MlstmParams {
  const void* x;                         // rows [q (heads*dim) | k (heads*dim) | v | g (heads*vdim)]
  int64_t row_stride;
  int k_off, v_off, g_off;
  const void* h;                         // [rows, width] the gates' input (recurrent kernel)
  const void* w_if;                      // [2 heads, width]: w_i then w_f
  const float* b_if;                     // [2 heads]
  const float* pre_if;                   // [rows, 2 heads] w.h without bias (chunk kernel)
  int width;
  float cap, scale;
  const float* norm_w;                   // [heads * vdim]
  float eps;
  void* out;                             // [rows, heads * vdim]
  float *S, *n, *m;                      // pools
  const int* slots;
  const int* q_starts;
  const int* ctx_lens;
  int heads, dim, vdim;
};

__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }

// -------------------------------------------------------------------------------------------------
// Recurrent form.  A cluster of C CTAs owns one (head, sequence); CTA r holds columns
// [r vt, (r + 1) vt) of S, streamed from and to the pool.  n and m are carried by every CTA of the
// cluster and written by the first.  Grid (C, heads, sequences).
// -------------------------------------------------------------------------------------------------
constexpr int kRecThreads = 256, kRowsInFlight = 8;

template <typename T, int VEC>
__global__ void __launch_bounds__(kRecThreads, 3)
mlstm_recurrent_kernel(MlstmParams p, int vt) {
  extern __shared__ float sm[];
  __shared__ float s_part[kRecThreads / 32], s_part2[kRecThreads / 32];
  __shared__ float s_sq[2];
  const int C = gridDim.x, rank = blockIdx.x, head = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  float* sq = sm;
  float* sk = sq + p.dim;
  float* sn = sk + p.dim;
  float* sv = sn + p.dim;
  float* so = sv + vt;                              // [row groups, vt]
  const int v0 = rank * vt, nv = max(0, min(vt, p.vdim - v0));
  const int cg_n = vt / VEC, rg_n = kRecThreads / cg_n;         // column groups, row groups
  const int cgi = tid % cg_n, rgi = tid / cg_n;
  const bool mine = rgi < rg_n && cgi * VEC < nv;
  pdl_wait();
  pdl_launch();
  const int q0 = p.q_starts[seq], tn = p.q_starts[seq + 1] - q0, ctx = p.ctx_lens[seq], slot = p.slots[seq];
  float* S = p.S + ((size_t)slot * p.heads + head) * p.dim * p.vdim + v0;
  float* gn = p.n + ((size_t)slot * p.heads + head) * p.dim;
  float* gm = p.m + (size_t)slot * p.heads + head;
  float m = ctx > 0 ? *gm : 0.f;
  for (int d = tid; d < p.dim; d += kRecThreads) sn[d] = ctx > 0 ? gn[d] : 0.f;
  const T* wi = (const T*)p.w_if + (size_t)head * p.width;
  const T* wf = (const T*)p.w_if + (size_t)(p.heads + head) * p.width;

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
    const T* h = (const T*)p.h + (size_t)(q0 + t) * p.width;
    const bool zero = ctx == 0 && t == 0;           // the state before this token is zero
    load_rows(rgi, zero);                           // on their way while the gates are computed
    for (int d = tid; d < p.dim; d += kRecThreads) {
      sq[d] = Cvt<T>::one(row[(size_t)head * p.dim + d]) * p.scale;
      sk[d] = Cvt<T>::one(row[p.k_off + (size_t)head * p.dim + d]);
    }
    for (int c = tid; c < nv; c += kRecThreads) sv[c] = Cvt<T>::one(row[p.v_off + (size_t)head * p.vdim + v0 + c]);
    float di = 0.f, df = 0.f;
    if constexpr (VEC == 4) {                       // also says that rows of h and w are vectors of eight
      for (int c = tid * 8; c < p.width; c += kRecThreads * 8) {
        float a[8], b[8], e[8];
        load8<T>(h + c, a);
        load8<T>(wi + c, b);
        load8<T>(wf + c, e);
#pragma unroll
        for (int j = 0; j < 8; ++j) { di += a[j] * b[j]; df += a[j] * e[j]; }
      }
    } else {
      for (int c = tid; c < p.width; c += kRecThreads) {
        const float a = Cvt<T>::one(h[c]);
        di += a * Cvt<T>::one(wi[c]);
        df += a * Cvt<T>::one(wf[c]);
      }
    }
    di = warp_sum(di);
    df = warp_sum(df);
    if ((tid & 31) == 0) { s_part[tid >> 5] = di; s_part2[tid >> 5] = df; }
    __syncthreads();
    di = df = 0.f;
#pragma unroll
    for (int w = 0; w < kRecThreads / 32; ++w) { di += s_part[w]; df += s_part2[w]; }
    const float gi = soft_cap(di + p.b_if[head], p.cap);
    const float gf = log_sigmoid(soft_cap(df + p.b_if[p.heads + head], p.cap));
    const float m_new = fmaxf(gf + m, gi);
    const float keep = expf(gf + m - m_new), add = expf(gi - m_new);
    m = m_new;

    float nq = 0.f;
    for (int d = tid; d < p.dim; d += kRecThreads) {
      const float v = sn[d] * keep + add * sk[d];
      sn[d] = v;
      nq += v * sq[d];
    }
    float o[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = 0.f;
    if (mine) {
      float v[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = sv[cgi * VEC + j] * add;
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
    nq = block_sum(nq, s_part);                     // also orders the writes of so before the reads below
    const float den = 1.f / (fmaxf(fabsf(nq), expf(-m)) + kDenEps);
    float ss = 0.f;
    for (int c = tid; c < nv; c += kRecThreads) {
      float a = 0.f;
      for (int g = 0; g < rg_n; ++g) a += so[g * vt + c];
      a *= den;
      so[c] = a;                                    // row 0 of this thread's own column
      ss += a * a;
    }
    ss = block_sum(ss, s_part);
    if (C > 1) {
      cg::cluster_group cl = cg::this_cluster();
      if (tid == 0) s_sq[t & 1] = ss;
      cl.sync();
      ss = 0.f;
      for (int r = 0; r < C; ++r) ss += *cl.map_shared_rank(&s_sq[t & 1], r);
    }
    const float inv = 1.f / sqrtf(ss / (float)p.vdim + p.eps);
    for (int c = tid; c < nv; c += kRecThreads) {
      const size_t col = (size_t)head * p.vdim + v0 + c;
      const float g = Cvt<T>::one(row[p.g_off + col]);
      ((T*)p.out)[(size_t)(q0 + t) * p.heads * p.vdim + col] =
          Cvt<T>::from(so[c] * inv * p.norm_w[col] / (1.f + expf(-g)));
    }
    __syncthreads();
  }
  if (C > 1) cg::this_cluster().sync();             // every CTA has read n and m, and its peers' sums
  if (rank == 0 && tn > 0) {
    for (int d = tid; d < p.dim; d += kRecThreads) gn[d] = sn[d];
    if (tid == 0) *gm = m;
  }
}

// -------------------------------------------------------------------------------------------------
// Chunkwise form, 16-bit activations.  With F_t the running sum of f inside the chunk, a_s = i_s - F_s
// and M_t = max(m_start, max_{s <= t} a_s), m_t = F_t + M_t and
//   o_t ~ sum_{s <= t} e^(a_s - M_t) (q_t.k_s) v_s + e^(m_start - M_t) q_t S_start
//   S_end = e^(m_start - M_L) S_start + sum_s e^(a_s - M_L) k_s v_s^T.
// A CTA of eight warps owns VT value columns of one (head, sequence) and walks the chunks; its slice
// of S stays in registers in 32 bits, as accumulators of the update, with n as one more row (the value
// matrix gets a column of ones).  32-bit operands enter the MMAs as hi + lo pairs, split once: S after
// its update, v times its gate weight at the start of a chunk.  A warp owns NTW groups of eight rows of
// k's columns (64 NTW >= dim).  Writes the cell's output before the
// head norm.  Grid (tiles of VT columns, heads, sequences).
// -------------------------------------------------------------------------------------------------
constexpr int kL = 64, kChunkThreads = 256;

template <int VT> __host__ __device__ constexpr int chunk_ldv() { return VT + 24; }

template <typename T, int VT, int NTW>
__global__ void __launch_bounds__(kChunkThreads, 1)
mlstm_chunk_kernel(MlstmParams p, int dimp, int* __restrict__ tickets) {
  constexpr int NT = VT / 16, MT = VT / 16 + 1, LDV = chunk_ldv<VT>();   // output: a warp has 16 rows, half of the columns
  extern __shared__ uint4 smem_raw[];
  __shared__ float s_a[kL], s_mx[kL], s_inter[kL], s_em[kL], s_w[kL];
  __shared__ float s_m, s_decay, s_mnext;
  __shared__ int s_last;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rw = warp & 3, cw = (warp >> 2) * (VT / 2);
  const int head = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * VT;
  pdl_wait();
  pdl_launch();
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0;
  if (qn <= 0) return;
  const int ctx = p.ctx_lens[seq], slot = p.slots[seq];
  const int vcols = min(VT, p.vdim - v0);
  const int ldk = dimp + 8, lds = dimp + 8;
  T* sq = reinterpret_cast<T*>(smem_raw);
  T* sk = sq + kL * ldk;
  T* sv = sk + kL * ldk;
  T* wh = sv + kL * LDV;                                          // v times its gate weight, hi and lo
  T* wl = wh + kL * LDV;
  T* sh = wl + kL * LDV;                                          // S transposed, hi and lo: [VT + 16][lds]
  T* sl = sh + (VT + 16) * lds;
  float* S = p.S + ((size_t)slot * p.heads + head) * p.dim * p.vdim + v0;
  float* gn = p.n + ((size_t)slot * p.heads + head) * p.dim;
  float* gm = p.m + (size_t)slot * p.heads + head;
  const int bytes = kL * (2 * ldk + 3 * LDV) * 2 + 2 * (VT + 16) * lds * 2;
  for (int i = tid; i < bytes / 16; i += kChunkThreads) smem_raw[i] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  for (int i = tid; i < kL; i += kChunkThreads) sv[i * LDV + VT] = Cvt<T>::from(1.f);
  // The state itself: rows mt * 16 + lane / 4 (+ 8), columns nt * 8 + 2 (lane % 4) (+ 1) of the transposed
  // slice, nt = warp + 8 i; the first row past the value columns is n.
  float acc[MT][NTW][4];
  const int col0 = warp * 8 + (lane & 3) * 2;
  auto each = [&](auto&& fn) {                       // fn(value, dim index, value column or -1 for n)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = col0 + i * 64 + (e & 1), v = mt * 16 + (lane >> 2) + (e >> 1) * 8;
          if (d < p.dim && (mt < MT - 1 ? v < vcols : v == VT)) fn(acc[mt][i][e], d, mt < MT - 1 ? v : -1);
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
  if (ctx > 0) {
    each([&](float& x, int d, int v) { x = v < 0 ? gn[d] : S[(size_t)d * p.vdim + v]; });
    publish();
  }
  if (tid == 0) s_m = ctx > 0 ? *gm : 0.f;
  const T* x = (const T*)p.x;
  const int r = tid >> 2, c0 = tid & 3;
  bool have_state = ctx > 0;
  // gate pre-activations of a chunk (warp 0; lane l holds tokens 2l and 2l + 1), fetched a chunk ahead
  float pi[2], pf[2];
  auto fetch_gates = [&](int base) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = base + 2 * lane + j;
      if (warp == 0 && t < qn) {
        const float* pre = p.pre_if + (size_t)(q0 + t) * 2 * p.heads;
        pi[j] = pre[head];
        pf[j] = pre[p.heads + head];
      }
    }
  };
  fetch_gates(0);
  __syncthreads();

  for (int base = 0; base < qn; base += kL) {
    const int len = min(kL, qn - base);
    {
      const bool ok = r < len;
      const T* row = x + (size_t)(q0 + base + (ok ? r : 0)) * p.row_stride;
      const T* qs = row + (size_t)head * p.dim;
      const T* ks = row + p.k_off + (size_t)head * p.dim;
      const T* vs = row + p.v_off + (size_t)head * p.vdim + v0;
      for (int c = c0; c < p.dim / 8; c += 4) {
        cp_async16(sq + r * ldk + c * 8, qs + c * 8, ok);
        cp_async16(sk + r * ldk + c * 8, ks + c * 8, ok);
      }
      for (int c = c0; c < vcols / 8; c += 4) cp_async16(sv + r * LDV + c * 8, vs + c * 8, ok);
      cp_async_commit();
    }
    if (warp == 0) {                                 // gates
      float gi[2], gf[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = 2 * lane + j;
        gi[j] = -INFINITY;                           // absent tokens add nothing and forget nothing
        gf[j] = 0.f;
        if (t < len) {
          gi[j] = soft_cap(pi[j] + p.b_if[head], p.cap);
          gf[j] = log_sigmoid(soft_cap(pf[j] + p.b_if[p.heads + head], p.cap));
        }
      }
      float f = gf[0] + gf[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, f, o);
        if (lane >= o) f += up;
      }
      const float F1 = f, F0 = f - gf[1];
      const float a0 = gi[0] - F0, a1 = gi[1] - F1;
      float mx = fmaxf(a0, a1);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, mx, o);
        if (lane >= o) mx = fmaxf(mx, up);
      }
      const float m0 = s_m;
      float before = __shfl_up_sync(0xffffffffu, mx, 1);
      if (lane == 0) before = -INFINITY;
      const float M0 = fmaxf(m0, fmaxf(before, a0)), M1 = fmaxf(m0, mx);
      const float ML = __shfl_sync(0xffffffffu, M1, 31), FL = __shfl_sync(0xffffffffu, F1, 31);
      const int t = 2 * lane;
      s_a[t] = a0; s_a[t + 1] = a1;
      s_mx[t] = M0; s_mx[t + 1] = M1;
      s_inter[t] = expf(m0 - M0) * p.scale; s_inter[t + 1] = expf(m0 - M1) * p.scale;
      s_em[t] = expf(-(F0 + M0)); s_em[t + 1] = expf(-(F1 + M1));
      s_w[t] = expf(a0 - ML); s_w[t + 1] = expf(a1 - ML);
      if (lane == 0) { s_decay = expf(m0 - ML); s_mnext = FL + ML; }
    }
    fetch_gates(base + kL);
    cp_async_wait<0>();
    __syncthreads();
    for (int i = c0; i < (VT + 16) / 8; i += 4) {     // four threads a row, eight columns at a time
      const int at = r * LDV + i * 8;
      const float w = s_w[r];
      float f[8];
      load8<T>(sv + at, f);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) split_pair<T>(f[2 * j] * w, f[2 * j + 1] * w, hi[j], lo[j]);
      *reinterpret_cast<uint4*>(wh + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(wl + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }

    const int r0 = rw * 16 + (lane >> 2), r1 = r0 + 8;
    if (rw * 16 < len) {
      float o[NT + 1][4];
#pragma unroll
      for (int i = 0; i <= NT; ++i)
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
          uint32_t bh[NT / 2 + 1][4], bl[NT / 2 + 1][4];
#pragma unroll
          for (int i = 0; i <= NT / 2; ++i) {       // the last pair of tiles starts with n
            const int at = ((i < NT / 2 ? cw + i * 16 : VT) + (lane & 7) + ((lane >> 4) & 1) * 8) * lds +
                           ((lane >> 3) & 1) * 8 + kk;
            ldsm4(bh[i], sh + at);
            ldsm4(bl[i], sl + at);
          }
#pragma unroll
          for (int i = 0; i <= NT; ++i) mma16816<T>(o[i], a, bh[i / 2][2 * (i & 1)], bh[i / 2][2 * (i & 1) + 1]);
#pragma unroll
          for (int i = 0; i <= NT; ++i) mma16816<T>(o[i], a, bl[i / 2][2 * (i & 1)], bl[i / 2][2 * (i & 1) + 1]);
        }
      }
      const float in0 = s_inter[r0], in1 = s_inter[r1], mx0 = s_mx[r0], mx1 = s_mx[r1];
#pragma unroll
      for (int i = 0; i <= NT; ++i) {
        o[i][0] *= in0;
        o[i][1] *= in0;
        o[i][2] *= in1;
        o[i][3] *= in1;
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int t = i * 8 + (lane & 3) * 2 + (j & 1);
          const float e = t <= (j < 2 ? r0 : r1) ? __expf(s_a[t] - (j < 2 ? mx0 : mx1)) : 0.f;
          s[i][j] *= e * p.scale;
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
          uint32_t b[4];
          ldsm4_t(b, bv + kk * 16 * LDV + VT);
          mma16816<T>(o[NT], hi, b[0], b[1]);
          mma16816<T>(o[NT], lo, b[0], b[1]);
        }
      }
      const float nq0 = __shfl_sync(0xffffffffu, o[NT][0], lane & ~3);
      const float nq1 = __shfl_sync(0xffffffffu, o[NT][2], lane & ~3);
      const float d0 = 1.f / (fmaxf(fabsf(nq0), s_em[r0]) + kDenEps);
      const float d1 = 1.f / (fmaxf(fabsf(nq1), s_em[r1]) + kDenEps);
      T* op = (T*)p.out + (size_t)(q0 + base) * p.heads * p.vdim + (size_t)head * p.vdim + v0;
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int c = cw + i * 8 + (lane & 3) * 2;
        if (c < vcols) {
          if (r0 < len)
            *reinterpret_cast<uint32_t*>(op + (size_t)r0 * p.heads * p.vdim + c) = Cvt<T>::down(o[i][0] * d0, o[i][1] * d0);
          if (r1 < len)
            *reinterpret_cast<uint32_t*>(op + (size_t)r1 * p.heads * p.vdim + c) = Cvt<T>::down(o[i][2] * d1, o[i][3] * d1);
        }
      }
    }
    __syncthreads();                                 // the old state has been read
    const float decay = s_decay;
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
    for (int mt = 0; mt < MT; ++mt) {                // 16 value columns, or the column of ones
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
    publish();
    if (tid == 0) s_m = s_mnext;
    have_state = true;
    __syncthreads();
  }
  each([&](float& x, int d, int v) {
    if (v >= 0) S[(size_t)d * p.vdim + v] = x;
  });
  // n and m, read by every CTA of this (head, sequence) at its start, are written by the last to end
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    int* tk = tickets + (size_t)seq * p.heads + head;
    s_last = atomicAdd(tk, 1) == (int)gridDim.x - 1;
    if (s_last) *tk = 0;
  }
  __syncthreads();
  if (s_last) {
    each([&](float& x, int d, int v) {
      if (v < 0) gn[d] = x;
    });
    if (tid == 0) *gm = s_m;
  }
}

// out = (o / rms(o) per head) * w * sigmoid(g); a warp per (row, head), in place allowed
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const T* o, const T* __restrict__ g, int64_t g_stride, const float* __restrict__ w,
                      float eps, T* out, int rows, int heads, int vdim) {
  const int lane = threadIdx.x & 31;
  const int64_t id = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  pdl_wait();
  pdl_launch();
  if (id >= (int64_t)rows * heads) return;
  const int64_t row = id / heads;
  const int head = (int)(id - row * heads);
  const T* op = o + row * heads * vdim + (int64_t)head * vdim;
  const T* gp = g + row * g_stride + (int64_t)head * vdim;
  const float* wp = w + (int64_t)head * vdim;
  T* dst = out + row * heads * vdim + (int64_t)head * vdim;
  float ss = 0.f;
  for (int c = lane * VEC; c < vdim; c += 32 * VEC) {
    if constexpr (VEC == 8) {
      float f[8];
      load8<T>(op + c, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
    } else {
      const float f = Cvt<T>::one(op[c]);
      ss += f * f;
    }
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)vdim + eps);
  for (int c = lane * VEC; c < vdim; c += 32 * VEC) {
    if constexpr (VEC == 8) {
      float f[8], e[8], v[8];
      load8<T>(op + c, f);
      load8<T>(gp + c, e);
      load8<float>(wp + c, v);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = f[j] * inv * v[j] / (1.f + __expf(-e[j]));
      store8<T>(dst + c, f);
    } else {
      dst[c] = Cvt<T>::from(Cvt<T>::one(op[c]) * inv * wp[c] / (1.f + expf(-Cvt<T>::one(gp[c]))));
    }
  }
}

size_t chunk_smem(int dimp, int vt) {
  return (size_t)kL * (2 * (dimp + 8) + 3 * (vt + 24)) * 2 + (size_t)2 * (vt + 16) * (dimp + 8) * 2;
}

template <typename T, int VT, int NTW>
int run_chunk_n(const MlstmParams& p, int num_seqs, int dimp, int* tickets, cudaStream_t st) {
  const size_t smem = chunk_smem(dimp, VT);
  DZ_CUDA_OK(allow_smem(mlstm_chunk_kernel<T, VT, NTW>, smem));
  DZ_CUDA_OK(launch_ex(mlstm_chunk_kernel<T, VT, NTW>, dim3((p.vdim + VT - 1) / VT, p.heads, num_seqs),
                       dim3(kChunkThreads), smem, 1, st, p, dimp, tickets));
  return DZ_OK;
}
template <typename T, int VT>
int run_chunk(const MlstmParams& p, int num_seqs, int dimp, int* tickets, cudaStream_t st) {
  if (dimp <= 64) return run_chunk_n<T, VT, 1>(p, num_seqs, dimp, tickets, st);
  if (dimp <= 128) return run_chunk_n<T, VT, 2>(p, num_seqs, dimp, tickets, st);
  if (dimp <= 256) return run_chunk_n<T, VT, 4>(p, num_seqs, dimp, tickets, st);
  return run_chunk_n<T, 32, 8>(p, num_seqs, dimp, tickets, st);
}

template <typename T>
int run_recurrent(const MlstmParams& p, int num_seqs, cudaStream_t st) {
  const bool vec = p.vdim % 4 == 0 && p.width % 8 == 0 && aligned16(p.h) && aligned16(p.w_if) && aligned16(p.S);
  const int v = vec ? 4 : 1;
  // columns per CTA: a slice of S of at most 64 KB, at most 8 CTAs (and never more column groups than threads)
  int c = 1;
  while (c < 8 && (size_t)p.dim * ((p.vdim + c - 1) / c) * 4 > 64 * 1024 && p.vdim / (2 * c) >= v) c *= 2;
  int vt = ((p.vdim + c - 1) / c + v - 1) / v * v;
  while (vt / v > kRecThreads && c < 8) { c *= 2; vt = ((p.vdim + c - 1) / c + v - 1) / v * v; }
  const int rg = kRecThreads / (vt / v > 0 ? vt / v : 1);
  const size_t smem = ((size_t)3 * p.dim + vt + (size_t)rg * vt) * 4;
  if (vt / v > kRecThreads || smem > kMaxDynSmem) return DZ_ERR_SHAPE;
  const dim3 grid(c, p.heads, num_seqs);
  if (vec) {
    DZ_CUDA_OK(allow_smem(mlstm_recurrent_kernel<T, 4>, smem));
    DZ_CUDA_OK(launch_ex(mlstm_recurrent_kernel<T, 4>, grid, dim3(kRecThreads), smem, c, st, p, vt));
  } else {
    DZ_CUDA_OK(allow_smem(mlstm_recurrent_kernel<T, 1>, smem));
    DZ_CUDA_OK(launch_ex(mlstm_recurrent_kernel<T, 1>, grid, dim3(kRecThreads), smem, c, st, p, vt));
  }
  return DZ_OK;
}

}  // namespace
}  // namespace dz

using namespace dz;

extern "C" {

// Whether dz_mlstm has a chunkwise kernel for these sizes (it then reads pre_if, else h and w_if).
int dz_mlstm_chunk_supported(int dim, int vdim, int dtype) {
  if (dtype != DZ_DTYPE_F16 && dtype != DZ_DTYPE_BF16) return 0;
  if (dim <= 0 || vdim <= 0 || dim % 8 || vdim % 8) return 0;
  const int dimp = (dim + 15) / 16 * 16;
  return dimp <= 512 && chunk_smem(dimp, 32) <= kMaxDynSmem;
}

size_t dz_mlstm_workspace_bytes(int num_seqs, int heads) {
  return num_seqs > 0 && heads > 0 ? (size_t)num_seqs * heads * 4 : 0;
}

int dz_mlstm(const dz_mlstm_args* a, void* stream) {
  if (!a || !a->x || !a->out || !a->S || !a->n || !a->m || !a->slots || !a->q_starts || !a->ctx_lens || !a->b_if ||
      !a->norm_weight)
    return DZ_ERR_INVALID_ARG;
  if (a->num_seqs < 0 || a->num_seqs > 65535 || a->rows < 0 || a->heads <= 0 || a->heads > 65535 || a->dim <= 0 ||
      a->vdim <= 0 || a->width <= 0 || !(a->cap > 0.f) || !is_float_dtype(a->dtype))
    return DZ_ERR_INVALID_ARG;
  const int64_t qk = (int64_t)a->heads * a->dim, vv = (int64_t)a->heads * a->vdim;
  if (a->k_off < 0 || a->v_off < 0 || a->g_off < 0 || a->row_stride < qk || a->row_stride < a->k_off + qk ||
      a->row_stride < a->v_off + vv || a->row_stride < a->g_off + vv)
    return DZ_ERR_INVALID_ARG;
  if (a->num_seqs == 0 || a->rows == 0) return DZ_OK;
  MlstmParams p = {a->x, a->row_stride, a->k_off, a->v_off, a->g_off, a->h, a->w_if, a->b_if, a->pre_if, a->width,
                   a->cap, a->scale, a->norm_weight, a->eps, a->out, a->S, a->n, a->m, a->slots, a->q_starts,
                   a->ctx_lens, a->heads, a->dim, a->vdim};
  cudaStream_t st = (cudaStream_t)stream;
  if (!a->chunkwise) {
    if (!a->h || !a->w_if) return DZ_ERR_INVALID_ARG;
    DZ_DISPATCH(a->dtype, return run_recurrent<T>(p, a->num_seqs, st));
    return DZ_OK;
  }
  if (!a->pre_if || !dz_mlstm_chunk_supported(a->dim, a->vdim, a->dtype)) return DZ_ERR_UNSUPPORTED;
  if (a->row_stride % 8 || a->k_off % 8 || a->v_off % 8 || a->g_off % 8 || !aligned16(a->x) || !aligned16(a->out))
    return DZ_ERR_ALIGNMENT;
  if (!a->workspace || a->workspace_bytes < dz_mlstm_workspace_bytes(a->num_seqs, a->heads)) return DZ_ERR_WORKSPACE;
  const int dimp = (a->dim + 15) / 16 * 16;
  int rc = DZ_OK;
  const bool wide = a->vdim > 32 && dimp <= 256 && chunk_smem(dimp, 64) <= kMaxDynSmem;
  DZ_DISPATCH16(a->dtype, rc = wide ? run_chunk<T, 64>(p, a->num_seqs, dimp, (int*)a->workspace, st)
                                    : run_chunk<T, 32>(p, a->num_seqs, dimp, (int*)a->workspace, st));
  if (rc) return rc;
  const unsigned blocks = (unsigned)(((int64_t)a->rows * a->heads + 7) / 8);
  DZ_DISPATCH16(a->dtype,
                DZ_CUDA_OK(launch_pdl(a->norm_weight && aligned16(a->norm_weight) ? head_norm_gate_kernel<T, 8>
                                                                                  : head_norm_gate_kernel<T, 1>,
                                      dim3(blocks), dim3(256), st, (const T*)a->out,
                                      (const T*)a->x + a->g_off, a->row_stride, a->norm_weight, a->eps, (T*)a->out,
                                      a->rows, a->heads, a->vdim)));
  return DZ_OK;
}

}  // extern "C"
