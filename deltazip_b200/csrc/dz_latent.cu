// Attention over a cached latent (the multi-head latent attention of "DeepSeek-V2: A Strong, Economical,
// and Efficient Mixture-of-Experts Language Model", DeepSeek-AI).  A token leaves one row
//
//   [ c (rank) | r (rot) ]      c = RMS norm of its latent,  r = its rotated key part, shared by all heads
//
// in the paged cache.  A head's key is [U_h c | r], its value V_h c, its query [a | b] with b rotated:
//
//   score = (a . U_h c + b . r) * scale = ([U_h^T a | b] . [c | r]) * scale,   output = V_h (sum p c).
//
// The left form expands a prompt's rows into keys and values (dz_latent_gather, a GEMM and
// dz_window_attention); the right one, for decoding and short portions, works on the rows as they lie,
// one key and value row for all heads (dz_latent_attention).
//
// Neighbouring components (2i, 2i + 1) are rotated by position * freq[i]; the angle is formed and brought
// into one turn in 64 bits, sine and cosine are 32-bit.  Scores, softmax weights and sums are 32-bit; a
// weight enters its product as a hi + lo pair of 16-bit numbers.
#include "dz_latent.cuh"
#include "dz_window_attention.cuh"

namespace dz {
namespace {

constexpr int kRowThreads = 128;

template <typename T> struct PairOf { using type = uint32_t; };
template <> struct PairOf<float> { using type = float2; };

template <typename T> __device__ __forceinline__ float2 load_pair(const T* p) {
  if constexpr (sizeof(T) == 2) return Cvt<T>::up(*reinterpret_cast<const uint32_t*>(p));
  else return *reinterpret_cast<const float2*>(p);
}
template <typename T> __device__ __forceinline__ void store_pair(T* p, float a, float b) {
  if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(p) = Cvt<T>::down(a, b);
  else *reinterpret_cast<float2*>(p) = make_float2(a, b);
}

template <typename T, bool PAIRS>
__device__ __forceinline__ void rotate(const T* src, T* dst, float2 cs) {
  float u, v;
  if constexpr (PAIRS) {
    const float2 x = load_pair<T>(src);
    u = x.x;
    v = x.y;
  } else {
    u = Cvt<T>::one(src[0]);
    v = Cvt<T>::one(src[1]);
  }
  const float a = u * cs.x - v * cs.y, b = v * cs.x + u * cs.y;
  if constexpr (PAIRS) {
    store_pair<T>(dst, a, b);
  } else {
    dst[0] = Cvt<T>::from(a);
    dst[1] = Cvt<T>::from(b);
  }
}

struct RowParams {
  const void* x;                         // rows [q: heads x (dim + rot) | ... | latent at l_off: rank + rot]
  int64_t row_stride;
  const long long* positions;
  const double* freq;                    // [rot / 2]
  int heads, dim, rot;
  void* q_out;                           // [rows, heads, rank + rot], its last rot columns; nullptr: in place
  int l_off, rank;                       // l_off < 0: the rows have no latent
  const float* norm_w;
  float eps;
  void* cache;                           // [slots, rank + rot]
  const long long* slots;
};

// The queries' rotation, and the latent's norm, its rotation and the cache append; a CTA per row.  VEC: the
// parts consist of whole vectors of eight.
template <typename T, bool PAIRS, bool VEC>
__global__ void __launch_bounds__(kRowThreads)
latent_rows_kernel(RowParams p) {
  extern __shared__ float2 s_cs[];
  __shared__ float s_part[kRowThreads / 32];
  pdl_wait();
  pdl_launch();
  const size_t row = blockIdx.x;
  const long long slot = p.l_off >= 0 ? p.slots[row] : -1;
  const int half = p.rot / 2;
  const double pos = (double)p.positions[row];
  for (int i = threadIdx.x; i < half; i += kRowThreads) {
    constexpr double kTurn = 6.283185307179586476925286766559;
    double a = pos * p.freq[i];
    a -= kTurn * rint(a * (1.0 / kTurn));
    float s, c;
    sincosf((float)a, &s, &c);
    s_cs[i] = make_float2(c, s);
  }
  const T* x = (const T*)p.x + row * p.row_stride;
  const T* lat = x + p.l_off;
  T* dst = (T*)p.cache + (size_t)slot * (p.rank + p.rot);
  float ss = 0.f;
  if (slot >= 0) {
    if constexpr (VEC) {
      for (int i = threadIdx.x * 8; i < p.rank; i += kRowThreads * 8) {
        float f[8];
        load8<T>(lat + i, f);
#pragma unroll
        for (int q = 0; q < 8; ++q) ss += f[q] * f[q];
      }
    } else {
      for (int i = threadIdx.x; i < p.rank; i += kRowThreads) {
        const float f = Cvt<T>::one(lat[i]);
        ss += f * f;
      }
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)p.rank + p.eps);        // also orders s_cs
  if constexpr (VEC) {
    const int per = p.rot / 8;
    for (int j = threadIdx.x; j < p.heads * per; j += kRowThreads) {
      const int head = j / per, i = (j - head * per) * 8;
      const T* src = x + (size_t)head * (p.dim + p.rot) + p.dim + i;
      T* to = p.q_out ? (T*)p.q_out + (row * p.heads + head) * (p.rank + p.rot) + p.rank + i : const_cast<T*>(src);
      float f[8];
      load8<T>(src, f);
#pragma unroll
      for (int q = 0; q < 8; q += 2) {
        const float2 cs = s_cs[(i + q) / 2];
        const float u = f[q], v = f[q + 1];
        f[q] = u * cs.x - v * cs.y;
        f[q + 1] = v * cs.x + u * cs.y;
      }
      store8<T>(to, f);
    }
  } else {
    for (int j = threadIdx.x; j < p.heads * half; j += kRowThreads) {
      const int head = j / half, i = j - head * half;
      const T* src = x + (size_t)head * (p.dim + p.rot) + p.dim + 2 * i;
      T* to = p.q_out ? (T*)p.q_out + (row * p.heads + head) * (p.rank + p.rot) + p.rank + 2 * i : const_cast<T*>(src);
      rotate<T, PAIRS>(src, to, s_cs[i]);
    }
  }
  if (slot < 0) return;
  if constexpr (VEC) {
    for (int i = threadIdx.x * 8; i < p.rank; i += kRowThreads * 8) {
      float f[8], w[8];
      load8<T>(lat + i, f);
      load8<float>(p.norm_w + i, w);
#pragma unroll
      for (int q = 0; q < 8; ++q) f[q] = f[q] * inv * w[q];
      store8<T>(dst + i, f);
    }
  } else {
    for (int i = threadIdx.x; i < p.rank; i += kRowThreads) dst[i] = Cvt<T>::from(Cvt<T>::one(lat[i]) * inv * p.norm_w[i]);
  }
  for (int i = threadIdx.x; i < half; i += kRowThreads)
    rotate<T, PAIRS>(lat + p.rank + 2 * i, dst + p.rank + 2 * i, s_cs[i]);
}

// Cached rows of positions 0, 1, ... of every sequence into consecutive rows; grid (positions / 8, sequences).
// A warp copies a row of `units` units of V.
template <typename V>
__global__ void __launch_bounds__(256)
latent_gather_kernel(const V* __restrict__ cache, const int* __restrict__ tables, int table_width, int block_size,
                     const int* __restrict__ starts, V* __restrict__ out, int units) {
  pdl_wait();
  pdl_launch();
  const int seq = blockIdx.y, row0 = starts[seq], n = starts[seq + 1] - row0;
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (t >= n) return;
  const size_t slot = (size_t)tables[(size_t)seq * table_width + t / block_size] * block_size + t % block_size;
  const V* src = cache + slot * units;
  V* dst = out + (size_t)(row0 + t) * units;
  for (int i = threadIdx.x & 31; i < units; i += 32) dst[i] = src[i];
}

// -------------------------------------------------------------------------------------------------
// All heads of a row against the cached rows, 16-bit, on warp MMAs: for what dz_latent_tc.cu does not take
// (pages that are not a multiple of eight tokens).  A CTA takes 16 MT heads (the MMA's M) of one row
// and a share of the keys, 64 per step, double-buffered through cp.async.  Eight warps: for the scores
// (16 keys) x (half of the row's columns), for the sums a share of the latent's columns.  Grid (head
// groups, rows, splits).
// -------------------------------------------------------------------------------------------------
constexpr int kKeys = 64, kLatentThreads = 256, kMaxGroups = 4;      // 16-column groups of the latent per warp
constexpr int kLdS = kKeys + 4, kLdP = kKeys + 8;

template <typename T, int MT>
__global__ void __launch_bounds__(kLatentThreads, 1)
latent_decode_kernel(LatentParams p) {
  constexpr int kHeads = 16 * MT, kPer = kLatentThreads / kHeads, kMine = kKeys / kPer;
  extern __shared__ uint4 smem_raw[];
  __shared__ float s_corr[kHeads], s_m[kHeads], s_l[kHeads];
  __shared__ int s_seq, s_last;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h0 = blockIdx.x * kHeads, row = blockIdx.y, split = blockIdx.z, live = min(kHeads, p.heads - h0);
  const int d = p.rank + p.rot, dp = (d + 15) / 16 * 16, ld = dp + 8;
  T* sq = reinterpret_cast<T*>(smem_raw);
  T* sk = sq + kHeads * ld;
  T* ph = sk + 2 * kKeys * ld;
  T* pl = ph + kHeads * kLdP;
  float* ss = reinterpret_cast<float*>(pl + kHeads * kLdP);          // [2][kHeads][kLdS]
  if (d < dp)                                                        // columns up to the MMA's K read as zero
    for (int i = tid; i < 2 * kKeys + kHeads; i += kLatentThreads)
      for (int c = d; c < dp; c += 8) *reinterpret_cast<uint4*>(sq + (size_t)i * ld + c) = make_uint4(0, 0, 0, 0);
  pdl_wait();
  pdl_launch();
  int seq = row, q0 = row;
  if (p.rows != p.num_seqs) {
    for (int s = tid; s < p.num_seqs; s += kLatentThreads)
      if (row >= p.q_starts[s] && row < p.q_starts[s + 1]) s_seq = s;
    __syncthreads();
    seq = s_seq;
    q0 = p.q_starts[seq];
  }
  const int n = p.ctx_lens[seq] + row - q0 + 1;                      // keys up to and with the row's own
  const int per = keys_per_split(n, p.splits);
  const int t0 = min(n, split * per), t1 = min(n, t0 + per);
  const int* table = p.tables + (size_t)seq * p.table_width;
  const T* cache = (const T*)p.cache;
  const int chunks = d / 8;
  for (int i = warp; i < kHeads; i += 8) {
    const bool ok = i < live;
    const T* src = (const T*)p.q + ((size_t)row * p.heads + h0 + (ok ? i : 0)) * d;
    for (int c = lane; c < chunks; c += 32) cp_async16(sq + i * ld + c * 8, src + c * 8, ok);
  }
  auto load = [&](int buf, int base) {
    for (int r = warp; r < kKeys; r += 8) {
      const int t = base + r;
      const bool ok = t < t1;
      const int tc = ok ? t : t0;
      const T* src = cache + ((size_t)table[tc / p.block_size] * p.block_size + tc % p.block_size) * d;
      T* dst = sk + (buf * kKeys + r) * ld;
      for (int c = lane; c < chunks; c += 32) cp_async16(dst + c * 8, src + c * 8, ok);
    }
  };
  float o[MT][kMaxGroups][2][4];
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int g = 0; g < kMaxGroups; ++g)
#pragma unroll
      for (int e = 0; e < 8; ++e) o[a][g][e >> 2][e & 3] = 0.f;
  float m = -INFINITY, l = 0.f;                                      // of the row of scores this thread shares
  const int groups = (p.rank + 15) / 16;
  const int kg = warp & 3, kh = warp >> 2, ksteps = dp / 16, kmid = (ksteps + 1) / 2;
  const int my = tid / kPer, sub = tid % kPer;
  const float scale2 = p.scale * kLog2e;
  const int tiles = t1 > t0 ? (t1 - t0 + kKeys - 1) / kKeys : 0;
  if (tiles) load(0, t0);
  cp_async_commit();
  for (int it = 0; it < tiles; ++it) {
    const int base = t0 + it * kKeys, buf = it & 1;
    if (it + 1 < tiles) {
      load(buf ^ 1, base + kKeys);
      cp_async_commit();
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const T* kt = sk + buf * kKeys * ld;
    {
      float s[MT][2][4];
#pragma unroll
      for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int e = 0; e < 8; ++e) s[a][e >> 2][e & 3] = 0.f;
      const T* aq = sq + (lane & 15) * ld + (lane >> 4) * 8;
      const T* bk = kt + (kg * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * ld + ((lane >> 3) & 1) * 8;
      const int k1 = kh ? ksteps : kmid;
#pragma unroll 4
      for (int k = kh ? kmid : 0; k < k1; ++k) {
        uint32_t b[4];
        ldsm4(b, bk + k * 16);
#pragma unroll
        for (int a = 0; a < MT; ++a) {
          uint32_t f[4];
          ldsm4(f, aq + a * 16 * ld + k * 16);
          mma16816<T>(s[a][0], f, b[0], b[1]);
          mma16816<T>(s[a][1], f, b[2], b[3]);
        }
      }
      float* sp = ss + (size_t)kh * kHeads * kLdS + (lane >> 2) * kLdS + kg * 16 + (lane & 3) * 2;
#pragma unroll
      for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          *reinterpret_cast<float2*>(sp + a * 16 * kLdS + j * 8) = make_float2(s[a][j][0], s[a][j][1]);
          *reinterpret_cast<float2*>(sp + (a * 16 + 8) * kLdS + j * 8) = make_float2(s[a][j][2], s[a][j][3]);
        }
    }
    __syncthreads();
    {
      const float* sp = ss + my * kLdS + sub * kMine;
      float v[kMine], mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < kMine; ++j) {
        v[j] = base + sub * kMine + j < t1 ? (sp[j] + sp[kHeads * kLdS + j]) * scale2 : -INFINITY;
        mx = fmaxf(mx, v[j]);
      }
#pragma unroll
      for (int w = kPer / 2; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      const float mn = fmaxf(m, mx), corr = exp2f(m - mn);          // the tile's first key is visible: mn is finite
      m = mn;
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < kMine; j += 2) {
        const float a = exp2f(v[j] - mn), b = exp2f(v[j + 1] - mn);
        sum += a + b;
        uint32_t hi, lo;
        split_pair<T>(a, b, hi, lo);
        *reinterpret_cast<uint32_t*>(ph + my * kLdP + sub * kMine + j) = hi;
        *reinterpret_cast<uint32_t*>(pl + my * kLdP + sub * kMine + j) = lo;
      }
      l = l * corr + sum;
      if (sub == 0) s_corr[my] = corr;
    }
    __syncthreads();
#pragma unroll
    for (int a = 0; a < MT; ++a) {
      const float c0 = s_corr[a * 16 + (lane >> 2)], c1 = s_corr[a * 16 + (lane >> 2) + 8];
      if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
        for (int g = 0; g < kMaxGroups; ++g)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            o[a][g][j][0] *= c0;
            o[a][g][j][1] *= c0;
            o[a][g][j][2] *= c1;
            o[a][g][j][3] *= c1;
          }
      }
    }
    const T* ap = ph + (lane & 15) * kLdP + (lane >> 4) * 8;
    const T* bv = kt + ((lane & 7) + ((lane >> 3) & 1) * 8) * ld + ((lane >> 4) & 1) * 8;
#pragma unroll
    for (int k = 0; k < kKeys / 16; ++k) {
      uint32_t hi[MT][4], lo[MT][4];
#pragma unroll
      for (int a = 0; a < MT; ++a) {
        ldsm4(hi[a], ap + a * 16 * kLdP + k * 16);
        ldsm4(lo[a], ap + kHeads * kLdP + a * 16 * kLdP + k * 16);
      }
#pragma unroll
      for (int g = 0; g < kMaxGroups; ++g) {
        if (warp + 8 * g < groups) {
          uint32_t b[4];
          ldsm4_t(b, bv + k * 16 * ld + (warp + 8 * g) * 16);
#pragma unroll
          for (int a = 0; a < MT; ++a) {
            mma16816<T>(o[a][g][0], hi[a], b[0], b[1]);
            mma16816<T>(o[a][g][1], hi[a], b[2], b[3]);
          }
#pragma unroll
          for (int a = 0; a < MT; ++a) {
            mma16816<T>(o[a][g][0], lo[a], b[0], b[1]);
            mma16816<T>(o[a][g][1], lo[a], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();                                                 // the buffer is loaded again two steps on
  }
  cp_async_wait<0>();
#pragma unroll
  for (int w = kPer / 2; w > 0; w >>= 1) l += __shfl_xor_sync(0xffffffffu, l, w);
  if (sub == 0) {
    float f = 1.f;
    if (p.splits == 1) {
      const float sk2 = p.sink && my < live ? p.sink[h0 + my] * kLog2e : -INFINITY, top = fmaxf(m, sk2);
      const float c = exp2f(m - top);
      f = c / (l * c + exp2f(sk2 - top));
    }
    s_corr[my] = f;
    s_m[my] = m;
    s_l[my] = l;
  }
  __syncthreads();
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int g = 0; g < kMaxGroups; ++g)
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int h = a * 16 + (lane >> 2) + (e >> 1) * 8, c = (warp + 8 * g) * 16 + j * 8 + (lane & 3) * 2;
          if (h < live && c < p.rank) {                              // rank is a multiple of eight
            const float f = s_corr[h], x = o[a][g][j][e] * f, y = o[a][g][j][e + 1] * f;
            const size_t at = (size_t)row * p.heads + h0 + h;
            if (p.splits == 1) {
              *reinterpret_cast<uint32_t*>((T*)p.out + at * p.rank + c) = Cvt<T>::down(x, y);
            } else {
              *reinterpret_cast<float2*>(p.partial + (at * p.splits + split) * partial_row(p.rank) + c) = make_float2(x, y);
            }
          }
        }
  if (p.splits == 1) return;
  if (tid < live) {
    float* pp = p.partial + (((size_t)row * p.heads + h0 + tid) * p.splits + split) * partial_row(p.rank) + p.rank;
    pp[0] = s_m[tid];
    pp[1] = s_l[tid];
  }
  merge_splits<T>(p, row, h0, live, &s_last, reinterpret_cast<float*>(smem_raw));
}

int head_tiles(int heads) { return heads <= 16 ? 1 : 2; }
int head_groups(int heads) { return (heads + 16 * head_tiles(heads) - 1) / (16 * head_tiles(heads)); }
size_t latent_smem(int heads, int d) {
  const size_t h = 16 * head_tiles(heads), ld = (d + 15) / 16 * 16 + 8;
  return (h + 2 * kKeys) * ld * 2 + 2 * h * kLdP * 2 + 2 * h * kLdS * 4;
}

bool tensor_core_shapes(int heads, int rank, int rot, int dtype) {
  return (dtype == DZ_DTYPE_F16 || dtype == DZ_DTYPE_BF16) && rank % 8 == 0 && (rank + rot) % 8 == 0 &&
         rank <= 16 * 8 * kMaxGroups && latent_smem(heads, rank + rot) <= kMaxDynSmem;
}

template <typename T, int MT>
int run_latent(const LatentParams& p, cudaStream_t st) {
  const size_t smem = latent_smem(p.heads, p.rank + p.rot);
  DZ_CUDA_OK(allow_smem(latent_decode_kernel<T, MT>, smem));
  DZ_CUDA_OK(launch_ex(latent_decode_kernel<T, MT>, dim3(head_groups(p.heads), p.rows, p.splits), dim3(kLatentThreads),
                       smem, 1, st, p));
  return DZ_OK;
}

}  // namespace
}  // namespace dz

using namespace dz;

extern "C" {

int dz_latent_rows(const dz_latent_rows_args* a, void* stream) {
  if (!a || !a->x || !a->positions || !a->freq || a->rows < 0 || a->heads <= 0 || a->dim < 0 || a->rot <= 0 || a->rot % 2 ||
      !is_float_dtype(a->dtype) || a->row_stride < (int64_t)a->heads * (a->dim + a->rot))
    return DZ_ERR_INVALID_ARG;
  if ((a->q_out || a->l_off >= 0) && a->rank <= 0) return DZ_ERR_INVALID_ARG;
  if (a->l_off >= 0 && (!a->norm_weight || !a->cache || !a->slots || a->row_stride < (int64_t)a->l_off + a->rank + a->rot))
    return DZ_ERR_INVALID_ARG;
  if (a->rot > 8192) return DZ_ERR_SHAPE;
  if (a->rows == 0) return DZ_OK;
  RowParams p = {a->x, a->row_stride, (const long long*)a->positions, a->freq, a->heads, a->dim, a->rot, a->q_out, a->l_off,
                 a->rank, a->norm_weight, a->eps, a->cache, (const long long*)a->slots};
  const bool pairs = a->dim % 2 == 0 && a->row_stride % 2 == 0 && ((a->q_out == nullptr && a->l_off < 0) || a->rank % 2 == 0) &&
                     (a->l_off < 0 || a->l_off % 2 == 0) && aligned16(a->x) && aligned16(a->q_out) && aligned16(a->cache);
  const bool vec = pairs && a->dim % 8 == 0 && a->rot % 8 == 0 && a->row_stride % 8 == 0 &&
                   ((a->q_out == nullptr && a->l_off < 0) || a->rank % 8 == 0) &&
                   (a->l_off < 0 || (a->l_off % 8 == 0 && aligned16(a->norm_weight)));
  DZ_DISPATCH(a->dtype, DZ_CUDA_OK(launch_ex(vec     ? latent_rows_kernel<T, true, true>
                                             : pairs ? latent_rows_kernel<T, true, false>
                                                     : latent_rows_kernel<T, false, false>,
                                             dim3(a->rows), dim3(kRowThreads), (size_t)(a->rot / 2) * 8, 1,
                                             (cudaStream_t)stream, p)));
  return DZ_OK;
}

int dz_latent_gather(const void* cache, const int32_t* block_tables, int table_width, int block_size, const int32_t* starts,
                     int num_seqs, int max_len, void* out, int row_size, int dtype, void* stream) {
  if (!cache || !block_tables || !starts || !out || table_width <= 0 || block_size <= 0 || num_seqs < 0 || max_len < 0 ||
      row_size <= 0 || !is_float_dtype(dtype))
    return DZ_ERR_INVALID_ARG;
  if (num_seqs > 65535) return DZ_ERR_SHAPE;
  if (num_seqs == 0 || max_len == 0) return DZ_OK;
  const size_t bytes = (size_t)row_size * (dtype == DZ_DTYPE_F32 ? 4 : 2);
  const dim3 grid((max_len + 7) / 8, num_seqs);
  cudaStream_t st = (cudaStream_t)stream;
  if (bytes % 16 == 0 && aligned16(cache) && aligned16(out)) {
    DZ_CUDA_OK(launch_pdl(latent_gather_kernel<uint4>, grid, dim3(256), st, (const uint4*)cache, block_tables, table_width,
                          block_size, starts, (uint4*)out, (int)(bytes / 16)));
  } else {
    DZ_CUDA_OK(launch_pdl(latent_gather_kernel<uint16_t>, grid, dim3(256), st, (const uint16_t*)cache, block_tables,
                          table_width, block_size, starts, (uint16_t*)out, (int)(bytes / 2)));
  }
  return DZ_OK;
}

// CTAs of one split of a launch: what a caller balances the number of splits with (0: no such kernel).
int dz_latent_attention_ctas(int rows, int heads, int rank, int rot, int dtype) {
  if (rows <= 0 || heads <= 0 || rank <= 0 || rot <= 0 || !tensor_core_shapes(heads, rank, rot, dtype)) return 0;
  return rows * head_groups(heads);
}

size_t dz_latent_attention_workspace_bytes(int rows, int heads, int rank, int splits) {
  if (rows <= 0 || heads <= 0 || rank <= 0 || splits <= 1) return 0;
  return kTicketBytes + (size_t)rows * heads * splits * partial_row(rank) * 4;
}

int dz_latent_attention(const dz_latent_attention_args* a, void* stream) {
  if (!a || !a->q || !a->cache || !a->block_tables || !a->q_starts || !a->ctx_lens || !a->out) return DZ_ERR_INVALID_ARG;
  if (a->num_seqs < 0 || a->rows < 0 || a->heads <= 0 || a->rank <= 0 || a->rot <= 0 || a->table_width <= 0 ||
      a->block_size <= 0 || a->splits < 1 || a->splits > 64 || !is_float_dtype(a->dtype))
    return DZ_ERR_INVALID_ARG;
  if (a->num_seqs == 0 || a->rows == 0) return DZ_OK;
  if (a->rows > 65535) return DZ_ERR_SHAPE;
  cudaStream_t st = (cudaStream_t)stream;
  const int d = a->rank + a->rot;
  if (!tensor_core_shapes(a->heads, a->rank, a->rot, a->dtype) || !aligned16(a->q) || !aligned16(a->cache) || !aligned16(a->out)) {
    AttnParams p = {};
    p.qkv = p.kv = a->q;
    p.row_stride = p.kv_stride = (int64_t)a->heads * d;
    p.out = a->out;
    p.k_cache = p.v_cache = a->cache;
    p.v_row = d;
    p.block_tables = a->block_tables;
    p.ring_blocks = a->table_width;
    p.block_size = a->block_size;
    p.q_starts = a->q_starts;
    p.ctx_lens = a->ctx_lens;
    p.heads = a->heads;
    p.kv_heads = 1;
    p.dim = d;
    p.vdim = a->rank;
    p.scale = a->scale;
    p.rows = p.kv_rows = a->rows;
    p.sink = a->sink;
    p.source = kKeysCached;
    return launch_attention_any(p, a->num_seqs, a->dtype, st);
  }
  LatentParams p = {a->q, a->cache, a->block_tables, a->table_width, a->block_size, a->q_starts, a->ctx_lens, a->num_seqs,
                    a->rows, a->heads, a->rank, a->rot, a->scale, a->sink, a->out, a->splits, nullptr, nullptr,
                    a->cache_rows, a->status};
  if (a->splits > 1) {
    if (!a->workspace || a->workspace_bytes < dz_latent_attention_workspace_bytes(a->rows, a->heads, a->rank, a->splits))
      return DZ_ERR_WORKSPACE;
    p.tickets = (int*)a->workspace;
    p.partial = (float*)((uint8_t*)a->workspace + kTicketBytes);
    if ((int64_t)a->rows * head_groups(a->heads) > kMaxTickets) return DZ_ERR_TOO_LARGE;
  }
  if (latent_tc_supported(p, a->dtype)) return launch_latent_tc(p, a->dtype, st);
  DZ_DISPATCH16(a->dtype, return head_tiles(a->heads) == 1 ? run_latent<T, 1>(p, st) : run_latent<T, 2>(p, st));
  return DZ_OK;
}

}  // extern "C"
