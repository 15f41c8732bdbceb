// Routed experts.  An entry is one (token, choice); entries are put in expert order on the device (nothing
// is read back), and a grouped GEMM runs every expert's matrix over its rows.
//
// The GEMM on tcgen05: 128 rows of an expert's matrix are the MMA's M, up to 256 of its entries the N, so a
// decode batch (a few rows per expert) and a prompt batch take the same kernel with different tile widths.
// Tiles (expert, rows of the matrix, entries) are dealt round-robin to one persistent CTA per SM, entries
// first, so that the CTAs running at a time share matrix tiles in L2; an expert's entries are cut into tiles
// of equal width.  Roles: a TMA warp (matrix tile and
// entry tile per 64-wide k step into a ring), an MMA warp (two TMEM accumulators), four epilogue warps
// (scale, activation, store) that drain one accumulator while the next tile fills the other.  Tiles may run
// past an expert's rows or entries: what is computed there is not stored.  All waits are bounded.
#include <algorithm>

#include "dz_elem.cuh"
#include "dz_tc.cuh"

namespace dz {
namespace {

// -------------------------------------------------------------------------------------------------
// Choice of experts: a warp per token.  Every round takes the largest logit that comes after the one
// before in (logit descending, number ascending) order.
// -------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
moe_route_kernel(const float* __restrict__ logits, int M, int experts, int top, int* __restrict__ ids,
                 float* __restrict__ scores) {
  pdl_wait();
  pdl_launch();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= M) return;
  const float* z = logits + (size_t)row * experts;
  float last = INFINITY;
  int last_i = -1;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int best_i = 0x7fffffff;
    for (int i = lane; i < experts; i += 32) {
      const float v = z[i];
      const bool after = v < last || (v == last && i > last_i);
      if (after && (v > best || best_i == 0x7fffffff)) { best = v; best_i = i; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float v = __shfl_xor_sync(0xffffffffu, best, o);
      const int i = __shfl_xor_sync(0xffffffffu, best_i, o);
      if (i != 0x7fffffff && (best_i == 0x7fffffff || v > best || (v == best && i < best_i))) { best = v; best_i = i; }
    }
    if (lane == 0) {
      const bool ok = best_i != 0x7fffffff;
      ids[(size_t)row * top + j] = ok ? best_i : -1;
      scores[(size_t)row * top + j] = ok ? 1.f / (1.f + expf(-best)) : 0.f;
    }
    last = best;
    last_i = best_i;
  }
}

// -------------------------------------------------------------------------------------------------
// Stable counting sort: a CTA per expert reads all ids twice -- how many come before its rows, then
// where each of its own goes.
// -------------------------------------------------------------------------------------------------
constexpr int kSortThreads = 1024, kSortPer = 4;

__global__ void __launch_bounds__(kSortThreads)
moe_sort_kernel(const int* __restrict__ ids, const float* __restrict__ scores, int entries, int experts,
                int* __restrict__ offsets, int* __restrict__ place, int* __restrict__ order, float* __restrict__ sorted) {
  __shared__ int s_warp[32], s_less[32];
  const int e = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_wait();
  pdl_launch();
  int less = 0, mine = 0;
  for (int i = tid; i < entries; i += kSortThreads) {
    const int id = ids[i];
    less += id >= 0 && id < e;
    mine += id == e;
    if (e == 0 && (id < 0 || id >= experts)) place[i] = -1;
  }
  less = __reduce_add_sync(0xffffffffu, less);
  mine = __reduce_add_sync(0xffffffffu, mine);
  if (lane == 0) { s_less[warp] = less; s_warp[warp] = mine; }
  __syncthreads();
  less = __reduce_add_sync(0xffffffffu, s_less[lane]);
  mine = __reduce_add_sync(0xffffffffu, s_warp[lane]);
  __syncthreads();
  if (tid == 0) offsets[e] = less;
  if (e == experts - 1) {
    if (tid == 0) offsets[experts] = less + mine;
    for (int i = less + mine + tid; i < entries; i += kSortThreads) order[i] = -1;
  }
  if (mine == 0) return;
  int at = less;
  for (int base = 0; base < entries; base += kSortThreads * kSortPer) {
    const int i0 = base + tid * kSortPer;
    int n = 0;
#pragma unroll
    for (int j = 0; j < kSortPer; ++j) n += i0 + j < entries && ids[i0 + j] == e;
    int before = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += up;
    }
    if (lane == 31) s_warp[warp] = before;
    __syncthreads();
    const int w = s_warp[lane];
    const int ahead = __reduce_add_sync(0xffffffffu, lane < warp ? w : 0), all = __reduce_add_sync(0xffffffffu, w);
    int to = at + ahead + before - n;
#pragma unroll
    for (int j = 0; j < kSortPer; ++j)
      if (i0 + j < entries && ids[i0 + j] == e) {
        place[i0 + j] = to;
        order[to] = i0 + j;
        sorted[to] = scores[i0 + j];
        ++to;
      }
    at += all;
    __syncthreads();
  }
}

template <typename V>
__global__ void __launch_bounds__(128)
moe_gather_kernel(const V* __restrict__ x, const int* __restrict__ order, int top, V* __restrict__ out, int units) {
  pdl_wait();
  pdl_launch();
  const int entry = order[blockIdx.x];
  if (entry < 0) return;
  const V* src = x + (size_t)(entry / top) * units;
  V* dst = out + (size_t)blockIdx.x * units;
  for (int i = threadIdx.x; i < units; i += 128) dst[i] = src[i];
}

// -------------------------------------------------------------------------------------------------
// Grouped GEMM
// -------------------------------------------------------------------------------------------------
struct MoeParams {
  const void* x;                         // [rows, K] sorted
  const void* weights;                   // [experts, N, K]
  const int* offsets;
  const float* scale;
  void* y;                               // [rows, N]
  int rows, N, K, experts, act;
  int nt, stages, tmem_cols;             // tensor-core form: entries per tile, ring size
  int* status;
};

template <int ACT> __device__ __forceinline__ float moe_act(float v) {
  if (ACT == DZ_ACT_RELU2) return v > 0.f ? v * v : 0.f;
  if (ACT == DZ_ACT_SILU) return v / (1.f + expf(-v));
  if (ACT == DZ_ACT_GELU_TANH) return 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
  return v;
}

// Any type, any sizes: 32 entries x 64 matrix rows per CTA, 32 of K at a time.
constexpr int kAnyE = 32, kAnyN = 64, kAnyK = 32;

template <typename T, int ACT>
__global__ void __launch_bounds__(256)
moe_gemm_any_kernel(MoeParams p) {
  __shared__ float sx[kAnyK][kAnyE + 1], sw[kAnyK][kAnyN + 1];
  __shared__ int s_e, s_row, s_end;
  pdl_wait();
  pdl_launch();
  const int tid = threadIdx.x;
  if (tid == 0) {
    int left = blockIdx.y;
    s_e = -1;
    for (int e = 0; e < p.experts; ++e) {
      const int o = p.offsets[e], n = p.offsets[e + 1] - o, tiles = (n + kAnyE - 1) / kAnyE;
      if (left < tiles) {
        s_e = e;
        s_row = o + left * kAnyE;
        s_end = o + n;
        break;
      }
      left -= tiles;
    }
  }
  __syncthreads();
  if (s_e < 0) return;
  const int row0 = s_row, end = s_end, n0 = blockIdx.x * kAnyN;
  const T* x = (const T*)p.x;
  const T* w = (const T*)p.weights + (size_t)s_e * p.N * p.K;
  const int tx = tid & 15, ty = tid >> 4;
  float acc[2][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += kAnyK) {
    for (int i = tid; i < kAnyK * kAnyE; i += 256) {
      const int r = i / kAnyK, k = i % kAnyK;
      sx[k][r] = row0 + r < end && k0 + k < p.K ? Cvt<T>::one(x[(size_t)(row0 + r) * p.K + k0 + k]) : 0.f;
    }
    for (int i = tid; i < kAnyK * kAnyN; i += 256) {
      const int r = i / kAnyK, k = i % kAnyK;
      sw[k][r] = n0 + r < p.N && k0 + k < p.K ? Cvt<T>::one(w[(size_t)(n0 + r) * p.K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < kAnyK; ++k) {
      const float a0 = sx[k][ty], a1 = sx[k][ty + 16];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float b = sw[k][tx + 16 * j];
        acc[0][j] += a0 * b;
        acc[1][j] += a1 * b;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int row = row0 + ty + 16 * i;
    if (row >= end) continue;
    const float sc = p.scale ? p.scale[row] : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      if (n < p.N) ((T*)p.y)[(size_t)row * p.N + n] = Cvt<T>::from(moe_act<ACT>(acc[i][j] * sc));
    }
  }
}

constexpr int kMoeThreads = 192, kMaxStages = 10, kMaxExperts = 1024;    // warp 0 TMA, 1 MMA + TMEM, 2..5 epilogue
constexpr int kWTile = 128 * 128;                                         // bytes of 128 matrix rows x 64 k

constexpr int kXBox = 64;                                                 // entries per copy

struct Tile { int e, row, count, n0; };

template <typename T, int ACT>
__global__ void __launch_bounds__(kMoeThreads, 1)
moe_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const MoeParams p) {
  constexpr int DT = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
  extern __shared__ uint8_t smem_dyn[];
  __shared__ __align__(8) uint64_t s_full[kMaxStages], s_empty[kMaxStages], s_acc_full[2], s_acc_empty[2];
  __shared__ int s_off[kMaxExperts + 1], s_first[kMaxExperts + 1];        // first row, first tile of every expert
  __shared__ int s_abort;
  __shared__ uint32_t s_tmem_base;
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  const uint32_t s_w = (smem_u32(smem_dyn) + 1023u) & ~1023u;
  const uint32_t x_bytes = p.nt * 128, s_x = s_w + p.stages * kWTile;
  if (threadIdx.x == 0) {
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(smem_u32(&s_full[i]), 1);
      mbar_init(smem_u32(&s_empty[i]), 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(smem_u32(&s_acc_full[i]), 1);
      mbar_init(smem_u32(&s_acc_empty[i]), 128);
    }
    s_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    fence_proxy_async();
    asm volatile("prefetch.tensormap [%0];" ::"l"(&map_w) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&map_x) : "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem_base)),
                 "r"(p.tmem_cols)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_wait();
  pdl_launch();
  const int tiles_n = (p.N + 127) / 128;
  for (int i = threadIdx.x; i <= p.experts; i += kMoeThreads) s_off[i] = p.offsets[i];
  __syncthreads();
  if (warp == 0) {                                                        // prefix sum of the experts' tiles
    int carry = 0;
    for (int b = 0; b < p.experts; b += 32) {
      const int e = b + lane;
      int n = e < p.experts ? (s_off[e + 1] - s_off[e] + p.nt - 1) / p.nt * tiles_n : 0;
      const int own = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, n, o);
        if (lane >= o) n += up;
      }
      if (e < p.experts) s_first[e] = carry + n - own;
      carry += __shfl_sync(0xffffffffu, n, 31);
    }
    if (lane == 0) s_first[p.experts] = carry;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const int total = s_first[p.experts];
  const int ksteps = (p.K + kBlockK - 1) / kBlockK;
  const uint32_t tmem_base = s_tmem_base;
  volatile int* abort_flag = &s_abort;
  auto tile = [&](int vt) {
    int lo = 0, hi = p.experts;                                           // s_first[lo] <= vt < s_first[hi]
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (s_first[mid] <= vt) lo = mid; else hi = mid;
    }
    // as few tiles as hold the expert's entries, of equal width
    const int rows = s_off[lo + 1] - s_off[lo], across = (rows + p.nt - 1) / p.nt, i = vt - s_first[lo];
    const int t = i % across, width = ((rows + across - 1) / across + 15) / 16 * 16;
    return Tile{lo, s_off[lo] + t * width, min(width, rows - t * width), i / across * 128};
  };

  if (warp == 0) {
    Ring r(p.stages, 1);
    for (int vt = blockIdx.x; vt < total; vt += gridDim.x) {
      const Tile t = tile(vt);
      const int wrow = t.e * p.N + t.n0, box = min(kXBox, p.nt), boxes = (t.count + box - 1) / box;
      for (int ks = 0; ks < ksteps; ++ks) {
        mbar_wait(smem_u32(&s_empty[r.idx]), r.par, abort_flag, p.status);
        __syncwarp();
        const uint32_t full = smem_u32(&s_full[r.idx]);
        warp_mbar_expect_tx(full, kWTile + boxes * box * 128);
        warp_tma_load_2d(s_w + r.idx * kWTile, &map_w, ks * kBlockK, wrow, full);
        for (int b = 0; b < boxes; ++b)
          warp_tma_load_2d(s_x + r.idx * x_bytes + b * box * 128, &map_x, ks * kBlockK, t.row + b * box, full);
        r.advance();
      }
    }
  } else if (warp == 1) {
    Ring r(p.stages, 0);
    int it = 0;
    for (int vt = blockIdx.x; vt < total; vt += gridDim.x, ++it) {
      const int a = it & 1;
      const uint32_t idesc = make_idesc<DT>((tile(vt).count + 15) / 16 * 16, false), acc = tmem_base + a * p.nt;
      mbar_wait(smem_u32(&s_acc_empty[a]), ((it >> 1) & 1) ^ 1, abort_flag, p.status);
      tc_fence_after();
      for (int ks = 0; ks < ksteps; ++ks) {
        mbar_wait(smem_u32(&s_full[r.idx]), r.par, abort_flag, p.status);
        __syncwarp();
        tc_fence_after();
        const uint32_t w = desc_lo(s_w + r.idx * kWTile), x = desc_lo(s_x + r.idx * x_bytes);
#pragma unroll
        for (int k = 0; k < 4; ++k) warp_umma_ss(acc, w + 2 * k, x + 2 * k, idesc, ks > 0 || k > 0);
        warp_umma_commit(smem_u32(&s_empty[r.idx]));
        r.advance();
      }
      warp_umma_commit(smem_u32(&s_acc_full[a]));
    }
  } else {
    const int q = warp & 3;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(q * 32) << 16);
    int it = 0;
    for (int vt = blockIdx.x; vt < total; vt += gridDim.x, ++it) {
      const int a = it & 1;
      const Tile t = tile(vt);
      const int n = t.n0 + q * 32 + lane;
      T* y = (T*)p.y + (size_t)t.row * p.N + n;
      mbar_wait(smem_u32(&s_acc_full[a]), (it >> 1) & 1, abort_flag, p.status);
      tc_fence_after();
      for (int c8 = 0; c8 < t.count; c8 += 8) {
        uint32_t v[8];
        tmem_ld8(lane_addr + a * p.nt + c8, v);
        tmem_wait_ld();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          if (c8 + i < t.count && n < p.N) {
            float f = __uint_as_float(v[i]);
            if (p.scale) f *= p.scale[t.row + c8 + i];
            y[(size_t)(c8 + i) * p.N] = Cvt<T>::from(moe_act<ACT>(f));
          }
        }
      }
      tc_fence_before();
      mbar_arrive(smem_u32(&s_acc_empty[a]));
    }
  }

  tc_fence_before();
  __syncthreads();
  if (s_abort) {                                                          // let copies and MMAs under way end
    const unsigned long long t0 = globaltimer();
    while (globaltimer() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(p.tmem_cols) : "memory");
  }
}

template <typename T, int ACT>
int run_any(const MoeParams& p, cudaStream_t st) {
  const int64_t most = (int64_t)std::min(p.experts, p.rows) + p.rows / kAnyE;        // token tiles there can be
  if (most > 65535) return DZ_ERR_SHAPE;
  DZ_CUDA_OK(launch_pdl(moe_gemm_any_kernel<T, ACT>, dim3((p.N + kAnyN - 1) / kAnyN, (unsigned)most), dim3(256), st, p));
  return DZ_OK;
}

template <typename T, int ACT>
int run_tc(MoeParams p, int typical, cudaStream_t st) {
  constexpr int kDt = std::is_same<T, __nv_bfloat16>::value;
  p.nt = 16;
  while (p.nt < 256 && p.nt < typical) p.nt *= 2;
  p.stages = std::min<int>(kMaxStages, (200 * 1024) / (kWTile + p.nt * 128));
  p.tmem_cols = std::max(32, 2 * p.nt);
  CUtensorMap map_w, map_x;
  int rc = make_map(&map_w, p.weights, p.experts * p.N, p.K, 128, kDt);
  if (!rc) rc = make_map(&map_x, p.x, p.rows, p.K, std::min(p.nt, kXBox), kDt);
  if (rc) return rc;
  int dev = 0, sms = 0;
  DZ_CUDA_OK(cudaGetDevice(&dev));
  DZ_CUDA_OK(cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev));
  const size_t smem = (size_t)p.stages * (kWTile + p.nt * 128) + 1024;
  DZ_CUDA_OK(allow_smem(moe_gemm_tc_kernel<T, ACT>, smem));
  DZ_CUDA_OK(launch_ex(moe_gemm_tc_kernel<T, ACT>, dim3(sms), dim3(kMoeThreads), smem, 1, st, map_w, map_x, p));
  return DZ_OK;
}

template <typename T, int ACT>
int run_gemm(const MoeParams& p, int typical, cudaStream_t st) {
  if constexpr (sizeof(T) == 2) {
    if (p.K % 8 == 0 && p.experts <= kMaxExperts && (int64_t)p.experts * p.N < (1ll << 31) && aligned16(p.x) &&
        aligned16(p.weights))
      return run_tc<T, ACT>(p, typical, st);
  }
  return run_any<T, ACT>(p, st);
}

}  // namespace
}  // namespace dz

using namespace dz;

extern "C" {

int dz_moe_route(const float* logits, int M, int experts, int top, int32_t* ids, float* scores, void* stream) {
  if (!logits || !ids || !scores || M < 0 || experts <= 0 || top <= 0 || top > experts) return DZ_ERR_INVALID_ARG;
  if (M == 0) return DZ_OK;
  DZ_CUDA_OK(launch_pdl(moe_route_kernel, dim3((M + 7) / 8), dim3(256), (cudaStream_t)stream, logits, M, experts, top, ids,
                        scores));
  return DZ_OK;
}

int dz_moe_sort(const int32_t* ids, const float* scores, int entries, int experts, int32_t* offsets, int32_t* place,
                int32_t* order, float* sorted_scores, void* stream) {
  if (!ids || !scores || !offsets || !place || !order || !sorted_scores || entries < 0 || experts <= 0 || experts > 65535)
    return DZ_ERR_INVALID_ARG;
  DZ_CUDA_OK(launch_pdl(moe_sort_kernel, dim3(experts), dim3(kSortThreads), (cudaStream_t)stream, ids, scores, entries,
                        experts, offsets, place, order, sorted_scores));
  return DZ_OK;
}

int dz_moe_gather(const void* x, const int32_t* order, int entries, int top, void* out, int width, int dtype, void* stream) {
  if (!x || !order || !out || entries < 0 || top <= 0 || width <= 0 || !is_float_dtype(dtype)) return DZ_ERR_INVALID_ARG;
  if (entries == 0) return DZ_OK;
  const size_t bytes = (size_t)width * (dtype == DZ_DTYPE_F32 ? 4 : 2);
  cudaStream_t st = (cudaStream_t)stream;
  if (bytes % 16 == 0 && aligned16(x) && aligned16(out)) {
    DZ_CUDA_OK(launch_pdl(moe_gather_kernel<uint4>, dim3(entries), dim3(128), st, (const uint4*)x, order, top, (uint4*)out,
                          (int)(bytes / 16)));
  } else {
    DZ_CUDA_OK(launch_pdl(moe_gather_kernel<uint16_t>, dim3(entries), dim3(128), st, (const uint16_t*)x, order, top,
                          (uint16_t*)out, (int)(bytes / 2)));
  }
  return DZ_OK;
}

int dz_moe_gemm(const void* x, const void* weights, const int32_t* offsets, const float* scale, void* y, int rows, int N,
                int K, int experts, int act, int typical, int dtype, int* status, void* stream) {
  if (!x || !weights || !offsets || !y || rows < 0 || N <= 0 || K <= 0 || experts <= 0 || !is_float_dtype(dtype))
    return DZ_ERR_INVALID_ARG;
  if (rows == 0) return DZ_OK;
  const MoeParams p = {x, weights, offsets, scale, y, rows, N, K, experts, act, 0, 0, 0, status};
  cudaStream_t st = (cudaStream_t)stream;
  switch (act) {
    case DZ_ACT_NONE: DZ_DISPATCH(dtype, return (run_gemm<T, DZ_ACT_NONE>(p, typical, st))); break;
    case DZ_ACT_RELU2: DZ_DISPATCH(dtype, return (run_gemm<T, DZ_ACT_RELU2>(p, typical, st))); break;
    case DZ_ACT_SILU: DZ_DISPATCH(dtype, return (run_gemm<T, DZ_ACT_SILU>(p, typical, st))); break;
    case DZ_ACT_GELU_TANH: DZ_DISPATCH(dtype, return (run_gemm<T, DZ_ACT_GELU_TANH>(p, typical, st))); break;
  }
  return DZ_ERR_INVALID_ARG;
}

}  // extern "C"
