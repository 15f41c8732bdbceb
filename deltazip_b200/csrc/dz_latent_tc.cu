// Attention over cached latents on the 5th-generation tensor cores: up to 32 heads of one row against a
// share of its sequence's cached rows [c | r], 64 per tile, two tiles in shared memory.
//
//   scores   S [heads, keys]      = Q K^T     Q and K as they lie, 64 columns of the row per slab
//   sums     O^T [latent, heads] += V^T P^T   V = the rows' first `rank` columns, read where they lie
//                                             ("MN-major"), 128 of them per MMA tile
//
// With the heads along N the sums fit the tensor memory beside the scores and the MMAs are as long as there
// are heads.  A weight is a hi + lo pair of 16-bit numbers; the his and the los are neighbouring columns of
// one MMA, so that V is read once for both, and their sums are added at the end.  The scores' M is 128 with
// the heads in the first lanes; what the others hold comes from whatever lies behind Q and is never read.
//
// Roles: warps 0 and 4 softmax (a lane owns a head, a warp half of a tile's keys: scores from TMEM, running
// maximum, exponentials, weights into shared memory), warps 1 and 3 copies (half of the columns each; TMA,
// one box per slab and run of rows that lie together in a page), warp 2 MMA issue, warps 8-11 rescaling of
// the sums (rare: the maximum is moved only when it has grown by more than 2^8).  All waits are bounded.
#include <algorithm>
#include <numeric>

#include "dz_latent.cuh"
#include "dz_tc.cuh"

namespace dz {
namespace {

constexpr int kTile = 64, kRing = 2, kTcThreads = 384, kTcHeads = 32, kMaxTiles = 4;   // tiles of 128 latent columns
constexpr int kSlabK = kTile * 128, kSlabH = kTcHeads * 128;                           // bytes: 64 keys, 32 heads x 64 columns
constexpr float kGrowth = 8.f, kLog2 = 1.4426950408889634f;
constexpr int kTmemCols = 512, kTmemO = 2 * kTile, kPairs = 2 * kTcHeads;              // S, S | O^T (hi | lo) per 128 of the latent

template <typename T>
__global__ void __launch_bounds__(kTcThreads, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                        const LatentParams p, int run) {
  constexpr int DT = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
  extern __shared__ uint8_t smem_dyn[];
  __shared__ uint64_t b_full[kRing][2], b_empty[kRing], b_s[2], b_dec[2], b_p[2], b_pv[2], b_o, b_q, b_tail[2];
  __shared__ float s_f[kTcHeads], s_out[kTcHeads], s_top[2][2][kTcHeads], s_sum[kTcHeads];
  __shared__ int s_need[2], s_seq, s_abort, s_last;
  __shared__ uint32_t s_tmem;
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;
  const int h0 = blockIdx.x * kTcHeads, row = blockIdx.y, split = blockIdx.z, live = min(kTcHeads, p.heads - h0);
  const int d = p.rank + p.rot, slabs = (d + 63) / 64, tiles_m = (p.rank + 127) / 128;
  const int hn = p.heads <= 16 ? 16 : 32;                              // the MMAs' N
  const int stage = slabs * kSlabK;
  const uint32_t s_k = (smem_u32(smem_dyn) + 1023u) & ~1023u, s_q = s_k + kRing * stage, s_p = s_q + slabs * kSlabH;
  volatile int* abort_flag = &s_abort;
  if (tid == 0) {
    for (int i = 0; i < kRing; ++i) {
      mbar_init(smem_u32(&b_full[i][0]), 1);
      mbar_init(smem_u32(&b_full[i][1]), 1);
      mbar_init(smem_u32(&b_empty[i]), 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(smem_u32(&b_s[i]), 1);
      mbar_init(smem_u32(&b_dec[i]), 2);
      mbar_init(smem_u32(&b_p[i]), 6);
      mbar_init(smem_u32(&b_pv[i]), 1);
    }
    mbar_init(smem_u32(&b_o), 1);
    mbar_init(smem_u32(&b_q), 1);
    mbar_init(smem_u32(&b_tail[0]), 1);
    mbar_init(smem_u32(&b_tail[1]), 1);
    s_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    fence_proxy_async();
    asm volatile("prefetch.tensormap [%0];" ::"l"(&map_q) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&map_k) : "memory");
  }
  if (warp == 3) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "n"(kTmemCols)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_wait();
  pdl_launch();
  int seq = row, q0 = row;
  if (p.rows != p.num_seqs) {
    for (int s = tid; s < p.num_seqs; s += kTcThreads)
      if (row >= p.q_starts[s] && row < p.q_starts[s + 1]) s_seq = s;
    __syncthreads();
    seq = s_seq;
    q0 = p.q_starts[seq];
  }
  const int n = p.ctx_lens[seq] + row - q0 + 1;                        // keys up to and with the row's own
  const int per = keys_per_split(n, p.splits);
  const int t0 = min(n, split * per), t1 = min(n, t0 + per);
  const int tiles = (t1 - t0 + kTile - 1) / kTile;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = s_tmem;

  const int half = (slabs + 1) / 2;                                    // slabs of the first copy warp
  if (warp == 1 || warp == 3) {
    // ---- copies ----
    const int* table = p.tables + (size_t)seq * p.table_width;
    const int part = warp >> 1, c0 = part ? half : 0, c1 = part ? slabs : half;
    if (tiles > 0 && part == 0) {
      warp_mbar_expect_tx(smem_u32(&b_q), slabs * hn * 128);
      for (int i = 0; i < slabs; ++i) warp_tma_load_2d(s_q + i * kSlabH, &map_q, i * 64, row * p.heads + h0, smem_u32(&b_q));
    }
    for (int j = 0; j < tiles; ++j) {
      const int st = j % kRing, base = t0 + j * kTile, valid = min(kTile, t1 - base);
      const uint32_t dst = s_k + st * stage, full = smem_u32(&b_full[st][part]);
      // the cache row of every run of rows of the tile, a lane each
      const int runs = (valid + run - 1) / run, t = base + lane * run;
      const int at = lane < runs ? table[t / p.block_size] * p.block_size + t % p.block_size : 0;
      bar_wait(&b_empty[st], ((j / kRing) & 1) ^ 1, abort_flag, p.status);
      __syncwarp();
      const bool tail = valid < kTile;
      const uint32_t bar = tail ? smem_u32(&b_tail[part]) : full;      // at most one tile of a CTA is cut
      warp_mbar_expect_tx(bar, runs * run * (c1 - c0) * 128);
      for (int r = 0; r < runs; ++r) {
        const int from = __shfl_sync(0xffffffffu, at, r);
        for (int c = c0; c < c1; ++c) warp_tma_load_2d(dst + c * kSlabK + r * run * 128, &map_k, c * 64, from, bar);
      }
      if (tail) {                                                      // rows past the end must not count: make them zero
        bar_wait(&b_tail[part], 0, abort_flag, p.status);
        for (int i = valid * 8 + lane; i < kTile * 8; i += 32)
          for (int c = c0; c < c1; ++c) sts128(dst + c * kSlabK + i * 16, make_uint4(0, 0, 0, 0));
        fence_proxy_async();
        __syncwarp();
        if (lane == 0) mbar_arrive(full);
      }
    }
  } else if (warp == 2) {
    // ---- MMA issue ----
    if (tiles > 0) {
      const uint32_t id_s = make_idesc<DT>(kTile, false), id_o = make_idesc<DT>(2 * hn, false) | (1u << 15);   // A transposed
      auto scores = [&](int j) {
        const int st = j % kRing;
        const uint32_t a = desc_lo(s_q), b = desc_lo(s_k + st * stage);
        auto slab = [&](int c, int n) {                                // n MMAs of 16 columns
          for (int k = 0; k < n; ++k)
            warp_umma_ss(tmem + (j & 1) * kTile, a + c * (kSlabH >> 4) + k * 2, b + c * (kSlabK >> 4) + k * 2, id_s, c + k > 0);
        };
        for (int part = 0; part < 2; ++part) {
          bar_wait(&b_full[st][part], (j / kRing) & 1, abort_flag, p.status);
          __syncwarp();
          tc_fence_after();
          const int c1 = part ? slabs : half;
          int c = part ? half : 0;
          for (; c < min(c1, d / 64); ++c) slab(c, 4);
          if (c < c1) slab(c, (d % 64 + 15) / 16);
        }
        warp_umma_commit(smem_u32(&b_s[j & 1]));
      };
      bar_wait(&b_q, 0, abort_flag, p.status);
      scores(0);
      for (int j = 0; j < tiles; ++j) {
        const int st = j % kRing, buf = j & 1;
        // the next tile's scores under this one's softmax, if it is here in time
        bool ahead = j + 1 >= tiles;
        for (int i = 0; i < 4096 && !ahead; ++i) {
          if (__any_sync(0xffffffffu, mbar_test(smem_u32(&b_p[buf]), (j >> 1) & 1))) break;
          if (__any_sync(0xffffffffu, mbar_test(smem_u32(&b_full[(j + 1) % kRing][0]), ((j + 1) / kRing) & 1) &&
                                          mbar_test(smem_u32(&b_full[(j + 1) % kRing][1]), ((j + 1) / kRing) & 1))) {
            scores(j + 1);
            ahead = true;
          }
        }
        bar_wait(&b_p[buf], (j >> 1) & 1, abort_flag, p.status);
        __syncwarp();
        tc_fence_after();
        const uint32_t w = desc_lo(s_p + buf * 2 * kSlabH);
        for (int m = 0; m < tiles_m; ++m) {
          const uint32_t v = desc_lo_mn(s_k + st * stage + m * 2 * kSlabK, kSlabK), o = tmem + kTmemO + m * kPairs;
#pragma unroll
          for (int k = 0; k < kTile / 16; ++k)                         // 16 keys: 2048 bytes of v, 32 of p
            warp_umma_ss(o, v + k * 128, w + k * 2, id_o, (j > 0 || k > 0) ? 1u : 0u);
        }
        warp_umma_commit(smem_u32(&b_empty[st]));
        warp_umma_commit(smem_u32(&b_pv[buf]));
        if (!ahead) scores(j + 1);
      }
      warp_umma_commit(smem_u32(&b_o));
    }
  } else if (warp == 0 || warp == 4) {
    // ---- softmax ----
    constexpr int kMine = kTile / 2;
    const int part = warp >> 2;
    const float scale2 = p.scale * kLog2;
    float m = -INFINITY, l = 0.f;
    for (int j = 0; j < tiles; ++j) {
      const int buf = j & 1, valid = min(kTile, t1 - t0 - j * kTile) - part * kMine;
      bar_wait(&b_s[buf], (j >> 1) & 1, abort_flag, p.status);
      __syncwarp();
      tc_fence_after();
      float s[kMine];
      tmem_ld32(tmem + buf * kTile + part * kMine, s);
      tmem_wait_ld();
      if (lane >= live) {                                              // lanes without a head
#pragma unroll
        for (int c = 0; c < kMine; ++c) s[c] = 0.f;
      }
      if (valid < kMine) {
#pragma unroll
        for (int c = 0; c < kMine; ++c) s[c] = c < valid ? s[c] : -INFINITY;
      }
      float mx[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int c = 4; c < kMine; ++c) mx[c & 3] = fmaxf(mx[c & 3], s[c]);
      float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
      s_top[buf][part][lane] = top;
      named_bar_sync(1, 64);
      top = fmaxf(top, s_top[buf][part ^ 1][lane]) * scale2;           // the tile's first key is there: finite
      float f = 1.f;
      if (j == 0) {
        m = top;
      } else if (top > m + kGrowth) {
        f = ex2(m - top);
        m = top;
        l *= f;
      }
      const bool need = __any_sync(0xffffffffu, f != 1.f);             // the same in both warps
      if (j >= 2) bar_wait(&b_pv[buf], ((j >> 1) - 1) & 1, abort_flag, p.status);       // these weights have been used
      const uint32_t ph = s_p + buf * 2 * kSlabH, pl = ph + hn * 128;
      float sum[2] = {0.f, 0.f};
#pragma unroll
      for (int c = 0; c < kMine / 8; ++c) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float a = ex2(fmaf(s[c * 8 + 2 * i], scale2, -m)), b = ex2(fmaf(s[c * 8 + 2 * i + 1], scale2, -m));
          sum[0] += a;
          sum[1] += b;
          split_pair<T>(a, b, hi[i], lo[i]);
        }
        if (lane < hn) {
          const uint32_t at = swizzled(lane, part * (kMine / 8) + c, kSlabH);
          sts128(ph + at, make_uint4(hi[0], hi[1], hi[2], hi[3]));
          sts128(pl + at, make_uint4(lo[0], lo[1], lo[2], lo[3]));
        }
      }
      l += sum[0] + sum[1];
      if (part == 0) {
        s_f[lane] = f;
        if (lane == 0) s_need[buf] = need;
      }
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(smem_u32(&b_dec[buf]));
        mbar_arrive(smem_u32(&b_p[buf]));
      }
      if (need) bar_wait(&b_p[buf], (j >> 1) & 1, abort_flag, p.status);                // s_f is written again next
    }
    if (part == 1) s_sum[lane] = l;
    named_bar_sync(1, 64);
    if (part == 0 && lane < live) {
      l += s_sum[lane];
      float f = 1.f;
      if (p.splits == 1) {
        const float sk2 = p.sink ? p.sink[h0 + lane] * kLog2 : -INFINITY, top = fmaxf(m, sk2), c = exp2f(m - top);
        f = c / (l * c + exp2f(sk2 - top));
      } else {
        float* pp = p.partial + (((size_t)row * p.heads + h0 + lane) * p.splits + split) * partial_row(p.rank) + p.rank;
        pp[0] = m;
        pp[1] = l;
      }
      s_out[lane] = f;
    }
  } else if (warp >= 8) {
    // ---- rescaling ----
    const uint32_t t_o = tmem + kTmemO + ((uint32_t)((warp & 3) * 32) << 16);
    for (int j = 0; j < tiles; ++j) {
      const int buf = j & 1;
      bar_wait(&b_dec[buf], (j >> 1) & 1, abort_flag, p.status);
      if (s_need[buf]) {                                               // never the first tile
        bar_wait(&b_pv[(j - 1) & 1], ((j - 1) >> 1) & 1, abort_flag, p.status);         // O holds the products so far
        tc_fence_after();
        for (int i = 0; i < tiles_m * kPairs; i += kPairs)
          for (int part = 0; part < 2 * hn; part += 32) {               // 32 columns: his, los, or 16 of each
            float o[32];
            tmem_ld32(t_o + i + part, o);
            tmem_wait_ld();
#pragma unroll
            for (int c = 0; c < 32; ++c) o[c] *= s_f[c & (hn - 1)];
            tmem_st16(t_o + i + part, reinterpret_cast<const uint32_t*>(o));
            tmem_st16(t_o + i + part + 16, reinterpret_cast<const uint32_t*>(o + 16));
          }
        tmem_wait_st();
        tc_fence_before();
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&b_p[buf]));
    }
    if (tiles > 0) bar_wait(&b_o, 0, abort_flag, p.status);
  }
  __syncthreads();
  tc_fence_after();
  {
    // ---- output, by all warps ----
    // small loops: this code runs once, and fetching it costs more than running it
    const uint32_t t_o = tmem + kTmemO + ((uint32_t)((warp & 3) * 32) << 16);
    const size_t at = (size_t)row * p.heads + h0;
    const int step = p.splits == 1 ? p.rank : p.splits * partial_row(p.rank);        // from a head to the next
#pragma unroll 1
    for (int i = warp >> 2; i < tiles_m; i += kTcThreads / 128) {
      const int c = i * 128 + (warp & 3) * 32 + lane;
      T* out = (T*)p.out + at * p.rank + c;
      float* part = p.partial + (at * p.splits + split) * partial_row(p.rank) + c;
#pragma unroll 1
      for (int h = 0; h < live; h += 8) {
        uint32_t hi[8], lo[8];
        tmem_ld8(t_o + i * kPairs + h, hi);
        tmem_ld8(t_o + i * kPairs + hn + h, lo);
        tmem_wait_ld();
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float o = tiles > 0 ? __uint_as_float(hi[e]) + __uint_as_float(lo[e]) : 0.f;
          if (h + e < live && c < p.rank) {
            if (p.splits == 1) out[(h + e) * step] = Cvt<T>::from(o * s_out[h + e]);
            else part[(h + e) * step] = o;
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (s_abort) {                                                       // let copies and MMAs under way end
    const unsigned long long t = globaltimer();
    while (globaltimer() - t < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 3) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(kTmemCols) : "memory");
  }
  if (p.splits > 1) merge_splits<T>(p, row, h0, live, &s_last, reinterpret_cast<float*>(smem_dyn));
}

size_t tc_smem(int d) {
  const size_t slabs = (d + 63) / 64;
  // the scores' MMAs read 128 rows from the last slab of Q on, the sums' a whole number of slab pairs
  return slabs * (kRing * kSlabK + kSlabH) + std::max<size_t>(4 * kSlabH, 128 * 128) + 1024;
}

template <typename T>
int run_tc(const LatentParams& p, cudaStream_t st) {
  constexpr int kDt = std::is_same<T, __nv_bfloat16>::value;
  const int d = p.rank + p.rot, hn = p.heads <= 16 ? 16 : 32, run = std::gcd(p.block_size, kTile);
  CUtensorMap map_q, map_k;
  int rc = make_map(&map_q, p.q, p.rows * p.heads, d, hn, kDt);
  if (!rc) rc = make_map(&map_k, p.cache, (int)p.cache_rows, d, run, kDt);
  if (rc) return rc;
  const size_t smem = tc_smem(d);
  DZ_CUDA_OK(allow_smem(latent_decode_tc_kernel<T>, smem));
  DZ_CUDA_OK(launch_ex(latent_decode_tc_kernel<T>, dim3(latent_tc_groups(p.heads), p.rows, p.splits), dim3(kTcThreads), smem, 1,
                       st, map_q, map_k, p, run));
  return DZ_OK;
}

}  // namespace

int latent_tc_groups(int heads) { return (heads + kTcHeads - 1) / kTcHeads; }

bool latent_tc_supported(const LatentParams& p, int dtype) {
  return (dtype == DZ_DTYPE_F16 || dtype == DZ_DTYPE_BF16) && (p.rank + p.rot) % 8 == 0 && p.rank % 8 == 0 &&
         p.rank <= 128 * kMaxTiles && tc_smem(p.rank + p.rot) <= kMaxDynSmem && p.block_size % 8 == 0 && p.scale > 0.f && p.cache_rows > 0 &&
         p.cache_rows < (1ll << 31) && (int64_t)p.rows * p.heads < (1ll << 31) && p.status;
}

int launch_latent_tc(const LatentParams& p, int dtype, cudaStream_t st) {
  return dtype == DZ_DTYPE_BF16 ? run_tc<__nv_bfloat16>(p, st) : run_tc<__half>(p, st);
}

}  // namespace dz
