// Small device helpers shared by the decoder-layer kernels: conversions between the storage types
// and float, reductions, asynchronous copies, the 16-bit warp MMA and launches with programmatic
// stream serialization.
#pragma once

#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <math.h>

#include "dz_common.cuh"

namespace dz {

template <typename T> struct Cvt;
template <> struct Cvt<__half> {
  static __device__ __forceinline__ float2 up(uint32_t v) {
    return __half22float2(*reinterpret_cast<const __half2*>(&v));
  }
  static __device__ __forceinline__ uint32_t down(float a, float b) {
    __half2 h = __floats2half2_rn(a, b);
    return *reinterpret_cast<uint32_t*>(&h);
  }
  static __device__ __forceinline__ float round(float a) { return __half2float(__float2half_rn(a)); }
  static __device__ __forceinline__ float one(__half v) { return __half2float(v); }
  static __device__ __forceinline__ __half from(float v) { return __float2half_rn(v); }
};
template <> struct Cvt<__nv_bfloat16> {
  static __device__ __forceinline__ float2 up(uint32_t v) {
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v));
  }
  static __device__ __forceinline__ uint32_t down(float a, float b) {
    __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<uint32_t*>(&h);
  }
  static __device__ __forceinline__ float round(float a) {
    return __bfloat162float(__float2bfloat16_rn(a));
  }
  static __device__ __forceinline__ float one(__nv_bfloat16 v) { return __bfloat162float(v); }
  static __device__ __forceinline__ __nv_bfloat16 from(float v) { return __float2bfloat16_rn(v); }
};
template <> struct Cvt<float> {
  static __device__ __forceinline__ float one(float v) { return v; }
  static __device__ __forceinline__ float from(float v) { return v; }
};

// Eight consecutive elements as floats (the address is a multiple of eight elements).
template <typename T> __device__ __forceinline__ void load8(const T* p, float (&f)[8]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 v = Cvt<T>::up(w[j]);
    f[2 * j] = v.x;
    f[2 * j + 1] = v.y;
  }
}
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
template <typename T> __device__ __forceinline__ void store8(T* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(Cvt<T>::down(f[0], f[1]), Cvt<T>::down(f[2], f[3]),
                                            Cvt<T>::down(f[4], f[5]), Cvt<T>::down(f[6], f[7]));
}
template <> __device__ __forceinline__ void store8<float>(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Sum over the block (a multiple of 32 threads, at most 1024); `part` holds one float per warp.
// Every thread of the block must call it; it starts and ends with the block in step.
__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += part[i];
  return t;
}

__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

// -- 16-byte asynchronous copies into shared memory (zero-filled when `ok` is false) -------------
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(ok ? 16 : 0)
               : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// -- warp-level 16-bit MMA, 32-bit accumulation ----------------------------------------------------
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)) : "memory");
}
__device__ __forceinline__ void ldsm2_t(uint32_t& r0, uint32_t& r1, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];"
               : "=r"(r0), "=r"(r1) : "r"(smem_addr(p)) : "memory");
}
template <typename T>
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1);
template <>
__device__ __forceinline__ void mma16816<__nv_bfloat16>(float (&c)[4], const uint32_t (&a)[4], uint32_t b0,
                                                        uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
template <>
__device__ __forceinline__ void mma16816<__half>(float (&c)[4], const uint32_t (&a)[4], uint32_t b0,
                                                 uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// A pair of floats as hi + lo 16-bit pairs (together about twice the mantissa of one): 32-bit
// quantities enter an MMA as two products.
template <typename T>
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = Cvt<T>::down(a, b);
  const float2 h = Cvt<T>::up(hi);
  lo = Cvt<T>::down(a - h.x, b - h.y);
}

// -- launches --------------------------------------------------------------------------------------
template <typename K, typename... Args>
cudaError_t launch_ex(K kern, dim3 grid, dim3 block, size_t smem, int cluster_x, cudaStream_t st, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = cluster_x;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = cluster_x > 1 ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, kern, args...);
}
template <typename K, typename... Args>
cudaError_t launch_pdl(K kern, dim3 grid, dim3 block, cudaStream_t st, Args... args) {
  return launch_ex(kern, grid, block, 0, 1, st, args...);
}
// Dynamic shared memory above 48 KB has to be granted per kernel and device; the attribute is
// cheap to set, so it is set before every such launch.
template <typename K> inline cudaError_t allow_smem(K kern, size_t bytes) {
  if (bytes <= 48 * 1024) return cudaSuccess;
  return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}
constexpr size_t kMaxDynSmem = 220 * 1024;

// Workspaces that hold both tickets (zero between launches) and other scratch start with the tickets,
// and with room for this many whatever the launch needs: no launch's scratch may lie where the tickets of
// another one of the same workspace are.
constexpr int kMaxTickets = 65536;
constexpr size_t kTicketBytes = (size_t)kMaxTickets * 4;

inline bool is_float_dtype(int d) { return d == DZ_DTYPE_F16 || d == DZ_DTYPE_BF16 || d == DZ_DTYPE_F32; }

}  // namespace dz

// Runs STMT with `T` bound to the storage type of a DZ_DTYPE_* code.
#define DZ_DISPATCH(dtype, ...)                                              \
  switch (dtype) {                                                           \
    case DZ_DTYPE_F16: { using T = __half; __VA_ARGS__; break; }             \
    case DZ_DTYPE_BF16: { using T = __nv_bfloat16; __VA_ARGS__; break; }     \
    case DZ_DTYPE_F32: { using T = float; __VA_ARGS__; break; }              \
    default: return DZ_ERR_INVALID_ARG;                                      \
  }
#define DZ_DISPATCH16(dtype, ...)                                            \
  switch (dtype) {                                                           \
    case DZ_DTYPE_F16: { using T = __half; __VA_ARGS__; break; }             \
    case DZ_DTYPE_BF16: { using T = __nv_bfloat16; __VA_ARGS__; break; }     \
    default: return DZ_ERR_INVALID_ARG;                                      \
  }
