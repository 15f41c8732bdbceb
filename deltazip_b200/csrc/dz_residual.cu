// Steps around a decoder layer whose residual stream is kept in 32-bit floats: token embedding with
// a norm or a scale, residual update fused with the next sublayer's norm (or with a plain cast, where
// the stream is an operand of a projection itself) and with the sum over a token's routed experts, and
// the activation of a feed-forward, gated or not.
// Norms are x / sqrt(mean(x^2) + eps) * (offset + w): offset 0 is the plain RMS norm, offset 1 the
// form whose weight is stored around zero.  All are passes over [tokens, width] arrays, HBM-bound.
#include "dz_elem.cuh"

namespace dz {
namespace {

constexpr int kThreads = 256;
constexpr int kMaxVec = 8;              // eight-element vectors a thread keeps in registers

// Rows of another matrix that are summed into a token's row: entry j of row r is row
// index[r * count + j] of `rows` (negative: none).
template <typename T> struct RowSum {
  const T* rows;
  const int* index;
  int count;
};

// v = [residual] + [delta] + [vec] + [sum of routed rows]; residual = v; out = norm(v) or v, one CTA per
// token row.
template <typename T, typename D>
__global__ void __launch_bounds__(kThreads)
residual_norm_vec_kernel(float* __restrict__ residual, const D* __restrict__ delta, int replace,
                         const float* __restrict__ vec, RowSum<T> sum, const float* __restrict__ w, float w_offset,
                         T* __restrict__ out, int64_t out_stride, int width, float eps) {
  __shared__ float s_part[kThreads / 32];
  const int nvec = width / 8;
  float* res = residual + (size_t)blockIdx.x * width;
  const D* dl = delta ? delta + (size_t)blockIdx.x * width : nullptr;
  T* o = out + (size_t)blockIdx.x * out_stride;
  pdl_wait();
  pdl_launch();
  float v[kMaxVec][8];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kMaxVec; ++j) {
    const int i = threadIdx.x + j * kThreads;
    if (i < nvec) {
#pragma unroll
      for (int q = 0; q < 8; ++q) v[j][q] = 0.f;
      if (!replace) load8<float>(res + i * 8, v[j]);
      if (dl) {
        float d[8];
        load8<D>(dl + i * 8, d);
#pragma unroll
        for (int q = 0; q < 8; ++q) v[j][q] += d[q];
      }
      if (vec) {
        float d[8];
        load8<float>(vec + i * 8, d);
#pragma unroll
        for (int q = 0; q < 8; ++q) v[j][q] += d[q];
      }
      for (int e = 0; e < sum.count; ++e) {
        const int row = sum.index[(size_t)blockIdx.x * sum.count + e];
        if (row < 0) continue;
        float d[8];
        load8<T>(sum.rows + (size_t)row * width + i * 8, d);
#pragma unroll
        for (int q = 0; q < 8; ++q) v[j][q] += d[q];
      }
      if (dl || vec || sum.count) store8<float>(res + i * 8, v[j]);
#pragma unroll
      for (int q = 0; q < 8; ++q) ss += v[j][q] * v[j][q];
    }
  }
  float inv = 1.f;
  if (w) inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)width + eps);
#pragma unroll
  for (int j = 0; j < kMaxVec; ++j) {
    const int i = threadIdx.x + j * kThreads;
    if (i < nvec) {
      if (w) {
        float f[8];
        load8<float>(w + i * 8, f);
#pragma unroll
        for (int q = 0; q < 8; ++q) v[j][q] = v[j][q] * inv * (w_offset + f[q]);
      }
      store8<T>(o + i * 8, v[j]);
    }
  }
}

// The same for any width and alignment: an element per step, the row re-read for the second pass.
template <typename T, typename D>
__global__ void __launch_bounds__(kThreads)
residual_norm_any_kernel(float* __restrict__ residual, const D* __restrict__ delta, int replace,
                         const float* __restrict__ vec, RowSum<T> sum, const float* __restrict__ w, float w_offset,
                         T* __restrict__ out, int64_t out_stride, int width, float eps) {
  __shared__ float s_part[kThreads / 32];
  float* res = residual + (size_t)blockIdx.x * width;
  const D* dl = delta ? delta + (size_t)blockIdx.x * width : nullptr;
  T* o = out + (size_t)blockIdx.x * out_stride;
  pdl_wait();
  pdl_launch();
  float ss = 0.f;
  for (int i = threadIdx.x; i < width; i += kThreads) {
    float v = replace ? 0.f : res[i];
    if (dl) v += Cvt<D>::one(dl[i]);
    if (vec) v += vec[i];
    for (int e = 0; e < sum.count; ++e) {
      const int row = sum.index[(size_t)blockIdx.x * sum.count + e];
      if (row >= 0) v += Cvt<T>::one(sum.rows[(size_t)row * width + i]);
    }
    if (dl || vec || sum.count) res[i] = v;
    ss += v * v;
  }
  float inv = 1.f;
  if (w) inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)width + eps);
  for (int i = threadIdx.x; i < width; i += kThreads)      // a thread reads back its own writes
    o[i] = Cvt<T>::from(w ? res[i] * inv * (w_offset + w[i]) : res[i]);
}

// x = scale * table[token], or its norm where there is a weight; residual = x in 32 bits, and optionally
// a copy in T into a column slice of a wider matrix.  Ids outside the table give a zero row.
template <typename T>
__global__ void __launch_bounds__(kThreads)
embed_norm_kernel(const long long* __restrict__ tokens, const T* __restrict__ table, long long vocab,
                  float scale, const float* __restrict__ w, float w_offset, float* __restrict__ residual,
                  T* __restrict__ copy, int64_t copy_stride, int width, float eps) {
  __shared__ float s_part[kThreads / 32];
  pdl_wait();
  pdl_launch();
  const long long tok = tokens[blockIdx.x];
  const bool ok = tok >= 0 && tok < vocab;
  const T* src = table + (size_t)(ok ? tok : 0) * width;
  float inv = 1.f;
  if (w) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < width; i += kThreads) {
      const float v = Cvt<T>::one(src[i]) * scale;
      ss += v * v;
    }
    inv = 1.f / sqrtf(block_sum(ss, s_part) / (float)width + eps);
  }
  for (int i = threadIdx.x; i < width; i += kThreads) {
    float v = ok ? Cvt<T>::one(src[i]) * scale : 0.f;
    if (w) v = v * inv * (w_offset + w[i]);
    residual[(size_t)blockIdx.x * width + i] = v;
    if (copy) copy[(size_t)blockIdx.x * copy_stride + i] = Cvt<T>::from(v);
  }
}

__device__ __forceinline__ float silu(float z, bool exact) { return z / (1.f + (exact ? expf(-z) : __expf(-z))); }
__device__ __forceinline__ float gelu_tanh(float z, bool exact) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  // tanh(u) = 1 - 2 / (1 + e^(2u)), so 0.5 (1 + tanh u) = 1 - 1 / (1 + e^(2u))
  return exact ? 0.5f * z * (1.f + tanhf(u)) : z * (1.f - 1.f / (1.f + __expf(2.f * u)));
}
__device__ __forceinline__ float relu2(float z) { return z > 0.f ? z * z : 0.f; }
template <int ACT> __device__ __forceinline__ float act_fn(float z, bool exact) {
  return ACT == DZ_ACT_SILU ? silu(z, exact) : ACT == DZ_ACT_RELU2 ? relu2(z) : gelu_tanh(z, exact);
}

// out[m, i] = act(x[m, i]), times x[m, inter + i] where GATED; computed in float and rounded once
template <typename T, int ACT, int VEC, bool GATED>
__global__ void __launch_bounds__(kThreads)
act_kernel(const T* __restrict__ x, int64_t x_stride, T* __restrict__ out, int inter) {
  constexpr bool kExact = sizeof(T) == 4;
  const T* g = x + (size_t)blockIdx.x * x_stride;
  const T* u = g + inter;
  T* o = out + (size_t)blockIdx.x * inter;
  pdl_wait();
  pdl_launch();
  for (int i = (blockIdx.y * kThreads + threadIdx.x) * VEC; i < inter; i += gridDim.y * kThreads * VEC) {
    if constexpr (VEC == 8) {
      float a[8], b[8];
      load8<T>(g + i, a);
      if constexpr (GATED) load8<T>(u + i, b);
#pragma unroll
      for (int q = 0; q < 8; ++q) a[q] = act_fn<ACT>(a[q], kExact) * (GATED ? b[q] : 1.f);
      store8<T>(o + i, a);
    } else {
      o[i] = Cvt<T>::from(act_fn<ACT>(Cvt<T>::one(g[i]), kExact) * (GATED ? Cvt<T>::one(u[i]) : 1.f));
    }
  }
}

template <typename T, typename D>
cudaError_t run_residual_norm(float* residual, const void* delta, int replace, const float* vec, RowSum<void> sum,
                              const float* w, float w_offset, void* out, int64_t out_stride, int M, int width,
                              float eps, cudaStream_t st) {
  const bool vecs = width % 8 == 0 && width <= 8 * kMaxVec * kThreads && out_stride % 8 == 0 && aligned16(out) &&
                    aligned16(residual) && aligned16(delta) && aligned16(vec) && aligned16(w) && aligned16(sum.rows);
  return launch_pdl(vecs ? residual_norm_vec_kernel<T, D> : residual_norm_any_kernel<T, D>, dim3(M), dim3(kThreads),
                    st, residual, (const D*)delta, replace, vec, RowSum<T>{(const T*)sum.rows, sum.index, sum.count}, w,
                    w_offset, (T*)out, out_stride, width, eps);
}

template <typename T, int ACT, bool GATED>
cudaError_t run_act(const void* x, int64_t x_stride, void* out, int M, int inter, cudaStream_t st) {
  const bool vecs = inter % 8 == 0 && x_stride % 8 == 0 && aligned16(x) && aligned16(out);
  const int per = kThreads * (vecs ? 8 : 1);
  const dim3 grid(M, (inter + per - 1) / per);
  return launch_pdl(vecs ? act_kernel<T, ACT, 8, GATED> : act_kernel<T, ACT, 1, GATED>, grid, dim3(kThreads), st,
                    (const T*)x, x_stride, (T*)out, inter);
}

}  // namespace
}  // namespace dz

using namespace dz;

extern "C" {

int dz_embed_norm(const int64_t* tokens, const void* table, int64_t vocab, float scale, const float* weight,
                  float weight_offset, float* residual, void* copy, int64_t copy_stride, int M, int width, float eps,
                  int dtype, void* stream) {
  if (!tokens || !table || !residual || M < 0 || width <= 0 || vocab <= 0) return DZ_ERR_INVALID_ARG;
  if (M == 0) return DZ_OK;
  DZ_DISPATCH(dtype, DZ_CUDA_OK(launch_pdl(embed_norm_kernel<T>, dim3(M), dim3(kThreads), (cudaStream_t)stream,
                                           (const long long*)tokens, (const T*)table, (long long)vocab, scale, weight,
                                           weight_offset, residual, (T*)copy, copy_stride, width, eps)));
  return DZ_OK;
}

int dz_residual_norm(float* residual, const void* delta, int delta_dtype, int replace, const float* vec,
                     const void* sum_rows, const int32_t* sum_index, int sum_count, const float* weight,
                     float weight_offset, void* out, int64_t out_stride, int M, int width, float eps, int dtype,
                     void* stream) {
  if (!residual || !out || M < 0 || width <= 0 || out_stride < width || (replace && !delta)) return DZ_ERR_INVALID_ARG;
  if (delta && delta_dtype != dtype && delta_dtype != DZ_DTYPE_F32) return DZ_ERR_INVALID_ARG;
  if (sum_count < 0 || (sum_count > 0 && (!sum_rows || !sum_index))) return DZ_ERR_INVALID_ARG;
  if (M == 0) return DZ_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const RowSum<void> sum = {sum_rows, sum_index, sum_count};
  if (delta && delta_dtype == DZ_DTYPE_F32) {
    DZ_DISPATCH(dtype, DZ_CUDA_OK((run_residual_norm<T, float>(residual, delta, replace, vec, sum, weight, weight_offset,
                                                               out, out_stride, M, width, eps, st))));
  } else {
    DZ_DISPATCH(dtype, DZ_CUDA_OK((run_residual_norm<T, T>(residual, delta, replace, vec, sum, weight, weight_offset,
                                                           out, out_stride, M, width, eps, st))));
  }
  return DZ_OK;
}

int dz_gated_act(const void* x, int64_t x_stride, void* out, int M, int inter, int act, int dtype, void* stream) {
  if (!x || !out || M < 0 || inter <= 0 || x_stride < 2 * (int64_t)inter) return DZ_ERR_INVALID_ARG;
  if (M == 0) return DZ_OK;
  cudaStream_t st = (cudaStream_t)stream;
  switch (act) {
    case DZ_ACT_SILU: DZ_DISPATCH(dtype, DZ_CUDA_OK((run_act<T, DZ_ACT_SILU, true>(x, x_stride, out, M, inter, st)))); break;
    case DZ_ACT_GELU_TANH:
      DZ_DISPATCH(dtype, DZ_CUDA_OK((run_act<T, DZ_ACT_GELU_TANH, true>(x, x_stride, out, M, inter, st))));
      break;
    case DZ_ACT_RELU2: DZ_DISPATCH(dtype, DZ_CUDA_OK((run_act<T, DZ_ACT_RELU2, true>(x, x_stride, out, M, inter, st)))); break;
    default: return DZ_ERR_INVALID_ARG;
  }
  return DZ_OK;
}

int dz_act(const void* x, int64_t x_stride, void* out, int M, int inter, int act, int dtype, void* stream) {
  if (!x || !out || M < 0 || inter <= 0 || x_stride < (int64_t)inter) return DZ_ERR_INVALID_ARG;
  if (M == 0) return DZ_OK;
  cudaStream_t st = (cudaStream_t)stream;
  switch (act) {
    case DZ_ACT_SILU: DZ_DISPATCH(dtype, DZ_CUDA_OK((run_act<T, DZ_ACT_SILU, false>(x, x_stride, out, M, inter, st)))); break;
    case DZ_ACT_GELU_TANH:
      DZ_DISPATCH(dtype, DZ_CUDA_OK((run_act<T, DZ_ACT_GELU_TANH, false>(x, x_stride, out, M, inter, st))));
      break;
    case DZ_ACT_RELU2: DZ_DISPATCH(dtype, DZ_CUDA_OK((run_act<T, DZ_ACT_RELU2, false>(x, x_stride, out, M, inter, st)))); break;
    default: return DZ_ERR_INVALID_ARG;
  }
  return DZ_OK;
}

}  // extern "C"
