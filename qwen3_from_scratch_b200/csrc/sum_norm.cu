// What a block whose sub-layers run side by side does to the float32 residual stream between two layers: everything the
// layer before left open goes into the stream, and the rows are normed once for both sub-layers.
//
//   stream += sum_i term_i,   term_i = delta_i, or delta_i / sqrt(mean(delta_i^2) + term_eps) * weight_i * scale_i
//   r = 1 / sqrt(mean(stream^2) + eps);   out_1 = stream * r * w_1;   out_2 = stream * r * w_2
//
// Up to three terms; the second norm's output is optional.  With `rows` the same for chosen rows only, the stream left as
// it is (the model's last norm).  All arithmetic float32, sums in an order that depends on the width alone.
#include "common.cuh"

namespace q3 {

constexpr int SN_TERMS = 3;

template <typename T>
struct SumTerms {
  const T* delta[SN_TERMS];
  const float* weight[SN_TERMS];  // null: the term is the delta as it is
  float scale[SN_TERMS];
  int count;
  float eps;
};

template <typename T, int V>
struct alignas(sizeof(T) * V) SnPack { T v[V]; };

// One block per row; V values per access (4 where width and pointers allow it, else 1).
template <typename T, int V>
__global__ void sum_norm_kernel(float* __restrict__ stream, SumTerms<T> terms, const float* __restrict__ w1,
                                T* __restrict__ out1, const float* __restrict__ w2, T* __restrict__ out2,
                                const int* __restrict__ rows, int W, float eps) {
  extern __shared__ float row_buf[];
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int t = rows ? rows[blockIdx.x] : blockIdx.x;
  float factor[SN_TERMS];
#pragma unroll
  for (int k = 0; k < SN_TERMS; ++k) {
    factor[k] = 1.f;
    if (k < terms.count && terms.weight[k]) {
      float ss = 0.f;
      for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
        const SnPack<T, V> d = *reinterpret_cast<const SnPack<T, V>*>(terms.delta[k] + (size_t)t * W + i);
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(to_float(d.v[e]), to_float(d.v[e]), ss);
      }
      factor[k] = terms.scale[k] / sqrtf(block_sum(ss, red) / (float)W + terms.eps);
    }
  }
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    SnPack<float, V> x = *reinterpret_cast<const SnPack<float, V>*>(stream + (size_t)t * W + i);
#pragma unroll
    for (int k = 0; k < SN_TERMS; ++k) {
      if (k >= terms.count) continue;
      const SnPack<T, V> d = *reinterpret_cast<const SnPack<T, V>*>(terms.delta[k] + (size_t)t * W + i);
      if (terms.weight[k]) {
        const SnPack<float, V> wt = *reinterpret_cast<const SnPack<float, V>*>(terms.weight[k] + i);
#pragma unroll
        for (int e = 0; e < V; ++e) x.v[e] = fmaf(to_float(d.v[e]) * factor[k], wt.v[e], x.v[e]);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) x.v[e] += to_float(d.v[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      row_buf[i + e] = x.v[e];
      ss = fmaf(x.v[e], x.v[e], ss);
    }
    if (!rows && terms.count) *reinterpret_cast<SnPack<float, V>*>(stream + (size_t)t * W + i) = x;
  }
  const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)W + eps);
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    const SnPack<float, V> a = *reinterpret_cast<const SnPack<float, V>*>(w1 + i);
    SnPack<T, V> y;
#pragma unroll
    for (int e = 0; e < V; ++e) y.v[e] = from_float<T>(row_buf[i + e] * r * a.v[e]);
    *reinterpret_cast<SnPack<T, V>*>(out1 + (size_t)blockIdx.x * W + i) = y;
    if (w2) {
      const SnPack<float, V> b = *reinterpret_cast<const SnPack<float, V>*>(w2 + i);
#pragma unroll
      for (int e = 0; e < V; ++e) y.v[e] = from_float<T>(row_buf[i + e] * r * b.v[e]);
      *reinterpret_cast<SnPack<T, V>*>(out2 + (size_t)blockIdx.x * W + i) = y;
    }
  }
}

template <typename T>
static int sum_norm_launch(float* stream, const void* const* delta, const float* const* weight, const float* scale, int count,
                           float term_eps, const float* w1, void* out1, const float* w2, void* out2, const int* rows, int n,
                           int W, float eps, cudaStream_t cuda_stream) {
  SumTerms<T> terms{};
  terms.count = count;
  terms.eps = term_eps;
  bool wide = W % 4 == 0 && (uintptr_t)stream % 16 == 0 && (uintptr_t)w1 % 16 == 0 && (uintptr_t)w2 % 16 == 0 &&
              (uintptr_t)out1 % 16 == 0 && (uintptr_t)out2 % 16 == 0;
  for (int k = 0; k < count; ++k) {
    terms.delta[k] = (const T*)delta[k];
    terms.weight[k] = weight[k];
    terms.scale[k] = scale[k];
    wide = wide && (uintptr_t)delta[k] % 16 == 0 && (uintptr_t)weight[k] % 16 == 0;
  }
  const size_t smem = (size_t)W * sizeof(float);
  int threads = ((W + 3) / 4 + 31) / 32 * 32;
  threads = threads < 64 ? 64 : (threads > 512 ? 512 : threads);
  if (wide)
    launch(sum_norm_kernel<T, 4>, dim3(n), dim3(threads), smem, cuda_stream, stream, terms, w1, (T*)out1, w2, (T*)out2, rows,
           W, eps);
  else
    launch(sum_norm_kernel<T, 1>, dim3(n), dim3(threads), smem, cuda_stream, stream, terms, w1, (T*)out1, w2, (T*)out2, rows,
           W, eps);
  if (!rows) note_stream_written();
  return launch_status();
}

}  // namespace q3

// stream: float32 [T, W]; delta0..2: [T, W] in `dtype` or null (the first `count` are used); weight0..2: float32 [W] or null
// (the term as it is); w1, out1 and w2, out2 (or both null): the norms' weights (float32 [W]) and outputs [n, W] in `dtype`;
// rows: int32 [R] or null.
extern "C" int q3_sum_norm(float* stream, const void* delta0, const float* weight0, float scale0, const void* delta1,
                           const float* weight1, float scale1, const void* delta2, const float* weight2, float scale2,
                           int count, float term_eps, const float* w1, void* out1, const float* w2, void* out2,
                           const int* rows, int R, int dtype, int T, int W, float eps, cudaStream_t cuda_stream) {
  const int n = rows ? R : T;
  if (n <= 0) return 0;
  if (W <= 0 || W > 12000 || count < 0 || count > q3::SN_TERMS || !w1 || !out1 || (w2 && !out2)) return Q3_ERR_SIZE;
  const void* delta[3] = {delta0, delta1, delta2};
  const float* weight[3] = {weight0, weight1, weight2};
  const float scale[3] = {scale0, scale1, scale2};
  if (dtype == Q3_F32)
    return q3::sum_norm_launch<float>(stream, delta, weight, scale, count, term_eps, w1, out1, w2, out2, rows, n, W, eps,
                                      cuda_stream);
  if (dtype == Q3_BF16)
    return q3::sum_norm_launch<__nv_bfloat16>(stream, delta, weight, scale, count, term_eps, w1, out1, w2, out2, rows, n, W,
                                              eps, cuda_stream);
  return Q3_ERR_DTYPE;
}
