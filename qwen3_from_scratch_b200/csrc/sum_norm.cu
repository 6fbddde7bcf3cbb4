// What a block does to the float32 residual stream between two sub-layers: everything that was left open goes into the
// stream, and the rows are normed, copied or mixed with the rows before them for what comes next.
//
//   stream += sum_i term_i,   term_i = d_i, or d_i / sqrt(mean(d_i^2) + term_eps) * weight_i * scale_i,   d_i = delta_i (+ bias_i)
//   sum_norm  r = 1 / sqrt(mean(stream^2) + eps);   out_1 = stream * r * w_1;   out_2 = stream * r * w_2
//             (without w_1: out_1 = the new rows as they are, or nothing)
//   sum_mix   out_m[t] = x_t + (x_{t-1} - x_t) * mu_m for several mu_m, x the stream; what lies before a portion's first
//             token comes from a state slot, which then receives the portion's last row.  Terms only in a step of single
//             tokens (a longer portion's rows are read by the blocks of their neighbours).
//
// Up to three terms; the second norm's output is optional.  With `rows` the same for chosen rows only, the stream left as
// it is (the model's last norm).  All arithmetic float32, sums in an order that depends on the width alone.
#include "common.cuh"

namespace q3 {

constexpr int SN_TERMS = 3;

template <typename T>
struct SumTerms {
  const T* delta[SN_TERMS];
  const float* bias[SN_TERMS];    // null: none
  const float* weight[SN_TERMS];  // null: the term is the delta as it is
  float scale[SN_TERMS];
  int count;
  float eps;
};

template <typename T, int V>
struct alignas(sizeof(T) * V) SnPack { T v[V]; };

// V values of term k from column i on.
template <typename T, int V>
__device__ __forceinline__ SnPack<float, V> sum_term(const SumTerms<T>& terms, int k, size_t row, int i) {
  const SnPack<T, V> d = *reinterpret_cast<const SnPack<T, V>*>(terms.delta[k] + row + i);
  SnPack<float, V> x;
#pragma unroll
  for (int e = 0; e < V; ++e) x.v[e] = to_float(d.v[e]);
  if (terms.bias[k]) {
    const SnPack<float, V> b = *reinterpret_cast<const SnPack<float, V>*>(terms.bias[k] + i);
#pragma unroll
    for (int e = 0; e < V; ++e) x.v[e] += b.v[e];
  }
  return x;
}

// What the terms of row t are multiplied by, by the whole block.  N: how many terms there may be.
template <typename T, int V, int N>
__device__ __forceinline__ void sum_factors(const SumTerms<T>& terms, int t, int W, float* red, float (&factor)[N]) {
#pragma unroll
  for (int k = 0; k < N; ++k) {
    factor[k] = 1.f;
    if (k < terms.count && terms.weight[k]) {
      float ss = 0.f;
      for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
        const SnPack<float, V> d = sum_term<T, V>(terms, k, (size_t)t * W, i);
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(d.v[e], d.v[e], ss);
      }
      factor[k] = terms.scale[k] / sqrtf(block_sum(ss, red) / (float)W + terms.eps);
    }
  }
}

// A thread's first V values of row t of the stream, asked for before the terms' statistics are worked out.
template <int V>
__device__ __forceinline__ SnPack<float, V> sum_first(const float* __restrict__ stream, int t, int W) {
  SnPack<float, V> x{};
  if ((int)threadIdx.x * V < W) x = *reinterpret_cast<const SnPack<float, V>*>(stream + (size_t)t * W + threadIdx.x * V);
  return x;
}

// V values of the new row t from column i on; `first`: what sum_first returned.
template <typename T, int V, int N>
__device__ __forceinline__ SnPack<float, V> sum_values(const float* __restrict__ stream, const SumTerms<T>& terms,
                                                       const float (&factor)[N], const SnPack<float, V>& first, int t,
                                                       int W, int i) {
  SnPack<float, V> x = first;
  if (i != (int)threadIdx.x * V) x = *reinterpret_cast<const SnPack<float, V>*>(stream + (size_t)t * W + i);
#pragma unroll
  for (int k = 0; k < N; ++k) {
    if (k >= terms.count) continue;
    const SnPack<float, V> d = sum_term<T, V>(terms, k, (size_t)t * W, i);
    if (terms.weight[k]) {
      const SnPack<float, V> wt = *reinterpret_cast<const SnPack<float, V>*>(terms.weight[k] + i);
#pragma unroll
      for (int e = 0; e < V; ++e) x.v[e] = fmaf(d.v[e] * factor[k], wt.v[e], x.v[e]);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) x.v[e] += d.v[e];
    }
  }
  return x;
}

// One block per row; V values per access (4 where width and pointers allow it, else 1).
template <typename T, int V, int N>
__global__ void sum_norm_kernel(float* __restrict__ stream, SumTerms<T> terms, const float* __restrict__ w1,
                                T* __restrict__ out1, const float* __restrict__ w2, T* __restrict__ out2,
                                const int* __restrict__ rows, int W, float eps) {
  extern __shared__ float row_buf[];
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int t = rows ? rows[blockIdx.x] : blockIdx.x;
  const SnPack<float, V> row = sum_first<V>(stream, t, W);
  float factor[N];
  sum_factors<T, V, N>(terms, t, W, red, factor);
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    const SnPack<float, V> x = sum_values<T, V, N>(stream, terms, factor, row, t, W, i);
    if (!rows && terms.count) *reinterpret_cast<SnPack<float, V>*>(stream + (size_t)t * W + i) = x;
    if (!w1) {
      if (out1) {
        SnPack<T, V> y;
#pragma unroll
        for (int e = 0; e < V; ++e) y.v[e] = from_float<T>(x.v[e]);
        *reinterpret_cast<SnPack<T, V>*>(out1 + (size_t)blockIdx.x * W + i) = y;
      }
      continue;
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      row_buf[i + e] = x.v[e];
      ss = fmaf(x.v[e], x.v[e], ss);
    }
  }
  if (!w1) return;
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

// One block per token, as above.  mu: [M, W]; out: [M, T, W]; state: [num_slots, W].
template <typename T, int V>  // at most one term
__global__ void sum_mix_kernel(float* __restrict__ stream, SumTerms<T> terms, const float* __restrict__ mu, int M,
                               float* __restrict__ state, const int* __restrict__ q_start, const int* __restrict__ tok_seq,
                               const int* __restrict__ slot_ids, int num_slots, T* __restrict__ out, int W, int* status) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, b = tok_seq[t], slot = slot_ids[b];
  const bool live = slot >= 0 && slot < num_slots;
  if (!live && threadIdx.x == 0) atomicOr(status, Q3_STATUS_BAD_POSITION);
  const bool first = t == q_start[b];
  const int last = q_start[b + 1] - 1;
  float* st = live ? state + (size_t)slot * W : nullptr;
  const SnPack<float, V> row = sum_first<V>(stream, t, W);
  float factor[1];
  sum_factors<T, V, 1>(terms, t, W, red, factor);
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    const SnPack<float, V> x = sum_values<T, V, 1>(stream, terms, factor, row, t, W, i);
    if (terms.count) *reinterpret_cast<SnPack<float, V>*>(stream + (size_t)t * W + i) = x;
    SnPack<float, V> p{};
    if (live) {
      p = *reinterpret_cast<const SnPack<float, V>*>((first ? st : stream + (size_t)(t - 1) * W) + i);
      // the element's old state has been read by this thread and by nobody else: it may be renewed now
      if (first)
        *reinterpret_cast<SnPack<float, V>*>(st + i) =
            last == t ? x : *reinterpret_cast<const SnPack<float, V>*>(stream + (size_t)last * W + i);
    }
    for (int m = 0; m < M; ++m) {
      const SnPack<float, V> u = *reinterpret_cast<const SnPack<float, V>*>(mu + (size_t)m * W + i);
      SnPack<T, V> y;
#pragma unroll
      for (int e = 0; e < V; ++e) y.v[e] = from_float<T>(live ? fmaf(p.v[e] - x.v[e], u.v[e], x.v[e]) : 0.f);
      *reinterpret_cast<SnPack<T, V>*>(out + ((size_t)m * gridDim.x + t) * W + i) = y;
    }
  }
}

static int sum_norm_threads(int W) {
  const int threads = ((W + 3) / 4 + 31) / 32 * 32;
  return threads < 64 ? 64 : (threads > 512 ? 512 : threads);
}

template <typename T>
static bool sum_terms_of(SumTerms<T>& terms, const void* const* delta, const float* const* bias, const float* const* weight,
                         const float* scale, int count, float term_eps) {
  bool wide = true;
  terms.count = count;
  terms.eps = term_eps;
  for (int k = 0; k < count; ++k) {
    terms.delta[k] = (const T*)delta[k];
    terms.bias[k] = bias[k];
    terms.weight[k] = weight[k];
    terms.scale[k] = scale[k];
    wide = wide && (uintptr_t)delta[k] % 16 == 0 && (uintptr_t)weight[k] % 16 == 0 && (uintptr_t)bias[k] % 16 == 0;
  }
  return wide;
}

template <typename T>
static int sum_norm_launch(float* stream, const void* const* delta, const float* const* bias, const float* const* weight,
                           const float* scale, int count, float term_eps, const float* w1, void* out1, const float* w2, void* out2, const int* rows, int n,
                           int W, float eps, cudaStream_t cuda_stream) {
  SumTerms<T> terms{};
  bool wide = sum_terms_of(terms, delta, bias, weight, scale, count, term_eps) && W % 4 == 0 && (uintptr_t)stream % 16 == 0 && (uintptr_t)w1 % 16 == 0 && (uintptr_t)w2 % 16 == 0 &&
              (uintptr_t)out1 % 16 == 0 && (uintptr_t)out2 % 16 == 0;
  const size_t smem = w1 ? (size_t)W * sizeof(float) : 0;
  const int threads = sum_norm_threads(W);
  auto go = [&](auto kernel) {
    launch(kernel, dim3(n), dim3(threads), smem, cuda_stream, stream, terms, w1, (T*)out1, w2, (T*)out2, rows, W, eps);
  };
  if (wide && count <= 1) go(sum_norm_kernel<T, 4, 1>);
  else if (wide) go(sum_norm_kernel<T, 4, SN_TERMS>);
  else go(sum_norm_kernel<T, 1, SN_TERMS>);
  if (!rows) note_stream_written();
  return launch_status();
}

template <typename T>
static int sum_mix_launch(float* stream, const void* delta, const float* bias, const float* weight, float scale, float term_eps,
                          const float* mu, int M, float* state, const int* q_start, const int* tok_seq, const int* slot_ids,
                          int num_slots, void* out, int n, int W, int* status, cudaStream_t cuda_stream) {
  SumTerms<T> terms{};
  const bool wide = sum_terms_of(terms, &delta, &bias, &weight, &scale, delta ? 1 : 0, term_eps) && W % 4 == 0 &&
                    (uintptr_t)stream % 16 == 0 && (uintptr_t)mu % 16 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)out % 16 == 0;
  auto go = [&](auto kernel) {
    launch(kernel, dim3(n), dim3(sum_norm_threads(W)), 0, cuda_stream, stream, terms, mu, M, state, q_start, tok_seq, slot_ids,
           num_slots, (T*)out, W, status);
  };
  if (wide) go(sum_mix_kernel<T, 4>);
  else go(sum_mix_kernel<T, 1>);
  if (delta) note_stream_written();
  return launch_status();
}

}  // namespace q3

// stream: float32 [T, W]; delta0..2: [T, W] in `dtype` or null (the first `count` are used); bias0..2: float32 [W] or null;
// weight0..2: float32 [W] or null (the term as it is); w1, out1 and w2, out2 (or both null): the norms' weights (float32 [W])
// and outputs [n, W] in `dtype`; without w1, out1 (or null) receives the new rows as they are; rows: int32 [R] or null.
extern "C" int q3_sum_norm(float* stream, const void* delta0, const float* bias0, const float* weight0, float scale0,
                           const void* delta1, const float* bias1, const float* weight1, float scale1, const void* delta2,
                           const float* bias2, const float* weight2, float scale2, int count,
                           float term_eps, const float* w1, void* out1, const float* w2, void* out2, const int* rows, int R,
                           int dtype, int T, int W, float eps, cudaStream_t cuda_stream) {
  const int n = rows ? R : T;
  if (n <= 0) return 0;
  if (W <= 0 || W > 12000 || count < 0 || count > q3::SN_TERMS || (w1 && !out1) || (w2 && (!w1 || !out2)))
    return Q3_ERR_SIZE;
  const void* delta[3] = {delta0, delta1, delta2};
  const float* bias[3] = {bias0, bias1, bias2};
  const float* weight[3] = {weight0, weight1, weight2};
  const float scale[3] = {scale0, scale1, scale2};
  if (dtype == Q3_F32)
    return q3::sum_norm_launch<float>(stream, delta, bias, weight, scale, count, term_eps, w1, out1, w2, out2, rows, n, W,
                                      eps, cuda_stream);
  if (dtype == Q3_BF16)
    return q3::sum_norm_launch<__nv_bfloat16>(stream, delta, bias, weight, scale, count, term_eps, w1, out1, w2, out2, rows,
                                              n, W, eps, cuda_stream);
  return Q3_ERR_DTYPE;
}

// stream: float32 [T, W]; delta: [T, W] in `dtype` or null (a step of single tokens only), with bias, weight, scale as above;
// mu: float32 [M, W]; state: float32 [num_slots, W]; out: [M, T, W] in `dtype`.
extern "C" int q3_sum_mix(float* stream, const void* delta, const float* bias, const float* weight, float scale, float term_eps,
                          const float* mu, int M, float* state, const int* q_start, const int* tok_seq, const int* slot_ids,
                          int num_slots, void* out, int dtype, int T, int B, int W, int* status, cudaStream_t cuda_stream) {
  if (T <= 0) return 0;
  if (W <= 0 || M <= 0 || M > 64 || num_slots <= 0 || (delta && T != B)) return Q3_ERR_SIZE;
  if (dtype == Q3_F32)
    return q3::sum_mix_launch<float>(stream, delta, bias, weight, scale, term_eps, mu, M, state, q_start, tok_seq, slot_ids,
                                     num_slots, out, T, W, status, cuda_stream);
  if (dtype == Q3_BF16)
    return q3::sum_mix_launch<__nv_bfloat16>(stream, delta, bias, weight, scale, term_eps, mu, M, state, q_start, tok_seq,
                                             slot_ids, num_slots, out, T, W, status, cuda_stream);
  return Q3_ERR_DTYPE;
}
