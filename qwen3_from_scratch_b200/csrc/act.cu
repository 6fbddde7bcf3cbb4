// SwiGLU gate on the merged gate/up projection:
//   out[t, i] = up[t, i] * gate[t, i] * sigmoid(gate[t, i])      (or another gate of gated_f)
// with gate = columns [0, I) and up = columns [I, 2I) of the [T, 2I] input.
// (or, with `interleave8`, gate and up alternating in blocks of eight columns, the layout the
// fused skinny product wants of its weight).  An optional bias (float32, in the order of the columns) is added first.  The
// gate is evaluated in float32 and the product rounded once.
// Reference: models/feedback.py:28-34 (up * silu(gate)), kernels/triton/feedback.py:145-158.
#include "common.cuh"

namespace q3 {

template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int I, size_t total,
                              int interleave8, int act, const float* __restrict__ bias, float limit) {
  pdl_wait();
  pdl_launch_dependents();
  const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const size_t t = idx / I;
  const int i = (int)(idx - t * I);
  const T* row = gate_up + t * 2 * (size_t)I;
  const int gate_col = interleave8 ? ((i >> 3) << 4) + (i & 7) : i;
  const int up_col = interleave8 ? gate_col + 8 : I + i;
  const float g = to_float(row[gate_col]) + (bias ? bias[gate_col] : 0.f);
  const float u = to_float(row[up_col]) + (bias ? bias[up_col] : 0.f);
  out[idx] = from_float<T>(gated_f(g, u, act, limit));
}

// Eight outputs per thread with 16-byte accesses (bfloat16, I a multiple of 8).
__global__ void swiglu_bf16x8_kernel(const __nv_bfloat16* __restrict__ gate_up, __nv_bfloat16* __restrict__ out,
                                     int I, size_t total8, int interleave8, int act, const float* __restrict__ bias,
                                     float limit) {
  pdl_wait();
  pdl_launch_dependents();
  const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total8) return;
  const int per_row = I >> 3;
  const size_t t = idx / per_row;
  const int j = (int)(idx - t * per_row);  // block of eight outputs
  const __nv_bfloat16* row = gate_up + t * 2 * (size_t)I;
  const int gate_col = interleave8 ? 16 * j : 8 * j, up_col = interleave8 ? 16 * j + 8 : I + 8 * j;
  const uint4 gv = *reinterpret_cast<const uint4*>(row + gate_col);
  const uint4 uv = *reinterpret_cast<const uint4*>(row + up_col);
  const uint32_t gw[4] = {gv.x, gv.y, gv.z, gv.w}, uw[4] = {uv.x, uv.y, uv.z, uv.w};
  uint32_t ow[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    float g0 = __uint_as_float(gw[k] << 16), g1 = __uint_as_float(gw[k] & 0xffff0000u);
    float u0 = __uint_as_float(uw[k] << 16), u1 = __uint_as_float(uw[k] & 0xffff0000u);
    if (bias) {
      const float2 bg = *reinterpret_cast<const float2*>(bias + gate_col + 2 * k);
      const float2 bu = *reinterpret_cast<const float2*>(bias + up_col + 2 * k);
      g0 += bg.x, g1 += bg.y, u0 += bu.x, u1 += bu.y;
    }
    __nv_bfloat162 o = __floats2bfloat162_rn(gated_f(g0, u0, act, limit), gated_f(g1, u1, act, limit));
    ow[k] = *reinterpret_cast<uint32_t*>(&o);
  }
  *reinterpret_cast<uint4*>(out + t * (size_t)I + 8 * j) = make_uint4(ow[0], ow[1], ow[2], ow[3]);
}

}  // namespace q3

// gate_up: [T, 2I]; out: [T, I]; both in `dtype`.  interleave8: columns 16j..16j+7 gate, 16j+8..16j+15 up.
// act: Q3_ACT_SILU, Q3_ACT_RELU, Q3_ACT_GELU_TANH or Q3_ACT_RELU_SQ, applied to the gate, or Q3_ACT_LIMITED with its limit.
// bias: float32 [2I] in the order of the columns, or null.
extern "C" int q3_gated_act(const void* gate_up, void* out, int dtype, int T, int I, int interleave8, int act,
                            const float* bias, float limit, cudaStream_t stream) {
  if (act < Q3_ACT_SILU || act == Q3_ACT_NONE || act > Q3_ACT_LIMITED) return Q3_ERR_SIZE;
  if (T <= 0 || I <= 0) return 0;
  if (interleave8 && I % 8) return Q3_ERR_SIZE;
  const size_t total = (size_t)T * I;
  const int threads = 256;
  const size_t blocks = (total + threads - 1) / threads;
  if (blocks > 0x7fffffffull) return Q3_ERR_SIZE;
  if (dtype == Q3_BF16 && I % 8 == 0 && (uintptr_t)gate_up % 16 == 0 && (uintptr_t)out % 16 == 0 &&
      (uintptr_t)bias % 8 == 0) {
    const size_t total8 = total / 8;
    q3::launch(q3::swiglu_bf16x8_kernel, dim3((unsigned)((total8 + threads - 1) / threads)), dim3(threads), 0, stream, 
        (const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, I, total8, interleave8, act, bias, limit);
    return q3::launch_status();
  }
  if (dtype == Q3_F32)
    q3::launch(q3::swiglu_kernel<float>, dim3((unsigned)blocks), dim3(threads), 0, stream, (const float*)gate_up, (float*)out, I, total, interleave8, act, bias, limit);
  else if (dtype == Q3_BF16)
    q3::launch(q3::swiglu_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(threads), 0, stream, 
        (const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, I, total, interleave8, act, bias, limit);
  else
    return Q3_ERR_DTYPE;
  return q3::launch_status();
}

extern "C" int q3_swiglu(const void* gate_up, void* out, int dtype, int T, int I, int interleave8,
                         cudaStream_t stream) {
  return q3_gated_act(gate_up, out, dtype, T, I, interleave8, Q3_ACT_SILU, nullptr, 0.f, stream);
}

namespace q3 {

// out = act(x), element by element, evaluated in float32 (the feed-forward without a gate).
template <typename T>
__global__ void act_kernel(const T* __restrict__ x, T* __restrict__ out, size_t total, int act) {
  pdl_wait();
  pdl_launch_dependents();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < total) out[i] = from_float<T>(activate(to_float(x[i]), act));
}

// Eight values per thread with 16-byte accesses (bfloat16, a multiple of eight values, aligned).
__global__ void act_bf16x8_kernel(const __nv_bfloat16* __restrict__ x, __nv_bfloat16* __restrict__ out, size_t total8,
                                  int act) {
  pdl_wait();
  pdl_launch_dependents();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total8) return;
  const uint4 v = reinterpret_cast<const uint4*>(x)[i];
  const uint32_t in[4] = {v.x, v.y, v.z, v.w};
  uint32_t ow[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float a = __uint_as_float(in[k] << 16), b = __uint_as_float(in[k] & 0xffff0000u);
    __nv_bfloat162 o = __floats2bfloat162_rn(activate(a, act), activate(b, act));
    ow[k] = *reinterpret_cast<uint32_t*>(&o);
  }
  reinterpret_cast<uint4*>(out)[i] = make_uint4(ow[0], ow[1], ow[2], ow[3]);
}

}  // namespace q3

// out = act(x) over `total` values in `dtype`; out may be x.
extern "C" int q3_act(const void* x, void* out, int dtype, long long total, int act, cudaStream_t stream) {
  if (act < Q3_ACT_SILU || (act > Q3_ACT_GELU_TANH && act != Q3_ACT_RELU_SQ)) return Q3_ERR_SIZE;
  if (total <= 0) return 0;
  const int threads = 256;
  if (dtype == Q3_BF16 && total % 8 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)out % 16 == 0) {
    const size_t total8 = (size_t)total / 8;
    q3::launch(q3::act_bf16x8_kernel, dim3((unsigned)((total8 + threads - 1) / threads)), dim3(threads), 0, stream,
               (const __nv_bfloat16*)x, (__nv_bfloat16*)out, total8, act);
    return q3::launch_status();
  }
  const long long blocks = (total + threads - 1) / threads;
  if (blocks > 0x7fffffffll) return Q3_ERR_SIZE;
  if (dtype == Q3_F32)
    q3::launch(q3::act_kernel<float>, dim3((unsigned)blocks), dim3(threads), 0, stream, (const float*)x, (float*)out,
               (size_t)total, act);
  else if (dtype == Q3_BF16)
    q3::launch(q3::act_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(threads), 0, stream, (const __nv_bfloat16*)x,
               (__nv_bfloat16*)out, (size_t)total, act);
  else
    return Q3_ERR_DTYPE;
  return q3::launch_status();
}
