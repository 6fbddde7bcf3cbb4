// A feed-forward of routed experts: every token goes through `top` of E small feed-forwards W_down act(W_up h),
// chosen by a router, and the results are added with the router's weights.
//
//   moe_route      logits z = W_r h in float32, scores s = sigmoid(z), or softmax(z) over all experts; the `top` experts
//                  with the largest s + bias[e] are chosen (ties: the lower index).  With `groups` > 1 the experts form
//                  equal groups of neighbours and only experts of the `keep` groups with the largest best member can be
//                  chosen.  Their weights are s * scale (the bias takes no part in the weights), divided by the sum
//                  of the chosen s (+ 1e-20) with `renorm`.  A bias of the logits themselves (`zbias`) is added before
//                  anything else.  With `share` the router's matrix has one more row w_s, and share[t] =
//                  sigmoid(w_s h): what a shared expert's output is multiplied by.  A block per token or per eight; in
//                  bfloat16, up to MR_MAX_ROWS rows of the router, per sixteen on the tensor cores: the router's float32
//                  numbers as three bfloat16 ones whose sum they are, so that every product is exact and the sums float32.
//   moe_pair_up    for every (token, chosen expert) pair: act(W_up[e] h), a warp per output value; the pair's expert
//                  weight is streamed once per pair.  For a few tokens (decoding) and the float32 run.
//   moe_pair_down  out[t] = base[t] + sum_k weight[t, k] W_down[e_k] a[t, k]: a warp per output value, the chosen
//                  experts in the order the router listed them.
//
// Gated experts (`gate_block` > 0): W_down (act(W_gate h) * (W_up h)); the stack `up` then holds 2 F rows per
// expert, gate and up rows alternating in blocks of `gate_block` rows (gate_block = F: all gate rows, then all up
// rows); the limited form of a gate (gated_f) takes `limit`.  `in_wts` (or null): the router's weight multiplies what the expert reads (both of its first products)
// instead of what it returns; the caller then passes ones as `wts` to the second kernel.
//
// Sums over a row are taken lane by lane in ascending order and then across the warp, so a token's result does not
// depend on the batch.  `base_wts` (or null): base[t] counts times base_wts[t].  The expert weights are stacked: up [E, F, W], down [E, W, F].
#include "attn_mma.cuh"

namespace q3 {

constexpr int MOE_MAX_TOP = 32;

__device__ __forceinline__ void load4(const float* p, float (&x)[4]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  x[0] = v.x, x[1] = v.y, x[2] = v.z, x[3] = v.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&x)[4]) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
  x[0] = a.x, x[1] = a.y, x[2] = b.x, x[3] = b.y;
}

// Order-preserving key of a float: larger floats have larger keys (minus infinity 0x7fffff), NaN the smallest one, 1;
// 0 is kept free for entries that cannot be chosen (any more).
__device__ __forceinline__ unsigned choice_key(float v) {
  if (v != v) return 1u;
  const unsigned u = __float_as_uint(v);
  return u & 0x80000000u ? ~u : u | 0x80000000u;
}

// What a router does with a token's logits, by one warp.  score [E]: the logits (softmax) or the scores (sigmoid); key [E]
// scratch; kept [groups] scratch.  With up to 32 experts everything stays in the lanes.
struct Choice {
  int E, top, softmax, groups, keep, renorm;
  float scale;
};

__device__ __forceinline__ void choose_experts(const Choice& c, float* score, unsigned* key, unsigned* kept,
                                               const float* __restrict__ bias, int* __restrict__ ids, float* __restrict__ wts,
                                               int lane) {
  const int E = c.E, per = E / c.groups;
  float mx = -INFINITY, sum = 0.f;
  if (c.softmax) {  // the sum's order is the lanes' and then the warp's: a token's scores do not depend on the batch
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, score[e]);
    mx = warp_max(mx);
    for (int e = lane; e < E; e += 32) sum += expf(score[e] - mx);
    sum = warp_sum(sum);
  }
  // the score of expert e and what it is chosen by: without a bias the logits themselves (the same order, no underflow)
  auto make = [&](int e, float& s) {
    const float z = score[e];
    s = c.softmax ? expf(z - mx) / sum : z;
    return choice_key(bias ? s + bias[e] : z);
  };
  float total = 0.f, my_score = 0.f;
  int mine = -1;  // lane k keeps the k-th choice (top <= MOE_MAX_TOP = 32)
  if (E <= 32) {
    float s = 0.f;
    unsigned k = lane < E ? make(lane, s) : 0u;
    if (c.groups > 1) {  // the best group is the one of the best expert outside the groups kept so far
      const int n = lane / per;
      unsigned mask = 0;
      for (int i = 0; i < c.keep; ++i) {
        const unsigned v = (mask >> n) & 1u ? 0u : k;
        const unsigned best = __reduce_max_sync(0xffffffffu, v);
        const int at = __ffs(__ballot_sync(0xffffffffu, v == best && v)) - 1;
        mask |= 1u << (at / per);
      }
      if (!((mask >> n) & 1u)) k = 0;
    }
    for (int i = 0; i < c.top; ++i) {
      const unsigned best = __reduce_max_sync(0xffffffffu, k);
      const int at = __ffs(__ballot_sync(0xffffffffu, k == best && k)) - 1;
      const float sc = __shfl_sync(0xffffffffu, s, at);
      total += sc;
      if (lane == i) {
        mine = at;
        my_score = sc;
      }
      if (lane == at) k = 0;
    }
  } else {
    for (int e = lane; e < E; e += 32) {
      float s;
      key[e] = make(e, s);
      score[e] = s;
    }
    auto best_of = [&](bool groups_left) {  // the largest key, the lowest index among equals
      unsigned best = 0, at = 0x7fffffff;
      for (int e = lane; e < E; e += 32)
        if (key[e] > best && !(groups_left && kept[e / per])) {
          best = key[e];
          at = e;
        }
      const unsigned top = __reduce_max_sync(0xffffffffu, best);
      return (int)__reduce_min_sync(0xffffffffu, best == top ? at : 0x7fffffffu);
    };
    if (c.groups > 1) {
      for (int n = lane; n < c.groups; n += 32) kept[n] = 0;
      __syncwarp();
      for (int i = 0; i < c.keep; ++i) {
        const int e = best_of(true);
        __syncwarp();
        if (lane == 0) kept[e / per] = 1;
        __syncwarp();
      }
      for (int e = lane; e < E; e += 32)
        if (!kept[e / per]) key[e] = 0;
    }
    __syncwarp();
    for (int i = 0; i < c.top; ++i) {
      const int e = best_of(false);
      const float sc = score[e];
      total += sc;
      if (lane == i) {
        mine = e;
        my_score = sc;
      }
      __syncwarp();
      if (lane == 0) key[e] = 0;
      __syncwarp();
    }
  }
  if (lane < c.top) {
    ids[lane] = mine;
    wts[lane] = c.renorm ? my_score / (total + 1e-20f) * c.scale : my_score * c.scale;
  }
}

// TOK tokens to a block: a warp's share of an expert's row is loaded once for all of them, and with TOK > 1 the tokens' rows
// wait in shared memory (the form for many tokens, W a multiple of 4).  The order of a dot product's additions is the same.
template <typename T, int TOK>
__global__ void moe_route_kernel(const T* __restrict__ h, const float* __restrict__ wr, const float* __restrict__ bias,
                                 const float* __restrict__ zbias, int* __restrict__ ids, float* __restrict__ wts,
                                 float* __restrict__ share, int Ttot, int W, Choice c) {
  extern __shared__ __align__(16) float score[];  // [TOK][E] scores, [TOK][E] keys, [TOK][groups] flags, TOK > 1: [TOK][W] rows
  unsigned* key = reinterpret_cast<unsigned*>(score + TOK * c.E);
  unsigned* kept = key + TOK * c.E;
  T* rows = reinterpret_cast<T*>(score + ((TOK * (2 * c.E + c.groups) + 3) & ~3));
  pdl_wait();
  pdl_launch_dependents();
  const int t0 = blockIdx.x * TOK;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const T* row = h + (size_t)t0 * W;
  const int rows_of_router = c.E + (share ? 1 : 0);
  auto leave = [&](int k, int e, float dot) {
    if (e == c.E) {  // the shared expert's row
      if (t0 + k < Ttot) share[t0 + k] = sigmoid_f(dot);
      return;
    }
    if (zbias) dot += zbias[e];
    score[k * c.E + e] = c.softmax ? dot : 1.0f / (1.0f + expf(-dot));
  };
  if constexpr (TOK > 1) {
    constexpr int PER = 4;
    const int live = min(TOK, Ttot - t0);
    struct alignas(sizeof(T) * PER) Pack { T v[PER]; };
    for (int i = threadIdx.x * PER; i < TOK * W; i += blockDim.x * PER)
      *reinterpret_cast<Pack*>(rows + i) = *reinterpret_cast<const Pack*>(row + (i < live * W ? i : i % W));
    __syncthreads();
    for (int e = warp; e < rows_of_router; e += nwarps) {
      const float* w = wr + (size_t)e * W;
      float dot[TOK];
#pragma unroll
      for (int k = 0; k < TOK; ++k) dot[k] = 0.f;
#pragma unroll 4
      for (int i = 4 * lane; i < W; i += 128) {
        const float4 wv = *reinterpret_cast<const float4*>(w + i);
#pragma unroll
        for (int k = 0; k < TOK; ++k) {
          float x[4];
          load4(rows + k * W + i, x);
          dot[k] = fmaf(x[0], wv.x, dot[k]);
          dot[k] = fmaf(x[1], wv.y, dot[k]);
          dot[k] = fmaf(x[2], wv.z, dot[k]);
          dot[k] = fmaf(x[3], wv.w, dot[k]);
        }
      }
#pragma unroll
      for (int k = 0; k < TOK; ++k) {
        dot[k] = warp_sum(dot[k]);
        if (lane == 0) leave(k, e, dot[k]);
      }
    }
  } else {
    // four values per lane and turn where the rows allow it, so that a warp has its loads in flight together
    const bool by4 = (W & 3) == 0 && ((uintptr_t)row & (4 * sizeof(T) - 1)) == 0 && ((uintptr_t)wr & 15) == 0;
    for (int e = warp; e < rows_of_router; e += nwarps) {
      const float* w = wr + (size_t)e * W;
      float dot = 0.f;
      if (by4) {
#pragma unroll 8
        for (int i = 4 * lane; i < W; i += 128) {
          const float4 wv = *reinterpret_cast<const float4*>(w + i);
          float x[4];
          load4(row + i, x);
          dot = fmaf(x[0], wv.x, dot);
          dot = fmaf(x[1], wv.y, dot);
          dot = fmaf(x[2], wv.z, dot);
          dot = fmaf(x[3], wv.w, dot);
        }
      } else {
        for (int i = lane; i < W; i += 32) dot = fmaf(to_float(row[i]), w[i], dot);
      }
      dot = warp_sum(dot);
      if (lane == 0) leave(0, e, dot);
    }
  }
  __syncthreads();
  for (int k = warp; k < TOK && t0 + k < Ttot; k += nwarps)
    choose_experts(c, score + k * c.E, key + k * c.E, kept + k * c.groups, bias, ids + (size_t)(t0 + k) * c.top,
                   wts + (size_t)(t0 + k) * c.top, lane);
}

// Sixteen tokens to a block; the warps share the sum over W, in groups of 32 values of which lane t of a row takes
// k = 8 t .. 8 t + 7 (see gemm_skinny.cu), and meet in shared memory in order.  A warp's first MR_BATCH groups of the router are
// asked for before the wait on the kernel before.  W a multiple of 8.
constexpr int MR_TOK = 16, MR_WARPS = 16, MR_MAX_ROWS = 40, MR_BATCH = 2;

template <int NT>  // tiles of eight router rows
__global__ void __launch_bounds__(MR_WARPS * 32)
moe_route_mma_kernel(const __nv_bfloat16* __restrict__ h, const float* __restrict__ wr, const float* __restrict__ bias,
                     const float* __restrict__ zbias, int* __restrict__ ids, float* __restrict__ wts, float* __restrict__ share,
                     int Ttot, int W, Choice c) {
  extern __shared__ __align__(16) float score[];  // [16][E] scores, [16][E] keys, [16][groups] flags; before them the partial sums
  float(*part)[MR_TOK][8 * NT + 1] = reinterpret_cast<float(*)[MR_TOK][8 * NT + 1]>(score + ((MR_TOK * (2 * c.E + c.groups) + 3) & ~3));
  unsigned* key = reinterpret_cast<unsigned*>(score + MR_TOK * c.E);
  unsigned* kept = key + MR_TOK * c.E;
  const int t0 = blockIdx.x * MR_TOK, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tid4 = lane & 3;
  const int rows = c.E + (share ? 1 : 0);
  const int groups32 = (W + 31) / 32, per = (groups32 + MR_WARPS - 1) / MR_WARPS;
  const int g_lo = warp * per, g_hi = min(groups32, g_lo + per);
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  float4 wv[MR_BATCH][NT][2];
  auto fetch = [&](int g0) {
#pragma unroll
    for (int u = 0; u < MR_BATCH; ++u)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int k = (g0 + u) * 32 + 8 * tid4, e = nt * 8 + gid;
        const bool in = g0 + u < g_hi && k < W && e < rows;
        const float4* p = reinterpret_cast<const float4*>(wr + (size_t)e * W + k);
        wv[u][nt][0] = in ? p[0] : make_float4(0.f, 0.f, 0.f, 0.f);
        wv[u][nt][1] = in ? p[1] : make_float4(0.f, 0.f, 0.f, 0.f);
      }
  };
  fetch(g_lo);
  pdl_wait();
  pdl_launch_dependents();
  const __nv_bfloat16* x_lo = h + (size_t)min(t0 + gid, Ttot - 1) * W;
  const __nv_bfloat16* x_hi = h + (size_t)min(t0 + gid + 8, Ttot - 1) * W;
  for (int g0 = g_lo; g0 < g_hi; g0 += MR_BATCH) {
    uint4 lo[MR_BATCH], hi[MR_BATCH];
#pragma unroll
    for (int u = 0; u < MR_BATCH; ++u) {
      const int k = (g0 + u) * 32 + 8 * tid4;
      const bool in = g0 + u < g_hi && k < W;
      lo[u] = in ? *reinterpret_cast<const uint4*>(x_lo + k) : make_uint4(0, 0, 0, 0);
      hi[u] = in ? *reinterpret_cast<const uint4*>(x_hi + k) : make_uint4(0, 0, 0, 0);
    }
    if (g0 > g_lo) fetch(g0);
#pragma unroll
    for (int u = 0; u < MR_BATCH; ++u) {
      const uint32_t a0[4] = {lo[u].x, hi[u].x, lo[u].y, hi[u].y}, a1[4] = {lo[u].z, hi[u].z, lo[u].w, hi[u].w};
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        float w[8] = {wv[u][nt][0].x, wv[u][nt][0].y, wv[u][nt][0].z, wv[u][nt][0].w,
                      wv[u][nt][1].x, wv[u][nt][1].y, wv[u][nt][1].z, wv[u][nt][1].w};
#pragma unroll
        for (int piece = 0; piece < 3; ++piece) {  // the upper eight bits, the middle, the lower
          uint32_t b[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 p = __floats2bfloat162_rn(w[2 * i], w[2 * i + 1]);
            const float2 f = __bfloat1622float2(p);
            b[i] = *reinterpret_cast<const uint32_t*>(&p);
            w[2 * i] -= f.x;
            w[2 * i + 1] -= f.y;
          }
          mma_bf16(acc[nt], a0, b[0], b[1]);
          mma_bf16(acc[nt], a1, b[2], b[3]);
        }
      }
    }
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int j = 0; j < 4; ++j) part[warp][gid + 8 * (j >> 1)][nt * 8 + 2 * tid4 + (j & 1)] = acc[nt][j];
  __syncthreads();
  for (int i = threadIdx.x; i < MR_TOK * rows; i += MR_WARPS * 32) {
    const int k = i / rows, e = i - k * rows;
    float dot = 0.f;
#pragma unroll
    for (int w = 0; w < MR_WARPS; ++w) dot += part[w][k][e];
    if (e == c.E) {
      if (t0 + k < Ttot) share[t0 + k] = sigmoid_f(dot);
      continue;
    }
    if (zbias) dot += zbias[e];
    score[k * c.E + e] = c.softmax ? dot : sigmoid_f(dot);
  }
  __syncthreads();
  for (int k = warp; k < MR_TOK && t0 + k < Ttot; k += MR_WARPS)
    choose_experts(c, score + k * c.E, key + k * c.E, kept + k * c.groups, bias, ids + (size_t)(t0 + k) * c.top,
                   wts + (size_t)(t0 + k) * c.top, lane);
}

// grid (pairs, ceil(F / warps)).  a[pair, f] = act(sum_i up[e, f, i] h[t, i]), t = pair / top.
template <typename T>
__global__ void moe_pair_up_kernel(const T* __restrict__ h, const T* __restrict__ up, const int* __restrict__ ids,
                                   T* __restrict__ a, int W, int F, int E, int top, int act, int gate_block,
                                   const float* __restrict__ in_wts, float limit) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const int f = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int pair = blockIdx.x;
  if (f >= F) return;
  const int e = ids[pair];
  if (e < 0 || e >= E) {
    if (lane == 0) a[(size_t)pair * F + f] = from_float<T>(0.f);
    return;
  }
  const T* row = h + (size_t)(pair / top) * W;
  const float in_scale = in_wts ? in_wts[pair] : 1.f;
  if (gate_block > 0) {
    const size_t gate_row = (size_t)(f / gate_block) * 2 * gate_block + f % gate_block;
    const T* wg = up + ((size_t)e * 2 * F + gate_row) * W;
    const T* wu = wg + (size_t)gate_block * W;
    float dg = 0.f, du = 0.f;
    for (int i = lane; i < W; i += 32) {
      const float x = to_float(row[i]);
      dg = fmaf(x, to_float(wg[i]), dg);
      du = fmaf(x, to_float(wu[i]), du);
    }
    dg = warp_sum(dg) * in_scale;
    du = warp_sum(du) * in_scale;
    if (lane == 0) a[(size_t)pair * F + f] = from_float<T>(gated_f(dg, du, act, limit));
    return;
  }
  const T* w = up + ((size_t)e * F + f) * W;
  float dot = 0.f;
  for (int i = lane; i < W; i += 32) dot = fmaf(to_float(row[i]), to_float(w[i]), dot);
  dot = warp_sum(dot) * in_scale;
  if (lane == 0) a[(size_t)pair * F + f] = from_float<T>(activate(dot, act));
}

// grid (T, ceil(W / warps)).  out[t, c] = base[t, c] + sum_k wts[t, k] sum_f down[e_k, c, f] a[t * top + k, f].
template <typename T>
__global__ void moe_pair_down_kernel(const T* __restrict__ a, const T* __restrict__ down, const int* __restrict__ ids,
                                     const float* __restrict__ wts, const T* __restrict__ base,
                                     const float* __restrict__ base_wts, T* __restrict__ out, int W, int F, int E, int top) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const int c = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int t = blockIdx.x;
  if (c >= W) return;
  float acc = base ? to_float(base[(size_t)t * W + c]) : 0.f;
  if (base_wts) acc *= base_wts[t];
  for (int k = 0; k < top; ++k) {
    const int e = ids[(size_t)t * top + k];
    if (e < 0 || e >= E) continue;
    const T* row = a + ((size_t)t * top + k) * F;
    const T* w = down + ((size_t)e * W + c) * F;
    float dot = 0.f;
    for (int i = lane; i < F; i += 32) dot = fmaf(to_float(row[i]), to_float(w[i]), dot);
    acc = fmaf(wts[(size_t)t * top + k], warp_sum(dot), acc);
  }
  if (lane == 0) out[(size_t)t * W + c] = from_float<T>(acc);
}

}  // namespace q3

#define Q3_BY_DTYPE(dtype, ...)                 \
  if ((dtype) == Q3_F32) { using E_ = float; __VA_ARGS__; }  \
  else if ((dtype) == Q3_BF16) { using E_ = __nv_bfloat16; __VA_ARGS__; } \
  else return Q3_ERR_DTYPE;

// h: [T, W] in `dtype`; wr: float32 [E, W]; bias: float32 [E] or null; ids: int32 [T, top]; wts: float32 [T, top].
// softmax: scores by softmax instead of a sigmoid; groups, keep: see the head of the file (1, 1: no groups); renorm: the
// weights divided by the chosen scores' sum.  zbias: float32 [E] or null, added to the logits.  share: float32 [T] or null; with
// it wr is [E + 1, W] and share[t] receives the sigmoid of the last row's product.
extern "C" int q3_moe_route(const void* h, const float* wr, const float* bias, const float* zbias, int* ids, float* wts,
                            float* share, int dtype, int T, int W, int E, int top, float scale, int softmax, int groups,
                            int keep, int renorm, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (W <= 0 || E <= 0 || top <= 0 || top > E || top > q3::MOE_MAX_TOP || E > 4096) return Q3_ERR_SIZE;
  if (groups <= 0 || E % groups || keep <= 0 || keep > groups || top > keep * (E / groups)) return Q3_ERR_SIZE;
  if ((size_t)(2 * E + groups + 3) * sizeof(float) > 48 * 1024) return Q3_ERR_SIZE;
  const q3::Choice choice{E, top, softmax, groups, keep, renorm, scale};
  const int rows = E + (share ? 1 : 0);
  if (dtype == Q3_BF16 && rows <= q3::MR_MAX_ROWS && W % 8 == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)wr % 16 == 0) {
    auto go = [&](auto kernel, int tiles) {
      q3::launch(kernel, dim3((T + q3::MR_TOK - 1) / q3::MR_TOK), dim3(q3::MR_WARPS * 32),
                 ((size_t)((q3::MR_TOK * (2 * E + groups) + 3) & ~3) + q3::MR_WARPS * q3::MR_TOK * (8 * tiles + 1)) * sizeof(float),
                 stream, (const __nv_bfloat16*)h, wr, bias, zbias, ids, wts,
                 share, T, W, choice);
      return q3::launch_status();
    };
    if (rows <= 8) return go(q3::moe_route_mma_kernel<1>, 1);
    if (rows <= 16) return go(q3::moe_route_mma_kernel<2>, 2);
    if (rows <= 24) return go(q3::moe_route_mma_kernel<3>, 3);
    return go(q3::moe_route_mma_kernel<5>, 5);
  }
  // many tokens: eight to a block, so that the experts' rows are read an eighth as often
  constexpr int MANY = 8;
  const size_t es = dtype == Q3_F32 ? 4 : 2;
  const size_t smem_many = (size_t)((MANY * (2 * E + groups) + 3) & ~3) * sizeof(float) + (size_t)MANY * W * es;
  if (T >= 4 * MANY * 32 && W % 4 == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)wr % 16 == 0 && smem_many <= 96 * 1024) {
    const int threads = 32 * (E < 8 ? (E < 4 ? 2 : 4) : 8);
    Q3_BY_DTYPE(dtype, {
      auto kernel = q3::moe_route_kernel<E_, MANY>;
      static bool configured = false;
      if (!configured) {
        const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024);
        if (err != cudaSuccess) return (int)err;
        configured = true;
      }
      q3::launch(kernel, dim3((T + MANY - 1) / MANY), dim3(threads), smem_many, stream, (const E_*)h, wr, bias, zbias, ids, wts, share, T,
                 W, choice);
    })
    return q3::launch_status();
  }
  Q3_BY_DTYPE(dtype, {
    auto kernel = q3::moe_route_kernel<E_, 1>;
    q3::launch(kernel, dim3(T), dim3(E >= 16 ? 512 : (E >= 8 ? 256 : 128)), (size_t)(2 * E + groups + 3) * sizeof(float), stream,
               (const E_*)h, wr, bias, zbias, ids, wts, share, T, W, choice);
  })
  return q3::launch_status();
}

// a: [T * top, F] = act(up[ids] h); out: [T, W] = base + sum_k wts down[ids] a.  act: a Q3_ACT_* code.
// gate_block > 0: gated experts (see the head of the file; only they take Q3_ACT_LIMITED, with its limit); in_wts: float32
// [T * top] or null; base_wts: float32 [T] or null.
extern "C" int q3_moe_pairs(const void* h, const void* up, const void* down, const int* ids, const float* wts,
                            const void* base, void* a, void* out, int dtype, int T, int W, int F, int E, int top, int act,
                            int gate_block, const float* in_wts, const float* base_wts, float limit, cudaStream_t stream) {
  if (gate_block < 0 || (gate_block > 0 && F % gate_block)) return Q3_ERR_SIZE;
  if (T <= 0) return 0;
  if (W <= 0 || F <= 0 || E <= 0 || top <= 0 || (long long)T * top > 0x7fffffffll || F > 4 * 65535 || W > 4 * 65535 || act < 0 || act > Q3_ACT_LIMITED ||
      (act == Q3_ACT_LIMITED && gate_block == 0))
    return Q3_ERR_SIZE;
  const int warps = 4;
  Q3_BY_DTYPE(dtype, q3::launch(q3::moe_pair_up_kernel<E_>, dim3(T * top, (F + warps - 1) / warps), dim3(warps * 32), 0,
                                stream, (const E_*)h, (const E_*)up, ids, (E_*)a, W, F, E, top, act, gate_block, in_wts, limit))
  int code = q3::launch_status();
  if (code) return code;
  Q3_BY_DTYPE(dtype, q3::launch(q3::moe_pair_down_kernel<E_>, dim3(T, (W + warps - 1) / warps), dim3(warps * 32), 0, stream,
                                (const E_*)a, (const E_*)down, ids, wts, (const E_*)base, base_wts, (E_*)out, W, F, E,
                                top))
  return q3::launch_status();
}
