// Matrix memories without a softmax: per head a state S [D, Dv], float32, zero for a new request, carried from token to
// token of a request.
//
//   decayed   S <- decay_h S + k v^T;  o = S^T q                  (a fixed decay per head: retention, lightning attention)
//   delta     g = exp(-exp(A_log_h) softplus(a + dt_bias_h)),  beta = sigmoid(b),  q and k brought to length one
//             S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q                    (the gated delta rule)
//   channel   o = (S + diag(u) k v^T)^T q;  S <- diag(w) S + k v^T     (a decay w per token and key channel, given by its
//             logarithm; the token itself is read with a bonus u per head and channel, before it enters: RWKV's time mixing)
//
//   memory_scan    walks the tokens of every request in order.  A block owns one head of one request and a slice of the
//                  Dv columns; L lanes share a column, each with 4 J of its rows in registers.  A chunk of tokens' q, k,
//                  v is copied into shared memory while the chunk before is walked, then widened (with its activation,
//                  its length, its scalars) once per chunk.  In the delta rule both sums over a column that a token
//                  needs, S^T k and S^T q of the state before the token, are taken together: with p = S_old^T k and
//                  r = S_old^T q,  u = beta (v - g p),  o = g r + (k . q) u,  S = g S_old + k u^T.
//                  The state is read at the start and written at the end, so a prompt in portions walks exactly as the
//                  whole prompt does.  It is kept column by column, [slots, H, Dv, D].
//   low_rank_decay the logarithms of the channel form's decays: -exp(W_2 tanh(low) + w_0) for the rows `low` that a first,
//                  narrow projection left, all in float32.
//   memory_out     o divided by the root mean square of its part of the row (one part, or one per head), times an
//                  optional weight, times sigmoid or silu of a gate: the operand of the output projection.
//   rotate_columns rotation of the first `dims` values of every head (value i with i + dims / 2), in place.
//
// Decays, their logarithms, lengths, sums, gates and the state are float32 in every run; q, k, v come as the projection
// (or the short convolution) left them.
#include "attn_mma.cuh"

namespace q3 {

constexpr int LM_THREADS = 128, LM_WARPS = 4;
enum MemoryRule { LM_DECAYED = 0, LM_DELTA = 1, LM_CHANNEL = 2 };

// Where the operands of a step lie: x [T, ld] with q (G heads of D), k, v (H heads of Dv) at columns of it; for the
// delta rule the pre-activations b and a (H each) at columns of `gates` [T, ldg].
template <typename T>
struct MemoryIn {
  const T* x;
  int ld, q_col, k_col, v_col;
  const T* gates;
  int ldg, b_col, a_col;
  const float *A_log, *dt_bias;     // delta [H]
  const float *decay, *decay_m1;    // decayed [H]: the decay and the decay minus one
  const float *logw, *bonus;        // channel: the decays' logarithms [T, H * D], u [H, D]
  float q_scale;
  int act;                          // Q3_ACT_SILU or Q3_ACT_NONE, on q, k and v
  int vec;                          // rows and slices are made of aligned 16-byte pieces
};

template <typename T>
__device__ __forceinline__ void lm_copy(T* dst, const T* src, int n, int vec, int first, int step) {
  if (vec) {
    constexpr int PER = 16 / sizeof(T);
    for (int i = first * PER; i < n; i += step * PER) cp_async_16(dst + i, src + i, 16);
  } else {
    for (int i = first; i < n; i += step) dst[i] = src[i];
  }
}

template <typename T, int L, int J, int CPT, int RULE>
__global__ void __launch_bounds__(LM_THREADS)
memory_scan_kernel(MemoryIn<T> in, float* __restrict__ state, const int* __restrict__ q_start,
                   const int* __restrict__ slot_ids, int num_slots, float* __restrict__ out, int H, int G, int D, int Dv,
                   int* status) {
  constexpr int DP = 4 * L * J;                     // a row of q or k in shared memory, zeros beyond D
  constexpr int CHUNK = DP <= 128 ? 16 : 2048 / DP; // tokens of a chunk
  constexpr int COLS = (LM_THREADS / L) * CPT;      // columns of a block
  constexpr bool EXACT = sizeof(T) == 4, DELTA = RULE == LM_DELTA, CHANNEL = RULE == LM_CHANNEL;
  extern __shared__ __align__(16) unsigned char lm_smem[];
  float* q_s = reinterpret_cast<float*>(lm_smem);   // [CHUNK][DP]
  float* k_s = q_s + CHUNK * DP;
  float* v_s = k_s + CHUNK * DP;                    // [CHUNK][COLS]
  float* o_s = v_s + CHUNK * COLS;                  // [CHUNK][COLS]
  float* g_s = o_s + CHUNK * COLS;                  // [CHUNK][4]: g, g - 1, beta, k . q; channel: q . (u k)
  float* w_s = g_s + 4 * CHUNK;                     // channel: [CHUNK][DP] decays minus one, then [2][CHUNK][DP] logarithms
  T* raw = reinterpret_cast<T*>(w_s + (CHANNEL ? 3 * CHUNK * DP : 0));  // [2][q: CHUNK][DP] [k] [v: CHUNK][COLS]
  constexpr int RAW = CHUNK * (2 * DP + COLS);

  const int b = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * COLS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int l = threadIdx.x % L, grp = threadIdx.x / L;
  const int slot = slot_ids[b];
  const int t0 = q_start[b], t1 = q_start[b + 1];
  if (slot < 0 || slot >= num_slots) {
    pdl_wait();
    pdl_launch_dependents();
    if (threadIdx.x == 0) atomicOr(status, Q3_STATUS_BAD_POSITION);
    for (int t = t0; t < t1; ++t)
      for (int c = threadIdx.x; c < COLS && col0 + c < Dv; c += LM_THREADS) out[((size_t)t * H + h) * Dv + col0 + c] = 0.f;
    return;
  }
  // the slot was last written by an earlier step: its state may be read ahead of the wait
  float* st = state + ((size_t)slot * H + h) * (size_t)Dv * D;
  const bool d4 = (D & 3) == 0;
  float S[CPT][J][4];
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
    const int col = col0 + grp * CPT + c;
#pragma unroll
    for (int j = 0; j < J; ++j) {
      const int d = 4 * (l + L * j);
      S[c][j][0] = S[c][j][1] = S[c][j][2] = S[c][j][3] = 0.f;
      if (col < Dv && d < D) {
        const float* p = st + (size_t)col * D + d;
        if (d4) {
          const float4 v = *reinterpret_cast<const float4*>(p);
          S[c][j][0] = v.x, S[c][j][1] = v.y, S[c][j][2] = v.z, S[c][j][3] = v.w;
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (d + i < D) S[c][j][i] = p[i];
        }
      }
    }
  }
  float rate = 0.f, bias = 0.f, dec = 1.f, dec1 = 0.f;
  if (DELTA) {
    rate = -expf(in.A_log[h]);
    bias = in.dt_bias[h];
  } else if (!CHANNEL) {
    dec = in.decay[h];
    dec1 = in.decay_m1[h];
  }
  const int hk = h / (H / G);
  const int vn = min(COLS, Dv - col0);
  pdl_wait();
  pdl_launch_dependents();

  auto fetch = [&](int c0, int buf) {  // a chunk's rows as they are
    T* r = raw + buf * RAW;
    const int cn = min(CHUNK, t1 - c0);
    for (int c = warp; c < cn; c += LM_WARPS) {
      const T* row = in.x + (size_t)(c0 + c) * in.ld;
      lm_copy(r + c * DP, row + in.q_col + hk * D, D, in.vec, lane, 32);
      lm_copy(r + (CHUNK + c) * DP, row + in.k_col + hk * D, D, in.vec, lane, 32);
      lm_copy(r + 2 * CHUNK * DP + c * COLS, row + in.v_col + h * Dv + col0, vn, in.vec, lane, 32);
      if constexpr (CHANNEL)
        lm_copy(w_s + (1 + buf) * CHUNK * DP + c * DP, in.logw + ((size_t)(c0 + c) * H + h) * D, D, in.vec, lane, 32);
    }
    cp_async_commit();
  };

  int buf = 0;
  if (t0 < t1) fetch(t0, 0);
  for (int c0 = t0; c0 < t1; c0 += CHUNK, buf ^= 1) {
    const int cn = min(CHUNK, t1 - c0);
    cp_async_wait<0>();
    __syncthreads();  // the chunk has arrived, and the chunk before has been walked and written by everybody
    if (c0 + CHUNK < t1) fetch(c0 + CHUNK, buf ^ 1);
    const T* r = raw + buf * RAW;
    for (int c = warp; c < cn; c += LM_WARPS) {
      const T *rq = r + c * DP, *rk = r + (CHUNK + c) * DP, *rv = r + 2 * CHUNK * DP + c * COLS;
      float fq = in.q_scale, fk = 1.f;
      if (DELTA) {
        float sq = 0.f, sk = 0.f, kq = 0.f;
        for (int d = lane; d < D; d += 32) {
          const float qv = to_float(rq[d]), kv = to_float(rk[d]);
          sq = fmaf(qv, qv, sq);
          sk = fmaf(kv, kv, sk);
          kq = fmaf(qv, kv, kq);
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        kq = warp_sum(kq);
        fq = in.q_scale / sqrtf(sq + 1e-6f);
        fk = 1.0f / sqrtf(sk + 1e-6f);
        if (lane == 0) {
          const T* gr = in.gates + (size_t)(c0 + c) * in.ldg;
          const float pre = to_float(gr[in.a_col + h]) + bias;
          const float lg = rate * softplus_f(pre);
          g_s[4 * c] = expf(lg);
          g_s[4 * c + 1] = expm1f(lg);
          g_s[4 * c + 2] = sigmoid_f(to_float(gr[in.b_col + h]));
          g_s[4 * c + 3] = kq * fq * fk;
        }
      }
      [[maybe_unused]] float own = 0.f;
      for (int d = lane; d < DP; d += 32) {
        float qv = 0.f, kv = 0.f;
        if (d < D) {
          qv = to_float(rq[d]);
          kv = to_float(rk[d]);
          if (in.act == Q3_ACT_SILU) {
            qv = silu_f(qv);
            kv = silu_f(kv);
          }
        }
        q_s[c * DP + d] = qv * fq;
        k_s[c * DP + d] = kv * fk;
        if constexpr (CHANNEL) {
          w_s[c * DP + d] = d < D ? expm1f(w_s[(1 + buf) * CHUNK * DP + c * DP + d]) : 0.f;
          if (d < D) own = fmaf(qv * fq, in.bonus[(size_t)h * D + d] * kv, own);
        }
      }
      if constexpr (CHANNEL) {
        own = warp_sum(own);
        if (lane == 0) g_s[4 * c] = own;
      }
      for (int d = lane; d < COLS; d += 32) {
        float v = d < vn ? to_float(rv[d]) : 0.f;
        if (in.act == Q3_ACT_SILU) v = silu_f(v);
        v_s[c * COLS + d] = v;
      }
    }
    __syncthreads();
#pragma unroll 4
    for (int c = 0; c < cn; ++c) {
      float kk[J][4], qq[J][4];
#pragma unroll
      for (int j = 0; j < J; ++j) {
        const float4 kv = *reinterpret_cast<const float4*>(k_s + c * DP + 4 * (l + L * j));
        const float4 qv = *reinterpret_cast<const float4*>(q_s + c * DP + 4 * (l + L * j));
        kk[j][0] = kv.x, kk[j][1] = kv.y, kk[j][2] = kv.z, kk[j][3] = kv.w;
        qq[j][0] = qv.x, qq[j][1] = qv.y, qq[j][2] = qv.z, qq[j][3] = qv.w;
      }
      float vv[CPT], o[CPT];
#pragma unroll
      for (int i = 0; i < CPT; ++i) vv[i] = v_s[c * COLS + grp * CPT + i];
      if constexpr (DELTA) {
        const float4 gs = *reinterpret_cast<const float4*>(g_s + 4 * c);
        float p[CPT], rr[CPT];
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          float pa[4] = {0.f, 0.f, 0.f, 0.f}, ra[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
          for (int j = 0; j < J; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              pa[e] = fmaf(S[i][j][e], kk[j][e], pa[e]);
              ra[e] = fmaf(S[i][j][e], qq[j][e], ra[e]);
            }
          p[i] = (pa[0] + pa[1]) + (pa[2] + pa[3]);
          rr[i] = (ra[0] + ra[1]) + (ra[2] + ra[3]);
        }
#pragma unroll
        for (int w = L >> 1; w > 0; w >>= 1)
#pragma unroll
          for (int i = 0; i < CPT; ++i) {
            p[i] += __shfl_xor_sync(0xffffffffu, p[i], w);
            rr[i] += __shfl_xor_sync(0xffffffffu, rr[i], w);
          }
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          const float gp = EXACT ? fmaf(gs.y, p[i], p[i]) : gs.x * p[i];
          const float u = gs.z * (vv[i] - gp);
          o[i] = fmaf(gs.w, u, EXACT ? fmaf(gs.y, rr[i], rr[i]) : gs.x * rr[i]);
#pragma unroll
          for (int j = 0; j < J; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e)
              S[i][j][e] = EXACT ? S[i][j][e] + fmaf(gs.y, S[i][j][e], kk[j][e] * u) : fmaf(gs.x, S[i][j][e], kk[j][e] * u);
        }
      } else if constexpr (CHANNEL) {
        float w1[J][4];
#pragma unroll
        for (int j = 0; j < J; ++j) {
          const float4 wv = *reinterpret_cast<const float4*>(w_s + c * DP + 4 * (l + L * j));
          w1[j][0] = wv.x, w1[j][1] = wv.y, w1[j][2] = wv.z, w1[j][3] = wv.w;
        }
        const float own = g_s[4 * c];
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          float ra[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
          for (int j = 0; j < J; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              ra[e] = fmaf(S[i][j][e], qq[j][e], ra[e]);
              S[i][j][e] += fmaf(w1[j][e], S[i][j][e], kk[j][e] * vv[i]);
            }
          o[i] = (ra[0] + ra[1]) + (ra[2] + ra[3]);
        }
#pragma unroll
        for (int w = L >> 1; w > 0; w >>= 1)
#pragma unroll
          for (int i = 0; i < CPT; ++i) o[i] += __shfl_xor_sync(0xffffffffu, o[i], w);
#pragma unroll
        for (int i = 0; i < CPT; ++i) o[i] = fmaf(own, vv[i], o[i]);
      } else {
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          float ra[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
          for (int j = 0; j < J; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              S[i][j][e] = EXACT ? S[i][j][e] + fmaf(dec1, S[i][j][e], kk[j][e] * vv[i])
                                 : fmaf(dec, S[i][j][e], kk[j][e] * vv[i]);
              ra[e] = fmaf(S[i][j][e], qq[j][e], ra[e]);
            }
          o[i] = (ra[0] + ra[1]) + (ra[2] + ra[3]);
        }
#pragma unroll
        for (int w = L >> 1; w > 0; w >>= 1)
#pragma unroll
          for (int i = 0; i < CPT; ++i) o[i] += __shfl_xor_sync(0xffffffffu, o[i], w);
      }
      if (l == 0)
#pragma unroll
        for (int i = 0; i < CPT; ++i) o_s[c * COLS + grp * CPT + i] = o[i];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < cn * COLS; i += LM_THREADS) {
      const int c = i / COLS, d = i - c * COLS;
      if (d < vn) out[((size_t)(c0 + c) * H + h) * Dv + col0 + d] = o_s[i];
    }
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
    const int col = col0 + grp * CPT + c;
#pragma unroll
    for (int j = 0; j < J; ++j) {
      const int d = 4 * (l + L * j);
      if (col < Dv && d < D) {
        float* p = st + (size_t)col * D + d;
        if (d4) {
          *reinterpret_cast<float4*>(p) = make_float4(S[c][j][0], S[c][j][1], S[c][j][2], S[c][j][3]);
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (d + i < D) p[i] = S[c][j][i];
        }
      }
    }
  }
}

template <typename T, int L, int J, int CPT, int RULE>
static int memory_scan_launch(const MemoryIn<T>& in, float* state, const int* q_start, const int* slot_ids, int num_slots,
                              float* out, int B, int H, int G, int D, int Dv, int* status, cudaStream_t stream) {
  constexpr int DP = 4 * L * J, CHUNK = DP <= 128 ? 16 : 2048 / DP, COLS = (LM_THREADS / L) * CPT;
  constexpr size_t smem = sizeof(float) * (size_t)(CHUNK * (2 * DP + 2 * COLS) + 4 * CHUNK + (RULE == LM_CHANNEL ? 3 * CHUNK * DP : 0)) +
                          2 * sizeof(T) * (size_t)CHUNK * (2 * DP + COLS);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(memory_scan_kernel<T, L, J, CPT, RULE>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  MemoryIn<T> args = in;
  // 16-byte pieces: rows, columns, heads and slices all start on one
  constexpr int PER = 16 / sizeof(T);
  args.vec = (uintptr_t)in.x % 16 == 0 && in.ld % PER == 0 && in.q_col % PER == 0 && in.k_col % PER == 0 &&
             in.v_col % PER == 0 && D % PER == 0 && Dv % PER == 0 && COLS % PER == 0 && (uintptr_t)in.logw % 16 == 0;
  launch(memory_scan_kernel<T, L, J, CPT, RULE>, dim3((Dv + COLS - 1) / COLS, H, B), dim3(LM_THREADS), smem, stream, args,
         state, q_start, slot_ids, num_slots, out, H, G, D, Dv, status);
  return launch_status();
}

template <typename T, int RULE>
static int memory_scan_sizes(const MemoryIn<T>& in, float* state, const int* q_start, const int* slot_ids, int num_slots,
                             float* out, int B, int H, int G, int D, int Dv, int* status, cudaStream_t stream) {
#define Q3_LM(L, J)                                                                                                     \
  {                                                                                                                     \
    const long long wide = (long long)B * H * ((Dv + 2 * (LM_THREADS / L) - 1) / (2 * (LM_THREADS / L)));               \
    if (wide >= 4LL * sm_count())                                                                                       \
      return memory_scan_launch<T, L, J, 2, RULE>(in, state, q_start, slot_ids, num_slots, out, B, H, G, D, Dv, status, \
                                                   stream);                                                             \
    return memory_scan_launch<T, L, J, 1, RULE>(in, state, q_start, slot_ids, num_slots, out, B, H, G, D, Dv, status,  \
                                                 stream);                                                               \
  }
  if (D <= 32) Q3_LM(4, 2)
  if (D <= 64) Q3_LM(4, 4)
  if (D <= 128) Q3_LM(8, 4)
  if (D <= 256) Q3_LM(16, 4)
  Q3_LM(32, 4)
#undef Q3_LM
}

// ---------------------------------------------------------------- decays from a low-rank projection
// logw[t, c] = -exp(sum_r w2[c, r] tanh(low[t, r]) + w0[c]), at least LR_LEAST (whose exponential is zero in float32).
// low: [T, ld]; w2t: [R, C]; w0: [C]; logw: [T, C].  Every sum runs over r in order, so that a token's decays do not depend on how
// many there are.  For many tokens a block takes LR_TT of them and LR_TC channels, a thread 4 x 8; for a few, a warp per token and
// LF_C channels, with all of their weights in shared memory.
constexpr int LR_R = 32, LR_TT = 64, LR_TC = 128, LR_THREADS = LR_TT * LR_TC / 32;
constexpr int LF_T = 8, LF_C = 32, LF_MAX_R = 256;
constexpr float LR_LEAST = -104.f;

__device__ __forceinline__ float log_decay_of(float sum, float w0) { return fmaxf(-expf(sum + w0), LR_LEAST); }

__global__ void __launch_bounds__(LR_THREADS, 4)
low_rank_decay_kernel(const float* __restrict__ low, int ld, const float* __restrict__ w2t, const float* __restrict__ w0,
                      float* __restrict__ logw, int Ttot, int C, int R) {
  __shared__ __align__(16) float a_s[LR_R][LR_TT + 4], w_s[LR_R][LR_TC + 4];
  const int t0 = blockIdx.y * LR_TT, c0 = blockIdx.x * LR_TC;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;  // channels 4 tx .. and 64 + 4 tx .., tokens 4 ty .. 4 ty + 3
  auto weights = [&](int r0) {
#pragma unroll 4
    for (int i = threadIdx.x; i < LR_TC * LR_R; i += LR_THREADS) {
      const int c = i % LR_TC, r = i / LR_TC;
      w_s[r][c] = c0 + c < C && r0 + r < R ? w2t[(size_t)(r0 + r) * C + c0 + c] : 0.f;
    }
  };
  weights(0);  // they do not depend on the kernel before this one
  pdl_wait();
  pdl_launch_dependents();
  float acc[2][4][4] = {};
  for (int r0 = 0; r0 < R; r0 += LR_R) {
    if (r0 > 0) {
      __syncthreads();
      weights(r0);
    }
#pragma unroll 4
    for (int i = threadIdx.x; i < LR_TT * LR_R; i += LR_THREADS) {
      const int t = i / LR_R, r = i % LR_R;
      a_s[r][t] = t0 + t < Ttot && r0 + r < R ? tanhf(low[(size_t)(t0 + t) * ld + r0 + r]) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int r = 0; r < LR_R; ++r) {
      const float4 av = *reinterpret_cast<const float4*>(&a_s[r][4 * ty]);
      const float a[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        const float4 w = *reinterpret_cast<const float4*>(&w_s[r][64 * p + 4 * tx]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          acc[p][i][0] = fmaf(a[i], w.x, acc[p][i][0]);
          acc[p][i][1] = fmaf(a[i], w.y, acc[p][i][1]);
          acc[p][i][2] = fmaf(a[i], w.z, acc[p][i][2]);
          acc[p][i][3] = fmaf(a[i], w.w, acc[p][i][3]);
        }
      }
    }
  }
  const bool by4 = (C & 3) == 0;
#pragma unroll
  for (int p = 0; p < 2; ++p) {
    const int c = c0 + 64 * p + 4 * tx;
    if (c >= C) continue;
    float off[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) off[j] = c + j < C ? w0[c + j] : 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = t0 + 4 * ty + i;
      if (t >= Ttot) continue;
      float* dst = logw + (size_t)t * C + c;
      const float v[4] = {log_decay_of(acc[p][i][0], off[0]), log_decay_of(acc[p][i][1], off[1]),
                          log_decay_of(acc[p][i][2], off[2]), log_decay_of(acc[p][i][3], off[3])};
      if (by4) {
        *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (c + j < C) dst[j] = v[j];
      }
    }
  }
}

__global__ void __launch_bounds__(LF_T * 32)
low_rank_decay_few_kernel(const float* __restrict__ low, int ld, const float* __restrict__ w2t, const float* __restrict__ w0,
                          float* __restrict__ logw, int Ttot, int C, int R) {
  extern __shared__ float lf_smem[];  // [R][LF_C] weights, [LF_T][R] inputs
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * LF_C + lane, t = blockIdx.y * LF_T + warp;
  float* w_s = lf_smem;
  float* a_s = lf_smem + R * LF_C + warp * R;
#pragma unroll 8
  for (int r = warp; r < R; r += LF_T) w_s[r * LF_C + lane] = c < C ? w2t[(size_t)r * C + c] : 0.f;
  const float off = c < C ? w0[c] : 0.f;
  pdl_wait();
  pdl_launch_dependents();
  if (t < Ttot)
    for (int r = lane; r < R; r += 32) a_s[r] = tanhf(low[(size_t)t * ld + r]);
  __syncthreads();
  if (t >= Ttot || c >= C) return;
  float acc = 0.f;
#pragma unroll 8
  for (int r = 0; r < R; ++r) acc = fmaf(a_s[r], w_s[r * LF_C + lane], acc);
  logw[(size_t)t * C + c] = log_decay_of(acc, off);
}

// ---------------------------------------------------------------- the norm and the gate behind a memory
// A unit (LANES lanes of a warp, or with WHOLE a block) per (token, part), V values per access.  o: float32 [T, n]; gates at g_col of
// proj; weight [n] (w_stride = width of a part), [width] shared by the parts (w_stride = 0), or null.
template <typename T, int V>
struct alignas(sizeof(T) * V) LmPack { T v[V]; };

template <typename T, int V, bool WHOLE, int LANES = 32>
__global__ void memory_out_kernel(const float* __restrict__ o, const T* __restrict__ proj, int ld, int g_col,
                                  const float* __restrict__ w, int w_stride, float eps, int gate, T* __restrict__ out,
                                  int ldo, int n, int parts, int units) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  int unit = WHOLE ? blockIdx.x : blockIdx.x * (blockDim.x / LANES) + threadIdx.x / LANES;
  const bool live = unit < units;
  if (WHOLE || LANES == 32) {
    if (!live) return;
  } else {
    unit = min(unit, units - 1);  // lanes of one warp stay together for the sum
  }
  const int first = WHOLE ? threadIdx.x : threadIdx.x % LANES, step = WHOLE ? blockDim.x : LANES;
  const int t = unit / parts, part = unit - t * parts, width = n / parts, c0 = part * width;
  const float* row = o + (size_t)t * n + c0;
  const T* gr = proj + (size_t)t * ld + g_col + c0;
  const float* wr = w ? w + (size_t)part * w_stride : nullptr;
  T* dst = out + (size_t)t * ldo + c0;
  float ss = 0.f;
#pragma unroll 4
  for (int i = first * V; i < width; i += step * V) {
    const LmPack<float, V> x = *reinterpret_cast<const LmPack<float, V>*>(row + i);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(x.v[e], x.v[e], ss);
  }
  if (WHOLE) {
    ss = block_sum(ss, red);
  } else {
#pragma unroll
    for (int w = LANES / 2; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
    if (!live) return;
  }
  const float inv = 1.0f / sqrtf(ss / (float)width + eps);
#pragma unroll 4
  for (int i = first * V; i < width; i += step * V) {
    const LmPack<float, V> x = *reinterpret_cast<const LmPack<float, V>*>(row + i);
    const LmPack<T, V> g = *reinterpret_cast<const LmPack<T, V>*>(gr + i);
    LmPack<float, V> wv;
    if (wr) wv = *reinterpret_cast<const LmPack<float, V>*>(wr + i);
    LmPack<T, V> y;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float gv = to_float(g.v[e]);
      float v = x.v[e] * inv;
      if (wr) v *= wv.v[e];
      y.v[e] = from_float<T>(v * (gate == Q3_ACT_SILU ? silu_f(gv) : sigmoid_f(gv)));
    }
    *reinterpret_cast<LmPack<T, V>*>(dst + i) = y;
  }
}

// grid (T).  x: rows of ld values; `heads` vectors of D values from column `col`.
template <typename T>
__global__ void rotate_columns_kernel(T* __restrict__ x, int ld, int col, int heads, int D, int dims,
                                      const float* __restrict__ freq, float mag, const int* __restrict__ positions) {
  extern __shared__ float cs[];  // [dims / 2] cosines, then sines
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, half = dims >> 1;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, c;
    sincosf(pos * freq[i], &sn, &c);
    cs[i] = c * mag;
    cs[half + i] = sn * mag;
  }
  __syncthreads();
  T* row = x + (size_t)t * ld + col;
  for (int e = threadIdx.x; e < heads * half; e += blockDim.x) {
    const int h = e / half, i = e - h * half;
    T* p = row + (size_t)h * D + i;
    const float u = to_float(p[0]), v = to_float(p[half]);
    p[0] = from_float<T>(u * cs[i] - v * cs[half + i]);
    p[half] = from_float<T>(v * cs[i] + u * cs[half + i]);
  }
}

}  // namespace q3

#define Q3_BY_DTYPE(dtype, ...)                 \
  if ((dtype) == Q3_F32) { using E = float; __VA_ARGS__; }  \
  else if ((dtype) == Q3_BF16) { using E = __nv_bfloat16; __VA_ARGS__; } \
  else return Q3_ERR_DTYPE;

// The largest key size the scan takes.
extern "C" int q3_memory_max_dim() { return 512; }

// x: [T, ld] in `dtype` with q (G * D), k (G * D) and v (H * Dv) at the given columns; head h reads q and k of head
// h / (H / G).  state: float32 [num_slots, H, Dv, D]; out: float32 [T, H * Dv].  q is multiplied by q_scale.
// decay and decay_m1 (float32 [H]): fixed decays and decays minus one; or null, and then the delta rule with the
// pre-activations b and a at columns of gates [T, ldg] and A_log, dt_bias (float32 [H]).
extern "C" int q3_memory_scan(const void* x, int ld, int q_col, int k_col, int v_col, const void* gates, int ldg, int b_col,
                              int a_col, const float* A_log, const float* dt_bias, const float* decay,
                              const float* decay_m1, float q_scale, int act, float* state, const int* q_start,
                              const int* slot_ids, int num_slots, float* out, int dtype, int B, int H, int G, int D, int Dv,
                              int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || H > 65535 || B > 65535 || D <= 0 || D > 512 || Dv <= 0 || num_slots <= 0 ||
      (act != Q3_ACT_SILU && act != Q3_ACT_NONE))
    return Q3_ERR_SIZE;
  if (!decay && (!gates || !A_log || !dt_bias || act != Q3_ACT_NONE)) return Q3_ERR_SIZE;
  if (decay && !decay_m1) return Q3_ERR_SIZE;
#define Q3_LM_DTYPE(E)                                                                                                     \
  {                                                                                                                        \
    const q3::MemoryIn<E> in{(const E*)x, ld, q_col, k_col, v_col, (const E*)gates, ldg, b_col, a_col, A_log, dt_bias,     \
                             decay, decay_m1, nullptr, nullptr, q_scale, act, 0};                                                            \
    if (decay)                                                                                                             \
      return q3::memory_scan_sizes<E, q3::LM_DECAYED>(in, state, q_start, slot_ids, num_slots, out, B, H, G, D, Dv, status, stream); \
    return q3::memory_scan_sizes<E, q3::LM_DELTA>(in, state, q_start, slot_ids, num_slots, out, B, H, G, D, Dv, status, stream);   \
  }
  if (dtype == Q3_F32) Q3_LM_DTYPE(float)
  if (dtype == Q3_BF16) Q3_LM_DTYPE(__nv_bfloat16)
#undef Q3_LM_DTYPE
  return Q3_ERR_DTYPE;
}

// The channel form (see the head of the file): x as above with one query/key head per value head; logw: float32 [T, H * D],
// the logarithms of the decays; bonus: float32 [H, D].
extern "C" int q3_channel_memory_scan(const void* x, int ld, int q_col, int k_col, int v_col, const float* logw,
                                      const float* bonus, float* state, const int* q_start, const int* slot_ids, int num_slots,
                                      float* out, int dtype, int B, int H, int D, int Dv, int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H <= 0 || H > 65535 || B > 65535 || D <= 0 || D > 512 || Dv <= 0 || num_slots <= 0 || !logw || !bonus) return Q3_ERR_SIZE;
  Q3_BY_DTYPE(dtype, {
    const q3::MemoryIn<E> in{(const E*)x, ld, q_col, k_col, v_col, nullptr, 0, 0, 0, nullptr, nullptr, nullptr, nullptr, logw,
                             bonus, 1.0f, Q3_ACT_NONE, 0};
    return q3::memory_scan_sizes<E, q3::LM_CHANNEL>(in, state, q_start, slot_ids, num_slots, out, B, H, H, D, Dv, status, stream);
  })
}

// low: float32 rows of ld values (the first R are read); w2t: float32 [R, C]; w0: float32 [C]; logw: float32 [T, C].
extern "C" int q3_low_rank_decay(const float* low, int ld, const float* w2t, const float* w0, float* logw, int T, int C, int R,
                                 cudaStream_t stream) {
  if (T <= 0) return 0;
  if (C <= 0 || R <= 0 || R > ld || T > q3::LF_T * 65535) return Q3_ERR_SIZE;
  if ((uintptr_t)logw % 16) return Q3_ERR_ALIGN;
  if (T <= 128 && R <= q3::LF_MAX_R)
    q3::launch(q3::low_rank_decay_few_kernel, dim3((C + q3::LF_C - 1) / q3::LF_C, (T + q3::LF_T - 1) / q3::LF_T), dim3(q3::LF_T * 32),
               (size_t)R * (q3::LF_C + q3::LF_T) * sizeof(float), stream, low, ld, w2t, w0, logw, T, C, R);
  else
    q3::launch(q3::low_rank_decay_kernel, dim3((C + q3::LR_TC - 1) / q3::LR_TC, (T + q3::LR_TT - 1) / q3::LR_TT), dim3(q3::LR_THREADS),
               0, stream, low, ld, w2t, w0, logw, T, C, R);
  return q3::launch_status();
}

// weight: float32 [n], [n / parts] with weight_shared, or null.  gate: Q3_ACT_SILU, or Q3_ACT_NONE for a sigmoid.
extern "C" int q3_memory_out(const float* o, const void* proj, int ld, int g_col, const float* weight, int weight_shared,
                             float eps, int gate, void* out, int ldo, int dtype, int T, int n, int parts,
                             cudaStream_t stream) {
  if (T <= 0) return 0;
  if (n <= 0 || parts <= 0 || n % parts || parts > 65535 || ldo < n) return Q3_ERR_SIZE;
  const int width = n / parts, shared = weight_shared ? 0 : width;
  const long long units = (long long)T * parts;
  if (units > 0x7fffffffll) return Q3_ERR_SIZE;
  const size_t es = dtype == Q3_F32 ? 4 : 2;
  const bool by4 = width % 4 == 0 && n % 4 == 0 && ld % 4 == 0 && g_col % 4 == 0 && ldo % 4 == 0 && (uintptr_t)o % 16 == 0 &&
                   (uintptr_t)proj % (4 * es) == 0 && (uintptr_t)out % (4 * es) == 0 && (uintptr_t)weight % 16 == 0;
  // a block per part where parts are long, else a warp per part
  const bool whole = width >= 512;
  const int threads = whole ? (width >= 2048 ? 512 : 256) : 128;
  const int lanes = !by4 || whole || width > 64 ? 32 : (width > 32 ? 16 : 8);  // short parts: several to a warp
  const unsigned grid = (unsigned)(whole ? units : (units * lanes + threads - 1) / threads);
#define Q3_MEMORY_OUT(V, WHOLE, LANES)                                                                                         \
  Q3_BY_DTYPE(dtype, {                                                                                                   \
    auto kernel = q3::memory_out_kernel<E, V, WHOLE, LANES>;                                                                    \
    q3::launch(kernel, dim3(grid), dim3(threads), 0, stream, o, (const E*)proj, ld, g_col, weight, shared, eps, gate, (E*)out, \
               ldo, n, parts, (int)units);                                                                               \
  })
  if (by4 && whole) { Q3_MEMORY_OUT(4, true, 32) }
  else if (by4 && lanes == 16) { Q3_MEMORY_OUT(4, false, 16) }
  else if (by4 && lanes == 8) { Q3_MEMORY_OUT(4, false, 8) }
  else if (by4) { Q3_MEMORY_OUT(4, false, 32) }
  else if (whole) { Q3_MEMORY_OUT(1, true, 32) }
  else { Q3_MEMORY_OUT(1, false, 32) }
#undef Q3_MEMORY_OUT
  return q3::launch_status();
}

// In place: `heads` vectors of D values from column `col` of x [T, ld].
extern "C" int q3_rotate_columns(void* x, int ld, int col, int heads, int D, int dims, const float* freq, float mag,
                                 const int* positions, int dtype, int T, cudaStream_t stream) {
  if (T <= 0 || dims == 0 || heads <= 0) return 0;
  if (dims < 0 || dims % 2 || dims > D || dims > 8192 || col < 0 || col + heads * D > ld) return Q3_ERR_SIZE;
  Q3_BY_DTYPE(dtype, q3::launch(q3::rotate_columns_kernel<E>, dim3(T), dim3(256), (size_t)dims * sizeof(float), stream,
                                (E*)x, ld, col, heads, D, dims, freq, mag, positions))
  return q3::launch_status();
}
