// The channel form of the matrix memories in linear_memory.cu (a decay per token and key channel, a bonus for the token
// itself) as matrix products on the tensor cores: bfloat16 run, prompt portions.
//
// A request's portion is cut into chunks of CC = 64 tokens and these into four parts of CP = 16.  With b_t the sum of the
// log-decays of the chunk's tokens up to and including t (per key channel d), b_-1 = 0, and S_in the state a chunk starts from:
//
//   o_t   = sum_{s < t} m_ts v_s + m_tt v_t + (q_t e^{b_{t-1}})^T S_in,     m_ts = sum_d q_td k_sd e^{b_{t-1,d} - b_{s,d}},
//   S_out = diag(e^{b_last}) S_in + sum_s (k_s e^{b_last - b_s}) v_s^T      m_tt = sum_d q_td u_d k_td
//
//   channel_chunk_state   every chunk's state reached from zero, and its b_last
//   memory carry          chunk after chunk, element by element; leaves every chunk's S_in and the request's last state
//   channel_chunk_output  the outputs of all chunks side by side
//
// No exponent is ever positive.  A decay per channel does not factor out of q_t . k_s, and e^{-b_s} alone can overflow; so
// for t in part i and s in an earlier part the sum is split at the start of part i, b_{t-1} - b_s = (b_{t-1} - B_i) + (B_i -
// b_s), and both factors are products on the tensor cores; within a part (136 pairs) the exponential is taken pair by pair.
// Sums of log-decays are kept relative to their part's start, so a fast decay earlier in the chunk does not cost the later
// ones their last digits.
//
// v is bfloat16 as the projection left it.  Everything else that enters a product carries a decay or is the state: float32,
// split into two bfloat16 halves and multiplied in two products (three where both operands are split, the product of the
// lower halves left out), about 16 bits.  Accumulation is float32.  The float32 run walks token by token (linear_memory.cu).
#include "attn_mma.cuh"

namespace q3 {

constexpr int CC = 64, CP = 16, CPARTS = CC / CP;  // tokens of a chunk, of a part, parts of a chunk
constexpr int CM_THREADS = 256;

__device__ __forceinline__ void cm_split_pack(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16(a - f.x, b - f.y);
}
__device__ __forceinline__ float2 cm_pair(const __nv_bfloat16* p) {  // two neighbouring values
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}

// The logarithms are kept in units of the base-2 exponential.
constexpr float CM_LOG2E = 1.4426950408889634f;
__device__ __forceinline__ float cm_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct ChannelMma {
  const __nv_bfloat16* x;  // [T, ld]: q, k (H heads of D), v (H heads of D) at columns
  int ld, q_col, k_col, v_col;
  const float* logw;   // [T, H, D]
  const float* bonus;  // [H, D]
  int H, num_slots;
  const int *q_start, *slot_ids;
  float* state;    // [slots, H, D, D]: value by value, the keys' channels side by side
  float* records;  // per chunk [H, D, D]: chunk j of request b is record q_start[b] / CC + b + j
  float* totals;   // per chunk [H, D]: b_last (base 2)
  float* out;      // [T, H, D]
  int* status;
};

// D values of each of the chunk's `len` rows to dst [CC][D + 8]; zeros beyond the chunk's end.
template <int D>
__device__ __forceinline__ void cm_rows(__nv_bfloat16* dst, const __nv_bfloat16* __restrict__ src, int ld, int len) {
  for (int i = threadIdx.x; i < CC * (D / 8); i += CM_THREADS) {
    const int t = i / (D / 8), c = (i % (D / 8)) * 8;
    cp_async_16(dst + t * (D + 8) + c, src + (size_t)min(t, len - 1) * ld + c, t < len ? 16 : 0);
  }
  cp_async_commit();
}

// ---------------------------------------------------------------- the state a chunk reaches from zero
// grid (requests, chunks, H).  Shared memory: k weighted, two halves [CC][D + 8] each; v [CC][D + 8]; [PARTS][D] sums.
template <int D>
__global__ void __launch_bounds__(CM_THREADS, 2)
channel_chunk_state_kernel(ChannelMma in) {
  constexpr int PN = D + 8;
  constexpr int PARTS = CM_THREADS / D, PT = CC / PARTS;  // a thread takes PT tokens of one channel
  constexpr int MT = D / 16, WN = (8 / MT) < (D / 16) ? (8 / MT) : (D / 16), NT = D / 8 / WN;
  extern __shared__ __align__(16) unsigned char cm_smem[];
  __nv_bfloat16* k_hi = reinterpret_cast<__nv_bfloat16*>(cm_smem);
  __nv_bfloat16* k_lo = k_hi + CC * PN;
  __nv_bfloat16* vs = k_lo + CC * PN;
  float* sum_s = reinterpret_cast<float*>(vs + CC * PN);
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x, h = blockIdx.z, H = in.H;
  const int slot = in.slot_ids[b];
  const int start = in.q_start[b], t0 = start + blockIdx.y * CC, t1 = in.q_start[b + 1];
  if (t0 >= t1 || slot < 0 || slot >= in.num_slots) return;
  const int len = min(CC, t1 - t0);
  cm_rows<D>(vs, in.x + (size_t)t0 * in.ld + in.v_col + h * D, in.ld, len);
  {
    const int d = threadIdx.x % D, part = threadIdx.x / D;
    float lw[PT], kv[PT], total = 0.f;
#pragma unroll
    for (int i = 0; i < PT; ++i) {
      const int t = part * PT + i;
      lw[i] = t < len ? CM_LOG2E * in.logw[((size_t)(t0 + t) * H + h) * D + d] : 0.f;
      kv[i] = t < len ? __bfloat162float(in.x[(size_t)(t0 + t) * in.ld + in.k_col + h * D + d]) : 0.f;
    }
#pragma unroll
    for (int i = PT - 1; i >= 0; --i) total += lw[i];
    sum_s[part * D + d] = total;
    __syncthreads();
    float after = 0.f;  // the log-decays of everything behind the token
    for (int p = PARTS - 1; p > part; --p) after += sum_s[p * D + d];
    if (part == 0) in.totals[((size_t)(start / CC + b + blockIdx.y) * H + h) * D + d] = after + total;
#pragma unroll
    for (int i = PT - 1; i >= 0; --i) {
      const float v = kv[i] * cm_exp2(after);
      const __nv_bfloat16 hi = __float2bfloat16_rn(v);
      k_hi[(part * PT + i) * PN + d] = hi;
      k_lo[(part * PT + i) * PN + d] = __float2bfloat16_rn(v - __bfloat162float(hi));
      after += lw[i];
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tid4 = lane & 3;
  if (warp >= MT * WN) return;
  const int prow = (warp % MT) * 16, n0 = (warp / MT) * (D / WN);
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < CC / 16; ++kk) {
    uint32_t va[4];  // A[value][s]: the stored [s][value] tile, transposed on the way
    ldmatrix_x4_trans(va, vs + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * PN + prow + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      const int at = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PN + n0 + np * 16 + (lane >> 4) * 8;
      uint32_t hb[4], lb[4];
      ldmatrix_x4_trans(hb, k_hi + at);
      ldmatrix_x4_trans(lb, k_lo + at);
      mma_bf16(acc[2 * np], va, hb[0], hb[1]);
      mma_bf16(acc[2 * np + 1], va, hb[2], hb[3]);
      mma_bf16(acc[2 * np], va, lb[0], lb[1]);
      mma_bf16(acc[2 * np + 1], va, lb[2], lb[3]);
    }
  }
  float* rec = in.records + ((size_t)(start / CC + b + blockIdx.y) * H + h) * D * D;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r)
      *reinterpret_cast<float2*>(rec + (size_t)(prow + gid + 8 * r) * D + n0 + i * 8 + 2 * tid4) =
          make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
}

// grid (requests, H * D * D / 1024): four state values (channels d .. d + 3 of one value) a thread.  The records' "reached
// from zero" become "the state the chunk starts from", the last state goes to the slot.
__global__ void channel_chunk_carry_kernel(ChannelMma in, int D) {
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x, H = in.H;
  const size_t all = (size_t)H * D * D, e = ((size_t)blockIdx.y * blockDim.x + threadIdx.x) * 4;
  const int slot = in.slot_ids[b];
  if (e >= all || slot < 0 || slot >= in.num_slots) return;
  const int t0 = in.q_start[b], chunks = (in.q_start[b + 1] - t0 + CC - 1) / CC;
  if (chunks <= 0) return;
  float4 S = *reinterpret_cast<const float4*>(in.state + (size_t)slot * all + e);
  float* rec = in.records + (size_t)(t0 / CC + b) * all + e;
  const float* tot = in.totals + (size_t)(t0 / CC + b) * H * D + (e / ((size_t)D * D)) * D + e % D;
  constexpr int AHEAD = 8;  // chunks whose loads are in flight together
  for (int j0 = 0; j0 < chunks; j0 += AHEAD, rec += AHEAD * all, tot += (size_t)AHEAD * H * D) {
    float4 reached[AHEAD], keep[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
      if (j0 + k < chunks) {
        reached[k] = *reinterpret_cast<const float4*>(rec + (size_t)k * all);
        keep[k] = *reinterpret_cast<const float4*>(tot + (size_t)k * H * D);
      }
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
      if (j0 + k < chunks) {
        *reinterpret_cast<float4*>(rec + (size_t)k * all) = S;
        S.x = fmaf(cm_exp2(keep[k].x), S.x, reached[k].x);
        S.y = fmaf(cm_exp2(keep[k].y), S.y, reached[k].y);
        S.z = fmaf(cm_exp2(keep[k].z), S.z, reached[k].z);
        S.w = fmaf(cm_exp2(keep[k].w), S.w, reached[k].w);
      }
  }
  *reinterpret_cast<float4*>(in.state + (size_t)slot * all + e) = S;
}

// ---------------------------------------------------------------- what a chunk's tokens read
template <int D>
struct ChannelOut {
  static constexpr int PN = D + 8, PB = D + 4, PM = CC + 4;
  static constexpr int P = D < 64 ? D : 64;                  // values of a state tile
  static constexpr int ROWS = CC * PN * 2;                   // bytes of 64 rows of q, k or v
  static constexpr int SUMS = CPARTS * (CP + 1) * PB * 4;    // exclusive sums of the parts: row n, the first n tokens
  static constexpr int STARTS = (CPARTS + 1) * D * 4, BONUS = D * 4, MAT = CC * PM * 4;
  static constexpr size_t SMEM = 3 * ROWS + SUMS + STARTS + BONUS + MAT;
};

// grid (requests, chunks, H): warps i and i + 4 share the chunk's tokens 16 i .. 16 i + 15.
template <int D>
__global__ void __launch_bounds__(CM_THREADS, 2)
channel_chunk_output_kernel(ChannelMma in) {
  using S = ChannelOut<D>;
  constexpr int PN = S::PN, PB = S::PB, PM = S::PM, P = S::P, NTW = P / 16;  // NTW: column tiles of a warp per state tile
  extern __shared__ __align__(16) unsigned char cm_smem[];
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(cm_smem);  // [CC][PN]
  __nv_bfloat16* ks = qs + CC * PN;                               // [CC][PN]; later the state's upper halves [P][PN]
  __nv_bfloat16* vs = ks + CC * PN;                               // [CC][PN]; later the state's lower halves
  float* sums = reinterpret_cast<float*>(vs + CC * PN);           // [CPARTS][CP + 1][PB]
  float* starts = sums + CPARTS * (CP + 1) * PB;                  // [CPARTS + 1][D]: the parts' log-decays before part i
  float* us = starts + (CPARTS + 1) * D;                          // [D]
  float* mat = us + D;                                            // [CC][PM]: m_ts
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x, h = blockIdx.z, H = in.H;
  const int slot = in.slot_ids[b];
  const int start = in.q_start[b], t0 = start + blockIdx.y * CC, t1 = in.q_start[b + 1];
  if (t0 >= t1) return;
  const int len = min(CC, t1 - t0);
  if (slot < 0 || slot >= in.num_slots) {
    if (threadIdx.x == 0) atomicOr(in.status, Q3_STATUS_BAD_POSITION);
    for (int i = threadIdx.x; i < len * D; i += CM_THREADS) in.out[((size_t)(t0 + i / D) * H + h) * D + i % D] = 0.f;
    return;
  }
  cm_rows<D>(qs, in.x + (size_t)t0 * in.ld + in.q_col + h * D, in.ld, len);
  cm_rows<D>(ks, in.x + (size_t)t0 * in.ld + in.k_col + h * D, in.ld, len);
  cm_rows<D>(vs, in.x + (size_t)t0 * in.ld + in.v_col + h * D, in.ld, len);
  for (int c = threadIdx.x; c < CPARTS * D; c += CM_THREADS) {
    const int part = c / D, d = c % D;
    float lw[CP], sum = 0.f;
#pragma unroll
    for (int i = 0; i < CP; ++i) {
      const int t = part * CP + i;
      lw[i] = t < len ? CM_LOG2E * in.logw[((size_t)(t0 + t) * H + h) * D + d] : 0.f;
    }
    float* dst = sums + part * (CP + 1) * PB + d;
#pragma unroll
    for (int i = 0; i < CP; ++i) {
      dst[i * PB] = sum;
      sum += lw[i];
    }
    dst[CP * PB] = sum;
  }
  for (int d = threadIdx.x; d < D; d += CM_THREADS) us[d] = in.bonus[(size_t)h * D + d];
  __syncthreads();
  for (int d = threadIdx.x; d < D; d += CM_THREADS) {
    float sum = 0.f;
#pragma unroll
    for (int part = 0; part < CPARTS; ++part) {
      starts[part * D + d] = sum;
      sum += sums[(part * (CP + 1) + CP) * PB + d];
    }
    starts[CPARTS * D + d] = sum;
  }
  cp_async_wait<0>();
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tid4 = lane & 3;
  const int part = warp & 3, hf = warp >> 2;
  const float* mine = sums + part * (CP + 1) * PB;  // row n: the log-decays of the part's first n tokens

  // m_ts of earlier parts: the 8-token column tiles of parity hf, up to three of them
  {
    float g[CPARTS - 1][4];
#pragma unroll
    for (int i = 0; i < CPARTS - 1; ++i) g[i][0] = g[i][1] = g[i][2] = g[i][3] = 0.f;
    for (int kk = 0; kk < D / 16 && part > 0; ++kk) {
      uint32_t qh[4], ql[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) {  // registers: row gid (+ 8 for odd r), channels + 8 for r >= 2
        const int row = gid + (r & 1) * 8, d = kk * 16 + 2 * tid4 + (r >> 1) * 8;
        const float2 q = cm_pair(qs + (part * CP + row) * PN + d);
        const float2 e = *reinterpret_cast<const float2*>(mine + row * PB + d);
        cm_split_pack(q.x * cm_exp2(e.x), q.y * cm_exp2(e.y), qh[r], ql[r]);
      }
#pragma unroll
      for (int i = 0; i < CPARTS - 1; ++i) {
        if (i >= part) continue;
        const int s = i * CP + hf * 8 + gid;  // this lane's key
        uint32_t kh[2], kl[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int d = kk * 16 + 2 * tid4 + r * 8;
          const float2 k = cm_pair(ks + s * PN + d);
          const float2 e = *reinterpret_cast<const float2*>(sums + (i * (CP + 1) + hf * 8 + gid + 1) * PB + d);
          const float2 from = *reinterpret_cast<const float2*>(starts + i * D + d);
          const float2 to = *reinterpret_cast<const float2*>(starts + part * D + d);
          cm_split_pack(k.x * cm_exp2(to.x - from.x - e.x), k.y * cm_exp2(to.y - from.y - e.y), kh[r], kl[r]);
        }
        mma_bf16(g[i], qh, kh[0], kh[1]);
        mma_bf16(g[i], qh, kl[0], kl[1]);
        mma_bf16(g[i], ql, kh[0], kh[1]);
      }
    }
#pragma unroll
    for (int i = 0; i < CPARTS - 1; ++i) {
      if (i >= part) continue;
#pragma unroll
      for (int r = 0; r < 2; ++r)
        *reinterpret_cast<float2*>(mat + (part * CP + gid + 8 * r) * PM + i * CP + hf * 8 + 2 * tid4) =
            make_float2(g[i][2 * r], g[i][2 * r + 1]);
    }
  }
  // m_ts within the part, pair by pair: a lane takes one t and the s = c, c + 4, c + 8, c + 12
  {
    const int t = lane & 15, c = (lane >> 4) + 2 * hf;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int d = 0; d < D; d += 4) {
      const float2 q0 = cm_pair(qs + (part * CP + t) * PN + d), q1 = cm_pair(qs + (part * CP + t) * PN + d + 2);
      const float4 bt = *reinterpret_cast<const float4*>(mine + t * PB + d);
      const float4 u = *reinterpret_cast<const float4*>(us + d);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int s = c + 4 * j;
        const float2 k0 = cm_pair(ks + (part * CP + s) * PN + d), k1 = cm_pair(ks + (part * CP + s) * PN + d + 2);
        const float4 bs = *reinterpret_cast<const float4*>(mine + (s + 1) * PB + d);
        const bool own = s == t;
        // beyond the diagonal the exponent would be positive: held at zero, the sum is not used
        const float w0 = own ? u.x : cm_exp2(fminf(bt.x - bs.x, 0.f)), w1 = own ? u.y : cm_exp2(fminf(bt.y - bs.y, 0.f));
        const float w2 = own ? u.z : cm_exp2(fminf(bt.z - bs.z, 0.f)), w3 = own ? u.w : cm_exp2(fminf(bt.w - bs.w, 0.f));
        acc[j] = fmaf(q0.x * k0.x, w0, acc[j]);
        acc[j] = fmaf(q0.y * k0.y, w1, acc[j]);
        acc[j] = fmaf(q1.x * k1.x, w2, acc[j]);
        acc[j] = fmaf(q1.y * k1.y, w3, acc[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = c + 4 * j;
      mat[(part * CP + t) * PM + part * CP + s] = s <= t ? acc[j] : 0.f;
    }
  }
  __syncthreads();
  float acc[D / P][NTW][4];
#pragma unroll
  for (int p = 0; p < D / P; ++p)
#pragma unroll
    for (int i = 0; i < NTW; ++i) acc[p][i][0] = acc[p][i][1] = acc[p][i][2] = acc[p][i][3] = 0.f;
  // m v, over this part and the earlier ones
  for (int kk = 0; kk <= part; ++kk) {
    uint32_t mh[4], ml[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const float2 m = *reinterpret_cast<const float2*>(mat + (part * CP + gid + (r & 1) * 8) * PM + kk * 16 + 2 * tid4 + (r >> 1) * 8);
      cm_split_pack(m.x, m.y, mh[r], ml[r]);
    }
#pragma unroll
    for (int p = 0; p < D / P; ++p)
#pragma unroll
      for (int np = 0; np < NTW / 2; ++np) {
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PN + p * P + hf * (P / 2) + np * 16 + (lane >> 4) * 8);
        mma_bf16(acc[p][2 * np], mh, vb[0], vb[1]);
        mma_bf16(acc[p][2 * np + 1], mh, vb[2], vb[3]);
        mma_bf16(acc[p][2 * np], ml, vb[0], vb[1]);
        mma_bf16(acc[p][2 * np + 1], ml, vb[2], vb[3]);
      }
  }
  // (q e^{b_{t-1}})^T S_in, P values of the state at a time
  const float* rec = in.records + ((size_t)(start / CC + b + blockIdx.y) * H + h) * D * D;
  __nv_bfloat16 *s_hi = ks, *s_lo = vs;
#pragma unroll
  for (int p = 0; p < D / P; ++p) {
    __syncthreads();  // keys and values, or the tile before, have been read
    for (int i = threadIdx.x; i < P * D / 4; i += CM_THREADS) {
      const float4 v = *reinterpret_cast<const float4*>(rec + (size_t)p * P * D + 4 * i);
      uint2 hi, lo;
      cm_split_pack(v.x, v.y, hi.x, lo.x);
      cm_split_pack(v.z, v.w, hi.y, lo.y);
      const int at = (4 * i / D) * PN + (4 * i) % D;
      *reinterpret_cast<uint2*>(s_hi + at) = hi;
      *reinterpret_cast<uint2*>(s_lo + at) = lo;
    }
    __syncthreads();
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t qh[4], ql[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int row = gid + (r & 1) * 8, d = kk * 16 + 2 * tid4 + (r >> 1) * 8;
        const float2 q = cm_pair(qs + (part * CP + row) * PN + d);
        const float2 e = *reinterpret_cast<const float2*>(mine + row * PB + d);
        const float2 f = *reinterpret_cast<const float2*>(starts + part * D + d);
        cm_split_pack(q.x * cm_exp2(e.x + f.x), q.y * cm_exp2(e.y + f.y), qh[r], ql[r]);
      }
#pragma unroll
      for (int np = 0; np < NTW / 2; ++np) {
        const int at = (hf * (P / 2) + np * 16 + (lane & 7) + ((lane >> 4) << 3)) * PN + kk * 16 + ((lane >> 3) & 1) * 8;
        uint32_t hb[4], lb[4];
        ldmatrix_x4(hb, s_hi + at);
        ldmatrix_x4(lb, s_lo + at);
        mma_bf16(acc[p][2 * np], qh, hb[0], hb[1]);
        mma_bf16(acc[p][2 * np + 1], qh, hb[2], hb[3]);
        mma_bf16(acc[p][2 * np], qh, lb[0], lb[1]);
        mma_bf16(acc[p][2 * np + 1], qh, lb[2], lb[3]);
        mma_bf16(acc[p][2 * np], ql, hb[0], hb[1]);
        mma_bf16(acc[p][2 * np + 1], ql, hb[2], hb[3]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = part * CP + gid + 8 * r;
    if (t >= len) continue;
    float* dst = in.out + ((size_t)(t0 + t) * H + h) * D + hf * (P / 2) + 2 * tid4;
#pragma unroll
    for (int p = 0; p < D / P; ++p)
#pragma unroll
      for (int i = 0; i < NTW; ++i)
        *reinterpret_cast<float2*>(dst + p * P + i * 8) = make_float2(acc[p][i][2 * r], acc[p][i][2 * r + 1]);
  }
}

template <int D>
static int channel_mma_launch(const ChannelMma& in, int B, int max_q_len, cudaStream_t stream) {
  constexpr size_t smem_state = 3 * sizeof(__nv_bfloat16) * CC * (D + 8) + sizeof(float) * CM_THREADS;
  constexpr size_t smem_out = ChannelOut<D>::SMEM;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(channel_chunk_state_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_state);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(channel_chunk_output_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_out);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int chunks = (max_q_len + CC - 1) / CC;
  if (chunks > 65535 || in.H > 65535) return Q3_ERR_SIZE;
  const size_t all = (size_t)in.H * D * D;
  launch(channel_chunk_state_kernel<D>, dim3(B, chunks, in.H), dim3(CM_THREADS), smem_state, stream, in);
  launch(channel_chunk_carry_kernel, dim3(B, (unsigned)((all / 4 + 255) / 256)), dim3(256), 0, stream, in, D);
  launch(channel_chunk_output_kernel<D>, dim3(B, chunks, in.H), dim3(CM_THREADS), smem_out, stream, in);
  return launch_status();
}

}  // namespace q3

// Tokens per chunk of the matrix form.
extern "C" int q3_channel_chunk() { return q3::CC; }

// 1 if the matrix form takes keys of D and values of Dv values.
extern "C" int q3_channel_mma_takes(int D, int Dv) { return D == Dv && (D == 32 || D == 64 || D == 128) ? 1 : 0; }

// The arguments of q3_channel_memory_scan (bfloat16, Dv = D).  records: float32, T / 64 + B + 1 records of H * D * D; totals:
// float32, as many of H * D.
extern "C" int q3_channel_memory_scan_mma(const void* x, int ld, int q_col, int k_col, int v_col, const float* logw,
                                          const float* bonus, float* state, const int* q_start, const int* slot_ids,
                                          int num_slots, float* out, float* records, float* totals, int T, int B,
                                          int max_q_len, int H, int D, int* status, cudaStream_t stream) {
  if (B <= 0 || T <= 0 || max_q_len <= 0) return 0;
  if (H <= 0 || !q3_channel_mma_takes(D, D) || num_slots <= 0 || !records || !totals || !logw || !bonus) return Q3_ERR_SIZE;
  if (ld % 8 || q_col % 8 || k_col % 8 || v_col % 8 || (uintptr_t)x % 16 || (uintptr_t)state % 16 || (uintptr_t)records % 16 ||
      (uintptr_t)totals % 16 || (uintptr_t)out % 8)
    return Q3_ERR_ALIGN;
  const q3::ChannelMma in{(const __nv_bfloat16*)x, ld, q_col, k_col, v_col, logw, bonus, H, num_slots, q_start, slot_ids,
                          state, records, totals, out, status};
  if (D == 32) return q3::channel_mma_launch<32>(in, B, max_q_len, stream);
  if (D == 64) return q3::channel_mma_launch<64>(in, B, max_q_len, stream);
  return q3::channel_mma_launch<128>(in, B, max_q_len, stream);
}
