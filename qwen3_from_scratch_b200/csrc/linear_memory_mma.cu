// The matrix memories of linear_memory.cu in their matrix form, on the tensor cores (bfloat16 run, prompt portions).
//
// A request's portion is cut into chunks of LC = 64 tokens.  With b_t the sum of the log-decays of the chunk's tokens up
// to and including t, and S_in the state a chunk starts from:
//
//   decayed   o_t   = sum_{s <= t} e^{b_t - b_s} (q_t . k_s) v_s  +  e^{b_t} S_in^T q_t
//             S_out = e^{b_last} S_in + sum_s e^{b_last - b_s} k_s v_s^T
//   delta     the same with u_s in place of v_s, where the rule u_t = beta_t (v_t - g_t S_{t-1}^T k_t) unrolls to
//             (I + A) U = diag(beta) (V - diag(e^b) K S_in),   A[t, s] = beta_t e^{b_t - b_s} (k_t . k_s)  for s < t
//             so with Tm = (I + A)^-1 (unit lower triangular):  U = Tm diag(beta) V - (Tm diag(beta e^b) K) S_in = U0 - W S_in
//
// (no exponent is ever positive).  Launches:
//   decayed: memory_chunk_state (every chunk's state reached from zero), memory_chunk_carry (chunk after chunk, leaves S_in),
//            memory_chunk_output
//   delta:   delta_chunk_prepare (Tm, W, U0 of every chunk side by side), delta_chunk_walk (chunk after chunk with the state
//            in registers: U = U0 - W S, the next state; leaves U and S_in), memory_chunk_output
//
// What enters a product must be bfloat16.  q, k and v are (the projection, the convolution or the rotation left them so;
// lengths and decays multiply finished sums or the other operand).  Everything that carries a decay, a length, beta, Tm, W,
// U or the state is float32 and is split into two bfloat16 halves, v = hi + lo, lo = bf16(v - hi), and multiplied in two
// products (three where both operands are split, the product of the two lower halves left out), which keeps about 16 bits.
// Accumulation is float32.  The float32 run does not come here: it walks token by token (linear_memory.cu).
#include "attn_mma.cuh"

namespace q3 {

constexpr int LC = 64;  // tokens per chunk
constexpr int LMM_THREADS = 128;

__device__ __forceinline__ void lm_split(float v, float& hi, float& lo) {
  hi = __bfloat162float(__float2bfloat16_rn(v));
  lo = v - hi;  // rounded when it is packed
}
__device__ __forceinline__ void lm_split_pack(float a, float b, uint32_t& hi, uint32_t& lo) {
  float ah, al, bh, bl;
  lm_split(a, ah, al);
  lm_split(b, bh, bl);
  hi = pack_bf16(ah, bh);
  lo = pack_bf16(al, bl);
}
__device__ __forceinline__ uint32_t silu_pair(uint32_t w) {  // rounded to bfloat16: the hardware's exponential and division do
  const float a = __uint_as_float(w << 16), b = __uint_as_float(w & 0xffff0000u);
  return pack_bf16(__fdividef(a, 1.0f + __expf(-a)), __fdividef(b, 1.0f + __expf(-b)));
}

// N values of each of the chunk's `len` rows from src (row pitch ld) to dst [LC][N + 8]; zeros beyond the chunk's end.
template <int N>
__device__ __forceinline__ void lm_rows(__nv_bfloat16* dst, const __nv_bfloat16* __restrict__ src, int ld, int len, bool silu) {
  for (int i = threadIdx.x; i < LC * (N / 8); i += blockDim.x) {
    const int t = i / (N / 8), c = i % (N / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (t < len) {
      v = *reinterpret_cast<const uint4*>(src + (size_t)t * ld + c * 8);
      if (silu) v = make_uint4(silu_pair(v.x), silu_pair(v.y), silu_pair(v.z), silu_pair(v.w));
    }
    *reinterpret_cast<uint4*>(dst + t * (N + 8) + c * 8) = v;
  }
}

// Sum of squares of N values of a shared-memory row, two threads per row (row = threadIdx.x / 2): both get the row's sum.
template <int N>
__device__ __forceinline__ float lm_row_squares(const __nv_bfloat16* rows) {
  const int t = threadIdx.x >> 1, half = threadIdx.x & 1;
  float ss = 0.f;
  for (int d = half * (N / 2); d < (half + 1) * (N / 2); ++d) {
    const float v = __bfloat162float(rows[t * (N + 8) + d]);
    ss = fmaf(v, v, ss);
  }
  return ss + __shfl_xor_sync(0xffffffffu, ss, 1);
}

struct MemoryMma {
  const __nv_bfloat16* x;  // [T, ld]: q, k (G heads of D), v (H heads of Dv) at columns
  int ld, q_col, k_col, v_col;
  const __nv_bfloat16* gates;  // delta: [T, ldg] with b and a (H each) at columns
  int ldg, b_col, a_col;
  const float *A_log, *dt_bias;  // delta [H]
  const float* log_decay;        // decayed [H]
  float q_scale;
  int silu;
  int H, G, Dv, num_slots;
  const int *q_start, *slot_ids;
  float* state;    // [slots, H, Dv, D]
  float* records;  // per chunk [H, Dv, D]: chunk j of request b is record q_start[b] / LC + b + j
  // delta: per token and head
  __nv_bfloat16 *w_hi, *w_lo;  // [T, H, D]
  float* u;                    // [T, H, Dv]: U0, then U
  float* scal;                 // [T, H, 2]: b_t, 1 / |k_t|
  float* out;                  // [T, H, Dv]
  int* status;
};

// ---------------------------------------------------------------- decayed: the state a chunk reaches from zero
// grid (requests, chunks, H * Dv / P): P value rows of one head.
template <int D, int P>
__global__ void __launch_bounds__(LMM_THREADS)
memory_chunk_state_kernel(MemoryMma in) {
  constexpr int PN = D + 8, PX = P + 8;
  constexpr int MT = P / 16, WN = 4 / MT, NT = D / 8 / WN;  // row tiles; column groups of the warps; column tiles per warp
  extern __shared__ __align__(16) unsigned char lmm_smem[];
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(lmm_smem);  // [LC][PN]
  __nv_bfloat16* v_hi = ks + LC * PN;                              // [LC][PX]: the weighted values
  __nv_bfloat16* v_lo = v_hi + LC * PX;
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x, tiles = in.Dv / P, h = blockIdx.z / tiles, p0 = (blockIdx.z % tiles) * P;
  const int slot = in.slot_ids[b];
  const int start = in.q_start[b], t0 = start + blockIdx.y * LC, t1 = in.q_start[b + 1];
  if (t0 >= t1 || slot < 0 || slot >= in.num_slots) return;
  const int len = min(LC, t1 - t0), hk = h / (in.H / in.G);
  lm_rows<D>(ks, in.x + (size_t)t0 * in.ld + in.k_col + hk * D, in.ld, len, in.silu);
  const float lg = in.log_decay[h];
  for (int i = threadIdx.x; i < LC * (P / 2); i += blockDim.x) {
    const int t = i / (P / 2), c = (i % (P / 2)) * 2;
    uint32_t hi = 0, lo = 0;
    if (t < len) {
      uint32_t raw = *reinterpret_cast<const uint32_t*>(in.x + (size_t)(t0 + t) * in.ld + in.v_col + h * in.Dv + p0 + c);
      if (in.silu) raw = silu_pair(raw);
      const int n = len - 1 - t;
      const float w = n == 0 ? 1.f : __expf(lg * (float)n);
      lm_split_pack(w * __uint_as_float(raw << 16), w * __uint_as_float(raw & 0xffff0000u), hi, lo);
    }
    *reinterpret_cast<uint32_t*>(v_hi + t * PX + c) = hi;
    *reinterpret_cast<uint32_t*>(v_lo + t * PX + c) = lo;
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tid4 = lane & 3;
  const int prow = (warp % MT) * 16, n0 = (warp / MT) * (D / WN);
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < LC / 16; ++kk) {
    uint32_t ah[4], al[4];  // A[p][s]: the stored [s][p] tile, transposed on the way
    const int at = (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * PX + prow + ((lane >> 3) & 1) * 8;
    ldmatrix_x4_trans(ah, v_hi + at);
    ldmatrix_x4_trans(al, v_lo + at);
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      uint32_t kb[4];
      ldmatrix_x4_trans(kb, ks + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PN + n0 + np * 16 + (lane >> 4) * 8);
      mma_bf16(acc[2 * np], ah, kb[0], kb[1]);
      mma_bf16(acc[2 * np + 1], ah, kb[2], kb[3]);
      mma_bf16(acc[2 * np], al, kb[0], kb[1]);
      mma_bf16(acc[2 * np + 1], al, kb[2], kb[3]);
    }
  }
  float* rec = in.records + (size_t)(start / LC + b + blockIdx.y) * in.H * in.Dv * D + ((size_t)h * in.Dv + p0) * D;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r)
      *reinterpret_cast<float2*>(rec + (size_t)(prow + gid + 8 * r) * D + n0 + i * 8 + 2 * tid4) =
          make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
}

// grid (requests, H * Dv * D / 1024): four state values a thread.  The records' "reached from zero" become "the state the
// chunk starts from", the last state goes to the slot.
__global__ void memory_chunk_carry_kernel(MemoryMma in, int D) {
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x;
  const size_t all = (size_t)in.H * in.Dv * D, e = ((size_t)blockIdx.y * blockDim.x + threadIdx.x) * 4;
  const int slot = in.slot_ids[b];
  if (e >= all || slot < 0 || slot >= in.num_slots) return;
  const int t0 = in.q_start[b], total = in.q_start[b + 1] - t0, chunks = (total + LC - 1) / LC;
  if (chunks <= 0) return;
  const float lg = in.log_decay[(int)(e / ((size_t)in.Dv * D))];
  const float whole = __expf(lg * (float)LC), tail = __expf(lg * (float)(total - (chunks - 1) * LC));
  float4 S = *reinterpret_cast<const float4*>(in.state + (size_t)slot * all + e);
  float* rec = in.records + (size_t)(t0 / LC + b) * all + e;
  constexpr int AHEAD = 8;  // chunks whose loads are in flight together
  for (int j0 = 0; j0 < chunks; j0 += AHEAD, rec += AHEAD * all) {
    float4 reached[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
      if (j0 + k < chunks) reached[k] = *reinterpret_cast<const float4*>(rec + (size_t)k * all);
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
      if (j0 + k < chunks) {
        *reinterpret_cast<float4*>(rec + (size_t)k * all) = S;
        const float g = j0 + k == chunks - 1 ? tail : whole;
        S.x = fmaf(g, S.x, reached[k].x);
        S.y = fmaf(g, S.y, reached[k].y);
        S.z = fmaf(g, S.z, reached[k].z);
        S.w = fmaf(g, S.w, reached[k].w);
      }
  }
  *reinterpret_cast<float4*>(in.state + (size_t)slot * all + e) = S;
}

// ---------------------------------------------------------------- both: what a chunk's tokens read
// grid (requests, chunks, H): warp w owns the chunk's tokens 16 w .. 16 w + 15; the values in tiles of P.
template <int D, int P, bool DELTA>
__global__ void __launch_bounds__(LMM_THREADS)
memory_chunk_output_kernel(MemoryMma in) {
  constexpr int PN = D + 8, PX = P + 8;
  extern __shared__ __align__(16) unsigned char lmm_smem[];
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(lmm_smem);  // [LC][PN]
  __nv_bfloat16* ks = qs + LC * PN;                                // [LC][PN]
  __nv_bfloat16* s_hi = ks + LC * PN;                              // [P][PN]
  __nv_bfloat16* s_lo = s_hi + P * PN;                             // [P][PN]
  __nv_bfloat16* vs = s_lo + P * PN;                               // [LC][PX]
  __nv_bfloat16* v_lo = vs + LC * PX;                              // [LC][PX], delta only
  float* b_s = reinterpret_cast<float*>(v_lo + (DELTA ? LC * PX : 0));  // [LC]
  float* rk_s = b_s + LC;                                               // [LC], delta only
  float* rq_s = rk_s + LC;
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x, h = blockIdx.z, H = in.H, Dv = in.Dv;
  const int slot = in.slot_ids[b];
  const int start = in.q_start[b], t0 = start + blockIdx.y * LC, t1 = in.q_start[b + 1];
  if (t0 >= t1) return;
  const int len = min(LC, t1 - t0), hk = h / (H / in.G);
  if (slot < 0 || slot >= in.num_slots) {
    if (threadIdx.x == 0) atomicOr(in.status, Q3_STATUS_BAD_POSITION);
    for (int i = threadIdx.x; i < len * Dv; i += blockDim.x) in.out[((size_t)(t0 + i / Dv) * H + h) * Dv + i % Dv] = 0.f;
    return;
  }
  lm_rows<D>(qs, in.x + (size_t)t0 * in.ld + in.q_col + hk * D, in.ld, len, in.silu);
  lm_rows<D>(ks, in.x + (size_t)t0 * in.ld + in.k_col + hk * D, in.ld, len, in.silu);
  const float lg = DELTA ? 0.f : in.log_decay[h];
  if (threadIdx.x < LC) {
    const int t = threadIdx.x;
    if (DELTA) {
      const float* sc = in.scal + ((size_t)(t0 + min(t, len - 1)) * H + h) * 2;
      b_s[t] = sc[0];
      rk_s[t] = sc[1];
    } else {
      b_s[t] = lg * (float)(t + 1);
    }
  }
  __syncthreads();
  if (DELTA) {
    const float ss = lm_row_squares<D>(qs);
    if ((threadIdx.x & 1) == 0) rq_s[threadIdx.x >> 1] = 1.0f / sqrtf(ss + 1e-6f);
    __syncthreads();
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tid4 = lane & 3;
  uint32_t qf[D / 16][4];  // this warp's rows of q as A fragments, for q k^T and for q S_in
#pragma unroll
  for (int kk = 0; kk < D / 16; ++kk) ldmatrix_x4(qf[kk], qs + (warp * 16 + (lane & 15)) * PN + kk * 16 + (lane >> 4) * 8);
  uint32_t m_hi[LC / 16][4], m_lo[LC / 16][4];
  const int tr[2] = {warp * 16 + gid, warp * 16 + gid + 8};
  {
    float g[LC / 8][4];
#pragma unroll
    for (int i = 0; i < LC / 8; ++i) g[i][0] = g[i][1] = g[i][2] = g[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk)
#pragma unroll
      for (int np = 0; np < LC / 16; ++np) {
        uint32_t kb[4];
        ldmatrix_x4(kb, ks + (np * 16 + (lane & 7) + ((lane >> 4) << 3)) * PN + kk * 16 + ((lane >> 3) & 1) * 8);
        mma_bf16(g[2 * np], qf[kk], kb[0], kb[1]);
        mma_bf16(g[2 * np + 1], qf[kk], kb[2], kb[3]);
      }
    // g[t][s] e^{b_t - b_s} for s <= t, in two halves, as A fragments
#pragma unroll
    for (int nt = 0; nt < LC / 8; ++nt) {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float m[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int s = nt * 8 + 2 * tid4 + j;
          float w;
          if (DELTA)
            w = __expf(b_s[tr[r]] - b_s[s]) * rk_s[s];
          else
            w = tr[r] == s ? 1.f : __expf(lg * (float)(tr[r] - s));
          m[j] = s <= tr[r] ? g[nt][2 * r + j] * w : 0.f;
        }
        const int reg = (nt & 1) * 2 + r;  // column tile 2 kk fills registers 0, 1 of step kk; 2 kk + 1 fills 2, 3
        lm_split_pack(m[0], m[1], m_hi[nt >> 1][reg], m_lo[nt >> 1][reg]);
      }
    }
  }
  const float* rec = in.records + (size_t)(start / LC + b + blockIdx.y) * H * Dv * D + (size_t)h * Dv * D;
  for (int p0 = 0; p0 < Dv; p0 += P) {
    __syncthreads();  // the tile before has been read
    for (int i = threadIdx.x; i < P * D / 4; i += blockDim.x) {
      const float4 v = *reinterpret_cast<const float4*>(rec + (size_t)p0 * D + 4 * i);
      const int p = (4 * i) / D, n = (4 * i) % D;
      uint2 hi, lo;
      lm_split_pack(v.x, v.y, hi.x, lo.x);
      lm_split_pack(v.z, v.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(s_hi + p * PN + n) = hi;
      *reinterpret_cast<uint2*>(s_lo + p * PN + n) = lo;
    }
    if (DELTA) {
      for (int i = threadIdx.x; i < LC * P / 4; i += blockDim.x) {
        const int t = (4 * i) / P, c = (4 * i) % P;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (t < len) v = *reinterpret_cast<const float4*>(in.u + ((size_t)(t0 + t) * H + h) * Dv + p0 + c);
        uint2 hi, lo;
        lm_split_pack(v.x, v.y, hi.x, lo.x);
        lm_split_pack(v.z, v.w, hi.y, lo.y);
        *reinterpret_cast<uint2*>(vs + t * PX + c) = hi;
        *reinterpret_cast<uint2*>(v_lo + t * PX + c) = lo;
      }
    } else {
      lm_rows<P>(vs, in.x + (size_t)t0 * in.ld + in.v_col + h * Dv + p0, in.ld, len, in.silu);
    }
    __syncthreads();
    float acc[P / 8][4], z[P / 8][4];
#pragma unroll
    for (int i = 0; i < P / 8; ++i) {
      acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
      z[i][0] = z[i][1] = z[i][2] = z[i][3] = 0.f;
    }
#pragma unroll
    for (int kk = 0; kk < LC / 16; ++kk)
#pragma unroll
      for (int dt = 0; dt < P / 16; ++dt) {
        const int at = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PX + dt * 16 + (lane >> 4) * 8;
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, vs + at);
        mma_bf16(acc[2 * dt], m_hi[kk], vb[0], vb[1]);
        mma_bf16(acc[2 * dt + 1], m_hi[kk], vb[2], vb[3]);
        mma_bf16(acc[2 * dt], m_lo[kk], vb[0], vb[1]);
        mma_bf16(acc[2 * dt + 1], m_lo[kk], vb[2], vb[3]);
        if (DELTA) {
          ldmatrix_x4_trans(vb, v_lo + at);
          mma_bf16(acc[2 * dt], m_hi[kk], vb[0], vb[1]);
          mma_bf16(acc[2 * dt + 1], m_hi[kk], vb[2], vb[3]);
        }
      }
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk)
#pragma unroll
      for (int dt = 0; dt < P / 16; ++dt) {
        const int at = (dt * 16 + (lane & 7) + ((lane >> 4) << 3)) * PN + kk * 16 + ((lane >> 3) & 1) * 8;
        uint32_t hb[4], lb[4];
        ldmatrix_x4(hb, s_hi + at);
        ldmatrix_x4(lb, s_lo + at);
        mma_bf16(z[2 * dt], qf[kk], hb[0], hb[1]);
        mma_bf16(z[2 * dt + 1], qf[kk], hb[2], hb[3]);
        mma_bf16(z[2 * dt], qf[kk], lb[0], lb[1]);
        mma_bf16(z[2 * dt + 1], qf[kk], lb[2], lb[3]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (tr[r] >= len) continue;
      const float e = __expf(b_s[tr[r]]);
      const float f = in.q_scale * (DELTA ? rq_s[tr[r]] : 1.f);
      float* dst = in.out + ((size_t)(t0 + tr[r]) * H + h) * Dv + p0;
#pragma unroll
      for (int i = 0; i < P / 8; ++i)
        *reinterpret_cast<float2*>(dst + i * 8 + 2 * tid4) =
            make_float2(f * fmaf(e, z[i][2 * r], acc[i][2 * r]), f * fmaf(e, z[i][2 * r + 1], acc[i][2 * r + 1]));
    }
  }
}

// ---------------------------------------------------------------- delta: Tm, W and U0 of a chunk
constexpr int TMP = LC + 1;  // pitch of the triangular matrices

// out[i][j] (rows r0.., columns c0.., n x n) = sign * sum_{k < n} L[i][k] R[k][j], L at rows/columns (lr, lc), R at (rr, rc).
__device__ __forceinline__ void tri_block(float* out, int r0, int c0, const float* L, int lr, int lc, const float* R, int rr, int rc,
                                          int n, float sign, int first, int step) {
  for (int e = first; e < n * n; e += step) {
    const int i = e / n, j = e % n;
    float acc = 0.f;
    for (int k = 0; k < n; ++k) acc = fmaf(L[(lr + i) * TMP + lc + k], R[(rr + k) * TMP + rc + j], acc);
    out[(r0 + i) * TMP + c0 + j] = sign * acc;
  }
}

// grid (requests, chunks, H), 128 threads.
template <int D, int P>
__global__ void __launch_bounds__(LMM_THREADS)
delta_chunk_prepare_kernel(MemoryMma in) {
  constexpr int PN = D + 8, PX = P + 8;
  extern __shared__ __align__(16) unsigned char lmm_smem[];
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(lmm_smem);  // [LC][PN]
  __nv_bfloat16* vs = ks + LC * PN;                                // [LC][PX]
  float* A = reinterpret_cast<float*>(vs + LC * PX);               // [LC][TMP]
  float* Tm = A + LC * TMP;                                        // [LC][TMP]
  float* X = Tm + LC * TMP;                                        // [32][TMP]: products on the way
  float* b_s = X + 32 * TMP;                                       // [LC] each
  float* rk_s = b_s + LC;
  float* be_s = rk_s + LC;
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x, h = blockIdx.z, H = in.H, Dv = in.Dv;
  const int slot = in.slot_ids[b];
  const int t0 = in.q_start[b] + blockIdx.y * LC, t1 = in.q_start[b + 1];
  if (t0 >= t1 || slot < 0 || slot >= in.num_slots) return;
  const int len = min(LC, t1 - t0), hk = h / (H / in.G);
  lm_rows<D>(ks, in.x + (size_t)t0 * in.ld + in.k_col + hk * D, in.ld, len, false);
  lm_rows<P>(vs, in.x + (size_t)t0 * in.ld + in.v_col + h * Dv, in.ld, len, false);
  if (threadIdx.x < LC) {
    const int t = threadIdx.x;
    float lg = 0.f, beta = 0.f;
    if (t < len) {
      const __nv_bfloat16* row = in.gates + (size_t)(t0 + t) * in.ldg;
      lg = -expf(in.A_log[h]) * softplus_f(__bfloat162float(row[in.a_col + h]) + in.dt_bias[h]);
      beta = sigmoid_f(__bfloat162float(row[in.b_col + h]));
    }
    // the inclusive sums of the log-decays: within each warp, then the first warp's total on the second
    const int l = t & 31;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, lg, o);
      if (l >= o) lg += up;
    }
    b_s[t] = lg;
    be_s[t] = beta;
  }
  for (int i = threadIdx.x; i < LC * TMP; i += blockDim.x) Tm[i] = 0.f;
  __syncthreads();
  {
    const float first = b_s[31];
    const float ss = lm_row_squares<D>(ks);
    __syncthreads();
    if ((threadIdx.x & 1) == 0) rk_s[threadIdx.x >> 1] = 1.0f / sqrtf(ss + 1e-6f);
    if (threadIdx.x >= 32 && threadIdx.x < LC) b_s[threadIdx.x] += first;
  }
  __syncthreads();
  if (threadIdx.x < len) {
    float* sc = in.scal + ((size_t)(t0 + threadIdx.x) * H + h) * 2;
    sc[0] = b_s[threadIdx.x];
    sc[1] = rk_s[threadIdx.x];
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tid4 = lane & 3;
  const int tr[2] = {warp * 16 + gid, warp * 16 + gid + 8};
  {
    float g[LC / 8][4];
#pragma unroll
    for (int i = 0; i < LC / 8; ++i) g[i][0] = g[i][1] = g[i][2] = g[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t kf[4];
      ldmatrix_x4(kf, ks + (warp * 16 + (lane & 15)) * PN + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int np = 0; np < LC / 16; ++np) {
        uint32_t kb[4];
        ldmatrix_x4(kb, ks + (np * 16 + (lane & 7) + ((lane >> 4) << 3)) * PN + kk * 16 + ((lane >> 3) & 1) * 8);
        mma_bf16(g[2 * np], kf, kb[0], kb[1]);
        mma_bf16(g[2 * np + 1], kf, kb[2], kb[3]);
      }
    }
#pragma unroll
    for (int nt = 0; nt < LC / 8; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = tr[j >> 1], s = nt * 8 + 2 * tid4 + (j & 1);
        A[t * TMP + s] = s < t ? be_s[t] * rk_s[t] * rk_s[s] * __expf(b_s[t] - b_s[s]) * g[nt][j] : 0.f;
      }
  }
  __syncthreads();
  // (I + A)^-1: the four 16 x 16 blocks of the diagonal by substitution, a column per thread; then pairs of blocks by
  // [[T1, 0], [-T2 A21 T1, T2]], to 32 and to 64
  if (threadIdx.x < LC) {
    const int base = threadIdx.x & ~15, j = threadIdx.x & 15;
    float col[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float acc = i == j ? 1.f : 0.f;
#pragma unroll
      for (int s = 0; s < i; ++s) acc = fmaf(-A[(base + i) * TMP + base + s], col[s], acc);
      col[i] = acc;  // zero above the diagonal: nothing but zeros has been summed
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) Tm[(base + i) * TMP + base + j] = col[i];
  }
  __syncthreads();
  {
    const int pair = threadIdx.x >> 6, r = pair * 32, at = threadIdx.x & 63;  // two pairs of 16-blocks, 64 threads each
    tri_block(X, pair * 16, 0, A, r + 16, r, Tm, r, r, 16, 1.f, at, 64);
    __syncthreads();
    tri_block(Tm, r + 16, r, Tm, r + 16, r + 16, X, pair * 16, 0, 16, -1.f, at, 64);
  }
  __syncthreads();
  tri_block(X, 0, 0, A, 32, 0, Tm, 0, 0, 32, 1.f, threadIdx.x, LMM_THREADS);
  __syncthreads();
  tri_block(Tm, 32, 0, Tm, 32, 32, X, 0, 0, 32, -1.f, threadIdx.x, LMM_THREADS);
  __syncthreads();
  // W = Tm diag(beta e^b / |k|) K, then U0 = Tm diag(beta) V: the factors on the columns of Tm, in two halves
#pragma unroll
  for (int which = 0; which < 2; ++which) {
    uint32_t hi[LC / 16][4], lo[LC / 16][4];
#pragma unroll
    for (int kk = 0; kk < LC / 16; ++kk)
#pragma unroll
      for (int reg = 0; reg < 4; ++reg) {
        const int t = tr[reg & 1], s = kk * 16 + (reg >> 1) * 8 + 2 * tid4;
        float f[2];
#pragma unroll
        for (int j = 0; j < 2; ++j)
          f[j] = Tm[t * TMP + s + j] * be_s[s + j] * (which == 0 ? rk_s[s + j] * __expf(b_s[s + j]) : 1.f);
        lm_split_pack(f[0], f[1], hi[kk][reg], lo[kk][reg]);
      }
    if (which == 0) {
      for (int n0 = 0; n0 < D; n0 += 64) {
        float acc[8][4];
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < LC / 16; ++kk)
#pragma unroll
          for (int dt = 0; dt < 4; ++dt) {
            uint32_t kb[4];
            ldmatrix_x4_trans(kb, ks + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PN + n0 + dt * 16 + (lane >> 4) * 8);
            mma_bf16(acc[2 * dt], hi[kk], kb[0], kb[1]);
            mma_bf16(acc[2 * dt + 1], hi[kk], kb[2], kb[3]);
            mma_bf16(acc[2 * dt], lo[kk], kb[0], kb[1]);
            mma_bf16(acc[2 * dt + 1], lo[kk], kb[2], kb[3]);
          }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          if (tr[r] >= len) continue;
          const size_t at = ((size_t)(t0 + tr[r]) * H + h) * D + n0 + 2 * tid4;
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            uint32_t ph, pl;
            lm_split_pack(acc[i][2 * r], acc[i][2 * r + 1], ph, pl);
            *reinterpret_cast<uint32_t*>(in.w_hi + at + i * 8) = ph;
            *reinterpret_cast<uint32_t*>(in.w_lo + at + i * 8) = pl;
          }
        }
      }
    } else {
      for (int p0 = 0; p0 < Dv; p0 += P) {
        if (p0 > 0) {
          __syncthreads();
          lm_rows<P>(vs, in.x + (size_t)t0 * in.ld + in.v_col + h * Dv + p0, in.ld, len, false);
          __syncthreads();
        }
        float acc[P / 8][4];
#pragma unroll
        for (int i = 0; i < P / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < LC / 16; ++kk)
#pragma unroll
          for (int dt = 0; dt < P / 16; ++dt) {
            uint32_t vb[4];
            ldmatrix_x4_trans(vb, vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PX + dt * 16 + (lane >> 4) * 8);
            mma_bf16(acc[2 * dt], hi[kk], vb[0], vb[1]);
            mma_bf16(acc[2 * dt + 1], hi[kk], vb[2], vb[3]);
            mma_bf16(acc[2 * dt], lo[kk], vb[0], vb[1]);
            mma_bf16(acc[2 * dt + 1], lo[kk], vb[2], vb[3]);
          }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          if (tr[r] >= len) continue;
          float* dst = in.u + ((size_t)(t0 + tr[r]) * H + h) * Dv + p0 + 2 * tid4;
#pragma unroll
          for (int i = 0; i < P / 8; ++i)
            *reinterpret_cast<float2*>(dst + i * 8) = make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
        }
      }
    }
  }
}

// ---------------------------------------------------------------- delta: chunk after chunk
// grid (Dv / 32, H, requests), two warps: a warp owns 16 value columns, S^T [16, D] in its accumulators.  A chunk's W, K and
// U0 are fetched while the chunk before is worked on.
constexpr int DW_WARPS = 2, DW_COLS = 16 * DW_WARPS, DW_UP = DW_COLS + 4;  // pitch of U0's rows in shared memory

template <int D>
__global__ void __launch_bounds__(32 * DW_WARPS)
delta_chunk_walk_kernel(MemoryMma in) {
  constexpr int PN = D + 8, THREADS = 32 * DW_WARPS;
  constexpr int STAGE = 3 * LC * PN * 2 + LC * DW_UP * 4 + 2 * LC * 4;  // bytes: W hi, W lo, K, U0, scalars
  extern __shared__ __align__(16) unsigned char lmm_smem[];
  float* f_s = reinterpret_cast<float*>(lmm_smem + 2 * STAGE);  // [LC]: e^{b_last - b_s} / |k_s|
  const int b = blockIdx.z, h = blockIdx.y, H = in.H, Dv = in.Dv, p0 = blockIdx.x * DW_COLS;
  const int slot = in.slot_ids[b];
  const int start = in.q_start[b], t1 = in.q_start[b + 1];
  pdl_wait();
  pdl_launch_dependents();
  if (slot < 0 || slot >= in.num_slots || start >= t1) return;  // the output kernel writes zeros for a bad slot
  const int hk = h / (H / in.G);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tid4 = lane & 3;

  auto fetch = [&](int t0, int stage) {
    unsigned char* base = lmm_smem + stage * STAGE;
    __nv_bfloat16* wh = reinterpret_cast<__nv_bfloat16*>(base);
    __nv_bfloat16 *wl = wh + LC * PN, *kk = wl + LC * PN;
    float* u0 = reinterpret_cast<float*>(kk + LC * PN);
    float* sc = u0 + LC * DW_UP;
    const int len = min(LC, t1 - t0);
    for (int i = threadIdx.x; i < LC * (D / 8); i += THREADS) {
      const int t = i / (D / 8), c = (i % (D / 8)) * 8;
      const int tt = min(t, len - 1), bytes = t < len ? 16 : 0;
      const size_t at = ((size_t)(t0 + tt) * H + h) * D + c;
      cp_async_16(wh + t * PN + c, in.w_hi + at, bytes);
      cp_async_16(wl + t * PN + c, in.w_lo + at, bytes);
      cp_async_16(kk + t * PN + c, in.x + (size_t)(t0 + tt) * in.ld + in.k_col + hk * D + c, bytes);
    }
    for (int i = threadIdx.x; i < LC * (DW_COLS / 4); i += THREADS) {
      const int t = i / (DW_COLS / 4), c = (i % (DW_COLS / 4)) * 4;
      cp_async_16(u0 + t * DW_UP + c, in.u + ((size_t)(t0 + min(t, len - 1)) * H + h) * Dv + p0 + c, t < len ? 16 : 0);
    }
    // the scalars: plain loads, 8 bytes a token, in flight with the rest until the barrier
    for (int t = threadIdx.x; t < LC; t += THREADS)
      *reinterpret_cast<float2*>(sc + 2 * t) =
          *reinterpret_cast<const float2*>(in.scal + ((size_t)(t0 + min(t, len - 1)) * H + h) * 2);
    cp_async_commit();
  };

  const int col = p0 + warp * 16 + gid;  // this thread's value columns: col and col + 8
  float* st = in.state + ((size_t)slot * H + h) * (size_t)Dv * D;
  float S[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const float2 v = *reinterpret_cast<const float2*>(st + (size_t)(col + 8 * r) * D + i * 8 + 2 * tid4);
      S[i][2 * r] = v.x;
      S[i][2 * r + 1] = v.y;
    }
  fetch(start, 0);
  int stage = 0;
  float* rec = in.records + (size_t)(start / LC + b) * H * Dv * D + (size_t)h * Dv * D;
  for (int t0 = start; t0 < t1; t0 += LC, stage ^= 1, rec += (size_t)H * Dv * D) {
    const int len = min(LC, t1 - t0);
    cp_async_wait<0>();
    __syncthreads();  // the chunk is there, and the other stage has been read by everybody
    if (t0 + LC < t1) fetch(t0 + LC, stage ^ 1);
    const unsigned char* base = lmm_smem + stage * STAGE;
    const __nv_bfloat16* wh = reinterpret_cast<const __nv_bfloat16*>(base);
    const __nv_bfloat16 *wl = wh + LC * PN, *kk_s = wl + LC * PN;
    const float* u0 = reinterpret_cast<const float*>(kk_s + LC * PN);
    const float* sc = u0 + LC * DW_UP;
    const float b_last = sc[2 * (len - 1)];
    for (int t = threadIdx.x; t < LC; t += THREADS) f_s[t] = t < len ? __expf(b_last - sc[2 * t]) * sc[2 * t + 1] : 0.f;
    // (W S)^T = S^T W^T: [16 columns, 64 tokens]
    float p[LC / 8][4];
#pragma unroll
    for (int i = 0; i < LC / 8; ++i) p[i][0] = p[i][1] = p[i][2] = p[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t sh[4], sl[4];
      lm_split_pack(S[2 * kk][0], S[2 * kk][1], sh[0], sl[0]);
      lm_split_pack(S[2 * kk][2], S[2 * kk][3], sh[1], sl[1]);
      lm_split_pack(S[2 * kk + 1][0], S[2 * kk + 1][1], sh[2], sl[2]);
      lm_split_pack(S[2 * kk + 1][2], S[2 * kk + 1][3], sh[3], sl[3]);
#pragma unroll
      for (int np = 0; np < LC / 16; ++np) {
        const int at = (np * 16 + (lane & 7) + ((lane >> 4) << 3)) * PN + kk * 16 + ((lane >> 3) & 1) * 8;
        uint32_t hb[4], lb[4];
        ldmatrix_x4(hb, wh + at);
        ldmatrix_x4(lb, wl + at);
        mma_bf16(p[2 * np], sh, hb[0], hb[1]);
        mma_bf16(p[2 * np + 1], sh, hb[2], hb[3]);
        mma_bf16(p[2 * np], sl, hb[0], hb[1]);
        mma_bf16(p[2 * np + 1], sl, hb[2], hb[3]);
        mma_bf16(p[2 * np], sh, lb[0], lb[1]);
        mma_bf16(p[2 * np + 1], sh, lb[2], lb[3]);
      }
    }
    // the state the chunk starts from, for the output kernel
#pragma unroll
    for (int i = 0; i < D / 8; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r)
        *reinterpret_cast<float2*>(rec + (size_t)(col + 8 * r) * D + i * 8 + 2 * tid4) = make_float2(S[i][2 * r], S[i][2 * r + 1]);
    __syncthreads();  // f_s
    const float keep = __expf(b_last);
#pragma unroll
    for (int i = 0; i < D / 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) S[i][j] *= keep;
#pragma unroll
    for (int nt = 0; nt < LC / 8; ++nt) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = nt * 8 + 2 * tid4 + (j & 1), c = warp * 16 + gid + 8 * (j >> 1);
        const float u = u0[t * DW_UP + c] - p[nt][j];
        if (t < len) in.u[((size_t)(t0 + t) * H + h) * Dv + p0 + c] = u;
        p[nt][j] = u * f_s[t];
      }
    }
    // S^T += (diag(f) U)^T K
#pragma unroll
    for (int kk = 0; kk < LC / 16; ++kk) {
      uint32_t uh[4], ul[4];
      lm_split_pack(p[2 * kk][0], p[2 * kk][1], uh[0], ul[0]);
      lm_split_pack(p[2 * kk][2], p[2 * kk][3], uh[1], ul[1]);
      lm_split_pack(p[2 * kk + 1][0], p[2 * kk + 1][1], uh[2], ul[2]);
      lm_split_pack(p[2 * kk + 1][2], p[2 * kk + 1][3], uh[3], ul[3]);
#pragma unroll
      for (int np = 0; np < D / 16; ++np) {
        uint32_t kb[4];
        ldmatrix_x4_trans(kb, kk_s + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PN + np * 16 + (lane >> 4) * 8);
        mma_bf16(S[2 * np], uh, kb[0], kb[1]);
        mma_bf16(S[2 * np + 1], uh, kb[2], kb[3]);
        mma_bf16(S[2 * np], ul, kb[0], kb[1]);
        mma_bf16(S[2 * np + 1], ul, kb[2], kb[3]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < D / 8; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r)
      *reinterpret_cast<float2*>(st + (size_t)(col + 8 * r) * D + i * 8 + 2 * tid4) = make_float2(S[i][2 * r], S[i][2 * r + 1]);
}

template <typename K>
static int lmm_configure(K kernel, size_t smem, bool& done) {
  if (done) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  done = true;
  return 0;
}

template <int D, int P>
static int memory_mma_launch(const MemoryMma& in, bool delta, int B, int max_q_len, cudaStream_t stream) {
  constexpr int PN = D + 8, PX = P + 8;
  constexpr size_t bf = sizeof(__nv_bfloat16);
  constexpr size_t smem_state = bf * (LC * PN + 2 * LC * PX);
  constexpr size_t smem_out = bf * (2 * LC * PN + 2 * P * PN + LC * PX) + 3 * LC * sizeof(float);
  constexpr size_t smem_out_delta = smem_out + bf * LC * PX;
  constexpr size_t smem_prep = bf * (LC * PN + LC * PX) + sizeof(float) * (2 * LC * TMP + 32 * TMP + 3 * LC);
  constexpr size_t smem_walk = 2 * (size_t)(3 * LC * PN * 2 + LC * DW_UP * 4 + 2 * LC * 4) + LC * sizeof(float);
  static bool c0 = false, c1 = false, c2 = false, c3 = false, c4 = false;
  const int chunks = (max_q_len + LC - 1) / LC;
  if (chunks > 65535 || in.H * (in.Dv / P) > 65535 || B > 65535) return Q3_ERR_SIZE;
  int code;
  if (delta) {
    if ((code = lmm_configure(delta_chunk_prepare_kernel<D, P>, smem_prep, c0))) return code;
    if ((code = lmm_configure(delta_chunk_walk_kernel<D>, smem_walk, c1))) return code;
    if ((code = lmm_configure(memory_chunk_output_kernel<D, P, true>, smem_out_delta, c2))) return code;
    launch(delta_chunk_prepare_kernel<D, P>, dim3(B, chunks, in.H), dim3(LMM_THREADS), smem_prep, stream, in);
    launch(delta_chunk_walk_kernel<D>, dim3(in.Dv / DW_COLS, in.H, B), dim3(32 * DW_WARPS), smem_walk, stream, in);
    launch(memory_chunk_output_kernel<D, P, true>, dim3(B, chunks, in.H), dim3(LMM_THREADS), smem_out_delta, stream, in);
    return launch_status();
  }
  if ((code = lmm_configure(memory_chunk_state_kernel<D, P>, smem_state, c3))) return code;
  if ((code = lmm_configure(memory_chunk_output_kernel<D, P, false>, smem_out, c4))) return code;
  const size_t all = (size_t)in.H * in.Dv * D;
  launch(memory_chunk_state_kernel<D, P>, dim3(B, chunks, in.H * (in.Dv / P)), dim3(LMM_THREADS), smem_state, stream, in);
  launch(memory_chunk_carry_kernel, dim3(B, (unsigned)((all / 4 + 255) / 256)), dim3(256), 0, stream, in, D);
  launch(memory_chunk_output_kernel<D, P, false>, dim3(B, chunks, in.H), dim3(LMM_THREADS), smem_out, stream, in);
  return launch_status();
}

}  // namespace q3

// Tokens per chunk of the matrix form.
extern "C" int q3_memory_chunk() { return q3::LC; }

// 1 if the matrix form takes keys of D and values of Dv values.
extern "C" int q3_memory_mma_takes(int D, int Dv) { return (D == 64 || D == 128) && Dv > 0 && Dv % 32 == 0 ? 1 : 0; }

// The arguments of q3_memory_scan (bfloat16) with log_decay (float32 [H]: the decays' logarithms) instead of the decays.
// records: float32, T / 64 + B + 1 records of H * Dv * D; the delta rule also takes w (bfloat16, 2 * T * H * D), u (float32
// [T, H, Dv]) and scal (float32 [T, H, 2]).
extern "C" int q3_memory_scan_mma(const void* x, int ld, int q_col, int k_col, int v_col, const void* gates, int ldg, int b_col,
                                  int a_col, const float* A_log, const float* dt_bias, const float* log_decay, float q_scale,
                                  int act, float* state, const int* q_start, const int* slot_ids, int num_slots, float* out,
                                  float* records, void* w, float* u, float* scal, int T, int B, int max_q_len, int H, int G,
                                  int D, int Dv, int* status, cudaStream_t stream) {
  if (B <= 0 || T <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || !q3_memory_mma_takes(D, Dv) || num_slots <= 0 || !records ||
      (act != Q3_ACT_SILU && act != Q3_ACT_NONE))
    return Q3_ERR_SIZE;
  const bool delta = log_decay == nullptr;
  if (delta && (!gates || !A_log || !dt_bias || !w || !u || !scal || act != Q3_ACT_NONE)) return Q3_ERR_SIZE;
  if (ld % 8 || q_col % 8 || k_col % 8 || v_col % 8 || (uintptr_t)x % 16 || (uintptr_t)state % 16 || (uintptr_t)records % 16 ||
      (uintptr_t)out % 8 || (uintptr_t)w % 16 || (uintptr_t)u % 16 || (uintptr_t)scal % 8)
    return Q3_ERR_ALIGN;
  q3::MemoryMma in{};
  in.x = (const __nv_bfloat16*)x;
  in.ld = ld, in.q_col = q_col, in.k_col = k_col, in.v_col = v_col;
  in.gates = (const __nv_bfloat16*)gates;
  in.ldg = ldg, in.b_col = b_col, in.a_col = a_col;
  in.A_log = A_log, in.dt_bias = dt_bias, in.log_decay = log_decay;
  in.q_scale = q_scale;
  in.silu = act == Q3_ACT_SILU;
  in.H = H, in.G = G, in.Dv = Dv, in.num_slots = num_slots;
  in.q_start = q_start, in.slot_ids = slot_ids;
  in.state = state, in.records = records;
  in.w_hi = (__nv_bfloat16*)w;
  in.w_lo = in.w_hi ? in.w_hi + (size_t)T * H * D : nullptr;
  in.u = u, in.scal = scal, in.out = out, in.status = status;
  if (D == 64) {
    if (Dv % 64 == 0) return q3::memory_mma_launch<64, 64>(in, delta, B, max_q_len, stream);
    return q3::memory_mma_launch<64, 32>(in, delta, B, max_q_len, stream);
  }
  if (Dv % 64 == 0) return q3::memory_mma_launch<128, 64>(in, delta, B, max_q_len, stream);
  return q3::memory_mma_launch<128, 32>(in, delta, B, max_q_len, stream);
}
