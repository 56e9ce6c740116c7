// The gated delta rule with one decay a head, from the convolved rows to the read-out in one launch:
//   q, k -> unit vectors, x / sqrt(sum x^2 + 1e-6);  q also times dim^(-1/2)
//   g = exp(-exp(A_log[h]) * softplus(a + dt_bias[h])),  beta = sigmoid(b)
//   S' = g S + k u^T  with  u = beta (v - g S^T k);  the read-out is S'^T q
// S [dim, vdim] a head in float32, carried from token to token and from step to step (state [slots, heads, dim, vdim]).
//
// With raw rows q, k, their factors rq and rk, and P = S^T k, R = S^T q taken of the state as the token finds it:
//   u = beta (v - g rk P);   o = g rq R + (rk rq k.q) u;   S <- g S + k (rk u)
// so one pass over the state gives both sums, the read-out waits for no second pass, and the chain from token to token is one
// product, a reduction over sixteen lanes and one update.
//
// k_delta_rule walks the tokens one by one (a decode step; 32-bit rows; any size).  A block of four warps owns 32 neighbouring
// value channels (columns of S) of one (sequence, head).  Sixteen lanes share four columns, each lane keeping a sixteenth of
// their rows in registers (rows 64 ii + 4 rg + e of row group rg), so that a 16-byte read of k or q from shared memory serves
// four columns.  A token's eight sums over the lanes (P and R of four columns) are handed over by halves, eight shuffles in all,
// and P handed back by four more.  CH tokens are staged at a time: their rows wait in registers as they were loaded while the
// tokens before them are worked on.  A token's sums run in a fixed order over its own rows, whatever the step: the same bits
// whole, in pieces or token by token, alone or in a batch.  A token takes some 600 cycles, whatever the sizes: the chain.
//
// k_delta_chunk takes 16 tokens at a time (bfloat16 rows of a long step).  With G_t = g_1 .. g_t of the chunk and the state S0
// in front of it,
//   (I + A) U = rhs,   A[t][s] = beta_t (G_t / G_s) rk_t rk_s k_t.k_s  (s < t),   rhs_t = beta_t (v_t - G_t rk_t k_t^T S0)
//   o_t = G_t rq_t q_t^T S0 + sum_{s <= t} M[t][s] u_s,   M[t][s] = (G_t / G_s) rq_t rk_s q_t.k_s
//   S   = G_16 S0 + sum_s (G_16 / G_s) rk_s k_s u_s^T
// so the chain from token to token becomes one from chunk to chunk, and all but the 16 x 16 inverse T = (I + A)^-1 are products.
// They run on the tensor cores (mma.m16n8k16) without giving up float32: the rows k and q are bfloat16 as they come, exactly,
// and what is float32 (S, rhs, U, T, M) enters as a sum of three bfloat16 terms, which hold its 24 bits; sums are float32.  The
// ratios are exponentials of differences of logarithms, so nothing overflows and a decay of 0 is no special case.
//   Warps 0 .. 3 own 16 columns each and keep S^T [16 columns][dim] as the accumulators of the update; two neighbouring
//   accumulator tiles are the A operand of the next chunk's product with k and q.  Three more warps run ahead, a barrier a chunk
//   between the stages: warp 6 loads the rows of chunk j + 4, warp 4 makes chunk j + 2's norms, decays and products of rows with
//   rows, warp 5 makes T and M of chunk j + 1 and leaves them split into their terms, while chunk j is worked on.  (One warp that
//   did all three took 5,900 cycles a chunk, twice what the columns' warps take.)
#include "common.cuh"
#include <cstddef>

namespace {
constexpr int DR_WARPS = 4, DR_THREADS = 32 * DR_WARPS, DR_COLS = 8 * DR_WARPS;

template <typename TA, int DIMP, bool VEC>
__global__ void __launch_bounds__(DR_THREADS)
k_delta_rule(const TA* __restrict__ qkv, int ld, const TA* __restrict__ a, int lda, const TA* __restrict__ b, int ldb,
             const float* __restrict__ A_log, const float* __restrict__ dt_bias, float* __restrict__ state, const int* __restrict__ seq_slot,
             const int* __restrict__ seq_first_row, float* __restrict__ out, int heads, int kv_heads, int dim, int vdim, float qscale) {
  constexpr int CH = DIMP > 128 ? 8 : 16;               // tokens staged at a time
  constexpr int RP = DIMP / 16;                         // rows of its four columns that a lane keeps
  constexpr int V = VEC ? 16 / (int)sizeof(TA) : 1;     // values of one load
  constexpr int PER = DIMP / V, NLD = (CH * PER + DR_THREADS - 1) / DR_THREADS;
  constexpr int NLV = CH * DR_COLS / DR_THREADS;
  constexpr int ROW = DIMP + 4;
  constexpr int G = DR_THREADS / CH;                    // threads that sum one token's squares
  __shared__ __align__(16) float sk[CH][ROW], sq[CH][ROW];
  __shared__ __align__(16) float sv[CH][DR_COLS];
  __shared__ float so[CH][DR_COLS];
  __shared__ float4 s_mul[CH];                          // g, beta, g rk, g rq
  __shared__ float2 s_end[CH];                          // rk, rk rq k.q
  __shared__ float s_g[CH], s_b[CH];
  const int seq = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * DR_COLS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int rg = lane & 15, lc = warp * 8 + (lane >> 4) * 4;       // row group; the lane's columns are col0 + lc .. + 3
  const int kvh = h / (heads / kv_heads), kd = kv_heads * dim;
  const float rate = expf(A_log[h]), bias = dt_bias[h];
  cima_pdl_wait();
  const int first = seq_first_row[seq], n = seq_first_row[seq + 1] - first;
  float* st = state + (((size_t)seq_slot[seq] * heads + h) * dim) * (size_t)vdim + col0 + lc;
  const int cols = min(4, vdim - col0 - lc);            // columns of the lane that exist
  const bool whole = cols == 4 && vdim % 4 == 0;         // (a slot's state starts on 16 bytes then)
  float S[RP][4];
#pragma unroll
  for (int j = 0; j < RP; j++) {
    const int row = (j >> 2) * 64 + rg * 4 + (j & 3);
    S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.f;
    if (row < dim) {
      if (whole) {
        const float4 t = *reinterpret_cast<const float4*>(st + (size_t)row * vdim);
        S[j][0] = t.x; S[j][1] = t.y; S[j][2] = t.z; S[j][3] = t.w;
      } else {
#pragma unroll
        for (int c = 0; c < 4; c++)
          if (c < cols) S[j][c] = st[(size_t)row * vdim + c];
      }
    }
  }

  struct __align__(VEC ? 16 : sizeof(TA)) Piece { TA e[V]; };
  Piece rk[NLD], rq[NLD];
  TA rv[NLV];
  const TA zero = cima_from_f32<TA>(0.f);
  TA za = zero, zb = zero;
  auto fetch = [&](int t0) {
    const int nt = min(CH, n - t0);
#pragma unroll
    for (int r = 0; r < NLD; r++) {
      const int idx = threadIdx.x + r * DR_THREADS;
      const int tt = idx / PER, i = (idx - tt * PER) * V;
      if (tt < nt && i < dim) {
        const TA* p = qkv + (size_t)(first + t0 + tt) * ld + (size_t)kvh * dim + i;
        rq[r] = *reinterpret_cast<const Piece*>(p);
        rk[r] = *reinterpret_cast<const Piece*>(p + kd);
      } else {
#pragma unroll
        for (int e = 0; e < V; e++) rq[r].e[e] = rk[r].e[e] = zero;
      }
    }
#pragma unroll
    for (int r = 0; r < NLV; r++) {
      const int idx = threadIdx.x + r * DR_THREADS;
      const int tt = idx / DR_COLS, cc = idx - tt * DR_COLS;
      rv[r] = tt < nt && col0 + cc < vdim ? qkv[(size_t)(first + t0 + tt) * ld + 2 * kd + (size_t)h * vdim + col0 + cc] : zero;
    }
    if ((int)threadIdx.x < nt) {
      za = a[(size_t)(first + t0 + threadIdx.x) * lda + h];
      zb = b[(size_t)(first + t0 + threadIdx.x) * ldb + h];
    }
  };
  if (n > 0) fetch(0);

  for (int t0 = 0; t0 < n; t0 += CH) {
    const int nt = min(CH, n - t0);
#pragma unroll
    for (int r = 0; r < NLD; r++) {
      const int idx = threadIdx.x + r * DR_THREADS;
      const int tt = idx / PER, i = (idx - tt * PER) * V;
      if (tt < CH) {
        float fk[V], fq[V];
#pragma unroll
        for (int e = 0; e < V; e++) { fk[e] = cima_to_f32<TA>(rk[r].e[e]); fq[e] = cima_to_f32<TA>(rq[r].e[e]); }
        if constexpr (V >= 4) {
#pragma unroll
          for (int e = 0; e < V; e += 4) {
            *reinterpret_cast<float4*>(&sk[tt][i + e]) = make_float4(fk[e], fk[e + 1], fk[e + 2], fk[e + 3]);
            *reinterpret_cast<float4*>(&sq[tt][i + e]) = make_float4(fq[e], fq[e + 1], fq[e + 2], fq[e + 3]);
          }
        } else {
          sk[tt][i] = fk[0];
          sq[tt][i] = fq[0];
        }
      }
    }
#pragma unroll
    for (int r = 0; r < NLV; r++) {
      const int idx = threadIdx.x + r * DR_THREADS;
      sv[idx / DR_COLS][idx % DR_COLS] = cima_to_f32<TA>(rv[r]);
    }
    if (threadIdx.x < CH) {
      const float z = cima_to_f32<TA>(za) + bias;
      s_g[threadIdx.x] = expf(-rate * (z > 20.f ? z : log1pf(expf(z))));
      s_b[threadIdx.x] = 1.0f / (1.0f + expf(-cima_to_f32<TA>(zb)));
    }
    __syncthreads();
    if (t0 + CH < n) fetch(t0 + CH);
    {                                                   // a token's three sums by G threads
      const int tt = threadIdx.x / G, sub = threadIdx.x % G;
      float kk = 0.f, qq = 0.f, kq = 0.f;
#pragma unroll
      for (int i = sub; i < DIMP; i += G) {
        const float x = sk[tt][i], y = sq[tt][i];
        kk = fmaf(x, x, kk);
        qq = fmaf(y, y, qq);
        kq = fmaf(x, y, kq);
      }
#pragma unroll
      for (int o = G / 2; o > 0; o >>= 1) {
        kk += __shfl_xor_sync(0xffffffffu, kk, o);
        qq += __shfl_xor_sync(0xffffffffu, qq, o);
        kq += __shfl_xor_sync(0xffffffffu, kq, o);
      }
      if (sub == 0) {
        const float fk = 1.0f / sqrtf(kk + 1e-6f), fq = qscale / sqrtf(qq + 1e-6f), g = s_g[tt];
        s_mul[tt] = make_float4(g, s_b[tt], g * fk, g * fq);
        s_end[tt] = make_float2(fk, fk * fq * kq);
      }
    }
    __syncthreads();
#pragma unroll 2
    for (int tt = 0; tt < nt; tt++) {
      float4 k4[RP / 4];
      float x[8];                                         // P of the four columns, then R
#pragma unroll
      for (int c = 0; c < 8; c++) x[c] = 0.f;
#pragma unroll
      for (int j = 0; j < RP; j += 4) {
        k4[j >> 2] = *reinterpret_cast<const float4*>(&sk[tt][(j >> 2) * 64 + rg * 4]);
        const float4 q4 = *reinterpret_cast<const float4*>(&sq[tt][(j >> 2) * 64 + rg * 4]);
        const float kk[4] = {k4[j >> 2].x, k4[j >> 2].y, k4[j >> 2].z, k4[j >> 2].w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int e = 0; e < 4; e++)
#pragma unroll
          for (int c = 0; c < 4; c++) {
            x[c] = fmaf(S[j + e][c], kk[e], x[c]);
            x[4 + c] = fmaf(S[j + e][c], qq[e], x[4 + c]);
          }
      }
      const float4 m = s_mul[tt], v4 = *reinterpret_cast<const float4*>(&sv[tt][lc]);
      const float2 z = s_end[tt];
      // handed over by halves: lane bits 8, 4, 2 say which of the eight sums a lane ends up with
#pragma unroll
      for (int d = 8; d >= 2; d >>= 1) {
        const bool upper = lane & d;
#pragma unroll
        for (int c = 0; c < d / 2; c++) {
          const float mine = upper ? x[c + d / 2] : x[c], other = upper ? x[c] : x[c + d / 2];
          x[c] = mine + __shfl_xor_sync(0xffffffffu, other, d);
        }
      }
      const float sum = x[0] + __shfl_xor_sync(0xffffffffu, x[0], 1);
      const float v[4] = {v4.x, v4.y, v4.z, v4.w};
      float u[4];
#pragma unroll
      for (int c = 0; c < 4; c++)                         // P of column c stands in lane 2 c of the sixteen
        u[c] = m.y * (v[c] - m.z * __shfl_sync(0xffffffffu, sum, (lane & 16) + 2 * c));
      const int own = (lane >> 1) & 3;                    // R of column c stands in lane 8 + 2 c
      const float uo = own & 2 ? (own & 1 ? u[3] : u[2]) : (own & 1 ? u[1] : u[0]);
      if ((lane & 9) == 8) so[tt][lc + own] = fmaf(z.y, uo, m.w * sum);
#pragma unroll
      for (int c = 0; c < 4; c++) u[c] *= z.x;
#pragma unroll
      for (int j = 0; j < RP; j += 4) {
        const float kk[4] = {k4[j >> 2].x, k4[j >> 2].y, k4[j >> 2].z, k4[j >> 2].w};
#pragma unroll
        for (int e = 0; e < 4; e++)
#pragma unroll
          for (int c = 0; c < 4; c++) S[j + e][c] = fmaf(kk[e], u[c], m.x * S[j + e][c]);
      }
    }
    __syncthreads();
    // (written before the next tokens' first barrier, read by nobody else before it: so is free again when it is written)
    for (int idx = threadIdx.x; idx < nt * DR_COLS; idx += DR_THREADS) {
      const int tt = idx / DR_COLS, cc = idx - tt * DR_COLS;
      if (col0 + cc < vdim) out[(size_t)(first + t0 + tt) * heads * vdim + (size_t)h * vdim + col0 + cc] = so[tt][cc];
    }
  }
  cima_pdl_trigger();        // the tokens are done: the next kernel may be set up while the state is stored
#pragma unroll
  for (int j = 0; j < RP; j++) {
    const int row = (j >> 2) * 64 + rg * 4 + (j & 3);
    if (row < dim) {
      if (whole) {
        *reinterpret_cast<float4*>(st + (size_t)row * vdim) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
      } else {
#pragma unroll
        for (int c = 0; c < 4; c++)
          if (c < cols) st[(size_t)row * vdim + c] = S[j][c];
      }
    }
  }
}


// ---------------------------------------------------------------------------------------------------- 16 tokens at a time
constexpr int DC_T = 16, DC_WARPS = 4, DC_COLS = 16 * DC_WARPS, DC_THREADS = 32 * (DC_WARPS + 3), DC_STAGES = 5;
constexpr int DC_TROW = 24, DC_VROW = DC_COLS + 8;      // padded rows of the 16 x 16 matrices' terms and of v

typedef __nv_bfloat16 bf16;
__device__ __forceinline__ void dc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void dc_ldmatrix(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((unsigned)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void dc_ldmatrix_trans(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((unsigned)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void dc_copy16(unsigned dst, const bf16* src) {             // 16 bytes, dst an address in shared memory
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src));
}
// x, y as a sum of three bfloat16 terms each, packed in pairs (x in the low half)
__device__ __forceinline__ void dc_split(float x, float y, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 hf = __bfloat1622float2(h);
  x -= hf.x; y -= hf.y;
  const __nv_bfloat162 m = __floats2bfloat162_rn(x, y);
  const float2 mf = __bfloat1622float2(m);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - mf.x, y - mf.y);
  hi = *reinterpret_cast<const uint32_t*>(&h); mid = *reinterpret_cast<const uint32_t*>(&m); lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <int DIMP>
struct __align__(16) DcShared {
  bf16 k[DC_STAGES][DC_T][DIMP + 8], q[DC_STAGES][DC_T][DIMP + 8], v[DC_STAGES][DC_T][DC_VROW];
  bf16 T[2][3][DC_T][DC_TROW], M[2][3][DC_T][DC_TROW];  // the terms of the inverse and of the read-out's matrix, [t][s]
  __align__(16) float kk[2][DC_T][DC_T + 4], qk[2][DC_T][DC_T + 4], A[DC_T][DC_T + 4];      // k_t.k_s, q_t.k_s
  double L[2][DC_T];                                    // logarithms of G_t, which may be large beside their differences
  float fk[2][DC_T], fq[2][DC_T], step[2][DC_T];        // rk, rq, beta
  float beta[2][DC_T], gk[2][DC_T], gq[2][DC_T], w[2][DC_T], gc[2];      // beta_t, G_t rk_t, G_t rq_t, (G_16 / G_s) rk_s, G_16
};

template <int DIMP>
__global__ void __launch_bounds__(DC_THREADS)
k_delta_chunk(const bf16* __restrict__ qkv, int ld, const bf16* __restrict__ a, int lda, const bf16* __restrict__ b, int ldb,
              const float* __restrict__ A_log, const float* __restrict__ dt_bias, float* __restrict__ state, const int* __restrict__ seq_slot,
              const int* __restrict__ seq_first_row, float* __restrict__ out, int heads, int kv_heads, int dim, int vdim, float qscale) {
  extern __shared__ __align__(16) unsigned char dc_smem[];
  DcShared<DIMP>& sm = *reinterpret_cast<DcShared<DIMP>*>(dc_smem);
  constexpr int KS = DIMP / 16, NT = DIMP / 8;
  const int seq = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * DC_COLS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g8 = lane >> 2, t4 = lane & 3;              // a fragment's row (and row + 8) and pair of columns
  const int kvh = h / (heads / kv_heads), kd = kv_heads * dim;
  const float rate = expf(A_log[h]), bias = dt_bias[h];
  cima_pdl_wait();
  const int first = seq_first_row[seq], n = seq_first_row[seq + 1] - first;
  const int chunks = (n + DC_T - 1) / DC_T;
  // what no copy reaches (dims and columns beyond the sizes) stays zero
  for (int i = threadIdx.x; i < (int)(sizeof(sm.k) + sizeof(sm.q) + sizeof(sm.v)) / 16; i += DC_THREADS) reinterpret_cast<uint4*>(&sm)[i] = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();
  // where the lane's pieces of a B operand lie for ldmatrix (rows of n, k contiguous; and its transposed form)
  const int b_row = (lane & 7) + 8 * (lane >> 4), b_col = 8 * ((lane >> 3) & 1);
  const int bt_row = (lane & 7) + 8 * ((lane >> 3) & 1), bt_col = 8 * (lane >> 4);

  // Every warp meets a barrier at the start of step j = -3 .. chunks - 1 and works on its own chunk of that step, if there is one.
  if (warp == DC_WARPS + 2) {
    // ------------------------------------------------------------------------------------------ the rows of chunk j + 4
    // A lane copies the same 16 bytes of every second (q, k) or fourth (v) token.  Beyond a sequence's end the last token's rows
    // are copied again: a token with step size 0 changes nothing, whatever its rows hold, as long as they are finite.
    constexpr int QL = DIMP / 8, QS = 32 / QL, VL = DC_COLS / 8, VS = 32 / VL;
    const int qt = lane / QL, qd = (lane % QL) * 8, vt = lane / VL, vd = (lane % VL) * 8;
    const bool q_ok = qd < dim, v_ok = col0 + vd < vdim;
    const bf16 *qp = qkv + (size_t)first * ld + (size_t)kvh * dim + qd, *vp = qkv + (size_t)first * ld + 2 * kd + (size_t)h * vdim + col0 + vd;
    const unsigned sq = (unsigned)__cvta_generic_to_shared(&sm.q[0][qt][qd]), sk = (unsigned)__cvta_generic_to_shared(&sm.k[0][qt][qd]);
    const unsigned sv = (unsigned)__cvta_generic_to_shared(&sm.v[0][vt][vd]);
    auto load = [&](int c) {
      if (c < chunks) {
        const int stage = c % DC_STAGES, t0 = c * DC_T, last = n - 1;
        const unsigned at = stage * (unsigned)(DC_T * (DIMP + 8) * 2), atv = stage * (unsigned)(DC_T * DC_VROW * 2);
        if (q_ok) {
#pragma unroll
          for (int r = 0; r < DC_T / QS; r++) {
            const bf16* p = qp + (size_t)min(t0 + qt + r * QS, last) * ld;
            dc_copy16(sq + at + r * QS * (DIMP + 8) * 2, p);
            dc_copy16(sk + at + r * QS * (DIMP + 8) * 2, p + kd);
          }
        }
        if (v_ok) {
#pragma unroll
          for (int r = 0; r < DC_T / VS; r++) dc_copy16(sv + atv + r * VS * DC_VROW * 2, vp + (size_t)min(t0 + vt + r * VS, last) * ld);
        }
      }
      asm volatile("cp.async.commit_group;\n" ::);
    };
    load(0);
    for (int j = -3; j < chunks; j++) {
      __syncthreads();
      load(j + 4);                                      // (into the place of chunk j - 1, which is done)
      asm volatile("cp.async.wait_group 1;\n" ::);      // chunk j + 3 is there at the next barrier
    }
    asm volatile("cp.async.wait_group 0;\n" ::);
    return;
  }
  if (warp == DC_WARPS) {
    // ------------------------------------------------------------------------------------------ norms, decays and row products of chunk j + 2
    bf16 za = __float2bfloat16_rn(0.f), zb = za;        // the next chunk's decay and step size of token `lane`
    auto numbers = [&](int c) {
      if (lane < DC_T && c * DC_T + lane < n) {
        za = a[(size_t)(first + c * DC_T + lane) * lda + h];
        zb = b[(size_t)(first + c * DC_T + lane) * ldb + h];
      }
    };
    numbers(0);
    for (int j = -3; j < chunks; j++) {
      __syncthreads();
      const int c = j + 2;
      if (c < 0 || c >= chunks) continue;
      const int stage = c % DC_STAGES, buf = c & 1, nt = min(DC_T, n - c * DC_T);
      // rows t = g8, g8 + 8; columns s = 2 t4, 2 t4 + 1 of the tiles s < 8 and s >= 8
      float gkk[2][4] = {}, gqk[2][4] = {}, gqq[2][4] = {};
#pragma unroll
      for (int i = 0; i < KS; i++) {
        uint32_t ak[4], aq[4], bk[4], bq[4];
        dc_ldmatrix(ak, &sm.k[stage][lane & 15][i * 16 + 8 * (lane >> 4)]);
        dc_ldmatrix(aq, &sm.q[stage][lane & 15][i * 16 + 8 * (lane >> 4)]);
        dc_ldmatrix(bk, &sm.k[stage][b_row][i * 16 + b_col]);
        dc_ldmatrix(bq, &sm.q[stage][b_row][i * 16 + b_col]);
#pragma unroll
        for (int x = 0; x < 2; x++) {
          dc_mma(gkk[x], ak, bk[2 * x], bk[2 * x + 1]);
          dc_mma(gqk[x], aq, bk[2 * x], bk[2 * x + 1]);
          dc_mma(gqq[x], aq, bq[2 * x], bq[2 * x + 1]);
        }
      }
      // a token of lane l < 16: logarithm of the decay, summed up over the chunk; a token beyond the end neither forgets nor writes
      double lg = 0.0;
      float be = 0.f;
      if (lane < nt) {
        const float z = __bfloat162float(za) + bias;
        lg = (double)fmaxf(-rate * (z > 20.f ? z : log1pf(expf(z))), -1e30f);
        be = 1.0f / (1.0f + expf(-__bfloat162float(zb)));
      }
      numbers(c + 1);
#pragma unroll
      for (int o = 1; o < DC_T; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, lg, o);
        if (lane >= o) lg += up;                        // (lanes from 16 on are not used)
      }
      if (lane < DC_T) { sm.L[buf][lane] = lg; sm.step[buf][lane] = be; }
#pragma unroll
      for (int x = 0; x < 2; x++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int t = g8 + 8 * e, s2 = 8 * x + 2 * t4;
          *reinterpret_cast<float2*>(&sm.kk[buf][t][s2]) = make_float2(gkk[x][2 * e], gkk[x][2 * e + 1]);
          *reinterpret_cast<float2*>(&sm.qk[buf][t][s2]) = make_float2(gqk[x][2 * e], gqk[x][2 * e + 1]);
        }
      if (t4 == (g8 >> 1)) {                            // the lane holds the squares of tokens g8 and g8 + 8
        const bool odd = g8 & 1;
        sm.fk[buf][g8] = 1.0f / sqrtf((odd ? gkk[0][1] : gkk[0][0]) + 1e-6f);
        sm.fk[buf][g8 + 8] = 1.0f / sqrtf((odd ? gkk[1][3] : gkk[1][2]) + 1e-6f);
        sm.fq[buf][g8] = qscale / sqrtf((odd ? gqq[0][1] : gqq[0][0]) + 1e-6f);
        sm.fq[buf][g8 + 8] = qscale / sqrtf((odd ? gqq[1][3] : gqq[1][2]) + 1e-6f);
      }
    }
    return;
  }
  if (warp == DC_WARPS + 1) {
    // ------------------------------------------------------------------------------------------ T and M of chunk j + 1
    for (int j = -3; j < chunks; j++) {
      __syncthreads();
      const int c = j + 1;
      if (c < 0 || c >= chunks) continue;
      const int buf = c & 1;
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int t = g8 + 8 * e;
        const double Lt = sm.L[buf][t];
        const float ft = sm.fk[buf][t] * sm.step[buf][t], fqt = sm.fq[buf][t];
#pragma unroll
        for (int x = 0; x < 2; x++) {
          const int s2 = 8 * x + 2 * t4;
          const float2 kk = *reinterpret_cast<const float2*>(&sm.kk[buf][t][s2]), qk = *reinterpret_cast<const float2*>(&sm.qk[buf][t][s2]);
          const float r0 = s2 <= t ? expf((float)(Lt - sm.L[buf][s2])) * sm.fk[buf][s2] : 0.f;
          const float r1 = s2 + 1 <= t ? expf((float)(Lt - sm.L[buf][s2 + 1])) * sm.fk[buf][s2 + 1] : 0.f;
          *reinterpret_cast<float2*>(&sm.A[t][s2]) = make_float2(s2 < t ? r0 * ft * kk.x : 0.f, s2 + 1 < t ? r1 * ft * kk.y : 0.f);
          uint32_t hi, mid, lo;
          dc_split(r0 * fqt * qk.x, r1 * fqt * qk.y, hi, mid, lo);
          *reinterpret_cast<uint32_t*>(&sm.M[buf][0][t][s2]) = hi;
          *reinterpret_cast<uint32_t*>(&sm.M[buf][1][t][s2]) = mid;
          *reinterpret_cast<uint32_t*>(&sm.M[buf][2][t][s2]) = lo;
        }
      }
      if (lane < DC_T) {
        const double lg = sm.L[buf][lane], total = sm.L[buf][DC_T - 1];
        const float G = expf((float)lg), fk = sm.fk[buf][lane];
        sm.beta[buf][lane] = sm.step[buf][lane];
        sm.gk[buf][lane] = G * fk;
        sm.gq[buf][lane] = G * sm.fq[buf][lane];
        sm.w[buf][lane] = expf((float)(total - lg)) * fk;
        if (lane == DC_T - 1) sm.gc[buf] = G;
      }
      __syncwarp();
      // column `lane` of T: T[t] = e_t - sum_{s < t} A[t][s] T[s]
      const int col = lane & 15;
      float T[DC_T];
#pragma unroll
      for (int t = 0; t < DC_T; t++) {
        float s0 = t == col ? 1.f : 0.f, s1 = 0.f;
#pragma unroll
        for (int x = 0; x < t; x += 4) {
          const float4 A4 = *reinterpret_cast<const float4*>(&sm.A[t][x]);        // (entries from t on are 0)
          s0 = fmaf(-A4.x, T[x], s0);
          if (x + 1 < t) s1 = fmaf(-A4.y, T[x + 1], s1);
          if (x + 2 < t) s0 = fmaf(-A4.z, T[x + 2], s0);
          if (x + 3 < t) s1 = fmaf(-A4.w, T[x + 3], s1);
        }
        T[t] = s0 + s1;
      }
      if (lane < DC_T) {
#pragma unroll
        for (int t = 0; t < DC_T; t++) {
          const bf16 hi = __float2bfloat16_rn(T[t]);
          const float r1 = T[t] - __bfloat162float(hi);
          const bf16 mid = __float2bfloat16_rn(r1);
          sm.T[buf][0][t][col] = hi;
          sm.T[buf][1][t][col] = mid;
          sm.T[buf][2][t][col] = __float2bfloat16_rn(r1 - __bfloat162float(mid));
        }
      }
      __syncwarp();                                     // (A is written again by other lanes)
    }
    return;
  }

  // ---------------------------------------------------------------------------------------------- 16 columns of the state
  // acc[j]: S^T, rows (columns of S) c0 = g8 and c0 + 8, dims 8 j + 2 t4 and the next
  const int c0 = warp * 16 + g8;
  float* st = state + (((size_t)seq_slot[seq] * heads + h) * dim) * (size_t)vdim + col0 + c0;
  const bool in0 = col0 + c0 < vdim, in1 = col0 + c0 + 8 < vdim;
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; j++)
#pragma unroll
    for (int y = 0; y < 2; y++) {
      const int d = 8 * j + 2 * t4 + y;
      acc[j][y] = in0 && d < dim ? st[(size_t)d * vdim] : 0.f;
      acc[j][2 + y] = in1 && d < dim ? st[(size_t)d * vdim + 8] : 0.f;
    }
  for (int j = -3; j < 0; j++) __syncthreads();         // (the other warps' first chunks)
  for (int c = 0; c < chunks; c++) {
    __syncthreads();
    const int stage = c % DC_STAGES, buf = c & 1, t0 = c * DC_T;
    // P = k^T S0 and R = q^T S0, transposed: the terms of S apart, the two small ones together
    float ph[2][4] = {}, pl[2][4] = {}, rh[2][4] = {}, rl[2][4] = {};
#pragma unroll
    for (int j = 0; j < KS; j++) {
      uint32_t hi[4], mid[4], lo[4], bk[4], bq[4];
#pragma unroll
      for (int x = 0; x < 2; x++)
#pragma unroll
        for (int e = 0; e < 2; e++)
          dc_split(acc[2 * j + x][2 * e], acc[2 * j + x][2 * e + 1], hi[2 * x + e], mid[2 * x + e], lo[2 * x + e]);
      dc_ldmatrix(bk, &sm.k[stage][b_row][j * 16 + b_col]);
      dc_ldmatrix(bq, &sm.q[stage][b_row][j * 16 + b_col]);
#pragma unroll
      for (int x = 0; x < 2; x++) {
        dc_mma(pl[x], lo, bk[2 * x], bk[2 * x + 1]);
        dc_mma(rl[x], lo, bq[2 * x], bq[2 * x + 1]);
        dc_mma(ph[x], hi, bk[2 * x], bk[2 * x + 1]);
        dc_mma(rh[x], hi, bq[2 * x], bq[2 * x + 1]);
        dc_mma(pl[x], mid, bk[2 * x], bk[2 * x + 1]);
        dc_mma(rl[x], mid, bq[2 * x], bq[2 * x + 1]);
      }
    }
    // rhs^T: columns c0, c0 + 8; tokens 8 x + 2 t4, + 1; as A operand of U^T = rhs^T T^T
    uint32_t hi[4], mid[4], lo[4];
#pragma unroll
    for (int x = 0; x < 2; x++) {
      const int t = 8 * x + 2 * t4;
      const float be0 = sm.beta[buf][t], be1 = sm.beta[buf][t + 1], gk0 = sm.gk[buf][t], gk1 = sm.gk[buf][t + 1];
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const float v0 = __bfloat162float(sm.v[stage][t][c0 + 8 * e]), v1 = __bfloat162float(sm.v[stage][t + 1][c0 + 8 * e]);
        dc_split(be0 * (v0 - gk0 * (ph[x][2 * e] + pl[x][2 * e])), be1 * (v1 - gk1 * (ph[x][2 * e + 1] + pl[x][2 * e + 1])),
                 hi[2 * x + e], mid[2 * x + e], lo[2 * x + e]);
      }
    }
    // the product of two float32 matrices, each as three terms: all pairs but those below 2^-24
    auto product = [&](float (&o)[2][4], const bf16 (&B)[3][DC_T][DC_TROW]) {
      float small[2][4] = {};
#pragma unroll
      for (int x = 0; x < 2; x++) {
        uint32_t b0[3], b1[3];
#pragma unroll
        for (int m = 0; m < 3; m++) {
          b0[m] = *reinterpret_cast<const uint32_t*>(&B[m][8 * x + g8][2 * t4]);
          b1[m] = *reinterpret_cast<const uint32_t*>(&B[m][8 * x + g8][2 * t4 + 8]);
        }
        dc_mma(small[x], lo, b0[0], b1[0]);
        dc_mma(small[x], hi, b0[2], b1[2]);
        dc_mma(small[x], mid, b0[1], b1[1]);
        dc_mma(small[x], mid, b0[0], b1[0]);
        dc_mma(small[x], hi, b0[1], b1[1]);
        dc_mma(o[x], hi, b0[0], b1[0]);
      }
#pragma unroll
      for (int x = 0; x < 2; x++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[x][e] += small[x][e];
    };
    float U[2][4] = {};
    product(U, sm.T[buf]);
#pragma unroll
    for (int x = 0; x < 2; x++)
#pragma unroll
      for (int e = 0; e < 2; e++) dc_split(U[x][2 * e], U[x][2 * e + 1], hi[2 * x + e], mid[2 * x + e], lo[2 * x + e]);
    float o[2][4];
#pragma unroll
    for (int x = 0; x < 2; x++) {
      const float q0 = sm.gq[buf][8 * x + 2 * t4], q1 = sm.gq[buf][8 * x + 2 * t4 + 1];
#pragma unroll
      for (int e = 0; e < 2; e++) {
        o[x][2 * e] = q0 * (rh[x][2 * e] + rl[x][2 * e]);
        o[x][2 * e + 1] = q1 * (rh[x][2 * e + 1] + rl[x][2 * e + 1]);
      }
    }
    product(o, sm.M[buf]);
#pragma unroll
    for (int x = 0; x < 2; x++)
#pragma unroll
      for (int y = 0; y < 2; y++) {
        const int t = t0 + 8 * x + 2 * t4 + y;
        if (t < n) {
          float* dst = out + ((size_t)(first + t) * heads + h) * vdim + col0 + c0;
          if (in0) dst[0] = o[x][y];
          if (in1) dst[8] = o[x][2 + y];
        }
      }
    // S^T <- G S^T + (w U)^T k
#pragma unroll
    for (int x = 0; x < 2; x++) {
      const float w0 = sm.w[buf][8 * x + 2 * t4], w1 = sm.w[buf][8 * x + 2 * t4 + 1];
#pragma unroll
      for (int e = 0; e < 2; e++) dc_split(w0 * U[x][2 * e], w1 * U[x][2 * e + 1], hi[2 * x + e], mid[2 * x + e], lo[2 * x + e]);
    }
    const float G = sm.gc[buf];
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      uint32_t bk[4];
      dc_ldmatrix_trans(bk, &sm.k[stage][bt_row][j * 8 + bt_col]);
#pragma unroll
      for (int x = 0; x < 2; x++) {
        float add[4] = {0.f, 0.f, 0.f, 0.f};
        dc_mma(add, lo, bk[2 * x], bk[2 * x + 1]);
        dc_mma(add, mid, bk[2 * x], bk[2 * x + 1]);
        dc_mma(add, hi, bk[2 * x], bk[2 * x + 1]);
#pragma unroll
        for (int e = 0; e < 4; e++) acc[j + x][e] = fmaf(G, acc[j + x][e], add[e]);
      }
    }
  }
  cima_pdl_trigger();
#pragma unroll
  for (int j = 0; j < NT; j++)
#pragma unroll
    for (int y = 0; y < 2; y++) {
      const int d = 8 * j + 2 * t4 + y;
      if (in0 && d < dim) st[(size_t)d * vdim] = acc[j][y];
      if (in1 && d < dim) st[(size_t)d * vdim + 8] = acc[j][2 + y];
    }
}

template <int DIMP>
int launch_delta_chunk(const void* qkv, int ld, const void* a, int lda, const void* b, int ldb, const float* A_log, const float* dt_bias,
                       float* state, const int* seq_slot, const int* seq_first_row, float* out, int n_seqs, int heads, int kv_heads, int dim,
                       int vdim, cudaStream_t stream) {
  const dim3 grid((vdim + DC_COLS - 1) / DC_COLS, heads, n_seqs);
  typedef DcShared<DIMP> Sh;
  static_assert(offsetof(Sh, k) % 16 == 0 && offsetof(Sh, q) % 16 == 0 && offsetof(Sh, v) % 16 == 0 && offsetof(Sh, A) % 16 == 0 &&
                offsetof(Sh, kk) % 8 == 0 && offsetof(Sh, qk) % 8 == 0 && offsetof(Sh, L) % 8 == 0 && offsetof(Sh, T) % 4 == 0 &&
                offsetof(Sh, M) % 4 == 0 && (DIMP + 8) * 2 % 16 == 0 && DC_VROW * 2 % 16 == 0 && DC_TROW * 2 % 4 == 0 && (DC_T + 4) * 4 % 16 == 0,
                "what is read 16 (8, 4) bytes at a time starts there");
  constexpr size_t smem = sizeof(Sh);
  static bool raised = false;
  if (smem > 48 * 1024 && !raised) {
    cudaError_t e = cudaFuncSetAttribute(k_delta_chunk<DIMP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return cima_fail((int)e, "delta_rule: cannot raise shared memory to %zu bytes: %s", smem, cudaGetErrorString(e));
    raised = true;
  }
  return cima_launch(k_delta_chunk<DIMP>, grid, dim3(DC_THREADS), smem, stream, 1, (const bf16*)qkv, ld, (const bf16*)a, lda, (const bf16*)b, ldb, A_log,
                     dt_bias, state, seq_slot, seq_first_row, out, heads, kv_heads, dim, vdim, 1.0f / sqrtf((float)dim));
}

template <typename TA, int DIMP>
int launch_delta_rule(const void* qkv, int ld, const void* a, int lda, const void* b, int ldb, const float* A_log, const float* dt_bias,
                      float* state, const int* seq_slot, const int* seq_first_row, float* out, int n_seqs, int heads, int kv_heads, int dim,
                      int vdim, cudaStream_t stream) {
  const dim3 grid((vdim + DR_COLS - 1) / DR_COLS, heads, n_seqs);
  const float qscale = 1.0f / sqrtf((float)dim);
  constexpr int V = 16 / (int)sizeof(TA);
  const bool vec = dim % V == 0 && ld % V == 0 && ((uintptr_t)qkv & 15) == 0;
#define RUN(VEC) return cima_launch(k_delta_rule<TA, DIMP, VEC>, grid, dim3(DR_THREADS), (size_t)0, stream, 1, (const TA*)qkv, ld, (const TA*)a, lda, \
                                    (const TA*)b, ldb, A_log, dt_bias, state, seq_slot, seq_first_row, out, heads, kv_heads, dim, vdim, qscale)
  if (vec) RUN(true);
  RUN(false);
#undef RUN
}
}  // namespace

// qkv [T, ld]: a row's q heads, k heads (kv_heads of dim values each), v heads (heads of vdim); a, b [T, lda / ldb]: one number a head;
// all of dtype.  A_log, dt_bias [heads] float32.  chunked: 16 tokens at a time (bfloat16, sizes and strides multiples of 8, dim <= 128).  out [T, heads * vdim] float32.
extern "C" int cima_delta_rule(const void* qkv, int ld, const void* a, int lda, const void* b, int ldb, int dtype, const float* A_log,
                               const float* dt_bias, float* state, const int* seq_slot, const int* seq_first_row, float* out, int T, int n_seqs,
                               int heads, int kv_heads, int dim, int vdim, int chunked, cudaStream_t stream) {
  if (T <= 0 || n_seqs <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || heads > 65535 || n_seqs > 65535)
    return cima_fail(CIMA_E_SIZE, "delta_rule: %d heads on %d key heads in %d sequences are not accepted", heads, kv_heads, n_seqs);
  if (dim <= 0 || dim > 256 || vdim <= 0) return cima_fail(CIMA_E_SIZE, "delta_rule: key size %d must lie in 1..256 and value size %d be positive", dim, vdim);
  if (ld < 2 * kv_heads * dim + heads * vdim || lda < heads || ldb < heads) return cima_fail(CIMA_E_SIZE, "delta_rule: rows of %d, %d and %d values do not hold the heads", ld, lda, ldb);
  if ((uintptr_t)state & 15) return cima_fail(CIMA_E_ARG, "delta_rule: the state must start on 16 bytes");
  if (!qkv || !a || !b || !A_log || !dt_bias || !state || !out) return cima_fail(CIMA_E_ARG, "delta_rule: the rows, the heads' numbers, the state and the output are needed");
  int rc;
  if (chunked) {
    if (dtype != CIMA_BF16 || dim > 128 || dim % 8 || vdim % 8 || ld % 8 || ((uintptr_t)qkv & 15))
      return cima_fail(CIMA_E_SIZE, "delta_rule: 16 tokens at a time take bfloat16 rows (stride %d) and key and value sizes %d and %d in multiples of 8, at most 128 for keys", ld, dim, vdim);
    if (dim <= 64) rc = launch_delta_chunk<64>(qkv, ld, a, lda, b, ldb, A_log, dt_bias, state, seq_slot, seq_first_row, out, n_seqs, heads, kv_heads, dim, vdim, stream);
    else rc = launch_delta_chunk<128>(qkv, ld, a, lda, b, ldb, A_log, dt_bias, state, seq_slot, seq_first_row, out, n_seqs, heads, kv_heads, dim, vdim, stream);
    return rc ? rc : cima_launch_result();
  }
#define SIZES(TA) { if (dim <= 64) RUN(TA, 64); else if (dim <= 128) RUN(TA, 128); else RUN(TA, 256); }
#define RUN(TA, D) rc = launch_delta_rule<TA, D>(qkv, ld, a, lda, b, ldb, A_log, dt_bias, state, seq_slot, seq_first_row, out, n_seqs, heads, kv_heads, dim, vdim, stream)
  if (dtype == CIMA_F32) SIZES(float)
  else if (dtype == CIMA_BF16) SIZES(__nv_bfloat16)
  else return cima_fail(CIMA_E_DTYPE, "delta_rule: dtype code %d is neither float32 nor bfloat16", dtype);
#undef RUN
#undef SIZES
  return rc ? rc : cima_launch_result();
}
