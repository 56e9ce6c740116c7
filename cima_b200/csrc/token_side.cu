// A token's own input to a layer: z[t, j] = act(sum_k x[t, k] W[j, k]) * D[tok_t, col + j], D the model's side table.
//
// token_side_few    the whole of it for the few rows of a decode step, straight from the float32 stream: a warp takes two
//                   outputs j, its lanes stride the two rows of W by 16 bytes and hold the sums of all rows (at most 8); a fixed
//                   shuffle tree adds the lanes.  A row's sum does not depend on what else is in the step.
// token_side_apply  behind a product of many rows: z <- act(z) * D[tok, col + j] in place
#include "common.cuh"

namespace {
constexpr int TS_ROWS = 8, TS_OUTS = 2, TS_WARPS = 4;

template <typename TW> struct TsVec;                          // weights of one 16-byte load
template <> struct TsVec<float> { static constexpr int N = 4; };
template <> struct TsVec<__nv_bfloat16> { static constexpr int N = 8; };

template <typename TW, typename TA>
__global__ void __launch_bounds__(TS_WARPS * 32)
k_token_side_few(const float* __restrict__ x, const TW* __restrict__ w, const TA* __restrict__ table, int ldt, const int* __restrict__ tokens,
                 int col, TA* __restrict__ z, int T, int dim, int W, int vocab, int act, int vec) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int j0 = (blockIdx.x * TS_WARPS + warp) * TS_OUTS;
  if (j0 >= dim) return;
  const int j1 = min(j0 + 1, dim - 1);                        // (an odd last output is computed twice and stored once)
  const TW *w0 = w + (size_t)j0 * W, *w1 = w + (size_t)j1 * W;
  constexpr int V = TsVec<TW>::N;
  float acc[TS_OUTS][TS_ROWS];
#pragma unroll
  for (int o = 0; o < TS_OUTS; o++)
#pragma unroll
    for (int r = 0; r < TS_ROWS; r++) acc[o][r] = 0.f;
  if (vec) {
    // the first weights depend on no kernel: they are requested before the wait
    uint4 n0 = make_uint4(0u, 0u, 0u, 0u), n1 = n0;
    if (lane * V < W) { n0 = *reinterpret_cast<const uint4*>(w0 + lane * V); n1 = *reinterpret_cast<const uint4*>(w1 + lane * V); }
    cima_pdl_wait();
    for (int k = lane * V; k < W; k += 32 * V) {
      const uint4 c0 = n0, c1 = n1;
      const int kn = k + 32 * V;
      if (kn < W) { n0 = *reinterpret_cast<const uint4*>(w0 + kn); n1 = *reinterpret_cast<const uint4*>(w1 + kn); }
      const TW *a = reinterpret_cast<const TW*>(&c0), *b = reinterpret_cast<const TW*>(&c1);
      float4 xv[TS_ROWS][V / 4];
#pragma unroll
      for (int r = 0; r < TS_ROWS; r++)
#pragma unroll
        for (int q = 0; q < V / 4; q++)
          xv[r][q] = r < T ? *reinterpret_cast<const float4*>(x + (size_t)r * W + k + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int q = 0; q < V / 4; q++) {
        const float a0 = cima_to_f32<TW>(a[4 * q]), a1 = cima_to_f32<TW>(a[4 * q + 1]), a2 = cima_to_f32<TW>(a[4 * q + 2]), a3 = cima_to_f32<TW>(a[4 * q + 3]);
        const float b0 = cima_to_f32<TW>(b[4 * q]), b1 = cima_to_f32<TW>(b[4 * q + 1]), b2 = cima_to_f32<TW>(b[4 * q + 2]), b3 = cima_to_f32<TW>(b[4 * q + 3]);
#pragma unroll
        for (int r = 0; r < TS_ROWS; r++) {
          const float4 f = xv[r][q];
          acc[0][r] = fmaf(f.x, a0, acc[0][r]); acc[0][r] = fmaf(f.y, a1, acc[0][r]);
          acc[0][r] = fmaf(f.z, a2, acc[0][r]); acc[0][r] = fmaf(f.w, a3, acc[0][r]);
          acc[1][r] = fmaf(f.x, b0, acc[1][r]); acc[1][r] = fmaf(f.y, b1, acc[1][r]);
          acc[1][r] = fmaf(f.z, b2, acc[1][r]); acc[1][r] = fmaf(f.w, b3, acc[1][r]);
        }
      }
    }
  } else {
    cima_pdl_wait();
    for (int k = lane; k < W; k += 32) {
      const float a = cima_to_f32<TW>(w0[k]), b = cima_to_f32<TW>(w1[k]);
#pragma unroll
      for (int r = 0; r < TS_ROWS; r++) {
        const float f = r < T ? x[(size_t)r * W + k] : 0.f;
        acc[0][r] = fmaf(f, a, acc[0][r]);
        acc[1][r] = fmaf(f, b, acc[1][r]);
      }
    }
  }
  cima_pdl_trigger();
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int q = 0; q < TS_OUTS; q++)
#pragma unroll
      for (int r = 0; r < TS_ROWS; r++) acc[q][r] += __shfl_xor_sync(0xffffffffu, acc[q][r], o);
  // lane (q, r) = q * TS_ROWS + r finishes output j0 + q of row r
#pragma unroll
  for (int q = 0; q < TS_OUTS; q++)
#pragma unroll
    for (int r = 0; r < TS_ROWS; r++)
      if (lane == q * TS_ROWS + r && r < T && j0 + q < dim) {
        int tok = tokens[r];
        tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
        const float e = cima_to_f32<TA>(table[(size_t)tok * ldt + col + j0 + q]);
        z[(size_t)r * dim + j0 + q] = cima_from_f32<TA>(cima_gate_act(acc[q][r], act) * e);
      }
}

template <typename TA>
__global__ void __launch_bounds__(256)
k_token_side_apply(TA* __restrict__ z, const TA* __restrict__ table, int ldt, const int* __restrict__ tokens, int col, size_t total, int dim,
                   int vocab, int act) {
  cima_pdl_wait();
  cima_pdl_trigger();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / dim;
    int tok = tokens[t];
    tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
    z[i] = cima_from_f32<TA>(cima_gate_act(cima_to_f32<TA>(z[i]), act) * cima_to_f32<TA>(table[(size_t)tok * ldt + col + (int)(i - t * dim)]));
  }
}

// Four neighbouring values a thread (dim, col and the table's rows multiples of 4, aligned).
template <typename TA> struct TsFour;
template <> struct TsFour<float> { typedef float4 T; };
template <> struct TsFour<__nv_bfloat16> { typedef uint2 T; };
template <typename TA>
__global__ void __launch_bounds__(256)
k_token_side_apply4(TA* __restrict__ z, const TA* __restrict__ table, int ldt, const int* __restrict__ tokens, int col, size_t groups, int dim,
                    int vocab, int act) {
  cima_pdl_wait();
  cima_pdl_trigger();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < groups; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / (dim / 4);
    const int j = 4 * (int)(i - t * (dim / 4));
    typedef typename TsFour<TA>::T F;
    int tok = tokens[t];
    tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
    F v = *reinterpret_cast<const F*>(z + t * dim + j);
    const F e = *reinterpret_cast<const F*>(table + (size_t)tok * ldt + col + j);
    TA* vp = reinterpret_cast<TA*>(&v);
    const TA* ep = reinterpret_cast<const TA*>(&e);
#pragma unroll
    for (int q = 0; q < 4; q++) vp[q] = cima_from_f32<TA>(cima_gate_act(cima_to_f32<TA>(vp[q]), act) * cima_to_f32<TA>(ep[q]));
    *reinterpret_cast<F*>(z + t * dim + j) = v;
  }
}
}  // namespace

// x [T, W] float32 with T <= 8, w [dim, W] (wdtype), table [vocab, ldt] and z [T, dim] of dtype; col: the layer's first column of the table.
extern "C" int cima_token_side_few(const float* x, const void* w, int wdtype, const void* table, int ldt, int dtype, const int* tokens, int col,
                                   void* z, int T, int dim, int W, int vocab, int act, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (T > TS_ROWS) return cima_fail(CIMA_E_SIZE, "token_side_few: %d rows; this kernel takes at most %d", T, TS_ROWS);
  if (dim <= 0 || W <= 0 || vocab <= 0 || col < 0 || ldt < col + dim) return cima_fail(CIMA_E_SIZE, "token_side_few: %d values from column %d on exceed a table's rows of %d (width %d)", dim, col, ldt, W);
  if (act < 0 || act >= CIMA_ACT_COUNT) return cima_fail(CIMA_E_ARG, "token_side_few: activation code %d is unknown", act);
  const int vec = W % (wdtype == CIMA_F32 ? 4 : 8) == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0;
  const dim3 grid((unsigned)((dim + TS_OUTS * TS_WARPS - 1) / (TS_OUTS * TS_WARPS)));
  int rc;
#define RUN(TW, TA) rc = cima_launch(k_token_side_few<TW, TA>, grid, dim3(TS_WARPS * 32), (size_t)0, stream, 1, x, (const TW*)w, (const TA*)table, ldt, tokens, col, (TA*)z, T, dim, W, vocab, act, vec)
  if (wdtype == CIMA_F32 && dtype == CIMA_F32) RUN(float, float);
  else if (wdtype == CIMA_BF16 && dtype == CIMA_BF16) RUN(__nv_bfloat16, __nv_bfloat16);
  else if (wdtype == CIMA_F32 && dtype == CIMA_BF16) RUN(float, __nv_bfloat16);
  else return cima_fail(CIMA_E_DTYPE, "token_side_few: weights of dtype code %d with rows of %d are not accepted", wdtype, dtype);
#undef RUN
  return rc ? rc : cima_launch_result();
}

// z [T, dim] in place, z and the table of one dtype.
extern "C" int cima_token_side_apply(void* z, const void* table, int ldt, int dtype, const int* tokens, int col, int T, int dim, int vocab, int act,
                                     cudaStream_t stream) {
  if (T <= 0) return 0;
  if (dim <= 0 || vocab <= 0 || col < 0 || ldt < col + dim) return cima_fail(CIMA_E_SIZE, "token_side_apply: %d values from column %d on exceed a table's rows of %d", dim, col, ldt);
  if (act < 0 || act >= CIMA_ACT_COUNT) return cima_fail(CIMA_E_ARG, "token_side_apply: activation code %d is unknown", act);
  const size_t bytes = dtype == CIMA_F32 ? 16 : 8;
  const bool four = dim % 4 == 0 && col % 4 == 0 && ldt % 4 == 0 && (((uintptr_t)z | (uintptr_t)table) & (bytes - 1)) == 0;
  const size_t work = (size_t)T * dim / (four ? 4 : 1);
  const unsigned grid = (unsigned)((work + 255) / 256 > 148 * 16 ? 148 * 16 : (work + 255) / 256);
  int rc;
#define RUN(TA) rc = four ? cima_launch(k_token_side_apply4<TA>, dim3(grid), dim3(256), (size_t)0, stream, 1, (TA*)z, (const TA*)table, ldt, tokens, col, work, dim, vocab, act) \
                          : cima_launch(k_token_side_apply<TA>, dim3(grid), dim3(256), (size_t)0, stream, 1, (TA*)z, (const TA*)table, ldt, tokens, col, work, dim, vocab, act)
  if (dtype == CIMA_F32) RUN(float);
  else if (dtype == CIMA_BF16) RUN(__nv_bfloat16);
  else return cima_fail(CIMA_E_DTYPE, "token_side_apply: dtype code %d is neither float32 nor bfloat16", dtype);
#undef RUN
  return rc ? rc : cima_launch_result();
}
