// A token's own input to a layer: z[t, j] = act(sum_k x[t, k] W[j, k]) * D[tok_t, col + j], D the model's side table.
//
// token_side_few    the whole of it for the few rows of a decode step, straight from the float32 stream: a block takes four
//                   outputs j, its eight warps share k in interleaved pieces of 16 bytes a lane and hold the sums of all rows (at
//                   most 8); the lanes are added by a shuffle tree, the warps in their order.  A row's sum does not depend on what
//                   else is in the step.
// token_side_apply  behind a product of many rows: z <- act(z) * D[tok, col + j] in place
#include "common.cuh"

namespace {
constexpr int TS_ROWS = 8, TS_OUTS = 4, TS_WARPS = 8;

template <typename TW> struct TsVec;                          // weights of one 16-byte load
template <> struct TsVec<float> { static constexpr int N = 4; };
template <> struct TsVec<__nv_bfloat16> { static constexpr int N = 8; };

// VEC false: one value a lane at a time (any width, any alignment).
template <typename TW, typename TA, bool VEC>
__global__ void __launch_bounds__(TS_WARPS * 32)
k_token_side_few(const float* __restrict__ x, const TW* __restrict__ w, const TA* __restrict__ table, int ldt, const int* __restrict__ tokens,
                 int col, TA* __restrict__ z, int T, int dim, int W, int vocab, int act) {
  constexpr int V = VEC ? TsVec<TW>::N : 1;
  constexpr int STEP = TS_WARPS * 32 * V;
  __shared__ float part[TS_WARPS][TS_OUTS * TS_ROWS];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int j0 = blockIdx.x * TS_OUTS;
  struct __align__(VEC ? 16 : sizeof(TW)) Piece { TW e[V]; };
  const TW* wr[TS_OUTS];
#pragma unroll
  for (int o = 0; o < TS_OUTS; o++) wr[o] = w + (size_t)min(j0 + o, dim - 1) * W;      // (outputs beyond the last are not stored)
  float acc[TS_OUTS][TS_ROWS];
#pragma unroll
  for (int o = 0; o < TS_OUTS; o++)
#pragma unroll
    for (int r = 0; r < TS_ROWS; r++) acc[o][r] = 0.f;
  // the first weights depend on no kernel: they are requested before the wait
  const int k0 = (warp * 32 + lane) * V;
  Piece c[TS_OUTS];
#pragma unroll
  for (int o = 0; o < TS_OUTS; o++)
    if (k0 < W) c[o] = *reinterpret_cast<const Piece*>(wr[o] + k0);
  cima_pdl_wait();
  for (int k = k0; k < W; k += STEP) {
    float xv[TS_ROWS][V];
#pragma unroll
    for (int r = 0; r < TS_ROWS; r++) {
      if constexpr (VEC) {
#pragma unroll
        for (int q = 0; q < V; q += 4) {
          const float4 f = r < T ? *reinterpret_cast<const float4*>(x + (size_t)r * W + k + q) : make_float4(0.f, 0.f, 0.f, 0.f);
          xv[r][q] = f.x; xv[r][q + 1] = f.y; xv[r][q + 2] = f.z; xv[r][q + 3] = f.w;
        }
      } else {
        xv[r][0] = r < T ? x[(size_t)r * W + k] : 0.f;
      }
    }
#pragma unroll
    for (int o = 0; o < TS_OUTS; o++)
#pragma unroll
      for (int q = 0; q < V; q++) {
        const float wv = cima_to_f32<TW>(c[o].e[q]);
#pragma unroll
        for (int r = 0; r < TS_ROWS; r++) acc[o][r] = fmaf(xv[r][q], wv, acc[o][r]);
      }
    if (k + STEP < W) {
#pragma unroll
      for (int o = 0; o < TS_OUTS; o++) c[o] = *reinterpret_cast<const Piece*>(wr[o] + k + STEP);
    }
  }
  cima_pdl_trigger();
  // 32 sums over the 32 lanes, handed over by halves: after the step of distance d a lane holds half as many sums, of its half
  // of the pairs; in the end lane l holds sum number l, added up over all lanes in a fixed order
  float s[TS_OUTS * TS_ROWS];
#pragma unroll
  for (int o = 0; o < TS_OUTS; o++)
#pragma unroll
    for (int r = 0; r < TS_ROWS; r++) s[o * TS_ROWS + r] = acc[o][r];
#pragma unroll
  for (int d = 16; d > 0; d >>= 1) {
    const bool upper = lane & d;
#pragma unroll
    for (int i = 0; i < d; i++) {
      const float mine = upper ? s[i + d] : s[i], other = upper ? s[i] : s[i + d];
      s[i] = mine + __shfl_xor_sync(0xffffffffu, other, d);
    }
  }
  part[warp][lane] = s[0];
  __syncthreads();
  if (warp == 0) {
    float v = 0.f;
#pragma unroll
    for (int q = 0; q < TS_WARPS; q++) v += part[q][lane];
    const int o = lane / TS_ROWS, r = lane % TS_ROWS;
    if (r < T && j0 + o < dim) {
      int tok = tokens[r];
      tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
      const float e = cima_to_f32<TA>(table[(size_t)tok * ldt + col + j0 + o]);
      z[(size_t)r * dim + j0 + o] = cima_from_f32<TA>(cima_gate_act(v, act) * e);
    }
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
  const bool vec = W % (wdtype == CIMA_F32 ? 4 : 8) == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0;
  const dim3 grid((unsigned)((dim + TS_OUTS - 1) / TS_OUTS));
  int rc;
#define RUN_V(TW, TA, VEC) cima_launch(k_token_side_few<TW, TA, VEC>, grid, dim3(TS_WARPS * 32), (size_t)0, stream, 1, x, (const TW*)w, (const TA*)table, ldt, tokens, col, (TA*)z, T, dim, W, vocab, act)
#define RUN(TW, TA) rc = vec ? RUN_V(TW, TA, true) : RUN_V(TW, TA, false)
  if (wdtype == CIMA_F32 && dtype == CIMA_F32) RUN(float, float);
  else if (wdtype == CIMA_BF16 && dtype == CIMA_BF16) RUN(__nv_bfloat16, __nv_bfloat16);
  else if (wdtype == CIMA_F32 && dtype == CIMA_BF16) RUN(float, __nv_bfloat16);
  else return cima_fail(CIMA_E_DTYPE, "token_side_few: weights of dtype code %d with rows of %d are not accepted", wdtype, dtype);
#undef RUN
#undef RUN_V
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
