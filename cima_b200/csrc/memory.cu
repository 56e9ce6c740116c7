// Linear recurrences whose state is a float32 matrix a head, S [dim, vdim], that nothing reads back before it is written
// (no delta), carried from token to token and from step to step (state [slots, heads, dim, vdim], zeroed when a slot opens):
//
//   channel form   S <- diag(g_t) S + k_t v_t^T;           o_t = S^T (c q_t)        g_t one decay a head and key channel
//   scalar form    S <- a_t S + b_t k_t v_t^T;             o_t = S^T (c q_t)        a_t, b_t one number a head
//                  n <- a_t n + b_t k_t;                   r_t = n . (c q_t)        the normaliser's row beside the matrix
//
// with one constant c.  A block owns 256 CPT / LANES value channels (columns of S) of one (sequence, head): a thread has CPT
// neighbouring columns, LANES lanes of a warp share them, and each keeps its part of the rows in registers (rows 4 LANES ii +
// 4 rg + e of row group rg).  In the scalar form the first block of a head has a ninth warp: it keeps n as one more column
// whose value is 1.  Tokens are walked in order, 16 (8 for key sizes above 128) at a time: the next ones travel from global
// memory into registers while the current ones are worked on from shared memory.  No token's read-out feeds the next
// update, so four tokens are taken together: their updates follow one another row by row, and their sums over the lanes
// are formed in one go.  A token's own arithmetic is the same wherever it stands among them.  Everything is float32 but the
// loads of q, k, v.
//
// Long steps are cut into segments of `seg` tokens that run side by side (three launches):
//   PHASE 1   every segment but a sequence's last, from S = 0, without read-out: what it adds, E, and the product of its
//             decays, D
//   combine   the state in front of every segment: S_0 = the stored state, S_(i+1) = D_i S_i + E_i
//   PHASE 2   every segment from the state in front of it, with read-out; a sequence's last one stores the state
// PHASE 0 is the one launch for steps that are not cut.  The decays are at most 1, so nothing grows and nothing is divided
// by.  A segment's borders depend on the step's rows of its own sequence only.
#include "common.cuh"

namespace {
constexpr int MEM_COL_WARPS = 8;

struct MemArgs {
  const void *q, *k, *v;
  int ldq, ldk, ldv;
  const float* g;              // channel form: [T, heads * dim];  scalar form: [T, heads, 2] = (a, b)
  float* state;                // [slots, heads, dim, vdim]
  float* nstate;               // scalar form: [slots, heads, dim]
  float* buf;                  // segments: [units, heads, dim, vdim]
  float* nbuf;                 // scalar form: [units, heads, dim]
  float* dbuf;                 // products of decays: channel form [units, heads, dim], scalar form [units, heads]
  const int *seq_slot, *seq_first_row;
  float* out;                  // [T, heads * vdim]
  float* nout;                 // scalar form: [T, heads]
  int heads, dim, vdim, seg, max_segs;
  float qscale;
};

template <typename TA, int DIMP, bool SCALAR, int CPT, int LANES, int PHASE>
__global__ void __launch_bounds__(288)
k_memory(const __grid_constant__ MemArgs a) {
  cima_pdl_wait();
  constexpr int RP = DIMP / LANES;                      // rows of a column that one lane keeps
  constexpr int GW = 32 / LANES;                        // groups of columns of a warp
  constexpr int CH = DIMP > 128 ? 8 : 16;               // tokens staged at a time
  constexpr int COLS = MEM_COL_WARPS * GW * CPT;
  constexpr int NLD = CH * DIMP / 256;                  // values of k (and of q, of g) a thread stages
  constexpr int NLV = (CH * COLS + 255) / 256;
  constexpr bool READ = PHASE != 1;
  __shared__ __align__(16) float sk[CH][DIMP];
  __shared__ __align__(16) float sq[READ ? CH : 1][DIMP];
  __shared__ __align__(16) float sg[SCALAR ? 1 : CH][DIMP];
  __shared__ float sv[CH][COLS];
  __shared__ float so[READ ? CH : 1][COLS + 1];         // the last column: the normaliser's sums
  __shared__ float2 sab[CH];
  const int h = blockIdx.y, col0 = blockIdx.x * COLS;
  const int seq = PHASE == 0 ? blockIdx.z : blockIdx.z / a.max_segs;
  const int sidx = PHASE == 0 ? 0 : blockIdx.z - seq * a.max_segs;
  const int all0 = a.seq_first_row[seq], all = a.seq_first_row[seq + 1] - all0;
  const int first = all0 + (PHASE == 0 ? 0 : sidx * a.seg);
  int n = all, last = 1;
  if (PHASE != 0) {
    const int left = all - sidx * a.seg;
    if (left <= 0) return;
    last = left <= a.seg;
    if (PHASE == 1 && last) return;
    n = min(left, a.seg);
  }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rg = lane / GW;
  const bool extra = warp == MEM_COL_WARPS;             // the ninth warp: the normaliser, or (PHASE 1) the decays' product
  const int lc = extra ? 0 : (warp * GW + lane % GW) * CPT;      // the thread's columns are col0 + lc + x
  const int heads = a.heads, dim = a.dim, vdim = a.vdim;
  const TA* q = static_cast<const TA*>(a.q);
  const TA* k = static_cast<const TA*>(a.k);
  const TA* v = static_cast<const TA*>(a.v);
  const size_t unit = PHASE == 0 ? (size_t)a.seq_slot[seq] : (size_t)blockIdx.z;
  float* st = (PHASE == 0 ? a.state : a.buf) + ((unit * heads + h) * dim) * (size_t)vdim + col0 + lc;
  float* nst = SCALAR ? (PHASE == 0 ? a.nstate : a.nbuf) + (unit * heads + h) * dim : nullptr;
  float S[CPT][RP];
#pragma unroll
  for (int x = 0; x < CPT; x++)
#pragma unroll
    for (int j = 0; j < RP; j++) {
      const int row = (j >> 2) * (4 * LANES) + rg * 4 + (j & 3);
      float s = 0.f;
      if (READ && row < dim) {
        if (!extra) { if (col0 + lc + x < vdim) s = st[(size_t)row * vdim + x]; }
        else if (SCALAR && x == 0) s = nst[row];
      }
      S[x][j] = s;
    }
  float D[SCALAR ? 1 : DIMP / 32];                      // the product of the decays (PHASE 1; the ninth warp, a channel every 32)
#pragma unroll
  for (int i = 0; i < (SCALAR ? 1 : DIMP / 32); i++) D[i] = 1.f;

  TA rk[NLD], rq[READ ? NLD : 1], rv[NLV];
  float rgt[SCALAR ? 1 : NLD];
  float2 rab = make_float2(1.f, 0.f);
  const TA zero = cima_from_f32<TA>(0.f);
  auto fetch = [&](int t0) {
    const int nt = min(CH, n - t0);
    if (!extra) {
#pragma unroll
      for (int r = 0; r < NLD; r++) {
        const int idx = tid + r * 256;
        const int tt = idx / DIMP, i = idx - tt * DIMP;
        const size_t row = (size_t)(first + t0 + tt);
        const bool ok = tt < nt && i < dim;
        rk[r] = ok ? k[row * a.ldk + (size_t)h * dim + i] : zero;
        if (READ) rq[r] = ok ? q[row * a.ldq + (size_t)h * dim + i] : zero;
        if (!SCALAR) rgt[r] = ok ? a.g[(row * heads + h) * dim + i] : 1.f;
      }
#pragma unroll
      for (int r = 0; r < NLV; r++) {
        const int idx = tid + r * 256;
        const int tt = idx / COLS, cc = idx - tt * COLS;
        rv[r] = (tt < nt && col0 + cc < vdim) ? v[(size_t)(first + t0 + tt) * a.ldv + (size_t)h * vdim + col0 + cc] : zero;
      }
      if (SCALAR && tid < CH) rab = tid < nt ? *reinterpret_cast<const float2*>(a.g + ((size_t)(first + t0 + tid) * heads + h) * 2) : make_float2(1.f, 0.f);
    }
  };
  if (n > 0) fetch(0);
  for (int t0 = 0; t0 < n; t0 += CH) {
    const int nt = min(CH, n - t0);
    __syncthreads();
    if (!extra) {
#pragma unroll
      for (int r = 0; r < NLD; r++) {
        const int idx = tid + r * 256;
        const int tt = idx / DIMP, i = idx - tt * DIMP;
        sk[tt][i] = cima_to_f32<TA>(rk[r]);
        if (READ) sq[tt][i] = cima_to_f32<TA>(rq[r]) * a.qscale;
        if (!SCALAR) sg[tt][i] = rgt[r];
      }
#pragma unroll
      for (int r = 0; r < NLV; r++) {
        const int idx = tid + r * 256;
        if (idx < CH * COLS) sv[idx / COLS][idx % COLS] = cima_to_f32<TA>(rv[r]);
      }
      if (SCALAR && tid < CH) sab[tid] = rab;
    }
    __syncthreads();
    if (t0 + CH < n) fetch(t0 + CH);
    constexpr int TB = 4;
    const bool works = !extra || (SCALAR && blockIdx.x == 0);
    if (works) {
      for (int tt = 0; tt < nt; tt += TB) {
        float o[TB * CPT];                               // [token][column]
#pragma unroll
        for (int y = 0; y < TB; y++) {
#pragma unroll
          for (int x = 0; x < CPT; x++) o[y * CPT + x] = 0.f;
          if (tt + y < nt) {
            float u[CPT], f = 1.f;
            if (SCALAR) {
              const float2 ab = sab[tt + y];
              f = ab.x;
#pragma unroll
              for (int x = 0; x < CPT; x++) u[x] = (extra ? 1.0f : sv[tt + y][lc + x]) * ab.y;
            } else {
#pragma unroll
              for (int x = 0; x < CPT; x++) u[x] = sv[tt + y][lc + x];
            }
            float p[CPT];
#pragma unroll
            for (int x = 0; x < CPT; x++) p[x] = 0.f;
#pragma unroll
            for (int j = 0; j < RP; j += 4) {
              const int i = (j >> 2) * (4 * LANES) + rg * 4;
              const float4 k4 = *reinterpret_cast<const float4*>(&sk[tt + y][i]);
              float4 g4 = make_float4(f, f, f, f);
              if (!SCALAR) g4 = *reinterpret_cast<const float4*>(&sg[tt + y][i]);
              float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f);
              if (READ) q4 = *reinterpret_cast<const float4*>(&sq[tt + y][i]);
#pragma unroll
              for (int x = 0; x < CPT; x++) {
                S[x][j] = fmaf(k4.x, u[x], g4.x * S[x][j]);
                S[x][j + 1] = fmaf(k4.y, u[x], g4.y * S[x][j + 1]);
                S[x][j + 2] = fmaf(k4.z, u[x], g4.z * S[x][j + 2]);
                S[x][j + 3] = fmaf(k4.w, u[x], g4.w * S[x][j + 3]);
                if (READ) {
                  o[y * CPT + x] = fmaf(S[x][j], q4.x, o[y * CPT + x]); p[x] = fmaf(S[x][j + 1], q4.y, p[x]);
                  o[y * CPT + x] = fmaf(S[x][j + 2], q4.z, o[y * CPT + x]); p[x] = fmaf(S[x][j + 3], q4.w, p[x]);
                }
              }
            }
            if (READ) {
#pragma unroll
              for (int x = 0; x < CPT; x++) o[y * CPT + x] += p[x];
            }
            if (PHASE == 1 && SCALAR) D[0] *= f;
          }
        }
        if (READ) {
          // sums over the LANES lanes of a column group, a tree of pairs over the lanes' distance LANES / 2, ..., 1
          // (as long as a lane has more than one value it keeps one half and hands the other over: in the end it holds one of them)
          int n_own = TB * CPT, base = 0;
#pragma unroll
          for (int m = LANES / 2; m > 0; m >>= 1) {
            if (n_own > 1) {
              n_own >>= 1;
              const bool up = (rg & m) != 0;
              if (up) base += n_own;
#pragma unroll
              for (int i = 0; i < TB * CPT / 2; i++)
                if (i < n_own) {
                  const float keep = up ? o[i + n_own] : o[i], give = up ? o[i] : o[i + n_own];
                  o[i] = keep + __shfl_xor_sync(0xffffffffu, give, m * GW);
                }
            } else {
              o[0] += __shfl_xor_sync(0xffffffffu, o[0], m * GW);
            }
          }
          static_assert(TB * CPT <= LANES, "a lane ends with one value");
          const int y = base / CPT, x = base % CPT;
          if (tt + y < nt) {                              // (lanes with the same value write the same sum)
            if (!extra) so[tt + y][lc + x] = o[0];
            else if (x == 0 && lane % GW == 0) so[tt + y][COLS] = o[0];
          }
        }
      }
    } else if (PHASE == 1 && !SCALAR && blockIdx.x == 0) {
      for (int tt = 0; tt < nt; tt++)
#pragma unroll
        for (int i = 0; i < (SCALAR ? 1 : DIMP / 32); i++) D[i] *= sg[tt][lane + 32 * i];
    }
    if (READ) {
      __syncthreads();
      for (int idx = tid; idx < nt * COLS; idx += blockDim.x) {
        const int tt = idx / COLS, cc = idx - tt * COLS;
        if (col0 + cc < vdim) a.out[((size_t)(first + t0 + tt) * heads + h) * vdim + col0 + cc] = so[tt][cc];
      }
      if (SCALAR && blockIdx.x == 0 && tid < nt) a.nout[(size_t)(first + t0 + tid) * heads + h] = so[tid][COLS];
    }
  }
  cima_pdl_trigger();        // the tokens are done: the next kernel may be set up while the state is stored
  if (PHASE == 2) {
    if (!last) return;       // only the state behind the sequence's last token is kept
    const size_t slot = (size_t)a.seq_slot[seq];
    st = a.state + ((slot * heads + h) * dim) * (size_t)vdim + col0 + lc;
    nst = SCALAR ? a.nstate + (slot * heads + h) * dim : nullptr;
  }
#pragma unroll
  for (int x = 0; x < CPT; x++)
#pragma unroll
    for (int j = 0; j < RP; j++) {
      const int row = (j >> 2) * (4 * LANES) + rg * 4 + (j & 3);
      if (row < dim) {
        if (!extra) { if (col0 + lc + x < vdim) st[(size_t)row * vdim + x] = S[x][j]; }
        else if (SCALAR && x == 0 && blockIdx.x == 0 && lane % GW == 0) nst[row] = S[x][j];
      }
    }
  if (PHASE == 1 && extra && blockIdx.x == 0) {
    if (SCALAR) {
      if (lane == 0) a.dbuf[unit * heads + h] = D[0];
    } else {
#pragma unroll
      for (int i = 0; i < (SCALAR ? 1 : DIMP / 32); i++)
        if (lane + 32 * i < dim) a.dbuf[(unit * heads + h) * dim + lane + 32 * i] = D[i];
    }
  }
}

// buf (and nbuf) turn from what every segment adds into the state in front of it.  A thread an element of a head's state.
template <bool SCALAR>
__global__ void __launch_bounds__(256)
k_memory_combine(const __grid_constant__ MemArgs a) {
  cima_pdl_wait();
  const int per = a.dim * a.vdim, total = per + (SCALAR ? a.dim : 0);
  const int e = blockIdx.x * 256 + threadIdx.x, h = blockIdx.y, seq = blockIdx.z;
  if (e >= total) return;
  const int rows = a.seq_first_row[seq + 1] - a.seq_first_row[seq];
  const int segs = (rows + a.seg - 1) / a.seg;
  const size_t slot = (size_t)a.seq_slot[seq];
  const bool is_n = e >= per;
  const size_t size = is_n ? a.dim : per;
  const int off = is_n ? e - per : e;
  float* base = is_n ? a.nbuf : a.buf;
  const float* from = is_n ? a.nstate : a.state;
  const int chan = off / a.vdim;
  float S = from[(slot * a.heads + h) * size + off];
  for (int s0 = 0; s0 < segs; s0 += 8) {                 // eight segments' values requested before the first is used
    float E[8], D[8];
#pragma unroll
    for (int i = 0; i < 8; i++) {
      const int s = s0 + i;
      const size_t unit = (size_t)seq * a.max_segs + (s < segs - 1 ? s : 0);
      const bool ok = s < segs - 1;                       // what the last segment adds was not made
      E[i] = ok ? base[(unit * a.heads + h) * size + off] : 0.f;
      D[i] = ok ? (SCALAR ? a.dbuf[unit * a.heads + h] : a.dbuf[(unit * a.heads + h) * a.dim + chan]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 8; i++) {
      const int s = s0 + i;
      if (s < segs) base[(((size_t)seq * a.max_segs + s) * a.heads + h) * size + off] = S;
      S = fmaf(D[i], S, E[i]);
    }
  }
}

template <typename TA, bool SCALAR, int PHASE>
int launch_memory(const MemArgs& a, int n_units, cudaStream_t stream) {
  // PHASE 0 (few tokens a sequence, or many sequences): 32 columns a block, so that more blocks share the state's traffic.
  // Segments: 64 columns, two a thread, so that a read of k, q and g from shared memory serves both (four a thread over 16
  // lanes measured the same: the kernel issues 0.6 to 0.7 instructions a cycle and scheduler either way).
  constexpr int CPT = PHASE == 0 ? 1 : 2;
  constexpr int cols = 32 * CPT;
  const dim3 grid((unsigned)((a.vdim + cols - 1) / cols), (unsigned)a.heads, (unsigned)n_units);
  const dim3 block(SCALAR || PHASE == 1 ? 288 : 256);
#define RUN(D) return cima_launch(k_memory<TA, D, SCALAR, CPT, 8, PHASE>, grid, block, (size_t)0, stream, 1, a)
  if (a.dim <= 32) RUN(32);
  if (a.dim <= 64) RUN(64);
  if (a.dim <= 128) RUN(128);
  RUN(256);
#undef RUN
}

template <typename TA, bool SCALAR>
int run_memory(const MemArgs& a, int n_seqs, cudaStream_t stream) {
  if (a.max_segs <= 1) return launch_memory<TA, SCALAR, 0>(a, n_seqs, stream);
  if (int rc = launch_memory<TA, SCALAR, 1>(a, n_seqs * a.max_segs, stream)) return rc;
  const unsigned blocks = (unsigned)((a.dim * (a.vdim + (SCALAR ? 1 : 0)) + 255) / 256);
  if (int rc = cima_launch(k_memory_combine<SCALAR>, dim3(blocks, (unsigned)a.heads, (unsigned)n_seqs), dim3(256), (size_t)0, stream, 1, a)) return rc;
  return launch_memory<TA, SCALAR, 2>(a, n_seqs * a.max_segs, stream);
}

// The decays of the channel form from a low-rank projection: g = sigmoid(W2 a + b)^(1 / tau), a thread a channel for
// ROWS rows at a time, the row's rank values in shared memory.
constexpr int DECAY_ROWS = 8;
// (the logarithm's absolute error decides the factor's relative one, so log(1 + e) serves where log1p would cost twice as much)
__device__ __forceinline__ float decay_of(float z, float inv_tau) { return expf((fminf(z, 0.f) - logf(1.0f + expf(-fabsf(z)))) * inv_tau); }
template <typename TA, typename TW>
__global__ void __launch_bounds__(128)
k_channel_decay(const TA* __restrict__ a1, int lda, const TW* __restrict__ w2, const float* __restrict__ bias, float inv_tau,
                float* __restrict__ g, int T, int rank, int channels) {
  cima_pdl_wait();
  cima_pdl_trigger();
  extern __shared__ float sa[];                          // [rank][DECAY_ROWS]
  const int row0 = blockIdx.y * DECAY_ROWS;
  for (int idx = threadIdx.x; idx < rank * DECAY_ROWS; idx += 128) {
    const int r = idx / rank, i = idx - r * rank;
    sa[i * DECAY_ROWS + r] = row0 + r < T ? cima_to_f32<TA>(a1[(size_t)(row0 + r) * lda + i]) : 0.f;
  }
  const int c = blockIdx.x * 128 + threadIdx.x;
  __syncthreads();
  if (c >= channels) return;
  float acc[DECAY_ROWS];
#pragma unroll
  for (int r = 0; r < DECAY_ROWS; r++) acc[r] = 0.f;
  const TW* wp = w2 + (size_t)c * rank;
  for (int i0 = 0; i0 < rank; i0 += 8) {
    float w[8];
#pragma unroll
    for (int i = 0; i < 8; i++) w[i] = i0 + i < rank ? cima_to_f32<TW>(wp[i0 + i]) : 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++)
      if (i0 + i < rank) {
#pragma unroll
        for (int r = 0; r < DECAY_ROWS; r++) acc[r] = fmaf(w[i], sa[(i0 + i) * DECAY_ROWS + r], acc[r]);
      }
  }
  const float b = bias[c];
#pragma unroll
  for (int r = 0; r < DECAY_ROWS; r++)
    if (row0 + r < T) g[(size_t)(row0 + r) * channels + c] = decay_of(acc[r] + b, inv_tau);
}

// The same for ranks of at most 16: the channel's weights stay in registers, and a block takes DECAY_GROUPS times as many rows.
constexpr int DECAY_GROUPS = 4;
template <typename TA, typename TW>
__global__ void __launch_bounds__(128)
k_channel_decay16(const TA* __restrict__ a1, int lda, const TW* __restrict__ w2, const float* __restrict__ bias, float inv_tau,
                  float* __restrict__ g, int T, int rank, int channels, int rows_per_block) {
  const int c = blockIdx.x * 128 + threadIdx.x;
  const int cc = min(c, channels - 1);
  float w[16];                                           // weights and bias do not depend on the kernel in front
#pragma unroll
  for (int i = 0; i < 16; i++) w[i] = i < rank ? cima_to_f32<TW>(w2[(size_t)cc * rank + i]) : 0.f;
  const float b = bias[cc];
  cima_pdl_wait();
  cima_pdl_trigger();
  __shared__ __align__(16) float sa[16][DECAY_ROWS * DECAY_GROUPS];
  const int row0 = blockIdx.y * rows_per_block, rows = min(rows_per_block, T - row0);
  for (int idx = threadIdx.x; idx < 16 * rows_per_block; idx += 128) {
    const int r = idx >> 4, i = idx & 15;
    sa[i][r] = r < rows && i < rank ? cima_to_f32<TA>(a1[(size_t)(row0 + r) * lda + i]) : 0.f;
  }
  __syncthreads();
  if (c >= channels) return;
  for (int r0 = 0; r0 < rows; r0 += 4) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < 16; i++) {
      const float4 x = *reinterpret_cast<const float4*>(&sa[i][r0]);
      acc[0] = fmaf(w[i], x.x, acc[0]); acc[1] = fmaf(w[i], x.y, acc[1]);
      acc[2] = fmaf(w[i], x.z, acc[2]); acc[3] = fmaf(w[i], x.w, acc[3]);
    }
#pragma unroll
    for (int r = 0; r < 4; r++)
      if (r0 + r < rows) g[(size_t)(row0 + r0 + r) * channels + c] = decay_of(acc[r] + b, inv_tau);
  }
}

// The scalar form's numbers from the gates' projections, with a running maximum m a head (state [slots, heads]):
//   i = cap tanh((zi + bi) / cap),  f = log sigmoid(cap tanh((zf + bf) / cap));   m' = max(f + m, i)
//   (a, b) = (exp(f + m - m'), exp(i - m')),   floor = exp(-m')
// A warp a (sequence, head), 32 tokens at a time: a lane a token for the gates and the exponentials, every lane the same
// chain of maxima in the tokens' order (so m has the same bits in every cutting).
template <typename TA>
__global__ void __launch_bounds__(128)
k_scalar_gates(const TA* __restrict__ z, int ldz, const float* __restrict__ bi, const float* __restrict__ bf, float cap,
               float* __restrict__ mstate, const int* __restrict__ seq_slot, const int* __restrict__ seq_first_row,
               float* __restrict__ ab, float* __restrict__ floor_, int n_seqs, int heads) {
  cima_pdl_wait();
  cima_pdl_trigger();
  __shared__ float2 fi[4][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int u = blockIdx.x * 4 + warp;
  if (u >= n_seqs * heads) return;
  const int seq = u / heads, h = u - seq * heads;
  const int first = seq_first_row[seq], n = seq_first_row[seq + 1] - first;
  float* mp = mstate + (size_t)seq_slot[seq] * heads + h;
  float m = *mp;
  const float b_i = bi[h], b_f = bf[h], inv = 1.0f / cap;
  auto zi_of = [&](int t) { return t < n ? cima_to_f32<TA>(z[(size_t)(first + t) * ldz + h]) : 0.f; };
  auto zf_of = [&](int t) { return t < n ? cima_to_f32<TA>(z[(size_t)(first + t) * ldz + heads + h]) : 0.f; };
  float zi = zi_of(lane), zf = zf_of(lane);
  for (int t0 = 0; t0 < n; t0 += 32) {
    const int nt = min(32, n - t0);
    const float i = cap * tanhf((zi + b_i) * inv);
    const float f = cima_log_sigmoid(cap * tanhf((zf + b_f) * inv));
    zi = zi_of(t0 + 32 + lane);
    zf = zf_of(t0 + 32 + lane);
    __syncwarp();
    fi[warp][lane] = lane < nt ? make_float2(f, i) : make_float2(0.f, -INFINITY);      // behind the end: m stays
    __syncwarp();
    float before = m, after = m;
#pragma unroll
    for (int t = 0; t < 32; t++) {
      const float2 x = fi[warp][t];
      const float next = fmaxf(x.x + m, x.y);
      if (t == lane) { before = m; after = next; }
      m = next;
    }
    if (lane < nt) {
      const size_t at = (size_t)(first + t0 + lane) * heads + h;
      *reinterpret_cast<float2*>(ab + at * 2) = make_float2(expf(f + before - after), expf(i - after));
      floor_[at] = expf(-after);
    }
  }
  if (lane == 0) *mp = m;
}

// The same for many tokens a sequence: a block a (sequence, head).  Seven warps make a tile's gates and, two tiles later, its
// exponentials; between them the first warp walks the chain of maxima, which is the same chain in the same order.
constexpr int GATE_TILE = 224;
template <typename TA>
__global__ void __launch_bounds__(256)
k_scalar_gates_long(const TA* __restrict__ z, int ldz, const float* __restrict__ bi, const float* __restrict__ bf, float cap,
                    float* __restrict__ mstate, const int* __restrict__ seq_slot, const int* __restrict__ seq_first_row,
                    float* __restrict__ ab, float* __restrict__ floor_, int heads) {
  cima_pdl_wait();
  cima_pdl_trigger();
  __shared__ float2 fi[3][GATE_TILE];
  __shared__ float mm[2][GATE_TILE + 1];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int first = seq_first_row[seq], n = seq_first_row[seq + 1] - first;
  const int tiles = (n + GATE_TILE - 1) / GATE_TILE;
  float* mp = mstate + (size_t)seq_slot[seq] * heads + h;
  const float b_i = bi[h], b_f = bf[h], inv = 1.0f / cap;
  float m = *mp;
  for (int it = 0; it < tiles + 2; it++) {
    if (tid >= 32) {
      const int w = tid - 32;
      if (it < tiles) {
        const int t = it * GATE_TILE + w;
        float2 x = make_float2(0.f, -INFINITY);          // behind the end: m stays
        if (t < n) {
          const TA* zp = z + (size_t)(first + t) * ldz + h;
          x.y = cap * tanhf((cima_to_f32<TA>(zp[0]) + b_i) * inv);
          x.x = cima_log_sigmoid(cap * tanhf((cima_to_f32<TA>(zp[heads]) + b_f) * inv));
        }
        fi[it % 3][w] = x;
      }
      const int j = it - 2, t = j * GATE_TILE + w;
      if (j >= 0 && t < n) {
        const float2 x = fi[j % 3][w];
        const float before = mm[j & 1][w], after = mm[j & 1][w + 1];
        const size_t at = (size_t)(first + t) * heads + h;
        *reinterpret_cast<float2*>(ab + at * 2) = make_float2(expf(x.x + before - after), expf(x.y - after));
        floor_[at] = expf(-after);
      }
    } else if (it >= 1 && it <= tiles) {
      const int j = it - 1;
      if (tid == 0) mm[j & 1][0] = m;
      // sixteen tokens' gates in registers, the next sixteen on their way; a lane keeps its token's maximum
      constexpr int U = 16;
      float2 x[U], nx[U];
#pragma unroll
      for (int u = 0; u < U; u++) nx[u] = fi[j % 3][u];
      for (int t = 0; t < GATE_TILE; t += U) {
#pragma unroll
        for (int u = 0; u < U; u++) x[u] = nx[u];
        if (t + U < GATE_TILE) {
#pragma unroll
          for (int u = 0; u < U; u++) nx[u] = fi[j % 3][t + U + u];
        }
        float mine = m;
#pragma unroll
        for (int u = 0; u < U; u++) {
          m = fmaxf(x[u].x + m, x[u].y);
          if (u == tid) mine = m;
        }
        if (tid < U) mm[j & 1][t + tid + 1] = mine;
      }
    }
    __syncthreads();
  }
  if (tid == 0) *mp = m;
}
}  // namespace

// q, k [T, >= heads * dim], v [T, >= heads * vdim] of one dtype (rows of ldq / ldk / ldv values).  scalar 0: g [T, heads * dim] the
// channels' decays; scalar 1: g [T, heads, 2] the pairs (a, b), with nstate [slots, heads, dim] and nout [T, heads].  out [T, heads * vdim]
// float32.  max_segs > 1 cuts every sequence's rows into segments of seg tokens (at most max_segs of them) and needs buf
// [n_seqs * max_segs, heads, dim, vdim], dbuf [n_seqs * max_segs, heads(, dim)] and, scalar, nbuf [n_seqs * max_segs, heads, dim].
extern "C" int cima_memory(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, int dtype, const float* g, int scalar,
                           float* state, float* nstate, const int* seq_slot, const int* seq_first_row, float* out, float* nout,
                           float qscale, int T, int n_seqs, int heads, int dim, int vdim, int seg, int max_segs, float* buf,
                           float* nbuf, float* dbuf, cudaStream_t stream) {
  if (T <= 0 || n_seqs <= 0) return 0;
  if (max_segs < 1) max_segs = 1;
  if (heads <= 0 || heads > 65535 || (long long)n_seqs * max_segs > 65535)
    return cima_fail(CIMA_E_SIZE, "memory: %d heads in %d sequences of %d segments exceed one launch", heads, n_seqs, max_segs);
  if (dim <= 0 || dim > 256 || vdim <= 0) return cima_fail(CIMA_E_SIZE, "memory: key size %d must lie in 1..256 and value size %d be positive", dim, vdim);
  if (!q || !k || !v || !g || !state || !out || (scalar && (!nstate || !nout))) return cima_fail(CIMA_E_ARG, "memory: q, k, v, the decays, the state and the output are needed");
  if (max_segs > 1 && (seg <= 0 || !buf || !dbuf || (scalar && !nbuf))) return cima_fail(CIMA_E_ARG, "memory: segments of %d tokens need their buffers", seg);
  const MemArgs a{q, k, v, ldq, ldk, ldv, g, state, nstate, buf, nbuf, dbuf, seq_slot, seq_first_row, out, nout, heads, dim, vdim, seg, max_segs, qscale};
  int rc;
  if (dtype == CIMA_F32) rc = scalar ? run_memory<float, true>(a, n_seqs, stream) : run_memory<float, false>(a, n_seqs, stream);
  else if (dtype == CIMA_BF16) rc = scalar ? run_memory<__nv_bfloat16, true>(a, n_seqs, stream) : run_memory<__nv_bfloat16, false>(a, n_seqs, stream);
  else return cima_fail(CIMA_E_DTYPE, "memory: dtype code %d is neither float32 nor bfloat16", dtype);
  return rc ? rc : cima_launch_result();
}

// a1 [T, lda] (adtype): the rank values of a row; w2 [channels, rank] (wdtype); g [T, channels] float32.
extern "C" int cima_channel_decay(const void* a1, int adtype, int lda, const void* w2, int wdtype, const float* bias, float inv_tau,
                                  float* g, int T, int rank, int channels, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rank <= 0 || rank > 1024 || channels <= 0) return cima_fail(CIMA_E_SIZE, "channel_decay: rank %d must lie in 1..1024 and %d channels be positive", rank, channels);
  if ((T + DECAY_ROWS - 1) / DECAY_ROWS > 65535) return cima_fail(CIMA_E_SIZE, "channel_decay: %d rows exceed one launch; the caller cuts them", T);
  const dim3 grid((unsigned)((channels + 127) / 128), (unsigned)((T + DECAY_ROWS - 1) / DECAY_ROWS));
  const size_t smem = (size_t)rank * DECAY_ROWS * sizeof(float);
  int rc;
  const int per = T <= 64 ? DECAY_ROWS : DECAY_ROWS * DECAY_GROUPS;      // (few rows: more blocks; a row's sum is the same either way)
  const dim3 grid16(grid.x, (unsigned)((T + per - 1) / per));
#define RUN(TA, TW) rc = rank <= 16 ? cima_launch(k_channel_decay16<TA, TW>, grid16, dim3(128), (size_t)0, stream, 1, (const TA*)a1, lda, (const TW*)w2, bias, inv_tau, g, T, rank, channels, per) \
                                    : cima_launch(k_channel_decay<TA, TW>, grid, dim3(128), smem, stream, 1, (const TA*)a1, lda, (const TW*)w2, bias, inv_tau, g, T, rank, channels)
  if (adtype == CIMA_F32 && wdtype == CIMA_F32) RUN(float, float);
  else if (adtype == CIMA_F32 && wdtype == CIMA_BF16) RUN(float, __nv_bfloat16);
  else if (adtype == CIMA_BF16 && wdtype == CIMA_BF16) RUN(__nv_bfloat16, __nv_bfloat16);
  else if (adtype == CIMA_BF16 && wdtype == CIMA_F32) RUN(__nv_bfloat16, float);
  else return cima_fail(CIMA_E_DTYPE, "channel_decay: dtype codes %d and %d are not float32 or bfloat16", adtype, wdtype);
#undef RUN
  return rc ? rc : cima_launch_result();
}

// max_rows: most rows of a sequence (from 128 on a block walks a head's tokens in tiles; the numbers are the same).
// z [T, ldz]: the input gates' projections of all heads, then the forget gates'; ab [T, heads, 2] and floor [T, heads] float32.
extern "C" int cima_scalar_gates(const void* z, int dtype, int ldz, const float* bi, const float* bf, float cap, float* mstate,
                                 const int* seq_slot, const int* seq_first_row, float* ab, float* floor_, int T, int n_seqs, int heads,
                                 int max_rows, cudaStream_t stream) {
  if (T <= 0 || n_seqs <= 0) return 0;
  if (heads <= 0 || !(cap > 0.f) || ldz < 2 * heads) return cima_fail(CIMA_E_SIZE, "scalar_gates: %d heads in rows of %d values, cap %g: the cap must be positive and a row hold two values a head", heads, ldz, (double)cap);
  const dim3 grid((unsigned)(((long long)n_seqs * heads + 3) / 4));
  int rc;
  if (max_rows >= 128 && n_seqs <= 65535) {
    const dim3 blocks((unsigned)heads, (unsigned)n_seqs);
    if (dtype == CIMA_F32) rc = cima_launch(k_scalar_gates_long<float>, blocks, dim3(256), (size_t)0, stream, 1, (const float*)z, ldz, bi, bf, cap, mstate, seq_slot, seq_first_row, ab, floor_, heads);
    else if (dtype == CIMA_BF16) rc = cima_launch(k_scalar_gates_long<__nv_bfloat16>, blocks, dim3(256), (size_t)0, stream, 1, (const __nv_bfloat16*)z, ldz, bi, bf, cap, mstate, seq_slot, seq_first_row, ab, floor_, heads);
    else return cima_fail(CIMA_E_DTYPE, "scalar_gates: dtype code %d is neither float32 nor bfloat16", dtype);
    return rc ? rc : cima_launch_result();
  }
  if (dtype == CIMA_F32) rc = cima_launch(k_scalar_gates<float>, grid, dim3(128), (size_t)0, stream, 1, (const float*)z, ldz, bi, bf, cap, mstate, seq_slot, seq_first_row, ab, floor_, n_seqs, heads);
  else if (dtype == CIMA_BF16) rc = cima_launch(k_scalar_gates<__nv_bfloat16>, grid, dim3(128), (size_t)0, stream, 1, (const __nv_bfloat16*)z, ldz, bi, bf, cap, mstate, seq_slot, seq_first_row, ab, floor_, n_seqs, heads);
  else return cima_fail(CIMA_E_DTYPE, "scalar_gates: dtype code %d is neither float32 nor bfloat16", dtype);
  return rc ? rc : cima_launch_result();
}
