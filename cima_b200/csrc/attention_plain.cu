// Plain causal grouped-query attention: one warp per (query row, head), keys visited one by one
// with a running (max, sum, accumulator) in float32.  It is the attention of the true 32-bit path
// and the fallback for head sizes the fast kernels do not take.  Two sources of keys and values:
//   step  - the step's own qkv buffer (a prompt that starts at position 0: key j of a sequence is
//           its row j), used for prefill;
//   cache - the layer's pages through the slot's block table, used for decoding.
// Head h reads kv head h / (heads / kv_heads); score = q.k * scale; a query at position p sees
// keys j <= p, and with window w > 0 only p - j < w (src/kernels.cu:458-491, :700-712); with `keep_first` f > 0 the
// first f positions stay visible beyond the window (at their own positions).  `v_group` neighbouring key heads share
// one value head (1: a value head for every key head): value head = key head / v_group, and a row of the step holds
// nkv / v_group value heads behind its key heads.
// A head's softmax may hold one more entry without a value: `sink` entries of score 0, or exp(head_sink[h]).
// `gate_col` > 0: the row's own buffer holds a gate value for every value of the result from that column on (heads of hd
// values like the queries'); the result leaves times the gate's sigmoid.
// `slopes` (or null), one number a head: slopes[h] * (p - j) is taken off the scaled score of key j for a query at position p.
// A row's result depends only on its own sequence: same bits alone or in any batch.
#include "common.cuh"

template <typename TA, bool FROM_CACHE, int NI>       // NI: values of a head per lane (head_dim <= 32 NI)
__global__ void __launch_bounds__(128)
k_attention_plain(const TA* __restrict__ qkv, int ld, const TA* __restrict__ cache, CimaPaged pg,
                  const int* __restrict__ row_pos, const int* __restrict__ row_seq,
                  const int* __restrict__ seq_slot, const int* __restrict__ seq_first_row,
                  TA* __restrict__ out, int ldo, int T, int nh, int nkv, int hd, float scale, int window, float sink, int keep_first, int v_group,
                  const float* __restrict__ head_sink, int gate_col, const float* __restrict__ slopes) {
  cima_pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int row = blockIdx.x * (blockDim.x >> 5) + warp;
  const int h = blockIdx.y;
  if (row >= T) return;
  const int kvh = h / (nh / nkv);
  const int pos = row_pos[row];
  const int seq = row_seq[row];
  const int slot = FROM_CACHE ? seq_slot[seq] : 0;
  const int first = FROM_CACHE ? 0 : seq_first_row[seq];
  const int vh = kvh / v_group;
  const int kcol = (nh + kvh) * hd, vcol = (nh + nkv + vh) * hd;

  float q[NI], acc[NI];
  const TA* qp = qkv + (size_t)row * ld + (size_t)h * hd;
#pragma unroll
  for (int i = 0; i < NI; i++) {
    const int d = lane + 32 * i;
    q[i] = d < hd ? cima_to_f32<TA>(qp[d]) : 0.f;
    acc[i] = 0.f;
  }
  const float slope = slopes ? slopes[h] : 0.f;
  float m = -1e30f, l = 0.f;
  const int lo = (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;
  const int kept = min(keep_first, lo);         // the first positions that stay visible below the window
  for (int j = kept > 0 ? 0 : lo; j <= pos; j++) {
    if (j == kept && j < lo) j = lo;
    const TA *kp, *vp;
    if (FROM_CACHE) {
      kp = cache + pg.offset(slot, j, 0, kvh);
      vp = cache + pg.offset(slot, j, 1, vh);
    } else {
      kp = qkv + (size_t)(first + j) * ld + kcol;
      vp = qkv + (size_t)(first + j) * ld + vcol;
    }
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NI; i++) {
      const int d = lane + 32 * i;
      if (d < hd) s = fmaf(q[i], cima_to_f32<TA>(kp[d]), s);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    s = s * scale - slope * (float)(pos - j);
    const float m2 = fmaxf(m, s);
    const float corr = expf(m - m2), p = expf(s - m2);
#pragma unroll
    for (int i = 0; i < NI; i++) {
      const int d = lane + 32 * i;
      if (d < hd) acc[i] = acc[i] * corr + p * cima_to_f32<TA>(vp[d]);
    }
    l = l * corr + p;
    m = m2;
  }
  TA* op = out + (size_t)row * ldo + (size_t)h * hd;
  // `sink` entries of score 0 that carry no value (0: an ordinary softmax); or, with `head_sink`, one entry whose score is
  // the head's own number (neither scaled nor attached to a value)
  l += head_sink ? expf(head_sink[h] - m) : sink * expf(-m);
  const float inv = l > 0.f ? 1.0f / l : 0.f;
#pragma unroll
  for (int i = 0; i < NI; i++) {
    const int d = lane + 32 * i;
    if (d < hd) {
      const float gate = gate_col > 0 ? cima_sigmoid(cima_to_f32<TA>(qkv[(size_t)row * ld + gate_col + (size_t)h * hd + d])) : 1.0f;
      op[d] = cima_from_f32<TA>(acc[i] * inv * gate);
    }
  }
}

// from_cache 0: keys/values of the step (seq_first_row needed); 1: of the cache (table, seq_slot needed).
extern "C" int cima_attention_plain(const void* qkv, int dtype, int ld, const void* cache, const int* table,
                                    int table_width, int ring, int page_size, const int* row_pos,
                                    const int* row_seq, const int* seq_slot, const int* seq_first_row, void* out,
                                    int ldo, int T, int nh, int nkv, int hd, float scale, int window,
                                    int from_cache, int planes, float sink, int keep_first, int v_group, const float* head_sink,
                                    int gate_col, const float* slopes, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (hd <= 0 || hd > 1024) return cima_fail(CIMA_E_SIZE, "attention_plain: head_dim %d is outside 1..1024", hd);
  if (planes != 1 && planes != 2) return cima_fail(CIMA_E_ARG, "attention_plain: %d planes; pages hold keys | values (2) or one shared vector (1)", planes);
  if (nh <= 0 || nkv <= 0 || nh % nkv) return cima_fail(CIMA_E_SIZE, "attention_plain: %d heads are not a multiple of %d kv heads", nh, nkv);
  if (nh > 65535) return cima_fail(CIMA_E_SIZE, "attention_plain: %d heads exceed one launch", nh);
  if (keep_first < 0 || v_group < 1 || nkv % v_group) return cima_fail(CIMA_E_ARG, "attention_plain: keep_first %d must not be negative and %d kv heads be a multiple of v_group %d", keep_first, nkv, v_group);
  if (from_cache && (!cache || !table)) return cima_fail(CIMA_E_ARG, "attention_plain: decoding needs the cache and its block table");
  if (gate_col < 0 || (gate_col > 0 && gate_col + nh * hd > ld)) return cima_fail(CIMA_E_ARG, "attention_plain: %d gate values from column %d on exceed the rows of %d", nh * hd, gate_col, ld);
  CimaPaged pg{table, table_width, ring, page_size, nkv, hd, planes};
  dim3 grid((T + 3) / 4, nh);
#define LAUNCH(TA, FC) { int rc_ = hd <= 256 ? LAUNCH_NI(TA, FC, 8) : LAUNCH_NI(TA, FC, 32); if (rc_) return rc_; }
#define LAUNCH_NI(TA, FC, NI) cima_launch(k_attention_plain<TA, FC, NI>, dim3(grid), dim3(128), (size_t)(0), stream, 1, (const TA*)qkv, ld, (const TA*)cache, pg, \
    row_pos, row_seq, seq_slot, seq_first_row, (TA*)out, ldo, T, nh, nkv, hd, scale, window, sink, keep_first, v_group, head_sink, gate_col, slopes)
  if (dtype == CIMA_F32) { if (from_cache) LAUNCH(float, true) else LAUNCH(float, false) }
  else if (dtype == CIMA_BF16) { if (from_cache) LAUNCH(__nv_bfloat16, true) else LAUNCH(__nv_bfloat16, false) }
  else return cima_fail(CIMA_E_DTYPE, "attention_plain: dtype code %d is neither float32 nor bfloat16", dtype);
#undef LAUNCH
#undef LAUNCH_NI
  return cima_launch_result();
}
