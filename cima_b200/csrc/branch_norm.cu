// The norm on a sublayer's output, in front of the sum (post-norm inside the branch):
//   x <- x + y / sqrt(mean(y^2) + eps) * w                      x, y [T, W] float32, x in place
// and, in the same pass, the rows that the next reader takes: h = x in another dtype, or with a second norm's weight w2
//   h = x / sqrt(mean(x^2) + eps2) * w2
// A block a row.  Rows whose width is a multiple of 4 are kept in registers between the sums and the stores (NV groups of
// four columns a thread, every load requested before the first use); any other width walks column by column.  All sums
// in a fixed order.
#include "common.cuh"

namespace {
template <typename TH>
__device__ __forceinline__ void store4(TH* p, float4 v) {
  if constexpr (sizeof(TH) == 2) {
    uint2 t;
    __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&t);
    h2[0] = __floats2bfloat162_rn(v.x, v.y);
    h2[1] = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = t;
  } else {
    *reinterpret_cast<float4*>(p) = v;
  }
}

template <typename TH, int NV>
__global__ void __launch_bounds__(256)
k_branch_norm4(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, TH* __restrict__ h,
               const float* __restrict__ w2, int W4, float eps, float eps2) {
  cima_pdl_wait();
  cima_pdl_trigger();
  __shared__ float red[32];
  const size_t row = blockIdx.x;
  float4* xr = reinterpret_cast<float4*>(x) + row * W4;
  const float4* yr = reinterpret_cast<const float4*>(y) + row * W4;
  float4 xv[NV], yv[NV], wv[NV];
#pragma unroll
  for (int j = 0; j < NV; j++) {
    const int c = min((int)(threadIdx.x + j * blockDim.x), W4 - 1);        // (beyond the row: its last columns, which are then not used)
    yv[j] = yr[c];
    xv[j] = xr[c];
    wv[j] = reinterpret_cast<const float4*>(w)[c];
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; j++)
    if ((int)(threadIdx.x + j * blockDim.x) < W4)
      ss += fmaf(yv[j].x, yv[j].x, yv[j].y * yv[j].y) + fmaf(yv[j].z, yv[j].z, yv[j].w * yv[j].w);
  ss = cima_block_sum(ss, red);
  const float W = 4.0f * (float)W4;
  const float r = 1.0f / sqrtf(ss / W + eps);
  float s2 = 0.f;
#pragma unroll
  for (int j = 0; j < NV; j++) {
    const int c = threadIdx.x + j * blockDim.x;
    xv[j].x += yv[j].x * r * wv[j].x;
    xv[j].y += yv[j].y * r * wv[j].y;
    xv[j].z += yv[j].z * r * wv[j].z;
    xv[j].w += yv[j].w * r * wv[j].w;
    if (c < W4) {
      xr[c] = xv[j];
      if (h && !w2) store4<TH>(h + (row * W4 + c) * 4, xv[j]);
      s2 += fmaf(xv[j].x, xv[j].x, xv[j].y * xv[j].y) + fmaf(xv[j].z, xv[j].z, xv[j].w * xv[j].w);
    }
  }
  if (!w2) return;
  s2 = cima_block_sum(s2, red);
  const float r2 = 1.0f / sqrtf(s2 / W + eps2);
#pragma unroll
  for (int j = 0; j < NV; j++) {
    const int c = threadIdx.x + j * blockDim.x;
    if (c < W4) {
      const float4 v = reinterpret_cast<const float4*>(w2)[c];
      store4<TH>(h + (row * W4 + c) * 4, make_float4(xv[j].x * r2 * v.x, xv[j].y * r2 * v.y, xv[j].z * r2 * v.z, xv[j].w * r2 * v.w));
    }
  }
}

template <typename TH>
__global__ void __launch_bounds__(256)
k_branch_norm(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, TH* __restrict__ h,
              const float* __restrict__ w2, int W, float eps, float eps2) {
  cima_pdl_wait();
  cima_pdl_trigger();
  __shared__ float red[32];
  const size_t base = (size_t)blockIdx.x * W;
  float ss = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) ss = fmaf(y[base + c], y[base + c], ss);
  ss = cima_block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / (float)W + eps);
  float s2 = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const float v = x[base + c] + y[base + c] * r * w[c];
    x[base + c] = v;
    if (h && !w2) h[base + c] = cima_from_f32<TH>(v);
    s2 = fmaf(v, v, s2);
  }
  if (!w2) return;
  s2 = cima_block_sum(s2, red);
  const float r2 = 1.0f / sqrtf(s2 / (float)W + eps2);
  for (int c = threadIdx.x; c < W; c += blockDim.x) h[base + c] = cima_from_f32<TH>(x[base + c] * r2 * w2[c]);      // (each thread reads what it wrote)
}

template <typename TH>
int launch_branch_norm(float* x, const float* y, const float* w, void* h, const float* w2, int T, int W, float eps, float eps2, cudaStream_t stream) {
  const bool vec = W % 4 == 0 && (((uintptr_t)x | (uintptr_t)y | (uintptr_t)w | (uintptr_t)w2) & 15) == 0 && ((uintptr_t)h & (4 * sizeof(TH) - 1)) == 0;
  const int W4 = W / 4;
#define RUN(NV, B) return cima_launch(k_branch_norm4<TH, NV>, dim3(T), dim3(B), (size_t)0, stream, 1, x, y, w, (TH*)h, w2, W4, eps, eps2)
  if (vec && W4 <= 128) RUN(1, 128);
  if (vec && W4 <= 256) RUN(1, 256);
  if (vec && W4 <= 384) RUN(3, 128);
  if (vec && W4 <= 512) RUN(2, 256);
  if (vec && W4 <= 1024) RUN(4, 256);
  if (vec && W4 <= 2048) RUN(8, 256);
#undef RUN
  return cima_launch(k_branch_norm<TH>, dim3(T), dim3(256), (size_t)0, stream, 1, x, y, w, (TH*)h, w2, W, eps, eps2);
}
}  // namespace

// h (hdtype) may be null; w2 (with its eps2) may be null, and goes with h.
extern "C" int cima_branch_norm(float* x, const float* y, const float* w, void* h, int hdtype, const float* w2, int T, int W, float eps,
                                float eps2, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (W <= 0) return cima_fail(CIMA_E_SIZE, "branch_norm: width %d must be positive", W);
  if (w2 && !h) return cima_fail(CIMA_E_ARG, "branch_norm: the second norm needs rows to write to");
  int rc;
  if (!h || hdtype == CIMA_F32) rc = launch_branch_norm<float>(x, y, w, h, w2, T, W, eps, eps2, stream);
  else if (hdtype == CIMA_BF16) rc = launch_branch_norm<__nv_bfloat16>(x, y, w, h, w2, T, W, eps, eps2, stream);
  else return cima_fail(CIMA_E_DTYPE, "branch_norm: dtype code %d is neither float32 nor bfloat16", hdtype);
  return rc ? rc : cima_launch_result();
}
