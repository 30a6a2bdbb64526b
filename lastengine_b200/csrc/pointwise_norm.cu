// The pointwise norm y = tanh(alpha x) w + b (a number alpha, vectors w and b; no statistics of the row), alone and fused with
// a sum into the residual stream.  No number of a row depends on another, so a sublayer's result can be normed, added and
// the new stream normed again for the next sublayer in one pass over the row.  All float; results that feed matrix
// products are stored in the activation type.
#include "common.cuh"

__device__ __forceinline__ float pnorm(float x, float alpha, float w, float b) { return fmaf(tanhf(alpha * x), w, b); }
__device__ __forceinline__ float4 pnorm4(float4 x, float alpha, float4 w, float4 b) {
  return make_float4(pnorm(x.x, alpha, w.x, b.x), pnorm(x.y, alpha, w.y, b.y), pnorm(x.z, alpha, w.z, b.z), pnorm(x.w, alpha, w.w, b.w));
}

// out[m] = norm(x[rows ? rows[m] : m]), or out += it (ADD; out is float then)
template <typename TO, int VEC, bool ADD>
__global__ void __launch_bounds__(256)
pointwise_norm_kernel(TO* __restrict__ out, const float* __restrict__ x, const int* __restrict__ rows, float alpha,
                      const float* __restrict__ w, const float* __restrict__ b, int D) {
  pdl_wait();
  const int i = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (i >= D) return;
  const size_t m = blockIdx.x;
  const float* xi = x + (size_t)(rows ? rows[m] : m) * D + i;
  TO* o = out + m * D + i;
  if (VEC == 4) {
    float4 r = pnorm4(load4(xi), alpha, load4(w + i), load4(b + i));
    if (ADD) {
      const float4 old = load4(o);
      r = make_float4(old.x + r.x, old.y + r.y, old.z + r.z, old.w + r.w);
    }
    store4(o, r);
  } else {
    const float r = pnorm(*xi, alpha, w[i], b[i]);
    *o = from_f32<TO>(ADD ? to_f32(*o) + r : r);
  }
}

LEB_API int leb_pointwise_norm(void* out, int out_dtype, const float* x, const int* rows, float alpha, const float* w,
                               const float* b, int M, int D, int add, cudaStream_t st) {
  if (M <= 0 || D <= 0) return 0;
  LEB_REQUIRE(out_dtype == LEB_F32 || out_dtype == LEB_BF16, "leb_pointwise_norm: unknown dtype %d", out_dtype);
  LEB_REQUIRE(!add || out_dtype == LEB_F32, "leb_pointwise_norm: the added form writes the float residual");
  const bool vec = D % 4 == 0 && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)b | (uintptr_t)out) & 15) == 0;
  const int n = vec ? D / 4 : D, threads = n >= 256 ? 256 : (n + 31) / 32 * 32;
  LebPlainLaunches plain(true);
  const dim3 grid(M, ceil_div(n, threads)), block(threads);
#define LEB_PN(TO, V, A) leb_launch(pointwise_norm_kernel<TO, V, A>, grid, block, 0, st, (TO*)out, x, rows, alpha, w, b, D)
  if (out_dtype == LEB_BF16) { if (vec) LEB_PN(bf16, 4, false); else LEB_PN(bf16, 1, false); }
  else if (add) { if (vec) LEB_PN(float, 4, true); else LEB_PN(float, 1, true); }
  else { if (vec) LEB_PN(float, 4, false); else LEB_PN(float, 1, false); }
#undef LEB_PN
  LEB_CHECK_LAUNCH("leb_pointwise_norm");
  return 0;
}

// x[m] += norm1(y[m]); with h also h[m] = norm2(x[m]) of the new row.  y = y1, or c1 y1 + c2 y2 where a sublayer left its result
// in two parts.  A thread takes VEC columns of R rows one after the other, so the vectors are read once for them.
template <typename TH, int VEC, int R>
__global__ void __launch_bounds__(256)
pointwise_norm_sum_kernel(float* __restrict__ x, const float* __restrict__ y1, float c1, const float* __restrict__ y2, float c2,
                          float alpha1, const float* __restrict__ w1, const float* __restrict__ b1, TH* __restrict__ h,
                          float alpha2, const float* __restrict__ w2, const float* __restrict__ b2, int M, int D) {
  pdl_wait();
  const int i = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (i >= D) return;
  if (VEC == 4) {
    const float4 wa = load4(w1 + i), ba = load4(b1 + i);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 wb = h ? load4(w2 + i) : zero, bb = h ? load4(b2 + i) : zero;
    float4 xv[R], yv[R];
#pragma unroll
    for (int r = 0; r < R; r++) {
      const size_t m = (size_t)blockIdx.x * R + r;
      if (m < M) {
        xv[r] = load4(x + m * D + i);
        yv[r] = load4(y1 + m * D + i);
        if (y2) {
          const float4 t = load4(y2 + m * D + i);
          yv[r] = make_float4(c1 * yv[r].x + c2 * t.x, c1 * yv[r].y + c2 * t.y, c1 * yv[r].z + c2 * t.z, c1 * yv[r].w + c2 * t.w);
        }
      }
    }
#pragma unroll
    for (int r = 0; r < R; r++) {
      const size_t m = (size_t)blockIdx.x * R + r;
      if (m >= M) break;
      const float4 d = pnorm4(yv[r], alpha1, wa, ba);
      const float4 v = make_float4(xv[r].x + d.x, xv[r].y + d.y, xv[r].z + d.z, xv[r].w + d.w);
      store4(x + m * D + i, v);
      if (h) store4(h + m * D + i, pnorm4(v, alpha2, wb, bb));
    }
  } else {
    for (int r = 0; r < R; r++) {
      const size_t m = (size_t)blockIdx.x * R + r;
      if (m >= M) break;
      float y = y1[m * D + i];
      if (y2) y = c1 * y + c2 * y2[m * D + i];
      const float v = x[m * D + i] + pnorm(y, alpha1, w1[i], b1[i]);
      x[m * D + i] = v;
      if (h) h[m * D + i] = from_f32<TH>(pnorm(v, alpha2, w2[i], b2[i]));
    }
  }
}

LEB_API int leb_pointwise_norm_sum(float* x, const float* y1, float c1, const float* y2, float c2, float alpha1,
                                   const float* w1, const float* b1, void* h, int h_dtype, float alpha2, const float* w2,
                                   const float* b2, int M, int D, cudaStream_t st) {
  if (M <= 0 || D <= 0) return 0;
  LEB_REQUIRE(!h || (w2 && b2), "leb_pointwise_norm_sum: the second norm needs its vectors");
  LEB_REQUIRE(!h || h_dtype == LEB_F32 || h_dtype == LEB_BF16, "leb_pointwise_norm_sum: unknown dtype %d", h_dtype);
  const bool vec = D % 4 == 0 && (((uintptr_t)x | (uintptr_t)y1 | (uintptr_t)y2 | (uintptr_t)w1 | (uintptr_t)b1 | (uintptr_t)h |
                                   (uintptr_t)w2 | (uintptr_t)b2) & 15) == 0;
  const int n = vec ? D / 4 : D;
  const int threads = n >= 256 && M > 64 ? 256 : (n >= 128 ? 128 : (n + 31) / 32 * 32);
  const int R = M > 256 ? 4 : 1;      // many rows: a block keeps its columns' vectors for four of them
  const dim3 grid(ceil_div(M, R), ceil_div(n, threads)), block(threads);
  const bool b16 = h && h_dtype == LEB_BF16;
  LebPlainLaunches plain(true);
#define LEB_PNS(TH, V, R_) \
  leb_launch(pointwise_norm_sum_kernel<TH, V, R_>, grid, block, 0, st, x, y1, c1, y2, c2, alpha1, w1, b1, (TH*)h, alpha2, w2, b2, M, D)
#define LEB_PNS2(TH)                                                  \
  {                                                                   \
    if (vec) { if (R == 4) LEB_PNS(TH, 4, 4); else LEB_PNS(TH, 4, 1); } \
    else { if (R == 4) LEB_PNS(TH, 1, 4); else LEB_PNS(TH, 1, 1); }     \
  }
  if (b16) LEB_PNS2(bf16)
  else LEB_PNS2(float)
#undef LEB_PNS2
#undef LEB_PNS
  LEB_CHECK_LAUNCH("leb_pointwise_norm_sum");
  return 0;
}

// What a product over [x | x0] needs of the stream x: out[m * ld + i] = x[m, i] in the activation type, and (fill) x[m, i] =
// vec[i] (null: 0) afterwards, so that the product, added onto x, leaves W [x | x0] + vec there.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
stream_columns_kernel(T* __restrict__ out, int ld, float* __restrict__ x, const float* __restrict__ vec, int fill, int D) {
  pdl_wait();
  const int i = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (i >= D) return;
  const size_t m = blockIdx.x;
  if (VEC == 4) {
    store4(out + m * ld + i, load4(x + m * D + i));
    if (fill) store4(x + m * D + i, vec ? load4(vec + i) : make_float4(0.f, 0.f, 0.f, 0.f));
  } else {
    out[m * ld + i] = from_f32<T>(x[m * D + i]);
    if (fill) x[m * D + i] = vec ? vec[i] : 0.f;
  }
}

LEB_API int leb_stream_columns(void* out, int ld, int dtype, float* x, const float* vec, int fill, int M, int D, cudaStream_t st) {
  if (M <= 0 || D <= 0) return 0;
  LEB_REQUIRE(dtype == LEB_F32 || dtype == LEB_BF16, "leb_stream_columns: unknown dtype %d", dtype);
  const bool v4 = D % 4 == 0 && ld % 4 == 0 && (((uintptr_t)x | (uintptr_t)vec | (uintptr_t)out) & 15) == 0;
  const int n = v4 ? D / 4 : D, threads = n >= 128 ? 128 : (n + 31) / 32 * 32;
  const dim3 grid(M, ceil_div(n, threads)), block(threads);
  LebPlainLaunches plain(true);
#define LEB_SC(T, V) leb_launch(stream_columns_kernel<T, V>, grid, block, 0, st, (T*)out, ld, x, vec, fill, D)
  if (dtype == LEB_F32) { if (v4) LEB_SC(float, 4); else LEB_SC(float, 1); }
  else { if (v4) LEB_SC(bf16, 4); else LEB_SC(bf16, 1); }
#undef LEB_SC
  LEB_CHECK_LAUNCH("leb_stream_columns");
  return 0;
}
