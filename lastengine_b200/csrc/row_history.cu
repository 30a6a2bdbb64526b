// Kernels of parts that look one row back: the embedding of token pairs and the mixing of every row with the row before
// it.  What a sequence's next step needs of its last row (a token, a row of numbers) is state per slot.  Who reads the old
// state of a sequence also writes the new one, in this order, so one launch does both for steps of any number of rows.
#include "common.cuh"

// x[m] = table[tok] * scale + pairs[(prev * mul_prev + tok * mul_cur) mod buckets], the row number `buckets` for a
// sequence's first token; prev is the row before within the step, or the sequence's last token (state [slot]).
template <typename T>
__global__ void __launch_bounds__(256)
embed_pairs_kernel(float* __restrict__ x, const T* __restrict__ table, const T* __restrict__ pairs, const int* __restrict__ tokens,
                   const int* __restrict__ row_seq, const int* __restrict__ row_pos, const int* __restrict__ seq_slot,
                   const int* __restrict__ seq_qstart, const int* __restrict__ seq_qlen, int* __restrict__ state, int D, int V,
                   int buckets, long long mul_prev, long long mul_cur, float scale) {
  __shared__ int pair_row;
  pdl_wait();
  const size_t m = blockIdx.x;
  if (threadIdx.x == 0) {
    const int b = row_seq[m], slot = seq_slot[b], q0 = seq_qstart[b];
    const bool opens = (int)m == q0;
    int prev = -1;
    if (!opens) prev = tokens[m - 1];
    else if (row_pos[m] > 0 && slot >= 0) prev = state[slot];
    if (opens && slot >= 0) state[slot] = tokens[q0 + (seq_qlen ? seq_qlen[b] : 1) - 1];
    pair_row = prev < 0 ? buckets : (int)(((long long)prev * mul_prev + (long long)tokens[m] * mul_cur) % buckets);
  }
  __syncthreads();
  int tok = tokens[m];
  tok = tok < 0 ? 0 : (tok >= V ? V - 1 : tok);
  const int pr = min(max(pair_row, 0), buckets);
  const T* a = table + (size_t)tok * D;
  const T* p = pairs + (size_t)pr * D;
  float* o = x + m * D;
  if (D % 4 == 0 && (((uintptr_t)a | (uintptr_t)p | (uintptr_t)o) & (sizeof(T) == 4 ? 15 : 7)) == 0 && ((uintptr_t)o & 15) == 0) {
    for (int i = threadIdx.x * 4; i < D; i += blockDim.x * 4) {
      const float4 u = load4(a + i), v = load4(p + i);
      store4(o + i, make_float4(u.x * scale + v.x, u.y * scale + v.y, u.z * scale + v.z, u.w * scale + v.w));
    }
  } else {
    for (int i = threadIdx.x; i < D; i += blockDim.x) o[i] = to_f32(a[i]) * scale + to_f32(p[i]);
  }
}

LEB_API int leb_embed_pairs(float* x, const void* table, const void* pairs, int dtype, const int* tokens, const int* row_seq,
                            const int* row_pos, const int* seq_slot, const int* seq_qstart, const int* seq_qlen, int* state,
                            int M, int D, int V, int buckets, long long mul_prev, long long mul_cur, float scale,
                            cudaStream_t st) {
  if (M <= 0) return 0;
  LEB_REQUIRE(buckets >= 1 && mul_prev >= 0 && mul_cur >= 0, "leb_embed_pairs: %d buckets, factors %lld and %lld", buckets,
              mul_prev, mul_cur);
  LebPlainLaunches plain(true);
  const dim3 grid(M), block(D >= 1024 ? 256 : 128);
  if (dtype == LEB_F32)
    leb_launch(embed_pairs_kernel<float>, grid, block, 0, st, x, (const float*)table, (const float*)pairs, tokens, row_seq, row_pos,
               seq_slot, seq_qstart, seq_qlen, state, D, V, buckets, mul_prev, mul_cur, scale);
  else if (dtype == LEB_BF16)
    leb_launch(embed_pairs_kernel<bf16>, grid, block, 0, st, x, (const bf16*)table, (const bf16*)pairs, tokens, row_seq, row_pos,
               seq_slot, seq_qstart, seq_qlen, state, D, V, buckets, mul_prev, mul_cur, scale);
  else
    return leb_fail("leb_embed_pairs: unknown table dtype %d", dtype);
  LEB_CHECK_LAUNCH("leb_embed_pairs");
  return 0;
}

// mix[s][m] = h[m] + (h_before[m] - h[m]) * mu[s] for s < n_mix: every row with the row before it (zeros before the
// sequence's first; the carried row, state [slot][D], in front of the step's).  A thread takes VEC columns of a row.
template <typename T, int VEC>
__global__ void __launch_bounds__(128)
row_shift_mix_kernel(T* __restrict__ mix, const T* __restrict__ h, const float* __restrict__ mu, float* __restrict__ state,
                     const int* __restrict__ row_seq, const int* __restrict__ seq_slot, const int* __restrict__ seq_qstart,
                     const int* __restrict__ seq_qlen, int M, int D, int n_mix) {
  pdl_wait();
  const int i = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (i >= D) return;
  const size_t m = blockIdx.x;
  const int b = row_seq[m], q0 = seq_qstart[b];
  float now[VEC], old[VEC];
  auto get = [&](float* o, auto p) {
    if (VEC == 4) {
      const float4 v = load4(p);
      o[0] = v.x; o[1 % VEC] = v.y; o[2 % VEC] = v.z; o[3 % VEC] = v.w;
    } else {
      o[0] = to_f32(*p);
    }
  };
  get(now, h + m * D + i);
  if ((int)m != q0) {
    get(old, h + (m - 1) * D + i);
  } else {
    const int slot = seq_slot[b];
    if (slot >= 0) {
      float* sp = state + (size_t)slot * D + i;
      get(old, (const float*)sp);
      float last[VEC];
      get(last, h + (size_t)(q0 + (seq_qlen ? seq_qlen[b] : 1) - 1) * D + i);
#pragma unroll
      for (int e = 0; e < VEC; e++) sp[e] = last[e];
    } else {
#pragma unroll
      for (int e = 0; e < VEC; e++) old[e] = 0.f;
    }
  }
  for (int s = 0; s < n_mix; s++) {
    float w[VEC], o[VEC];
    get(w, mu + (size_t)s * D + i);
#pragma unroll
    for (int e = 0; e < VEC; e++) o[e] = fmaf(old[e] - now[e], w[e], now[e]);
    T* dst = mix + ((size_t)s * M + m) * D + i;
    if (VEC == 4) store4(dst, make_float4(o[0], o[1 % VEC], o[2 % VEC], o[3 % VEC]));
    else *dst = from_f32<T>(o[0]);
  }
}

LEB_API int leb_row_shift_mix(void* mix, const void* h, int dtype, const float* mu, float* state, const int* row_seq,
                              const int* seq_slot, const int* seq_qstart, const int* seq_qlen, int M, int D, int n_mix,
                              cudaStream_t st) {
  if (M <= 0 || D <= 0 || n_mix <= 0) return 0;
  LEB_REQUIRE(dtype == LEB_F32 || dtype == LEB_BF16, "leb_row_shift_mix: unknown dtype %d", dtype);
  const bool vec = D % 4 == 0 && (((uintptr_t)mix | (uintptr_t)h | (uintptr_t)mu | (uintptr_t)state) & 15) == 0;
  const int n = vec ? D / 4 : D;
  const dim3 grid(M, ceil_div(n, 128)), block(128);
  LebPlainLaunches plain(true);
#define LEB_RSM(T, V) \
  leb_launch(row_shift_mix_kernel<T, V>, grid, block, 0, st, (T*)mix, (const T*)h, mu, state, row_seq, seq_slot, seq_qstart, seq_qlen, M, D, n_mix)
  if (dtype == LEB_F32) { if (vec) LEB_RSM(float, 4); else LEB_RSM(float, 1); }
  else { if (vec) LEB_RSM(bf16, 4); else LEB_RSM(bf16, 1); }
#undef LEB_RSM
  LEB_CHECK_LAUNCH("leb_row_shift_mix");
  return 0;
}

// The decay of a recurrence from a low-rank pair: out[m, c] = exp(-exp(sum_j tanh(low[m, j]) w2[j, c] + w0[c])), all
// float (w2 [rank, C], so that neighbouring threads read neighbouring numbers).  A block takes R rows x 128 VEC
// channels, a thread VEC neighbouring ones; the rows' tanh values stay in shared memory, a slab of ranks at a time.
constexpr int LRD_SLAB = 64;
template <int R, int VEC>
__global__ void __launch_bounds__(128)
low_rank_decay_kernel(float* __restrict__ out, const float* __restrict__ low, int ldl, const float* __restrict__ w2,
                      const float* __restrict__ w0, int M, int C, int rank) {
  __shared__ __align__(16) float ts[LRD_SLAB][R];
  pdl_wait();
  const int m0 = blockIdx.x * R, c = (blockIdx.y * 128 + threadIdx.x) * VEC;
  float acc[R][VEC];
#pragma unroll
  for (int r = 0; r < R; r++)
#pragma unroll
    for (int e = 0; e < VEC; e++) acc[r][e] = 0.f;
  auto get = [&](float* o, const float* p) {
    if (VEC == 4) {
      const float4 v = load4(p);
      o[0] = v.x; o[1 % VEC] = v.y; o[2 % VEC] = v.z; o[3 % VEC] = v.w;
    } else {
      o[0] = *p;
    }
  };
  for (int j0 = 0; j0 < rank; j0 += LRD_SLAB) {
    const int nj = min(LRD_SLAB, rank - j0);
    __syncthreads();
    for (int idx = threadIdx.x; idx < R * nj; idx += 128) {
      const int r = idx / nj, j = idx - r * nj;
      ts[j][r] = m0 + r < M ? tanhf(low[(size_t)(m0 + r) * ldl + j0 + j]) : 0.f;
    }
    __syncthreads();
    if (c < C) {
      for (int j = 0; j < nj; j += 4) {
        float wv[4][VEC];      // four rows of w2 are asked for before the first is used
#pragma unroll
        for (int q = 0; q < 4; q++) {
          if (j + q < nj) get(wv[q], w2 + (size_t)(j0 + j + q) * C + c);
          else
#pragma unroll
            for (int e = 0; e < VEC; e++) wv[q][e] = 0.f;
        }
#pragma unroll
        for (int q = 0; q < 4; q++)
          if (j + q < nj)
#pragma unroll
            for (int r = 0; r < R; r++) {
              const float t = ts[j + q][r];
#pragma unroll
              for (int e = 0; e < VEC; e++) acc[r][e] = fmaf(t, wv[q][e], acc[r][e]);
            }
      }
    }
  }
  if (c >= C) return;
  float z0[VEC];
  get(z0, w0 + c);
#pragma unroll
  for (int r = 0; r < R; r++) {
    if (m0 + r >= M) break;
    float o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) o[e] = expf(-expf(acc[r][e] + z0[e]));
    float* dst = out + (size_t)(m0 + r) * C + c;
    if (VEC == 4) store4(dst, make_float4(o[0], o[1 % VEC], o[2 % VEC], o[3 % VEC]));
    else *dst = o[0];
  }
}

LEB_API int leb_low_rank_decay(float* out, const float* low, int ldl, const float* w2, const float* w0, int M, int C, int rank,
                               cudaStream_t st) {
  if (M <= 0 || C <= 0) return 0;
  LEB_REQUIRE(rank >= 1, "leb_low_rank_decay: a rank of %d", rank);
  LebPlainLaunches plain(true);
  const bool vec = C % 4 == 0 && (((uintptr_t)out | (uintptr_t)w2 | (uintptr_t)w0) & 15) == 0;
#define LEB_LRD(R_, V_) \
  leb_launch(low_rank_decay_kernel<R_, V_>, dim3(ceil_div(M, R_), ceil_div(C, 128 * V_)), dim3(128), 0, st, out, low, ldl, w2, w0, M, C, rank)
  // a few rows: a channel a thread, so that a decode step has blocks for more SMs
  if (M <= 16) LEB_LRD(1, 1);
  else if (vec) LEB_LRD(8, 4);
  else LEB_LRD(8, 1);
#undef LEB_LRD
  LEB_CHECK_LAUNCH("leb_low_rank_decay");
  return 0;
}
