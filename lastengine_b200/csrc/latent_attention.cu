// Latent attention: every head's keys and values are linear images of one cached latent vector
// per position, plus one rotated key part that all heads share.
//
//   c_q = rmsnorm(W_dq h),  q_h = W_uq,h c_q = [q_h^n (dim) | q_h^r (rot)]      q_h^r rotated by position
//   [a | r] = W_dkv h,  c = rmsnorm(a) (rank),  k^r = rotate(r) (rot)              cached: [c | k^r]
//   k_h = W_uk,h c,  v_h = W_uv,h c
//   s_h(i, j) = scale (q_h^n . k_h(j) + q_h^r . k^r(j)),  j <= i (and in i's window or chunk where a layer has one)
//   p = softmax over {s_h(i, j)} and one more logit sink_h that has no key and no value
//   o_h = sum_j p_j v_h(j)
//
// Only [c | k^r] is cached, one row of rank + rot numbers per position and layer, whatever the
// number of heads.  The kernels never form k_h or v_h: since q^n . (W_uk c) = (W_uk^T q^n) . c, a
// query is taken into the latent space once (t_h = W_uk,h^T q_h^n, a product grouped by head),
// attention runs with the one cached row as key ([c | k^r] against [t_h | q_h^r]) and its first
// `rank` numbers as value, and the result u_h = sum_j p_j c(j) goes through W_uv,h afterwards
// (again a product grouped by head).  All heads of a row share every key they read.
//
// Kernels here: the preparation of a step's rows (both norms, the rotation of k^r, the cache
// write), the split of q into its unrotated part (head-major, for the grouped product) and its
// rotated part, the attention itself with its merge of key-range splits, and the turn of a
// head-major result back to rows.  Norms, angles, sine and cosine, scores, softmax and the value
// sums are float; sinf/cosf are the full-range versions.
#include "common.cuh"

// Rotation of the first `rot_dims` of a vector's numbers: pair t is (2t, 2t + 1), or with `neox` (t, t + rot_dims / 2);
// (u, v) -> (u cos a - v sin a, v cos a + u sin a), a = pos * inv_freq[t]; the rest passes unchanged.  The unit t of
// such a vector of `rot` numbers is pair t while t < rot_dims / 2, then single numbers.
template <typename T, typename CT>
__device__ __forceinline__ void rotate_unit(CT* __restrict__ dst, const T* __restrict__ src, int t, float pos,
                                            const float* __restrict__ inv_freq, int rot_dims, int neox) {
  const int half = rot_dims / 2;
  if (t >= half) {
    const int d = rot_dims + t - half;
    dst[d] = from_f32<CT>(to_f32(src[d]));
    return;
  }
  const int ia = neox ? t : 2 * t, ib = neox ? t + half : 2 * t + 1;
  const float u = to_f32(src[ia]), v = to_f32(src[ib]);
  const float a = pos * inv_freq[t];
  const float c = cosf(a), s = sinf(a);
  dst[ia] = from_f32<CT>(u * c - v * s);
  dst[ib] = from_f32<CT>(v * c + u * s);
}

// The cache row [c | k^r] of row m: lat = `rank` numbers of the latent before its norm, then `rot` of the shared key part
// before its rotation.  By the whole block; rows of padding sequences touch no cache.
template <typename T, typename CT>
__device__ __forceinline__ void latent_cache_row(const T* __restrict__ lat, int m, CT* __restrict__ pool,
                                                 const int* __restrict__ block_table, int bt_width,
                                                 const int* __restrict__ row_seq, const int* __restrict__ row_pos,
                                                 const int* __restrict__ seq_slot, const float* __restrict__ wkv, float eps,
                                                 const float* __restrict__ inv_freq, int rot_dims, int neox, int rank, int rot,
                                                 int page_size, float* red) {
  const int b = row_seq[m], pos = row_pos[m];
  float ss = 0.f;
  for (int i = threadIdx.x; i < rank; i += blockDim.x) {
    const float v = to_f32(lat[i]);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  if (seq_slot[b] < 0) return;      // a padding sequence touches no cache
  const int page = block_table[(size_t)b * bt_width + pos / page_size];
  if (page < 0) return;
  const float r = 1.0f / sqrtf(ss / (float)rank + eps);
  CT* dst = pool + ((size_t)page * page_size + pos % page_size) * (size_t)(rank + rot);
  for (int i = threadIdx.x; i < rank; i += blockDim.x) dst[i] = from_f32<CT>(to_f32(lat[i]) * r * wkv[i]);
  for (int t = threadIdx.x; t < rot - rot_dims / 2; t += blockDim.x)
    rotate_unit<T, CT>(dst + rank, lat + rank, t, (float)pos, inv_freq, rot_dims, neox);
}

// Row m of q [H * (dim + rot)] -> qn [H, M, dim_p] (the unrotated parts, head-major, zeros from dim to dim_p) and
// qr [M, H, rot] (the rotated parts).  By the whole block; `wide`: 16-byte pieces.
template <typename T>
__device__ __forceinline__ void latent_split_row(T* __restrict__ qn, T* __restrict__ qr, const T* __restrict__ row, int m,
                                                 float pos, const float* __restrict__ inv_freq, int rot_dims, int neox, int M,
                                                 int H, int dim, int dim_p, int rot, bool wide) {
  const int hw = dim + rot;
  constexpr int PER = 16 / (int)sizeof(T);          // elements of a 16-byte piece
  if (wide) {
    const int pieces = dim / PER;
    for (int i = threadIdx.x; i < H * pieces; i += blockDim.x) {
      const int h = i / pieces, c = i - h * pieces;
      reinterpret_cast<uint4*>(qn + ((size_t)h * M + m) * dim)[c] = reinterpret_cast<const uint4*>(row + h * hw)[c];
    }
  } else {
    for (int i = threadIdx.x; i < H * dim_p; i += blockDim.x) {
      const int h = i / dim_p, d = i - h * dim_p;
      qn[((size_t)h * M + m) * dim_p + d] = d < dim ? row[h * hw + d] : from_f32<T>(0.f);
    }
  }
  const int units = rot - rot_dims / 2;
  for (int i = threadIdx.x; i < H * units; i += blockDim.x) {
    const int h = i / units, t = i - h * units;
    rotate_unit<T, T>(qr + ((size_t)m * H + h) * rot, row + h * hw + dim, t, pos, inv_freq, rot_dims, neox);
  }
}

// One block per row.  in [M, ld_in]: columns [0, q_rank) the query latent before its norm, then
// (own_kv) `rank` columns of the key/value latent before its norm and `rot` columns of the shared
// key part before its rotation.  Leaves cq [M, q_rank] = rmsnorm(.) * wq and, for rows of live
// sequences, the cache row [c | k^r] at the row's position.
template <typename T, typename CT>
__global__ void __launch_bounds__(256)
latent_prep_kernel(T* __restrict__ cq, const T* __restrict__ in, int ld_in, CT* __restrict__ pool,
                   const int* __restrict__ block_table, int bt_width, const int* __restrict__ row_seq,
                   const int* __restrict__ row_pos, const int* __restrict__ seq_slot,
                   const float* __restrict__ wq, const float* __restrict__ wkv, float eps,
                   const float* __restrict__ inv_freq, int rot_dims, int neox, int q_rank, int rank, int rot,
                   int page_size) {
  __shared__ float red[33];
  pdl_wait();
  const int m = blockIdx.x;
  const T* row = in + (size_t)m * ld_in;
  float ss = 0.f;
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) {
    const float v = to_f32(row[i]);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / (float)q_rank + eps);
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x)
    cq[(size_t)m * q_rank + i] = from_f32<T>(to_f32(row[i]) * r * wq[i]);
  if (!pool) return;
  latent_cache_row<T, CT>(row + q_rank, m, pool, block_table, bt_width, row_seq, row_pos, seq_slot, wkv, eps, inv_freq, rot_dims,
                          neox, rank, rot, page_size, red);
}

// q [M, H * (dim + rot)] -> qn and qr, one block per row.
template <typename T>
__global__ void __launch_bounds__(256)
latent_q_split_kernel(T* __restrict__ qn, T* __restrict__ qr, const T* __restrict__ q,
                      const int* __restrict__ row_pos, const float* __restrict__ inv_freq, int rot_dims, int neox,
                      int M, int H, int dim, int dim_p, int rot, int wide) {
  pdl_wait();
  const int m = blockIdx.x;
  latent_split_row<T>(qn, qr, q + (size_t)m * H * (dim + rot), m, (float)row_pos[m], inv_freq, rot_dims, neox, M, H, dim, dim_p, rot,
                      wide != 0);
}

// Both jobs in one launch where q comes straight from a projection of the row (no query latent): in [M, ld_in] holds
// q [H * (dim + rot)], then (with `pool`) `rank` latent columns and `rot` columns of the shared key part.  Blocks (m, 0)
// split q, blocks (m, 1) write the cache row.
template <typename T>
__global__ void __launch_bounds__(256)
latent_rows_kernel(T* __restrict__ qn, T* __restrict__ qr, const T* __restrict__ in, int ld_in, T* __restrict__ pool,
                   const int* __restrict__ block_table, int bt_width, const int* __restrict__ row_seq,
                   const int* __restrict__ row_pos, const int* __restrict__ seq_slot, const float* __restrict__ wkv, float eps,
                   const float* __restrict__ inv_freq, int rot_dims, int neox, int M, int H, int dim, int dim_p, int rank,
                   int rot, int page_size, int wide) {
  __shared__ float red[33];
  pdl_wait();
  const int m = blockIdx.x;
  const T* row = in + (size_t)m * ld_in;
  if (blockIdx.y == 0)
    latent_split_row<T>(qn, qr, row, m, (float)row_pos[m], inv_freq, rot_dims, neox, M, H, dim, dim_p, rot, wide != 0);
  else
    latent_cache_row<T, T>(row + H * (dim + rot), m, pool, block_table, bt_width, row_seq, row_pos, seq_slot, wkv, eps, inv_freq,
                           rot_dims, neox, rank, rot, page_size, red);
}

// in [H, M, w] -> out [M, H * w], one piece per thread: an element, or 16 bytes where the rows allow it
template <typename P>
__global__ void heads_to_rows_kernel(P* __restrict__ out, const P* __restrict__ in, int M, int H, int w) {
  pdl_wait();
  const size_t total = (size_t)M * H * w;
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const size_t m = i / ((size_t)H * w);
  const int r = (int)(i - m * H * w);
  const int h = r / w, d = r - h * w;
  out[i] = in[((size_t)h * M + m) * w + d];
}

// ---------------------------------------------------------------------------------------------
// The attention.  Block = 4 warps: one sequence, a chunk of HC <= 8 heads, QT rows (QT * HC <= 32
// query vectors), one split of the key range.  Per tile of 32 cached rows, staged once as float
// for all of the block's query vectors: lane = key for the scores, lane = dimension for the sums
// of c.  A query vector is [t_h (rank) | q_h^r (rot)].
#define LAT_WARPS 4
#define LAT_RPW 8
#define LAT_NEG (-1e30f)

template <typename T, typename CT, int HDL>      // rank <= 32 * HDL
__global__ void __launch_bounds__(32 * LAT_WARPS)
latent_attention_kernel(T* __restrict__ out, int ld_out, float* __restrict__ part, const T* __restrict__ qt,
                        const T* __restrict__ qr, const CT* __restrict__ pool,
                        const int* __restrict__ block_table, int bt_width, const int* __restrict__ seq_slot,
                        const int* __restrict__ seq_pos0, const int* __restrict__ seq_qstart,
                        const int* __restrict__ seq_qlen, const float* __restrict__ sink, int M, int H,
                        int rank, int rot, int page_size, int window, int chunk, float scale, int QT, int HC,
                        int n_splits) {
  extern __shared__ float sm[];
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int hc = blockIdx.y;
  const int b = blockIdx.z / n_splits, split = blockIdx.z % n_splits;
  const int slot = seq_slot[b];
  const int qlen = seq_qlen[b];
  const int row_lo = blockIdx.x * QT;
  if (row_lo >= qlen) return;
  const int nrows = min(QT, qlen - row_lo);
  const int nheads = min(HC, H - hc * HC);
  const int q0 = seq_qstart[b];
  const int pos0 = seq_pos0[b];
  const int R = QT * HC;
  const int dk = rank + rot;
  const int KS = dk + 1;           // lanes read different staged rows at the same column

  float* q_s = sm;                 // [R][dk]
  float* k_s = q_s + R * dk;       // [32][dk + 1]
  float* p_s = k_s + 32 * KS;      // [LAT_WARPS][32]

  if (slot < 0) {                  // a padding sequence: defined output, no cache access
    for (int r = warp; r < R; r += LAT_WARPS) {
      const int i = r / HC, j = r % HC;
      if (i >= nrows || j >= nheads) continue;
      const int h = hc * HC + j;
      const size_t m = (size_t)q0 + row_lo + i;
      if (n_splits == 1) {
        for (int d = lane; d < ld_out; d += 32) out[((size_t)h * M + m) * ld_out + d] = from_f32<T>(0.f);
      } else {
        float* pp = part + ((m * H + h) * n_splits + split) * (size_t)(rank + 2);
        if (lane == 0) { pp[0] = LAT_NEG; pp[1] = 0.f; }
        for (int d = lane; d < rank; d += 32) pp[2 + d] = 0.f;
      }
    }
    return;
  }

  for (int idx = threadIdx.x; idx < R * dk; idx += blockDim.x) {
    const int r = idx / dk, d = idx - r * dk;
    const int i = r / HC, j = r % HC;
    float v = 0.f;
    if (i < nrows && j < nheads) {
      const int h = hc * HC + j;
      const size_t m = (size_t)q0 + row_lo + i;
      v = d < rank ? to_f32(qt[((size_t)h * M + m) * rank + d]) : to_f32(qr[(m * H + h) * rot + (d - rank)]);
    }
    q_s[idx] = v;
  }

  const int kv_len = pos0 + qlen;
  const int pos_hi = pos0 + row_lo + nrows - 1;
  const int tile_first = first_key(pos0 + row_lo, window, chunk) / 32, tile_end = pos_hi / 32 + 1;
  const int per_split = (tile_end - tile_first + n_splits - 1) / n_splits;
  const int t_lo = tile_first + split * per_split;
  const int t_hi = min(tile_end, t_lo + per_split);

  float mx[LAT_RPW], l[LAT_RPW], acc[LAT_RPW][HDL];
#pragma unroll
  for (int ri = 0; ri < LAT_RPW; ri++) {
    mx[ri] = LAT_NEG;
    l[ri] = 0.f;
#pragma unroll
    for (int jj = 0; jj < HDL; jj++) acc[ri][jj] = 0.f;
  }

  for (int tile = t_lo; tile < t_hi; tile++) {
    const int key0 = tile * 32;
    const int page = block_table[(size_t)b * bt_width + key0 / page_size];
    const size_t base = ((size_t)(page < 0 ? 0 : page) * page_size + key0 % page_size) * dk;
    __syncthreads();               // the previous tile has been consumed (and q_s is written, first time round)
    for (int idx = threadIdx.x; idx < 32 * dk; idx += blockDim.x) {
      const int kk = idx / dk, d = idx - kk * dk;
      float kv = 0.f;
      if (page >= 0 && key0 + kk < kv_len) kv = to_f32(pool[base + idx]);   // beyond the sequence the pool holds stale bits
      k_s[kk * KS + d] = kv;
    }
    __syncthreads();
#pragma unroll
    for (int ri = 0; ri < LAT_RPW; ri++) {
      const int r = warp + ri * LAT_WARPS;
      if (r >= R) break;
      const int i = r / HC, j = r % HC;
      if (i >= nrows || j >= nheads) continue;
      const int qpos = pos0 + row_lo + i;
      const int lo = first_key(qpos, window, chunk);
      if (key0 > qpos || key0 + 31 < lo) continue;   // the whole tile lies after this row, or before what it reads
      const float* qv = q_s + r * dk;
      const float* kr = k_s + lane * KS;
      float s = 0.f;
      for (int d = 0; d < dk; d++) s += qv[d] * kr[d];
      s *= scale;
      const bool valid = key0 + lane <= qpos && key0 + lane >= lo;
      s = valid ? s : LAT_NEG;
      const float mn = fmaxf(mx[ri], warp_max(s));
      const float p = valid ? expf(s - mn) : 0.f;
      const float corr = expf(mx[ri] - mn);
      l[ri] = l[ri] * corr + warp_sum(p);
      mx[ri] = mn;
      p_s[warp * 32 + lane] = p;
      __syncwarp();
#pragma unroll
      for (int jj = 0; jj < HDL; jj++) {
        const int d = lane + 32 * jj;
        if (d < rank) {
          float a = 0.f;
#pragma unroll 8
          for (int kk = 0; kk < 32; kk++) a += p_s[warp * 32 + kk] * k_s[kk * KS + d];
          acc[ri][jj] = acc[ri][jj] * corr + a;
        }
      }
      __syncwarp();
    }
  }

#pragma unroll
  for (int ri = 0; ri < LAT_RPW; ri++) {
    const int r = warp + ri * LAT_WARPS;
    if (r >= R) break;
    const int i = r / HC, j = r % HC;
    if (i >= nrows || j >= nheads) continue;
    const int h = hc * HC + j;
    const size_t m = (size_t)q0 + row_lo + i;
    if (n_splits == 1) {
      // the sink joins the denominator: one more logit, not scaled, without a value
      const float sk = sink ? sink[h] : LAT_NEG;
      const float mn = fmaxf(mx[ri], sk);
      const float corr = expf(mx[ri] - mn);
      const float den = l[ri] * corr + (sink ? expf(sk - mn) : 0.f);
      const float inv = den > 0.f ? corr / den : 0.f;
      T* o = out + ((size_t)h * M + m) * ld_out;
#pragma unroll
      for (int jj = 0; jj < HDL; jj++) {
        const int d = lane + 32 * jj;
        if (d < rank) o[d] = from_f32<T>(acc[ri][jj] * inv);
      }
      for (int d = rank + lane; d < ld_out; d += 32) o[d] = from_f32<T>(0.f);
    } else {
      float* pp = part + ((m * H + h) * n_splits + split) * (size_t)(rank + 2);
      if (lane == 0) { pp[0] = mx[ri]; pp[1] = l[ri]; }
#pragma unroll
      for (int jj = 0; jj < HDL; jj++) {
        const int d = lane + 32 * jj;
        if (d < rank) pp[2 + d] = acc[ri][jj];
      }
    }
  }
}

// Merge of the key-range splits of one (row, head), with the sink as one more term of the
// denominator: out = sum_s acc_s e^(m_s - m) / (sum_s l_s e^(m_s - m) + e^(sink - m)).
// The first warp turns the splits' maxima and sums into one factor each; then a thread per number of the latent adds the
// splits' sums, sixteen loads at a time (n_splits <= 64).
template <typename T>
__global__ void __launch_bounds__(512)
latent_merge_kernel(T* __restrict__ out, int ld_out, const float* __restrict__ part, const float* __restrict__ sink, int M,
                    int H, int rank, int n_splits) {
  __shared__ float f_s[64];
  pdl_wait();
  const size_t m = blockIdx.x;
  const int h = blockIdx.y;
  const size_t step = rank + 2;
  const float* pp = part + ((m * H + h) * n_splits) * step;
  if (threadIdx.x < 32) {
    const int s0 = threadIdx.x, s1 = threadIdx.x + 32;
    const float m0 = s0 < n_splits ? pp[s0 * step] : LAT_NEG, m1 = s1 < n_splits ? pp[s1 * step] : LAT_NEG;
    const float l0 = s0 < n_splits ? pp[s0 * step + 1] : 0.f, l1 = s1 < n_splits ? pp[s1 * step + 1] : 0.f;
    const float sk = sink ? sink[h] : LAT_NEG;
    const float mn = fmaxf(sk, warp_max(fmaxf(m0, m1)));
    const float e0 = expf(m0 - mn), e1 = expf(m1 - mn);
    const float den = warp_sum(l0 * e0 + l1 * e1) + (sink ? expf(sk - mn) : 0.f);
    const float inv = den > 0.f ? 1.0f / den : 0.f;
    f_s[s0] = e0 * inv;
    f_s[s1] = e1 * inv;
  }
  __syncthreads();
  T* o = out + ((size_t)h * M + m) * ld_out;
  for (int d = threadIdx.x; d < ld_out; d += blockDim.x) {
    float a = 0.f;
    if (d < rank) {
      for (int s0 = 0; s0 < n_splits; s0 += 16) {
        float v[16];
#pragma unroll
        for (int q = 0; q < 16; q++) v[q] = s0 + q < n_splits ? pp[(s0 + q) * step + 2 + d] : 0.f;
#pragma unroll
        for (int q = 0; q < 16; q++) a += s0 + q < n_splits ? v[q] * f_s[s0 + q] : 0.f;
      }
    }
    o[d] = from_f32<T>(a);
  }
}

// ---------------------------------------------------------------------------------------------
// Whether the unrotated parts of q move in 16-byte pieces: sizes, the row stride and the addresses on that grid.
static bool latent_wide(int dtype, int dim, int dim_p, int stride, uintptr_t addr) {
  const int per = dtype == LEB_BF16 ? 8 : 4;
  return dim_p == dim && dim % per == 0 && stride % per == 0 && (addr & 15) == 0;
}

LEB_API int leb_latent_rows(void* qn, void* qr, const void* in, int ld_in, int dtype, void* pool, const int* block_table,
                            int bt_width, const int* row_seq, const int* row_pos, const int* seq_slot, const float* wkv,
                            float eps, const float* inv_freq, int rot_dims, int neox, int M, int H, int dim, int dim_p,
                            int rank, int rot, int page_size, cudaStream_t st) {
  if (M <= 0) return 0;
  LEB_REQUIRE(H >= 1 && dim >= 1 && dim_p >= dim && rot >= 0, "leb_latent_rows: sizes out of range");
  LEB_REQUIRE(!pool || (rank >= 1 && wkv && block_table && row_seq && seq_slot),
              "leb_latent_rows: a cache write needs the latent's size, its norm weight and the step's tables");
  LEB_REQUIRE(row_pos && rot_dims >= 0 && rot_dims <= rot && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq),
              "leb_latent_rows: %d rotated dimensions of %d", rot_dims, rot);
  LEB_REQUIRE(dtype == LEB_F32 || dtype == LEB_BF16, "leb_latent_rows: unknown dtype %d", dtype);
  const int wide = latent_wide(dtype, dim, dim_p, dim + rot, (uintptr_t)in | (uintptr_t)qn) && ld_in % (dtype == LEB_BF16 ? 8 : 4) == 0;
  LebPlainLaunches plain(true);
  const dim3 grid(M, pool ? 2 : 1), block(256);
  if (dtype == LEB_F32)
    leb_launch(latent_rows_kernel<float>, grid, block, 0, st, (float*)qn, (float*)qr, (const float*)in, ld_in, (float*)pool,
               block_table, bt_width, row_seq, row_pos, seq_slot, wkv, eps, inv_freq, rot_dims, neox, M, H, dim, dim_p, rank, rot,
               page_size, wide);
  else
    leb_launch(latent_rows_kernel<bf16>, grid, block, 0, st, (bf16*)qn, (bf16*)qr, (const bf16*)in, ld_in, (bf16*)pool,
               block_table, bt_width, row_seq, row_pos, seq_slot, wkv, eps, inv_freq, rot_dims, neox, M, H, dim, dim_p, rank, rot,
               page_size, wide);
  LEB_CHECK_LAUNCH("leb_latent_rows");
  return 0;
}

LEB_API int leb_latent_prep(void* cq, const void* in, int ld_in, int dtype, void* pool, const int* block_table,
                            int bt_width, const int* row_seq, const int* row_pos, const int* seq_slot,
                            const float* wq, const float* wkv, float eps, const float* inv_freq, int rot_dims,
                            int neox, int M, int q_rank, int rank, int rot, int page_size, cudaStream_t st) {
  if (M <= 0) return 0;
  LEB_REQUIRE(q_rank >= 1 && wq, "leb_latent_prep: the query latent needs a width and a norm weight");
  LEB_REQUIRE(!pool || (rank >= 1 && rot >= 0 && wkv && block_table && row_seq && row_pos && seq_slot),
              "leb_latent_prep: a cache write needs the latent's sizes, its norm weight and the step's tables");
  LEB_REQUIRE(rot_dims >= 0 && rot_dims <= rot && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq),
              "leb_latent_prep: %d rotated dimensions of %d", rot_dims, rot);
  LebPlainLaunches plain(true);
  if (dtype == LEB_F32)
    leb_launch(latent_prep_kernel<float, float>, dim3(M), dim3(128), 0, st, (float*)cq, (const float*)in, ld_in,
               (float*)pool, block_table, bt_width, row_seq, row_pos, seq_slot, wq, wkv, eps, inv_freq, rot_dims, neox,
               q_rank, rank, rot, page_size);
  else if (dtype == LEB_BF16)
    leb_launch(latent_prep_kernel<bf16, bf16>, dim3(M), dim3(128), 0, st, (bf16*)cq, (const bf16*)in, ld_in,
               (bf16*)pool, block_table, bt_width, row_seq, row_pos, seq_slot, wq, wkv, eps, inv_freq, rot_dims, neox,
               q_rank, rank, rot, page_size);
  else
    return leb_fail("leb_latent_prep: unknown dtype %d", dtype);
  LEB_CHECK_LAUNCH("leb_latent_prep");
  return 0;
}

LEB_API int leb_latent_q_split(void* qn, void* qr, const void* q, int dtype, const int* row_pos,
                               const float* inv_freq, int rot_dims, int neox, int M, int H, int dim, int dim_p, int rot,
                               cudaStream_t st) {
  if (M <= 0) return 0;
  LEB_REQUIRE(H >= 1 && dim >= 1 && dim_p >= dim && rot >= 0, "leb_latent_q_split: sizes out of range");
  LEB_REQUIRE(rot_dims >= 0 && rot_dims <= rot && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq),
              "leb_latent_q_split: %d rotated dimensions of %d", rot_dims, rot);
  const int wide = latent_wide(dtype, dim, dim_p, dim + rot, (uintptr_t)q | (uintptr_t)qn);
  LebPlainLaunches plain(true);
  if (dtype == LEB_F32)
    leb_launch(latent_q_split_kernel<float>, dim3(M), dim3(256), 0, st, (float*)qn, (float*)qr, (const float*)q,
               row_pos, inv_freq, rot_dims, neox, M, H, dim, dim_p, rot, wide);
  else if (dtype == LEB_BF16)
    leb_launch(latent_q_split_kernel<bf16>, dim3(M), dim3(256), 0, st, (bf16*)qn, (bf16*)qr, (const bf16*)q, row_pos,
               inv_freq, rot_dims, neox, M, H, dim, dim_p, rot, wide);
  else
    return leb_fail("leb_latent_q_split: unknown dtype %d", dtype);
  LEB_CHECK_LAUNCH("leb_latent_q_split");
  return 0;
}

LEB_API int leb_heads_to_rows(void* out, const void* in, int dtype, int M, int H, int w, cudaStream_t st) {
  if ((size_t)M * H * w == 0) return 0;
  LEB_REQUIRE(dtype == LEB_F32 || dtype == LEB_BF16, "leb_heads_to_rows: unknown dtype %d", dtype);
  LebPlainLaunches plain(true);
  const int per16 = dtype == LEB_F32 ? 4 : 8;      // elements of a 16-byte piece
  if (w % per16 == 0 && (((uintptr_t)out | (uintptr_t)in) & 15) == 0) {
    const size_t total = (size_t)M * H * (w / per16);
    leb_launch(heads_to_rows_kernel<uint4>, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, st, (uint4*)out,
               (const uint4*)in, M, H, w / per16);
  } else {
    const size_t total = (size_t)M * H * w;
    const dim3 grid((unsigned)((total + 255) / 256)), block(256);
    if (dtype == LEB_F32) leb_launch(heads_to_rows_kernel<float>, grid, block, 0, st, (float*)out, (const float*)in, M, H, w);
    else leb_launch(heads_to_rows_kernel<bf16>, grid, block, 0, st, (bf16*)out, (const bf16*)in, M, H, w);
  }
  LEB_CHECK_LAUNCH("leb_heads_to_rows");
  return 0;
}

template <typename T, int HDL>
static int launch_latent(void* out, int ld_out, float* part, const void* qt, const void* qr, const void* pool,
                         const int* block_table, int bt_width, const int* seq_slot, const int* seq_pos0,
                         const int* seq_qstart, const int* seq_qlen, const float* sink, int M, int B, int H, int rank,
                         int rot, int page_size, int window, int chunk, float scale, int max_qlen, int n_splits,
                         cudaStream_t st) {
  const int HC = H < 8 ? H : 8;
  int QT = 32 / HC;
  if (QT > max_qlen) QT = max_qlen;
  const int R = QT * HC;
  const int dk = rank + rot;
  const size_t smem = ((size_t)R * dk + 32 * (dk + 1) + LAT_WARPS * 32) * sizeof(float);
  auto kern = latent_attention_kernel<T, T, HDL>;
  static size_t smem_set = 0;
  if (smem > 48 * 1024 && smem > smem_set) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return leb_fail("leb_latent_attention: shared memory %zu: %s", smem, cudaGetErrorString(e));
    smem_set = smem;
  }
  dim3 grid(ceil_div(max_qlen, QT), ceil_div(H, HC), B * n_splits);
  LEB_REQUIRE(grid.y <= 65535 && grid.z <= 65535, "leb_latent_attention: grid too large (%u, %u)", grid.y, grid.z);
  leb_launch(kern, grid, dim3(32 * LAT_WARPS), smem, st, (T*)out, ld_out, part, (const T*)qt, (const T*)qr,
             (const T*)pool, block_table, bt_width, seq_slot, seq_pos0, seq_qstart, seq_qlen, sink, M, H, rank, rot,
             page_size, window, chunk, scale, QT, HC, n_splits);
  LEB_CHECK_LAUNCH("leb_latent_attention");
  return 0;
}

// The tensor-core kernel for bfloat16 (latent_attention_mma.cu) and its switch (on by default; off for comparisons).
extern "C" int leb_latent_attention_mma_supported(int rank, int rot, int page_size);
extern "C" int leb_latent_attention_mma(void* out, float* part, const void* qt, const void* qr, const void* pool,
                                        const int* block_table, int bt_width, const int* seq_slot, const int* seq_pos0,
                                        const int* seq_qstart, const int* seq_qlen, const float* sink, int M, int B, int H,
                                        int rank, int rot, int page_size, int window, int chunk, int wide,
                                        float scale, int max_qlen, int n_splits, cudaStream_t st);
static int g_latent_mma = 1;
LEB_API void leb_set_latent_mma(int on) { g_latent_mma = on ? 1 : 0; }

// qt [H, M, rank] (queries taken into the latent space), qr [M, H, rot] (rotated parts), pool
// [page][page_size][rank + rot], sink [H] float or null; out [H, M, ld_out] (ld_out >= rank, the
// rest zeros).  window / chunk > 0: a row reads its last `window` positions / its own chunk only; wide: the weights of
// the tensor-core kernel enter the product with the values as two terms (the general kernel's are float anyway).  part: float scratch of M*H*n_splits*(rank+2), used when n_splits > 1 (then every
// sequence brings one row).
LEB_API int leb_latent_attention(void* out, int ld_out, float* part, const void* qt, const void* qr, const void* pool,
                                 int dtype, const int* block_table, int bt_width, const int* seq_slot,
                                 const int* seq_pos0, const int* seq_qstart, const int* seq_qlen, const float* sink,
                                 int M, int B, int H, int rank, int rot, int page_size, int window, int chunk, int wide,
                                 float scale, int max_qlen, int n_splits, cudaStream_t st) {
  if (M <= 0 || B <= 0) return 0;
  LEB_REQUIRE(rank >= 1 && rank <= 512, "leb_latent_attention: latent size %d outside 1..512", rank);
  LEB_REQUIRE(rot >= 0 && rot <= 256, "leb_latent_attention: %d rotated dimensions outside 0..256", rot);
  LEB_REQUIRE(ld_out >= rank, "leb_latent_attention: result rows of %d for a latent of %d", ld_out, rank);
  LEB_REQUIRE(page_size % 32 == 0, "leb_latent_attention: page size %d is not a multiple of 32", page_size);
  LEB_REQUIRE(n_splits >= 1 && n_splits <= 64 && (n_splits == 1 || (max_qlen == 1 && part)),
              "leb_latent_attention: up to 64 splits, and they need single-row sequences and scratch");
  LebPlainLaunches plain(true);
  int rc;
  const bool mma = g_latent_mma && dtype == LEB_BF16 && ld_out == rank && leb_latent_attention_mma_supported(rank, rot, page_size) &&
                   (((uintptr_t)qt | (uintptr_t)qr | (uintptr_t)pool) & 15) == 0;
#define LEB_LAT(T, L)                                                                                              \
  launch_latent<T, L>(out, ld_out, part, qt, qr, pool, block_table, bt_width, seq_slot, seq_pos0, seq_qstart, seq_qlen, \
                      sink, M, B, H, rank, rot, page_size, window, chunk, scale, max_qlen, n_splits, st)
#define LEB_LAT_T(T) \
  (rank <= 32 ? LEB_LAT(T, 1) : rank <= 64 ? LEB_LAT(T, 2) : rank <= 128 ? LEB_LAT(T, 4) : rank <= 256 ? LEB_LAT(T, 8) : LEB_LAT(T, 16))
  if (mma)
    rc = leb_latent_attention_mma(out, part, qt, qr, pool, block_table, bt_width, seq_slot, seq_pos0, seq_qstart, seq_qlen,
                                  sink, M, B, H, rank, rot, page_size, window, chunk, wide, scale, max_qlen, n_splits, st);
  else if (dtype == LEB_F32) rc = LEB_LAT_T(float);
  else if (dtype == LEB_BF16) rc = LEB_LAT_T(bf16);
  else return leb_fail("leb_latent_attention: unknown dtype %d", dtype);
#undef LEB_LAT_T
#undef LEB_LAT
  if (rc) return rc;
  if (n_splits > 1) {
    dim3 grid(M, H), block(ld_out >= 512 ? 512 : ceil_div(ld_out, 32) * 32);
    if (dtype == LEB_F32)
      leb_launch(latent_merge_kernel<float>, grid, block, 0, st, (float*)out, ld_out, part, sink, M, H, rank, n_splits);
    else
      leb_launch(latent_merge_kernel<bf16>, grid, block, 0, st, (bf16*)out, ld_out, part, sink, M, H, rank, n_splits);
    LEB_CHECK_LAUNCH("leb_latent_attention merge");
  }
  return 0;
}
