// RMSNorm on q and k (per head, or over the whole projected row), rotary position encoding, and the write of k and v into the
// paged cache, one launch for all rows of a step.
//
// Order as in the reference (src/dense.rs:119-128): norm each head of q and k over head_dim with
// the shared [head_dim] weights and the model's eps, then rotate, then append k and v at the
// token's position.  Rotation (src/dense.rs:103-111): half = rope_dim/2, angle_i = pos * inv_freq[i]
// with inv_freq[i] = theta^(-2i/rope_dim) (divided by a frequency factor where the model has one);
// split-half pairing (i, i+half) or adjacent pairing (2i, 2i+1); a' = a cos - b sin,
// b' = a sin + b cos.  The reference does the three jobs in one decode launch too
// (src/cuda/dense.cu:80-93); here the same launch also serves prompts.
// Norm, angle, sine and cosine are float; sinf/cosf are the full-range versions.
//
// Cache layout of one layer: keys [page][kv_head][page_size][head_dim]; values transposed,
// [page][kv_head][head_dim][page_size], so that the positions of a page are contiguous for each
// dimension (the tensor-core attention kernels contract over positions and read them 8 at a
// time).  The page of position p of sequence b is block_table[b][p / page_size].
#include "common.cuh"

constexpr int ROPE_WARPS = 8;   // warps of a block; each takes one head of the block's row
constexpr int VT_ROWS = 32;     // rows of a value tile
constexpr int VT_DIMS = 64;     // dimensions of a value tile

// A tile of VT_ROWS rows of one kv head's values, turned through shared memory so that a warp
// writes 32 consecutive positions of one dimension (64 bytes in bfloat16) instead of 32
// scattered elements.  Every row's page and offset is looked up on its own, so rows of
// different sequences or pages in one tile are fine.
template <typename T, typename CT>
__device__ __forceinline__ void store_value_tile(
    int t, const T* __restrict__ v_in, int kv_stride, CT* __restrict__ v_pool,
    const int* __restrict__ block_table, int bt_width, const int* __restrict__ row_seq,
    const int* __restrict__ row_pos, const int* __restrict__ seq_slot, int M, int nkv, int hd,
    int page_size, int v_norm, float eps, int vin) {      // hd: the head's width in the pool; vin <= hd: in v_in (the rest is stored as zeros)
  constexpr int LD = VT_DIMS + (sizeof(CT) == 2 ? 2 : 1);     // odd number of 32-bit words
  __shared__ CT tile[VT_ROWS * LD];
  __shared__ long long dst[VT_ROWS];                          // element offset of (row, dim 0), or -1
  __shared__ float rs[VT_ROWS];                               // 1 / root mean square of the row's head, or 1
  const int kvh = t % nkv, m0 = (t / nkv) * VT_ROWS;
  if (threadIdx.x < VT_ROWS) {
    int m = m0 + threadIdx.x;
    long long off = -1;
    if (m < M) {
      int b = row_seq[m], pos = row_pos[m];
      if (seq_slot[b] >= 0) {
        int page = block_table[(size_t)b * bt_width + pos / page_size];
        if (page >= 0) off = ((long long)page * nkv + kvh) * hd * page_size + pos % page_size;
      }
    }
    dst[threadIdx.x] = off;
  }
  // values divided by their root mean square over the head (no weight) where the layer asks for it
  for (int r = threadIdx.x >> 5; r < VT_ROWS; r += blockDim.x >> 5) {
    float ss = 0.f;
    if (v_norm && m0 + r < M)
      for (int d = threadIdx.x & 31; d < vin; d += 32) {
        float x = to_f32(v_in[(size_t)(m0 + r) * kv_stride + (size_t)kvh * vin + d]);
        ss += x * x;
      }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) rs[r] = v_norm ? 1.0f / sqrtf(ss / (float)vin + eps) : 1.f;
  }
  for (int d0 = 0; d0 < hd; d0 += VT_DIMS) {
    int nd = min(VT_DIMS, hd - d0);
    __syncthreads();
    for (int i = threadIdx.x; i < VT_ROWS * VT_DIMS; i += blockDim.x) {
      int r = i / VT_DIMS, d = i % VT_DIMS;
      if (d < nd && m0 + r < M)
        tile[r * LD + d] = d0 + d < vin
            ? from_f32<CT>(to_f32(v_in[(size_t)(m0 + r) * kv_stride + (size_t)kvh * vin + d0 + d]) * rs[r])
            : from_f32<CT>(0.f);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < VT_ROWS * VT_DIMS; i += blockDim.x) {
      int d = i / VT_ROWS, r = i % VT_ROWS;
      if (d < nd && dst[r] >= 0) v_pool[dst[r] + (size_t)(d0 + d) * page_size] = tile[r * LD + d];
    }
  }
}

// Blocks (x < M, y): row x, heads [8y, 8y + 8) of its q and k heads, one per warp: norm, rotate
// (sine and cosine of the row's position are computed once per block, not per head), write q
// and the cached k.  Blocks (x in [M, M + tiles * nkv), y = 0): a value tile.
template <typename T, typename CT>
__global__ void __launch_bounds__(ROPE_WARPS * 32) qk_rope_store_kernel(
    T* __restrict__ q_out, const T* __restrict__ q_in, int q_stride, const T* __restrict__ k_in,
    const T* __restrict__ v_in, int kv_stride, CT* __restrict__ k_pool, CT* __restrict__ v_pool,
    const int* __restrict__ block_table, int bt_width, const int* __restrict__ row_seq,
    const int* __restrict__ row_pos, const int* __restrict__ seq_slot,
    const float* __restrict__ q_norm_w, const float* __restrict__ k_norm_w, float eps,
    const float* __restrict__ inv_freq, int rope_dim, int neox, int M, int nh, int nkv, int hd,
    int page_size, int vd, int v_norm, int hin, int vin,     // hin <= hd, vin <= vd: a head's width in q_in/k_in and v_in
    float temp_coef, float temp_every) {                     // q times query_temperature(position) (coef 0: as it is)
  extern __shared__ float sm[];
  pdl_trigger();   // the kernel after this one may start and wait (see common.cuh)
  pdl_wait();
  int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if ((int)blockIdx.x >= M) {
    if (blockIdx.y == 0)
      store_value_tile<T, CT>(blockIdx.x - M, v_in, kv_stride, v_pool, block_table, bt_width, row_seq, row_pos,
                              seq_slot, M, nkv, vd, page_size, v_norm, eps, vin);
    return;
  }
  // ---- one row: q and k heads ----
  int m = blockIdx.x;
  int b = row_seq[m];
  int slot = seq_slot[b];
  int pos = row_pos[m];
  int half = rope_dim / 2;
  float* cs = sm;                                   // [half] cosine, [half] sine
  float* v = sm + 2 * half + warp * hd;             // one head vector per warp
  if (inv_freq) {
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      float th = (float)pos * inv_freq[i];
      cs[i] = cosf(th);
      cs[half + i] = sinf(th);
    }
  }
  __syncthreads();
  int total = nh + (k_in ? nkv : 0);
  long long kdst = -1;
  if (k_in && slot >= 0) {
    int page = block_table[(size_t)b * bt_width + pos / page_size];
    if (page >= 0) kdst = ((long long)page * nkv * page_size + pos % page_size) * hd;
  }
  int head = blockIdx.y * ROPE_WARPS + warp;
  if (head < total) {
    bool is_q = head < nh;
    if (!is_q && kdst < 0) return;  // padding rows and positions outside a window own no cache
    const T* src = is_q ? q_in + (size_t)m * q_stride + (size_t)head * hin
                        : k_in + (size_t)m * kv_stride + (size_t)(head - nh) * hin;
    const float* nw = is_q ? q_norm_w : k_norm_w;
    float ss = 0.f;
    for (int i = lane; i < hd; i += 32) {
      float x = i < hin ? to_f32(src[i]) : 0.f;      // a head stored wider than it is: zeros behind it
      v[i] = x;
      ss += x * x;
    }
    if (nw) {
      ss = warp_sum(ss);
      float r = 1.0f / sqrtf(ss / (float)hin + eps);
      __syncwarp();
      for (int i = lane; i < hin; i += 32) v[i] = v[i] * r * nw[i];
    }
    __syncwarp();
    if (inv_freq) {
      for (int i = lane; i < half; i += 32) {
        float c = cs[i], s = cs[half + i];
        int ia = neox ? i : 2 * i, ib = neox ? i + half : 2 * i + 1;
        float a = v[ia], bb = v[ib];
        v[ia] = a * c - bb * s;
        v[ib] = a * s + bb * c;
      }
    }
    __syncwarp();
    if (is_q) {
      T* o = q_out + ((size_t)m * nh + head) * hd;
      const float factor = query_temperature(pos, temp_coef, temp_every);
      for (int i = lane; i < hd; i += 32) o[i] = from_f32<T>(v[i] * factor);
    } else {
      CT* o = k_pool + kdst + (size_t)(head - nh) * page_size * hd;
      for (int i = lane; i < hd; i += 32) o[i] = from_f32<CT>(v[i]);
    }
  }
}

// The usual case (split-half pairing over the whole head, head size 64 or 128) without shared
// memory: a lane holds elements lane, lane + 32, ... of a head, so both halves of a rotation
// pair are in the same lane.  A warp takes `per_warp` consecutive heads of its row, four at a
// time so that their loads are in flight together; sine and cosine are formed once per warp.
// Same operations in the same order as the kernel above: the results are the same bit for bit.
template <typename T, typename CT, int EPL>
__global__ void __launch_bounds__(ROPE_WARPS * 32) qk_rope_store_lanes_kernel(
    T* __restrict__ q_out, const T* __restrict__ q_in, int q_stride, const T* __restrict__ k_in,
    const T* __restrict__ v_in, int kv_stride, CT* __restrict__ k_pool, CT* __restrict__ v_pool,
    const int* __restrict__ block_table, int bt_width,
    const int* __restrict__ row_seq, const int* __restrict__ row_pos, const int* __restrict__ seq_slot,
    const float* __restrict__ q_norm_w, const float* __restrict__ k_norm_w, float eps,
    const float* __restrict__ inv_freq, int M, int nh, int nkv, int page_size, int per_warp, int vd, int v_norm, int vin,
    float temp_coef, float temp_every) {
  constexpr int HD = EPL * 32, NP = EPL / 2, U = 4;
  pdl_trigger();   // the kernel after this one may start and wait (see common.cuh)
  pdl_wait();
  if ((int)blockIdx.x >= M) {
    if (blockIdx.y == 0)
      store_value_tile<T, CT>(blockIdx.x - M, v_in, kv_stride, v_pool, block_table, bt_width, row_seq, row_pos,
                              seq_slot, M, nkv, vd, page_size, v_norm, eps, vin);
    return;
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int m = blockIdx.x;
  const int total = nh + (k_in ? nkv : 0);
  const int h0 = (blockIdx.y * ROPE_WARPS + warp) * per_warp;
  if (h0 >= total) return;
  const int h1 = min(h0 + per_warp, total);
  const int b = row_seq[m], pos = row_pos[m];
  long long kdst = -1;
  if (h1 > nh && seq_slot[b] >= 0) {
    const int page = block_table[(size_t)b * bt_width + pos / page_size];
    if (page >= 0) kdst = ((long long)page * nkv * page_size + pos % page_size) * HD;
  }
  float c[NP], sn[NP], wq[EPL], wk[EPL];
#pragma unroll
  for (int p = 0; p < NP; p++) {
    const float th = inv_freq ? (float)pos * inv_freq[lane + 32 * p] : 0.f;     // no rotation: turned by zero
    c[p] = cosf(th);
    sn[p] = sinf(th);
  }
#pragma unroll
  for (int e = 0; e < EPL; e++) {
    wq[e] = q_norm_w ? q_norm_w[lane + 32 * e] : 1.f;
    wk[e] = k_norm_w ? k_norm_w[lane + 32 * e] : 1.f;
  }
  const float factor = query_temperature(pos, temp_coef, temp_every);
  for (int hb = h0; hb < h1; hb += U) {
    float x[U][EPL];
#pragma unroll
    for (int u = 0; u < U; u++) {
      const int head = hb + u;
      if (head < h1) {
        const T* src = head < nh ? q_in + (size_t)m * q_stride + (size_t)head * HD
                                 : k_in + (size_t)m * kv_stride + (size_t)(head - nh) * HD;
#pragma unroll
        for (int e = 0; e < EPL; e++) x[u][e] = to_f32(src[lane + 32 * e]);
      } else {
#pragma unroll
        for (int e = 0; e < EPL; e++) x[u][e] = 0.f;
      }
    }
#pragma unroll
    for (int u = 0; u < U; u++) {
      const int head = hb + u;
      if (head >= h1) break;
      const bool is_q = head < nh;
      if (!is_q && kdst < 0) continue;
      if (is_q ? q_norm_w != nullptr : k_norm_w != nullptr) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < EPL; e++) ss += x[u][e] * x[u][e];
        ss = warp_sum(ss);
        const float r = 1.0f / sqrtf(ss / (float)HD + eps);
#pragma unroll
        for (int e = 0; e < EPL; e++) x[u][e] = x[u][e] * r * (is_q ? wq[e] : wk[e]);
      }
#pragma unroll
      for (int p = 0; p < NP; p++) {
        const float a = x[u][p], bb = x[u][p + NP];
        x[u][p] = a * c[p] - bb * sn[p];
        x[u][p + NP] = a * sn[p] + bb * c[p];
      }
      if (is_q) {
        T* o = q_out + ((size_t)m * nh + head) * HD;
#pragma unroll
        for (int e = 0; e < EPL; e++) o[lane + 32 * e] = from_f32<T>(x[u][e] * factor);
      } else {
        CT* o = k_pool + kdst + (size_t)(head - nh) * page_size * HD;
#pragma unroll
        for (int e = 0; e < EPL; e++) o[lane + 32 * e] = from_f32<CT>(x[u][e]);
      }
    }
  }
}

// The same job where q and k are normed over their whole projected row (all heads at once, a weight per number of the
// row) instead of head by head.  Block (m, 0): row m's q, block (m, 1): its k (sum of squares, norm, rotation, q out or
// cache write); blocks (x >= M, 0): value tiles as above.
// FAST (bfloat16, adjacent pairs, heads stored as wide as they are and a multiple of 8): a thread keeps its pieces of
// eight numbers in registers (up to NC of them) between the sum and the rotation.
template <typename T, typename CT, bool FAST, int NC>
__global__ void __launch_bounds__(256) qk_row_norm_rope_store_kernel(
    T* __restrict__ q_out, const T* __restrict__ q_in, int q_stride, const T* __restrict__ k_in,
    const T* __restrict__ v_in, int kv_stride, CT* __restrict__ k_pool, CT* __restrict__ v_pool,
    const int* __restrict__ block_table, int bt_width, const int* __restrict__ row_seq,
    const int* __restrict__ row_pos, const int* __restrict__ seq_slot,
    const float* __restrict__ q_norm_w, const float* __restrict__ k_norm_w, float eps,
    const float* __restrict__ inv_freq, int rope_dim, int neox, int M, int nh, int nkv, int hd,
    int page_size, int vd, int hin, int vin) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33];
  pdl_wait();
  if ((int)blockIdx.x >= M) {
    if (blockIdx.y == 0)
      store_value_tile<T, CT>(blockIdx.x - M, v_in, kv_stride, v_pool, block_table, bt_width, row_seq, row_pos,
                              seq_slot, M, nkv, vd, page_size, 0, eps, vin);
    return;
  }
  const int m = blockIdx.x;
  const bool is_q = blockIdx.y == 0;
  const int b = row_seq[m], pos = row_pos[m];
  const int heads = is_q ? nh : nkv, n = heads * hin, half = rope_dim / 2;
  CT* kbase = nullptr;
  if (!is_q) {
    if (seq_slot[b] < 0) return;     // padding rows and positions outside what the layer keeps own no cache
    const int page = block_table[(size_t)b * bt_width + pos / page_size];
    if (page < 0) return;
    kbase = k_pool + ((size_t)page * nkv * page_size + pos % page_size) * hd;
  }
  const T* src = is_q ? q_in + (size_t)m * q_stride : k_in + (size_t)m * kv_stride;
  const float* nw = is_q ? q_norm_w : k_norm_w;
  float* cs = sm;                    // [half] cosine, [half] sine
  float* row = sm + rope_dim;        // [heads * hin] (not FAST)
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float th = (float)pos * inv_freq[i];
    cs[i] = cosf(th);
    cs[half + i] = sinf(th);
  }
  float ss = 0.f;
  if constexpr (FAST) {
    const int pieces = n / 8, ppd = hd / 8;
    uint4 v[NC];
#pragma unroll
    for (int c = 0; c < NC; c++) {
      const int p = threadIdx.x + c * 256;
      if (p < pieces) {
        v[c] = reinterpret_cast<const uint4*>(src)[p];
        const bf16* e = reinterpret_cast<const bf16*>(&v[c]);
#pragma unroll
        for (int j = 0; j < 8; j++) ss += to_f32(e[j]) * to_f32(e[j]);
      }
    }
    ss = block_sum(ss, red);
    const float r = 1.0f / sqrtf(ss / (float)n + eps);
#pragma unroll
    for (int c = 0; c < NC; c++) {
      const int p = threadIdx.x + c * 256;
      if (p >= pieces) break;
      const int h = p / ppd, d0 = (p - h * ppd) * 8;
      const bf16* e = reinterpret_cast<const bf16*>(&v[c]);
      const float4 wa = reinterpret_cast<const float4*>(nw)[2 * p], wb = reinterpret_cast<const float4*>(nw)[2 * p + 1];
      const float ww[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
      uint4 o;
      uint32_t* op = reinterpret_cast<uint32_t*>(&o);
#pragma unroll
      for (int j = 0; j < 4; j++) {
        float a = to_f32(e[2 * j]) * r * ww[2 * j], bb = to_f32(e[2 * j + 1]) * r * ww[2 * j + 1];
        const int pi = d0 / 2 + j;
        if (pi < half) {
          const float c0 = cs[pi], s0 = cs[half + pi];
          const float a2 = a * c0 - bb * s0;
          bb = a * s0 + bb * c0;
          a = a2;
        }
        __nv_bfloat162 two = __floats2bfloat162_rn(a, bb);
        op[j] = *reinterpret_cast<uint32_t*>(&two);
      }
      CT* dst = is_q ? (CT*)(q_out + ((size_t)m * nh + h) * hd) : kbase + (size_t)h * page_size * hd;
      *reinterpret_cast<uint4*>(dst + d0) = o;
    }
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      const float x = to_f32(src[i]);
      row[i] = x;
      ss += x * x;
    }
    ss = block_sum(ss, red);
    const float r = 1.0f / sqrtf(ss / (float)n + eps);
    // units of a head: `half` rotated pairs, then the numbers that pass, then the zeros a wider stored head ends with
    const int units = half + hd - rope_dim;
    for (int i = threadIdx.x; i < heads * units; i += blockDim.x) {
      const int h = i / units, u = i - h * units;
      const float* hv = row + h * hin;
      const float* hw = nw + h * hin;
      T* qo = q_out + ((size_t)m * nh + h) * hd;
      CT* ko = is_q ? nullptr : kbase + (size_t)h * page_size * hd;
      if (u < half) {
        const int ia = neox ? u : 2 * u, ib = neox ? u + half : 2 * u + 1;
        const float a = hv[ia] * r * hw[ia], bb = hv[ib] * r * hw[ib];
        const float oa = a * cs[u] - bb * cs[half + u], ob = a * cs[half + u] + bb * cs[u];
        if (is_q) { qo[ia] = from_f32<T>(oa); qo[ib] = from_f32<T>(ob); }
        else { ko[ia] = from_f32<CT>(oa); ko[ib] = from_f32<CT>(ob); }
      } else {
        const int d = rope_dim + u - half;
        const float a = d < hin ? hv[d] * r * hw[d] : 0.f;
        if (is_q) qo[d] = from_f32<T>(a);
        else ko[d] = from_f32<CT>(a);
      }
    }
  }
}

// q, k and v of a step's rows: the root mean square of the whole q row and of the whole k row (weights [nh * hin] and
// [nkv * hin]), rotation of every head, q out and the write of k and v into the pages.  k_in null: q alone.
LEB_API int leb_qk_row_norm_rope_store(void* q_out, const void* q_in, int q_stride, const void* k_in,
                                       const void* v_in, int kv_stride, void* k_pool, void* v_pool,
                                       int dtype, const int* block_table, int bt_width, const int* row_seq,
                                       const int* row_pos, const int* seq_slot, const float* q_norm_w,
                                       const float* k_norm_w, float eps, const float* inv_freq, int rope_dim,
                                       int neox, int M, int nh, int nkv, int hd, int page_size, int vd,
                                       int hin, int vin, cudaStream_t st) {
  if (M <= 0) return 0;
  if (!inv_freq) rope_dim = 0;
  if (hin <= 0) hin = hd;
  if (vd <= 0) vd = hd;
  if (vin <= 0) vin = vd;
  LEB_REQUIRE(nh >= 1 && nkv >= 1 && hd >= 1 && hin <= hd && vin <= vd && rope_dim >= 0 && rope_dim <= hin && rope_dim % 2 == 0,
              "leb_qk_row_norm_rope_store: heads %d/%d of %d (stored %d), %d rotated, values of %d (stored %d)", nh, nkv, hin, hd,
              rope_dim, vin, vd);
  LEB_REQUIRE(q_norm_w && (!k_in || k_norm_w), "leb_qk_row_norm_rope_store: the rows' norm weights are required");
  LEB_REQUIRE(dtype == LEB_F32 || dtype == LEB_BF16, "leb_qk_row_norm_rope_store: unknown dtype %d", dtype);
  const int tiles = k_in ? ceil_div(M, VT_ROWS) * nkv : 0;
  LebPlainLaunches plain(true);
  const dim3 grid(M + tiles, k_in ? 2 : 1), block(256);
  const int wide = (nh > nkv ? nh : nkv) * hin;
  const uintptr_t al = (uintptr_t)q_out | (uintptr_t)q_in | (uintptr_t)k_in | (uintptr_t)k_pool | (uintptr_t)q_norm_w | (uintptr_t)k_norm_w;
  const bool fast = dtype == LEB_BF16 && (!neox || rope_dim == 0) && hin == hd && hd % 8 == 0 && wide <= 8 * 256 * 4 &&
                    (al & 15) == 0 && q_stride % 8 == 0 && kv_stride % 8 == 0;
#define LEB_QRN_ARGS(T)                                                                                                    \
  (T*)q_out, (const T*)q_in, q_stride, (const T*)k_in, (const T*)v_in, kv_stride, (T*)k_pool, (T*)v_pool, block_table,     \
      bt_width, row_seq, row_pos, seq_slot, q_norm_w, k_norm_w, eps, inv_freq, rope_dim, neox, M, nh, nkv, hd, page_size, vd, hin, vin
  if (fast) {
    const size_t smem = (size_t)rope_dim * sizeof(float);
    if (wide <= 8 * 256) leb_launch(qk_row_norm_rope_store_kernel<bf16, bf16, true, 1>, grid, block, smem, st, LEB_QRN_ARGS(bf16));
    else if (wide <= 8 * 256 * 2) leb_launch(qk_row_norm_rope_store_kernel<bf16, bf16, true, 2>, grid, block, smem, st, LEB_QRN_ARGS(bf16));
    else leb_launch(qk_row_norm_rope_store_kernel<bf16, bf16, true, 4>, grid, block, smem, st, LEB_QRN_ARGS(bf16));
  } else {
    const size_t smem = (size_t)(rope_dim + wide) * sizeof(float);
    LEB_REQUIRE(smem <= 200 * 1024, "leb_qk_row_norm_rope_store: a row of %d numbers does not fit shared memory", wide);
    static bool set = false;
    if (smem > 40 * 1024 && !set) {
      cudaFuncSetAttribute(qk_row_norm_rope_store_kernel<float, float, false, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      cudaFuncSetAttribute(qk_row_norm_rope_store_kernel<bf16, bf16, false, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      set = true;
    }
    if (dtype == LEB_F32)
      leb_launch(qk_row_norm_rope_store_kernel<float, float, false, 1>, grid, block, smem, st, LEB_QRN_ARGS(float));
    else
      leb_launch(qk_row_norm_rope_store_kernel<bf16, bf16, false, 1>, grid, block, smem, st, LEB_QRN_ARGS(bf16));
  }
#undef LEB_QRN_ARGS
  LEB_CHECK_LAUNCH("leb_qk_row_norm_rope_store");
  return 0;
}

LEB_API int leb_qk_rope_store(void* q_out, const void* q_in, int q_stride, const void* k_in,
                              const void* v_in, int kv_stride, void* k_pool, void* v_pool,
                              int dtype, const int* block_table, int bt_width, const int* row_seq,
                              const int* row_pos, const int* seq_slot, const float* q_norm_w,
                              const float* k_norm_w, float eps, const float* inv_freq, int rope_dim,
                              int neox, int M, int nh, int nkv, int hd, int page_size, int vd, int v_norm,
                              int hin, int vin, float temp_coef, float temp_every, cudaStream_t st) {
  if (M <= 0) return 0;
  if (!inv_freq) rope_dim = 0;
  LEB_REQUIRE(temp_coef == 0.f || temp_every > 0.f, "leb_qk_rope_store: a temperature that rises every %g positions", temp_every);
  LEB_REQUIRE(hd >= 2 && hd <= 512, "leb_qk_rope_store: head_dim %d outside 2..512", hd);
  LEB_REQUIRE(rope_dim <= hd && rope_dim % 2 == 0, "leb_qk_rope_store: rope_dim %d does not fit head_dim %d", rope_dim, hd);
  if (vd <= 0) vd = hd;      // values as wide as keys
  if (hin <= 0) hin = hd;    // heads come as wide as they are stored
  if (vin <= 0) vin = vd;
  LEB_REQUIRE(hin <= hd && vin <= vd && rope_dim <= hin, "leb_qk_rope_store: heads of %d/%d do not fit their stored width %d/%d", hin, vin, hd, vd);
  int tiles = k_in ? ceil_div(M, VT_ROWS) * nkv : 0;
  int total = nh + (k_in ? nkv : 0);
  dim3 block(32 * ROPE_WARPS);
  if (dtype == LEB_BF16 && (inv_freq ? neox && rope_dim == hd : temp_coef != 0.f) && hin == hd && (hd == 64 || hd == 128)) {
    // heads per warp: one while the launch is small, up to all of a row's over 8 warps
    int per_warp = 1;
    const long long n_sm = sm_count();
    while (per_warp * ROPE_WARPS < total && (long long)M * ceil_div(total, per_warp * ROPE_WARPS) > 4 * n_sm) per_warp++;
    dim3 grid(M + tiles, ceil_div(total, per_warp * ROPE_WARPS));
    if (hd == 64)
      leb_launch(qk_rope_store_lanes_kernel<bf16, bf16, 2>, grid, block, 0, st,
          (bf16*)q_out, (const bf16*)q_in, q_stride, (const bf16*)k_in, (const bf16*)v_in, kv_stride,
          (bf16*)k_pool, (bf16*)v_pool, block_table, bt_width, row_seq, row_pos, seq_slot, q_norm_w,
          k_norm_w, eps, inv_freq, M, nh, nkv, page_size, per_warp, vd, v_norm, vin, temp_coef, temp_every);
    else
      leb_launch(qk_rope_store_lanes_kernel<bf16, bf16, 4>, grid, block, 0, st,
          (bf16*)q_out, (const bf16*)q_in, q_stride, (const bf16*)k_in, (const bf16*)v_in, kv_stride,
          (bf16*)k_pool, (bf16*)v_pool, block_table, bt_width, row_seq, row_pos, seq_slot, q_norm_w,
          k_norm_w, eps, inv_freq, M, nh, nkv, page_size, per_warp, vd, v_norm, vin, temp_coef, temp_every);
    LEB_CHECK_LAUNCH("leb_qk_rope_store");
    return 0;
  }
  dim3 grid(M + tiles, ceil_div(total, ROPE_WARPS));
  size_t smem = (size_t)(rope_dim + ROPE_WARPS * hd) * sizeof(float);
  if (dtype == LEB_F32)
    leb_launch(qk_rope_store_kernel<float, float>, grid, block, smem, st,
        (float*)q_out, (const float*)q_in, q_stride, (const float*)k_in, (const float*)v_in,
        kv_stride, (float*)k_pool, (float*)v_pool, block_table, bt_width, row_seq, row_pos,
        seq_slot, q_norm_w, k_norm_w, eps, inv_freq, rope_dim, neox, M, nh, nkv, hd, page_size, vd, v_norm, hin, vin,
        temp_coef, temp_every);
  else if (dtype == LEB_BF16)
    leb_launch(qk_rope_store_kernel<bf16, bf16>, grid, block, smem, st,
        (bf16*)q_out, (const bf16*)q_in, q_stride, (const bf16*)k_in, (const bf16*)v_in, kv_stride,
        (bf16*)k_pool, (bf16*)v_pool, block_table, bt_width, row_seq, row_pos, seq_slot, q_norm_w,
        k_norm_w, eps, inv_freq, rope_dim, neox, M, nh, nkv, hd, page_size, vd, v_norm, hin, vin,
        temp_coef, temp_every);
  else
    return leb_fail("leb_qk_rope_store: unknown dtype %d", dtype);
  LEB_CHECK_LAUNCH("leb_qk_rope_store");
  return 0;
}
