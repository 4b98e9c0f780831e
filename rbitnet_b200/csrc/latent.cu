// Attention through latents: what stands between the down-projections and the attention kernels.
//
//   latent_norm_append_kernel  rows float32 [T, ...] of the stacked down-projections, holding the query latent (q_rank
//                              values at q_off), the key/value latent (kv_rank values at kv_off) and, right behind
//                              it, a key part of rot_dim values that all heads share.  Each latent is divided by its
//                              root mean square (eps inside the root) and multiplied by its weight; the key part is
//                              turned by position.  The query latent leaves as a row of the compute dtype for the
//                              up-projection; the other two are what the cache keeps per position: one "head" of
//                              `width` values [latent | turned key part | zeros] in the sequence's page.
//   latent_queries_few_kernel  query heads [q_c (D) | q_r (R)] into the latent's space, for few rows: per head
//                              [W_h q_c | turned q_r | zeros] of the cache row's width
//   latent_turn_kernel         for many rows the product W_h q_c is a product of its own; this kernel fills in the rest
//                              of every head's row, [turned q_r | zeros]
//
// All arithmetic is float32.
#include "rb_rotary.cuh"

namespace {

template <typename T>
__global__ void __launch_bounds__(256) latent_norm_append_kernel(
    T* __restrict__ cq, const float* __restrict__ rows, int64_t ld, int q_off, int kv_off, int q_rank, int kv_rank,
    int rot_dim, const float* __restrict__ wq, const float* __restrict__ wkv, float eps, const double* __restrict__ freq,
    float magnitude, int interleaved, RbPagedLayer cache, int width, const int* __restrict__ tok_pos,
    const int* __restrict__ tok_slot) {
  rb_pdl_launch_dependents();
  __shared__ float scratch[33];
  extern __shared__ float s_sincos[];
  rb_pdl_wait();
  const int t = blockIdx.x;
  const int pos = tok_pos[t];
  const float* row = rows + (int64_t)t * ld;
  // (the block's last threads make the sines and cosines while the others start on the sums)
  for (int i = (int)(blockDim.x - 1 - threadIdx.x); i < rot_dim / 2; i += blockDim.x)
    angle_sincos(pos, freq[i], magnitude, &s_sincos[i], &s_sincos[rot_dim / 2 + i]);
  float ss = 0.f;
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) ss = fmaf(row[q_off + i], row[q_off + i], ss);
  ss = rb_block_sum(ss, scratch);
  const float rq = 1.0f / sqrtf(ss / (float)q_rank + eps);
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x)
    cq[(int64_t)t * q_rank + i] = rb_from_float<T>(row[q_off + i] * rq * wq[i]);
  ss = 0.f;
  for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) ss = fmaf(row[kv_off + i], row[kv_off + i], ss);
  ss = rb_block_sum(ss, scratch);                            // also the barrier after the table's writes
  const float rk = 1.0f / sqrtf(ss / (float)kv_rank + eps);
  T* dst = reinterpret_cast<T*>(cache.k) + rb_page_offset(cache, tok_slot[t], pos, 0);
  const float* key = row + kv_off + kv_rank;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float y = 0.f;
    if (i < kv_rank) {
      y = row[kv_off + i] * rk * wkv[i];
    } else if (i < kv_rank + rot_dim) {
      auto val = [&](int e) { return key[e]; };
      y = turned(val, i - kv_rank, rot_dim, interleaved, s_sincos);
    }
    dst[i] = rb_from_float<T>(y);
  }
}

// A warp makes one value of one head's row for up to eight rows at a time, its lanes sharing the D inner values, so
// that the head's matrix is read once; a value of the turned part is made by a lane per row.
constexpr int FEW_ROWS = 8;
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) latent_queries_few_kernel(
    T* __restrict__ out, const T* __restrict__ q, const T* __restrict__ W, const double* __restrict__ freq, float magnitude,
    int interleaved, const int* __restrict__ tok_pos, int M, int H, int D, int R, int C, int width) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, n = blockIdx.x * 8 + warp;
  if (n >= width) return;
  const int Dq = D + R;
  const int64_t ldq = (int64_t)H * Dq, ldo = (int64_t)H * width;
  const T* qh = q + (int64_t)h * Dq;
  T* dst = out + (int64_t)h * width + n;
  if (n >= C) {
    for (int m = lane; m < M; m += 32) {
      float y = 0.f;
      const int e = n - C;
      if (e < R) {
        const int half = R >> 1;
        int pair, other;
        bool first;
        if (interleaved) { pair = e >> 1; first = (e & 1) == 0; other = first ? e + 1 : e - 1; }
        else { first = e < half; pair = first ? e : e - half; other = first ? e + half : e - half; }
        float sn, cs;
        angle_sincos(tok_pos[m], freq[pair], magnitude, &sn, &cs);
        const float me = rb_to_float<T>(qh[(int64_t)m * ldq + D + e]), ot = rb_to_float<T>(qh[(int64_t)m * ldq + D + other]);
        y = first ? me * cs - ot * sn : me * cs + ot * sn;
      }
      dst[(int64_t)m * ldo] = rb_from_float<T>(y);
    }
    return;
  }
  const T* w = W + ((int64_t)h * C + n) * D;
  for (int m0 = 0; m0 < M; m0 += FEW_ROWS) {
    float acc[FEW_ROWS];
#pragma unroll
    for (int i = 0; i < FEW_ROWS; ++i) acc[i] = 0.f;
    if (VEC) {
      for (int k = lane * 4; k < D; k += 128) {
        float wv[4];
        rb_load4(w + k, wv);
#pragma unroll
        for (int i = 0; i < FEW_ROWS; ++i) {
          if (m0 + i < M) {
            float av[4];
            rb_load4(qh + (int64_t)(m0 + i) * ldq + k, av);
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i] = fmaf(av[j], wv[j], acc[i]);
          }
        }
      }
    } else {
      for (int k = lane; k < D; k += 32) {
        const float wv = rb_to_float<T>(w[k]);
#pragma unroll
        for (int i = 0; i < FEW_ROWS; ++i)
          if (m0 + i < M) acc[i] = fmaf(rb_to_float<T>(qh[(int64_t)(m0 + i) * ldq + k]), wv, acc[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < FEW_ROWS; ++i) {
      const float v = rb_warp_sum(acc[i]);
      if (lane == 0 && m0 + i < M) dst[(int64_t)(m0 + i) * ldo] = rb_from_float<T>(v);
    }
  }
}

// A block per token: columns C .. width-1 of every head's row.
template <typename T>
__global__ void __launch_bounds__(256) latent_turn_kernel(T* __restrict__ out, const T* __restrict__ q,
                                                          const double* __restrict__ freq, float magnitude, int interleaved,
                                                          const int* __restrict__ tok_pos, int H, int D, int R, int C,
                                                          int width) {
  rb_pdl_launch_dependents();
  extern __shared__ float s_sincos[];
  rb_pdl_wait();
  const int t = blockIdx.x, pos = tok_pos[t];
  for (int i = threadIdx.x; i < R / 2; i += blockDim.x)
    angle_sincos(pos, freq[i], magnitude, &s_sincos[i], &s_sincos[R / 2 + i]);
  __syncthreads();
  const int rest = width - C;
  for (int i = threadIdx.x; i < H * rest; i += blockDim.x) {
    const int h = i / rest, e = i - h * rest;
    const T* src = q + ((int64_t)t * H + h) * (D + R) + D;
    float y = 0.f;
    if (e < R) {
      auto val = [&](int k) { return rb_to_float<T>(src[k]); };
      y = turned(val, e, R, interleaved, s_sincos);
    }
    out[((int64_t)t * H + h) * width + C + e] = rb_from_float<T>(y);
  }
}

}  // namespace

RB_EXPORT int rb_latent_norm_append(void* cq, int dtype, const float* rows, int64_t ld, int q_off, int kv_off, int q_rank,
                                    int kv_rank, int rot_dim, const float* wq, const float* wkv, float eps,
                                    const double* freq, float magnitude, int interleaved, void* pool, const int* page_table,
                                    int max_pages, int page_size, int width, const int* tok_pos, const int* tok_slot, int T,
                                    cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(q_rank > 0 && kv_rank > 0 && rot_dim >= 0 && rot_dim % 2 == 0 && width >= kv_rank + rot_dim && page_size > 0,
             "rb_latent_norm_append: bad sizes q_rank=%d kv_rank=%d rot_dim=%d width=%d", q_rank, kv_rank, rot_dim, width);
  RB_REQUIRE(rot_dim == 0 || freq != nullptr, "rb_latent_norm_append: a turned part without frequencies");
  RbPagedLayer cache{pool, pool, page_table, max_pages, page_size, 1, width};
  const int threads = (q_rank > 512 || kv_rank > 512) ? 256 : 128;
  const size_t smem = (size_t)(rot_dim > 0 ? rot_dim : 1) * sizeof(float);
#define GO(TT) RB_LAUNCH("latent_norm_append_kernel", (latent_norm_append_kernel<TT>), T, threads, smem, stream, (TT*)cq, rows, ld, q_off, kv_off, q_rank, kv_rank, rot_dim, wq, wkv, eps, freq, magnitude, interleaved, cache, width, tok_pos, tok_slot)
  if (dtype == RB_F32) GO(float);
  else if (dtype == RB_BF16) GO(__nv_bfloat16);
  else RB_FAIL("rb_latent_norm_append: unknown dtype %d", dtype);
#undef GO
  RB_CHECK_LAUNCH("rb_latent_norm_append");
  return 0;
}

// out [M, H * width] from q [M, H * (D + R)] and W [H, C, D] (dtype of all three: dtype).  Any number of rows is right; up
// to 16 is what it is for.
RB_EXPORT int rb_latent_queries_few(void* out, const void* q, const void* W, int dtype, const double* freq, float magnitude,
                                    int interleaved, const int* tok_pos, int M, int H, int D, int R, int C, int width,
                                    cudaStream_t stream) {
  if (M == 0) return 0;
  RB_REQUIRE(M > 0 && H > 0 && H <= 65535 && D > 0 && C > 0 && R >= 0 && R % 2 == 0 && width >= C + R,
             "rb_latent_queries_few: bad sizes H=%d D=%d R=%d C=%d width=%d", H, D, R, C, width);
  RB_REQUIRE(R == 0 || freq != nullptr, "rb_latent_queries_few: a turned part without frequencies");
  const dim3 grid((width + 7) / 8, H);
  const int elem = dtype == RB_F32 ? 4 : 2;
  const bool vec = D % 4 == 0 && R % 4 == 0 && (uintptr_t)q % (4 * elem) == 0 && (uintptr_t)W % (4 * elem) == 0;
#define GO(TT, V) RB_LAUNCH("latent_queries_few_kernel", (latent_queries_few_kernel<TT, V>), grid, 256, 0, stream, (TT*)out, (const TT*)q, (const TT*)W, freq, magnitude, interleaved, tok_pos, M, H, D, R, C, width)
  if (dtype == RB_F32) { if (vec) GO(float, true); else GO(float, false); }
  else if (dtype == RB_BF16) { if (vec) GO(__nv_bfloat16, true); else GO(__nv_bfloat16, false); }
  else RB_FAIL("rb_latent_queries_few: unknown dtype %d", dtype);
#undef GO
  RB_CHECK_LAUNCH("rb_latent_queries_few");
  return 0;
}

// Columns C .. width-1 of every head's row of out [T, H * width]: the last R values of q's heads turned, then zeros.
RB_EXPORT int rb_latent_turn(void* out, const void* q, int dtype, const double* freq, float magnitude, int interleaved,
                             const int* tok_pos, int T, int H, int D, int R, int C, int width, cudaStream_t stream) {
  if (T == 0 || width == C) return 0;
  RB_REQUIRE(H > 0 && D > 0 && C > 0 && R >= 0 && R % 2 == 0 && width >= C + R,
             "rb_latent_turn: bad sizes H=%d D=%d R=%d C=%d width=%d", H, D, R, C, width);
  RB_REQUIRE(R == 0 || freq != nullptr, "rb_latent_turn: a turned part without frequencies");
  const size_t smem = (size_t)(R > 0 ? R : 1) * sizeof(float);
#define GO(TT) RB_LAUNCH("latent_turn_kernel", (latent_turn_kernel<TT>), T, 256, smem, stream, (TT*)out, (const TT*)q, freq, magnitude, interleaved, tok_pos, H, D, R, C, width)
  if (dtype == RB_F32) GO(float);
  else if (dtype == RB_BF16) GO(__nv_bfloat16);
  else RB_FAIL("rb_latent_turn: unknown dtype %d", dtype);
#undef GO
  RB_CHECK_LAUNCH("rb_latent_turn");
  return 0;
}

RB_CHECK_READER(latent)
