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

// A block per token.  STAGED: the row's values wait in shared memory between the sums and the values made from them.
template <typename T, bool STAGED>
__global__ void __launch_bounds__(256) latent_norm_append_kernel(
    T* __restrict__ cq, const float* __restrict__ rows, int64_t ld, int q_off, int kv_off, int q_rank, int kv_rank,
    int rot_dim, const float* __restrict__ wq, const float* __restrict__ wkv, float eps, const double* __restrict__ freq,
    float magnitude, int interleaved, RbPagedLayer cache, int width, const int* __restrict__ tok_pos,
    const int* __restrict__ tok_slot) {
  rb_pdl_launch_dependents();
  __shared__ float scratch[66];
  extern __shared__ float s_mem[];
  float* s_sincos = s_mem;
  float* s_row = s_mem + (rot_dim > 0 ? rot_dim : 1);
  rb_pdl_wait();
  const int t = blockIdx.x;
  const int pos = tok_pos[t];
  const float* q = rows + (int64_t)t * ld + q_off;
  const float* kv = rows + (int64_t)t * ld + kv_off;        // the latent, then the key part
  float sq = 0.f, sk = 0.f;
#pragma unroll 4
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) {
    const float v = q[i];
    if (STAGED) s_row[i] = v;
    sq = fmaf(v, v, sq);
  }
#pragma unroll 2
  for (int i = threadIdx.x; i < kv_rank + rot_dim; i += blockDim.x) {
    const float v = kv[i];
    if (STAGED) s_row[q_rank + i] = v;
    if (i < kv_rank) sk = fmaf(v, v, sk);
  }
  // (the block's last threads make the sines and cosines, while the first are still at the latents' ends)
  for (int i = (int)(blockDim.x - 1 - threadIdx.x); i < rot_dim / 2; i += blockDim.x)
    angle_sincos(pos, freq[i], magnitude, &s_sincos[i], &s_sincos[rot_dim / 2 + i]);
  const float2 sums = rb_block_sum2(sq, sk, scratch);       // also the barrier after the shared memory's writes
  const float rq = 1.0f / sqrtf(sums.x / (float)q_rank + eps);
  const float rk = 1.0f / sqrtf(sums.y / (float)kv_rank + eps);
  if (STAGED) { q = s_row; kv = s_row + q_rank; }
  for (int i = threadIdx.x; i < q_rank; i += blockDim.x) cq[(int64_t)t * q_rank + i] = rb_from_float<T>(q[i] * rq * wq[i]);
  T* dst = reinterpret_cast<T*>(cache.k) + rb_page_offset(cache, tok_slot[t], pos, 0);
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float y = 0.f;
    if (i < kv_rank) {
      y = kv[i] * rk * wkv[i];
    } else if (i < kv_rank + rot_dim) {
      auto val = [&](int e) { return kv[kv_rank + e]; };
      y = turned(val, i - kv_rank, rot_dim, interleaved, s_sincos);
    }
    dst[i] = rb_from_float<T>(y);
  }
}

// blockIdx.x < dot_blocks: a warp makes four values of W_h q_c of one head for up to eight rows at a time, its lanes
// sharing the D inner values, so that the head's matrix is read once and the rows once for four values.  The blocks
// beyond: a thread per value of the turned part and of the zeros behind it.  VEC: four values a load.
constexpr int FEW_ROWS = 8, FEW_OUTS = 4, FEW_WARPS = 4;
template <typename T, bool VEC>
__global__ void __launch_bounds__(FEW_WARPS * 32) latent_queries_few_kernel(
    T* __restrict__ out, const T* __restrict__ q, const T* __restrict__ W, const double* __restrict__ freq, float magnitude,
    int interleaved, const int* __restrict__ tok_pos, int M, int H, int D, int R, int C, int width, int dot_blocks) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, Dq = D + R;
  const int64_t ldq = (int64_t)H * Dq, ldo = (int64_t)H * width;
  const T* qh = q + (int64_t)h * Dq;
  T* dst = out + (int64_t)h * width;
  if ((int)blockIdx.x >= dot_blocks) {
    const int rest = width - C, n_blocks = gridDim.x - dot_blocks;
    for (int i = (blockIdx.x - dot_blocks) * blockDim.x + threadIdx.x; i < rest * M; i += n_blocks * blockDim.x) {
      const int m = i / rest, e = i - m * rest;
      float y = 0.f;
      if (e < R) {
        const int half = R >> 1;
        int pair, other;
        bool first;
        if (interleaved) { pair = e >> 1; first = (e & 1) == 0; other = first ? e + 1 : e - 1; }
        else { first = e < half; pair = first ? e : e - half; other = first ? e + half : e - half; }
        float sn, cs;
        angle_sincos(tok_pos[m], freq[pair], magnitude, &sn, &cs);
        const float me = rb_to_float<T>(qh[m * ldq + D + e]), ot = rb_to_float<T>(qh[m * ldq + D + other]);
        y = first ? me * cs - ot * sn : me * cs + ot * sn;
      }
      dst[m * ldo + C + e] = rb_from_float<T>(y);
    }
    return;
  }
  const int n0 = (blockIdx.x * FEW_WARPS + warp) * FEW_OUTS;
  if (n0 >= C) return;
  const T* w = W + ((int64_t)h * C + n0) * D;
  for (int m0 = 0; m0 < M; m0 += FEW_ROWS) {
    float acc[FEW_OUTS * FEW_ROWS];
#pragma unroll
    for (int i = 0; i < FEW_OUTS * FEW_ROWS; ++i) acc[i] = 0.f;
    constexpr int V = VEC ? 4 : 1;
    for (int k = lane * V; k < D; k += 32 * V) {
      float wv[FEW_OUTS][4];
#pragma unroll
      for (int o = 0; o < FEW_OUTS; ++o) {
        const bool have = n0 + o < C;
        if (VEC) {
          if (have) rb_load4(w + (int64_t)o * D + k, wv[o]);
          else wv[o][0] = wv[o][1] = wv[o][2] = wv[o][3] = 0.f;
        } else {
          wv[o][0] = have ? rb_to_float<T>(w[(int64_t)o * D + k]) : 0.f;
        }
      }
#pragma unroll
      for (int i = 0; i < FEW_ROWS; ++i) {
        if (m0 + i < M) {
          float av[4];
          if (VEC) rb_load4(qh + (int64_t)(m0 + i) * ldq + k, av);
          else av[0] = rb_to_float<T>(qh[(int64_t)(m0 + i) * ldq + k]);
#pragma unroll
          for (int o = 0; o < FEW_OUTS; ++o)
#pragma unroll
            for (int j = 0; j < V; ++j) acc[o * FEW_ROWS + i] = fmaf(av[j], wv[o][j], acc[o * FEW_ROWS + i]);
        }
      }
    }
    const float v = rb_warp_sum32(acc, lane);
    const int n = n0 + lane / FEW_ROWS, m = m0 + lane % FEW_ROWS;
    if (n < C && m < M) dst[m * ldo + n] = rb_from_float<T>(v);
  }
}

// A block per token: columns C .. width-1 of every head's row.  A thread turns a pair at a time; PAIRS2: two neighbouring
// pairs of the half layout, whose values lie side by side.
template <typename T, bool PAIRS2>
__global__ void __launch_bounds__(256) latent_turn_kernel(T* __restrict__ out, const T* __restrict__ q,
                                                          const double* __restrict__ freq, float magnitude, int interleaved,
                                                          const int* __restrict__ tok_pos, int H, int D, int R, int C,
                                                          int width) {
  rb_pdl_launch_dependents();
  extern __shared__ float s_sincos[];
  rb_pdl_wait();
  const int t = blockIdx.x, pos = tok_pos[t], half = R >> 1;
  for (int i = threadIdx.x; i < half; i += blockDim.x)
    angle_sincos(pos, freq[i], magnitude, &s_sincos[i], &s_sincos[half + i]);
  __syncthreads();
  constexpr int P = PAIRS2 ? 2 : 1;
  const int per = half / P;                              // work items of a head
  for (int i = threadIdx.x; i < H * per; i += blockDim.x) {
    const int h = i / per, pair = (i - h * per) * P;
    const T* src = q + ((int64_t)t * H + h) * (D + R) + D;
    T* dst = out + ((int64_t)t * H + h) * width + C;
    const int ia = interleaved ? 2 * pair : pair, ib = interleaved ? 2 * pair + 1 : pair + half;
    float u[2], v[2];
#pragma unroll
    for (int j = 0; j < P; ++j) { u[j] = rb_to_float<T>(src[ia + j]); v[j] = rb_to_float<T>(src[ib + j]); }
#pragma unroll
    for (int j = 0; j < P; ++j) {
      const float sn = s_sincos[pair + j], cs = s_sincos[half + pair + j];
      const float a = u[j] * cs - v[j] * sn, b = v[j] * cs + u[j] * sn;
      u[j] = a;
      v[j] = b;
    }
    if (PAIRS2) {
      rb_store2(dst + ia, u[0], u[1]);
      rb_store2(dst + ib, v[0], v[1]);
    } else {
      dst[ia] = rb_from_float<T>(u[0]);
      dst[ib] = rb_from_float<T>(v[0]);
    }
  }
  const int pad = width - C - R;
  for (int i = threadIdx.x; i < H * pad; i += blockDim.x) {
    const int h = i / pad;
    out[((int64_t)t * H + h) * width + C + R + (i - h * pad)] = rb_from_float<T>(0.f);
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
  size_t smem = (size_t)(rot_dim > 0 ? rot_dim : 1) * sizeof(float);
  const size_t row_bytes = (size_t)(q_rank + kv_rank + rot_dim) * sizeof(float);
  const bool staged = smem + row_bytes <= 40 * 1024;
  if (staged) smem += row_bytes;
#define GO1(TT, ST) RB_LAUNCH("latent_norm_append_kernel", (latent_norm_append_kernel<TT, ST>), T, threads, smem, stream, (TT*)cq, rows, ld, q_off, kv_off, q_rank, kv_rank, rot_dim, wq, wkv, eps, freq, magnitude, interleaved, cache, width, tok_pos, tok_slot)
#define GO(TT) do { if (staged) GO1(TT, true); else GO1(TT, false); } while (0)
  if (dtype == RB_F32) GO(float);
  else if (dtype == RB_BF16) GO(__nv_bfloat16);
  else RB_FAIL("rb_latent_norm_append: unknown dtype %d", dtype);
#undef GO
#undef GO1
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
  const int dot_blocks = (C + FEW_OUTS * FEW_WARPS - 1) / (FEW_OUTS * FEW_WARPS);
  const int rest_blocks = width > C ? ((width - C) * (M < 16 ? M : 16) + FEW_WARPS * 32 - 1) / (FEW_WARPS * 32) : 0;
  const dim3 grid(dot_blocks + rest_blocks, H);
  const int elem = dtype == RB_F32 ? 4 : 2;
  const bool vec = D % 4 == 0 && R % 4 == 0 && (uintptr_t)q % (4 * elem) == 0 && (uintptr_t)W % (4 * elem) == 0;
#define GO(TT, V) RB_LAUNCH("latent_queries_few_kernel", (latent_queries_few_kernel<TT, V>), grid, FEW_WARPS * 32, 0, stream, (TT*)out, (const TT*)q, (const TT*)W, freq, magnitude, interleaved, tok_pos, M, H, D, R, C, width, dot_blocks)
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
  // two values side by side: every head's parts begin on an even value
  const bool pairs2 = !interleaved && R % 4 == 0 && D % 2 == 0 && C % 2 == 0 && width % 2 == 0;
#define GO1(TT, P2) RB_LAUNCH("latent_turn_kernel", (latent_turn_kernel<TT, P2>), T, 256, smem, stream, (TT*)out, (const TT*)q, freq, magnitude, interleaved, tok_pos, H, D, R, C, width)
#define GO(TT) do { if (pairs2) GO1(TT, true); else GO1(TT, false); } while (0)
  if (dtype == RB_F32) GO(float);
  else if (dtype == RB_BF16) GO(__nv_bfloat16);
  else RB_FAIL("rb_latent_turn: unknown dtype %d", dtype);
#undef GO
#undef GO1
  RB_CHECK_LAUNCH("rb_latent_turn");
  return 0;
}

RB_CHECK_READER(latent)
