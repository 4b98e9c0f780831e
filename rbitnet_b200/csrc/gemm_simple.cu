// Plain tiled matrix product on the CUDA cores: C[M,N] (+)= alpha * A[M,K] * W[N,K]^T.
//
// This is the true 32-bit path's product (FFMA with float32 accumulation, no
// tensor-core or reduced-precision mode) and the product for shapes that the
// tensor-core kernel refuses.  W is row-major [out, in], the layout the
// reference indexes as w[i + o*n_in] (crates/bitnet-core/src/llama/model.rs:67-91),
// so no weight is transposed at load.  Each output element is one sequential
// float32 sum over k in ascending order, whatever M is: a row's result does not
// depend on which other rows are in the batch.
#include "rb_common.cuh"

namespace {

constexpr int BM = 64, BN = 64, BK = 16, TM = 4, TN = 4;  // 256 threads, 4x4 outputs each

// What happens to a finished sum before it is stored or added (null: nothing): bias[n] is added, and the value is
// multiplied by sigmoid(gate[row * ldg + z * gate_batch + n * gate_step]), z the number of the product (a head); a step of
// 0 is one gate for all of a product's values.
struct Tail {
  const float* bias = nullptr;
  const float* gate = nullptr;
  int64_t ldg = 0;
  int64_t gate_batch = 0;
  int gate_step = 1;
};
__device__ __forceinline__ float finished(const Tail& tail, float v, int64_t row, int n, int64_t z) {
  if (tail.bias != nullptr) v += tail.bias[n];
  if (tail.gate != nullptr) v *= 1.0f / (1.0f + expf(-tail.gate[row * tail.ldg + z * tail.gate_batch + n * tail.gate_step]));
  return v;
}

template <typename TA, typename TC>
__global__ void __launch_bounds__(256) gemm_simple_kernel(TC* __restrict__ C, int64_t ldc,
                                                         const TA* __restrict__ A, int64_t lda,
                                                         const TA* __restrict__ W, int64_t ldw, int M, int N,
                                                         int K, int accumulate, float alpha, Tail tail, int64_t batch_c,
                                                         int64_t batch_a, int64_t batch_w) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  // blockIdx.z: one of several independent products of equal sizes, their operands a fixed distance apart
  C += blockIdx.z * batch_c;
  A += blockIdx.z * batch_a;
  W += blockIdx.z * batch_w;
  __shared__ float As[BK][BM + 1];
  __shared__ float Ws[BK][BN + 1];
  const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  float acc[TM][TN];
#pragma unroll
  for (int i = 0; i < TM; ++i)
#pragma unroll
    for (int j = 0; j < TN; ++j) acc[i][j] = 0.f;

  for (int k0 = 0; k0 < K; k0 += BK) {
    // 64x16 elements of each operand, 256 threads -> 4 each
    for (int e = threadIdx.x; e < BM * BK; e += 256) {
      const int r = e / BK, c = e % BK;
      const int gm = m0 + r, gn = n0 + r, gk = k0 + c;
      As[c][r] = (gm < M && gk < K) ? rb_to_float<TA>(A[(int64_t)gm * lda + gk]) : 0.f;
      Ws[c][r] = (gn < N && gk < K) ? rb_to_float<TA>(W[(int64_t)gn * ldw + gk]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < BK; ++kk) {
      float a[TM], w[TN];
#pragma unroll
      for (int i = 0; i < TM; ++i) a[i] = As[kk][ty * TM + i];
#pragma unroll
      for (int j = 0; j < TN; ++j) w[j] = Ws[kk][tx * TN + j];
#pragma unroll
      for (int i = 0; i < TM; ++i)
#pragma unroll
        for (int j = 0; j < TN; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < TM; ++i) {
    const int gm = m0 + ty * TM + i;
    if (gm >= M) continue;
#pragma unroll
    for (int j = 0; j < TN; ++j) {
      const int gn = n0 + tx * TN + j;
      if (gn >= N) continue;
      TC* p = C + (int64_t)gm * ldc + gn;
      float v = finished(tail, alpha == 1.0f ? acc[i][j] : acc[i][j] * alpha, gm, gn, blockIdx.z);
      if (accumulate) v += rb_to_float<TC>(*p);
      *p = rb_from_float<TC>(v);
    }
  }
}


// The same product with tiles of 128 x 128 and 8 x 8 outputs per thread, for many rows: every value read from shared
// memory feeds eight multiply-adds instead of four.  Each output element is still one sequential float32 sum over k in
// ascending order.
constexpr int LM = 128, LN = 128, LK = 16;

template <typename TA, typename TC>
__global__ void __launch_bounds__(256) gemm_simple_large_kernel(TC* __restrict__ C, int64_t ldc, const TA* __restrict__ A,
                                                               int64_t lda, const TA* __restrict__ W, int64_t ldw, int M,
                                                               int N, int K, int accumulate, float alpha, Tail tail, int64_t batch_c,
                                                               int64_t batch_a, int64_t batch_w) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  C += blockIdx.z * batch_c;
  A += blockIdx.z * batch_a;
  W += blockIdx.z * batch_w;
  __shared__ __align__(16) float As[LK][LM + 4];
  __shared__ __align__(16) float Ws[LK][LN + 4];
  const int m0 = blockIdx.y * LM, n0 = blockIdx.x * LN;
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;      // outputs: rows ty*4 + {0..3} and 64 + ty*4 + {0..3}, columns likewise with tx
  float acc[8][8];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += LK) {
#pragma unroll
    for (int e = threadIdx.x; e < LM * LK; e += 256) {
      const int r = e / LK, c = e % LK;
      const int gm = m0 + r, gn = n0 + r, gk = k0 + c;
      As[c][r] = (gm < M && gk < K) ? rb_to_float<TA>(A[(int64_t)gm * lda + gk]) : 0.f;
      Ws[c][r] = (gn < N && gk < K) ? rb_to_float<TA>(W[(int64_t)gn * ldw + gk]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < LK; ++kk) {
      const float4 a0 = *reinterpret_cast<const float4*>(&As[kk][ty * 4]);
      const float4 a1 = *reinterpret_cast<const float4*>(&As[kk][64 + ty * 4]);
      const float4 w0 = *reinterpret_cast<const float4*>(&Ws[kk][tx * 4]);
      const float4 w1 = *reinterpret_cast<const float4*>(&Ws[kk][64 + tx * 4]);
      const float a[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
      const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int gm = m0 + (i < 4 ? ty * 4 + i : 64 + ty * 4 + i - 4);
    if (gm >= M) continue;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int gn = n0 + (j < 4 ? tx * 4 + j : 64 + tx * 4 + j - 4);
      if (gn >= N) continue;
      TC* p = C + (int64_t)gm * ldc + gn;
      float v = finished(tail, alpha == 1.0f ? acc[i][j] : acc[i][j] * alpha, gm, gn, blockIdx.z);
      if (accumulate) v += rb_to_float<TC>(*p);
      *p = rb_from_float<TC>(v);
    }
  }
}

// Few rows (a decode step) times one matrix per head: a warp makes four outputs of one head for up to eight rows at a
// time, its lanes sharing K, so that the head's matrix is read once, the rows once for four outputs, and heads x N / 16
// blocks are at work instead of a few tiles.  float32 sums (a lane's share in ascending order, then the lanes' shares in a
// fixed tree).  Head h's input values start at column h * head_a of a row.  VEC: four values a load.
constexpr int FEW_ROWS = 8, FEW_OUTS = 4, FEW_WARPS = 4;
template <typename TA, typename TC, bool VEC>
__global__ void __launch_bounds__(FEW_WARPS * 32) per_head_few_rows_kernel(
    TC* __restrict__ C, int64_t ldc, const TA* __restrict__ A, int64_t lda, int head_a, const TA* __restrict__ W, int M, int N,
    int K, Tail tail) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, n0 = (blockIdx.x * FEW_WARPS + warp) * FEW_OUTS;
  if (n0 >= N) return;
  const TA* w = W + ((int64_t)h * N + n0) * K;
  const TA* a = A + (int64_t)h * head_a;
  for (int m0 = 0; m0 < M; m0 += FEW_ROWS) {
    float acc[FEW_OUTS * FEW_ROWS];
#pragma unroll
    for (int i = 0; i < FEW_OUTS * FEW_ROWS; ++i) acc[i] = 0.f;
    constexpr int V = VEC ? 4 : 1;
    for (int k = lane * V; k < K; k += 32 * V) {
      float wv[FEW_OUTS][4];
#pragma unroll
      for (int o = 0; o < FEW_OUTS; ++o) {
        const bool have = n0 + o < N;
        if (VEC) {
          if (have) rb_load4(w + (int64_t)o * K + k, wv[o]);
          else wv[o][0] = wv[o][1] = wv[o][2] = wv[o][3] = 0.f;
        } else {
          wv[o][0] = have ? rb_to_float<TA>(w[(int64_t)o * K + k]) : 0.f;
        }
      }
#pragma unroll
      for (int i = 0; i < FEW_ROWS; ++i) {
        if (m0 + i < M) {
          float av[4];
          if (VEC) rb_load4(a + (int64_t)(m0 + i) * lda + k, av);
          else av[0] = rb_to_float<TA>(a[(int64_t)(m0 + i) * lda + k]);
#pragma unroll
          for (int o = 0; o < FEW_OUTS; ++o)
#pragma unroll
            for (int j = 0; j < V; ++j) acc[o * FEW_ROWS + i] = fmaf(av[j], wv[o][j], acc[o * FEW_ROWS + i]);
        }
      }
    }
    const float v = rb_warp_sum32(acc, lane);
    const int n = n0 + lane / FEW_ROWS, m = m0 + lane % FEW_ROWS;
    if (n < N && m < M) C[(int64_t)m * ldc + (int64_t)h * N + n] = rb_from_float<TC>(finished(tail, v, m, n, h));
  }
}

thread_local Tail t_tail;          // of this thread's next call
Tail take_tail() {
  const Tail t = t_tail;
  t_tail = Tail();
  return t;
}

}  // namespace

// The next rb_gemm_simple, rb_gemm_simple_batched or rb_per_head_few_rows call of this thread adds bias[n] (float32, or
// null) to every finished sum and multiplies it by sigmoid(gate[row * ldg + z * gate_batch + n * gate_step]) (float32, or
// null; z: the number of the product or head).
RB_EXPORT int rb_gemm_simple_next(const float* bias, const float* gate, int64_t ldg, int64_t gate_batch, int gate_step) {
  t_tail.gate_step = gate_step;
  t_tail.bias = bias; t_tail.gate = gate; t_tail.ldg = ldg; t_tail.gate_batch = gate_batch;
  return 0;
}

// C[m, h * N + n] = sum_k A[m, h * head_a + k] * W[h, n, k] for few rows m (any number is right; up to 16 is what it is for).
RB_EXPORT int rb_per_head_few_rows(void* C, int64_t ldc, int c_dtype, const void* A, int64_t lda, int head_a, const void* W,
                                   int a_dtype, int M, int H, int N, int K, cudaStream_t stream) {
  const Tail tail = take_tail();
  if (M == 0 || N == 0 || H == 0) return 0;
  RB_REQUIRE(M > 0 && N > 0 && K > 0 && H > 0 && H <= 65535 && head_a >= K, "rb_per_head_few_rows: bad sizes M=%d H=%d N=%d K=%d (%d apart)",
             M, H, N, K, head_a);
  const dim3 grid((N + FEW_OUTS * FEW_WARPS - 1) / (FEW_OUTS * FEW_WARPS), H);
  const int elem = a_dtype == RB_F32 ? 4 : 2;
  const bool vec = K % 4 == 0 && head_a % 4 == 0 && lda % 4 == 0 && (uintptr_t)A % (4 * elem) == 0 && (uintptr_t)W % (4 * elem) == 0;
#define LAUNCH(TA, TC)                                                                                                  \
  do {                                                                                                                  \
    if (vec) RB_LAUNCH("per_head_few_rows_kernel", (per_head_few_rows_kernel<TA, TC, true>), grid, FEW_WARPS * 32, 0, stream, (TC*)C, ldc, (const TA*)A, lda, head_a, (const TA*)W, M, N, K, tail); \
    else RB_LAUNCH("per_head_few_rows_kernel", (per_head_few_rows_kernel<TA, TC, false>), grid, FEW_WARPS * 32, 0, stream, (TC*)C, ldc, (const TA*)A, lda, head_a, (const TA*)W, M, N, K, tail);    \
  } while (0)
  if (a_dtype == RB_F32 && c_dtype == RB_F32) LAUNCH(float, float);
  else if (a_dtype == RB_BF16 && c_dtype == RB_F32) LAUNCH(__nv_bfloat16, float);
  else if (a_dtype == RB_BF16 && c_dtype == RB_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else RB_FAIL("rb_per_head_few_rows: unsupported dtypes a=%d c=%d", a_dtype, c_dtype);
#undef LAUNCH
  RB_CHECK_LAUNCH("rb_per_head_few_rows");
  return 0;
}

// a_dtype: dtype of A and W; c_dtype: dtype of C.  accumulate: C += instead of C =.
// alpha multiplies the finished sum (1.0 leaves it as it is).
// n_batch products at once: product z reads A + z*batch_a and W + z*batch_w and writes C + z*batch_c
// (distances in elements); block-diagonal matrices are the use.
RB_EXPORT int rb_gemm_simple_batched(void* C, int64_t ldc, int c_dtype, const void* A, int64_t lda, const void* W,
                                     int64_t ldw, int a_dtype, int M, int N, int K, int accumulate, float alpha,
                                     int n_batch, int64_t batch_c, int64_t batch_a, int64_t batch_w,
                                     cudaStream_t stream) {
  const Tail tail = take_tail();
  if (M == 0 || N == 0 || n_batch == 0) return 0;
  RB_REQUIRE(M > 0 && N > 0 && K > 0, "rb_gemm_simple: bad sizes M=%d N=%d K=%d", M, N, K);
  if (M >= 256 && N >= LN) {
    // many rows: the larger tiles
    dim3 lgrid((N + LN - 1) / LN, (M + LM - 1) / LM, n_batch);
    RB_REQUIRE(lgrid.y <= 65535 && n_batch >= 1 && n_batch <= 65535, "rb_gemm_simple: M=%d, %d products: too large for one launch", M, n_batch);
#define LLAUNCH(TA, TC)                                                                                            \
  RB_LAUNCH("gemm_simple_large_kernel", (gemm_simple_large_kernel<TA, TC>), lgrid, 256, 0, stream, (TC*)C, ldc,     \
            (const TA*)A, lda, (const TA*)W, ldw, M, N, K, accumulate, alpha, tail, batch_c, batch_a, batch_w)
    if (a_dtype == RB_F32 && c_dtype == RB_F32) LLAUNCH(float, float);
    else if (a_dtype == RB_BF16 && c_dtype == RB_F32) LLAUNCH(__nv_bfloat16, float);
    else if (a_dtype == RB_BF16 && c_dtype == RB_BF16) LLAUNCH(__nv_bfloat16, __nv_bfloat16);
    else RB_FAIL("rb_gemm_simple: unsupported dtypes a=%d c=%d", a_dtype, c_dtype);
#undef LLAUNCH
    RB_CHECK_LAUNCH("rb_gemm_simple");
    return 0;
  }
  dim3 grid((N + BN - 1) / BN, (M + BM - 1) / BM, n_batch);
  RB_REQUIRE(grid.y <= 65535 && n_batch >= 1 && n_batch <= 65535, "rb_gemm_simple: M=%d, %d products: too large for one launch", M, n_batch);
#define LAUNCH(TA, TC)                                                                                     \
  RB_LAUNCH("gemm_simple_kernel", (gemm_simple_kernel<TA, TC>), grid, 256, 0, stream, (TC*)C, ldc, (const TA*)A, \
            lda, (const TA*)W, ldw, M, N, K, accumulate, alpha, tail, batch_c, batch_a, batch_w)
  if (a_dtype == RB_F32 && c_dtype == RB_F32) LAUNCH(float, float);
  else if (a_dtype == RB_BF16 && c_dtype == RB_F32) LAUNCH(__nv_bfloat16, float);
  else if (a_dtype == RB_BF16 && c_dtype == RB_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else RB_FAIL("rb_gemm_simple: unsupported dtypes a=%d c=%d", a_dtype, c_dtype);
#undef LAUNCH
  RB_CHECK_LAUNCH("rb_gemm_simple");
  return 0;
}

RB_EXPORT int rb_gemm_simple(void* C, int64_t ldc, int c_dtype, const void* A, int64_t lda, const void* W,
                             int64_t ldw, int a_dtype, int M, int N, int K, int accumulate,
                             float alpha, cudaStream_t stream) {
  return rb_gemm_simple_batched(C, ldc, c_dtype, A, lda, W, ldw, a_dtype, M, N, K, accumulate, alpha, 1, 0, 0, 0, stream);
}
