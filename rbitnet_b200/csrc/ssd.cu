// A state-space mixer with one decay per head and token (the recurrence of Mamba-2):
//
//   S_t = exp(-exp(A_h) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D_h x_t,   v_t = y_t silu(z_t)
//
// per head h; S [N state rows, P value columns] is float32, zero at a sequence's start, kept per slot as
// [slot][head][N][P].  B_t and C_t [N] belong to the head's group (head h reads group h / (heads / groups)), dt_t =
// softplus(raw + dt_bias_h).  rows: the mixer's stacked projection, float32 [T, ...], holding z, the channels [x | B | C]
// and raw dt at given columns; the channels pass a short causal convolution with a bias and SiLU first.  A step's rows of
// one sequence are a run; the state is read at a run's start and written at its end.
//
//   ssd_conv_kernel        convolution and SiLU of all channels, in the compute dtype (a thread keeps the last rows of its
//                          channels in registers while it goes down the rows)
//   ssd_step_kernel        one token per sequence, all of it in one launch: convolution (whose ring of inputs moves on),
//                          dt, the state's step, the read-out and the gate
//   ssd_scan_kernel        runs of any length token by token: the plain form
//   ssd_chunk_*            runs of several tokens in chunks of 64, on the tensor cores (below)
#include "rb_common.cuh"

namespace {

__device__ __forceinline__ float ssd_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float ssd_silu(float v) { return v / (1.0f + expf(-v)); }
// The same two with the hardware's exponential and reciprocal, for the chunked kernels (error a few units of float32, far
// below that of the bfloat16 channels they work on).
__device__ __forceinline__ float ssd_exp_fast(float v) { return __expf(v); }
__device__ __forceinline__ float ssd_silu_fast(float v) { return __fdividef(v, 1.0f + __expf(-v)); }

// ---------------------------------------------------------------- short convolution and SiLU
// u[t, c] = silu(bias[c] + sum_d taps[c, K-1-d] x_(t-d)[c]), zeros before a sequence's start, rows before a run from the
// ring tail[slot][K][C] (the input of position q in row q mod K).  A block takes `per_block` rows; V channels a thread.
template <typename TO, int K, int V>
__global__ void __launch_bounds__(128) ssd_conv_kernel(TO* __restrict__ u, int64_t ldu, const float* __restrict__ x, int64_t ldx,
                                                       int x_off, const float* __restrict__ taps, const float* __restrict__ bias,
                                                       const float* __restrict__ tail, const int* __restrict__ tok_first,
                                                       const int* __restrict__ tok_slot, const int* __restrict__ tok_pos, int T,
                                                       int C, int per_block) {
  rb_pdl_launch_dependents();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  float w[K][V], b[V], hist[K][V];                       // hist[d]: the input d rows back (d = 0: this row's)
#pragma unroll
  for (int i = 0; i < V; ++i) {
    b[i] = bias[c + i];
#pragma unroll
    for (int d = 0; d < K; ++d) w[d][i] = taps[(int64_t)(c + i) * K + K - 1 - d];
  }
  rb_pdl_wait();
  const int t0 = blockIdx.x * per_block, t1 = min(T, t0 + per_block);
  auto load = [&](const float* src, float (&to)[V]) {
    if (V == 4) {
      const float4 f = *reinterpret_cast<const float4*>(src);
      to[0] = f.x; if (V > 1) { to[1 % V] = f.y; to[2 % V] = f.z; to[3 % V] = f.w; }
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) to[i] = src[i];
    }
  };
  int last_first = -1;
  constexpr int AHEAD = 8;                               // rows on their way at a time
  for (int ta = t0; ta < t1; ta += AHEAD) {
  float in[AHEAD][V];
#pragma unroll
  for (int r = 0; r < AHEAD; ++r)
    if (ta + r < t1) load(x + (int64_t)(ta + r) * ldx + x_off + c, in[r]);
#pragma unroll
  for (int r = 0; r < AHEAD; ++r) {
    const int t = ta + r;
    if (t >= t1) break;
    const int first = tok_first != nullptr ? tok_first[t] : t;
    if (first != last_first) {                           // a new run, or the block's first row: fetch the rows before
      last_first = first;
      const int slot = tok_slot[t], pos = tok_pos[t];
#pragma unroll
      for (int d = 1; d < K; ++d) {
        if (pos - d < 0) {
#pragma unroll
          for (int i = 0; i < V; ++i) hist[d][i] = 0.f;
        } else if (t - d >= first) {
          load(x + (int64_t)(t - d) * ldx + x_off + c, hist[d]);
        } else {
          load(tail + ((int64_t)slot * K + (pos - d) % K) * C + c, hist[d]);
        }
      }
    }
    float y[V];
#pragma unroll
    for (int i = 0; i < V; ++i) hist[0][i] = in[r][i];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      float acc = b[i];
#pragma unroll
      for (int d = 0; d < K; ++d) acc = fmaf(w[d][i], hist[d][i], acc);
      y[i] = sizeof(TO) == 2 ? ssd_silu_fast(acc) : ssd_silu(acc);
    }
    TO* dst = u + (int64_t)t * ldu + c;
    if (V == 4) {
      const float yy[4] = {y[0], y[1 % V], y[2 % V], y[3 % V]};
      rb_store4(dst, yy);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) dst[i] = rb_from_float<TO>(y[i]);
    }
#pragma unroll
    for (int d = K - 1; d > 0; --d)
#pragma unroll
      for (int i = 0; i < V; ++i) hist[d][i] = hist[d - 1][i];
  }
  }
}

// Any number of taps, value by value.
template <typename TO>
__global__ void __launch_bounds__(128) ssd_conv_any_kernel(TO* __restrict__ u, int64_t ldu, const float* __restrict__ x, int64_t ldx,
                                                           int x_off, const float* __restrict__ taps,
                                                           const float* __restrict__ bias, const float* __restrict__ tail,
                                                           const int* __restrict__ tok_first, const int* __restrict__ tok_slot,
                                                           const int* __restrict__ tok_pos, int T, int C, int K) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  const int t = blockIdx.x;
  const int first = tok_first != nullptr ? tok_first[t] : t, slot = tok_slot[t], pos = tok_pos[t];
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
    float acc = bias[c];
    for (int d = 0; d < K && d <= pos; ++d) {
      const float v = t - d >= first ? x[(int64_t)(t - d) * ldx + x_off + c] : tail[((int64_t)slot * K + (pos - d) % K) * C + c];
      acc = fmaf(taps[(int64_t)c * K + K - 1 - d], v, acc);
    }
    u[(int64_t)t * ldu + c] = rb_from_float<TO>(ssd_silu(acc));
  }
}

// ---------------------------------------------------------------- one token per sequence
// grid (rows, H, tiles of up to 64 value columns), 256 threads.  A thread owns V neighbouring columns of every NL-th state
// row.  The first tile of a group's first head moves the ring on for the group's B and C, every block for its own x.
constexpr int STEP_NT = 256;
constexpr int STEP_COLS = 64;
constexpr int STEP_HELD = 8;            // state rows a thread holds at a time

// KT: the convolution's taps (0: any number, from K).
template <int V, int KT>
__global__ void __launch_bounds__(STEP_NT, 3) ssd_step_kernel(
    float* __restrict__ out, const float* __restrict__ rows, int64_t ld, int z_off, int x_off, int dt_off,
    const float* __restrict__ taps, const float* __restrict__ conv_bias, const float* __restrict__ dt_bias,
    const float* __restrict__ A_log, const float* __restrict__ D_skip, float* __restrict__ state, float* __restrict__ tail,
    const int* __restrict__ tok_slot, const int* __restrict__ tok_pos, int H, int P, int N, int G, int K_, int cols) {
  rb_pdl_launch_dependents();
  extern __shared__ float s_step[];
  float* sx = s_step;                   // [cols] x
  float* sB = sx + STEP_COLS;           // [N]
  float* sC = sB + N;                   // [N]
  float* red = sC + N;                  // [NL][pw]
  const int K = KT > 0 ? KT : K_;
  const int t = blockIdx.x, h = blockIdx.y, tile = blockIdx.z, p0 = tile * cols;
  const int pw = min(cols, P - p0);                          // columns of this block
  const int groups_of = H / G, grp = h / groups_of;
  const int inner = H * P, C = inner + 2 * G * N;
  const int PV = (pw + V - 1) / V;                           // threads across the columns
  const int NL = STEP_NT / PV;                               // state rows side by side
  const int pc = (threadIdx.x % PV) * V, nl = threadIdx.x / PV;
  const bool mine = nl < NL;
  const int slot = tok_slot[t], pos = tok_pos[t];
  const float a = expf(A_log[h]), dtb = dt_bias[h], skip = D_skip[h];
  const int n_ch = pw + 2 * N;                               // channels this block convolves: its x, the group's B and C
  auto channel = [&](int i) {
    return i < pw ? h * P + p0 + i : (i < pw + N ? inner + grp * N + (i - pw) : inner + G * N + grp * N + (i - pw - N));
  };
  // the weights of a thread's first two channels do not depend on the kernel before this one
  constexpr int CPT = KT > 0 ? 2 : 1, KW = KT > 0 ? KT : 1;
  float w[CPT][KW], cb[CPT];
  if (KT > 0) {
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      const int i = threadIdx.x + j * STEP_NT;
      if (i < n_ch) {
        const int c = channel(i);
        cb[j] = conv_bias[c];
#pragma unroll
        for (int d = 0; d < KW; ++d) w[j][d] = taps[(int64_t)c * KW + KW - 1 - d];
      }
    }
  }
  rb_pdl_wait();
  const float* row = rows + (int64_t)t * ld;
  float* S = state + ((int64_t)slot * H + h) * N * P + p0 + pc;
  float held[STEP_HELD][V];
  auto fetch = [&](int n0) {
#pragma unroll
    for (int i = 0; i < STEP_HELD; ++i) {
      const int n = n0 + i * NL + nl;
      if (mine && n < N) {
        if (V == 4) {
          const float4 f = *reinterpret_cast<const float4*>(S + (int64_t)n * P);
          held[i][0] = f.x; held[i][1 % V] = f.y; held[i][2 % V] = f.z; held[i][3 % V] = f.w;
        } else {
          held[i][0] = S[(int64_t)n * P];
        }
      }
    }
  };
  const bool write_bc = tile == 0 && h % groups_of == 0;
  auto put = [&](int i, int c, float now, float acc) {
    if (K > 1 && (i < pw || write_bc)) tail[((int64_t)slot * K + pos % K) * C + c] = now;
    const float y = ssd_silu(acc);
    if (i < pw) sx[i] = y;
    else sB[i - pw] = y;                                     // B, then C behind it
  };
  const float raw_dt = row[dt_off + h];
  const float z = threadIdx.x < pw ? row[z_off + h * P + p0 + threadIdx.x] : 0.f;
  int done = 0;
  if (KT > 0) {
    float in[CPT][KW];
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      const int i = threadIdx.x + j * STEP_NT;
      if (i < n_ch) {
        const int c = channel(i);
        in[j][0] = row[x_off + c];
#pragma unroll
        for (int d = 1; d < KW; ++d) in[j][d] = d <= pos ? tail[((int64_t)slot * KW + (pos - d) % KW) * C + c] : 0.f;
      }
    }
    fetch(0);                                                // the state is on its way while the channels are convolved
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      const int i = threadIdx.x + j * STEP_NT;
      if (i < n_ch) {
        float acc = cb[j];
#pragma unroll
        for (int d = 0; d < KW; ++d) acc = fmaf(w[j][d], in[j][d], acc);
        put(i, channel(i), in[j][0], acc);
      }
    }
    done = CPT * STEP_NT;
  } else {
    fetch(0);
  }
  for (int i = done + threadIdx.x; i < n_ch; i += STEP_NT) {
    const int c = channel(i);
    const float now = row[x_off + c];
    float acc = fmaf(taps[(int64_t)c * K + K - 1], now, conv_bias[c]);
    for (int d = 1; d < K && d <= pos; ++d)
      acc = fmaf(taps[(int64_t)c * K + K - 1 - d], tail[((int64_t)slot * K + (pos - d) % K) * C + c], acc);
    put(i, c, now, acc);
  }
  const float dt = ssd_softplus(raw_dt + dtb);
  const float decay = expf(-a * dt);
  __syncthreads();
  float y[V], xdt[V];
#pragma unroll
  for (int k = 0; k < V; ++k) {
    y[k] = 0.f;
    xdt[k] = mine && pc + k < pw ? sx[pc + k] * dt : 0.f;
  }
  for (int n0 = 0; n0 < N; n0 += STEP_HELD * NL) {
    if (n0 > 0) fetch(n0);
#pragma unroll
    for (int i = 0; i < STEP_HELD; ++i) {
      const int n = n0 + i * NL + nl;
      if (mine && n < N) {
        const float b = sB[n], cc = sC[n];
#pragma unroll
        for (int k = 0; k < V; ++k) {
          held[i][k] = fmaf(decay, held[i][k], b * xdt[k]);
          y[k] = fmaf(cc, held[i][k], y[k]);
        }
        if (V == 4) *reinterpret_cast<float4*>(S + (int64_t)n * P) = make_float4(held[i][0], held[i][1 % V], held[i][2 % V], held[i][3 % V]);
        else S[(int64_t)n * P] = held[i][0];
      }
    }
  }
  if (mine) {
#pragma unroll
    for (int k = 0; k < V; ++k)
      if (pc + k < pw) red[nl * pw + pc + k] = y[k];
  }
  __syncthreads();
  if (threadIdx.x < pw) {
    const int p = threadIdx.x;
    float acc = skip * sx[p];
    for (int i = 0; i < NL; ++i) acc += red[i * pw + p];
    out[(int64_t)t * inner + h * P + p0 + p] = acc * ssd_silu(z);
  }
}

// ---------------------------------------------------------------- token by token, any run
// grid (runs, H, tiles of 16 value columns), 256 threads: column = thread % 16, state rows thread / 16 + 16 r.
constexpr int SCAN_NT = 256;
constexpr int SCAN_COLS = 16;
constexpr int SCAN_ROWS = SCAN_NT / SCAN_COLS;

template <typename TU, int R>
__global__ void __launch_bounds__(SCAN_NT) ssd_scan_kernel(
    float* __restrict__ out, const TU* __restrict__ u, int64_t ldu, const float* __restrict__ rows, int64_t ld, int z_off, int dt_off,
    const float* __restrict__ dt_bias, const float* __restrict__ A_log, const float* __restrict__ D_skip, float* __restrict__ state,
    const int* __restrict__ seq_first, const int* __restrict__ seq_count, const int* __restrict__ tok_slot, int H, int P, int N,
    int G) {
  rb_pdl_launch_dependents();
  __shared__ float red[2][SCAN_NT / 32][SCAN_COLS];
  const int run = blockIdx.x, h = blockIdx.y;
  const int p = blockIdx.z * SCAN_COLS + threadIdx.x % SCAN_COLS, nr = threadIdx.x / SCAN_COLS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int inner = H * P, grp = h / (H / G);
  const bool in = p < P;
  const float a = expf(A_log[h]), dtb = dt_bias[h], skip = D_skip[h];
  rb_pdl_wait();
  const int first = seq_first != nullptr ? seq_first[run] : run, n_tok = seq_count != nullptr ? seq_count[run] : 1;
  const int slot = tok_slot[first];
  float* St = state + ((int64_t)slot * H + h) * N * P + p;
  float S[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int n = nr + r * SCAN_ROWS;
    S[r] = in && n < N ? St[(int64_t)n * P] : 0.f;
  }
  for (int i = 0; i < n_tok; ++i) {
    const int64_t t = first + i;
    const TU* ur = u + t * ldu;
    const float dt = ssd_softplus(rows[t * ld + dt_off + h] + dtb);
    const float decay = expf(-a * dt);
    const float x = in ? rb_to_float<TU>(ur[h * P + p]) : 0.f;
    const float xdt = x * dt;
    float y = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int n = nr + r * SCAN_ROWS;
      if (n < N) {
        S[r] = fmaf(decay, S[r], rb_to_float<TU>(ur[inner + grp * N + n]) * xdt);
        y = fmaf(rb_to_float<TU>(ur[inner + G * N + grp * N + n]), S[r], y);
      }
    }
    y += __shfl_xor_sync(0xffffffffu, y, 16);                // the warp's two rows of this column
    if (lane < SCAN_COLS) red[i & 1][warp][lane] = y;
    __syncthreads();                                         // (two buffers: the next token writes the other one)
    if (threadIdx.x < SCAN_COLS && in) {
      float acc = skip * x;
#pragma unroll
      for (int w = 0; w < SCAN_NT / 32; ++w) acc += red[i & 1][w][threadIdx.x];
      out[t * inner + h * P + p] = acc * ssd_silu(rows[t * ld + z_off + h * P + p]);
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int n = nr + r * SCAN_ROWS;
    if (in && n < N) St[(int64_t)n * P] = S[r];
  }
}

// ---------------------------------------------------------------- runs of several tokens: chunks of 64
// Within a chunk that starts from the state S0, with L_i the sum of the decays' logarithms over the chunk's tokens up to
// and including i:
//   y_i   = e^{L_i} S0^T C_i + sum_{j <= i} (C_i . B_j) e^{L_i - L_j} dt_j x_j + D x_i
//   S_end = e^{L_end} S0 + sum_j e^{L_end - L_j} dt_j B_j x_j^T
// Three kernels: every chunk's sum over its own tokens and e^{L_end} (all chunks at once); the walk over a run's chunks,
// value by value of the state, which leaves in each chunk's place the state it starts from; every chunk's outputs (all at
// once).  No exponent is of a positive number.  L is summed in float64, because what enters an exponential is a difference
// of two sums that may be large.
// The products run on mma.sync with bfloat16 operands and float32 accumulators.  x, B and C are bfloat16 values (the
// convolution's results); whatever else enters a product is float32 and is cut into three bfloat16 terms (high, middle,
// low: 24 bits together), one product each, so that the sums are those of float32 operands.  A chunk's missing tokens
// count as dt = 0 and x = B = C = 0.
constexpr int CH = 64;                  // tokens of a chunk
constexpr int CH_NT = 128;              // four warps of 16 rows
constexpr int CH_P = 64;                // value columns of a block
constexpr int LDZ = CH_P + 8;           // row stride of the tile of z (float32)
constexpr int SL = 64;                  // state rows that the output kernel holds at a time
constexpr int LDX = CH_P + 8;           // row stride of tiles of columns: ldmatrix rows in different banks

__device__ __forceinline__ uint32_t s_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_pair(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// Two values as three pairs of bfloat16 terms each; what is left of a value after its first two terms is exact in float32.
__device__ __forceinline__ void split3(float a, float b, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  hi = pack_pair(a, b);
  a -= __uint_as_float(hi << 16);
  b -= __uint_as_float(hi & 0xffff0000u);
  mid = pack_pair(a, b);
  lo = pack_pair(a - __uint_as_float(mid << 16), b - __uint_as_float(mid & 0xffff0000u));
}

// One warp: dt and L of the chunk's tokens into s_dt [64] and s_L [64] (float64).
__device__ __forceinline__ void chunk_decays(const float* __restrict__ rows, int64_t ld, int col, int64_t row0, int m, float a,
                                             float dt_bias, double* s_L, float* s_dt, int lane) {
  float d[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int i = 2 * lane + k;
    d[k] = i < m ? ssd_softplus(rows[(row0 + i) * ld + col] + dt_bias) : 0.f;
    s_dt[i] = d[k];
  }
  const double l0 = -(double)(a * d[0]), l1 = l0 - (double)(a * d[1]);       // over this lane's two tokens
  double before = l1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, before, o);
    if (lane >= o) before += v;
  }
  before -= l1;                                                              // over the tokens before them
  s_L[2 * lane] = before + l0;
  s_L[2 * lane + 1] = before + l1;
}

// A tile [64 rows][width] of bfloat16 values from u's columns col.., zeros beyond row m and column `live`.  vec: 16-byte
// pieces (every column and stride a multiple of 8 values), which are only asked for: see tiles_landed.
__device__ __forceinline__ void tiles_landed() { asm volatile("cp.async.wait_all;" ::: "memory"); }
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, int ldd, int width, const __nv_bfloat16* __restrict__ u, int64_t ldu,
                                          int64_t row0, int m, int col, int live, bool vec) {
  if (vec) {
    const int w8 = width >> 3;
    for (int i = threadIdx.x; i < CH * w8; i += CH_NT) {
      const int r = i / w8, c = (i - r * w8) << 3;
      const bool in = r < m && c < live;
      const int bytes = in ? 16 : 0;                                    // none: the piece is filled with zeros
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s_addr(dst + r * ldd + c)),
                   "l"(in ? u + (row0 + r) * ldu + col + c : u), "r"(bytes) : "memory");
    }
  } else {
    for (int i = threadIdx.x; i < CH * width; i += CH_NT) {
      const int r = i / width, c = i - r * width;
      dst[r * ldd + c] = r < m && c < live ? u[(row0 + r) * ldu + col + c] : __float2bfloat16_rn(0.f);
    }
  }
}

// FULL: every block has all of its 64 columns.
// grid (chunks, H, tiles of 64 columns).  sums [chunks][H][N][P], ends [chunks][H].
template <bool FULL>
__global__ void __launch_bounds__(CH_NT, 4) ssd_chunk_sum_kernel(
    float* __restrict__ sums, float* __restrict__ ends, const __nv_bfloat16* __restrict__ u, int64_t ldu,
    const float* __restrict__ rows, int64_t ld, int dt_off, const float* __restrict__ dt_bias, const float* __restrict__ A_log,
    const int* __restrict__ chunk_row, const int* __restrict__ chunk_len, int H, int P, int N, int G, int vec) {
  rb_pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t s_bytes[];
  const int NP = (N + 15) & ~15, LDB = NP + 8;
  double* s_L = reinterpret_cast<double*>(s_bytes);
  float* s_dt = reinterpret_cast<float*>(s_L + CH);
  __nv_bfloat16* sB = reinterpret_cast<__nv_bfloat16*>(s_dt + CH);      // [64][LDB]
  __nv_bfloat16* sX = sB + CH * LDB;                                    // three of [64][LDX]: the weighted x in three terms
  const int chunk = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * CH_P, pw = min(CH_P, P - p0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int inner = H * P, grp = h / (H / G);
  const float a = expf(A_log[h]), dtb = dt_bias[h];
  rb_pdl_wait();
  const int64_t row0 = chunk_row[chunk];
  const int m = chunk_len[chunk];
  load_tile(sB, LDB, NP, u, ldu, row0, m, inner + grp * N, N, vec != 0);
  load_tile(sX, LDX, CH_P, u, ldu, row0, m, h * P + p0, pw, vec != 0);
  if (warp == 0) chunk_decays(rows, ld, dt_off + h, row0, m, a, dtb, s_L, s_dt, lane);
  tiles_landed();
  __syncthreads();
  const double L_end = s_L[CH - 1];
  for (int i = threadIdx.x; i < CH * (CH_P / 2); i += CH_NT) {          // x in place: its owner reads it first
    const int r = i / (CH_P / 2), c = (i % (CH_P / 2)) * 2;
    __nv_bfloat16* at = sX + r * LDX + c;
    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(at));
    const float w = s_dt[r] * ssd_exp_fast((float)(L_end - s_L[r]));
    uint32_t hi, mid, lo;
    split3(x.x * w, x.y * w, hi, mid, lo);
    *reinterpret_cast<uint32_t*>(at) = hi;
    *reinterpret_cast<uint32_t*>(at + CH * LDX) = mid;
    *reinterpret_cast<uint32_t*>(at + 2 * CH * LDX) = lo;
  }
  if (threadIdx.x == 0 && blockIdx.z == 0) ends[(int64_t)chunk * H + h] = expf((float)L_end);
  __syncthreads();
  float* dst = sums + ((int64_t)chunk * H + h) * N * P + p0;
  const int g = lane >> 2, t4 = lane & 3;
  for (int nb = warp * 16; nb < NP; nb += 64) {                         // 16 state rows at a time
    float acc[CH_P / 8][4];
#pragma unroll
    for (int i = 0; i < CH_P / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < CH / 16; ++kk) {
      if (!FULL && kk * 16 >= m) break;
      uint32_t A[4];
      ldsm4t(A, s_addr(sB + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * LDB + nb + ((lane >> 3) & 1) * 8));
#pragma unroll
      for (int part = 0; part < 3; ++part) {
#pragma unroll
        for (int dn = 0; dn < CH_P / 8; dn += 2) {
          if (!FULL && dn * 8 >= pw) break;
          uint32_t b[4];
          ldsm4t(b, s_addr(sX + part * CH * LDX + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDX + (dn + (lane >> 4)) * 8));
          mma_16816(acc[dn], A, b[0], b[1]);
          mma_16816(acc[dn + 1], A, b[2], b[3]);
        }
      }
    }
    const bool pairs = P % 2 == 0;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int n = nb + g + 8 * half;
      if (n >= N) continue;
#pragma unroll
      for (int dn = 0; dn < CH_P / 8; ++dn) {
        const int p = dn * 8 + t4 * 2;
        if (p >= pw) break;
        if (pairs) {
          *reinterpret_cast<float2*>(dst + (int64_t)n * P + p) = make_float2(acc[dn][2 * half], acc[dn][2 * half + 1]);
        } else {
          dst[(int64_t)n * P + p] = acc[dn][2 * half];
          if (p + 1 < pw) dst[(int64_t)n * P + p + 1] = acc[dn][2 * half + 1];
        }
      }
    }
  }
}

// grid (runs, H, pieces of a state), 128 threads, V values each: sums[chunk] <- the state the chunk starts from; and
// the ring of the convolution's last inputs is brought up to the run's end (tail [n_slots, K, C], null with one tap).
template <int V>
__global__ void __launch_bounds__(128) ssd_chunk_walk_kernel(float* __restrict__ sums, const float* __restrict__ ends,
                                                             float* __restrict__ state, const int* __restrict__ seq_first,
                                                             const int* __restrict__ seq_count,
                                                             const int* __restrict__ run_chunk0, const int* __restrict__ tok_slot,
                                                             int H, int64_t NP_, float* __restrict__ tail,
                                                             const float* __restrict__ rows, int64_t ld, int x_off,
                                                             const int* __restrict__ tok_pos, int C, int K) {
  rb_pdl_launch_dependents();
  const int run = blockIdx.x, h = blockIdx.y;
  const int64_t e = ((int64_t)blockIdx.z * 128 + threadIdx.x) * V;
  rb_pdl_wait();
  const int first = seq_first[run], n_tok = seq_count[run], n_chunks = (n_tok + CH - 1) / CH, chunk0 = run_chunk0[run];
  if (K > 1) {
    // the ring of the convolution's inputs moves on to the run's end (the convolution is done)
    const int slot = tok_slot[first], last = first + n_tok - 1, pos = tok_pos[last];
    for (int c = (h * gridDim.z + blockIdx.z) * 128 + threadIdx.x; c < C; c += H * gridDim.z * 128)
      for (int back = 0; back < K - 1 && back < n_tok; ++back)
        tail[((int64_t)slot * K + (pos - back) % K) * C + c] = rows[(int64_t)(last - back) * ld + x_off + c];
  }
  if (e >= NP_) return;
  float* st = state + ((int64_t)tok_slot[first] * H + h) * NP_ + e;
  float S[V];
#pragma unroll
  for (int k = 0; k < V; ++k) S[k] = st[k];
  constexpr int AHEAD = 8;
  const int64_t step = (int64_t)H * NP_;
  float* at = sums + ((int64_t)chunk0 * H + h) * NP_ + e;
  for (int c0 = 0; c0 < n_chunks; c0 += AHEAD) {
    float v[AHEAD][V], d[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (c0 + i < n_chunks) {
        const float* src = at + (int64_t)(c0 + i) * step;
        if (V == 4) {
          const float4 f = *reinterpret_cast<const float4*>(src);
          v[i][0] = f.x; v[i][1 % V] = f.y; v[i][2 % V] = f.z; v[i][3 % V] = f.w;
        } else {
          v[i][0] = src[0];
        }
        d[i] = ends[(int64_t)(chunk0 + c0 + i) * H + h];
      }
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (c0 + i < n_chunks) {
        float* dst = at + (int64_t)(c0 + i) * step;
        if (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(S[0], S[1 % V], S[2 % V], S[3 % V]);
        else dst[0] = S[0];
#pragma unroll
        for (int k = 0; k < V; ++k) S[k] = fmaf(d[i], S[k], v[i][k]);
      }
    }
  }
#pragma unroll
  for (int k = 0; k < V; ++k) st[k] = S[k];
}

// grid (chunks, H, tiles of 64 columns).  starts: what the walk left.  out [T, H * P] = v (see the top of the file).
template <bool FULL>
__global__ void __launch_bounds__(CH_NT, 3) ssd_chunk_out_kernel(
    float* __restrict__ out, const float* __restrict__ starts, const __nv_bfloat16* __restrict__ u, int64_t ldu,
    const float* __restrict__ rows, int64_t ld, int z_off, int dt_off, const float* __restrict__ dt_bias,
    const float* __restrict__ A_log, const float* __restrict__ D_skip, const int* __restrict__ chunk_row,
    const int* __restrict__ chunk_len, int H, int P, int N, int G, int vec) {
  rb_pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t s_bytes[];
  const int NP = (N + 15) & ~15, LDB = NP + 8;
  double* s_L = reinterpret_cast<double*>(s_bytes);
  float* s_dt = reinterpret_cast<float*>(s_L + CH);
  __nv_bfloat16* sC = reinterpret_cast<__nv_bfloat16*>(s_dt + CH);      // [64][LDB]
  __nv_bfloat16* sB = sC + CH * LDB;                                    // [64][LDB]
  __nv_bfloat16* sX = sB + CH * LDB;                                    // [64][LDX]
  __nv_bfloat16* sS = sX + CH * LDX;                                    // three of [64][LDX]: 64 state rows in three terms
  const int chunk = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * CH_P, pw = min(CH_P, P - p0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int inner = H * P, grp = h / (H / G);
  const float a = expf(A_log[h]), dtb = dt_bias[h], skip = D_skip[h];
  rb_pdl_wait();
  const int64_t row0 = chunk_row[chunk];
  const int m = chunk_len[chunk];
  const float* start = starts + ((int64_t)chunk * H + h) * N * P + p0;
  // a thread's part of 64 state rows: four columns of every eighth row, fetched ahead
  constexpr int HELD = SL * (CH_P / 4) / CH_NT;
  const bool quads = P % 4 == 0;
  const int sc = (threadIdx.x % (CH_P / 4)) * 4, sr = threadIdx.x / (CH_P / 4);
  float4 held[HELD];
  auto fetch = [&](int n0) {
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
      const int n = n0 + sr + i * (CH_NT / (CH_P / 4));
      held[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (n < N && sc < pw) {
        const float* src = start + (int64_t)n * P + sc;
        if (quads) {
          held[i] = *reinterpret_cast<const float4*>(src);
        } else {
          held[i].x = src[0];
          if (sc + 1 < pw) held[i].y = src[1];
          if (sc + 2 < pw) held[i].z = src[2];
          if (sc + 3 < pw) held[i].w = src[3];
        }
      }
    }
  };
  fetch(0);
  load_tile(sC, LDB, NP, u, ldu, row0, m, inner + G * N + grp * N, N, vec != 0);
  load_tile(sB, LDB, NP, u, ldu, row0, m, inner + grp * N, N, vec != 0);
  load_tile(sX, LDX, CH_P, u, ldu, row0, m, h * P + p0, pw, vec != 0);
  if (warp == 0) chunk_decays(rows, ld, dt_off + h, row0, m, a, dtb, s_L, s_dt, lane);
  constexpr int part_elems = SL * LDX;
  const int rb = warp * 16;                                             // this warp's 16 tokens
  const bool active = rb < m;
  float acc[CH_P / 8][4], G_[CH / 8][4];
#pragma unroll
  for (int i = 0; i < CH_P / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int i = 0; i < CH / 8; ++i) G_[i][0] = G_[i][1] = G_[i][2] = G_[i][3] = 0.f;
  for (int n0 = 0; n0 < NP; n0 += SL) {                                 // 64 state rows at a time
    if (n0 > 0) __syncthreads();                                        // everybody has left the slice before
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
      uint2 hi, mid, lo;
      split3(held[i].x, held[i].y, hi.x, mid.x, lo.x);
      split3(held[i].z, held[i].w, hi.y, mid.y, lo.y);
      __nv_bfloat16* at = sS + (sr + i * (CH_NT / (CH_P / 4))) * LDX + sc;
      *reinterpret_cast<uint2*>(at) = hi;
      *reinterpret_cast<uint2*>(at + part_elems) = mid;
      *reinterpret_cast<uint2*>(at + 2 * part_elems) = lo;
    }
    if (n0 == 0) tiles_landed();
    __syncthreads();
    if (n0 + SL < NP) fetch(n0 + SL);                                   // on its way while this slice is multiplied
    if (!active) continue;
    for (int kk = n0 / 16; kk < min(NP, n0 + SL) / 16; ++kk) {
      uint32_t A[4];
      ldsm4(A, s_addr(sC + (rb + (lane & 7) + ((lane >> 3) & 1) * 8) * LDB + kk * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int part = 0; part < 3; ++part) {                            // S0^T C
#pragma unroll
        for (int dn = 0; dn < CH_P / 8; dn += 2) {
          if (!FULL && dn * 8 >= pw) break;
          uint32_t b[4];
          ldsm4t(b, s_addr(sS + part * part_elems + (kk * 16 - n0 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDX + (dn + (lane >> 4)) * 8));
          mma_16816(acc[dn], A, b[0], b[1]);
          mma_16816(acc[dn + 1], A, b[2], b[3]);
        }
      }
#pragma unroll
      for (int j = 0; j < CH / 8; j += 2) {                             // C B^T, half of it where the rows are early
        if (j == CH / 16 && rb < CH / 2) break;
        uint32_t b[4];
        ldsm4(b, s_addr(sB + (j * 8 + (lane >> 4) * 8 + (lane & 7)) * LDB + kk * 16 + ((lane >> 3) & 1) * 8));
        mma_16816(G_[j], A, b[0], b[1]);
        mma_16816(G_[j + 1], A, b[2], b[3]);
      }
    }
  }
  // z comes into the state's place while the chunk's own tokens are multiplied
  float* sZ = reinterpret_cast<float*>(sS);                             // [64][LDZ]
  const bool staged = FULL && vec != 0 && ld % 4 == 0 && z_off % 4 == 0;
  if (staged) {
    __syncthreads();                                                    // everybody has left the last slice
    for (int i = threadIdx.x; i < CH * (CH_P / 4); i += CH_NT) {
      const int r = i / (CH_P / 4), c = (i % (CH_P / 4)) * 4;
      if (r < m)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s_addr(sZ + r * LDZ + c)),
                     "l"(rows + (row0 + r) * ld + z_off + h * P + p0 + c) : "memory");
    }
  }
  const int i0 = rb + g, i1 = rb + g + 8;
  const double L0 = s_L[i0], L1 = s_L[i1];
  {
    const float e0 = expf((float)L0), e1 = expf((float)L1);
#pragma unroll
    for (int dn = 0; dn < CH_P / 8; ++dn) {
      acc[dn][0] *= e0; acc[dn][1] *= e0;
      acc[dn][2] *= e1; acc[dn][3] *= e1;
    }
  }
#pragma unroll
  for (int kt = 0; kt < CH / 16; ++kt) {                                // 16 earlier tokens at a time
    if (kt * 16 > rb + 15 || !active) break;
    uint32_t Mp[3][4];
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int j = kt * 16 + q * 8 + t4 * 2;
      const double Lj0 = s_L[j], Lj1 = s_L[j + 1];
      const float d0 = s_dt[j], d1 = s_dt[j + 1];
      const float* c = G_[2 * kt + q];
      const float v00 = j <= i0 ? c[0] * d0 * ssd_exp_fast((float)(L0 - Lj0)) : 0.f;
      const float v01 = j + 1 <= i0 ? c[1] * d1 * ssd_exp_fast((float)(L0 - Lj1)) : 0.f;
      const float v10 = j <= i1 ? c[2] * d0 * ssd_exp_fast((float)(L1 - Lj0)) : 0.f;
      const float v11 = j + 1 <= i1 ? c[3] * d1 * ssd_exp_fast((float)(L1 - Lj1)) : 0.f;
      split3(v00, v01, Mp[0][2 * q], Mp[1][2 * q], Mp[2][2 * q]);
      split3(v10, v11, Mp[0][2 * q + 1], Mp[1][2 * q + 1], Mp[2][2 * q + 1]);
    }
#pragma unroll
    for (int dn = 0; dn < CH_P / 8; dn += 2) {
      if (!FULL && dn * 8 >= pw) break;
      uint32_t b[4];
      ldsm4t(b, s_addr(sX + (kt * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDX + (dn + (lane >> 4)) * 8));
#pragma unroll
      for (int part = 0; part < 3; ++part) {
        mma_16816(acc[dn], Mp[part], b[0], b[1]);
        mma_16816(acc[dn + 1], Mp[part], b[2], b[3]);
      }
    }
  }
  if (staged) {
    tiles_landed();
    __syncthreads();
  }
  if (!active) return;
  const bool pairs = P % 2 == 0 && ld % 2 == 0 && z_off % 2 == 0;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int i = rb + g + 8 * half;
    if (i >= m) continue;
    const float* z = rows + (row0 + i) * ld + z_off + h * P + p0;
    float* dst = out + (row0 + i) * inner + h * P + p0;
#pragma unroll
    for (int dn = 0; dn < CH_P / 8; ++dn) {
      const int p = dn * 8 + t4 * 2;
      if (!FULL && p >= pw) break;
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sX + i * LDX + p));
      const float y0 = fmaf(skip, x.x, acc[dn][2 * half]), y1 = fmaf(skip, x.y, acc[dn][2 * half + 1]);
      if (pairs) {
        const float2 zz = staged ? *reinterpret_cast<const float2*>(sZ + i * LDZ + p) : *reinterpret_cast<const float2*>(z + p);
        *reinterpret_cast<float2*>(dst + p) = make_float2(y0 * ssd_silu_fast(zz.x), y1 * ssd_silu_fast(zz.y));
      } else {
        dst[p] = y0 * ssd_silu_fast(z[p]);
        if (p + 1 < pw) dst[p + 1] = y1 * ssd_silu_fast(z[p + 1]);
      }
    }
  }
}

inline int chunk_sum_smem(int N) {
  const int NP = (N + 15) & ~15;
  return CH * 12 + (CH * (NP + 8) + 3 * CH * LDX) * 2;
}
inline int chunk_out_smem(int N) {
  const int NP = (N + 15) & ~15;
  return CH * 12 + (2 * CH * (NP + 8) + CH * LDX + 3 * SL * LDX) * 2;
}

}  // namespace

// u [T, ldu] (the first C columns) = silu(convolution + bias) of columns x_off .. of rows x.  See ssd_conv_kernel.
RB_EXPORT int rb_ssd_conv(void* u, int u_dtype, int64_t ldu, const float* x, int64_t ldx, int x_off, const float* taps,
                          const float* bias, const float* tail, const int* tok_first, const int* tok_slot, const int* tok_pos, int T,
                          int C, int K, cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(C > 0 && K >= 1 && ldu >= C && (K == 1 || tail != nullptr), "rb_ssd_conv: bad sizes C=%d K=%d", C, K);
  RB_REQUIRE(u_dtype == RB_F32 || u_dtype == RB_BF16, "rb_ssd_conv: unknown dtype %d", u_dtype);
  const bool vec = C % 4 == 0 && x_off % 4 == 0 && ldx % 4 == 0 && ldu % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)u % 16 == 0;
  const int lanes = vec ? C / 4 : C;
  const int by = (lanes + 127) / 128;
  int per_block = 16;
  while (per_block > 1 && (int64_t)((T + per_block - 1) / per_block) * by < 2 * rb_sm_count()) per_block /= 2;
  const dim3 grid((T + per_block - 1) / per_block, by);
#define GO(TO, KK, V) RB_LAUNCH("ssd_conv_kernel", (ssd_conv_kernel<TO, KK, V>), grid, 128, 0, stream, (TO*)u, ldu, x, ldx, x_off, taps, bias, tail, tok_first, tok_slot, tok_pos, T, C, per_block)
#define PICK(TO)                                                                                                          \
  do {                                                                                                                    \
    if (K == 1) { if (vec) GO(TO, 1, 4); else GO(TO, 1, 1); }                                                             \
    else if (K == 2) { if (vec) GO(TO, 2, 4); else GO(TO, 2, 1); }                                                        \
    else if (K == 3) { if (vec) GO(TO, 3, 4); else GO(TO, 3, 1); }                                                        \
    else if (K == 4) { if (vec) GO(TO, 4, 4); else GO(TO, 4, 1); }                                                        \
    else RB_LAUNCH("ssd_conv_any_kernel", (ssd_conv_any_kernel<TO>), dim3(T, (C + 127) / 128 < 64 ? (C + 127) / 128 : 64), 128, 0, stream, \
                   (TO*)u, ldu, x, ldx, x_off, taps, bias, tail, tok_first, tok_slot, tok_pos, T, C, K);                  \
  } while (0)
  if (u_dtype == RB_F32) PICK(float);
  else PICK(__nv_bfloat16);
#undef PICK
#undef GO
  RB_CHECK_LAUNCH("rb_ssd_conv");
  return 0;
}

// T rows, each a run of one token.  out [T, H * P] float32; state [n_slots, H, N, P]; tail [n_slots, K, H P + 2 G N].
RB_EXPORT int rb_ssd_step(float* out, const float* rows, int64_t ld, int z_off, int x_off, int dt_off, const float* taps,
                          const float* conv_bias, const float* dt_bias, const float* A_log, const float* D_skip, float* state,
                          float* tail, const int* tok_slot, const int* tok_pos, int T, int H, int P, int N, int G, int K,
                          cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(H > 0 && H <= 65535 && P > 0 && N > 0 && G > 0 && H % G == 0 && K >= 1 && (K == 1 || tail != nullptr),
             "rb_ssd_step: bad sizes H=%d P=%d N=%d G=%d K=%d", H, P, N, G, K);
  const int cols = P < STEP_COLS ? P : STEP_COLS;
  const dim3 grid(T, H, (P + cols - 1) / cols);
  const size_t smem = (size_t)(STEP_COLS + 2 * N + 4 * STEP_NT) * sizeof(float);
  RB_REQUIRE(smem <= 48 * 1024, "rb_ssd_step: a state of %d rows is more than a block's shared memory holds", N);
#define GO(V, KT) RB_LAUNCH("ssd_step_kernel", (ssd_step_kernel<V, KT>), grid, STEP_NT, smem, stream, out, rows, ld, z_off, x_off, dt_off, taps, conv_bias, dt_bias, A_log, D_skip, state, tail, tok_slot, tok_pos, H, P, N, G, K, cols)
#define PICK(V)                \
  do {                         \
    if (K == 2) GO(V, 2);      \
    else if (K == 3) GO(V, 3); \
    else if (K == 4) GO(V, 4); \
    else GO(V, 0);             \
  } while (0)
  if (P % 4 == 0) PICK(4);
  else PICK(1);
#undef PICK
#undef GO
  RB_CHECK_LAUNCH("rb_ssd_step");
  return 0;
}

// Runs of any length, token by token.  u: the convolved channels [x | B | C] (u_dtype, rows ldu apart).
RB_EXPORT int rb_ssd_scan(float* out, const void* u, int u_dtype, int64_t ldu, const float* rows, int64_t ld, int z_off, int dt_off,
                          const float* dt_bias, const float* A_log, const float* D_skip, float* state, const int* seq_first,
                          const int* seq_count, const int* tok_slot, int n_runs, int H, int P, int N, int G, cudaStream_t stream) {
  if (n_runs == 0) return 0;
  RB_REQUIRE(H > 0 && H <= 65535 && P > 0 && N > 0 && G > 0 && H % G == 0 && N <= 64 * SCAN_ROWS,
             "rb_ssd_scan: bad sizes H=%d P=%d N=%d G=%d (at most %d state rows)", H, P, N, G, 64 * SCAN_ROWS);
  const dim3 grid(n_runs, H, (P + SCAN_COLS - 1) / SCAN_COLS);
  const int need = (N + SCAN_ROWS - 1) / SCAN_ROWS;
#define GO(TU, R) RB_LAUNCH("ssd_scan_kernel", (ssd_scan_kernel<TU, R>), grid, SCAN_NT, 0, stream, out, (const TU*)u, ldu, rows, ld, z_off, dt_off, dt_bias, A_log, D_skip, state, seq_first, seq_count, tok_slot, H, P, N, G)
#define PICK(TU)                       \
  do {                                 \
    if (need <= 2) GO(TU, 2);          \
    else if (need <= 4) GO(TU, 4);     \
    else if (need <= 8) GO(TU, 8);     \
    else if (need <= 16) GO(TU, 16);   \
    else GO(TU, 64);                   \
  } while (0)
  if (u_dtype == RB_F32) PICK(float);
  else if (u_dtype == RB_BF16) PICK(__nv_bfloat16);
  else RB_FAIL("rb_ssd_scan: unknown dtype %d", u_dtype);
#undef PICK
#undef GO
  RB_CHECK_LAUNCH("rb_ssd_scan");
  return 0;
}

// Whether runs of several tokens take the chunked kernels (bfloat16 channels).
RB_EXPORT int rb_ssd_chunked_supports(int P, int N) { return P > 0 && N > 0 && chunk_out_smem(N) <= 224 * 1024; }

// Floats of scratch per (chunk, head).
RB_EXPORT long long rb_ssd_chunk_floats(int P, int N) { return (long long)P * N + 1; }

// Runs of several tokens in chunks of 64.  chunk_row, chunk_len: every chunk of every run, the runs' chunks in order;
// run_chunk0[r]: the first chunk of run r.  scratch: n_chunks * H * rb_ssd_chunk_floats(P, N) floats.
// It also brings the ring of the convolution's last inputs (columns x_off .. of rows) up to the runs' ends.
RB_EXPORT int rb_ssd_chunked(float* out, const void* u, int64_t ldu, const float* rows, int64_t ld, int z_off, int x_off, int dt_off,
                             const float* dt_bias, const float* A_log, const float* D_skip, float* state, float* tail,
                             float* scratch, const int* seq_first, const int* seq_count, const int* run_chunk0,
                             const int* chunk_row, const int* chunk_len, const int* tok_slot, const int* tok_pos, int n_runs,
                             int n_chunks, int H, int P, int N, int G, int K, cudaStream_t stream) {
  if (n_runs == 0 || n_chunks == 0) return 0;
  const int C = H * P + 2 * G * N;
  RB_REQUIRE(H > 0 && H <= 65535 && G > 0 && H % G == 0 && rb_ssd_chunked_supports(P, N) && (uintptr_t)scratch % 16 == 0 &&
                 (K == 1 || tail != nullptr),
             "rb_ssd_chunked: bad sizes H=%d P=%d N=%d G=%d", H, P, N, G);
  const bool full = P % CH_P == 0;
  const int vec = P % 8 == 0 && N % 8 == 0 && ldu % 8 == 0 && (uintptr_t)u % 16 == 0;
  static RbOncePerDevice configured;
  if (configured.first()) {
    RB_CUDA(cudaFuncSetAttribute(ssd_chunk_sum_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
    RB_CUDA(cudaFuncSetAttribute(ssd_chunk_out_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
    RB_CUDA(cudaFuncSetAttribute(ssd_chunk_sum_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
    RB_CUDA(cudaFuncSetAttribute(ssd_chunk_out_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
  }
  const int64_t NPv = (int64_t)N * P;
  float* sums = scratch;
  float* ends = scratch + (int64_t)n_chunks * H * NPv;
  const dim3 grid(n_chunks, H, (P + CH_P - 1) / CH_P);
  const __nv_bfloat16* ub = (const __nv_bfloat16*)u;
  RB_LAUNCH("ssd_chunk_sum_kernel", (full ? ssd_chunk_sum_kernel<true> : ssd_chunk_sum_kernel<false>), grid, CH_NT, chunk_sum_smem(N), stream, sums, ends, ub, ldu, rows, ld, dt_off,
            dt_bias, A_log, chunk_row, chunk_len, H, P, N, G, vec);
  RB_CHECK_LAUNCH("rb_ssd_chunked");
  if (NPv % 4 == 0)
    RB_LAUNCH("ssd_chunk_walk_kernel", (ssd_chunk_walk_kernel<4>), dim3(n_runs, H, (NPv / 4 + 127) / 128), 128, 0, stream, sums, ends, state,
              seq_first, seq_count, run_chunk0, tok_slot, H, NPv, tail, rows, ld, x_off, tok_pos, C, K);
  else
    RB_LAUNCH("ssd_chunk_walk_kernel", (ssd_chunk_walk_kernel<1>), dim3(n_runs, H, (NPv + 127) / 128), 128, 0, stream, sums, ends, state,
              seq_first, seq_count, run_chunk0, tok_slot, H, NPv, tail, rows, ld, x_off, tok_pos, C, K);
  RB_CHECK_LAUNCH("rb_ssd_chunked");
  RB_LAUNCH("ssd_chunk_out_kernel", (full ? ssd_chunk_out_kernel<true> : ssd_chunk_out_kernel<false>), grid, CH_NT, chunk_out_smem(N), stream, out, sums, ub, ldu, rows, ld, z_off,
            dt_off, dt_bias, A_log, D_skip, chunk_row, chunk_len, H, P, N, G, vec);
  RB_CHECK_LAUNCH("rb_ssd_chunked");
  return 0;
}
