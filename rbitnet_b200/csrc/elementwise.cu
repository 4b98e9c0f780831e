// Memory-bound kernels of the step: embedding gather, RMSNorm, rotation of q and k
// with the append to the paged cache, SiLU(gate)*up, and row gather.
// All arithmetic is float32 whatever the storage dtype.
#include "rb_common.cuh"

#include <stdarg.h>
#include <stdlib.h>
#include <string.h>

static thread_local char g_error[512];

void rb_set_error(const char* fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(g_error, sizeof(g_error), fmt, ap);
  va_end(ap);
}

RB_EXPORT const char* rb_last_error() { return g_error; }

bool rb_pdl_enabled() {
  static int v = -1;
  if (v < 0) {
    const char* e = getenv("RBITNET_PDL");
    v = (e && e[0] == '0') ? 0 : 1;
  }
  return v != 0;
}

RB_EXPORT int rb_abi_version() { return 2; }

RB_EXPORT int rb_device_sm_count() { return rb_sm_count(); }

// 1: the library was built with -DRB_CHECKED (cache addresses are checked before they are used).
RB_EXPORT int rb_is_checked_build() {
#ifdef RB_CHECKED
  return 1;
#else
  return 0;
#endif
}

// ---------------------------------------------------------------- embedding
// x[t, :] = table[ids[t], :] * scale as float32 (crates/bitnet-core/src/llama/model.rs:230-232;
// the reference has no multiplier, scale 1.0).
// An id outside [0, V) is refused on the host before the launch; the kernel
// writes zeros for one rather than read outside the table.
template <typename TW>
__global__ void embed_kernel(float* __restrict__ out, const TW* __restrict__ table,
                             const int* __restrict__ ids, int E, int V, float scale) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  // four values per thread and the whole row in flight at once: the rows come from anywhere in a
  // table far larger than L2, and a loop over the row would wait for memory once per turn
  const int t = blockIdx.x;
  const int id = ids[t];
  const bool ok = id >= 0 && id < V;
  const TW* row = table + (int64_t)(ok ? id : 0) * E;
  float* o = out + (int64_t)t * E;
  const int j = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
  if (j >= E) return;
  if ((E & 3) == 0) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (ok) {
      if constexpr (sizeof(TW) == 4) {
        v = *reinterpret_cast<const float4*>(row + j);
      } else {
        const uint2 raw = *reinterpret_cast<const uint2*>(row + j);
        const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&raw.x);
        const __nv_bfloat162 hi = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
        v = make_float4(__low2float(lo), __high2float(lo), __low2float(hi), __high2float(hi));
      }
    }
    if (scale != 1.0f) v = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
    *reinterpret_cast<float4*>(o + j) = v;
  } else {
    for (int i = j; i < min(E, j + 4); ++i) o[i] = ok ? rb_to_float<TW>(row[i]) * scale : 0.f;
  }
}

RB_EXPORT int rb_embed(float* out, const void* table, int table_dtype, const int* ids, int T, int E,
                       int V, float scale, cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(T > 0 && E > 0 && V > 0, "rb_embed: bad sizes T=%d E=%d V=%d", T, E, V);
  const int threads = 256;
  const dim3 grid(T, (E + threads * 4 - 1) / (threads * 4));
  RB_REQUIRE(grid.y <= 65535, "rb_embed: rows of %d values", E);
  if (table_dtype == RB_F32)
    RB_LAUNCH("embed_kernel", (embed_kernel<float>), grid, threads, 0, stream, out, (const float*)table, ids, E, V, scale);
  else if (table_dtype == RB_BF16)
    RB_LAUNCH("embed_kernel", (embed_kernel<__nv_bfloat16>), grid, threads, 0, stream, out, (const __nv_bfloat16*)table, ids, E, V, scale);
  else
    RB_FAIL("rb_embed: unknown dtype %d", table_dtype);
  RB_CHECK_LAUNCH("rb_embed");
  return 0;
}

// ---------------------------------------------------------------- RMSNorm
// y = x * w / sqrt(mean(x^2) + eps)  (crates/bitnet-core/src/llama/model.rs:93-100).
// x is the float32 residual stream.
template <typename TO> __device__ __forceinline__ void store4(TO* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void store4<float>(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 v;
  v.x = *reinterpret_cast<uint32_t*>(&lo);
  v.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = v;
}

// VEC: the width is a multiple of 4 and rows are read and written four values at a time.
template <typename TO, bool VEC>
__global__ void rmsnorm_kernel(TO* __restrict__ out, const float* __restrict__ x, const float* __restrict__ w,
                               int E, float eps) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  __shared__ float scratch[33];
  extern __shared__ __align__(16) float row[];  // E floats
  const int t = blockIdx.x;
  const float* xr = x + (int64_t)t * E;
  float ss = 0.f;
  if (VEC) {
    for (int j = threadIdx.x * 4; j < E; j += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(xr + j);
      *reinterpret_cast<float4*>(row + j) = v;
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int j = threadIdx.x; j < E; j += blockDim.x) {
      const float v = xr[j];
      row[j] = v;
      ss += v * v;
    }
  }
  ss = rb_block_sum(ss, scratch);
  const float r = 1.0f / sqrtf(ss / (float)E + eps);
  TO* o = out + (int64_t)t * E;
  if (VEC) {
    for (int j = threadIdx.x * 4; j < E; j += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(row + j);
      const float4 g = *reinterpret_cast<const float4*>(w + j);
      store4<TO>(o + j, v.x * g.x * r, v.y * g.y * r, v.z * g.z * r, v.w * g.w * r);
    }
  } else {
    for (int j = threadIdx.x; j < E; j += blockDim.x) o[j] = rb_from_float<TO>(row[j] * w[j] * r);
  }
}

// Rows of up to 4*NV*blockDim values (a multiple of 4) kept in registers: every load of a row
// is in flight before the first is used, and nothing goes through shared memory.
template <typename TO, int NV>
__global__ void rmsnorm_reg_kernel(TO* __restrict__ out, const float* __restrict__ x, const float* __restrict__ w,
                                   int E, float eps) {
  rb_pdl_launch_dependents();
  __shared__ float scratch[33];
  const int t = blockIdx.x;
  const float* xr = x + (int64_t)t * E;
  float4 v[NV], g[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {       // the norm's weights do not depend on the kernel before
    const int j = (threadIdx.x + i * blockDim.x) * 4;
    g[i] = j < E ? *reinterpret_cast<const float4*>(w + j) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  rb_pdl_wait();
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = (threadIdx.x + i * blockDim.x) * 4;
    v[i] = j < E ? *reinterpret_cast<const float4*>(xr + j) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  ss = rb_block_sum(ss, scratch);
  const float r = 1.0f / sqrtf(ss / (float)E + eps);
  TO* o = out + (int64_t)t * E;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = (threadIdx.x + i * blockDim.x) * 4;
    if (j < E) store4<TO>(o + j, v[i].x * g[i].x * r, v[i].y * g[i].y * r, v[i].z * g[i].z * r, v[i].w * g[i].w * r);
  }
}

template <typename TO>
static int launch_rmsnorm_reg(TO* out, const float* x, const float* w, int T, int E, float eps, cudaStream_t stream) {
  const int threads = E <= 1024 ? 128 : (E <= 4096 ? 256 : 1024);
  const int nv = (E / 4 + threads - 1) / threads;
  switch (nv) {
    case 1: RB_LAUNCH("rmsnorm_reg_kernel", (rmsnorm_reg_kernel<TO, 1>), T, threads, 0, stream, out, x, w, E, eps); break;
    case 2: RB_LAUNCH("rmsnorm_reg_kernel", (rmsnorm_reg_kernel<TO, 2>), T, threads, 0, stream, out, x, w, E, eps); break;
    case 3: RB_LAUNCH("rmsnorm_reg_kernel", (rmsnorm_reg_kernel<TO, 3>), T, threads, 0, stream, out, x, w, E, eps); break;
    default: RB_LAUNCH("rmsnorm_reg_kernel", (rmsnorm_reg_kernel<TO, 4>), T, threads, 0, stream, out, x, w, E, eps); break;
  }
  RB_CHECK_LAUNCH("rb_rmsnorm");
  return 0;
}

template <typename TO, bool VEC>
static int launch_rmsnorm(TO* out, const float* x, const float* w, int T, int E, float eps, cudaStream_t stream) {
  const int per = VEC ? 4 : 1;
  int threads = 128;
  while (threads < 1024 && threads * per * 2 <= E) threads *= 2;     // about two loads per thread
  const size_t smem = (size_t)E * sizeof(float);
  if (smem > 48 * 1024)
    RB_CUDA(cudaFuncSetAttribute(rmsnorm_kernel<TO, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  RB_LAUNCH("rmsnorm_kernel", (rmsnorm_kernel<TO, VEC>), T, threads, smem, stream, out, x, w, E, eps);
  RB_CHECK_LAUNCH("rb_rmsnorm");
  return 0;
}

RB_EXPORT int rb_rmsnorm(void* out, int out_dtype, const float* x, const float* w, int T, int E, float eps,
                         cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(T > 0 && E > 0, "rb_rmsnorm: bad sizes T=%d E=%d", T, E);
  RB_REQUIRE((size_t)E * 4 <= 200 * 1024, "rb_rmsnorm: width %d exceeds the %d floats one block can hold",
             E, 200 * 1024 / 4);
  const bool vec = E % 4 == 0 && ((uintptr_t)x % 16 == 0) && ((uintptr_t)w % 16 == 0) &&
                   ((uintptr_t)out % 16 == 0);
  if (vec && E <= 16384) {
    if (out_dtype == RB_F32)
      return launch_rmsnorm_reg<float>((float*)out, x, w, T, E, eps, stream);
    if (out_dtype == RB_BF16)
      return launch_rmsnorm_reg<__nv_bfloat16>((__nv_bfloat16*)out, x, w, T, E, eps, stream);
  }
  if (out_dtype == RB_F32)
    return vec ? launch_rmsnorm<float, true>((float*)out, x, w, T, E, eps, stream)
               : launch_rmsnorm<float, false>((float*)out, x, w, T, E, eps, stream);
  if (out_dtype == RB_BF16)
    return vec ? launch_rmsnorm<__nv_bfloat16, true>((__nv_bfloat16*)out, x, w, T, E, eps, stream)
               : launch_rmsnorm<__nv_bfloat16, false>((__nv_bfloat16*)out, x, w, T, E, eps, stream);
  RB_FAIL("rb_rmsnorm: unknown dtype %d", out_dtype);
}

// ---------------------------------------------------------------- rotation + cache append
// ---------------------------------------------------------------- tanh in place of a norm
// out = w * tanh(alpha * x) + b, value by value.  A thread keeps its V columns (their w and b in registers) and takes
// every gridDim.y-th row.
template <typename TO, int V>
__global__ void __launch_bounds__(256) tanh_norm_kernel(TO* __restrict__ out, const float* __restrict__ x,
                                                        const float* __restrict__ w, const float* __restrict__ b,
                                                        float alpha, int T, int E) {
  rb_pdl_launch_dependents();
  const int e = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  float ww[4], bb[4];
  if (e < E) {                                       // (weights: never written by a kernel)
    if (V == 4) { rb_load4(w + e, ww); rb_load4(b + e, bb); }
    else { ww[0] = w[e]; bb[0] = b[e]; }
  }
  rb_pdl_wait();
  if (e >= E) return;
#pragma unroll 4
  for (int t = blockIdx.y; t < T; t += gridDim.y) {
    const int64_t at = (int64_t)t * E + e;
    float v[4];
    if (V == 4) rb_load4(x + at, v);
    else v[0] = x[at];
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = fmaf(ww[j], rb_norm_tanh<TO>(alpha * v[j]), bb[j]);
    if (V == 4) rb_store4(out + at, v);
    else out[at] = rb_from_float<TO>(v[0]);
  }
}

RB_EXPORT int rb_tanh_norm(void* out, int out_dtype, const float* x, const float* w, const float* b, float alpha, int T, int E,
                           cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(T > 0 && E > 0, "rb_tanh_norm: bad sizes T=%d E=%d", T, E);
  const bool vec = E % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)b % 16 == 0 &&
                   (uintptr_t)out % 16 == 0;
  const int items = vec ? E / 4 : E, threads = items >= 256 ? 256 : (items >= 128 ? 128 : 64);
  const int bx = (items + threads - 1) / threads;
  int by = (rb_sm_count() * (2048 / threads) + bx - 1) / bx;            // every SM's threads once
  if (by > T) by = T;
  const dim3 grid(bx, by);
#define GO(TO, V) RB_LAUNCH("tanh_norm_kernel", (tanh_norm_kernel<TO, V>), grid, threads, 0, stream, (TO*)out, x, w, b, alpha, T, E)
  if (out_dtype == RB_F32) { if (vec) GO(float, 4); else GO(float, 1); }
  else if (out_dtype == RB_BF16) { if (vec) GO(__nv_bfloat16, 4); else GO(__nv_bfloat16, 1); }
  else RB_FAIL("rb_tanh_norm: unknown dtype %d", out_dtype);
#undef GO
  RB_CHECK_LAUNCH("rb_tanh_norm");
  return 0;
}

// ---------------------------------------------------------------- layer norm with weight and bias
// out = (x - mean) / sqrt(var + eps) * w + b, var the mean of the squared deviations; float32 sums, two passes over
// the row (the second over the deviations).  One block per row.
template <typename TO>
__global__ void __launch_bounds__(256) layernorm_kernel(TO* __restrict__ out, const float* __restrict__ x,
                                                        const float* __restrict__ w, const float* __restrict__ b, int E,
                                                        float eps) {
  rb_pdl_launch_dependents();
  __shared__ float scratch[33];
  rb_pdl_wait();
  const float* row = x + (int64_t)blockIdx.x * E;
  float s = 0.f;
  for (int e = threadIdx.x; e < E; e += blockDim.x) s += row[e];
  const float mean = rb_block_sum(s, scratch) / (float)E;
  float v = 0.f;
  for (int e = threadIdx.x; e < E; e += blockDim.x) { const float d = row[e] - mean; v = fmaf(d, d, v); }
  const float r = 1.0f / sqrtf(rb_block_sum(v, scratch) / (float)E + eps);
  TO* dst = out + (int64_t)blockIdx.x * E;
  for (int e = threadIdx.x; e < E; e += blockDim.x) dst[e] = rb_from_float<TO>((row[e] - mean) * r * w[e] + (b != nullptr ? b[e] : 0.f));
}

// The same with the row held in registers (NV groups of four values a thread, 16-byte accesses): the row is read once.
template <typename TO, int NV>
__global__ void __launch_bounds__(256) layernorm_reg_kernel(TO* __restrict__ out, const float* __restrict__ x,
                                                            const float* __restrict__ w, const float* __restrict__ b, int E,
                                                            float eps) {
  rb_pdl_launch_dependents();
  __shared__ float scratch[33];
  rb_pdl_wait();
  const float4* row = reinterpret_cast<const float4*>(x + (int64_t)blockIdx.x * E);
  const int E4 = E >> 2;
  float4 v[NV];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = threadIdx.x + i * 256;
    v[i] = e < E4 ? row[e] : make_float4(0.f, 0.f, 0.f, 0.f);
    s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
  }
  const float mean = rb_block_sum(s, scratch) / (float)E;
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = threadIdx.x + i * 256;
    if (e < E4) {
      v[i].x -= mean; v[i].y -= mean; v[i].z -= mean; v[i].w -= mean;
      q = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, q))));
    }
  }
  const float r = 1.0f / sqrtf(rb_block_sum(q, scratch) / (float)E + eps);
  TO* dst = out + (int64_t)blockIdx.x * E;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = threadIdx.x + i * 256;
    if (e < E4) {
      const float4 ww = reinterpret_cast<const float4*>(w)[e];
      const float4 bb = b != nullptr ? reinterpret_cast<const float4*>(b)[e] : make_float4(0.f, 0.f, 0.f, 0.f);
      store4<TO>(dst + 4 * e, v[i].x * r * ww.x + bb.x, v[i].y * r * ww.y + bb.y, v[i].z * r * ww.z + bb.z, v[i].w * r * ww.w + bb.w);
    }
  }
}

template <typename TO>
int launch_layernorm_reg(TO* out, const float* x, const float* w, const float* b, int T, int E, float eps, cudaStream_t stream) {
  const int groups = (E / 4 + 255) / 256;
  if (groups <= 1) RB_LAUNCH("layernorm_reg_kernel", (layernorm_reg_kernel<TO, 1>), T, 256, 0, stream, out, x, w, b, E, eps);
  else if (groups <= 2) RB_LAUNCH("layernorm_reg_kernel", (layernorm_reg_kernel<TO, 2>), T, 256, 0, stream, out, x, w, b, E, eps);
  else if (groups <= 4) RB_LAUNCH("layernorm_reg_kernel", (layernorm_reg_kernel<TO, 4>), T, 256, 0, stream, out, x, w, b, E, eps);
  else RB_LAUNCH("layernorm_reg_kernel", (layernorm_reg_kernel<TO, 8>), T, 256, 0, stream, out, x, w, b, E, eps);
  RB_CHECK_LAUNCH("rb_layernorm");
  return 0;
}

RB_EXPORT int rb_layernorm(void* out, int out_dtype, const float* x, const float* w, const float* b, int T, int E, float eps,
                           cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(E > 0, "rb_layernorm: width %d", E);
  if (E % 4 == 0 && E >= 512 && E <= 8192 && (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)b % 16 == 0 &&
      (uintptr_t)out % 16 == 0) {
    if (out_dtype == RB_F32) return launch_layernorm_reg<float>((float*)out, x, w, b, T, E, eps, stream);
    if (out_dtype == RB_BF16) return launch_layernorm_reg<__nv_bfloat16>((__nv_bfloat16*)out, x, w, b, T, E, eps, stream);
  }
  const int threads = E >= 1024 ? 256 : (E >= 256 ? 128 : 64);
  if (out_dtype == RB_F32)
    RB_LAUNCH("layernorm_kernel", (layernorm_kernel<float>), T, threads, 0, stream, (float*)out, x, w, b, E, eps);
  else if (out_dtype == RB_BF16)
    RB_LAUNCH("layernorm_kernel", (layernorm_kernel<__nv_bfloat16>), T, threads, 0, stream, (__nv_bfloat16*)out, x, w, b, E, eps);
  else
    RB_FAIL("rb_layernorm: unknown dtype %d", out_dtype);
  RB_CHECK_LAUNCH("rb_layernorm");
  return 0;
}

// ---------------------------------------------------------------- x += y, float32
__global__ void add_rows_kernel(float* __restrict__ x, const float* __restrict__ y, int64_t n) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) x[i] += y[i];
}

RB_EXPORT int rb_add_rows(float* x, const float* y, long long n, cudaStream_t stream) {
  if (n == 0) return 0;
  const long long most = (long long)rb_sm_count() * 16;
  const int blocks = (int)((n + 255) / 256 < most ? (n + 255) / 256 : most);
  RB_LAUNCH("add_rows_kernel", (add_rows_kernel), blocks, 256, 0, stream, x, y, (int64_t)n);
  RB_CHECK_LAUNCH("rb_add_rows");
  return 0;
}

// For every new token: rotate each q head and each k head by the token's
// position (angle = pos * inv_freq[i], float32; pairs (2i,2i+1) when
// `interleaved`, else (i, i+D/2)), write q to q_out[T,H,D], the rotated k and
// the raw v to the token's place in the paged cache.
// crates/bitnet-core/src/llama/model.rs:122-136 (rotation), :242-257 (append).
// `qkv` rows hold [H*D | Kh*D | Kh*D]; with write_kv == 0 only q is read (a
// layer that reads another layer's cache).  Only the first rot_dim values of a head are
// rotated (pairs (2i,2i+1) or (i, i+rot_dim/2) among them); the rest pass unchanged.
template <typename T>
__global__ void rotate_append_kernel(T* __restrict__ q_out, const T* __restrict__ qkv, int64_t qkv_stride,
                                     const float* __restrict__ inv_freq, const int* __restrict__ tok_pos,
                                     const int* __restrict__ tok_slot, RbPagedLayer cache, int H, int write_kv,
                                     int interleaved, int heads_per_block, int rot_dim) {
  rb_pdl_launch_dependents();
  const int t = blockIdx.x;
  const int D = cache.head_dim, Kh = cache.n_kv_heads;
  const int pos = tok_pos[t];
  const int slot = tok_slot[t];
  rb_pdl_wait();     // positions and slots were written before the step began; qkv comes from the kernel before
  const T* row = qkv + (int64_t)t * qkv_stride;
  auto value = [&](int64_t i) { return rb_to_float<T>(row[i]); };
  const int half = D / 2;
  const int n_rot_heads = H + (write_kv ? Kh : 0);
  const int n_heads = n_rot_heads + (write_kv ? Kh : 0);        // rotated heads, then the v heads
  const int h0 = blockIdx.y * heads_per_block, h1 = min(n_heads, h0 + heads_per_block);
  T* kdst = (T*)cache.k;
  T* vdst = (T*)cache.v;
  // one thread per pair of values: a rotated pair of a q or k head, or two neighbours of a v head
  for (int idx = threadIdx.x; idx < (h1 - h0) * half; idx += blockDim.x) {
    const int head = h0 + idx / half, i = idx % half;
    const int64_t src = (int64_t)head * D;  // q heads, k heads, v heads are contiguous in a row
    if (head >= n_rot_heads) {
      T* dst = vdst + rb_page_offset(cache, slot, pos, head - n_rot_heads);
      dst[2 * i] = rb_from_float<T>(value(src + 2 * i));
      dst[2 * i + 1] = rb_from_float<T>(value(src + 2 * i + 1));
      continue;
    }
    T* dst = head < H ? q_out + ((int64_t)t * H + head) * D : kdst + rb_page_offset(cache, slot, pos, head - H);
    const int rhalf = rot_dim / 2;
    if (i >= rhalf) {           // behind the rotated prefix: two neighbours, as they are
      const int a = rot_dim + 2 * (i - rhalf);
      dst[a] = rb_from_float<T>(value(src + a));
      dst[a + 1] = rb_from_float<T>(value(src + a + 1));
      continue;
    }
    int a, b;
    if (interleaved) { a = 2 * i; b = 2 * i + 1; } else { a = i; b = i + rhalf; }
    const float x0 = value(src + a);
    const float x1 = value(src + b);
    float sn, cs;
    sincosf((float)pos * inv_freq[i], &sn, &cs);
    const float y0 = x0 * cs - x1 * sn;
    const float y1 = x0 * sn + x1 * cs;
    dst[a] = rb_from_float<T>(y0);
    dst[b] = rb_from_float<T>(y1);
  }
}

// Many tokens, bfloat16 in and out, head_dim a multiple of 16: one block per token.  A thread owns
// eight rotation pairs (the same eight in every head), computes their sines and cosines once,
// and walks over the heads with 16-byte loads and stores; values are copied 16 bytes at a time.
constexpr int ROWS_MAX_PAIRS = 256;      // head sizes up to 512 take the many-token kernel
__global__ void __launch_bounds__(1024) rotate_append_rows_kernel(
    __nv_bfloat16* __restrict__ q_out, const __nv_bfloat16* __restrict__ qkv, int64_t qkv_stride,
    const float* __restrict__ inv_freq, const int* __restrict__ tok_pos, const int* __restrict__ tok_slot,
    RbPagedLayer cache, int H, int write_kv, int interleaved) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  const int t = blockIdx.x;
  const int D = cache.head_dim, Kh = cache.n_kv_heads;
  const int pos = tok_pos[t], slot = tok_slot[t];
  const __nv_bfloat16* row = qkv + (int64_t)t * qkv_stride;
  const int groups = D / 16;                       // groups of eight pairs per head
  const int lanes = blockDim.x / groups;           // threads that share a group walk different heads
  const int grp = threadIdx.x % groups, lane = threadIdx.x / groups;
  const int n_rot = H + (write_kv ? Kh : 0);
  __nv_bfloat16* kdst = (__nv_bfloat16*)cache.k;
  __nv_bfloat16* vdst = (__nv_bfloat16*)cache.v;
  // element offsets of the two 16-byte pieces this thread rotates in every head
  const int off_a = interleaved ? grp * 16 : grp * 8;
  const int off_b = interleaved ? grp * 16 + 8 : D / 2 + grp * 8;
  // the first head's values and the value rows are asked for before anything else, so that the loads
  // run while the sines and cosines are made (with one thread per head and group that is all of them)
  const bool active = lane < lanes && lane < n_rot;
  uint4 va = make_uint4(0, 0, 0, 0), vb = va, vv = va;
  if (active) {
    va = *reinterpret_cast<const uint4*>(row + (int64_t)lane * D + off_a);
    vb = *reinterpret_cast<const uint4*>(row + (int64_t)lane * D + off_b);
  }
  const int per_head = D / 8;
  const bool copies = write_kv && (int)threadIdx.x < Kh * per_head;
  if (copies) vv = *reinterpret_cast<const uint4*>(row + (int64_t)(H + Kh) * D + (int64_t)threadIdx.x * 8);
  // the token's D/2 sines and cosines, once per block
  __shared__ float s_sn[ROWS_MAX_PAIRS], s_cs[ROWS_MAX_PAIRS];
  for (int i = threadIdx.x; i < D / 2; i += blockDim.x) sincosf((float)pos * inv_freq[i], &s_sn[i], &s_cs[i]);
  __syncthreads();
  if (active) {
    float sn[8], cs[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) { sn[j] = s_sn[grp * 8 + j]; cs[j] = s_cs[grp * 8 + j]; }
    for (int head = lane; head < n_rot; head += lanes) {
      if (head != lane) {
        va = *reinterpret_cast<const uint4*>(row + (int64_t)head * D + off_a);
        vb = *reinterpret_cast<const uint4*>(row + (int64_t)head * D + off_b);
      }
      __nv_bfloat16* ea = reinterpret_cast<__nv_bfloat16*>(&va);
      __nv_bfloat16* eb = reinterpret_cast<__nv_bfloat16*>(&vb);
      if (interleaved) {
        // pairs (2i, 2i+1): pairs 0..3 lie in va, 4..7 in vb
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          __nv_bfloat16* e = j < 4 ? ea : eb;
          const int o = (j & 3) * 2;
          const float x0 = __bfloat162float(e[o]), x1 = __bfloat162float(e[o + 1]);
          e[o] = __float2bfloat16_rn(x0 * cs[j] - x1 * sn[j]);
          e[o + 1] = __float2bfloat16_rn(x0 * sn[j] + x1 * cs[j]);
        }
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const float x0 = __bfloat162float(ea[j]), x1 = __bfloat162float(eb[j]);
          ea[j] = __float2bfloat16_rn(x0 * cs[j] - x1 * sn[j]);
          eb[j] = __float2bfloat16_rn(x0 * sn[j] + x1 * cs[j]);
        }
      }
      __nv_bfloat16* dst = head < H ? q_out + ((int64_t)t * H + head) * D
                                    : kdst + rb_page_offset(cache, slot, pos, head - H);
      *reinterpret_cast<uint4*>(dst + off_a) = va;
      *reinterpret_cast<uint4*>(dst + off_b) = vb;
    }
  }
  if (write_kv) {
    const __nv_bfloat16* vsrc = row + (int64_t)(H + Kh) * D;
    for (int idx = threadIdx.x; idx < Kh * per_head; idx += blockDim.x) {
      const int kvh = idx / per_head, c = idx % per_head;
      if (idx != (int)threadIdx.x) vv = *reinterpret_cast<const uint4*>(vsrc + (int64_t)kvh * D + c * 8);
      *reinterpret_cast<uint4*>(vdst + rb_page_offset(cache, slot, pos, kvh) + c * 8) = vv;
    }
  }
}

// dtype: the type of qkv, of q_out and of the cache.
RB_EXPORT int rb_rotate_append(void* q_out, const void* qkv, int64_t qkv_stride, int dtype,
                               const float* inv_freq, const int* tok_pos, const int* tok_slot, void* cache_k,
                               void* cache_v, const int* page_table, int max_pages, int page_size, int T, int H,
                               int Kh, int D, int write_kv, int rot_dim, int interleaved, cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(D % 2 == 0 && D > 0, "rb_rotate_append: head_dim %d must be even", D);
  RB_REQUIRE(rot_dim >= 0 && rot_dim <= D && rot_dim % 2 == 0,
             "rb_rotate_append: the rotated prefix %d must be even and at most the head size %d", rot_dim, D);
  RB_REQUIRE(H > 0 && Kh >= 0 && page_size > 0, "rb_rotate_append: bad sizes H=%d Kh=%d page=%d", H, Kh, page_size);
  RbPagedLayer c{cache_k, cache_v, page_table, max_pages, page_size, Kh, D};
  const int threads = 256;
  // few tokens: spread a token's heads over several blocks so that enough blocks run
  const int n_heads = H + (write_kv ? 2 * Kh : 0);
  int by = T >= 128 ? 1 : (128 + T - 1) / T;
  if (by > n_heads) by = n_heads;
  const int hpb = (n_heads + by - 1) / by;
  const dim3 grid(T, (n_heads + hpb - 1) / hpb);
  if (dtype == RB_BF16 && T >= 32 && rot_dim == D && D % 16 == 0 && D <= 2 * ROWS_MAX_PAIRS &&
      qkv_stride % 8 == 0 && ((uintptr_t)qkv % 16 == 0) && ((uintptr_t)q_out % 16 == 0) &&
      ((uintptr_t)cache_k % 16 == 0) && ((uintptr_t)cache_v % 16 == 0)) {
    // one thread per (rotated head, group of eight pairs) where a block can hold them: one pass over the heads
    const int items = (H + (write_kv ? Kh : 0)) * (D / 16);
    const int rows_threads = items >= 1024 ? 1024 : (items < 128 ? 128 : (items + 31) / 32 * 32);
    RB_LAUNCH("rotate_append_rows_kernel", (rotate_append_rows_kernel), T, rows_threads, 0, stream, (__nv_bfloat16*)q_out,
              (const __nv_bfloat16*)qkv, qkv_stride, inv_freq, tok_pos, tok_slot, c, H, write_kv, interleaved);
    return 0;
  }
  if (dtype == RB_F32)
    RB_LAUNCH("rotate_append_kernel", (rotate_append_kernel<float>), grid, threads, 0, stream, (float*)q_out, (const float*)qkv, qkv_stride, inv_freq, tok_pos, tok_slot, c, H, write_kv, interleaved, hpb, rot_dim);
  else if (dtype == RB_BF16)
    RB_LAUNCH("rotate_append_kernel", (rotate_append_kernel<__nv_bfloat16>), grid, threads, 0, stream, (__nv_bfloat16*)q_out, (const __nv_bfloat16*)qkv, qkv_stride, inv_freq, tok_pos, tok_slot, c, H, write_kv, interleaved, hpb, rot_dim);
  else
    RB_FAIL("rb_rotate_append: unknown dtype %d", dtype);
  RB_CHECK_LAUNCH("rb_rotate_append");
  return 0;
}

// ---------------------------------------------------------------- SiLU(gate) * up
// out[t, j] = silu(gate[t, j]) * up[t, j], silu(v) = v / (1 + exp(-v)), in float32.
// crates/bitnet-core/src/llama/model.rs:116-120, 297-302
// block == 0: a row of gu is [gate (F) | up (F)].  block == B > 0: it is made of groups of 2B
// values, B of gate followed by the B of up for the same features (the row order the tensor-core
// gated product wants of its weights); `ld` is the row length of gu.
template <typename T, typename TI>
__global__ void silu_mul_kernel(T* __restrict__ out, const TI* __restrict__ gu, int64_t n, int F, int64_t ld, int block) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / F;
    const int j = (int)(i % F);
    const int64_t at_g = block > 0 ? (int64_t)(j / block) * 2 * block + j % block : j;
    const int64_t at_u = block > 0 ? at_g + block : (int64_t)F + j;
    const float g = rb_to_float<TI>(gu[t * ld + at_g]);
    const float u = rb_to_float<TI>(gu[t * ld + at_u]);
    out[i] = rb_from_float<T>(g / (1.0f + expf(-g)) * u);
  }
}

// in_dtype: dtype of gate_up (the output dtype, or RB_F32 for a bfloat16 output).
RB_EXPORT int rb_silu_mul(void* out, const void* gate_up, int dtype, int in_dtype, int T, int F, int64_t ld, int block,
                          cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(block >= 0 && (block == 0 ? ld >= 2 * (int64_t)F : ld >= ((int64_t)(F + block - 1) / block) * 2 * block),
             "rb_silu_mul: rows of %lld values do not hold %d features in blocks of %d", (long long)ld, F, block);
  const int64_t n = (int64_t)T * F;
  const int threads = 256;
  const int64_t most = (int64_t)rb_sm_count() * 16;
  const int blocks = (int)((n + threads - 1) / threads < most ? (n + threads - 1) / threads : most);
  if (dtype == RB_F32 && in_dtype == RB_F32)
    RB_LAUNCH("silu_mul_kernel", (silu_mul_kernel<float, float>), blocks, threads, 0, stream, (float*)out, (const float*)gate_up, n, F, ld, block);
  else if (dtype == RB_BF16 && in_dtype == RB_BF16)
    RB_LAUNCH("silu_mul_kernel", (silu_mul_kernel<__nv_bfloat16, __nv_bfloat16>), blocks, threads, 0, stream, (__nv_bfloat16*)out, (const __nv_bfloat16*)gate_up, n, F, ld, block);
  else if (dtype == RB_BF16 && in_dtype == RB_F32)
    RB_LAUNCH("silu_mul_kernel", (silu_mul_kernel<__nv_bfloat16, float>), blocks, threads, 0, stream, (__nv_bfloat16*)out, (const float*)gate_up, n, F, ld, block);
  else
    RB_FAIL("rb_silu_mul: unsupported dtypes %d <- %d", dtype, in_dtype);
  return 0;
}

// ---------------------------------------------------------------- row gather (float32 residual rows)
__global__ void gather_rows_kernel(float* __restrict__ out, const float* __restrict__ x,
                                   const int* __restrict__ rows, int E) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  // one element (or one group of four) per thread: the copies of a row are all in flight together
  const int r = blockIdx.x;
  const float* src = x + (int64_t)rows[r] * E;
  float* dst = out + (int64_t)r * E;
  const int j = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
  if ((E & 3) == 0) {
    if (j < E) *reinterpret_cast<float4*>(dst + j) = *reinterpret_cast<const float4*>(src + j);
  } else {
    for (int i = j; i < min(E, j + 4); ++i) dst[i] = src[i];
  }
}

RB_EXPORT int rb_gather_rows(float* out, const float* x, const int* rows, int R, int E, cudaStream_t stream) {
  if (R == 0) return 0;
  RB_REQUIRE(R <= 2147483647 && (E + 1023) / 1024 <= 65535, "rb_gather_rows: %d rows of %d", R, E);
  RB_LAUNCH("gather_rows_kernel", (gather_rows_kernel), dim3(R, (E + 1023) / 1024), 256, 0, stream, out, x, rows, E);
  RB_CHECK_LAUNCH("rb_gather_rows");
  return 0;
}

// ---------------------------------------------------------------- decode bookkeeping on the device
// After a decode step has sampled: the sampled ids become the next step's tokens and every
// position moves on by one, so that steps can follow one another without the host.  Only the first
// *n_live rows move (n_live null: all B): rows behind them belong to the padding sequence, which
// rewrites its position 0 at every step.
__global__ void decode_advance_kernel(int* __restrict__ token_ids, int* __restrict__ tok_pos,
                                      const int* __restrict__ sampled, int B, const int* __restrict__ n_live,
                                      const int* flag_a, const int* flag_b, int* __restrict__ flag_out) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  const int live = n_live != nullptr ? *n_live : B;
  if (i < B && i < live) {
    token_ids[i] = sampled[i];
    tok_pos[i] += 1;
  }
  // the error words of the kernels that wait on barriers travel with the step's results
  if (i == 0 && flag_out != nullptr) {
    const int a = flag_a != nullptr ? *flag_a : 0, b = flag_b != nullptr ? *flag_b : 0;
    *flag_out = a != 0 ? a : b;
  }
}

RB_EXPORT int rb_decode_advance(int* token_ids, int* tok_pos, const int* sampled, int B, const int* n_live,
                                const int* flag_a, const int* flag_b, int* flag_out, cudaStream_t stream) {
  if (B == 0) return 0;
  RB_LAUNCH("decode_advance_kernel", (decode_advance_kernel), (B + 127) / 128, 128, 0, stream, token_ids, tok_pos, sampled, B,
            n_live, flag_a, flag_b, flag_out);
  RB_CHECK_LAUNCH("rb_decode_advance");
  return 0;
}


// ---------------------------------------------------------------- norm over a whole projection + rotation of a prefix + cache append
// Rows of projections [q (H D) | k (Kh D) | v (Kh Dv) | ...].  Per token:
//   q <- q / rms(q over all H D values) * wq     (likewise k; skipped without weights)
//   the first rot_dim values of every q and k head turn by the position's angles; cos and sin are
//   multiplied by `magnitude`; the rest of the head passes;
//   q goes to q_out[T, H, Dc]; k and v go to the token's place in the paged cache, whose rows are
//   Dc wide: values behind D (Dv) are written as zeros, so kernels that know one head size serve
//   keys and values of different sizes.
// The angle is position * freq in float64, brought into (-pi, pi] before the float32 sine and cosine,
// so that it does not lose digits at large positions.  freq: rot_dim/2 float64 values.
__device__ __forceinline__ void rb_angle_sincos(int pos, double freq, float magnitude, float* sn, float* cs) {
  const double a = (double)pos * freq;
  const double turns = rint(a * 0.15915494309189535);
  const float r = (float)fma(-turns, 6.283185307179586, a);
  sincosf(r, sn, cs);
  *sn *= magnitude;
  *cs *= magnitude;
}

template <typename T>
__global__ void __launch_bounds__(256) norm_rotate_append_kernel(
    T* __restrict__ q_out, const T* __restrict__ proj, int64_t ld, const float* __restrict__ q_norm_w,
    const float* __restrict__ k_norm_w, float eps, const double* __restrict__ freq, float magnitude,
    const int* __restrict__ tok_pos, const int* __restrict__ tok_slot, RbPagedLayer cache, int H, int D, int Dv,
    int rot_dim, int interleaved, int write_kv, int heads_per_block) {
  rb_pdl_launch_dependents();
  __shared__ float scratch[33];
  extern __shared__ float s_sincos[];              // rot_dim/2 sines, then as many cosines, of this token's position
  const int t = blockIdx.x;
  const int Dc = cache.head_dim, Kh = cache.n_kv_heads;
  const int pos = tok_pos[t], slot = tok_slot[t];
  // once per token: the float64 angle is the costly part, and every head turns by the same angles
  for (int i = threadIdx.x; i < rot_dim / 2; i += blockDim.x)
    rb_angle_sincos(pos, freq[i], magnitude, &s_sincos[i], &s_sincos[rot_dim / 2 + i]);
  rb_pdl_wait();
  const T* row = proj + (int64_t)t * ld;
  float rq = 1.f, rk = 1.f;
  if (q_norm_w != nullptr) {
    float ss = 0.f;
    for (int e = threadIdx.x; e < H * D; e += blockDim.x) { const float v = rb_to_float<T>(row[e]); ss += v * v; }
    ss = rb_block_sum(ss, scratch);
    rq = 1.0f / sqrtf(ss / (float)(H * D) + eps);
  }
  if (k_norm_w != nullptr && write_kv) {
    float ss = 0.f;
    for (int e = threadIdx.x; e < Kh * D; e += blockDim.x) { const float v = rb_to_float<T>(row[H * D + e]); ss += v * v; }
    ss = rb_block_sum(ss, scratch);
    rk = 1.0f / sqrtf(ss / (float)(Kh * D) + eps);
  }
  const int n_rot_heads = H + (write_kv ? Kh : 0);
  const int rhalf = rot_dim / 2;
  __syncthreads();                                 // the table is complete (also without a norm's sums before)
  T* kdst = (T*)cache.k;
  T* vdst = (T*)cache.v;
  // With few tokens a token's heads (q heads, k heads, then v heads) are spread over several blocks, each of which
  // makes the norms' sums for itself.
  const int h0 = blockIdx.y * heads_per_block, h1 = h0 + heads_per_block;
  const int r0 = min(h0, n_rot_heads), r1 = min(h1, n_rot_heads);
  // one output value per thread and turn: a q or k head's value (normed, turned or passed), or padding
  for (int idx = threadIdx.x + r0 * Dc; idx < r1 * Dc; idx += blockDim.x) {
    const int head = idx / Dc, e = idx % Dc;
    const bool is_q = head < H;
    T* dst = is_q ? q_out + ((int64_t)t * H + head) * Dc : kdst + rb_page_offset(cache, slot, pos, head - H);
    if (e >= D) { dst[e] = rb_from_float<T>(0.f); continue; }
    const int base = head * D;          // q heads, then k heads, are contiguous in a row
    const float* nw = is_q ? q_norm_w : k_norm_w;
    const float fac = is_q ? rq : rk;
    auto value = [&](int i) { const float v = rb_to_float<T>(row[base + i]); return nw != nullptr ? v * fac * nw[base - (is_q ? 0 : H * D) + i] : v; };
    float y;
    if (e >= rot_dim) {
      y = value(e);
    } else {
      int pair, other;
      bool first;
      if (interleaved) { pair = e >> 1; first = (e & 1) == 0; other = first ? e + 1 : e - 1; }
      else { first = e < rhalf; pair = first ? e : e - rhalf; other = first ? e + rhalf : e - rhalf; }
      const float sn = s_sincos[pair], cs = s_sincos[rhalf + pair];
      const float me = value(e), ot = value(other);
      y = first ? me * cs - ot * sn : me * cs + ot * sn;
    }
    dst[e] = rb_from_float<T>(y);
  }
  if (write_kv) {
    const T* vsrc = row + (int64_t)(H + Kh) * D;
    const int v0 = min(max(h0 - n_rot_heads, 0), Kh), v1 = min(max(h1 - n_rot_heads, 0), Kh);
    for (int idx = threadIdx.x + v0 * Dc; idx < v1 * Dc; idx += blockDim.x) {
      const int kvh = idx / Dc, e = idx % Dc;
      vdst[rb_page_offset(cache, slot, pos, kvh) + e] = e < Dv ? vsrc[kvh * Dv + e] : rb_from_float<T>(0.f);
    }
  }
}

// The same for bfloat16 rows whose heads are made of whole groups of eight values (D, Dv, Dc and the rotated prefix
// multiples of 8, interleaved pairs, 16-byte aligned rows): a thread takes eight neighbouring values at a time, which
// hold four whole pairs, with one 16-byte load and one 16-byte store.
__global__ void __launch_bounds__(256) norm_rotate_append_rows_kernel(
    __nv_bfloat16* __restrict__ q_out, const __nv_bfloat16* __restrict__ proj, int64_t ld, const float* __restrict__ q_norm_w,
    const float* __restrict__ k_norm_w, float eps, const double* __restrict__ freq, float magnitude,
    const int* __restrict__ tok_pos, const int* __restrict__ tok_slot, RbPagedLayer cache, int H, int D, int Dv,
    int rot_dim, int heads_per_block) {
  rb_pdl_launch_dependents();
  __shared__ float scratch[33];
  extern __shared__ float s_sincos[];
  const int t = blockIdx.x;
  const int Dc = cache.head_dim, Kh = cache.n_kv_heads;
  const int pos = tok_pos[t], slot = tok_slot[t];
  for (int i = threadIdx.x; i < rot_dim / 2; i += blockDim.x)
    rb_angle_sincos(pos, freq[i], magnitude, &s_sincos[i], &s_sincos[rot_dim / 2 + i]);
  rb_pdl_wait();
  const __nv_bfloat16* row = proj + (int64_t)t * ld;
  auto sum_squares = [&](const __nv_bfloat16* src, int n) {
    float ss = 0.f;
    for (int e = threadIdx.x * 8; e < n; e += blockDim.x * 8) {
      const uint4 raw = *reinterpret_cast<const uint4*>(src + e);
      const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(p2[j]);
        ss += f.x * f.x + f.y * f.y;
      }
    }
    return rb_block_sum(ss, scratch);
  };
  float rq = 1.f, rk = 1.f;
  if (q_norm_w != nullptr) rq = 1.0f / sqrtf(sum_squares(row, H * D) / (float)(H * D) + eps);
  if (k_norm_w != nullptr) rk = 1.0f / sqrtf(sum_squares(row + H * D, Kh * D) / (float)(Kh * D) + eps);
  __syncthreads();
  const int n_rot_heads = H + Kh, per_head = Dc / 8;
  const int h0 = blockIdx.y * heads_per_block, h1 = h0 + heads_per_block;
  const int r0 = min(h0, n_rot_heads), r1 = min(h1, n_rot_heads);
  __nv_bfloat16* kdst = (__nv_bfloat16*)cache.k;
  __nv_bfloat16* vdst = (__nv_bfloat16*)cache.v;
  for (int idx = threadIdx.x + r0 * per_head; idx < r1 * per_head; idx += blockDim.x) {
    const int head = idx / per_head, e = (idx - head * per_head) * 8;
    const bool is_q = head < H;
    __nv_bfloat16* dst = is_q ? q_out + ((int64_t)t * H + head) * Dc : kdst + rb_page_offset(cache, slot, pos, head - H);
    uint4 out = make_uint4(0, 0, 0, 0);
    if (e < D) {
      const int base = head * D + e;
      const uint4 raw = *reinterpret_cast<const uint4*>(row + base);
      const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
      const float* nw = is_q ? q_norm_w : k_norm_w;
      const float fac = is_q ? rq : rk;
      float v[8];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(p2[j]);
        v[2 * j] = f.x;
        v[2 * j + 1] = f.y;
      }
      if (nw != nullptr) {
        const float* w = nw + (is_q ? base : base - H * D);
        const float4 wa = *reinterpret_cast<const float4*>(w), wb = *reinterpret_cast<const float4*>(w + 4);
        const float ww[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = v[j] * fac * ww[j];
      }
      if (e < rot_dim) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float sn = s_sincos[e / 2 + j], cs = s_sincos[rot_dim / 2 + e / 2 + j];
          const float a = v[2 * j], b = v[2 * j + 1];
          v[2 * j] = a * cs - b * sn;
          v[2 * j + 1] = b * cs + a * sn;
        }
      }
      __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
      for (int j = 0; j < 4; ++j) o2[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
    }
    *reinterpret_cast<uint4*>(dst + e) = out;
  }
  const __nv_bfloat16* vsrc = row + (int64_t)(H + Kh) * D;
  const int v0 = min(max(h0 - n_rot_heads, 0), Kh), v1 = min(max(h1 - n_rot_heads, 0), Kh);
  for (int idx = threadIdx.x + v0 * per_head; idx < v1 * per_head; idx += blockDim.x) {
    const int kvh = idx / per_head, e = (idx - kvh * per_head) * 8;
    const uint4 val = e < Dv ? *reinterpret_cast<const uint4*>(vsrc + kvh * Dv + e) : make_uint4(0, 0, 0, 0);
    *reinterpret_cast<uint4*>(vdst + rb_page_offset(cache, slot, pos, kvh) + e) = val;
  }
}

// The same rows with a norm per head AFTER the rotation: every q and k head is turned (a prefix of it) and then
// divided by its own root mean square over its D values (no weight).  A block per token (its heads spread over several
// blocks when tokens are few) makes the sines and cosines of the token's position once; then a warp per head, a lane
// holding every 32nd value of the head in registers (D up to 32 * HN_MAX).
constexpr int HN_MAX = 16;
template <typename T, int NG>      // NG: groups of 32 values a head's cache row holds at most
__global__ void __launch_bounds__(256) rotate_headnorm_append_kernel(
    T* __restrict__ q_out, const T* __restrict__ proj, int64_t ld, float eps, const double* __restrict__ freq, float magnitude,
    const int* __restrict__ tok_pos, const int* __restrict__ tok_slot, RbPagedLayer cache, int n_tokens, int H, int D, int Dv,
    int rot_dim, int interleaved, int write_kv, int heads_per_block) {
  rb_pdl_launch_dependents();
  extern __shared__ float s_sincos[];              // rot_dim/2 sines, then as many cosines, of this token's position
  rb_pdl_wait();
  const int Dc = cache.head_dim, Kh = cache.n_kv_heads;
  const int per_token = H + (write_kv ? 2 * Kh : 0);
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int pos = tok_pos[t], slot = tok_slot[t];
  const int rhalf = rot_dim / 2;
  for (int i = threadIdx.x; i < rhalf; i += blockDim.x)
    rb_angle_sincos(pos, freq[i], magnitude, &s_sincos[i], &s_sincos[rhalf + i]);
  __syncthreads();
  const T* row = proj + (int64_t)t * ld;
  const int h_end = min(per_token, (int)(blockIdx.y + 1) * heads_per_block);
  for (int head = blockIdx.y * heads_per_block + (threadIdx.x >> 5); head < h_end; head += blockDim.x >> 5) {
  if (head >= H + Kh) {
    // a value head: copied, padded with zeros
    const int kvh = head - H - Kh;
    T* dst = (T*)cache.v + rb_page_offset(cache, slot, pos, kvh);
    const T* src = row + (int64_t)(H + Kh) * D + kvh * Dv;
    for (int e = lane; e < Dc; e += 32) dst[e] = e < Dv ? src[e] : rb_from_float<T>(0.f);
    continue;
  }
  const bool is_q = head < H;
  T* dst = is_q ? q_out + ((int64_t)t * H + head) * Dc : (T*)cache.k + rb_page_offset(cache, slot, pos, head - H);
  const T* src = row + (int64_t)head * D;
  float y[NG];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int e = lane + 32 * i;
    y[i] = 0.f;
    if (e >= D) continue;
    const float me = rb_to_float<T>(src[e]);
    if (e >= rot_dim) {
      y[i] = me;
    } else {
      int pair, other;
      bool first;
      if (interleaved) { pair = e >> 1; first = (e & 1) == 0; other = first ? e + 1 : e - 1; }
      else { first = e < rhalf; pair = first ? e : e - rhalf; other = first ? e + rhalf : e - rhalf; }
      const float sn = s_sincos[pair], cs = s_sincos[rhalf + pair];
      const float ot = rb_to_float<T>(src[other]);
      y[i] = first ? me * cs - ot * sn : me * cs + ot * sn;
    }
    ss = fmaf(y[i], y[i], ss);
  }
  ss = rb_warp_sum(ss);
  const float r = 1.0f / sqrtf(ss / (float)D + eps);
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int e = lane + 32 * i;
    if (e < Dc) dst[e] = rb_from_float<T>(e < D ? y[i] * r : 0.f);
  }
  }
}

// dtype: the type of the projections, of q_out and of the cache.  Dc: the width of q_out's and the cache's heads.
// head_norm: the norm is one per head, after the rotation, without weights (q_norm_w and k_norm_w unused).
RB_EXPORT int rb_norm_rotate_append(void* q_out, const void* proj, int64_t ld, int dtype, const float* q_norm_w,
                                    const float* k_norm_w, float eps, const double* freq, float magnitude,
                                    const int* tok_pos, const int* tok_slot, void* cache_k, void* cache_v,
                                    const int* page_table, int max_pages, int page_size, int T, int H, int Kh, int D,
                                    int Dv, int Dc, int rot_dim, int interleaved, int write_kv, int head_norm,
                                    cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(H > 0 && Kh > 0 && D > 0 && Dv > 0 && Dc >= D && Dc >= Dv && page_size > 0,
             "rb_norm_rotate_append: bad sizes H=%d Kh=%d D=%d Dv=%d cache width %d", H, Kh, D, Dv, Dc);
  RB_REQUIRE(rot_dim >= 0 && rot_dim <= D && rot_dim % 2 == 0 && (rot_dim == 0 || freq != nullptr),
             "rb_norm_rotate_append: the rotated prefix %d must be even and at most the head size %d", rot_dim, D);
  RbPagedLayer c{cache_k, cache_v, page_table, max_pages, page_size, Kh, Dc};
  if (head_norm) {
    RB_REQUIRE(Dc <= 32 * HN_MAX, "rb_norm_rotate_append: a norm per head for heads of up to %d values (found %d)", 32 * HN_MAX, Dc);
    // few tokens: spread a token's heads over several blocks so that enough blocks run
    const int per_token = H + (write_kv ? 2 * Kh : 0);
    int by = T >= 128 ? 1 : (128 + T - 1) / T;
    if (by > per_token) by = per_token;
    const int hpb = (per_token + by - 1) / by;
    const dim3 blocks(T, (per_token + hpb - 1) / hpb);
    const int threads = hpb >= 4 ? 128 : (hpb >= 2 ? 64 : 32);
    const size_t table = (size_t)rot_dim * sizeof(float);
    const int groups = (Dc + 31) / 32;
#define HN_GO(NG)                                                                                                                  \
  do {                                                                                                                             \
    if (dtype == RB_F32)                                                                                                           \
      RB_LAUNCH("rotate_headnorm_append_kernel", (rotate_headnorm_append_kernel<float, NG>), blocks, threads, table, stream,       \
                (float*)q_out, (const float*)proj, ld, eps, freq, magnitude, tok_pos, tok_slot, c, T, H, D, Dv, rot_dim,           \
                interleaved, write_kv, hpb);                                                                                       \
    else if (dtype == RB_BF16)                                                                                                     \
      RB_LAUNCH("rotate_headnorm_append_kernel", (rotate_headnorm_append_kernel<__nv_bfloat16, NG>), blocks, threads, table,       \
                stream, (__nv_bfloat16*)q_out, (const __nv_bfloat16*)proj, ld, eps, freq, magnitude, tok_pos, tok_slot, c, T, H,   \
                D, Dv, rot_dim, interleaved, write_kv, hpb);                                                                       \
    else                                                                                                                           \
      RB_FAIL("rb_norm_rotate_append: unknown dtype %d", dtype);                                                                   \
  } while (0)
    if (groups <= 1) HN_GO(1);
    else if (groups <= 2) HN_GO(2);
    else if (groups <= 4) HN_GO(4);
    else if (groups <= 8) HN_GO(8);
    else HN_GO(16);
#undef HN_GO
    RB_CHECK_LAUNCH("rb_norm_rotate_append");
    return 0;
  }
  // few tokens: spread a token's heads over several blocks so that enough blocks run
  const int n_heads = H + (write_kv ? 2 * Kh : 0);
  int by = T >= 128 ? 1 : (128 + T - 1) / T;
  if (by > n_heads) by = n_heads;
  const int hpb = (n_heads + by - 1) / by;
  const dim3 grid(T, (n_heads + hpb - 1) / hpb);
  if (dtype == RB_BF16 && write_kv && interleaved && D % 8 == 0 && Dv % 8 == 0 && Dc % 8 == 0 && rot_dim % 8 == 0 && ld % 8 == 0 &&
      (uintptr_t)proj % 16 == 0 && (uintptr_t)q_out % 16 == 0 && (uintptr_t)cache_k % 16 == 0 && (uintptr_t)cache_v % 16 == 0 &&
      (uintptr_t)q_norm_w % 16 == 0 && (uintptr_t)k_norm_w % 16 == 0) {
    RB_LAUNCH("norm_rotate_append_rows_kernel", (norm_rotate_append_rows_kernel), grid, 256, (size_t)rot_dim * sizeof(float), stream,
              (__nv_bfloat16*)q_out, (const __nv_bfloat16*)proj, ld, q_norm_w, k_norm_w, eps, freq, magnitude, tok_pos, tok_slot,
              c, H, D, Dv, rot_dim, hpb);
    RB_CHECK_LAUNCH("rb_norm_rotate_append");
    return 0;
  }
  if (dtype == RB_F32)
    RB_LAUNCH("norm_rotate_append_kernel", (norm_rotate_append_kernel<float>), grid, 256, (size_t)rot_dim * sizeof(float), stream, (float*)q_out, (const float*)proj, ld, q_norm_w, k_norm_w, eps, freq, magnitude, tok_pos, tok_slot, c, H, D, Dv, rot_dim, interleaved, write_kv, hpb);
  else if (dtype == RB_BF16)
    RB_LAUNCH("norm_rotate_append_kernel", (norm_rotate_append_kernel<__nv_bfloat16>), grid, 256, (size_t)rot_dim * sizeof(float), stream, (__nv_bfloat16*)q_out, (const __nv_bfloat16*)proj, ld, q_norm_w, k_norm_w, eps, freq, magnitude, tok_pos, tok_slot, c, H, D, Dv, rot_dim, interleaved, write_kv, hpb);
  else
    RB_FAIL("rb_norm_rotate_append: unknown dtype %d", dtype);
  RB_CHECK_LAUNCH("rb_norm_rotate_append");
  return 0;
}

// ---------------------------------------------------------------- a gate per head on the attention's output
// out[t, h*Dv + j] = a[t, h*Dc + j] * sigmoid(gate[t*ldg + h]) for j < Dv: drops the padding of heads that are
// Dc wide and applies one gate value per head (no gate: gate == null), or one per value (per_value:
// gate[t*ldg + h*Dv + j]).
template <typename T>
__global__ void head_gate_kernel(T* __restrict__ out, const T* __restrict__ a, const T* __restrict__ gate, int64_t ldg,
                                 int64_t n, int H, int Dv, int Dc, int per_value) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / ((int64_t)H * Dv);
    const int r = (int)(i % ((int64_t)H * Dv));
    const int h = r / Dv, j = r % Dv;
    float v = rb_to_float<T>(a[(t * H + h) * Dc + j]);
    if (gate != nullptr) v *= 1.0f / (1.0f + expf(-rb_to_float<T>(gate[t * ldg + (per_value ? r : h)])));
    out[i] = rb_from_float<T>(v);
  }
}

// The same for bfloat16 rows in groups of eight values (Dv and Dc multiples of 8, 16-byte aligned rows).
__global__ void head_gate_rows_kernel(__nv_bfloat16* __restrict__ out, const __nv_bfloat16* __restrict__ a,
                                      const __nv_bfloat16* __restrict__ gate, int64_t ldg, int64_t n8, int H, int Dv, int Dc,
                                      int per_value) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  const int per_row = H * Dv / 8;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n8; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / per_row;
    const int r = (int)(i - t * per_row) * 8;
    const int h = r / Dv, j = r - h * Dv;
    const uint4 raw = *reinterpret_cast<const uint4*>(a + (t * H + h) * Dc + j);
    const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
    float v[8];
#pragma unroll
    for (int k = 0; k < 4; ++k) { const float2 f = __bfloat1622float2(p2[k]); v[2 * k] = f.x; v[2 * k + 1] = f.y; }
    if (gate != nullptr && per_value) {
      const uint4 graw = *reinterpret_cast<const uint4*>(gate + t * ldg + r);
      const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&graw);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 f = __bfloat1622float2(g2[k]);
        v[2 * k] *= 1.0f / (1.0f + expf(-f.x));
        v[2 * k + 1] *= 1.0f / (1.0f + expf(-f.y));
      }
    } else if (gate != nullptr) {
      const float g = 1.0f / (1.0f + expf(-__bfloat162float(gate[t * ldg + h])));
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] *= g;
    }
    uint4 res;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&res);
#pragma unroll
    for (int k = 0; k < 4; ++k) o2[k] = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
    *reinterpret_cast<uint4*>(out + t * (int64_t)H * Dv + r) = res;
  }
}

RB_EXPORT int rb_head_gate(void* out, const void* a, const void* gate, int64_t ldg, int dtype, int T, int H, int Dv, int Dc,
                           int per_value, cudaStream_t stream) {
  if (T == 0) return 0;
  const int64_t n = (int64_t)T * H * Dv;
  if (dtype == RB_BF16 && Dv % 8 == 0 && Dc % 8 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)a % 16 == 0 &&
      (gate == nullptr || !per_value || (ldg % 8 == 0 && (uintptr_t)gate % 16 == 0))) {
    const int64_t n8 = n / 8;
    const int64_t most8 = (int64_t)rb_sm_count() * 16;
    const int blocks8 = (int)((n8 + 255) / 256 < most8 ? (n8 + 255) / 256 : most8);
    RB_LAUNCH("head_gate_rows_kernel", (head_gate_rows_kernel), blocks8, 256, 0, stream, (__nv_bfloat16*)out, (const __nv_bfloat16*)a,
              (const __nv_bfloat16*)gate, ldg, n8, H, Dv, Dc, per_value);
    RB_CHECK_LAUNCH("rb_head_gate");
    return 0;
  }
  const int threads = 256;
  const int64_t most = (int64_t)rb_sm_count() * 16;
  const int blocks = (int)((n + threads - 1) / threads < most ? (n + threads - 1) / threads : most);
  if (dtype == RB_F32)
    RB_LAUNCH("head_gate_kernel", (head_gate_kernel<float>), blocks, threads, 0, stream, (float*)out, (const float*)a, (const float*)gate, ldg, n, H, Dv, Dc, per_value);
  else if (dtype == RB_BF16)
    RB_LAUNCH("head_gate_kernel", (head_gate_kernel<__nv_bfloat16>), blocks, threads, 0, stream, (__nv_bfloat16*)out, (const __nv_bfloat16*)a, (const __nv_bfloat16*)gate, ldg, n, H, Dv, Dc, per_value);
  else
    RB_FAIL("rb_head_gate: unknown dtype %d", dtype);
  RB_CHECK_LAUNCH("rb_head_gate");
  return 0;
}

// ---------------------------------------------------------------- gated activations
// kind 0: out = g' * sigmoid(alpha * g') * (u' + shift),  g' = min(g, limit),  u' = clamp(u, -limit, limit)
//         (limit <= 0: no limit).  alpha = 1, shift = 0 without a limit is SiLU(gate) * up.
// kind 1: out = gelu_tanh(g) * u, with gelu_tanh(g) = g * sigmoid(2 sqrt(2/pi) (g + 0.044715 g^3)), which is
//         g/2 * (1 + tanh(...)) written with one exponential
// bias (or null): a number per column of gu, added first.  Row layouts as rb_silu_mul.
template <typename T, typename TI>
__global__ void gated_act_kernel(T* __restrict__ out, const TI* __restrict__ gu, int64_t n, int F, int64_t ld, int block,
                                 int kind, float alpha, float limit, float shift, const float* __restrict__ bias) {
  rb_pdl_launch_dependents();
  rb_pdl_wait();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / F;
    const int j = (int)(i % F);
    const int64_t at_g = block > 0 ? (int64_t)(j / block) * 2 * block + j % block : j;
    const int64_t at_u = block > 0 ? at_g + block : (int64_t)F + j;
    float g = rb_to_float<TI>(gu[t * ld + at_g]);
    float u = rb_to_float<TI>(gu[t * ld + at_u]);
    if (bias != nullptr) { g += bias[at_g]; u += bias[at_u]; }
    if (kind == 1) {
      out[i] = rb_from_float<T>(g / (1.0f + expf(-1.5957691216057308f * (g + 0.044715f * g * g * g))) * u);
      continue;
    }
    if (kind == 2) {
      out[i] = rb_from_float<T>(fmaxf(g, 0.f) * u);
      continue;
    }
    if (limit > 0.f) {
      g = fminf(g, limit);
      u = fminf(fmaxf(u, -limit), limit);
    }
    out[i] = rb_from_float<T>(g / (1.0f + expf(-alpha * g)) * (u + shift));
  }
}

RB_EXPORT int rb_gated_act(void* out, const void* gate_up, int dtype, int in_dtype, int T, int F, int64_t ld, int block,
                           int kind, float alpha, float limit, float shift, const float* bias, cudaStream_t stream) {
  if (T == 0) return 0;
  RB_REQUIRE(kind >= 0 && kind <= 2, "rb_gated_act: activation %d is not built (0: limited swish, 1: gelu in its tanh form, 2: relu)", kind);
  RB_REQUIRE(block >= 0 && (block == 0 ? ld >= 2 * (int64_t)F : ld >= ((int64_t)(F + block - 1) / block) * 2 * block),
             "rb_gated_act: rows of %lld values do not hold %d features in blocks of %d", (long long)ld, F, block);
  const int64_t n = (int64_t)T * F;
  const int threads = 256;
  const int64_t most = (int64_t)rb_sm_count() * 16;
  const int blocks = (int)((n + threads - 1) / threads < most ? (n + threads - 1) / threads : most);
#define GO(TO, TI) RB_LAUNCH("gated_act_kernel", (gated_act_kernel<TO, TI>), blocks, threads, 0, stream, (TO*)out, (const TI*)gate_up, n, F, ld, block, kind, alpha, limit, shift, bias)
  if (dtype == RB_F32 && in_dtype == RB_F32) GO(float, float);
  else if (dtype == RB_BF16 && in_dtype == RB_BF16) GO(__nv_bfloat16, __nv_bfloat16);
  else if (dtype == RB_BF16 && in_dtype == RB_F32) GO(__nv_bfloat16, float);
  else RB_FAIL("rb_gated_act: unsupported dtypes %d <- %d", dtype, in_dtype);
#undef GO
  RB_CHECK_LAUNCH("rb_gated_act");
  return 0;
}

RB_CHECK_READER(elementwise)
