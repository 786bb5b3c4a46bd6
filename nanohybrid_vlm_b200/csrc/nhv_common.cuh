// Shared helpers for the sm_100a kernels of this engine.
//
// Every exported function is `extern "C"`, takes raw device pointers, sizes and the
// CUDA stream to launch on, allocates nothing and returns 0 or an error code; the text
// of the last error is read with nhv_last_error().  Python binds them with ctypes.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#define NHV_API extern "C" __attribute__((visibility("default")))

enum NhvDtype { NHV_F32 = 0, NHV_BF16 = 1 };

#ifdef NHV_OWN_ERROR_TEXT
// A file compiled into a library of its own (tests do that) keeps the text of its last error itself and exports
// nhv_last_error() for it.
#include <stdarg.h>
static char nhv_own_error_text[512];
static void nhv_set_error(const char* fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(nhv_own_error_text, sizeof(nhv_own_error_text), fmt, ap);
  va_end(ap);
}
NHV_API const char* nhv_last_error() { return nhv_own_error_text; }
#else
// Defined in elementwise.cu.
void nhv_set_error(const char* fmt, ...);
#endif

#define NHV_REQUIRE(cond, ...)                                  \
  do {                                                          \
    if (!(cond)) {                                              \
      nhv_set_error(__VA_ARGS__);                               \
      return 1;                                                 \
    }                                                           \
  } while (0)

#define NHV_CHECK_LAUNCH(name)                                                        \
  do {                                                                                \
    cudaError_t e_ = cudaPeekAtLastError();                                           \
    if (e_ != cudaSuccess) {                                                          \
      nhv_set_error("%s: launch failed: %s", name, cudaGetErrorString(e_));           \
      return 2;                                                                       \
    }                                                                                 \
  } while (0)

#define NHV_CUDA(call, name)                                                          \
  do {                                                                                \
    cudaError_t e_ = (call);                                                          \
    if (e_ != cudaSuccess) {                                                          \
      nhv_set_error("%s: %s", name, cudaGetErrorString(e_));                          \
      return 2;                                                                       \
    }                                                                                 \
  } while (0)

// Programmatic dependent launch.  Every kernel of this library is launched with the attribute that
// lets it start while the kernel before it in the stream is still running, and every kernel begins
// with pdl_prologue(): it lets the kernel after it start likewise, then waits until the kernel before
// it has completed and its writes are visible.  Nothing may be read that another kernel writes, and
// nothing written at all, before that wait; what a kernel does before it (fetching weights) overlaps
// with its predecessor's tail.  Launch latency and pipeline fill leave the critical path this way.
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;\n" ::); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;\n" ::: "memory"); }
__device__ __forceinline__ void pdl_prologue() {
  pdl_launch_dependents();
  pdl_wait();
}

template <typename... KArgs, typename... Args>
inline cudaError_t nhv_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                              Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

// Shared memory to ask for so that a kernel of few, long-running blocks gets its blocks spread over the SMs: the
// block scheduler fills an SM as far as resources allow, and behind another kernel's tail that can leave several
// such blocks on one SM and other SMs idle.  `need`: what the block uses; `blocks`: the grid.  With a grid of up to
// `sms` blocks each block takes an SM's whole shared memory, with up to 2 * sms half of it, and so on; large grids
// ask for what they need.
inline size_t nhv_spread_smem(size_t need, long blocks, int sms = 148) {
  const long per_sm = (blocks + sms - 1) / sms;
  if (per_sm > 6) return need;
  const size_t share = (size_t)(233472 / per_sm) - 1024;      // 228 KB an SM, 1 KB reserved per block
  const size_t most = 232448;                                  // 227 KB a block
  const size_t want = share < most ? share : most;
  return want > need ? want : need;
}

// Two fp32 values in one 64-bit register and the arithmetic on both at once (sm_100: one instruction does two
// fused multiply-adds, each rounded as the scalar one is).  A 16-byte read of four floats is two such pairs.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 f2_pack(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void f2_unpack(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 f2_fma(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 f2_mul(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ float f2_sum(f32x2 a, f32x2 b) {     // (a.lo + a.hi) + (b.lo + b.hi)
  float x, y, z, w;
  f2_unpack(a, x, y);
  f2_unpack(b, z, w);
  return (x + y) + (z + w);
}

// The first key that a query at position pos may see besides causality: with a sliding window the last `window`
// keys (window > 0), with chunked attention the keys of its own chunk of `chunk` positions counted from position 0
// (chunk > 0); both 0: every key.  The result does not fall as pos grows, so the bound of a block's first row
// holds for the block.
__host__ __device__ __forceinline__ int nhv_first_key(int pos, int window, int chunk) {
  if (pos < 0) return 0;
  int lo = window > 0 ? (pos - window + 1 > 0 ? pos - window + 1 : 0) : 0;
  if (chunk > 0) {
    const int c = (pos / chunk) * chunk;
    lo = c > lo ? c : lo;
  }
  return lo;
}

// Scores capped smoothly, cap * tanh(z) with z = raw * scale / cap, in log2 units, so that exp2 of it is the exponential of
// the capped score.  Two forms, chosen by a warp for a whole tile of scores:
//   small scores (|z| <= 1/2 throughout): z times a polynomial in z^2, the least worst error over that range (3e-9; fitted
//     to tanh(z) / z by least squares on Chebyshev points, reweighted by the error), multiply-adds only;
//   else cap log2(e) (1 - 2 / (1 + e^(2 z))): `in` = 2 log2(e) scale / cap turns a raw score into the exponent of 2.  Two
//     scores share one reciprocal (of the product of both denominators, whose exponents are kept below 2^60 so that it
//     cannot overflow: tanh is 1 to the last bit long before).
// The error is a few units of 2^-24 of the cap in both.
struct NhvScoreCap {
  float in, out;        // in == 0: scores are not capped; out = cap log2(e)
  float z, small;       // scale / cap; the raw score at |z| = 1/2
  float c[5];           // the polynomial's coefficients times out
};
inline NhvScoreCap nhv_score_cap(float scale, float cap) {
  NhvScoreCap c = {};
  if (cap > 0.f) {
    const float tanh_over_z[5] = {0.9999999312f, -0.3333277586f, 0.1332057123f, -0.05276213199f, 0.01673756908f};
    c.in = 2.0f * 1.4426950408889634f * scale / cap;
    c.out = cap * 1.4426950408889634f;
    c.z = scale / cap;
    c.small = 0.5f * cap / (scale < 0.f ? -scale : scale);
    for (int i = 0; i < 5; ++i) c.c[i] = tanh_over_z[i] * c.out;
  }
  return c;
}
__device__ __forceinline__ float nhv_cap_small(float raw, const NhvScoreCap& c) {
  const float z = raw * c.z, t = z * z;
  return z * fmaf(fmaf(fmaf(fmaf(c.c[4], t, c.c[3]), t, c.c[2]), t, c.c[1]), t, c.c[0]);
}
__device__ __forceinline__ void nhv_cap_scores(float& a, float& b, const NhvScoreCap& c) {
  float ea, eb, r;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(ea) : "f"(fminf(a * c.in, 60.f)));
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(eb) : "f"(fminf(b * c.in, 60.f)));
  ea += 1.f;
  eb += 1.f;
  asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(r) : "f"(ea * eb));
  r *= -2.0f * c.out;
  a = fmaf(r, eb, c.out);
  b = fmaf(r, ea, c.out);
}
// The scores of a warp's tile, N groups of four a thread (scores that a mask replaces later may be anything).
template <int N>
__device__ __forceinline__ void nhv_cap_tile(float (&s)[N][4], const NhvScoreCap& c) {
  float m = 0.f;
#pragma unroll
  for (int j = 0; j < N; ++j)
    m = fmaxf(fmaxf(m, fmaxf(fabsf(s[j][0]), fabsf(s[j][1]))), fmaxf(fabsf(s[j][2]), fabsf(s[j][3])));
  if (__all_sync(0xffffffffu, m <= c.small)) {
#pragma unroll
    for (int j = 0; j < N; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[j][e] = nhv_cap_small(s[j][e], c);
  } else {
#pragma unroll
    for (int j = 0; j < N; ++j) {
      nhv_cap_scores(s[j][0], s[j][1], c);
      nhv_cap_scores(s[j][2], s[j][3], c);
    }
  }
}

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// Round a float to the storage type and back: the value the next op would read.
template <typename T> __device__ __forceinline__ float round_to(float v) { return to_f32<T>(from_f32<T>(v)); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result.  `red` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nwarp ? red[lane] : 0.f;
    t = warp_sum(t);
    if (lane == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}
