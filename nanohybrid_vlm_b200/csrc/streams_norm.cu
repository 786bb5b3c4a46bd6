// A residual stream kept as S copies per token in 32-bit floats (hyper-connections), [tokens, S, width].
//
// Between two sub-blocks every copy is rebuilt from all of them and the output y of the sub-block before, and the next
// sub-block reads a weighted sum of the copies through an RMS norm:
//   x'_t = sum_s mix[s, t] x_s + write[t] y          (all t at once from the old copies; without y the copies stay)
//   u    = sum_t read[t] x'_t                        (read null: the plain sum)
//   out  = u / sqrt(mean(u^2) + eps) * w             rounded once to the storage type
// One launch does both: a token's copies are read once and written once.  src_streams 1: all copies are still equal
// (nothing has been written yet) and src holds one row per token.  rows: gather (out[r] of token rows[r]; no write).
// All sums are fp32.  One block per row; u lives in shared memory between the two passes.
#include "nhv_common.cuh"

constexpr int SN_MAX_STREAMS = 16;

template <typename T, int V> struct SnVec;      // V consecutive elements as floats
template <> struct SnVec<float, 4> {
  static __device__ __forceinline__ void load(float (&o)[4], const float* p) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct SnVec<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(float (&o)[4], const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    o[0] = a.x; o[1] = a.y; o[2] = b.x; o[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = raw;
  }
};
template <typename T> struct SnVec<T, 1> {
  static __device__ __forceinline__ void load(float (&o)[1], const T* p) { o[0] = to_f32<T>(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_f32<T>(v[0]); }
};

// S: the number of copies the loops are unrolled for; n (<= S) the number there are.
template <typename T, int S, int V>
__global__ void __launch_bounds__(S <= 8 ? 512 : 256) streams_rmsnorm_kernel(T* __restrict__ out, float* dst, const float* src, int src_streams,
                                       const T* __restrict__ y, const float* __restrict__ mix,
                                       const float* __restrict__ write, const float* __restrict__ read,
                                       const T* __restrict__ w, const int* __restrict__ rows, int n, int width, float eps) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[33];
  float m[S][S], wr[S], rd[S];                  // the weights are not another kernel's work: fetched before the wait
#pragma unroll
  for (int t = 0; t < S; ++t) {
    rd[t] = t < n ? (read ? read[t] : 1.f) : 0.f;
    wr[t] = (y && t < n) ? write[t] : 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s) m[s][t] = (y && s < n && t < n) ? mix[s * n + t] : 0.f;
  }
  pdl_prologue();
  const int r = blockIdx.x;
  const size_t tok = rows ? rows[r] : r;
  const float* x = src + tok * src_streams * width;
  const size_t step = src_streams == 1 ? 0 : width;
  float* xd = dst ? dst + tok * n * width : nullptr;
  const T* yr = y ? y + tok * width : nullptr;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
    float xs[S][V], u[V];
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (s < n) SnVec<float, V>::load(xs[s], x + s * step + c);
      else {
#pragma unroll
        for (int i = 0; i < V; ++i) xs[s][i] = 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) u[i] = 0.f;
    if (yr) {
      float yv[V];
      SnVec<T, V>::load(yv, yr + c);
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (t < n) {
          float nx[V];
#pragma unroll
          for (int i = 0; i < V; ++i) {
            float a = wr[t] * yv[i];
#pragma unroll
            for (int s = 0; s < S; ++s) a = fmaf(m[s][t], xs[s][i], a);
            nx[i] = a;
            u[i] = fmaf(rd[t], a, u[i]);
          }
          if (xd) SnVec<float, V>::store(xd + (size_t)t * width + c, nx);
        }
      }
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] = fmaf(rd[s], xs[s][i], u[i]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(u[i], u[i], ss);
    SnVec<float, V>::store(row + c, u);
  }
  const float total = block_sum(ss, red);
  const float rstd = 1.0f / sqrtf(total / (float)width + eps);
  T* o = out + (size_t)r * width;
  for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
    float u[V], wv[V];
    SnVec<float, V>::load(u, row + c);
    SnVec<T, V>::load(wv, w + c);
#pragma unroll
    for (int i = 0; i < V; ++i) u[i] = u[i] * rstd * wv[i];
    SnVec<T, V>::store(o + c, u);
  }
}

// src: [tokens, src_streams, width], src_streams 1 or n_streams; dst (may be src when src_streams == n_streams; null: the
// new copies are not kept): [tokens, n_streams, width]; y (or null): [tokens, width]; mix [n, n] indexed [from, to],
// write [n], read [n] (or null): float32; out: [n_rows, width].
NHV_API int nhv_streams_rmsnorm(int dtype, void* out, float* dst, const float* src, int src_streams, const void* y,
                                const float* mix, const float* write, const float* read, const void* w, const int* rows,
                                int n_rows, int n_streams, int width, float eps, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  NHV_REQUIRE(n_rows > 0 && width > 0 && out && src && w, "streams_rmsnorm: bad arguments");
  NHV_REQUIRE(n_streams >= 1 && n_streams <= SN_MAX_STREAMS, "streams_rmsnorm: 1 to %d streams, not %d", SN_MAX_STREAMS, n_streams);
  NHV_REQUIRE(src_streams == 1 || src_streams == n_streams, "streams_rmsnorm: the source has one row per token or all streams");
  NHV_REQUIRE(!y || (mix && write), "streams_rmsnorm: a sub-block's output comes with its mixing matrix and write vector");
  NHV_REQUIRE(!(dst && (!y || rows)), "streams_rmsnorm: new streams are written only where a sub-block's output joins, and not by a gather");
  NHV_REQUIRE(dst != src || src_streams == n_streams, "streams_rmsnorm: streams cannot be written over a single row per token");
  const size_t smem = (size_t)((width + 3) / 4 * 4) * sizeof(float);
  NHV_REQUIRE(smem <= 200 * 1024, "streams_rmsnorm: width %d is beyond the %d floats a row buffer holds", width, 200 * 1024 / 4);
  const int item = dtype == NHV_F32 ? 4 : 2;
  const bool vec = width % 4 == 0 && ((uintptr_t)out % (4 * item)) == 0 && ((uintptr_t)dst % 16) == 0 && ((uintptr_t)src % 16) == 0 &&
                   ((uintptr_t)y % (4 * item)) == 0 && ((uintptr_t)w % (4 * item)) == 0;
  const int per = vec && n_streams <= 8 ? 4 : 1;
  // registers for the matrix and the copies leave few threads an SM: many small blocks where there are many rows
  const int most = n_rows <= 148 && n_streams <= 8 && (vec || n_streams <= 4) ? 512 : 256;
  int threads = 32;
  while (threads < most && threads * per < width) threads <<= 1;
#define GO(T, S, V)                                                                                                  \
  do {                                                                                                               \
    if (smem > 48 * 1024)                                                                                            \
      NHV_CUDA(cudaFuncSetAttribute(streams_rmsnorm_kernel<T, S, V>, cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                    (int)smem), "streams_rmsnorm");                                                  \
    nhv_launch(streams_rmsnorm_kernel<T, S, V>, n_rows, threads, smem, stream, (T*)out, dst, src, src_streams,       \
               (const T*)y, mix, write, read, (const T*)w, rows, n_streams, width, eps);                             \
  } while (0)
#define PICK(T)                                                    \
  do {                                                             \
    if (!vec) {                                                    \
      if (n_streams <= 4) GO(T, 4, 1); else GO(T, 16, 1);          \
    } else if (n_streams <= 2) GO(T, 2, 4);                        \
    else if (n_streams == 3) GO(T, 3, 4);                          \
    else if (n_streams == 4) GO(T, 4, 4);                          \
    else if (n_streams <= 6) GO(T, 6, 4);                          \
    else if (n_streams <= 8) GO(T, 8, 4);                          \
    else GO(T, 16, 1);                                             \
  } while (0)
  if (dtype == NHV_F32) PICK(float);
  else if (dtype == NHV_BF16) PICK(__nv_bfloat16);
  else NHV_REQUIRE(false, "streams_rmsnorm: unknown dtype %d", dtype);
#undef PICK
#undef GO
  NHV_CHECK_LAUNCH("streams_rmsnorm");
  return 0;
}
