// Norms around a residual stream kept in 32-bit floats, for blocks that norm a sub-block's input and its output.
//
//   sandwich_stream:  s = stream[src] + y[src] / rms(y[src]) * (w_post + post_offset)
//                     stream[src] = s                                     (if write_stream)
//                     out[r] = s / rms(s) * (w_pre + pre_offset), rounded once to the storage type;  src = rows[r] or r
//   embed_rmsnorm:    stream[t] = e / rms(e) * (w + offset), e = table[ids[t]]
//
// rms(v) = sqrt(mean(v^2) + eps), each norm with its own eps.  Everything is computed in fp32.  One block per row; a row in
// steps of 8 up to 16,384 elements stays in registers between the passes, others in shared memory.
#include "nhv_common.cuh"
#include "nhv_vec8.cuh"

template <typename T, int CHUNKS>
__global__ void __launch_bounds__(512) sandwich_vec_kernel(T* __restrict__ out, float* __restrict__ stream, const T* __restrict__ y,
                                    const T* __restrict__ w_post, const T* __restrict__ w_pre, const int* __restrict__ rows,
                                    int width, float post_eps, float pre_eps, float post_offset, float pre_offset,
                                    int write_stream) {
  __shared__ float red[33];
  pdl_launch_dependents();
  float wp[CHUNKS][8];                                      // weights do not depend on the kernel before this one
#pragma unroll
  for (int k = 0; k < CHUNKS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c < width) nhv_load8(wp[k], w_post + c);
  }
  pdl_wait();
  const int r = blockIdx.x;
  const size_t src = (size_t)(rows ? rows[r] : r) * width;
  float s[CHUNKS][8], v[CHUNKS][8];
  float sy = 0.f;
#pragma unroll
  for (int k = 0; k < CHUNKS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c < width) {
      nhv_load8(v[k], y + src + c);
      nhv_load8(s[k], stream + src + c);
#pragma unroll
      for (int e = 0; e < 8; ++e) sy = fmaf(v[k][e], v[k][e], sy);
    }
  }
  const float ry = 1.0f / sqrtf(block_sum(sy, red) / (float)width + post_eps);
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < CHUNKS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c < width) {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        s[k][e] += v[k][e] * ry * (wp[k][e] + post_offset);
        ss = fmaf(s[k][e], s[k][e], ss);
      }
      if (write_stream) nhv_store8(stream + src + c, s[k]);
    }
  }
  const float rs = 1.0f / sqrtf(block_sum(ss, red) / (float)width + pre_eps);
#pragma unroll
  for (int k = 0; k < CHUNKS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c < width) {
      float w[8];
      nhv_load8(w, w_pre + c);
#pragma unroll
      for (int e = 0; e < 8; ++e) s[k][e] = s[k][e] * rs * (w[e] + pre_offset);
      nhv_store8(out + (size_t)r * width + c, s[k]);
    }
  }
}

template <typename T>
__global__ void sandwich_kernel(T* __restrict__ out, float* __restrict__ stream, const T* __restrict__ y,
                                const T* __restrict__ w_post, const T* __restrict__ w_pre, const int* __restrict__ rows,
                                int width, float post_eps, float pre_eps, float post_offset, float pre_offset,
                                int write_stream) {
  extern __shared__ float row[];
  __shared__ float red[33];
  pdl_prologue();
  const int r = blockIdx.x;
  const size_t src = (size_t)(rows ? rows[r] : r) * width;
  float sy = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = to_f32<T>(y[src + c]);
    row[c] = v;
    sy = fmaf(v, v, sy);
  }
  const float ry = 1.0f / sqrtf(block_sum(sy, red) / (float)width + post_eps);
  float ss = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float s = stream[src + c] + row[c] * ry * (to_f32<T>(w_post[c]) + post_offset);
    if (write_stream) stream[src + c] = s;
    row[c] = s;
    ss = fmaf(s, s, ss);
  }
  const float rs = 1.0f / sqrtf(block_sum(ss, red) / (float)width + pre_eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x)
    out[(size_t)r * width + c] = from_f32<T>(row[c] * rs * (to_f32<T>(w_pre[c]) + pre_offset));
}

static inline bool sw_aligned(const void* p) { return ((uintptr_t)p % 16) == 0; }

NHV_API int nhv_sandwich_stream(int dtype, void* out, float* stream_rows, const void* y, const void* w_post,
                                const void* w_pre, const int* rows, int n_rows, int width, float post_eps, float pre_eps,
                                float post_offset, float pre_offset, int write_stream, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  NHV_REQUIRE(n_rows > 0 && width > 0 && out && stream_rows && y && w_post && w_pre, "sandwich_stream: bad arguments");
  NHV_REQUIRE(!(rows && write_stream), "sandwich_stream: a gathered norm cannot write the stream back");
  const bool vec = width % 8 == 0 && width <= 16384 && sw_aligned(out) && sw_aligned(stream_rows) && sw_aligned(y) &&
                   sw_aligned(w_post) && sw_aligned(w_pre);
  if (vec) {
    // few rows: as many threads as a row has chunks of eight; many rows: two chunks a thread, so that a thread has more
    // loads on their way and an SM more rows
    const int chunks = width / 8, per = n_rows >= 256 && chunks > 64 ? 2 : 1;
    int threads = 32;
    while (threads < 512 && threads * per < chunks) threads <<= 1;
    const int need = (chunks + threads - 1) / threads;
#define GO(T, N)                                                                                                     \
  nhv_launch(sandwich_vec_kernel<T, N>, n_rows, threads, 0, stream, (T*)out, stream_rows, (const T*)y, (const T*)w_post, \
             (const T*)w_pre, rows, width, post_eps, pre_eps, post_offset, pre_offset, write_stream)
#define PICK(T)                 \
  do {                          \
    if (need <= 1) GO(T, 1);    \
    else if (need <= 2) GO(T, 2); \
    else GO(T, 4);              \
  } while (0)
    if (dtype == NHV_F32) PICK(float);
    else if (dtype == NHV_BF16) PICK(__nv_bfloat16);
    else NHV_REQUIRE(false, "sandwich_stream: unknown dtype %d", dtype);
#undef PICK
#undef GO
    NHV_CHECK_LAUNCH("sandwich_stream");
    return 0;
  }
  const size_t smem = (size_t)width * sizeof(float);
  NHV_REQUIRE(smem <= 200 * 1024, "sandwich_stream: width %d is beyond the %d floats a row buffer holds", width, 200 * 1024 / 4);
  int threads = 32;
  while (threads < 512 && threads * 4 < width) threads <<= 1;
#define GO(T)                                                                                                        \
  do {                                                                                                               \
    if (smem > 48 * 1024)                                                                                            \
      NHV_CUDA(cudaFuncSetAttribute(sandwich_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem),     \
               "sandwich_stream");                                                                                   \
    nhv_launch(sandwich_kernel<T>, n_rows, threads, smem, stream, (T*)out, stream_rows, (const T*)y,                 \
               (const T*)w_post, (const T*)w_pre, rows, width, post_eps, pre_eps, post_offset, pre_offset, write_stream); \
  } while (0)
  if (dtype == NHV_F32) GO(float);
  else if (dtype == NHV_BF16) GO(__nv_bfloat16);
  else NHV_REQUIRE(false, "sandwich_stream: unknown dtype %d", dtype);
#undef GO
  NHV_CHECK_LAUNCH("sandwich_stream");
  return 0;
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(512) embed_rmsnorm_kernel(float* __restrict__ out, const T* __restrict__ table, const int* __restrict__ ids,
                                     const T* __restrict__ w, int width, int vocab, float eps, float offset) {
  __shared__ float red[33];
  pdl_prologue();
  const int t = blockIdx.x, id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  const T* src = table + (size_t)(ok ? id : 0) * width;
  float ss = 0.f;
  if constexpr (VEC) {
    for (int c = threadIdx.x * 8; c < width; c += blockDim.x * 8) {
      float v[8];
      nhv_load8(v, src + c);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
    }
  } else {
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      const float v = to_f32<T>(src[c]);
      ss = fmaf(v, v, ss);
    }
  }
  const float r = ok ? 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps) : 0.f;      // an id outside the table: zeros
  if constexpr (VEC) {
    for (int c = threadIdx.x * 8; c < width; c += blockDim.x * 8) {
      float v[8], wv[8];
      nhv_load8(v, src + c);                                  // from the cache: the row was just read
      nhv_load8(wv, w + c);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = v[e] * r * (wv[e] + offset);
      nhv_store8(out + (size_t)t * width + c, v);
    }
    return;
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x)
    out[(size_t)t * width + c] = to_f32<T>(src[c]) * r * (to_f32<T>(w[c]) + offset);
}

NHV_API int nhv_embed_rmsnorm(int dtype, float* out, const void* table, const int* ids, const void* w, int n_tokens, int width,
                              int vocab, float eps, float offset, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  NHV_REQUIRE(n_tokens > 0 && width > 0 && vocab > 0, "embed_rmsnorm: bad sizes");
  const bool vec = width % 8 == 0 && sw_aligned(out) && sw_aligned(table) && sw_aligned(w);
  int threads = 32;
  while (threads < 512 && threads * (vec ? 8 : 4) < width) threads <<= 1;
#define GO(T, V)                                                                                                     \
  nhv_launch(embed_rmsnorm_kernel<T, V>, n_tokens, threads, 0, stream, out, (const T*)table, ids, (const T*)w, width, vocab, eps, offset)
  if (dtype == NHV_F32) { if (vec) GO(float, true); else GO(float, false); }
  else if (dtype == NHV_BF16) { if (vec) GO(__nv_bfloat16, true); else GO(__nv_bfloat16, false); }
  else NHV_REQUIRE(false, "embed_rmsnorm: unknown dtype %d", dtype);
#undef GO
  NHV_CHECK_LAUNCH("embed_rmsnorm");
  return 0;
}
