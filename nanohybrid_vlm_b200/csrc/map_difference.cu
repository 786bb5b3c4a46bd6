// Two attention maps per head brought together (differential attention): for head h of a token
//   o = a[2h] - share * a[2h + 1],   out[h] = o / sqrt(mean(o^2) + eps) * factor
// a [T, 2 H dv] holds the maps' outputs head by head, share is one number in device memory; the mean is over the head's
// dv elements.  Computed in fp32, rounded once.
#include "nhv_common.cuh"
#include "nhv_vec8.cuh"

// L lanes per head, CHUNKS times eight elements a lane.
template <typename T, int L, int CHUNKS>
__global__ void __launch_bounds__(256) map_difference_vec_kernel(T* __restrict__ out, int out_stride, const T* __restrict__ a,
                                                                 int a_stride, const float* __restrict__ share, float factor,
                                                                 float eps, int heads, int dv, long items) {
  pdl_prologue();
  const long item = (long)blockIdx.x * (256 / L) + threadIdx.x / L;
  const int lane = threadIdx.x & (L - 1);
  const bool live = item < items;
  const long t = live ? item / heads : 0;
  const int h = live ? (int)(item - t * heads) : 0;
  const float s = share[0];
  const T* a1 = a + (size_t)t * a_stride + (size_t)2 * h * dv;
  float o[CHUNKS][8];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < CHUNKS; ++k) {
    const int c = (lane + k * L) * 8;
    if (live && c < dv) {
      float x[8], y[8];
      nhv_load8(x, a1 + c);
      nhv_load8(y, a1 + dv + c);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        o[k][e] = fmaf(-s, y[e], x[e]);
        ss = fmaf(o[k][e], o[k][e], ss);
      }
    }
  }
#pragma unroll
  for (int m = L / 2; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  const float r = factor / sqrtf(ss / (float)dv + eps);
#pragma unroll
  for (int k = 0; k < CHUNKS; ++k) {
    const int c = (lane + k * L) * 8;
    if (live && c < dv) {
#pragma unroll
      for (int e = 0; e < 8; ++e) o[k][e] *= r;
      nhv_store8(out + (size_t)t * out_stride + (size_t)h * dv + c, o[k]);
    }
  }
}

// One warp per head, any size.
template <typename T>
__global__ void __launch_bounds__(128) map_difference_kernel(T* __restrict__ out, int out_stride, const T* __restrict__ a,
                                                             int a_stride, const float* __restrict__ share, float factor,
                                                             float eps, int heads, int dv, long items) {
  pdl_prologue();
  const long item = (long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= items) return;
  const long t = item / heads;
  const int h = (int)(item - t * heads);
  const float s = share[0];
  const T* a1 = a + (size_t)t * a_stride + (size_t)2 * h * dv;
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) {
    const float o = fmaf(-s, to_f32<T>(a1[dv + c]), to_f32<T>(a1[c]));
    ss = fmaf(o, o, ss);
  }
  const float r = factor / sqrtf(warp_sum(ss) / (float)dv + eps);
  for (int c = lane; c < dv; c += 32)
    out[(size_t)t * out_stride + (size_t)h * dv + c] = from_f32<T>(fmaf(-s, to_f32<T>(a1[dv + c]), to_f32<T>(a1[c])) * r);
}

NHV_API int nhv_map_difference(int dtype, void* out, int out_stride, const void* a, int a_stride, const float* share,
                               float factor, float eps, int n_rows, int heads, int dv, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  NHV_REQUIRE(n_rows > 0 && heads > 0 && dv > 0 && share && out_stride >= heads * dv && a_stride >= 2 * heads * dv,
              "map_difference: bad sizes");
  const long items = (long)n_rows * heads;
  const bool vec = dv % 8 == 0 && dv <= 512 && out_stride % 8 == 0 && a_stride % 8 == 0 && ((uintptr_t)out % 16) == 0 &&
                   ((uintptr_t)a % 16) == 0;
#define GO_VEC(T, L, CHUNKS)                                                                                             \
  nhv_launch(map_difference_vec_kernel<T, L, CHUNKS>, (unsigned)((items + 256 / L - 1) / (256 / L)), 256, 0, stream, (T*)out, \
             out_stride, (const T*)a, a_stride, share, factor, eps, heads, dv, items)
#define GO(T)                                                                                                         \
  do {                                                                                                                \
    if (!vec)                                                                                                         \
      nhv_launch(map_difference_kernel<T>, (unsigned)((items + 3) / 4), 128, 0, stream, (T*)out, out_stride,          \
                 (const T*)a, a_stride, share, factor, eps, heads, dv, items);                                        \
    else if (dv <= 64) GO_VEC(T, 8, 1);                                                                               \
    else if (dv <= 128) GO_VEC(T, 16, 1);                                                                             \
    else if (dv <= 256) GO_VEC(T, 32, 1);                                                                             \
    else GO_VEC(T, 32, 2);                                                                                            \
  } while (0)
  if (dtype == NHV_F32) GO(float);
  else if (dtype == NHV_BF16) GO(__nv_bfloat16);
  else NHV_REQUIRE(false, "map_difference: unknown dtype %d", dtype);
#undef GO
#undef GO_VEC
  NHV_CHECK_LAUNCH("map_difference");
  return 0;
}
