// Attention whose keys and values are one latent vector per token: what a token leaves in the cache, and the rotated
// part of its queries.
//
// One warp per (token, item).  Item 0 takes the token's row kv [rank + dr] of the down projection: the first `rank`
// elements are divided by their root mean square (eps inside the root) and multiplied by a weight [rank]: the latent;
// the last dr elements are one key part shared by all heads, of which the first rotary_dim rotate (element i with
// i + rotary_dim / 2, or (interleaved) element 2i with 2i + 1; angles from the table).  Both go to the token's slot of a page with one plane,
// [page][1][1][slot_in_page][row], row >= rank + dr, latent first; the rest of the row is cleared.
// Items 1 .. H take head h of q [T, H, dn + dr]: its last dr elements, rotated the same way, go to
// q_lat [T, H, rank + dr] behind the `rank` elements that a product with the keys' expansion fills.
// Norm and rotation are computed in fp32 and rounded once.
#include "nhv_common.cuh"
#include "nhv_vec8.cuh"

constexpr int LS_WARPS = 4;
constexpr int LS_MAX_ROW = 2048;

template <typename T>
__global__ void latent_rope_store_kernel(const T* __restrict__ kv, int kv_stride, const T* __restrict__ q, int q_stride,
                                         T* __restrict__ q_lat, int q_lat_stride, T* __restrict__ pages,
                                         const int* __restrict__ slot_mapping, const int* __restrict__ positions,
                                         const float* __restrict__ cos_sin, int rotary_dim, int max_position,
                                         int n_tokens, int H, int dn, int dr, int rank, int row, int page_size,
                                         int n_pages, float eps, const T* __restrict__ weight, int interleaved) {
  extern __shared__ float smem[];
  pdl_prologue();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long item = (long)blockIdx.x * LS_WARPS + warp;
  if (item >= (long)n_tokens * (H + 1)) return;
  const int t = (int)(item / (H + 1));
  const int which = (int)(item - (long)t * (H + 1));
  float* v = smem + (size_t)warp * (rank + dr);
  const float* cs = nullptr;
  const int half = rotary_dim >> 1;
  if (cos_sin) {
    int pos = positions[t];
    pos = pos < 0 ? 0 : (pos >= max_position ? max_position - 1 : pos);
    cs = cos_sin + (size_t)pos * rotary_dim;                    // cos[0..half) then sin[0..half)
  }
  auto turned = [&](const float* x, int c) {                    // element c of the rotated part x [dr]
    if (cs && interleaved && c < rotary_dim) {
      const int i = c >> 1;                                     // the pair (2i, 2i + 1) turns by angle i
      return (c & 1) ? x[c] * cs[i] + x[c - 1] * cs[half + i] : x[c] * cs[i] - x[c + 1] * cs[half + i];
    }
    if (cs && c < half) return x[c] * cs[c] - x[c + half] * cs[half + c];
    if (cs && c < rotary_dim) return x[c] * cs[c - half] + x[c - half] * cs[c];
    return x[c];
  };
  if (which == 0) {
    if (!pages) return;
    const int slot = slot_mapping[t];
    if (slot < 0 || slot >= n_pages * page_size) return;
    const T* src = kv + (size_t)t * kv_stride;
    for (int c = lane; c < rank + dr; c += 32) v[c] = to_f32<T>(src[c]);
    __syncwarp();
    float ss = 0.f;
    for (int c = lane; c < rank; c += 32) ss = fmaf(v[c], v[c], ss);
    ss = warp_sum(ss);
    const float r = 1.0f / sqrtf(ss / (float)rank + eps);
    T* dst = pages + (size_t)slot * row;
    for (int c = lane; c < rank; c += 32) dst[c] = from_f32<T>(v[c] * r * to_f32<T>(weight[c]));
    for (int c = lane; c < dr; c += 32) dst[rank + c] = from_f32<T>(turned(v + rank, c));
    for (int c = rank + dr + lane; c < row; c += 32) dst[c] = from_f32<T>(0.f);
  } else {
    const int h = which - 1;
    const T* src = q + (size_t)t * q_stride + (size_t)h * (dn + dr) + dn;
    for (int c = lane; c < dr; c += 32) v[c] = to_f32<T>(src[c]);
    __syncwarp();
    T* dst = q_lat + (size_t)t * q_lat_stride + (size_t)h * (rank + dr) + rank;
    for (int c = lane; c < dr; c += 32) dst[c] = from_f32<T>(turned(v, c));
  }
}

// The same in pieces of 8 elements (all sizes, offsets and strides in steps of 8): a warp takes a token's latent row (item
// 0), or 32 pieces of its queries' rotated parts (a head's dr / 8 pieces are neighbours).
template <typename T>
__global__ void latent_rope_store_vec_kernel(const T* __restrict__ kv, int kv_stride, const T* __restrict__ q, int q_stride,
                                             T* __restrict__ q_lat, int q_lat_stride, T* __restrict__ pages,
                                             const int* __restrict__ slot_mapping, const int* __restrict__ positions,
                                             const float* __restrict__ cos_sin, int rotary_dim, int max_position,
                                             int n_tokens, int items, int H, int dn, int dr, int rank, int row, int n_slots,
                                             float eps, const T* __restrict__ weight, int interleaved) {
  pdl_prologue();
  const int lane = threadIdx.x & 31, half = rotary_dim >> 1;
  const long item = (long)blockIdx.x * LS_WARPS + (threadIdx.x >> 5);
  if (item >= (long)n_tokens * items) return;
  const int t = (int)(item / items), which = (int)(item - (long)t * items);
  const float* cs = nullptr;
  if (cos_sin) {
    int pos = positions[t];
    pos = pos < 0 ? 0 : (pos >= max_position ? max_position - 1 : pos);
    cs = cos_sin + (size_t)pos * rotary_dim;                    // cos[0..half) then sin[0..half)
  }
  auto turn = [&](float (&x)[8], const T* part, int c0) {       // elements c0 .. c0 + 7 of the rotated part
    if (!cs || c0 >= rotary_dim) return;
    if (interleaved) {
#pragma unroll
      for (int k = 0; k < 8; k += 2) {
        const int i = (c0 + k) >> 1;
        const float co = cs[i], si = cs[half + i], a = x[k], b = x[k + 1];
        x[k] = a * co - b * si;
        x[k + 1] = b * co + a * si;
      }
    } else {                                                    // half is in steps of 8: the partners are one piece
      const bool first = c0 < half;
      const int i0 = first ? c0 : c0 - half;
      float p[8], co[8], si[8];
      nhv_load8(p, part + (first ? c0 + half : c0 - half));
      nhv_load8(co, cs + i0);
      nhv_load8(si, cs + half + i0);
#pragma unroll
      for (int k = 0; k < 8; ++k) x[k] = first ? x[k] * co[k] - p[k] * si[k] : x[k] * co[k] + p[k] * si[k];
    }
  };
  if (which == 0) {
    if (!pages) return;
    const int slot = slot_mapping[t];
    if (slot < 0 || slot >= n_slots) return;
    const T* src = kv + (size_t)t * kv_stride;
    T* dst = pages + (size_t)slot * row;
    float ss = 0.f;
    for (int c = lane * 8; c < rank; c += 256) {
      float x[8];
      nhv_load8(x, src + c);
#pragma unroll
      for (int k = 0; k < 8; ++k) ss = fmaf(x[k], x[k], ss);
    }
    ss = warp_sum(ss);
    const float r = 1.0f / sqrtf(ss / (float)rank + eps);
    for (int c = lane * 8; c < row; c += 256) {
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (c < rank) {
        float w[8];
        nhv_load8(x, src + c);
        nhv_load8(w, weight + c);
#pragma unroll
        for (int k = 0; k < 8; ++k) x[k] = x[k] * r * w[k];
      } else if (c < rank + dr) {
        nhv_load8(x, src + c);
        turn(x, src + rank, c - rank);
      }
      nhv_store8(dst + c, x);
    }
  } else {
    const int per = dr >> 3, e = (which - 1) * 32 + lane;
    if (e >= H * per) return;
    const int h = e / per, c0 = (e - h * per) * 8;
    const T* part = q + (size_t)t * q_stride + (size_t)h * (dn + dr) + dn;
    float x[8];
    nhv_load8(x, part + c0);
    turn(x, part, c0);
    nhv_store8(q_lat + (size_t)t * q_lat_stride + (size_t)h * (rank + dr) + rank + c0, x);
  }
}

NHV_API int nhv_latent_rope_store(int dtype, const void* kv, int kv_stride, const void* q, int q_stride, void* q_lat,
                                  int q_lat_stride, void* pages, const int* slot_mapping, const int* positions,
                                  const float* cos_sin, int rotary_dim, int max_position, int n_tokens, int H, int dn,
                                  int dr, int rank, int row, int page_size, int n_pages, float eps, const void* weight,
                                  int interleaved, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  NHV_REQUIRE(n_tokens > 0 && H > 0 && dn >= 0 && dr >= 0 && rank > 0, "latent_rope_store: bad sizes");
  NHV_REQUIRE(rank + dr <= LS_MAX_ROW, "latent_rope_store: a row of %d elements is beyond the supported %d", rank + dr, LS_MAX_ROW);
  NHV_REQUIRE(!cos_sin || (rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= dr && positions),
              "latent_rope_store: rotary_dim %d must be even and at most the rotated part %d, and needs positions", rotary_dim, dr);
  NHV_REQUIRE(pages == nullptr || (page_size > 0 && n_pages > 0 && slot_mapping && row >= rank + dr && weight),
              "latent_rope_store: the store needs pages whose rows hold the latent and the rotated part, a slot mapping and the norm's weight");
  auto on16 = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
  if (dr > 0 && dn % 8 == 0 && dr % 8 == 0 && rank % 8 == 0 && row % 8 == 0 && kv_stride % 8 == 0 && q_stride % 8 == 0 &&
      q_lat_stride % 8 == 0 && (!cos_sin || rotary_dim % (interleaved ? 8 : 16) == 0) && on16(kv) && on16(q) && on16(q_lat) &&
      on16(pages) && on16(weight) && on16(cos_sin)) {
    const int per_token = 1 + (H * (dr / 8) + 31) / 32;
    const int vec_blocks = (int)(((long)n_tokens * per_token + LS_WARPS - 1) / LS_WARPS);
#define LAUNCH(T)                                                                                                        \
  nhv_launch(latent_rope_store_vec_kernel<T>, vec_blocks, LS_WARPS * 32, 0, stream, (const T*)kv, kv_stride, (const T*)q, \
             q_stride, (T*)q_lat, q_lat_stride, (T*)pages, slot_mapping, positions, cos_sin, rotary_dim, max_position,   \
             n_tokens, per_token, H, dn, dr, rank, row, page_size * n_pages, eps, (const T*)weight, interleaved)
    if (dtype == NHV_F32) LAUNCH(float);
    else if (dtype == NHV_BF16) LAUNCH(__nv_bfloat16);
    else NHV_REQUIRE(false, "latent_rope_store: unknown dtype %d", dtype);
#undef LAUNCH
    NHV_CHECK_LAUNCH("latent_rope_store");
    return 0;
  }
  const long items = (long)n_tokens * (H + 1);
  const int blocks = (int)((items + LS_WARPS - 1) / LS_WARPS);
  const size_t smem = (size_t)LS_WARPS * (rank + dr) * sizeof(float);
#define LAUNCH(T)                                                                                                   \
  nhv_launch(latent_rope_store_kernel<T>, blocks, LS_WARPS * 32, smem, stream, (const T*)kv, kv_stride, (const T*)q, \
             q_stride, (T*)q_lat, q_lat_stride, (T*)pages, slot_mapping, positions, cos_sin, rotary_dim,            \
             max_position, n_tokens, H, dn, dr, rank, row, page_size, n_pages, eps, (const T*)weight, interleaved)
  if (dtype == NHV_F32) LAUNCH(float);
  else if (dtype == NHV_BF16) LAUNCH(__nv_bfloat16);
  else NHV_REQUIRE(false, "latent_rope_store: unknown dtype %d", dtype);
#undef LAUNCH
  NHV_CHECK_LAUNCH("latent_rope_store");
  return 0;
}
