// Queries and keys normed over their whole projection (all heads of a kind together), optionally rotated, and the
// key / value store, with values that may be mixed with the values of an earlier layer.
//
// One block per token (its row is read once for the sums and once more, from the caches, for what is stored) of the packed projection output qkv [T, nq*dk + nkv*dk + nkv*dv]:
//   q row [nq*dk]: x / sqrt(mean(x^2) + eps) * q_weight [nq*dk], then the rotation per head -> q_out [T, nq, q_head],
//                  q_head >= dk, zeros behind a head's dk elements
//   k row:         the same with k_weight [nkv*dk] -> the token's slot of the K pages
//   v row:         (1 - share) v + share v_first where v_first is given (the same token's row of another layer's values,
//                  share one float in device memory), else v -> the token's slot of the V pages
// eps < 0 leaves the norm out.  All of it in fp32, rounded once.  Rotation: the first rotary_dim elements of a head,
// element i with i + rotary_dim / 2, or (interleaved) 2i with 2i + 1; angles from a table of cosines, then sines.
// Cache pages of one layer: [page][K|V][kv_head][slot_in_page][row], row >= max(dk, dv); the elements of a row beyond
// the head's size are cleared.  slot_mapping[t] = page * page_size + slot_in_page, or -1 for "do not store".
#include "nhv_common.cuh"
#include "nhv_vec8.cuh"

template <typename T, int V> struct RowPiece;
template <typename T> struct RowPiece<T, 8> {
  static __device__ __forceinline__ void load(float (&o)[8], const T* p) { nhv_load8(o, p); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[8]) { nhv_store8(p, v); }
};
template <typename T> struct RowPiece<T, 1> {
  static __device__ __forceinline__ void load(float (&o)[1], const T* p) { o[0] = to_f32<T>(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_f32<T>(v[0]); }
};

template <typename T, int V, bool ROT>
__global__ void __launch_bounds__(512, V == 8 && !ROT ? 3 : 1) row_norm_store_kernel(const T* __restrict__ qkv, int qkv_stride, T* __restrict__ q_out, int q_out_stride,
                                      int q_head, T* __restrict__ kv_pages, const int* __restrict__ slot_mapping,
                                      const int* __restrict__ positions, const float* __restrict__ cos_sin, int rotary_dim,
                                      int max_position, int interleaved, int nq, int nkv, int dk, int dv, int row,
                                      int page_size, int n_pages, float eps, const T* __restrict__ q_weight,
                                      const T* __restrict__ k_weight, const T* __restrict__ v_first, int v_first_stride,
                                      const float* __restrict__ v_share) {
  __shared__ float2 red[33];
  pdl_prologue();
  const int t = blockIdx.x, nqd = nq * dk, nkd = nkv * dk;
  const T* src = qkv + (size_t)t * qkv_stride;
  int slot = -1;
  if (kv_pages) {
    slot = slot_mapping[t];
    if (slot >= n_pages * page_size) slot = -1;
  }
  float rq = 1.f, rk = 1.f;
  if (eps >= 0.f) {
    const int n_norm = slot >= 0 ? nqd + nkd : nqd;
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x * V; c < n_norm; c += blockDim.x * V) {
      float x[V];
      RowPiece<T, V>::load(x, src + c);
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < V; ++i) s = fmaf(x[i], x[i], s);
      if (c < nqd) sq += s; else sk += s;                    // V divides dk: a piece lies in one row
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    if (lane == 0) red[warp] = make_float2(sq, sk);
    __syncthreads();
    float2 both = lane < n_warps ? red[lane] : make_float2(0.f, 0.f);     // every warp sums the warps' sums for itself
    rq = 1.0f / sqrtf(warp_sum(both.x) / (float)nqd + eps);
    rk = 1.0f / sqrtf(warp_sum(both.y) / (float)nkd + eps);
  }
  const float* cs = nullptr;
  const int half = rotary_dim >> 1;
  if (ROT && cos_sin) {
    int pos = positions[t];
    pos = pos < 0 ? 0 : (pos >= max_position ? max_position - 1 : pos);
    cs = cos_sin + (size_t)pos * rotary_dim;                 // cos[0..half) then sin[0..half)
  }
  int page = 0, off = 0;
  if (slot >= 0) { page = slot / page_size; off = slot - page * page_size; }
  // pieces of V elements of every (padded) head: q heads of q_head, k and v heads of `row`
  const int qp = q_head / V, rp = row / V;
  const int n_q = nq * qp, n_kv = slot >= 0 ? nkv * rp : 0;
  for (int i = threadIdx.x; i < n_q + 2 * n_kv; i += blockDim.x) {
    const int kind = i < n_q ? 0 : (i < n_q + n_kv ? 1 : 2);
    const int e = kind == 0 ? i : i - n_q - (kind - 1) * n_kv;
    const int per = kind == 0 ? qp : rp;
    const int head = e / per, c0 = (e - head * per) * V;
    T* dst = kind == 0 ? q_out + (size_t)t * q_out_stride + (size_t)head * q_head + c0
                       : kv_pages + ((((size_t)page * 2 + (kind - 1)) * nkv + head) * page_size + off) * row + c0;
    float o[V];
#pragma unroll
    for (int k = 0; k < V; ++k) o[k] = 0.f;
    if (kind < 2) {
      if (c0 < dk) {
        const T* h = src + (kind == 0 ? 0 : nqd) + head * dk;
        const T* hw = eps >= 0.f ? (kind == 0 ? q_weight : k_weight) : nullptr;
        if (hw) hw += head * dk;
        const float r = kind == 0 ? rq : rk;
        auto normed = [&](int c) { return hw ? to_f32<T>(h[c]) * r * to_f32<T>(hw[c]) : to_f32<T>(h[c]) * r; };
        float x[V];
        RowPiece<T, V>::load(x, h + c0);
        float wv[V];
        if (hw) RowPiece<T, V>::load(wv, hw + c0);
#pragma unroll
        for (int k = 0; k < V; ++k) {
          const int c = c0 + k;
          float v = hw ? x[k] * r * wv[k] : x[k] * r;
          if (ROT && cs && c < rotary_dim) {
            if (interleaved) {
              const int a = c >> 1;
              v = (c & 1) ? v * cs[a] + normed(c - 1) * cs[half + a] : v * cs[a] - normed(c + 1) * cs[half + a];
            } else {
              v = c < half ? v * cs[c] - normed(c + half) * cs[half + c] : v * cs[c - half] + normed(c - half) * cs[c];
            }
          }
          o[k] = v;
        }
      }
    } else if (c0 < dv) {
      RowPiece<T, V>::load(o, src + nqd + nkd + head * dv + c0);
      if (v_first) {
        float f[V];
        RowPiece<T, V>::load(f, v_first + (size_t)t * v_first_stride + head * dv + c0);
        const float share = *v_share;
#pragma unroll
        for (int k = 0; k < V; ++k) o[k] = fmaf(share, f[k], (1.0f - share) * o[k]);
      }
    }
    RowPiece<T, V>::store(dst, o);
  }
}

NHV_API int nhv_row_norm_store(int dtype, const void* qkv, int qkv_stride, void* q_out, int q_out_stride, int q_head,
                               void* kv_pages, const int* slot_mapping, const int* positions, const float* cos_sin,
                               int rotary_dim, int max_position, int interleaved, int n_tokens, int nq, int nkv, int dk,
                               int dv, int row, int page_size, int n_pages, float eps, const void* q_weight,
                               const void* k_weight, const void* v_first, int v_first_stride, const float* v_share,
                               cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  NHV_REQUIRE(n_tokens > 0 && nq > 0 && nkv > 0 && dk > 0 && dv > 0 && q_head >= dk, "row_norm_store: bad sizes");
  NHV_REQUIRE(!cos_sin || (positions && rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= dk),
              "row_norm_store: rotary_dim %d must be even and at most the head size %d, and needs positions", rotary_dim, dk);
  NHV_REQUIRE(kv_pages == nullptr || (page_size > 0 && n_pages > 0 && slot_mapping && row >= dk && row >= dv),
              "row_norm_store: a key/value store needs pages whose rows hold a head, and a slot mapping");
  NHV_REQUIRE(!v_first || v_share, "row_norm_store: mixed values need their share");
  const int item = dtype == NHV_F32 ? 4 : 2;
  auto on8 = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
  const bool vec = dk % 8 == 0 && dv % 8 == 0 && q_head % 8 == 0 && row % 8 == 0 && (size_t)qkv_stride * item % 16 == 0 &&
                   (size_t)q_out_stride * item % 16 == 0 && (size_t)v_first_stride * item % 16 == 0 && on8(qkv) && on8(q_out) &&
                   on8(kv_pages) && on8(q_weight) && on8(k_weight) && on8(v_first);
  const int work = ((nq + nkv) * dk) / (vec ? 8 : 1);
  int threads = 64;
  while (threads < (n_tokens <= 148 ? 512 : 256) && threads < work) threads <<= 1;
#define GO2(T, V, R)                                                                                                    \
  do {                                                                                                                \
    nhv_launch(row_norm_store_kernel<T, V, R>, n_tokens, threads, 0, stream, (const T*)qkv, qkv_stride, (T*)q_out,    \
               q_out_stride, q_head, (T*)kv_pages, slot_mapping, positions, cos_sin, rotary_dim, max_position,        \
               interleaved, nq, nkv, dk, dv, row, page_size, n_pages, eps, (const T*)q_weight, (const T*)k_weight,    \
               (const T*)v_first, v_first_stride, v_share);                                                           \
  } while (0)
#define GO(T, V) do { if (cos_sin) GO2(T, V, true); else GO2(T, V, false); } while (0)
  if (dtype == NHV_F32) { if (vec) GO(float, 8); else GO(float, 1); }
  else if (dtype == NHV_BF16) { if (vec) GO(__nv_bfloat16, 8); else GO(__nv_bfloat16, 1); }
  else NHV_REQUIRE(false, "row_norm_store: unknown dtype %d", dtype);
#undef GO
#undef GO2
  NHV_CHECK_LAUNCH("row_norm_store");
  return 0;
}
