// From a packed projection to queries and cache rows, for attention layers whose heads pass a short filter over time,
// have several maps (independent query / key pairs over one value head) or a temperature on the queries.
//
// qkv [T, (nq + nkv) * maps * dk (+ nkv * dv)]: q heads, then k heads, then (unless v_from_k) v heads; a head's maps
// lie one behind the other.  Per token and (head, map):
//   taps (optional, [K][(nq + nkv) * maps * dk], one row per tap, the newest token's tap last):
//            y = sum_j taps[j] * u(t - K + 1 + j), t within the request; inputs before this step's portion come from
//            the request's state (its last K - 1 inputs, fp32, [slot][K - 1][channels], oldest first), zeros before
//            the request's start
//   v_from_k: the value of a KV head is its key head after the filter (maps == 1, dv == dk)
//   norm:    x / sqrt(mean(x^2) + eps) over the map's dk elements, times a weight [dk] of its kind (q or k)
//   rotation of the first rotary_dim elements (element i with i + rotary_dim / 2, angles from the table)
//   queries: times 1 + temp_coef * ln(floor((position + 1) / temp_every) + 1)   (temp_every 0: no temperature)
// and then
//   query (head h, map m) -> q_out[t, (h * maps + m) * q_head + m * dk ...], zeros elsewhere in its q_head elements,
//   key (head g, map m)   -> the token's K row of head g at m * dk,
// so that the product of a padded query with a whole key row is the score of its own map, and a KV head's maps are
// query heads of one group over one key / value row (any grouped-query kernel serves them).
// Everything is computed in fp32 and rounded once.  Rows of the cache: [page][K|V][kv_head][slot][row]; what a head leaves
// of a row is cleared.  slot_mapping[t] < 0: nothing is stored.
//
// The main kernel reads the old state of every request; a request that brings one token has its state moved on by the
// threads that read it, the others by a second launch (portions).
#include <math.h>

#include "nhv_common.cuh"
#include "nhv_vec8.cuh"

// Measured on B200 (4,096 tokens, 64 maps of 64 over 8 KV heads): what counts is how many warps an SM holds; more units or
// tokens per thread cost registers and lose (blocks of 256 with 3 units a thread: 94 us, these: 61 us).
constexpr int HS_THREADS = 128;
constexpr int HS_BLOCKS = 6;             // on an SM at least
constexpr int HS_BATCH = 2;              // units whose elements a thread asks for at once (no filter)
constexpr int HS_TOKENS = 2;             // tokens of a block in long steps (filters)
constexpr int HS_TAPS = 4;               // filters of up to so many taps run eight elements a lane
constexpr int HS_WARPS = 4;              // of the general kernel

template <typename T>
struct HeadsStore {
  const T* qkv;
  T* q_out;
  T* kv_pages;
  const T* q_weight;
  const T* k_weight;
  const T* taps;
  float* state;
  const int *slot_mapping, *positions, *cu_q, *q_start, *slots;
  const float* cos_sin;
  long state_stride;
  int qkv_stride, q_out_stride, q_head, rotary_dim, max_position, n_tokens, n_seqs, nq, nkv, maps, dk, dv, row, page_size,
      n_pages, K, v_from_k, units, temp_every, one_each;
  float eps, temp_coef;
};

// What a unit (head and map of a token) is and where its results go.
template <typename T>
struct HeadsUnit {
  int kind, map;                         // kind: 0 query, 1 key, 2 value
  int col;                               // its first column of qkv
  T* dst;                                // its padded query head, or its row of the cache (null: not stored)
  T* dst_v;                              // v_from_k: the value row
};

// A token's facts, the same for all its units.
struct HeadsToken {
  int pos;
  long row;                              // element offset of the token's K row of head 0 in the pages, or -1
  // for the filter: how many tokens of this portion lie before it, whether the portion is this token alone, and its
  // request's state (null: no slot; has_past: it holds inputs)
  int before, single, has_past;
  float* state;
};

template <typename T>
__device__ __forceinline__ HeadsToken heads_token(const HeadsStore<T>& p, int t) {
  HeadsToken k;
  k.pos = p.positions ? p.positions[t] : 0;
  k.row = -1;
  if (p.kv_pages) {
    const int slot = p.slot_mapping[t];
    if (slot >= 0 && slot < p.n_pages * p.page_size) {
      const int page = slot / p.page_size, off = slot - page * p.page_size;
      k.row = ((long)page * 2 * p.nkv * p.page_size + off) * p.row;
    }
  }
  k.before = k.single = k.has_past = 0;
  k.state = nullptr;
  if (p.taps) {
    int lo = t;                                             // a step of single tokens: one request each
    if (!p.one_each) {
      lo = 0;
      int hi = p.n_seqs - 1;
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (p.cu_q[mid] <= t) lo = mid; else hi = mid - 1;
      }
    }
    const int first = p.cu_q[lo], slot = p.slots[lo];
    k.before = t - first;
    k.single = p.cu_q[lo + 1] - first == 1;
    k.has_past = slot >= 0 && p.q_start[lo] > 0;
    if (slot >= 0) k.state = p.state + (size_t)slot * p.state_stride;
  }
  return k;
}

template <typename T>
__device__ __forceinline__ HeadsUnit<T> heads_unit(const HeadsStore<T>& p, int t, const HeadsToken& k, int x) {
  HeadsUnit<T> u;
  const int nqm = p.nq * p.maps, nkm = p.nkv * p.maps;
  auto head_of = [&](int i) { return p.maps == 1 ? i : p.maps == 2 ? i >> 1 : i / p.maps; };
  u.dst_v = nullptr;
  if (x < nqm) {
    u.kind = 0;
    u.map = x - head_of(x) * p.maps;
    u.col = x * p.dk;
    u.dst = p.q_out + (size_t)t * p.q_out_stride + (size_t)x * p.q_head;
    return u;
  }
  const int y = x - nqm;
  u.kind = y < nkm ? 1 : 2;
  const int g = u.kind == 1 ? head_of(y) : y - nkm;
  u.map = u.kind == 1 ? y - g * p.maps : 0;
  u.col = u.kind == 1 ? x * p.dk : (nqm + nkm) * p.dk + g * p.dv;
  u.dst = nullptr;
  if (k.row >= 0) {
    const size_t plane = (size_t)p.nkv * p.page_size * p.row;
    T* k_row = p.kv_pages + k.row + (size_t)g * p.page_size * p.row;
    u.dst = u.kind == 1 ? k_row : k_row + plane;
    if (p.v_from_k) u.dst_v = k_row + plane;
  }
  return u;
}

template <typename T>
__device__ __forceinline__ float heads_temperature(const HeadsStore<T>& p, int pos) {
  return p.temp_every > 0 ? 1.0f + p.temp_coef * logf((float)((pos + 1) / p.temp_every) + 1.0f) : 1.0f;
}

template <typename T>
__device__ __forceinline__ const float* heads_angles(const HeadsStore<T>& p, int pos) {
  if (!p.cos_sin) return nullptr;
  pos = pos < 0 ? 0 : (pos >= p.max_position ? p.max_position - 1 : pos);
  return p.cos_sin + (size_t)pos * p.rotary_dim;
}

// Eight elements as they lie in memory (so that many can be on their way in few registers), and as floats.
template <typename T>
struct Raw8 { uint4 w[sizeof(T) / 2]; };
template <typename T>
__device__ __forceinline__ void raw_load(Raw8<T>& r, const T* src) {
#pragma unroll
  for (int i = 0; i < (int)(sizeof(T) / 2); ++i) r.w[i] = reinterpret_cast<const uint4*>(src)[i];
}
template <typename T>
__device__ __forceinline__ void raw_get(float (&v)[8], const Raw8<T>& r) { nhv_load8(v, reinterpret_cast<const T*>(r.w)); }

// Norm, rotation, temperature and the store of one unit's chunk of eight; all lanes of a warp come here together.
// mine: this lane holds elements of a query or key; co / si: its cosines and sines (turns: its elements rotate).
struct HeadsLane {
  int c, partner, i0;
  bool first, turns;
};
template <typename T, int L>
__device__ __forceinline__ void heads_finish(const HeadsStore<T>& p, float (&v)[8], const HeadsUnit<T>& u, bool live, bool mine,
                                             const HeadsLane& lane, const float (&hw)[8], bool rotate, const float (&co)[8],
                                             const float (&si)[8], float temp) {
  const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  const int CH = p.dk / 8, c = lane.c;
  if (p.eps >= 0.f) {
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float r = 1.0f / sqrtf(ss / (float)p.dk + p.eps);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = v[e] * r * hw[e];
  }
  if (rotate) {
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float other = __shfl_sync(0xffffffffu, v[e], lane.partner, L);
      if (mine && lane.turns) v[e] = lane.first ? v[e] * co[e] - other * si[e] : v[e] * co[e] + other * si[e];
    }
  }
  if (!live || u.kind == 2 || !u.dst) return;
  const int from = u.map * CH;
  if (mine) {
    if (u.kind == 0) {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= temp;
    }
    nhv_store8(u.dst + (from + c) * 8, v);
  }
  if (u.kind == 0) {
    for (int y = c; y < p.q_head / 8; y += L)
      if (y < from || y >= from + CH) nhv_store8(u.dst + y * 8, zero);
  } else if (u.map == p.maps - 1) {
    for (int y = p.maps * CH + c; y < p.row / 8; y += L) nhv_store8(u.dst + y * 8, zero);
  }
}

template <typename T, int L>
__device__ __forceinline__ HeadsLane heads_lane(const HeadsStore<T>& p) {
  HeadsLane l;
  l.c = threadIdx.x & (L - 1);
  const int hc = (p.rotary_dim >> 1) / 8;
  l.first = l.c < hc;
  l.turns = l.c < 2 * hc;
  l.partner = l.turns ? (l.first ? l.c + hc : l.c - hc) : l.c;
  l.i0 = (l.first ? l.c : l.c - hc) * 8;
  return l;
}

// L lanes per unit, eight consecutive elements a lane: sizes in steps of 8, halves of the rotation too.

// Without a filter: a block per token (gridDim.x) and its units, or a share of them (gridDim.y); HS_BATCH of a thread's units
// are read before the first is worked on, its angles once for all of them.
template <typename T, int L>
__global__ void __launch_bounds__(HS_THREADS, HS_BLOCKS) heads_store_vec_kernel(const HeadsStore<T> p) {
  pdl_prologue();
  constexpr int GROUPS = HS_THREADS / L;
  const int t = blockIdx.x;
  const HeadsToken k = heads_token(p, t);
  const float temp = heads_temperature(p, k.pos);
  const HeadsLane lane = heads_lane<T, L>(p);
  const int c = lane.c, CH = p.dk / 8, step = gridDim.y * GROUPS;
  const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  const T* row = p.qkv + (size_t)t * p.qkv_stride;
  const float* cs = heads_angles(p, k.pos);
  float co[8], si[8];
  if (cs && lane.turns && c < CH) {
    nhv_load8(co, cs + lane.i0);
    nhv_load8(si, cs + (p.rotary_dim >> 1) + lane.i0);
  }
  for (int base = blockIdx.y * GROUPS; base < p.units; base += HS_BATCH * step) {
    Raw8<T> raw[HS_BATCH];
#pragma unroll
    for (int b = 0; b < HS_BATCH; ++b) {
      const int x = base + b * step + threadIdx.x / L;
      if (x < (p.nq + p.nkv) * p.maps && x < p.units && c < CH) raw_load(raw[b], row + (size_t)x * p.dk + c * 8);
    }
#pragma unroll
    for (int b = 0; b < HS_BATCH; ++b) {
      if (base + b * step >= p.units) break;                // the same for the whole block
      const int x = base + b * step + threadIdx.x / L;
      const bool live = x < p.units;
      const HeadsUnit<T> u = heads_unit(p, t, k, live ? x : 0);
      const bool mine = live && u.kind != 2 && c < CH;
      float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      float hw[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
      if (mine) {
        raw_get(v, raw[b]);
        const T* w = u.kind == 0 ? p.q_weight : p.k_weight;
        if (w) nhv_load8(hw, w + c * 8);
        if (u.dst_v) nhv_store8(u.dst_v + c * 8, v);
      }
      if (live && u.kind == 1 && u.dst_v)
        for (int y = CH + c; y < p.row / 8; y += L) nhv_store8(u.dst_v + y * 8, zero);
      if (live && u.kind == 2 && u.dst)                     // a value head as it is, the rest of its row cleared
        for (int y = c; y < p.row / 8; y += L) {
          float val[8];
          if (y < p.dv / 8) {
            nhv_load8(val, row + u.col + y * 8);
            nhv_store8(u.dst + y * 8, val);
          } else {
            nhv_store8(u.dst + y * 8, zero);
          }
        }
      heads_finish<T, L>(p, v, u, live, mine, lane, hw, cs != nullptr, co, si, temp);
    }
  }
}

// With a filter of up to TAPS taps: a block takes NT neighbouring tokens (gridDim.x) and all their units, or a share of them
// (gridDim.y); a unit's taps are read once for its tokens, and the inputs of all of them (and of the TAPS - 1 tokens before)
// before the first is worked on.
template <typename T, int L, int TAPS, int NT>
__global__ void __launch_bounds__(HS_THREADS, 4) heads_filter_vec_kernel(const HeadsStore<T> p) {
  __shared__ HeadsToken facts[NT];
  __shared__ float temps[NT];
  pdl_prologue();
  const int t0 = blockIdx.x * NT, n = min(NT, p.n_tokens - t0);
  if (threadIdx.x < n) {
    facts[threadIdx.x] = heads_token(p, t0 + threadIdx.x);
    temps[threadIdx.x] = heads_temperature(p, facts[threadIdx.x].pos);
  }
  __syncthreads();
  constexpr int GROUPS = HS_THREADS / L, X = TAPS - 1;
  const HeadsLane lane = heads_lane<T, L>(p);
  const int c = lane.c, CH = p.dk / 8, C = (p.nq + p.nkv) * p.maps * p.dk, skip = TAPS - p.K;
  const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  for (int base = blockIdx.y * GROUPS; base < p.units; base += gridDim.y * GROUPS) {
    const int x = base + threadIdx.x / L;
    const bool live = x < p.units;                          // a warp's lanes stay together for the exchanges below
    const int kind = x < p.nq * p.maps ? 0 : x < (p.nq + p.nkv) * p.maps ? 1 : 2;
    const bool mine = live && kind != 2 && c < CH;
    const int at = x * p.dk + c * 8;                        // the first of this lane's channels (queries and keys)
    Raw8<T> in[NT + X], tap[TAPS];                          // in[r]: the input of token t0 - X + r; taps right-aligned
    float hw[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
    if (mine) {
#pragma unroll
      for (int r = 0; r < NT + X; ++r) {
        const int t = t0 - X + r;
        if (r >= skip && t >= 0 && t < t0 + n) raw_load(in[r], p.qkv + (size_t)t * p.qkv_stride + at);
      }
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
        if (j >= skip) raw_load(tap[j], p.taps + (size_t)(j - skip) * C + at);
      const T* w = kind == 0 ? p.q_weight : p.k_weight;
      if (w) nhv_load8(hw, w + c * 8);
    }
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      if (i >= n) break;                                    // the same for the whole block
      const HeadsToken& k = facts[i];
      const HeadsUnit<T> u = heads_unit(p, t0 + i, k, live ? x : 0);
      float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (mine) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          const int back = X - j;
          if (j < skip) continue;
          float o[8], w[8];
          if (k.before >= back) raw_get(o, in[i + j]);
          else if (k.has_past) nhv_load8(o, k.state + (size_t)(p.K - 1 + k.before - back) * C + at);
          else continue;
          raw_get(w, tap[j]);
#pragma unroll
          for (int e = 0; e < 8; ++e) v[e] = fmaf(w[e], o[e], v[e]);
        }
        if (k.single && k.state && p.K > 1) {               // the only reader of these channels of this state
          float o[8];
          for (int j = 0; j + 2 < p.K; ++j) {
            if (k.has_past) {
              nhv_load8(o, k.state + (size_t)(j + 1) * C + at);
              nhv_store8(k.state + (size_t)j * C + at, o);
            } else {
              nhv_store8(k.state + (size_t)j * C + at, zero);
            }
          }
          raw_get(o, in[i + X]);
          nhv_store8(k.state + (size_t)(p.K - 2) * C + at, o);
        }
        if (u.dst_v) nhv_store8(u.dst_v + c * 8, v);
      }
      if (live && kind == 1 && u.dst_v)
        for (int y = CH + c; y < p.row / 8; y += L) nhv_store8(u.dst_v + y * 8, zero);
      if (live && kind == 2 && u.dst)
        for (int y = c; y < p.row / 8; y += L) {
          float val[8];
          if (y < p.dv / 8) {
            nhv_load8(val, p.qkv + (size_t)(t0 + i) * p.qkv_stride + u.col + y * 8);
            nhv_store8(u.dst + y * 8, val);
          } else {
            nhv_store8(u.dst + y * 8, zero);
          }
        }
      const float* cs = heads_angles(p, k.pos);
      float co[8], si[8];
      if (cs && mine && lane.turns) {
        nhv_load8(co, cs + lane.i0);
        nhv_load8(si, cs + (p.rotary_dim >> 1) + lane.i0);
      }
      heads_finish<T, L>(p, v, u, live, mine, lane, hw, cs != nullptr, co, si, temps[i]);
    }
  }
}

// One warp per unit, element by element, any size.
template <typename T>
__global__ void __launch_bounds__(HS_WARPS * 32) heads_store_kernel(const HeadsStore<T> p) {
  extern __shared__ float smem[];
  pdl_prologue();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long item = (long)blockIdx.x * HS_WARPS + warp;
  if (item >= (long)p.n_tokens * p.units) return;
  const int t = (int)(item / p.units);
  const HeadsToken k = heads_token(p, t);
  const HeadsUnit<T> u = heads_unit(p, t, k, (int)(item - (long)t * p.units));
  const T* src = p.qkv + (size_t)t * p.qkv_stride + u.col;
  if (u.kind == 2) {
    if (u.dst)
      for (int c = lane; c < p.row; c += 32) u.dst[c] = c < p.dv ? src[c] : from_f32<T>(0.f);
    return;
  }
  float* v = smem + (size_t)warp * p.dk;
  const int d = p.dk;
  if (p.taps) {
    const int C = (p.nq + p.nkv) * p.maps * d;
    for (int c = lane; c < d; c += 32) {
      const int at = u.col + c;
      float acc = 0.f;
      for (int j = 0; j < p.K; ++j) {
        const int back = p.K - 1 - j;
        float x;
        if (k.before >= back) x = to_f32<T>(*(src + c - (size_t)back * p.qkv_stride));
        else if (k.has_past) x = k.state[(size_t)(p.K - 1 + k.before - back) * C + at];
        else continue;
        acc = fmaf(to_f32<T>(p.taps[(size_t)j * C + at]), x, acc);
      }
      v[c] = acc;
      if (k.single && k.state && p.K > 1) {
        for (int j = 0; j + 2 < p.K; ++j)
          k.state[(size_t)j * C + at] = k.has_past ? k.state[(size_t)(j + 1) * C + at] : 0.f;
        k.state[(size_t)(p.K - 2) * C + at] = to_f32<T>(src[c]);
      }
    }
  } else {
    for (int c = lane; c < d; c += 32) v[c] = to_f32<T>(src[c]);
  }
  if (u.dst_v)
    for (int c = lane; c < p.row; c += 32) u.dst_v[c] = from_f32<T>(c < d ? v[c] : 0.f);
  if (p.eps >= 0.f) {
    float ss = 0.f;
    for (int c = lane; c < d; c += 32) ss = fmaf(v[c], v[c], ss);
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)d + p.eps);
    const T* hw = u.kind == 0 ? p.q_weight : p.k_weight;
    for (int c = lane; c < d; c += 32) v[c] = v[c] * r * (hw ? to_f32<T>(hw[c]) : 1.0f);
  }
  __syncwarp();
  if (!u.dst) return;
  const float* cs = heads_angles(p, k.pos);
  const int half = p.rotary_dim >> 1, from = u.map * d;
  const float f = u.kind == 0 ? heads_temperature(p, k.pos) : 1.0f;
  for (int c = lane; c < d; c += 32) {
    float y = v[c];
    if (cs && c < half) y = v[c] * cs[c] - v[c + half] * cs[half + c];
    else if (cs && c < p.rotary_dim) y = v[c] * cs[c - half] + v[c - half] * cs[c];
    u.dst[from + c] = from_f32<T>(y * f);
  }
  if (u.kind == 0) {
    for (int c = lane; c < p.q_head; c += 32)
      if (c < from || c >= from + d) u.dst[c] = from_f32<T>(0.f);
  } else if (u.map == p.maps - 1) {
    for (int c = p.maps * d + lane; c < p.row; c += 32) u.dst[c] = from_f32<T>(0.f);
  }
}

// The state of the requests that bring more than one token, moved on (behind the main kernel, which reads it).
template <typename T>
__global__ void heads_state_kernel(const T* __restrict__ x, int x_stride, float* __restrict__ state, long state_stride,
                                   const int* __restrict__ cu_q, const int* __restrict__ q_start,
                                   const int* __restrict__ slots, int C, int K) {
  pdl_prologue();
  const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  const int slot = slots[s];
  const int first = cu_q[s], n = cu_q[s + 1] - first;
  if (c >= C || slot < 0 || n < 2) return;
  const bool has_past = q_start[s] > 0;
  float* st = state + (size_t)slot * state_stride;
  for (int j = 0; j + 1 < K; ++j) {                         // ascending: an entry is read before it is written over
    const int rel = n - (K - 1) + j;
    st[(size_t)j * C + c] = rel >= 0 ? to_f32<T>(x[(size_t)(first + rel) * x_stride + c])
                                     : (has_past ? st[(size_t)(K - 1 + rel) * C + c] : 0.f);
  }
}

template <typename T>
static int heads_store_launch(HeadsStore<T> p, bool portions, cudaStream_t stream) {
  const long items = (long)p.n_tokens * p.units;
  const int half = p.rotary_dim >> 1;
  auto ok16 = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
  const bool vec = p.dk % 8 == 0 && p.dk <= 256 && p.q_head % 8 == 0 && p.qkv_stride % 8 == 0 && p.q_out_stride % 8 == 0 &&
                   (!p.cos_sin || (half % 8 == 0 && ok16(p.cos_sin))) &&
                   (!p.kv_pages || (p.row % 8 == 0 && (p.v_from_k || p.dv % 8 == 0))) &&
                   (!p.taps || (p.K <= HS_TAPS && (p.K < 2 || p.state_stride % 4 == 0))) && ok16(p.qkv) && ok16(p.q_out) && ok16(p.kv_pages) &&
                   ok16(p.q_weight) && ok16(p.k_weight) && ok16(p.taps) && ok16(p.state);
  if (vec) {
    const int ch = p.dk / 8, L = ch <= 4 ? 4 : ch <= 8 ? 8 : ch <= 16 ? 16 : 32;
    // short steps: a block per share of a token's units; long steps: a block for all of them, with a filter for several tokens
    const int passes = (p.units + HS_THREADS / L - 1) / (HS_THREADS / L);
    const bool many = p.n_tokens >= 2048;
#define GO(L)                                                                                                        \
  do {                                                                                                               \
    if (!p.taps)                                                                                                     \
      nhv_launch(heads_store_vec_kernel<T, L>, dim3(p.n_tokens, p.n_tokens >= 592 ? 1 : passes), HS_THREADS, 0, stream, p); \
    else if (many)                                                                                                   \
      nhv_launch(heads_filter_vec_kernel<T, L, HS_TAPS, HS_TOKENS>, dim3((p.n_tokens + HS_TOKENS - 1) / HS_TOKENS),  \
                 HS_THREADS, 0, stream, p);                                                                          \
    else                                                                                                             \
      nhv_launch(heads_filter_vec_kernel<T, L, HS_TAPS, 1>, dim3(p.n_tokens, p.n_tokens >= 592 ? 1 : passes), HS_THREADS, 0, \
                 stream, p);                                                                                         \
  } while (0)
    if (L == 4) GO(4);
    else if (L == 8) GO(8);
    else if (L == 16) GO(16);
    else GO(32);
#undef GO
  } else {
    const size_t smem = (size_t)HS_WARPS * p.dk * sizeof(float);
    nhv_launch(heads_store_kernel<T>, (unsigned)((items + HS_WARPS - 1) / HS_WARPS), HS_WARPS * 32, smem, stream, p);
  }
  NHV_CHECK_LAUNCH("heads_store");
  if (p.taps && p.K > 1 && portions) {
    const int C = (p.nq + p.nkv) * p.maps * p.dk;
    nhv_launch(heads_state_kernel<T>, dim3(p.n_seqs, (C + 127) / 128), 128, 0, stream, p.qkv, p.qkv_stride, p.state,
               p.state_stride, p.cu_q, p.q_start, p.slots, C, p.K);
    NHV_CHECK_LAUNCH("heads_store (state)");
  }
  return 0;
}

// portions != 0: some request of the step brings more than one token; one_each != 0: every request brings exactly one (so
// that token t is request t's).
NHV_API int nhv_heads_store(int dtype, const void* qkv, int qkv_stride, void* q_out, int q_out_stride, int q_head,
                            void* kv_pages, const int* slot_mapping, const int* positions, const float* cos_sin,
                            int rotary_dim, int max_position, int n_tokens, int nq, int nkv, int maps, int dk, int dv,
                            int row, int page_size, int n_pages, float eps, const void* q_weight, const void* k_weight,
                            int v_from_k, float temp_coef, int temp_every, const void* taps, int K, float* state,
                            long state_stride, const int* cu_q, const int* q_start, const int* slots, int n_seqs,
                            int portions, int one_each, cudaStream_t stream) {
  if (n_tokens == 0 || n_seqs == 0) return 0;
  NHV_REQUIRE(n_tokens > 0 && nq > 0 && nkv >= 0 && maps > 0 && dk > 0 && dv > 0, "heads_store: bad sizes");
  NHV_REQUIRE(dk <= 2048, "heads_store: a head of %d elements is beyond the supported 2048", dk);
  NHV_REQUIRE(q_head >= maps * dk, "heads_store: a padded query head of %d elements does not hold %d maps of %d", q_head, maps, dk);
  NHV_REQUIRE(!cos_sin || (positions && rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= dk && max_position > 0),
              "heads_store: rotary_dim %d must be even and at most the head size %d", rotary_dim, dk);
  NHV_REQUIRE(temp_every >= 0 && (temp_every == 0 || positions), "heads_store: a temperature needs positions");
  NHV_REQUIRE(!kv_pages || (page_size > 0 && n_pages > 0 && slot_mapping && nkv > 0 && row >= maps * dk && row >= dv),
              "heads_store: a key/value store needs pages whose rows hold a head, and a slot mapping");
  NHV_REQUIRE(!v_from_k || (dv == dk && maps == 1), "heads_store: values taken from the keys have the keys' size and one map");
  NHV_REQUIRE(!taps || (K >= 1 && kv_pages && cu_q && q_start && slots), "heads_store: a filter over time needs keys of the layer's own and the step's requests");
  NHV_REQUIRE(!taps || K == 1 || (state && state_stride >= (long)(K - 1) * (nq + nkv) * maps * dk),
              "heads_store: the state holds fewer than (taps - 1) * channels floats");
  const int units = kv_pages ? (nq + nkv) * maps + (v_from_k ? 0 : nkv) : nq * maps;
#define GO(T)                                                                                                        \
  return heads_store_launch<T>(                                                                                      \
      HeadsStore<T>{(const T*)qkv, (T*)q_out, (T*)kv_pages, (const T*)q_weight, (const T*)k_weight, (const T*)taps,  \
                    state, slot_mapping, positions, cu_q, q_start, slots, cos_sin, state_stride, qkv_stride,         \
                    q_out_stride, q_head, cos_sin ? rotary_dim : 0, max_position, n_tokens, n_seqs, nq, nkv, maps,   \
                    dk, dv, row, page_size, n_pages, K, v_from_k, units, temp_every, one_each, eps, temp_coef},      \
      portions != 0, stream)
  if (dtype == NHV_F32) GO(float);
  if (dtype == NHV_BF16) GO(__nv_bfloat16);
#undef GO
  NHV_REQUIRE(false, "heads_store: unknown dtype %d", dtype);
  return 1;
}
