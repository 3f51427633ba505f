// Operators of decoder layers whose norm keeps no statistics and whose attention comes in several forms:
//   * the embedding with a hashed token-pair table (the previous token of a request is part of its state),
//   * the fp32 residual update fused with a tanh norm  tanh(alpha x) w + b  (plus what a pass of a looped
//     block adds in front of its first layer),
//   * rotary positions over strided "segments" (q, k, v of a merged projection, or the rotated slice of a
//     latent attention's queries and keys), in the paired or the half-split layout, with the biases of the
//     projections added first, an RMS norm per head or over all heads of a row where a segment asks for one,
//     and the cache write fused,
//   * the fp32 residual update of layers that norm a sublayer's OUTPUT,
//   * the step between an attention and its output projection: an elementwise sigmoid gate, optionally on
//     the unit-RMS difference of two attention maps.
// Everything is computed in fp32; 16-bit only at the loads and stores.
#include "common.cuh"
#include "ptx.cuh"

namespace spd {

constexpr int kMixThreads = 256;

__device__ __forceinline__ float mix_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// the request that owns row t of a ragged extend batch (empty entries share their successor's start)
__device__ __forceinline__ int row_request(const int32_t* __restrict__ extend_start_loc,
                                           const int32_t* __restrict__ extend_lens, int batch, int64_t t) {
  int lo = 0, hi = batch - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if ((int64_t)extend_start_loc[mid] <= t) lo = mid; else hi = mid - 1;
  }
  while (lo > 0 && extend_lens[lo] == 0) --lo;
  return lo;
}

// x[t] = table[id] * scale + pair[(prev * mul_prev + id * mul_cur) mod buckets]   (pair row `buckets` for a
// request's first token).  prev is the row before in the batch, or — for the first row of a request's portion
// — prev_state[slot]; the CTA of that first row also leaves the portion's last token in prev_state[slot].
template <typename T>
__global__ void __launch_bounds__(kMixThreads)
embed_pair_kernel(float* __restrict__ x, const T* __restrict__ table, const T* __restrict__ pair,
                  const int64_t* __restrict__ idx, int32_t* __restrict__ prev_state,
                  const int64_t* __restrict__ req_pool_indices, const int64_t* __restrict__ seq_lens,
                  const int64_t* __restrict__ out_cache_loc, const int32_t* __restrict__ prefix_lens,
                  const int32_t* __restrict__ extend_lens, const int32_t* __restrict__ extend_start_loc, int batch,
                  int64_t dim, int64_t table_rows, float scale, int64_t buckets, int64_t mul_prev, int64_t mul_cur) {
  griddep_wait();
  griddep_launch_dependents();
  const int64_t t = blockIdx.x;
  __shared__ int64_t s_prev;
  if (threadIdx.x == 0) {
    int64_t prev = -1;  // -1: the request's first token
    if (pair != nullptr) {
      if (seq_lens != nullptr) {
        const int64_t slot = req_pool_indices[t];
        if (seq_lens[t] > 1) prev = prev_state[slot];
        if (out_cache_loc == nullptr || out_cache_loc[t] != 0) prev_state[slot] = (int32_t)idx[t];  // not a padded row
      } else {
        const int r = row_request(extend_start_loc, extend_lens, batch, t);
        const int64_t first = extend_start_loc[r];
        if (t > first) {
          prev = idx[t - 1];
        } else {
          const int64_t slot = req_pool_indices[r];
          if (prefix_lens[r] > 0) prev = prev_state[slot];
          prev_state[slot] = (int32_t)idx[first + extend_lens[r] - 1];
        }
      }
    }
    s_prev = prev;
  }
  __syncthreads();
  int64_t id = idx[t];
  id = id < 0 ? 0 : (id >= table_rows ? table_rows - 1 : id);
  int64_t prow = buckets;
  if (s_prev >= 0) prow = (s_prev * mul_prev + id * mul_cur) % buckets;
  for (int64_t i = threadIdx.x; i < dim; i += kMixThreads) {
    float v = to_f32<T>(table[id * dim + i]) * scale;
    if (pair != nullptr) v += to_f32<T>(pair[prow * dim + i]);
    x[t * dim + i] = v;
  }
}

// x[row] += a[row] + x0[row] + vec (each optional; written back when any is given), then
// out[r] = tanh(alpha x[row]) w + b with row = rows ? rows[r] : r.
template <typename T>
__global__ void __launch_bounds__(kMixThreads)
residual_tanh_norm_kernel(T* __restrict__ out, float* __restrict__ x, const T* __restrict__ a,
                          const float* __restrict__ x0, const float* __restrict__ vec, const T* __restrict__ w,
                          const T* __restrict__ b, const int64_t* __restrict__ rows, int64_t dim, float alpha) {
  griddep_wait();
  griddep_launch_dependents();
  const int64_t r = blockIdx.x;
  const int64_t row = rows != nullptr ? rows[r] : r;
  float* xr = x + row * dim;
  const bool update = a != nullptr || x0 != nullptr || vec != nullptr;
  for (int64_t i = threadIdx.x; i < dim; i += kMixThreads) {
    float v = xr[i];
    if (update) {
      if (a != nullptr) v += to_f32<T>(a[row * dim + i]);
      if (x0 != nullptr) v += x0[row * dim + i];
      if (vec != nullptr) v += vec[i];
      xr[i] = v;
    }
    if (out != nullptr) out[r * dim + i] = from_f32<T>(tanhf(alpha * v) * to_f32<T>(w[i]) + to_f32<T>(b[i]));
  }
}

struct RotarySegment {
  const void* src;    // [tokens, ...]: head h of token t starts at src + t * src_row + h * src_head
  const float* bias;  // [heads * head_dim] or null, added before the rotation
  void* dst;          // head h of token t goes to dst + (to_pool ? loc[t] : t) * dst_row + h * dst_head
  int64_t src_row, dst_row;
  int32_t heads, head_dim, rot, src_head, dst_head, to_pool;
  const float* norm_w;  // [head_dim] (norm 2: [heads * head_dim]) or null (plain unit RMS); read when norm != 0
  int32_t norm;         // RMS norm after the bias and before the rotation: 1 over the head's channels, 2 over all heads
  float norm_eps;
};
struct RotarySegments {
  RotarySegment seg[4];
  int n;
};

// The first `rot` channels of every head turn by position * f_i (cos_sin [positions, rot_max] = cos || sin of
// rot_max / 2 angles each; a segment uses the first rot / 2 of both): paired layout, channel 2 i with 2 i + 1;
// half-split layout, channel i with i + rot / 2.  Channels >= rot are copied (plus bias).
template <typename T>
__global__ void __launch_bounds__(128)
rotary_segments_kernel(RotarySegments segs, const int64_t* __restrict__ positions, const int64_t* __restrict__ loc,
                       const float* __restrict__ cos_sin, int rot_max, int64_t max_positions, int paired) {
  griddep_wait();
  griddep_launch_dependents();
  const int64_t t = blockIdx.x;
  int64_t p = positions[t];
  p = p < 0 ? 0 : (p < max_positions ? p : max_positions - 1);
  const float* cs = cos_sin != nullptr ? cos_sin + p * rot_max : nullptr;
  const int half_max = rot_max >> 1;
  const int64_t slot = loc != nullptr ? loc[t] : 0;
  for (int sidx = 0; sidx < segs.n; ++sidx) {
    const RotarySegment& sg = segs.seg[sidx];
    const T* src = reinterpret_cast<const T*>(sg.src) + t * sg.src_row;
    T* dst = reinterpret_cast<T*>(sg.dst) + (sg.to_pool ? slot : t) * sg.dst_row;
    const int half = sg.rot >> 1;
    const int n = sg.heads * sg.head_dim;
    for (int idx = threadIdx.x; idx < n; idx += 128) {
      const int h = idx / sg.head_dim, d = idx - h * sg.head_dim;
      const float x = to_f32<T>(src[h * sg.src_head + d]) + (sg.bias != nullptr ? sg.bias[idx] : 0.f);
      float y = x;
      if (d < sg.rot) {
        int pd, i;
        bool first;
        if (paired) { pd = d ^ 1; i = d >> 1; first = (d & 1) == 0; }
        else { first = d < half; pd = first ? d + half : d - half; i = first ? d : d - half; }
        const float xp = to_f32<T>(src[h * sg.src_head + pd]) + (sg.bias != nullptr ? sg.bias[h * sg.head_dim + pd] : 0.f);
        const float c = cs[i], sn = cs[half_max + i];
        y = first ? x * c - xp * sn : x * c + xp * sn;
      }
      dst[h * sg.dst_head + d] = from_f32<T>(y);
    }
  }
}

// The same step in 16-byte pieces (every segment: head_dim, rot / 2 — rot in the paired layout —, the head and row
// strides multiples of the vector width; 16-byte aligned pointers).  A work item is one vector of a head: in the
// paired layout it holds whole pairs; in the half-split layout a vector of the first half is handled together with
// its partner vector of the second half.  Same arithmetic, element by element.
template <typename T>
__global__ void __launch_bounds__(128)
rotary_segments_vec_kernel(RotarySegments segs, const int64_t* __restrict__ positions, const int64_t* __restrict__ loc,
                           const float* __restrict__ cos_sin, int rot_max, int64_t max_positions, int paired) {
  griddep_wait();
  griddep_launch_dependents();
  constexpr int N = Vec16<T>::kN;
  const int64_t t = blockIdx.x;
  int64_t p = positions[t];
  p = p < 0 ? 0 : (p < max_positions ? p : max_positions - 1);
  const float* cs = cos_sin != nullptr ? cos_sin + p * rot_max : nullptr;
  const int half_max = rot_max >> 1;
  const int64_t slot = loc != nullptr ? loc[t] : 0;
  for (int sidx = 0; sidx < segs.n; ++sidx) {
    const RotarySegment& sg = segs.seg[sidx];
    const T* src = reinterpret_cast<const T*>(sg.src) + t * sg.src_row;
    T* dst = reinterpret_cast<T*>(sg.dst) + (sg.to_pool ? slot : t) * sg.dst_row;
    const int half = sg.rot >> 1;
    const int per_head = sg.head_dim / N;
    for (int item = threadIdx.x; item < sg.heads * per_head; item += 128) {
      const int h = item / per_head, d0 = (item - h * per_head) * N;
      const T* sp = src + h * sg.src_head;
      T* dp = dst + h * sg.dst_head;
      const float* bs = sg.bias != nullptr ? sg.bias + h * sg.head_dim : nullptr;
      if (d0 >= sg.rot || paired) {
        const Vec16<T> v = ldv(sp + d0);
        float x[N];
#pragma unroll
        for (int i = 0; i < N; ++i) x[i] = to_f32<T>(v.e()[i]) + (bs != nullptr ? bs[d0 + i] : 0.f);
        Vec16<T> o;
        if (d0 < sg.rot) {
#pragma unroll
          for (int i = 0; i < N; i += 2) {
            const float c = cs[(d0 + i) >> 1], sn = cs[half_max + ((d0 + i) >> 1)];
            o.e()[i] = from_f32<T>(x[i] * c - x[i + 1] * sn);
            o.e()[i + 1] = from_f32<T>(x[i + 1] * c + x[i] * sn);
          }
        } else {
#pragma unroll
          for (int i = 0; i < N; ++i) o.e()[i] = from_f32<T>(x[i]);
        }
        stv(dp + d0, o);
      } else if (d0 < half) {
        const Vec16<T> va = ldv(sp + d0), vb = ldv(sp + d0 + half);
        Vec16<T> oa, ob;
#pragma unroll
        for (int i = 0; i < N; ++i) {
          const float a = to_f32<T>(va.e()[i]) + (bs != nullptr ? bs[d0 + i] : 0.f);
          const float b = to_f32<T>(vb.e()[i]) + (bs != nullptr ? bs[d0 + half + i] : 0.f);
          const float c = cs[d0 + i], sn = cs[half_max + d0 + i];
          oa.e()[i] = from_f32<T>(a * c - b * sn);
          ob.e()[i] = from_f32<T>(b * c + a * sn);
        }
        stv(dp + d0, oa);
        stv(dp + d0 + half, ob);
      }  // vectors of the second half were written with their partners
    }
  }
}

// The form with per-head norms in 16-byte pieces (every segment turns whole heads or none in the half-split layout, its
// head_dim / (2 N) is a power of two of at most 32, strides and pointers aligned): a lane owns vector i of a head's
// first half and vector i of its second half — rotation partners — and the head's lanes sum their squares by shuffles.
// The items (lane, head) of all segments form one list, each segment starting at a warp boundary.
template <typename T>
__global__ void __launch_bounds__(256)
rotary_segments_norm_vec_kernel(RotarySegments segs, const int64_t* __restrict__ positions,
                                const int64_t* __restrict__ loc, const float* __restrict__ cos_sin, int rot_max,
                                int64_t max_positions) {
  griddep_wait();
  griddep_launch_dependents();
  constexpr int N = Vec16<T>::kN;
  const int64_t t = blockIdx.x;
  int64_t p = positions[t];
  p = p < 0 ? 0 : (p < max_positions ? p : max_positions - 1);
  const float* cs = cos_sin != nullptr ? cos_sin + p * rot_max : nullptr;
  const int half_max = rot_max >> 1;
  const int64_t slot = loc != nullptr ? loc[t] : 0;
  int total = 0;
  for (int sidx = 0; sidx < segs.n; ++sidx) total += (segs.seg[sidx].heads * (segs.seg[sidx].head_dim / (2 * N)) + 31) & ~31;
  for (int it = threadIdx.x; it < total; it += blockDim.x) {  // uniform over a warp
    int sidx = 0, item = it;
    for (;; ++sidx) {
      const int n = (segs.seg[sidx].heads * (segs.seg[sidx].head_dim / (2 * N)) + 31) & ~31;
      if (item < n) break;
      item -= n;
    }
    const RotarySegment& sg = segs.seg[sidx];
    const int gl = sg.head_dim / (2 * N), half = sg.head_dim >> 1;
    const int h = item / gl, d0 = (item - h * gl) * N;
    const bool on = h < sg.heads;
    const T* sp = reinterpret_cast<const T*>(sg.src) + t * sg.src_row + (on ? h : 0) * sg.src_head + d0;
    const Vec16<T> va = ldv(sp), vb = ldv(sp + half);
    float a[N], b[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {
      a[i] = to_f32<T>(va.e()[i]);
      b[i] = to_f32<T>(vb.e()[i]);
    }
    auto with4 = [&](const float* src, bool add) {  // add to / multiply by the head's fp32 vector
#pragma unroll
      for (int i = 0; i < N; i += 4) {
        const float4 x = *reinterpret_cast<const float4*>(src + d0 + i), y = *reinterpret_cast<const float4*>(src + half + d0 + i);
        if (add) {
          a[i] += x.x; a[i + 1] += x.y; a[i + 2] += x.z; a[i + 3] += x.w;
          b[i] += y.x; b[i + 1] += y.y; b[i + 2] += y.z; b[i + 3] += y.w;
        } else {
          a[i] *= x.x; a[i + 1] *= x.y; a[i + 2] *= x.z; a[i + 3] *= x.w;
          b[i] *= y.x; b[i + 1] *= y.y; b[i + 2] *= y.z; b[i + 3] *= y.w;
        }
      }
    };
    if (sg.bias != nullptr) with4(sg.bias + (on ? h : 0) * sg.head_dim, true);
    if (sg.norm) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < N; ++i) ss = fmaf(a[i], a[i], fmaf(b[i], b[i], ss));
      for (int m = 1; m < gl; m <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
      const float inv = 1.0f / sqrtf(ss / (float)sg.head_dim + sg.norm_eps);
#pragma unroll
      for (int i = 0; i < N; ++i) {
        a[i] *= inv;
        b[i] *= inv;
      }
      if (sg.norm_w != nullptr) with4(sg.norm_w, false);
    }
    if (sg.rot) {
#pragma unroll
      for (int i = 0; i < N; i += 4) {
        const float4 c4 = *reinterpret_cast<const float4*>(cs + d0 + i);
        const float4 s4 = *reinterpret_cast<const float4*>(cs + half_max + d0 + i);
        const float c[4] = {c4.x, c4.y, c4.z, c4.w}, sn[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = a[i + e], y = b[i + e];
          a[i + e] = x * c[e] - y * sn[e];
          b[i + e] = y * c[e] + x * sn[e];
        }
      }
    }
    if (on) {
      T* dp = reinterpret_cast<T*>(sg.dst) + (sg.to_pool ? slot : t) * sg.dst_row + h * sg.dst_head + d0;
      Vec16<T> oa, ob;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        oa.e()[i] = from_f32<T>(a[i]);
        ob.e()[i] = from_f32<T>(b[i]);
      }
      stv(dp, oa);
      stv(dp + half, ob);
    }
  }
}

// The same for any sizes and either layout: a warp per (token, head), the head's channels in shared memory between the norm and
// the rotation.  VEC consecutive channels per lane and step (head_dim a multiple of 32 VEC for every segment, rows and
// heads aligned to VEC elements), else VEC = 1.
constexpr int kRotNormMaxDim = 512;
template <typename T, int VEC>
struct alignas(sizeof(T) * VEC) RotVec {
  T e[VEC];
};
template <typename T, int VEC>
__global__ void __launch_bounds__(128)
rotary_segments_norm_kernel(RotarySegments segs, const int64_t* __restrict__ positions, const int64_t* __restrict__ loc,
                            const float* __restrict__ cos_sin, int rot_max, int64_t max_positions, int paired,
                            int dim_max) {
  griddep_wait();
  griddep_launch_dependents();
  extern __shared__ __align__(16) float rn_smem[];  // [4][dim_max]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* xs = rn_smem + warp * dim_max;
  const int64_t t = blockIdx.x;
  int64_t p = positions[t];
  p = p < 0 ? 0 : (p < max_positions ? p : max_positions - 1);
  const float* cs = cos_sin != nullptr ? cos_sin + p * rot_max : nullptr;
  const int half_max = rot_max >> 1;
  const int64_t slot = loc != nullptr ? loc[t] : 0;
  int h0 = 0;  // heads of the segments before this one: head number n of the token goes to warp n mod 4
  for (int sidx = 0; sidx < segs.n; ++sidx) {
    const RotarySegment& sg = segs.seg[sidx];
    const T* src = reinterpret_cast<const T*>(sg.src) + t * sg.src_row;
    T* dst = reinterpret_cast<T*>(sg.dst) + (sg.to_pool ? slot : t) * sg.dst_row;
    const int half = sg.rot >> 1, dim = sg.head_dim;
    for (int h = (warp - h0) & 3; h < sg.heads; h += 4) {
      const T* sp = src + h * sg.src_head;
      const float* bs = sg.bias != nullptr ? sg.bias + h * dim : nullptr;
      float ss = 0.f;
      for (int d0 = lane * VEC; d0 < dim; d0 += 32 * VEC) {
        const RotVec<T, VEC> v = *reinterpret_cast<const RotVec<T, VEC>*>(sp + d0);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const float x = to_f32<T>(v.e[e]) + (bs != nullptr ? bs[d0 + e] : 0.f);
          ss = fmaf(x, x, ss);
          xs[d0 + e] = x;
        }
      }
      float inv = 1.f;
      if (sg.norm) inv = 1.0f / sqrtf(warp_sum(ss) / (float)dim + sg.norm_eps);
      const float* nw = sg.norm ? sg.norm_w : nullptr;
      __syncwarp();
      for (int d0 = lane * VEC; d0 < dim; d0 += 32 * VEC) {
        RotVec<T, VEC> o;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const int d = d0 + e;
          float y = xs[d] * inv * (nw != nullptr ? nw[d] : 1.f);
          if (d < sg.rot) {
            int pd, i;
            bool first;
            if (paired) { pd = d ^ 1; i = d >> 1; first = (d & 1) == 0; }
            else { first = d < half; pd = first ? d + half : d - half; i = first ? d : d - half; }
            const float yp = xs[pd] * inv * (nw != nullptr ? nw[pd] : 1.f);
            const float c = cs[i], sn = cs[half_max + i];
            y = first ? y * c - yp * sn : y * c + yp * sn;
          }
          o.e[e] = from_f32<T>(y);
        }
        *reinterpret_cast<RotVec<T, VEC>*>(dst + h * sg.dst_head + d0) = o;
      }
      __syncwarp();  // the next head overwrites xs
    }
    h0 += sg.heads;
  }
}

// The form with norms over all heads of a row (norm 2; norm 0 segments beside them): one CTA per token sums the squares
// of every normed segment, then each work item — VEC channels of a head, in the rotated part together with their
// partners — is read again (from L1), scaled, rotated and written.  VEC > 1: head_dim, rot / 2 (rot in the paired
// layout), head and row strides multiples of VEC, 16-byte aligned pointers.
constexpr int kRowNormThreads = 256;
template <typename T, int VEC>
__global__ void __launch_bounds__(kRowNormThreads)
rotary_segments_rownorm_kernel(RotarySegments segs, const int64_t* __restrict__ positions,
                               const int64_t* __restrict__ loc, const float* __restrict__ cos_sin, int rot_max,
                               int64_t max_positions, int paired) {
  griddep_wait();
  griddep_launch_dependents();
  using V = RotVec<T, VEC>;
  __shared__ float red[4][kRowNormThreads / 32];
  const int64_t t = blockIdx.x;
  int64_t p = positions[t];
  p = p < 0 ? 0 : (p < max_positions ? p : max_positions - 1);
  const float* cs = cos_sin != nullptr ? cos_sin + p * rot_max : nullptr;
  const int half_max = rot_max >> 1;
  const int64_t slot = loc != nullptr ? loc[t] : 0;
  float ss[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int sidx = 0; sidx < 4; ++sidx) {
    if (sidx >= segs.n || segs.seg[sidx].norm != 2) continue;
    const RotarySegment& sg = segs.seg[sidx];
    const T* src = reinterpret_cast<const T*>(sg.src) + t * sg.src_row;
    const int per_head = sg.head_dim / VEC;
    for (int item = threadIdx.x; item < sg.heads * per_head; item += kRowNormThreads) {
      const int h = item / per_head, d0 = (item - h * per_head) * VEC;
      const V v = *reinterpret_cast<const V*>(src + h * sg.src_head + d0);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float x = to_f32<T>(v.e[i]) + (sg.bias != nullptr ? sg.bias[h * sg.head_dim + d0 + i] : 0.f);
        ss[sidx] = fmaf(x, x, ss[sidx]);
      }
    }
    ss[sidx] = warp_sum(ss[sidx]);
    if ((threadIdx.x & 31) == 0) red[sidx][threadIdx.x >> 5] = ss[sidx];
  }
  __syncthreads();
  for (int sidx = 0; sidx < segs.n; ++sidx) {
    const RotarySegment& sg = segs.seg[sidx];
    const T* src = reinterpret_cast<const T*>(sg.src) + t * sg.src_row;
    T* dst = reinterpret_cast<T*>(sg.dst) + (sg.to_pool ? slot : t) * sg.dst_row;
    float inv = 1.f;
    if (sg.norm == 2) {
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < kRowNormThreads / 32; ++i) sum += red[sidx][i];
      inv = 1.0f / sqrtf(sum / (float)(sg.heads * sg.head_dim) + sg.norm_eps);
    }
    const float* nw = sg.norm == 2 ? sg.norm_w : nullptr;
    const int half = sg.rot >> 1, per_head = sg.head_dim / VEC;
    for (int item = threadIdx.x; item < sg.heads * per_head; item += kRowNormThreads) {
      const int h = item / per_head, d0 = (item - h * per_head) * VEC;
      const T* sp = src + h * sg.src_head;
      T* dp = dst + h * sg.dst_head;
      auto read = [&](int d, float (&x)[VEC]) {
        const V v = *reinterpret_cast<const V*>(sp + d);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const int c = h * sg.head_dim + d + i;
          x[i] = (to_f32<T>(v.e[i]) + (sg.bias != nullptr ? sg.bias[c] : 0.f)) * inv * (nw != nullptr ? nw[c] : 1.f);
        }
      };
      auto write = [&](int d, const float (&x)[VEC]) {
        V v;
#pragma unroll
        for (int i = 0; i < VEC; ++i) v.e[i] = from_f32<T>(x[i]);
        *reinterpret_cast<V*>(dp + d) = v;
      };
      float a[VEC];
      if (d0 >= sg.rot) {
        read(d0, a);
        write(d0, a);
      } else if (VEC > 1 && paired) {
        read(d0, a);
#pragma unroll
        for (int i = 0; i + 1 < VEC; i += 2) {
          const float c = cs[(d0 + i) >> 1], sn = cs[half_max + ((d0 + i) >> 1)];
          const float x = a[i], y = a[i + 1];
          a[i] = x * c - y * sn;
          a[i + 1] = y * c + x * sn;
        }
        write(d0, a);
      } else {
        // the item of the pair's first channel turns both
        const int partner = paired ? d0 + 1 : d0 + half;
        if (paired ? (d0 & 1) != 0 : d0 >= half) continue;
        float b[VEC];
        read(d0, a);
        read(partner, b);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const int f = paired ? d0 >> 1 : d0 + i;
          const float c = cs[f], sn = cs[half_max + f];
          const float x = a[i], y = b[i];
          a[i] = x * c - y * sn;
          b[i] = y * c + x * sn;
        }
        write(d0, a);
        write(partner, b);
      }
    }
  }
}

// The same in 16-byte pieces that stay in registers between the sum and the rotation (half-split layout; head_dim, rot / 2,
// strides multiples of the vector width; weights, biases and table rows 16-byte aligned).  The items of all segments form
// one list — per head rot / (2 N) vectors that carry their rotation partner, then (head_dim - rot) / N single ones — of
// which a thread owns NI.
struct RowNormItems {
  int start[5];  // first item of each segment; start[n] = all items
};
template <typename T, int NI>
__global__ void __launch_bounds__(kRowNormThreads)
rotary_segments_rownorm_vec_kernel(RotarySegments segs, RowNormItems items, const int64_t* __restrict__ positions,
                                   const int64_t* __restrict__ loc, const float* __restrict__ cos_sin, int rot_max,
                                   int64_t max_positions) {
  griddep_wait();
  griddep_launch_dependents();
  constexpr int N = Vec16<T>::kN;
  __shared__ float red[4][kRowNormThreads / 32];
  const int64_t t = blockIdx.x;
  int seg_of[NI], col[NI];  // segment (-1: none), first channel within the row of heads
  Vec16<T> va[NI], vb[NI];
  float ss[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int u = 0; u < NI; ++u) {
    int item = (int)(threadIdx.x + u * blockDim.x);
    int s = 0;
    while (s < segs.n && item >= items.start[s + 1]) ++s;
    seg_of[u] = s < segs.n ? s : -1;
    if (s >= segs.n) continue;
    const RotarySegment& sg = segs.seg[s];
    item -= items.start[s];
    const int leads = sg.rot / (2 * N), per_head = leads + (sg.head_dim - sg.rot) / N;
    const int h = item / per_head, x = item - h * per_head;
    const int d0 = x < leads ? x * N : sg.rot + (x - leads) * N;
    col[u] = h * sg.head_dim + d0;
    const T* sp = reinterpret_cast<const T*>(sg.src) + t * sg.src_row + h * sg.src_head + d0;
    va[u] = ldv(sp);
    if (x < leads) vb[u] = ldv(sp + (sg.rot >> 1));
    if (x >= leads) seg_of[u] |= 8;  // no partner
  }
  int64_t p = positions[t];
  p = p < 0 ? 0 : (p < max_positions ? p : max_positions - 1);
  const float* cs = cos_sin != nullptr ? cos_sin + p * rot_max : nullptr;
  const int half_max = rot_max >> 1;
  const int64_t slot = loc != nullptr ? loc[t] : 0;
  auto with_vector = [&](const Vec16<T>& v, const float* bias, int c, float (&x)[N]) {
#pragma unroll
    for (int i = 0; i < N; ++i) x[i] = to_f32<T>(v.e()[i]);
    if (bias != nullptr) {
#pragma unroll
      for (int i = 0; i < N; i += 4) {
        const float4 b = *reinterpret_cast<const float4*>(bias + c + i);
        x[i] += b.x; x[i + 1] += b.y; x[i + 2] += b.z; x[i + 3] += b.w;
      }
    }
  };
#pragma unroll
  for (int u = 0; u < NI; ++u) {
    if (seg_of[u] < 0) continue;
    const RotarySegment& sg = segs.seg[seg_of[u] & 3];
    if (sg.norm != 2) continue;
    float x[N], sum = 0.f;
    with_vector(va[u], sg.bias, col[u], x);
#pragma unroll
    for (int i = 0; i < N; ++i) sum = fmaf(x[i], x[i], sum);
    if ((seg_of[u] & 8) == 0) {
      with_vector(vb[u], sg.bias, col[u] + (sg.rot >> 1), x);
#pragma unroll
      for (int i = 0; i < N; ++i) sum = fmaf(x[i], x[i], sum);
    }
#pragma unroll
    for (int s = 0; s < 4; ++s) ss[s] += (seg_of[u] & 3) == s ? sum : 0.f;
  }
#pragma unroll
  for (int s = 0; s < 4; ++s) {
    if (s >= segs.n || segs.seg[s].norm != 2) continue;
    ss[s] = warp_sum(ss[s]);
    if ((threadIdx.x & 31) == 0) red[s][threadIdx.x >> 5] = ss[s];
  }
  __syncthreads();
  const int warps = blockDim.x >> 5;
#pragma unroll
  for (int u = 0; u < NI; ++u) {
    if (seg_of[u] < 0) continue;
    const int s = seg_of[u] & 3;
    const RotarySegment& sg = segs.seg[s];
    float inv = 1.f;
    const float* nw = nullptr;
    if (sg.norm == 2) {
      float sum = 0.f;
      for (int i = 0; i < warps; ++i) sum += red[s][i];
      inv = 1.0f / sqrtf(sum / (float)(sg.heads * sg.head_dim) + sg.norm_eps);
      nw = sg.norm_w;
    }
    const int half = sg.rot >> 1;
    const int h = col[u] / sg.head_dim, d0 = col[u] - h * sg.head_dim;
    T* dp = reinterpret_cast<T*>(sg.dst) + (sg.to_pool ? slot : t) * sg.dst_row + h * sg.dst_head + d0;
    auto scaled = [&](const Vec16<T>& v, int c, float (&x)[N]) {
      with_vector(v, sg.bias, c, x);
#pragma unroll
      for (int i = 0; i < N; ++i) x[i] *= inv;
      if (nw != nullptr) {
#pragma unroll
        for (int i = 0; i < N; i += 4) {
          const float4 w = *reinterpret_cast<const float4*>(nw + c + i);
          x[i] *= w.x; x[i + 1] *= w.y; x[i + 2] *= w.z; x[i + 3] *= w.w;
        }
      }
    };
    float a[N];
    Vec16<T> o;
    scaled(va[u], col[u], a);
    if ((seg_of[u] & 8) == 0) {
      float b[N];
      Vec16<T> ob;
      scaled(vb[u], col[u] + half, b);
#pragma unroll
      for (int i = 0; i < N; i += 4) {
        const float4 c4 = *reinterpret_cast<const float4*>(cs + d0 + i);
        const float4 s4 = *reinterpret_cast<const float4*>(cs + half_max + d0 + i);
        const float c[4] = {c4.x, c4.y, c4.z, c4.w}, sn[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = a[i + e], y = b[i + e];
          a[i + e] = x * c[e] - y * sn[e];
          b[i + e] = y * c[e] + x * sn[e];
        }
      }
#pragma unroll
      for (int i = 0; i < N; ++i) ob.e()[i] = from_f32<T>(b[i]);
      stv(dp + half, ob);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) o.e()[i] = from_f32<T>(a[i]);
    stv(dp, o);
  }
}

// The residual update of a layer that norms its sublayer's output: x[row] += y / rms(y) * coef (y null: no update),
// then out = x in T, or (w given) x / rms(x) * (off + w).  One CTA per row; a row of up to NV vectors per thread stays
// in registers (VEC = 1: any size, read twice).
constexpr int kPostThreads = 256;
__device__ __forceinline__ float post_block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kPostThreads / 32; ++i) t += red[i];
  __syncthreads();
  return t;
}

template <typename T, int NV>
__global__ void __launch_bounds__(kPostThreads)
residual_postnorm_vec_kernel(T* __restrict__ out, float* __restrict__ x, const T* __restrict__ y,
                             const float* __restrict__ coef, const T* __restrict__ w, int64_t dim, float eps, float off) {
  griddep_wait();
  griddep_launch_dependents();
  constexpr int N = Vec16<T>::kN;
  __shared__ float red[kPostThreads / 32];
  const int64_t row = blockIdx.x;
  float xv[NV][N], yv[NV][N];
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int64_t i = ((int64_t)v * kPostThreads + threadIdx.x) * N;
    if (i < dim) {
#pragma unroll
      for (int e = 0; e < N; e += 4) {
        const float4 f = *reinterpret_cast<const float4*>(x + row * dim + i + e);
        xv[v][e] = f.x; xv[v][e + 1] = f.y; xv[v][e + 2] = f.z; xv[v][e + 3] = f.w;
      }
      if (y != nullptr) {
        const Vec16<T> a = ldv(y + row * dim + i);
#pragma unroll
        for (int e = 0; e < N; ++e) {
          yv[v][e] = to_f32<T>(a.e()[e]);
          ss = fmaf(yv[v][e], yv[v][e], ss);
        }
      }
    }
  }
  if (y != nullptr) {
    const float inv = 1.0f / sqrtf(post_block_sum(ss, red) / (float)dim + eps);
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int64_t i = ((int64_t)v * kPostThreads + threadIdx.x) * N;
      if (i < dim) {
#pragma unroll
        for (int e = 0; e < N; e += 4) {
          const float4 c = *reinterpret_cast<const float4*>(coef + i + e);
          xv[v][e] += yv[v][e] * inv * c.x;
          xv[v][e + 1] += yv[v][e + 1] * inv * c.y;
          xv[v][e + 2] += yv[v][e + 2] * inv * c.z;
          xv[v][e + 3] += yv[v][e + 3] * inv * c.w;
          *reinterpret_cast<float4*>(x + row * dim + i + e) =
              make_float4(xv[v][e], xv[v][e + 1], xv[v][e + 2], xv[v][e + 3]);
        }
      }
    }
  }
  if (out == nullptr) return;
  float inv = 1.f;
  if (w != nullptr) {
    ss = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v)
      if (((int64_t)v * kPostThreads + threadIdx.x) * N < dim) {
#pragma unroll
        for (int e = 0; e < N; ++e) ss = fmaf(xv[v][e], xv[v][e], ss);
      }
    inv = 1.0f / sqrtf(post_block_sum(ss, red) / (float)dim + eps);
  }
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int64_t i = ((int64_t)v * kPostThreads + threadIdx.x) * N;
    if (i < dim) {
      Vec16<T> o, wv;
      if (w != nullptr) wv = ldv(w + i);
#pragma unroll
      for (int e = 0; e < N; ++e)
        o.e()[e] = from_f32<T>(w != nullptr ? xv[v][e] * inv * (off + to_f32<T>(wv.e()[e])) : xv[v][e]);
      stv(out + row * dim + i, o);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(kPostThreads)
residual_postnorm_kernel(T* __restrict__ out, float* __restrict__ x, const T* __restrict__ y,
                         const float* __restrict__ coef, const T* __restrict__ w, int64_t dim, float eps, float off) {
  griddep_wait();
  griddep_launch_dependents();
  __shared__ float red[kPostThreads / 32];
  const int64_t row = blockIdx.x;
  float* xr = x + row * dim;
  float inv = 0.f, ss = 0.f;
  if (y != nullptr) {
    for (int64_t i = threadIdx.x; i < dim; i += kPostThreads) {
      const float a = to_f32<T>(y[row * dim + i]);
      ss = fmaf(a, a, ss);
    }
    inv = 1.0f / sqrtf(post_block_sum(ss, red) / (float)dim + eps);
  }
  ss = 0.f;
  for (int64_t i = threadIdx.x; i < dim; i += kPostThreads) {
    float v = xr[i];
    if (y != nullptr) {
      v += to_f32<T>(y[row * dim + i]) * inv * coef[i];
      xr[i] = v;
    }
    if (out != nullptr && w == nullptr) out[row * dim + i] = from_f32<T>(v);
    ss = fmaf(v, v, ss);
  }
  if (out == nullptr || w == nullptr) return;
  inv = 1.0f / sqrtf(post_block_sum(ss, red) / (float)dim + eps);
  for (int64_t i = threadIdx.x; i < dim; i += kPostThreads)  // a thread reads back the elements it wrote
    out[row * dim + i] = from_f32<T>(xr[i] * inv * (off + to_f32<T>(w[i])));
}

// out[t, h, c] = y[c] * sigmoid(gate[t, h * vdim + c]) with y = a[t, h, :] or, a2 given,
// y = unit_rms(a - lambda a2) * post  (unit RMS over the head's vdim values, eps inside the root).
template <typename T>
__global__ void __launch_bounds__(128)
heads_gate_kernel(T* __restrict__ out, const T* __restrict__ a, const T* __restrict__ a2, const T* __restrict__ gate,
                  int64_t tokens, int heads, int vdim, int64_t a_stride, int64_t gate_stride, int64_t out_stride,
                  float lambda, float eps, float post) {
  griddep_wait();
  griddep_launch_dependents();
  const int lane = threadIdx.x & 31;
  const int64_t item = blockIdx.x * 4ll + (threadIdx.x >> 5);
  if (item >= tokens * heads) return;
  const int64_t t = item / heads;
  const int h = (int)(item - t * heads);
  const T* ar = a + t * a_stride + (int64_t)h * vdim;
  const T* gr = gate + t * gate_stride + (int64_t)h * vdim;
  T* orow = out + t * out_stride + (int64_t)h * vdim;
  float mul = 1.f;
  const T* br = nullptr;
  if (a2 != nullptr) {
    br = a2 + t * a_stride + (int64_t)h * vdim;
    float ss = 0.f;
    for (int c = lane; c < vdim; c += 32) {
      const float d = to_f32<T>(ar[c]) - lambda * to_f32<T>(br[c]);
      ss += d * d;
    }
    ss = warp_sum(ss);
    mul = post / sqrtf(ss / (float)vdim + eps);
  }
  for (int c = lane; c < vdim; c += 32) {
    float y = to_f32<T>(ar[c]);
    if (br != nullptr) y = (y - lambda * to_f32<T>(br[c])) * mul;
    orow[c] = from_f32<T>(y * mix_sigmoid(to_f32<T>(gr[c])));
  }
}

}  // namespace spd

using namespace spd;

extern "C" {

int spd_embed_pair(float* x, const void* table, const void* pair, const int64_t* idx, int32_t* prev_state,
                   const int64_t* req_pool_indices, const int64_t* seq_lens, const int64_t* out_cache_loc,
                   const int32_t* prefix_lens, const int32_t* extend_lens, const int32_t* extend_start_loc,
                   int64_t batch, int64_t tokens, int64_t dim, int64_t table_rows, float scale, int64_t buckets,
                   int64_t mul_prev, int64_t mul_cur, int dtype, spd_stream_t stream) {
  SPD_REQUIRE(x && table && idx, SPD_E_BADARG, "spd_embed_pair: null pointer");
  SPD_REQUIRE(tokens >= 0 && dim > 0 && table_rows > 0, SPD_E_BADARG, "spd_embed_pair: bad sizes");
  if (pair != nullptr) {
    SPD_REQUIRE(prev_state && req_pool_indices && buckets > 0, SPD_E_BADARG,
                "spd_embed_pair: the pair table needs the previous-token state and the request slots");
    SPD_REQUIRE(seq_lens != nullptr || (prefix_lens && extend_lens && extend_start_loc), SPD_E_BADARG,
                "spd_embed_pair: extend needs prefix_lens, extend_lens and extend_start_loc");
    SPD_REQUIRE(seq_lens == nullptr || batch == tokens, SPD_E_BADARG, "spd_embed_pair: decode has one row per request");
    SPD_REQUIRE(batch > 0 && batch < (1ll << 31), SPD_E_BADARG, "spd_embed_pair: bad batch");
  }
  if (tokens == 0) return 0;
  SPD_DISPATCH_ANY(dtype, {
    SPD_CUDA(launch(embed_pair_kernel<T>, dim3((unsigned)tokens), dim3(kMixThreads), 0, as_stream(stream), pdl_enabled(),
                    x, (const T*)table, (const T*)pair, idx, prev_state, req_pool_indices, seq_lens, out_cache_loc,
                    prefix_lens, extend_lens, extend_start_loc, (int)batch, dim, table_rows, scale, buckets, mul_prev,
                    mul_cur));
  });
  return 0;
}

int spd_residual_tanh_norm(void* out, float* x, const void* a, const float* x0, const float* vec, const void* w,
                           const void* b, const int64_t* rows, int64_t n_rows, int64_t dim, float alpha, int dtype,
                           spd_stream_t stream) {
  SPD_REQUIRE(x && (out == nullptr) == (w == nullptr) && (w == nullptr) == (b == nullptr), SPD_E_BADARG,
              "spd_residual_tanh_norm: null pointer");
  SPD_REQUIRE(rows == nullptr || (a == nullptr && x0 == nullptr && vec == nullptr), SPD_E_BADARG,
              "spd_residual_tanh_norm: selected rows are read only");
  SPD_REQUIRE(n_rows >= 0 && dim > 0, SPD_E_BADARG, "spd_residual_tanh_norm: bad sizes");
  if (n_rows == 0) return 0;
  SPD_DISPATCH_ANY(dtype, {
    SPD_CUDA(launch(residual_tanh_norm_kernel<T>, dim3((unsigned)n_rows), dim3(kMixThreads), 0, as_stream(stream),
                    pdl_enabled(), (T*)out, x, (const T*)a, x0, vec, (const T*)w, (const T*)b, rows, dim, alpha));
  });
  return 0;
}

int spd_residual_postnorm(void* out, float* x, const void* y, const float* coef, const void* w, int64_t rows, int64_t dim,
                          float eps, float weight_offset, int dtype, spd_stream_t stream) {
  SPD_REQUIRE(x && (y == nullptr) == (coef == nullptr) && (out != nullptr || w == nullptr) && (out || y), SPD_E_BADARG,
              "spd_residual_postnorm: null pointer");
  SPD_REQUIRE(rows >= 0 && dim > 0, SPD_E_BADARG, "spd_residual_postnorm: bad sizes");
  if (rows == 0) return 0;
  SPD_DISPATCH_ANY(dtype, {
    constexpr int N = 16 / (int)sizeof(T);
    const int64_t nv = (dim / N + kPostThreads - 1) / kPostThreads;
    if (dim % N == 0 && nv <= 4 && aligned16(out) && aligned16(x) && aligned16(y) && aligned16(coef) && aligned16(w)) {
      auto kern = nv == 1   ? residual_postnorm_vec_kernel<T, 1>
                  : nv == 2 ? residual_postnorm_vec_kernel<T, 2>
                            : residual_postnorm_vec_kernel<T, 4>;
      SPD_CUDA(launch(kern, dim3((unsigned)rows), dim3(kPostThreads), 0, as_stream(stream), pdl_enabled(), (T*)out, x,
                      (const T*)y, coef, (const T*)w, dim, eps, weight_offset));
    } else {
      SPD_CUDA(launch(residual_postnorm_kernel<T>, dim3((unsigned)rows), dim3(kPostThreads), 0, as_stream(stream),
                      pdl_enabled(), (T*)out, x, (const T*)y, coef, (const T*)w, dim, eps, weight_offset));
    }
  });
  return 0;
}

int spd_rotary_segments(const spd_rotary_segment_t* segments, int num_segments, const int64_t* positions,
                        const int64_t* loc, const float* cos_sin, int rot_max, int64_t max_positions, int paired,
                        int64_t tokens, int dtype, spd_stream_t stream) {
  SPD_REQUIRE(segments && positions && num_segments >= 1 && num_segments <= 4, SPD_E_BADARG,
              "spd_rotary_segments: 1 to 4 segments");
  RotarySegments segs;
  segs.n = num_segments;
  for (int i = 0; i < num_segments; ++i) {
    const spd_rotary_segment_t& s = segments[i];
    SPD_REQUIRE(s.src && s.dst && s.heads > 0 && s.head_dim > 0 && s.rot >= 0 && s.rot <= s.head_dim && s.rot % 2 == 0 &&
                    s.rot <= rot_max, SPD_E_SHAPE, "spd_rotary_segments: segment %d: bad sizes", i);
    SPD_REQUIRE(s.rot == 0 || cos_sin != nullptr, SPD_E_BADARG, "spd_rotary_segments: rotation without a table");
    SPD_REQUIRE(!s.to_pool || loc != nullptr, SPD_E_BADARG, "spd_rotary_segments: a cache segment needs slot ids");
    segs.seg[i] = RotarySegment{s.src, s.bias, s.dst, s.src_row, s.dst_row, s.heads, s.head_dim, s.rot, s.src_head,
                                s.dst_head, s.to_pool, s.norm_w, s.norm, s.norm_eps};
  }
  if (tokens == 0) return 0;
  bool row_norm = false, head_norm = false;
  for (int i = 0; i < num_segments; ++i) {
    row_norm = row_norm || segs.seg[i].norm == 2;
    head_norm = head_norm || segs.seg[i].norm == 1;
    SPD_REQUIRE(segs.seg[i].norm >= 0 && segs.seg[i].norm <= 2, SPD_E_BADARG, "spd_rotary_segments: norm is 0, 1 or 2");
  }
  const int vecn = dtype == SPD_F32 ? 4 : 8;
  bool vec = true;
  for (int i = 0; i < num_segments; ++i) {
    const RotarySegment& s = segs.seg[i];
    vec = vec && s.head_dim % vecn == 0 && (paired ? s.rot : s.rot / 2) % vecn == 0 && s.src_head % vecn == 0 &&
          s.dst_head % vecn == 0 && s.src_row % vecn == 0 && s.dst_row % vecn == 0 && aligned16(s.src) && aligned16(s.dst);
  }
  if (row_norm) {
    SPD_REQUIRE(!head_norm, SPD_E_BADARG, "spd_rotary_segments: norms per head and per row in one launch");
    bool pieces = vec && !paired && rot_max % 8 == 0 && aligned16(cos_sin);
    RowNormItems items{};
    for (int i = 0; i < num_segments; ++i) {
      const RotarySegment& s = segs.seg[i];
      pieces = pieces && aligned16(s.bias) && aligned16(s.norm_w);
      items.start[i + 1] = items.start[i] + s.heads * (s.rot / (2 * vecn) + (s.head_dim - s.rot) / vecn);
    }
    const int total = items.start[num_segments];
    if (pieces && total <= 4 * kRowNormThreads) {
      const int ni = total <= kRowNormThreads ? 1 : total <= 2 * kRowNormThreads ? 2 : 4;
      const int threads = ((total + ni - 1) / ni + 31) / 32 * 32;
      SPD_DISPATCH_ANY(dtype, {
        auto kern = ni == 1   ? rotary_segments_rownorm_vec_kernel<T, 1>
                    : ni == 2 ? rotary_segments_rownorm_vec_kernel<T, 2>
                              : rotary_segments_rownorm_vec_kernel<T, 4>;
        SPD_CUDA(launch(kern, dim3((unsigned)tokens), dim3((unsigned)threads), 0, as_stream(stream), pdl_enabled(), segs,
                        items, positions, loc, cos_sin, rot_max, max_positions));
      });
      return 0;
    }
    SPD_DISPATCH_ANY(dtype, {
      auto kern = vec ? rotary_segments_rownorm_kernel<T, 16 / (int)sizeof(T)> : rotary_segments_rownorm_kernel<T, 1>;
      SPD_CUDA(launch(kern, dim3((unsigned)tokens), dim3(kRowNormThreads), 0, as_stream(stream), pdl_enabled(), segs,
                      positions, loc, cos_sin, rot_max, max_positions, paired));
    });
    return 0;
  }
  int dim_max = 0, step = 4;  // form with norms: the widest step every segment's sizes allow
  bool any_norm = false;
  for (int i = 0; i < num_segments; ++i) {
    const RotarySegment& s = segs.seg[i];
    any_norm = any_norm || s.norm != 0;
    dim_max = s.head_dim > dim_max ? s.head_dim : dim_max;
    const int64_t align = dtype == SPD_F32 ? 4 : 2;
    while (step > 1 && (s.head_dim % (32 * step) != 0 || s.src_head % step != 0 || s.dst_head % step != 0 ||
                        s.src_row % step != 0 || s.dst_row % step != 0 ||
                        reinterpret_cast<uintptr_t>(s.src) % (step * align) != 0 ||
                        reinterpret_cast<uintptr_t>(s.dst) % (step * align) != 0))
      step >>= 1;
  }
  if (any_norm) {
    SPD_REQUIRE(dim_max <= kRotNormMaxDim, SPD_E_SHAPE, "spd_rotary_segments: normed heads of %d channels (max %d)",
                dim_max, kRotNormMaxDim);
    const int pad = (dim_max + 3) / 4 * 4;
    const int nv = dtype == SPD_F32 ? 4 : 8;
    bool pieces = !paired && rot_max % 8 == 0 && aligned16(cos_sin);
    int items = 0;
    for (int i = 0; i < num_segments; ++i) {
      const RotarySegment& s = segs.seg[i];
      const int gl = s.head_dim / (2 * nv);
      pieces = pieces && s.head_dim % (2 * nv) == 0 && gl <= 32 && (gl & (gl - 1)) == 0 && (s.rot == 0 || s.rot == s.head_dim) &&
               s.src_head % nv == 0 && s.dst_head % nv == 0 && s.src_row % nv == 0 && s.dst_row % nv == 0 &&
               aligned16(s.src) && aligned16(s.dst) && aligned16(s.bias) && aligned16(s.norm_w);
      items += (s.heads * gl + 31) / 32 * 32;
    }
    if (pieces) {
      const int threads = items < 256 ? items : 256;
      SPD_DISPATCH_ANY(dtype, {
        SPD_CUDA(launch(rotary_segments_norm_vec_kernel<T>, dim3((unsigned)tokens), dim3((unsigned)threads), 0,
                        as_stream(stream), pdl_enabled(), segs, positions, loc, cos_sin, rot_max, max_positions));
      });
      return 0;
    }
    SPD_DISPATCH_ANY(dtype, {
      auto kern = step == 4   ? rotary_segments_norm_kernel<T, 4>
                  : step == 2 ? rotary_segments_norm_kernel<T, 2>
                              : rotary_segments_norm_kernel<T, 1>;
      SPD_CUDA(launch(kern, dim3((unsigned)tokens), dim3(128), sizeof(float) * 4 * (size_t)pad, as_stream(stream),
                      pdl_enabled(), segs, positions, loc, cos_sin, rot_max, max_positions, paired, pad));
    });
    return 0;
  }
  SPD_DISPATCH_ANY(dtype, {
    auto kern = vec ? rotary_segments_vec_kernel<T> : rotary_segments_kernel<T>;
    SPD_CUDA(launch(kern, dim3((unsigned)tokens), dim3(128), 0, as_stream(stream), pdl_enabled(), segs, positions, loc,
                    cos_sin, rot_max, max_positions, paired));
  });
  return 0;
}

int spd_heads_gate(void* out, const void* a, const void* a2, const void* gate, int64_t tokens, int heads, int vdim,
                   int64_t a_stride, int64_t gate_stride, int64_t out_stride, float lambda, float eps, float post,
                   int dtype, spd_stream_t stream) {
  SPD_REQUIRE(out && a && gate, SPD_E_BADARG, "spd_heads_gate: null pointer");
  SPD_REQUIRE(tokens >= 0 && heads > 0 && vdim > 0, SPD_E_BADARG, "spd_heads_gate: bad sizes");
  if (tokens == 0) return 0;
  const int64_t ctas = (tokens * heads + 3) / 4;
  SPD_REQUIRE(ctas < (1ll << 31), SPD_E_SHAPE, "spd_heads_gate: batch too large");
  SPD_DISPATCH_ANY(dtype, {
    SPD_CUDA(launch(heads_gate_kernel<T>, dim3((unsigned)ctas), dim3(128), 0, as_stream(stream), pdl_enabled(), (T*)out,
                    (const T*)a, (const T*)a2, (const T*)gate, tokens, heads, vdim, a_stride, gate_stride, out_stride,
                    lambda, eps, post));
  });
  return 0;
}

}  // extern "C"
