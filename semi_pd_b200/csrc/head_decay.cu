// Recurrent mixers whose state decays by ONE number per head and token, and the short causal convolution and the
// gated group norm that stand around them.  Per (request, head) an fp32 matrix state S [head_dim x v_dim] is carried:
//
//   dt_t = softplus(z_t + dt_bias_h),  w_t = exp(-exp(a_log_h) dt_t)
//   form 0 (state-space duality)  S_t = w_t S_(t-1) + dt_t k_t v_t^T ;  o_t = S_t^T q_t + skip_h v_t
//   form 1 (gated delta rule)     S' = w_t S_(t-1) ;  u_t = sigmoid(b_t) (v_t - S'^T k_t) ;  S_t = S' + k_t u_t^T ;
//                                 o_t = S_t^T q_t, with k and q brought to unit length per head (q also scaled)
//
// Decode and ragged extend (chunked prefill, mixed batches) are one kernel: a CTA owns (request, head, 32 value
// columns).  Eight lanes share a column pair, each with every eighth group of four state rows of the two columns in
// registers (as packed fp32 pairs), so a product with the state is three shuffles away from complete and a token needs
// no block-wide barrier.  The delta rule reads the state once per token and walks a prompt two tokens at a time, with
// the small products between the two taken beforehand (A = S^T of the state before the pair):
//   u_1 = b_1 (v_1 - w_1 A k_1),             o_1 = w_1 A q_1 + (k_1 . q_1) u_1
//   u_2 = b_2 (v_2 - w_2 (w_1 A k_2 + (k_1 . k_2) u_1)),
//   o_2 = w_2 (w_1 A q_2 + (k_1 . q_2) u_1) + (k_2 . q_2) u_2,        S <- w_2 (w_1 S + k_1 u_1^T) + k_2 u_2^T
// so that the chain of dependent steps (products, shuffles, u, update) is paid once per pair.
// Separate producer warps prepare the next block of tokens in shared memory (loads, unit length, the small products,
// step size, decay) while the consumer warps walk the current one; one block-wide barrier per token block.  The state is stored
// transposed, [v_dim][head_dim] per head, so that the eight lanes of a column read and write whole 128-byte lines.
// Every output element is summed in one fixed order, so o does not depend on how a prompt was cut or batched.  A
// request that starts at position 0 ignores what its state slots held before.
#include "common.cuh"
#include "ptx.cuh"

namespace spd {

constexpr int kHdTok = 16;       // tokens per block (extend); decode has its one token
constexpr int kHdCols = 32;      // value columns per CTA
constexpr int kHdConsumers = 4;  // warps: eight columns each

// two fp32 lanes in one 64-bit register pair
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(d)
      : "l"(reinterpret_cast<const uint64_t&>(a)), "l"(reinterpret_cast<const uint64_t&>(b)),
        "l"(reinterpret_cast<const uint64_t&>(c)));
  return reinterpret_cast<const float2&>(d);
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;"
      : "=l"(d)
      : "l"(reinterpret_cast<const uint64_t&>(a)), "l"(reinterpret_cast<const uint64_t&>(b)));
  return reinterpret_cast<const float2&>(d);
}
__device__ __forceinline__ float hd_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float hd_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float hd_silu(float z) { return z / (1.0f + expf(-z)); }
// the activations whose result is rounded to T: the fast exponential and division in 16-bit models
template <typename T>
__device__ __forceinline__ float silu_for(float z) { return silu_f32(z); }
template <>
__device__ __forceinline__ float silu_for<float>(float z) { return hd_silu(z); }

// the rows a request brings: first position, first row of the batch, count; false: nothing to do
struct RowSpan {
  int64_t pos0, row0;
  int n;
  bool keep;  // write the state back (not a padded row of a captured batch)
};
__device__ __forceinline__ bool row_span(RowSpan& s, int r, const int64_t* __restrict__ seq_lens,
                                         const int64_t* __restrict__ out_cache_loc,
                                         const int32_t* __restrict__ prefix_lens,
                                         const int32_t* __restrict__ extend_lens,
                                         const int32_t* __restrict__ extend_start_loc) {
  s.keep = true;
  if (seq_lens != nullptr) {
    s.pos0 = seq_lens[r] - 1;
    s.row0 = r;
    s.n = 1;
    if (out_cache_loc != nullptr && out_cache_loc[r] == 0) s.keep = false;
  } else {
    s.pos0 = prefix_lens[r];
    s.row0 = extend_start_loc[r];
    s.n = extend_lens[r];
  }
  return s.n > 0 && s.pos0 >= 0;
}

// four elements of a row, kept as raw words between their load and their use
template <typename T>
struct alignas(4 * sizeof(T)) Quad {
  uint32_t w[sizeof(T)];
  __device__ __forceinline__ float get(int i) const {
    if constexpr (sizeof(T) == 4) {
      return __uint_as_float(w[i]);
    } else {
      const float2 f = unpack2<T>(w[i >> 1]);
      return (i & 1) ? f.y : f.x;
    }
  }
};

template <typename T, int RPL, int TOK, int NPROD, int FORM, bool VEC>
__global__ void __launch_bounds__((kHdConsumers + NPROD) * 32, RPL <= 16 && sizeof(T) == 2 ? 2 : 1)
head_decay_kernel(float* __restrict__ o, const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                  const T* __restrict__ z, const T* __restrict__ b, float* __restrict__ state,
                  const int64_t* __restrict__ req_pool_indices, const int64_t* __restrict__ seq_lens,
                  const int64_t* __restrict__ out_cache_loc, const int32_t* __restrict__ prefix_lens,
                  const int32_t* __restrict__ extend_lens, const int32_t* __restrict__ extend_start_loc, int H, int Hk,
                  int dk, int dv, int64_t q_stride, int64_t k_stride, int64_t v_stride, int64_t z_stride,
                  int64_t b_stride, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                  const float* __restrict__ skip, float q_scale, float unit_eps) {
  constexpr int DKP = RPL * 8;             // padded head_dim
  constexpr int BUF = TOK * (2 * DKP + kHdCols + 4);
  extern __shared__ __align__(16) float hd_smem[];  // (TOK > 1 ? 2 : 1) x { q | k [TOK][DKP], v [TOK][32], scalars [TOK][4] }
  griddep_wait();
  const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kHdCols;
  const int hk = h / (H / Hk);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  RowSpan sp;
  if (!row_span(sp, r, seq_lens, out_cache_loc, prefix_lens, extend_lens, extend_start_loc)) return;
  const int n = sp.n;

  const int j = lane & 7;  // which eighth of the rows (chunks of four rows: j, j + 8, ...)
  const float dt_bias_h = dt_bias[h], rate_h = expf(a_log[h]);
  // Eight lanes prepare a token, a warp four tokens at a time, in ROUNDS rounds per block; tokens past the end become
  // ones that change nothing.  The raw values of a block are loaded a whole block before they are prepared.
  constexpr int ROUNDS = (TOK + 4 * NPROD - 1) / (4 * NPROD);
  Quad<T> rq[ROUNDS][RPL / 4], rk[ROUNDS][RPL / 4], rv[ROUNDS];
  T rz[ROUNDS], rb[ROUNDS];
  auto load4 = [](const T* p, int d, int dim) {  // p[d .. d + 3], zeros from dim on
    Quad<T> f;
    if constexpr (VEC) {
      f = d < dim ? *reinterpret_cast<const Quad<T>*>(p + d) : Quad<T>{};
    } else {
      float x[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] = d + e < dim ? to_f32<T>(p[d + e]) : 0.f;
      if constexpr (sizeof(T) == 4) {
#pragma unroll
        for (int e = 0; e < 4; ++e) f.w[e] = __float_as_uint(x[e]);
      } else {
        f.w[0] = pack2<T>(x[0], x[1]);
        f.w[1] = pack2<T>(x[2], x[3]);
      }
    }
    return f;
  };
  auto fetch = [&](int t0) {
    const int nt = n - t0 < TOK ? n - t0 : TOK;
#pragma unroll
    for (int x = 0; x < ROUNDS; ++x) {
      const int tt = (x * NPROD + warp - kHdConsumers) * 4 + (lane >> 3);
      const int64_t row = sp.row0 + t0 + (tt < nt ? tt : 0);
#pragma unroll
      for (int i = 0; i < RPL / 4; ++i) {
        rq[x][i] = load4(q + row * q_stride + (int64_t)hk * dk, i * 32 + j * 4, dk);
        rk[x][i] = load4(k + row * k_stride + (int64_t)hk * dk, i * 32 + j * 4, dk);
      }
      rv[x] = load4(v + row * v_stride + (int64_t)h * dv, col0 + j * 4, dv);
      rz[x] = z[row * z_stride + h];
      if (FORM == 1) rb[x] = b[row * b_stride + h];
    }
  };
  auto prepare = [&](int t0, float* buf) {
    const int nt = n - t0 < TOK ? n - t0 : TOK;
    float* qs = buf;
    float* ks = qs + TOK * DKP;
    float* vs = ks + TOK * DKP;
    float* sc = vs + TOK * kHdCols;
#pragma unroll
    for (int x = 0; x < ROUNDS; ++x) {
      const int tt = (x * NPROD + warp - kHdConsumers) * 4 + (lane >> 3);
      const bool ok = tt < nt;
      float qv[RPL], kv[RPL], vv[4];
#pragma unroll
      for (int i = 0; i < RPL; ++i) {
        qv[i] = ok ? rq[x][i / 4].get(i % 4) : 0.f;
        kv[i] = ok ? rk[x][i / 4].get(i % 4) : 0.f;
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) vv[i] = rv[x].get(i);
      const float dt = hd_softplus(to_f32<T>(rz[x]) + dt_bias_h);
      const float w = ok ? expf(-rate_h * dt) : 1.f;
      const float coef = !ok ? 0.f : FORM == 0 ? dt : hd_sigmoid(to_f32<T>(rb[x]));
      float kq = 0.f, kk = 0.f, kn = 0.f;  // k . q, and for the second token of a pair k_first . k and k_first . q
      if (FORM == 1) {
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
          sq = fmaf(qv[i], qv[i], sq);
          sk = fmaf(kv[i], kv[i], sk);
          kq = fmaf(kv[i], qv[i], kq);
          if (TOK > 1) {
            const float kp = __shfl_xor_sync(0xffffffffu, kv[i], 8);  // the pair's other token
            kk = fmaf(kp, kv[i], kk);
            kn = fmaf(kp, qv[i], kn);
          }
        }
#pragma unroll
        for (int m = 1; m < 8; m <<= 1) {
          sq += __shfl_xor_sync(0xffffffffu, sq, m);
          sk += __shfl_xor_sync(0xffffffffu, sk, m);
          kq += __shfl_xor_sync(0xffffffffu, kq, m);
          if (TOK > 1) {
            kk += __shfl_xor_sync(0xffffffffu, kk, m);
            kn += __shfl_xor_sync(0xffffffffu, kn, m);
          }
        }
        const float fq = q_scale / sqrtf(sq + unit_eps), fk = 1.0f / sqrtf(sk + unit_eps);
        kq *= fq * fk;
        if (TOK > 1) {
          const float fp = __shfl_xor_sync(0xffffffffu, fk, 8);
          kk *= fp * fk;
          kn *= fp * fq;
        }
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
          qv[i] *= fq;
          kv[i] *= fk;
        }
      } else if (q_scale != 1.f) {
#pragma unroll
        for (int i = 0; i < RPL; ++i) qv[i] *= q_scale;
      }
      if (tt < TOK) {
#pragma unroll
        for (int i = 0; i < RPL / 4; ++i) {
          const int d = tt * DKP + i * 32 + j * 4;
          *reinterpret_cast<float4*>(qs + d) = make_float4(qv[4 * i], qv[4 * i + 1], qv[4 * i + 2], qv[4 * i + 3]);
          *reinterpret_cast<float4*>(ks + d) = make_float4(kv[4 * i], kv[4 * i + 1], kv[4 * i + 2], kv[4 * i + 3]);
        }
        *reinterpret_cast<float4*>(vs + tt * kHdCols + j * 4) = make_float4(vv[0], vv[1], vv[2], vv[3]);
        if (j == 0) {
          *reinterpret_cast<float2*>(sc + tt * 4) = make_float2(w, coef);
          sc[tt * 4 + 2] = kq;
          if (FORM == 1 && (tt & 1)) {
            sc[tt * 4 + 3] = kk;
            sc[tt * 4 - 1] = kn;  // with the pair's first token: its k . q_next
          }
        }
      }
    }
  };

  const bool producer = warp >= kHdConsumers;
  const int c = col0 + (producer ? 0 : warp) * 8 + (lane >> 3) * 2;  // a consumer lane's columns c, c + 1
  float* st = state + ((int64_t)req_pool_indices[r] * H + h) * (int64_t)dk * dv;
  const bool rows4 = (dk & 3) == 0;
  float2 S[2][RPL / 2];
  if (!producer) {
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int i = 0; i < RPL / 4; ++i) {
        const int row = i * 32 + j * 4;
        float4 s4 = make_float4(0.f, 0.f, 0.f, 0.f);
        if (sp.pos0 > 0 && c + x < dv) {
          const float* src = st + (int64_t)(c + x) * dk + row;
          if (rows4) {
            if (row < dk) s4 = *reinterpret_cast<const float4*>(src);
          } else {
            if (row < dk) s4.x = src[0];
            if (row + 1 < dk) s4.y = src[1];
            if (row + 2 < dk) s4.z = src[2];
            if (row + 3 < dk) s4.w = src[3];
          }
        }
        S[x][2 * i] = make_float2(s4.x, s4.y);
        S[x][2 * i + 1] = make_float2(s4.z, s4.w);
      }
  } else {
    fetch(0);
    prepare(0, hd_smem);
    if (TOK > 1 && TOK < n) fetch(TOK);
  }
  const float sk_h = (FORM == 0 && skip != nullptr) ? skip[h] : 0.f;
  __syncthreads();

  for (int t0 = 0; t0 < n; t0 += TOK) {
    float* buf = hd_smem + (TOK > 1 && ((t0 / TOK) & 1) ? BUF : 0);
    if (producer) {
      if (TOK > 1 && t0 + TOK < n) {
        prepare(t0 + TOK, hd_smem + (((t0 / TOK) & 1) ? 0 : BUF));
        if (t0 + 2 * TOK < n) fetch(t0 + 2 * TOK);
      }
    } else {
      const int nt = n - t0 < TOK ? n - t0 : TOK;
      const float* qs = buf;
      const float* ks = qs + TOK * DKP;
      const float* vs = ks + TOK * DKP;
      const float* sc = vs + TOK * kHdCols;
      if (FORM == 1 && TOK > 1) {
        constexpr bool HOLD = RPL <= 16;  // the pair's keys stay in registers between the two passes
        for (int tt = 0; tt < nt; tt += 2) {
          const float4* k4 = reinterpret_cast<const float4*>(ks + tt * DKP) + j;
          const float4* q4 = reinterpret_cast<const float4*>(qs + tt * DKP) + j;
          const float4 s1 = *reinterpret_cast<const float4*>(sc + tt * 4);      // w, b, k . q, k . q_next
          const float4 s2 = *reinterpret_cast<const float4*>(sc + tt * 4 + 4);  // w, b, k . q, k . k_previous
          const float2 v1 = *reinterpret_cast<const float2*>(vs + tt * kHdCols + warp * 8 + (lane >> 3) * 2);
          const float2 v2 = *reinterpret_cast<const float2*>(vs + (tt + 1) * kHdCols + warp * 8 + (lane >> 3) * 2);
          float2 kr[2][HOLD ? RPL / 2 : 1];
          float2 acc[8];  // k_1, k_2, q_1, q_2 by column
#pragma unroll
          for (int i = 0; i < 8; ++i) acc[i] = make_float2(0.f, 0.f);
#pragma unroll
          for (int i = 0; i < RPL / 4; ++i) {
            const float4 f[4] = {k4[i * 8], k4[i * 8 + DKP / 4], q4[i * 8], q4[i * 8 + DKP / 4]};
#pragma unroll
            for (int y = 0; y < 4; ++y) {
              const float2 lo = make_float2(f[y].x, f[y].y), hi = make_float2(f[y].z, f[y].w);
              if (HOLD && y < 2) { kr[y][2 * i] = lo; kr[y][2 * i + 1] = hi; }
              acc[2 * y] = fma2(S[0][2 * i], lo, acc[2 * y]);
              acc[2 * y + 1] = fma2(S[1][2 * i], lo, acc[2 * y + 1]);
              acc[2 * y] = fma2(S[0][2 * i + 1], hi, acc[2 * y]);
              acc[2 * y + 1] = fma2(S[1][2 * i + 1], hi, acc[2 * y + 1]);
            }
          }
          // sum over the eight lanes; lane j ends with value j
          float p[8], t4[4], t2[2];
#pragma unroll
          for (int i = 0; i < 8; ++i) p[i] = acc[i].x + acc[i].y;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float got = __shfl_xor_sync(0xffffffffu, (j & 4) ? p[i] : p[i + 4], 4);
            t4[i] = ((j & 4) ? p[i + 4] : p[i]) + got;
          }
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float got = __shfl_xor_sync(0xffffffffu, (j & 2) ? t4[i] : t4[i + 2], 2);
            t2[i] = ((j & 2) ? t4[i + 2] : t4[i]) + got;
          }
          const float got = __shfl_xor_sync(0xffffffffu, (j & 1) ? t2[0] : t2[1], 1);
          const float mine = ((j & 1) ? t2[1] : t2[0]) + got;
          const int g0 = lane & 24;  // the eight lanes' first
          const float a10 = __shfl_sync(0xffffffffu, mine, g0), a11 = __shfl_sync(0xffffffffu, mine, g0 + 1);
          const float a20 = __shfl_sync(0xffffffffu, mine, g0 + 2), a21 = __shfl_sync(0xffffffffu, mine, g0 + 3);
          const float u10 = s1.y * (v1.x - s1.x * a10), u11 = s1.y * (v1.y - s1.x * a11);
          const float u20 = s2.y * (v2.x - s2.x * fmaf(s2.w, u10, s1.x * a20));
          const float u21 = s2.y * (v2.y - s2.x * fmaf(s2.w, u11, s1.x * a21));
          if (j >= 4) {  // lanes 4 - 7 hold the products with q_1 (two columns), q_2 (two columns)
            const float u1 = (j & 1) ? u11 : u10, u2 = (j & 1) ? u21 : u20;
            const float first = s1.x * mine;
            const float out = (j & 2) ? fmaf(s2.z, u2, s2.x * fmaf(s1.w, u1, first)) : fmaf(s1.z, u1, first);
            const int tok = tt + ((j >> 1) & 1), col = c + (j & 1);
            if (tok < nt && col < dv) o[((sp.row0 + t0 + tok) * H + h) * (int64_t)dv + col] = out;
          }
          const float w12 = s1.x * s2.x;
          const float2 wp = make_float2(w12, w12);
          const float2 x10 = make_float2(s2.x * u10, s2.x * u10), x11 = make_float2(s2.x * u11, s2.x * u11);
          const float2 x20 = make_float2(u20, u20), x21 = make_float2(u21, u21);
#pragma unroll
          for (int i = 0; i < RPL / 4; ++i) {
            float2 ka[2], kb[2];
            if (HOLD) {
              ka[0] = kr[0][HOLD ? 2 * i : 0]; ka[1] = kr[0][HOLD ? 2 * i + 1 : 0];
              kb[0] = kr[1][HOLD ? 2 * i : 0]; kb[1] = kr[1][HOLD ? 2 * i + 1 : 0];
            } else {
              const float4 f = k4[i * 8], e = k4[i * 8 + DKP / 4];
              ka[0] = make_float2(f.x, f.y); ka[1] = make_float2(f.z, f.w);
              kb[0] = make_float2(e.x, e.y); kb[1] = make_float2(e.z, e.w);
            }
#pragma unroll
            for (int y = 0; y < 2; ++y) {
              S[0][2 * i + y] = fma2(kb[y], x20, fma2(ka[y], x10, mul2(wp, S[0][2 * i + y])));
              S[1][2 * i + y] = fma2(kb[y], x21, fma2(ka[y], x11, mul2(wp, S[1][2 * i + y])));
            }
          }
        }
      } else
      for (int tt = 0; tt < nt; ++tt) {
        const float4* k4 = reinterpret_cast<const float4*>(ks + tt * DKP) + j;
        const float4* q4 = reinterpret_cast<const float4*>(qs + tt * DKP) + j;
        const float4 s = *reinterpret_cast<const float4*>(sc + tt * 4);  // decay, coefficient, k . q
        const float2 vv = *reinterpret_cast<const float2*>(vs + tt * kHdCols + warp * 8 + (lane >> 3) * 2);
        const float2 w2 = make_float2(s.x, s.x);
        float2 k2[RPL / 2];
        float out0, out1;
        if (FORM == 1) {
          float2 a0 = make_float2(0.f, 0.f), a1 = a0, b0 = a0, b1 = a0;  // S^T k and S^T q of the two columns
#pragma unroll
          for (int i = 0; i < RPL / 4; ++i) {
            const float4 kk = k4[i * 8], qq = q4[i * 8];
            k2[2 * i] = make_float2(kk.x, kk.y);
            k2[2 * i + 1] = make_float2(kk.z, kk.w);
            const float2 ql = make_float2(qq.x, qq.y), qh = make_float2(qq.z, qq.w);
            a0 = fma2(S[0][2 * i], k2[2 * i], a0);
            a1 = fma2(S[1][2 * i], k2[2 * i], a1);
            b0 = fma2(S[0][2 * i], ql, b0);
            b1 = fma2(S[1][2 * i], ql, b1);
            a0 = fma2(S[0][2 * i + 1], k2[2 * i + 1], a0);
            a1 = fma2(S[1][2 * i + 1], k2[2 * i + 1], a1);
            b0 = fma2(S[0][2 * i + 1], qh, b0);
            b1 = fma2(S[1][2 * i + 1], qh, b1);
          }
          float x0 = a0.x + a0.y, x1 = a1.x + a1.y, y0 = b0.x + b0.y, y1 = b1.x + b1.y;
#pragma unroll
          for (int m = 1; m < 8; m <<= 1) {
            x0 += __shfl_xor_sync(0xffffffffu, x0, m);
            x1 += __shfl_xor_sync(0xffffffffu, x1, m);
            y0 += __shfl_xor_sync(0xffffffffu, y0, m);
            y1 += __shfl_xor_sync(0xffffffffu, y1, m);
          }
          const float u0 = s.y * (vv.x - s.x * x0), u1 = s.y * (vv.y - s.x * x1);
          const float2 u0p = make_float2(u0, u0), u1p = make_float2(u1, u1);
#pragma unroll
          for (int i = 0; i < RPL / 2; ++i) {
            S[0][i] = fma2(k2[i], u0p, mul2(w2, S[0][i]));
            S[1][i] = fma2(k2[i], u1p, mul2(w2, S[1][i]));
          }
          out0 = fmaf(s.z, u0, s.x * y0);
          out1 = fmaf(s.z, u1, s.x * y1);
        } else {
          const float2 u0p = make_float2(s.y * vv.x, s.y * vv.x), u1p = make_float2(s.y * vv.y, s.y * vv.y);
          float2 b0 = make_float2(0.f, 0.f), b1 = b0;
#pragma unroll
          for (int i = 0; i < RPL / 4; ++i) {
            const float4 kk = k4[i * 8], qq = q4[i * 8];
            const float2 kl = make_float2(kk.x, kk.y), kh = make_float2(kk.z, kk.w);
            const float2 ql = make_float2(qq.x, qq.y), qh = make_float2(qq.z, qq.w);
            S[0][2 * i] = fma2(kl, u0p, mul2(w2, S[0][2 * i]));
            S[1][2 * i] = fma2(kl, u1p, mul2(w2, S[1][2 * i]));
            b0 = fma2(S[0][2 * i], ql, b0);
            b1 = fma2(S[1][2 * i], ql, b1);
            S[0][2 * i + 1] = fma2(kh, u0p, mul2(w2, S[0][2 * i + 1]));
            S[1][2 * i + 1] = fma2(kh, u1p, mul2(w2, S[1][2 * i + 1]));
            b0 = fma2(S[0][2 * i + 1], qh, b0);
            b1 = fma2(S[1][2 * i + 1], qh, b1);
          }
          float y0 = b0.x + b0.y, y1 = b1.x + b1.y;
#pragma unroll
          for (int m = 1; m < 8; m <<= 1) {
            y0 += __shfl_xor_sync(0xffffffffu, y0, m);
            y1 += __shfl_xor_sync(0xffffffffu, y1, m);
          }
          out0 = fmaf(sk_h, vv.x, y0);
          out1 = fmaf(sk_h, vv.y, y1);
        }
        if (j < 2 && c + j < dv)
          o[((sp.row0 + t0 + tt) * H + h) * (int64_t)dv + c + j] = j == 0 ? out0 : out1;
      }
    }
    __syncthreads();  // the next block is prepared; this one's buffer is free
  }
  if (!producer && sp.keep) {
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int i = 0; i < RPL / 4; ++i) {
        const int row = i * 32 + j * 4;
        if (c + x >= dv) continue;
        float* dst = st + (int64_t)(c + x) * dk + row;
        const float2 lo = S[x][2 * i], hi = S[x][2 * i + 1];
        if (rows4) {
          if (row < dk) *reinterpret_cast<float4*>(dst) = make_float4(lo.x, lo.y, hi.x, hi.y);
        } else {
          if (row < dk) dst[0] = lo.x;
          if (row + 1 < dk) dst[1] = lo.y;
          if (row + 2 < dk) dst[2] = hi.x;
          if (row + 3 < dk) dst[3] = hi.y;
        }
      }
  }
}

template <typename T, int RPL, int TOK, int NPROD, int FORM, bool VEC>
int head_decay_launch(dim3 grid, cudaStream_t stream, float* o, const void* q, const void* k, const void* v,
                      const void* z, const void* b, float* state, const int64_t* req_pool_indices,
                      const int64_t* seq_lens, const int64_t* out_cache_loc, const int32_t* prefix_lens,
                      const int32_t* extend_lens, const int32_t* extend_start_loc, int H, int Hk, int dk, int dv,
                      int64_t q_stride, int64_t k_stride, int64_t v_stride, int64_t z_stride, int64_t b_stride,
                      const float* dt_bias, const float* a_log, const float* skip, float q_scale, float unit_eps) {
  const size_t smem = sizeof(float) * (TOK > 1 ? 2 : 1) * (size_t)TOK * (2 * RPL * 8 + kHdCols + 4);
  static size_t configured = 0;
  if (smem > 48 * 1024 && smem > configured) {
    SPD_CUDA(cudaFuncSetAttribute(head_decay_kernel<T, RPL, TOK, NPROD, FORM, VEC>,
                                  cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  SPD_CUDA(launch(head_decay_kernel<T, RPL, TOK, NPROD, FORM, VEC>, grid, dim3((kHdConsumers + NPROD) * 32), smem, stream,
                  pdl_enabled(), o, (const T*)q, (const T*)k, (const T*)v, (const T*)z, (const T*)b, state,
                  req_pool_indices, seq_lens, out_cache_loc, prefix_lens, extend_lens, extend_start_loc, H, Hk, dk, dv,
                  q_stride, k_stride, v_stride, z_stride, b_stride, dt_bias, a_log, skip, q_scale, unit_eps));
  return 0;
}

// ------------------------------------------------------------------------------------------------
// short causal convolution per channel + SiLU: out[t, c] = silu(sum_i w[i, c] x[t - (TAPS - 1) + i, c] + bias[c]).
// The TAPS - 1 inputs before a request's first new row are kept in its state slot (fp32 [TAPS - 1][channels], oldest
// first; zeros at position 0); the slot then receives its last TAPS - 1 inputs.  One CTA per (request, slice of the
// channels, chunk of the request's rows); the CTA of the first chunk is the only one that touches the slot.
// ------------------------------------------------------------------------------------------------
constexpr int kConvThreads = 128;  // at most
constexpr int kConvChunk = 16;
constexpr int kConvMaxTaps = 8;

template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kConvThreads)
short_conv_kernel(T* __restrict__ out, const T* __restrict__ x, const T* __restrict__ w, const T* __restrict__ bias,
                  float* __restrict__ conv_state, const int64_t* __restrict__ req_pool_indices,
                  const int64_t* __restrict__ seq_lens, const int64_t* __restrict__ out_cache_loc,
                  const int32_t* __restrict__ prefix_lens, const int32_t* __restrict__ extend_lens,
                  const int32_t* __restrict__ extend_start_loc, int64_t channels, int64_t x_stride) {
  griddep_wait();
  griddep_launch_dependents();
  constexpr int HIST = TAPS - 1;
  const int r = blockIdx.x;
  const int64_t c = ((int64_t)blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= channels) return;
  RowSpan sp;
  if (!row_span(sp, r, seq_lens, out_cache_loc, prefix_lens, extend_lens, extend_start_loc)) return;
  const int t_lo = blockIdx.z * kConvChunk;
  if (t_lo >= sp.n) return;
  const int t_hi = t_lo + kConvChunk < sp.n ? t_lo + kConvChunk : sp.n;
  auto load = [&](const T* p, float* dst) {
    if constexpr (VEC == 1) {
      dst[0] = to_f32<T>(p[0]);
    } else {
      const Vec16<T> v = ldv(p);
#pragma unroll
      for (int e = 0; e < VEC; ++e) dst[e] = to_f32<T>(v.e()[e]);
    }
  };
  float wt[TAPS][VEC], bs[VEC], hist[HIST > 0 ? HIST : 1][VEC];
#pragma unroll
  for (int i = 0; i < TAPS; ++i) load(w + (int64_t)i * channels + c, wt[i]);
#pragma unroll
  for (int e = 0; e < VEC; ++e) bs[e] = 0.f;
  if (bias != nullptr) load(bias + c, bs);
  if (HIST > 0) {
    if (t_lo == 0) {
      float* slot = conv_state + (int64_t)req_pool_indices[r] * HIST * channels + c;
#pragma unroll
      for (int i = 0; i < HIST; ++i)
#pragma unroll
        for (int e = 0; e < VEC; ++e) hist[i][e] = sp.pos0 > 0 ? slot[(int64_t)i * channels + e] : 0.f;
      if (sp.keep) {
#pragma unroll
        for (int i = 0; i < HIST; ++i) {
          const int t = sp.n - HIST + i;  // which of the new rows becomes entry i (negative: an entry kept from before)
          float keep[VEC];
          if (t >= 0) {
            load(x + (sp.row0 + t) * x_stride + c, keep);
          } else {
#pragma unroll
            for (int jx = 0; jx < HIST; ++jx)
              if (jx == HIST + t) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) keep[e] = hist[jx][e];
              }
          }
#pragma unroll
          for (int e = 0; e < VEC; ++e) slot[(int64_t)i * channels + e] = keep[e];
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < HIST; ++i) load(x + (sp.row0 + t_lo - HIST + i) * x_stride + c, hist[i]);
    }
  }
#pragma unroll 4
  for (int t = t_lo; t < t_hi; ++t) {
    float cur[VEC], y[VEC];
    load(x + (sp.row0 + t) * x_stride + c, cur);
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = bs[e];
#pragma unroll
    for (int i = 0; i < HIST; ++i)
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = fmaf(wt[i][e], hist[i][e], y[e]);
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = silu_for<T>(fmaf(wt[HIST][e], cur[e], y[e]));
#pragma unroll
    for (int i = 0; i + 1 < HIST; ++i)
#pragma unroll
      for (int e = 0; e < VEC; ++e) hist[i][e] = hist[i + 1][e];
    if (HIST > 0) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) hist[HIST - 1][e] = cur[e];
    }
    T* dst = out + (sp.row0 + t) * channels + c;
    if constexpr (VEC == 1) {
      dst[0] = from_f32<T>(y[0]);
    } else {
      Vec16<T> v;
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.e()[e] = from_f32<T>(y[e]);
      stv(dst, v);
    }
  }
}

template <typename T, int VEC, int TAPS>
int short_conv_launch(int64_t batch, int64_t rows, cudaStream_t stream, void* out, const void* x, const void* w,
                      const void* bias, float* conv_state, const int64_t* req_pool_indices, const int64_t* seq_lens,
                      const int64_t* out_cache_loc, const int32_t* prefix_lens, const int32_t* extend_lens,
                      const int32_t* extend_start_loc, int64_t channels, int64_t x_stride) {
  // whole warps, the channels spread evenly over the fewest CTAs
  const int64_t vecs = (channels + VEC - 1) / VEC, ctas = (vecs + kConvThreads - 1) / kConvThreads;
  const int64_t threads = ((vecs + ctas - 1) / ctas + 31) / 32 * 32, per = threads * VEC;
  const int64_t chunks = (rows + kConvChunk - 1) / kConvChunk;
  SPD_REQUIRE(chunks <= 65535 && (channels + per - 1) / per <= 65535, SPD_E_SHAPE, "spd_short_conv: too many rows or channels");
  const dim3 grid((unsigned)batch, (unsigned)((channels + per - 1) / per), (unsigned)chunks);
  SPD_CUDA(launch(short_conv_kernel<T, VEC, TAPS>, grid, dim3((unsigned)threads), 0, stream, pdl_enabled(), (T*)out,
                  (const T*)x, (const T*)w, (const T*)bias, conv_state, req_pool_indices, seq_lens, out_cache_loc,
                  prefix_lens, extend_lens, extend_start_loc, channels, x_stride));
  return 0;
}

// ------------------------------------------------------------------------------------------------
// out = y silu(z) at unit RMS over each of `groups` equal parts of a row, times w: one CTA per (row, part), the gated
// part held in shared memory between the two passes
// ------------------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
gated_group_norm_kernel(T* __restrict__ out, const float* __restrict__ y, const T* __restrict__ z,
                        const T* __restrict__ w, int groups, int part, int64_t z_stride, float eps) {
  griddep_wait();
  griddep_launch_dependents();
  extern __shared__ __align__(16) float gn_smem[];  // [part]
  __shared__ float red[8];
  const int64_t t = blockIdx.x / groups;
  const int g = (int)(blockIdx.x - t * groups);
  const int64_t off = (int64_t)g * part, row = t * groups * (int64_t)part + off;
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < part; i += blockDim.x * VEC) {
    if constexpr (VEC == 1) {
      const float a = y[row + i] * hd_silu(to_f32<T>(z[t * z_stride + off + i]));
      gn_smem[i] = a;
      ss = fmaf(a, a, ss);
    } else {
      const Vec16<T> zv = ldv(z + t * z_stride + off + i);
#pragma unroll
      for (int e = 0; e < VEC; e += 4) {
        const float4 yv = *reinterpret_cast<const float4*>(y + row + i + e);
        float4 a;
        a.x = yv.x * hd_silu(to_f32<T>(zv.e()[e]));
        a.y = yv.y * hd_silu(to_f32<T>(zv.e()[e + 1]));
        a.z = yv.z * hd_silu(to_f32<T>(zv.e()[e + 2]));
        a.w = yv.w * hd_silu(to_f32<T>(zv.e()[e + 3]));
        *reinterpret_cast<float4*>(gn_smem + i + e) = a;
        ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
      }
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < (int)blockDim.x / 32; ++i) tot += red[i];
  const float inv = 1.0f / sqrtf(tot / (float)part + eps);
  // a thread reads back the elements it wrote
  for (int i = threadIdx.x * VEC; i < part; i += blockDim.x * VEC) {
    if constexpr (VEC == 1) {
      out[row + i] = from_f32<T>(gn_smem[i] * inv * to_f32<T>(w[off + i]));
    } else {
      const Vec16<T> wv = ldv(w + off + i);
      Vec16<T> ov;
#pragma unroll
      for (int e = 0; e < VEC; ++e) ov.e()[e] = from_f32<T>(gn_smem[i + e] * inv * to_f32<T>(wv.e()[e]));
      stv(out + row + i, ov);
    }
  }
}

}  // namespace spd

using namespace spd;

extern "C" {

int spd_head_decay(float* o, const void* q, const void* k, const void* v, const void* z, const void* b, float* state,
                   const int64_t* req_pool_indices, const int64_t* seq_lens, const int64_t* out_cache_loc,
                   const int32_t* prefix_lens, const int32_t* extend_lens, const int32_t* extend_start_loc,
                   int64_t batch, int num_heads, int num_k_heads, int head_dim, int v_dim, int64_t q_stride,
                   int64_t k_stride, int64_t v_stride, int64_t z_stride, int64_t b_stride, const float* dt_bias,
                   const float* a_log, const float* skip, int form, float q_scale, float unit_eps, int dtype,
                   spd_stream_t stream) {
  SPD_REQUIRE(o && q && k && v && z && state && req_pool_indices && dt_bias && a_log, SPD_E_BADARG,
              "spd_head_decay: null pointer");
  SPD_REQUIRE(form == 0 || (form == 1 && b != nullptr && skip == nullptr), SPD_E_BADARG, "spd_head_decay: form %d", form);
  SPD_REQUIRE(seq_lens != nullptr || (prefix_lens && extend_lens && extend_start_loc), SPD_E_BADARG,
              "spd_head_decay: extend needs prefix_lens, extend_lens and extend_start_loc");
  SPD_REQUIRE(num_heads > 0 && num_heads <= 65535 && num_k_heads > 0 && num_heads % num_k_heads == 0, SPD_E_SHAPE,
              "spd_head_decay: heads %d not a multiple of key heads %d", num_heads, num_k_heads);
  SPD_REQUIRE(head_dim > 0 && head_dim <= 256 && v_dim > 0 && v_dim <= 65535 * kHdCols, SPD_E_SHAPE,
              "spd_head_decay: head_dim %d above 256", head_dim);
  if (batch == 0) return 0;
  const dim3 grid((unsigned)batch, (unsigned)num_heads, (unsigned)((v_dim + kHdCols - 1) / kHdCols));
  const bool decode = seq_lens != nullptr;
#define SPD_HD_ARGS                                                                                                  \
  grid, as_stream(stream), o, q, k, v, z, b, state, req_pool_indices, seq_lens, out_cache_loc, prefix_lens,          \
      extend_lens, extend_start_loc, num_heads, num_k_heads, head_dim, v_dim, q_stride, k_stride, v_stride, z_stride, \
      b_stride, dt_bias, a_log, skip, q_scale, unit_eps
#define SPD_HD_SHAPE(RPL, VEC)                                                                    \
  do {                                                                                            \
    if (decode) return form == 0 ? head_decay_launch<T, RPL, 1, 1, 0, VEC>(SPD_HD_ARGS)           \
                                 : head_decay_launch<T, RPL, 1, 1, 1, VEC>(SPD_HD_ARGS);          \
    return form == 0 ? head_decay_launch<T, RPL, kHdTok, 2, 0, VEC>(SPD_HD_ARGS)                  \
                     : head_decay_launch<T, RPL, kHdTok, 2, 1, VEC>(SPD_HD_ARGS);                 \
  } while (0)
  SPD_DISPATCH_ANY(dtype, {
    // rows in groups of four elements; other sizes take one element-wise instantiation
    const bool vec = ((head_dim | v_dim | q_stride | k_stride | v_stride) & 3) == 0 &&
                     ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) &
                      (sizeof(Quad<T>) - 1)) == 0;
    if (!vec) SPD_HD_SHAPE(32, false);
    else if (head_dim <= 32) SPD_HD_SHAPE(4, true);
    else if (head_dim <= 64) SPD_HD_SHAPE(8, true);
    else if (head_dim <= 128) SPD_HD_SHAPE(16, true);
    else SPD_HD_SHAPE(32, true);
  });
#undef SPD_HD_SHAPE
#undef SPD_HD_ARGS
  return 0;
}

int spd_short_conv(void* out, const void* x, const void* w, const void* bias, float* conv_state,
                   const int64_t* req_pool_indices, const int64_t* seq_lens, const int64_t* out_cache_loc,
                   const int32_t* prefix_lens, const int32_t* extend_lens, const int32_t* extend_start_loc,
                   int64_t batch, int64_t total_rows, int64_t max_rows_per_request, int64_t channels, int taps,
                   int64_t x_stride, int dtype, spd_stream_t stream) {
  SPD_REQUIRE(out && x && w && req_pool_indices && (taps == 1 || conv_state), SPD_E_BADARG, "spd_short_conv: null pointer");
  SPD_REQUIRE(seq_lens != nullptr || (prefix_lens && extend_lens && extend_start_loc), SPD_E_BADARG,
              "spd_short_conv: extend needs prefix_lens, extend_lens and extend_start_loc");
  SPD_REQUIRE(channels > 0 && taps >= 1 && taps <= kConvMaxTaps && x_stride >= channels, SPD_E_SHAPE,
              "spd_short_conv: %d taps (max %d)", taps, kConvMaxTaps);
  if (batch == 0 || total_rows == 0) return 0;
  const int64_t rows = seq_lens != nullptr ? 1 : (max_rows_per_request > 0 ? max_rows_per_request : total_rows);
#define SPD_CONV_ARGS                                                                                               \
  batch, rows, as_stream(stream), out, x, w, bias, conv_state, req_pool_indices, seq_lens, out_cache_loc, prefix_lens, \
      extend_lens, extend_start_loc, channels, x_stride
#define SPD_CONV_TAPS(VEC)                                              \
  switch (taps) {                                                       \
    case 1: return short_conv_launch<T, VEC, 1>(SPD_CONV_ARGS);         \
    case 2: return short_conv_launch<T, VEC, 2>(SPD_CONV_ARGS);         \
    case 3: return short_conv_launch<T, VEC, 3>(SPD_CONV_ARGS);         \
    case 4: return short_conv_launch<T, VEC, 4>(SPD_CONV_ARGS);         \
    case 5: return short_conv_launch<T, VEC, 5>(SPD_CONV_ARGS);         \
    case 6: return short_conv_launch<T, VEC, 6>(SPD_CONV_ARGS);         \
    case 7: return short_conv_launch<T, VEC, 7>(SPD_CONV_ARGS);         \
    default: return short_conv_launch<T, VEC, 8>(SPD_CONV_ARGS);        \
  }
  SPD_DISPATCH_ANY(dtype, {
    constexpr int N = 16 / (int)sizeof(T);
    if (channels % N == 0 && x_stride % N == 0 && aligned16(out) && aligned16(x) && aligned16(w) && aligned16(bias)) {
      SPD_CONV_TAPS(N)
    } else {
      SPD_CONV_TAPS(1)
    }
  });
#undef SPD_CONV_TAPS
#undef SPD_CONV_ARGS
  return 0;
}

int spd_gated_group_norm(void* out, const float* y, const void* z, const void* w, int64_t rows, int groups, int part,
                         int64_t z_stride, float eps, int dtype, spd_stream_t stream) {
  SPD_REQUIRE(out && y && z && w, SPD_E_BADARG, "spd_gated_group_norm: null pointer");
  SPD_REQUIRE(rows >= 0 && groups > 0 && part > 0 && part <= 48 * 1024, SPD_E_SHAPE, "spd_gated_group_norm: bad sizes");
  SPD_REQUIRE(rows * groups < (1ll << 31), SPD_E_SHAPE, "spd_gated_group_norm: batch too large");
  if (rows == 0) return 0;
  const size_t smem = sizeof(float) * (size_t)part;
  SPD_DISPATCH_ANY(dtype, {
    constexpr int N = 16 / (int)sizeof(T);
    const bool vec = part % N == 0 && z_stride % N == 0 && aligned16(out) && aligned16(y) && aligned16(z) && aligned16(w);
    auto kern = vec ? gated_group_norm_kernel<T, N> : gated_group_norm_kernel<T, 1>;
    const int64_t per = vec ? part / N : part;
    const unsigned threads = per <= 32 ? 32 : per <= 64 ? 64 : per <= 128 ? 128 : 256;
    if (smem > 48 * 1024 - 64) {
      SPD_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    }
    SPD_CUDA(launch(kern, dim3((unsigned)(rows * groups)), dim3(threads), smem, as_stream(stream), pdl_enabled(), (T*)out,
                    y, (const T*)z, (const T*)w, groups, part, z_stride, eps));
  });
  return 0;
}

}  // extern "C"
