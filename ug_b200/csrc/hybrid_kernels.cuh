// Row kernels of the layer-list engine (hybrid_engine.cu): everything between the matrix products of a decoder whose
// layers are recurrent or latent-attention mixers with sandwich norms, input convolutions and a depth average; the residual
// update and the convolution also serve layers in the parallel form (parallel_kernels.cuh).
//
// T is the activation type (bf16, or f32 when the model runs in 32 bits).  Norms, the residual stream, the layer
// bank, gates and the recurrence are f32 whatever T is.  Every row buffer is `ld` elements wide (a multiple of 8, the
// model's width rounded up); the gains, convolution taps and weight rows behind the width are zero, so the padding
// stays zero everywhere and a mean is a sum over ld divided by the width.
#pragma once
#include <cuda_bf16.h>

#include "tc_ptx.cuh"
#include "ugb_internal.h"

namespace ugb_hybrid_k {

template <typename T> struct Act;
template <> struct Act<float> {
  static __device__ __forceinline__ float4 ld4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
  static __device__ __forceinline__ void st4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
  static __device__ __forceinline__ float round(float v) { return v; }
};
template <> struct Act<__nv_bfloat16> {
  static __device__ __forceinline__ float4 ld4(const __nv_bfloat16 *p) {
    const uint2 v = *reinterpret_cast<const uint2 *>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&v.y));
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void st4(__nv_bfloat16 *p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*(uint32_t *)&a, *(uint32_t *)&b);
  }
  static __device__ __forceinline__ float round(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }
};

// Gate functions in fp32; EXACT: correctly rounded division and full-precision exp, otherwise the hardware's exp2 and
// reciprocal (about 1e-6 relative): the block scan of a bf16 model is bound by the instructions of its gates.
template <bool EXACT> __device__ __forceinline__ float sigmoid_t(float x) {
  if constexpr (EXACT) return 1.0f / (1.0f + expf(-x));
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * -1.4426950408889634f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));   // e = inf gives 0
  return r;
}
__device__ __forceinline__ float sigmoid_f(float x) { return sigmoid_t<true>(x); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
// candidate of the minimal gated recurrent unit: u + 1/2 for u >= 0, sigmoid(u) below -- the larger of the two on either
// side, since sigmoid has slope at most 1/4 and equals 1/2 at 0
template <bool EXACT> __device__ __forceinline__ float gru_candidate(float u) { return fmaxf(u + 0.5f, sigmoid_t<EXACT>(u)); }

__device__ __forceinline__ float block_sum_256(float v, float *sm) {   // sm: 8 floats; all 256 threads
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  __syncthreads();                                                     // the previous use of sm is over
  if ((threadIdx.x & 31) == 0) sm[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) s += sm[i];
  return s;
}
__device__ __forceinline__ float sq4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }

// ------------------------------------------------------------- row update ---
// One CTA per row r, in this order:
//   y   = sum of the projection partials, or the embedding row of token id(r);  + sum_k routed[slot[r][k]];  + bias
//   x   = x + norm(y) * post_gain          (post_gain null: y itself; add_x 0: the stream starts here)
//   bank_out = x;  x = sum_j dwa[j] bank[j] + dwa[n_avg] x        (with a depth average)
//   copy = x rounded to T (twice, where a second place is given)
//   h   = norm(x) * gain, rounded to T     (gain null: none)
//   h   = h + sum_j conv[j] h_(-taps+1+j)  (conv set: one new position per sequence; the tail of earlier h's is the
//                                           sequence's state and moves on by one)
template <typename T> struct RowArgs {
  const int *tok = nullptr;            // embedding source: row r = (r / t, r % t) reads tok[(r / t) * tok_stride + tok_off + r % t]
  const T *embed = nullptr;
  int vocab = 0, t = 1, tok_stride = 1, tok_off = 0;
  const float *part = nullptr;         // or projection partials [n_part][rows][ld]
  int n_part = 0;
  size_t part_stride = 0;
  const float *routed = nullptr;       // rows of other products that belong to this one: slot[r][k] < 0 = none
  const int *slot = nullptr;
  int top = 0;
  const float *bias = nullptr;         // [ld], joins y
  const float *post_gain = nullptr;
  float *x = nullptr;
  int add_x = 1;
  float *bank_out = nullptr;
  const float *bank = nullptr;         // [n_avg] earlier results, bank_stride apart
  size_t bank_stride = 0;
  const float *dwa = nullptr;          // n_avg + 1 coefficients, null = no depth average
  int n_avg = 0;
  const float *gain = nullptr;
  T *h = nullptr;
  T *copy = nullptr, *copy2 = nullptr; // rows copy_ld apart
  size_t copy_ld = 0;
  int *zero = nullptr;                 // n_zero counters that the kernels behind this one want at zero
  int n_zero = 0;
  const float *conv = nullptr;         // [taps][ld]
  int taps = 0;
  T *tail = nullptr;                   // [rows][taps - 1][ld]
  int ld = 0;
  float inv_width = 0.f, eps = 0.f;
  int early = 0;                       // 1: x, bank and tail may be read before the wait for the preceding kernel
  ugb_status_word *status = nullptr;
};

// Taps of a fused convolution whose tail rows are held in registers from before the wait; longer ones are read late.
constexpr int ROW_TAPS = 4;

// STEP: few rows (a decode step), everything that can be requested early is; otherwise many rows, whose CTAs hide one
// another's latencies, and registers count.
template <typename T, int VPT, bool STEP>
__global__ void __launch_bounds__(256, (STEP || VPT > 2 ? 1 : 4))
row_update_kernel(RowArgs<T> a) {
  __shared__ float sm[8];
  const int r = blockIdx.x, nvec = a.ld >> 2;
  const size_t row0 = (size_t)r * a.ld;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 *xr = reinterpret_cast<float4 *>(a.x + row0);
  float4 v[VPT], pg[VPT], acc[VPT];
  float4 tl[STEP ? ROW_TAPS - 1 : 1][VPT];
  const bool short_conv = STEP && a.conv != nullptr && a.taps <= ROW_TAPS;
  // Weights, and what kernels before the predecessor wrote -- the residual row, the layer bank, the convolution tail --
  // are read ahead of the wait: every kernel of the chain lets its successor start only after its own wait has returned,
  // so when this kernel runs, everything up to its predecessor's predecessor is complete.
  if (!a.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    pg[i] = make_float4(1.f, 1.f, 1.f, 1.f);
    v[i] = acc[i] = zero;
    if (c < nvec) {
      if (a.add_x) v[i] = xr[c];
      if (a.post_gain) pg[i] = __ldg(reinterpret_cast<const float4 *>(a.post_gain) + c);
      if (STEP && short_conv) {
#pragma unroll
        for (int j = 0; j < (STEP ? ROW_TAPS - 1 : 1); ++j)
          tl[j][i] = j < a.taps - 1 ? Act<T>::ld4(a.tail + ((size_t)r * (a.taps - 1) + j) * a.ld + 4 * c) : zero;
      }
    }
  }
  if (a.dwa) {
    constexpr int U = STEP ? (VPT <= 2 ? 8 : (VPT <= 4 ? 4 : 2)) : (VPT <= 2 ? 4 : 2);  // bank rows in flight
    for (int j = 0; j < a.n_avg; j += U) {
      float4 q[U][VPT];
      float w[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const bool on = j + u < a.n_avg;
        w[u] = on ? __ldg(a.dwa + j + u) : 0.f;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int c = threadIdx.x + i * 256;
          q[u][i] = zero;
          if (on && c < nvec) q[u][i] = __ldcg(reinterpret_cast<const float4 *>(a.bank + (size_t)(j + u) * a.bank_stride + row0) + c);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          acc[i].x = fmaf(w[u], q[u][i].x, acc[i].x); acc[i].y = fmaf(w[u], q[u][i].y, acc[i].y);
          acc[i].z = fmaf(w[u], q[u][i].z, acc[i].z); acc[i].w = fmaf(w[u], q[u][i].w, acc[i].w);
        }
    }
  }
  if (a.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
  if (a.zero && r == 0)
    for (int i = threadIdx.x; i < a.n_zero; i += 256) a.zero[i] = 0;
  float4 y[VPT];
  if (a.tok) {
    const int id = a.tok[(size_t)(r / a.t) * a.tok_stride + a.tok_off + r % a.t];
    if (id < 0 || id >= a.vocab) {
      if (threadIdx.x == 0 && atomicCAS(&a.status->code, 0u, (unsigned)UGB_ERR_INVALID) == 0u) a.status->detail = r;
      return;
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      y[i] = c < nvec ? Act<T>::ld4(a.embed + (size_t)id * a.ld + 4 * c) : zero;
    }
  } else if (a.n_part == 1) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      y[i] = c < nvec ? __ldcs(reinterpret_cast<const float4 *>(a.part + row0) + c) : zero;
    }
  } else {
    constexpr int U = STEP ? (VPT <= 2 ? 8 : 4) : 1;      // split-K partials, added in order, U round trips in flight
#pragma unroll
    for (int i = 0; i < VPT; ++i) y[i] = zero;
    for (int s = 0; s < a.n_part; s += U) {
      float4 q[U][VPT];
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int c = threadIdx.x + i * 256;
          q[u][i] = zero;
          if (c < nvec && s + u < a.n_part)
            q[u][i] = __ldcs(reinterpret_cast<const float4 *>(a.part + (size_t)(s + u) * a.part_stride + row0) + c);
        }
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int i = 0; i < VPT; ++i) { y[i].x += q[u][i].x; y[i].y += q[u][i].y; y[i].z += q[u][i].z; y[i].w += q[u][i].w; }
    }
  }
  for (int k = 0; k < a.top; ++k) {
    const int to = __ldcg(a.slot + (size_t)r * a.top + k);
    if (to < 0) continue;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c >= nvec) continue;
      const float4 q = __ldcs(reinterpret_cast<const float4 *>(a.routed + (size_t)to * a.ld) + c);
      y[i].x += q.x; y[i].y += q.y; y[i].z += q.z; y[i].w += q.w;
    }
  }
  if (a.bias) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c >= nvec) continue;
      const float4 q = __ldg(reinterpret_cast<const float4 *>(a.bias) + c);
      y[i].x += q.x; y[i].y += q.y; y[i].z += q.z; y[i].w += q.w;
    }
  }
  float4 g2[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    g2[i] = zero;
    if (a.gain && c < nvec) g2[i] = __ldg(reinterpret_cast<const float4 *>(a.gain) + c);
  }
  float inv = 1.f;
  if (a.post_gain) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) ss += sq4(y[i]);
    inv = 1.0f / sqrtf(block_sum_256(ss, sm) * a.inv_width + a.eps);
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    v[i].x += y[i].x * inv * pg[i].x; v[i].y += y[i].y * inv * pg[i].y;
    v[i].z += y[i].z * inv * pg[i].z; v[i].w += y[i].w * inv * pg[i].w;
  }
  if (a.bank_out) {
    float4 *bo = reinterpret_cast<float4 *>(a.bank_out + row0);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c < nvec) bo[c] = v[i];
    }
  }
  if (a.dwa) {
    const float own = __ldg(a.dwa + a.n_avg);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      v[i].x = fmaf(own, v[i].x, acc[i].x); v[i].y = fmaf(own, v[i].y, acc[i].y);
      v[i].z = fmaf(own, v[i].z, acc[i].z); v[i].w = fmaf(own, v[i].w, acc[i].w);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c < nvec) xr[c] = v[i];
    if (a.copy && c < nvec) Act<T>::st4(a.copy + (size_t)r * a.copy_ld + 4 * c, v[i]);
    if (a.copy2 && c < nvec) Act<T>::st4(a.copy2 + (size_t)r * a.copy_ld + 4 * c, v[i]);
    ss += sq4(v[i]);
  }
  if (!a.gain) return;
  const float inv2 = 1.0f / sqrtf(block_sum_256(ss, sm) * a.inv_width + a.eps);
  auto fma4 = [](float4 w, float4 q, float4 &s) {
    s.x = fmaf(w.x, q.x, s.x); s.y = fmaf(w.y, q.y, s.y); s.z = fmaf(w.z, q.z, s.z); s.w = fmaf(w.w, q.w, s.w);
  };
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c >= nvec) continue;
    float4 h = make_float4(v[i].x * inv2 * g2[i].x, v[i].y * inv2 * g2[i].y, v[i].z * inv2 * g2[i].z, v[i].w * inv2 * g2[i].w);
    if (a.conv) {
      // what the convolution sees, now and later, is the rounded h
      h = make_float4(Act<T>::round(h.x), Act<T>::round(h.y), Act<T>::round(h.z), Act<T>::round(h.w));
      T *tp = a.tail + (size_t)r * (a.taps - 1) * a.ld + 4 * c;
      const float4 *cw = reinterpret_cast<const float4 *>(a.conv) + c;
      float4 s = zero;
      if (STEP && short_conv) {
        float4 w[ROW_TAPS];
#pragma unroll
        for (int j = 0; j < ROW_TAPS; ++j) w[j] = j < a.taps ? __ldg(cw + (size_t)j * (a.ld >> 2)) : zero;
#pragma unroll
        for (int j = 0; j < ROW_TAPS; ++j) {
          if (j < a.taps - 1) {
            const float4 q = tl[STEP && j < ROW_TAPS - 1 ? j : 0][i];
            fma4(w[j], q, s);
            if (j > 0) Act<T>::st4(tp + (size_t)(j - 1) * a.ld, q);
          } else if (j == a.taps - 1) {
            fma4(w[j], h, s);
            if (j > 0) Act<T>::st4(tp + (size_t)(j - 1) * a.ld, h);
          }
        }
      } else {
        for (int j = 0; j < a.taps; ++j) {
          const float4 q = j + 1 < a.taps ? Act<T>::ld4(tp + (size_t)j * a.ld) : h;
          if (j > 0) Act<T>::st4(tp + (size_t)(j - 1) * a.ld, q);
          fma4(__ldg(cw + (size_t)j * (a.ld >> 2)), q, s);
        }
      }
      h.x += s.x; h.y += s.y; h.z += s.z; h.w += s.w;
    }
    Act<T>::st4(a.h + row0 + 4 * c, h);
  }
}

// ------------------------------------------------------- causal convolution ---
// c[b, i] = sum_j w[j] h[b, i - (taps - 1) + j] over a block of t positions per sequence (rows h_ld apart), rows before the
// block from tail_in [b][taps - 1][ld]; the block's own last taps - 1 rows go to tail_out (a different buffer).
// out[b, i] = h[b, i] + c[b, i], or with ACT silu(c[b, i] + bias).
// One thread per 8 channels and CONV_STRIP positions; with TAPS > 0 (the tap count, when it is small) the rows of the
// strip slide through registers, all of them requested before the first is used; TAPS = 0 takes any tap count.
constexpr int CONV_STRIP = 8;
constexpr int CONV_TAPS = 4;

template <typename T> struct Row8 { float v[8]; };
struct alignas(16) Raw32 { uint4 a, b; };
template <typename T> struct RawRow8 { using type = uint4; };
template <> struct RawRow8<float> { using type = Raw32; };
template <typename T> __device__ __forceinline__ Row8<T> ld8(const T *p) {
  Row8<T> r;
  if constexpr (sizeof(T) == 2) {
    const uint4 u = *reinterpret_cast<const uint4 *>(p);
    const __nv_bfloat162 *h = reinterpret_cast<const __nv_bfloat162 *>(&u);
#pragma unroll
    for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h[e]); r.v[2 * e] = f.x; r.v[2 * e + 1] = f.y; }
  } else {
    const float4 a = Act<T>::ld4(p), b = Act<T>::ld4(p + 4);
    r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w; r.v[4] = b.x; r.v[5] = b.y; r.v[6] = b.z; r.v[7] = b.w;
  }
  return r;
}
template <typename T> __device__ __forceinline__ void st8(T *p, const Row8<T> &r) {
  if constexpr (sizeof(T) == 2) {
    uint4 u;
    uint32_t *w = reinterpret_cast<uint32_t *>(&u);
#pragma unroll
    for (int e = 0; e < 4; ++e) { __nv_bfloat162 b = __floats2bfloat162_rn(r.v[2 * e], r.v[2 * e + 1]); w[e] = *(uint32_t *)&b; }
    *reinterpret_cast<uint4 *>(p) = u;
  } else {
    Act<T>::st4(p, make_float4(r.v[0], r.v[1], r.v[2], r.v[3]));
    Act<T>::st4(p + 4, make_float4(r.v[4], r.v[5], r.v[6], r.v[7]));
  }
}

template <typename T, int TAPS, bool ACT = false>
__global__ void __launch_bounds__(128)
causal_conv_kernel(const T *__restrict__ h, size_t h_ld, const float *__restrict__ w, const float *__restrict__ bias,
                   const T *__restrict__ tail_in, T *__restrict__ tail_out, T *__restrict__ out, int t, int taps_any, int ld) {
  const int taps = TAPS > 0 ? TAPS : taps_any;
  const int c = blockIdx.y * blockDim.x + threadIdx.x, b = blockIdx.z;
  if (c >= ld >> 3) return;
  const T *hb = h + (size_t)b * t * h_ld + 8 * c;
  const T *ti = tail_in + (size_t)b * (taps - 1) * ld + 8 * c;
  T *to = tail_out + (size_t)b * (taps - 1) * ld + 8 * c;
  T *ob = out + (size_t)b * t * ld + 8 * c;
  auto row = [&](int i) { return i >= 0 ? ld8<T>(hb + (size_t)i * h_ld) : ld8<T>(ti + (size_t)(i + taps - 1) * ld); };
  Row8<float> bv{};
  if constexpr (ACT) bv = ld8<float>(bias + 8 * c);
  auto finish = [&](Row8<T> &o, const Row8<T> &x) {        // x: the position itself, the convolution's last input
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      if constexpr (ACT) { const float s = o.v[e] + bv.v[e]; o.v[e] = s * sigmoid_t<sizeof(T) == 4>(s); }
      else o.v[e] += x.v[e];
    }
  };
  const int i0 = blockIdx.x * CONV_STRIP, i1 = min(i0 + CONV_STRIP, t);
  if constexpr (TAPS > 0) {
    using Raw = typename RawRow8<T>::type;                 // rows wait as they are stored and are widened when used
    Raw q[CONV_STRIP + TAPS - 1];
#pragma unroll
    for (int k = 0; k < CONV_STRIP + TAPS - 1; ++k) {
      const int i = i0 - (TAPS - 1) + k;
      if (i < i1) q[k] = *reinterpret_cast<const Raw *>(i >= 0 ? hb + (size_t)i * h_ld : ti + (size_t)(i + TAPS - 1) * ld);
    }
    Row8<float> wv[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wv[j] = ld8<float>(w + (size_t)j * ld + 8 * c);
#pragma unroll
    for (int k = 0; k < CONV_STRIP; ++k) {
      if (i0 + k >= i1) break;
      Row8<T> o{}, x;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        x = ld8<T>(reinterpret_cast<const T *>(&q[k + j]));
#pragma unroll
        for (int e = 0; e < 8; ++e) o.v[e] = fmaf(wv[j].v[e], x.v[e], o.v[e]);
      }
      finish(o, x);
      st8<T>(ob + (size_t)(i0 + k) * ld, o);
    }
  } else {
    for (int i = i0; i < i1; ++i) {
      Row8<T> own{}, o{};
      for (int j = 0; j < taps; ++j) {
        own = row(i - (taps - 1) + j);
        const Row8<float> wv = ld8<float>(w + (size_t)j * ld + 8 * c);
#pragma unroll
        for (int e = 0; e < 8; ++e) o.v[e] = fmaf(wv.v[e], own.v[e], o.v[e]);
      }
      finish(o, own);
      st8<T>(ob + (size_t)i * ld, o);
    }
  }
  if (i1 == t)
    for (int j = 0; j < taps - 1; ++j) st8<T>(to + (size_t)j * ld, row(t - (taps - 1) + j));
}

// ---------------------------------------------------------- minimal GRU -----
// pre [n_part][rows][3 ld]: z, u and gate pre-activations side by side (split-K partials of one projection);
//   S = (1 - z) S + z c(u),  out = S silu(g),  z = sigmoid(pre_z + bz), u = pre_u + bu
// One new position per sequence: one thread per 4 channels, state [rows][ld] in place.
template <typename T>
__global__ void __launch_bounds__(128)
min_gru_step_kernel(const float *__restrict__ pre, int n_part, size_t part_stride, const float *__restrict__ bz,
                    const float *__restrict__ bu, float *__restrict__ state, T *__restrict__ out, int ld) {
  const int r = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  const bool on = c < ld >> 2;
  float4 z = make_float4(0.f, 0.f, 0.f, 0.f), u = z, g = z;
  if (on) {
    z = __ldg(reinterpret_cast<const float4 *>(bz) + c);
    u = __ldg(reinterpret_cast<const float4 *>(bu) + c);
  }
  // the state was written a step ago, by a kernel that is certainly complete (see row_update_kernel)
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (on) S = *reinterpret_cast<const float4 *>(state + (size_t)r * ld + 4 * c);
  ugb_pdl_wait();
  ugb_pdl_trigger();
  if (!on) return;
  const float *row = pre + (size_t)r * 3 * ld + 4 * c;
  auto add = [](float4 &d, float4 s) { d.x += s.x; d.y += s.y; d.z += s.z; d.w += s.w; };
  for (int s = 0; s < n_part; s += 4) {
    float4 q[4][3];
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int k = 0; k < 3; ++k) {
        q[e][k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s + e < n_part) q[e][k] = __ldcs(reinterpret_cast<const float4 *>(row + (size_t)(s + e) * part_stride + (size_t)k * ld));
      }
#pragma unroll
    for (int e = 0; e < 4; ++e) { add(z, q[e][0]); add(u, q[e][1]); add(g, q[e][2]); }
  }
  auto step = [](float S0, float zp, float up) {
    const float zz = sigmoid_f(zp);
    return (1.0f - zz) * S0 + zz * gru_candidate<true>(up);
  };
  S = make_float4(step(S.x, z.x, u.x), step(S.y, z.y, u.y), step(S.z, z.z, u.z), step(S.w, z.w, u.w));
  *reinterpret_cast<float4 *>(state + (size_t)r * ld + 4 * c) = S;
  Act<T>::st4(out + (size_t)r * ld + 4 * c, make_float4(S.x * silu_f(g.x), S.y * silu_f(g.y), S.z * silu_f(g.z), S.w * silu_f(g.w)));
}

// A block of t positions per sequence as a scan over time.  A lane is a channel; a warp takes STEPS consecutive
// positions, a CTA SCAN_WARPS warps' worth, a cluster of CTAs (grid.x) consecutive pieces of the sequence.  Each warp
// composes its positions into one affine map S -> A S + B held in registers, the maps meet in shared memory (warps)
// and distributed shared memory (CTAs), and every warp then replays its positions from its own incoming state.  The
// cluster walks the sequence in rounds of BLOCK * gridDim.x positions; all CTAs run every round.
// bf16 pre-activations: a lane takes two adjacent channels, so a warp reads 128 bytes of a row either way.
constexpr int SCAN_WARPS = 8;
template <typename TI> struct Scan {
  static constexpr int V = sizeof(TI) == 2 ? 2 : 1;        // channels per lane
  static constexpr int STEPS = 8;                          // positions per warp and round
  static constexpr int BLOCK = SCAN_WARPS * STEPS, COLUMNS = 32 * V;
};

// a lane's channels of one pre-activation row, as stored (32 bits either way)
template <int V> __device__ __forceinline__ void scan_widen(uint32_t raw, float (&f)[V]) {
  if constexpr (V == 2) {
    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&raw));
    f[0] = x.x; f[1] = x.y;
  } else f[0] = __uint_as_float(raw);
}

template <typename TI, typename T>
__global__ void __launch_bounds__(SCAN_WARPS * 32, 2)
min_gru_scan_kernel(const TI *__restrict__ pre, const float *__restrict__ bz, const float *__restrict__ bu,
                    float *__restrict__ state, T *__restrict__ out, int t, int ld) {
  constexpr int V = Scan<TI>::V, STEPS = Scan<TI>::STEPS, BLOCK = Scan<TI>::BLOCK, COLS = Scan<TI>::COLUMNS;
  constexpr bool EXACT = sizeof(T) == 4;
  __shared__ float agg_a[SCAN_WARPS][COLS], agg_b[SCAN_WARPS][COLS];
  __shared__ float tot[2][2][COLS];                        // [round parity][A, B][channel], read by the cluster
  __shared__ float enter[SCAN_WARPS][COLS];                // state entering each warp's positions
  __shared__ float carry[COLS];                            // state before the round
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int rank = blockIdx.x, n_cta = gridDim.x, b = blockIdx.z;
  const int c = blockIdx.y * COLS + lane * V;              // ld is a multiple of 8: a lane's channels are all in or all out
  const bool on = c < ld;
  float zb[V], ub[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    zb[e] = on ? bz[c + e] : 0.f;
    ub[e] = on ? bu[c + e] : 0.f;
  }
  if (threadIdx.x < COLS) {
    const int k = blockIdx.y * COLS + threadIdx.x;
    carry[threadIdx.x] = k < ld ? state[(size_t)b * ld + k] : 0.f;
  }
  const size_t base = (size_t)b * t;
  const TI *mine = pre + base * (size_t)(3 * ld) + c;
  uint32_t nz[STEPS], nu[STEPS], ng[STEPS];                // the coming round's rows, requested a round ahead
  auto fetch = [&](int i0) {
#pragma unroll
    for (int s = 0; s < STEPS; ++s) {
      nz[s] = nu[s] = ng[s] = 0u;
      if (on && i0 + s < t) {
        const TI *row = mine + (size_t)(i0 + s) * (3 * ld);
        nz[s] = __ldcs(reinterpret_cast<const uint32_t *>(row));
        nu[s] = __ldcs(reinterpret_cast<const uint32_t *>(row + ld));
        ng[s] = __ldcs(reinterpret_cast<const uint32_t *>(row + 2 * ld));
      }
    }
  };
  fetch(rank * BLOCK + warp * STEPS);
  int round = 0;
  for (int t0 = 0; t0 < t; t0 += BLOCK * n_cta, ++round) {
    const int i0 = t0 + rank * BLOCK + warp * STEPS;
    const bool whole = i0 + STEPS <= t;
    float a[STEPS][V], bb[STEPS][V];
    uint32_t g[STEPS];
#pragma unroll
    for (int s = 0; s < STEPS; ++s) { scan_widen<V>(nz[s], a[s]); scan_widen<V>(nu[s], bb[s]); g[s] = ng[s]; }
    fetch(i0 + BLOCK * n_cta);
    float A[V], B[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      A[e] = 1.f; B[e] = 0.f;
#pragma unroll
      for (int s = 0; s < STEPS; ++s) {
        const float z = sigmoid_t<EXACT>(a[s][e] + zb[e]);
        a[s][e] = 1.0f - z;
        bb[s][e] = z * gru_candidate<EXACT>(bb[s][e] + ub[e]);
        if (!whole && i0 + s >= t) { a[s][e] = 1.0f; bb[s][e] = 0.0f; }   // behind the block: leaves the state alone
        A[e] *= a[s][e];
        B[e] = fmaf(a[s][e], B[e], bb[s][e]);
      }
      // (the round before has left these arrays: all read them before its last barrier)
      agg_a[warp][lane * V + e] = A[e]; agg_b[warp][lane * V + e] = B[e];
    }
    __syncthreads();
    if (threadIdx.x < COLS) {                              // this CTA's map, a thread per channel
      float TA = 1.f, TB = 0.f;
#pragma unroll
      for (int w = 0; w < SCAN_WARPS; ++w) { TB = fmaf(agg_a[w][threadIdx.x], TB, agg_b[w][threadIdx.x]); TA *= agg_a[w][threadIdx.x]; }
      tot[round & 1][0][threadIdx.x] = TA; tot[round & 1][1][threadIdx.x] = TB;
    }
    // the parity of `tot` alternates, so one barrier per round separates a round's writes from the reads of the
    // round before the last
    if (n_cta > 1) ugb_tc::cluster_sync_all();
    if (threadIdx.x < COLS) {
      float in = carry[threadIdx.x], R = in;
      const uint32_t pa = ugb_tc::smem_u32(&tot[round & 1][0][threadIdx.x]), pb = ugb_tc::smem_u32(&tot[round & 1][1][threadIdx.x]);
      float va[8], vb[8];                                  // every CTA's map is requested before the first is used
#pragma unroll
      for (int q = 0; q < 8; ++q) {
        va[q] = 1.f; vb[q] = 0.f;
        if (q < n_cta) {
          asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(va[q]) : "r"(ugb_tc::mapa_u32(pa, (uint32_t)q)) : "memory");
          asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(vb[q]) : "r"(ugb_tc::mapa_u32(pb, (uint32_t)q)) : "memory");
        }
      }
#pragma unroll
      for (int q = 0; q < 8; ++q) {
        if (q == rank) in = R;                             // state entering this CTA's piece
        R = fmaf(va[q], R, vb[q]);
      }
      carry[threadIdx.x] = R;
#pragma unroll
      for (int w = 0; w < SCAN_WARPS; ++w) {
        enter[w][threadIdx.x] = in;
        in = fmaf(agg_a[w][threadIdx.x], in, agg_b[w][threadIdx.x]);
      }
    }
    __syncthreads();
    float S[V];
#pragma unroll
    for (int e = 0; e < V; ++e) S[e] = enter[warp][lane * V + e];
#pragma unroll
    for (int s = 0; s < STEPS; ++s) {
#pragma unroll
      for (int e = 0; e < V; ++e) S[e] = fmaf(a[s][e], S[e], bb[s][e]);
      float sg[V];
      scan_widen<V>(g[s], sg);
#pragma unroll
      for (int e = 0; e < V; ++e) sg[e] *= sigmoid_t<EXACT>(sg[e]);
      if (on && (whole || i0 + s < t)) {
        T *o = out + (base + i0 + s) * (size_t)ld + c;
        if constexpr (sizeof(T) == 4) {
#pragma unroll
          for (int e = 0; e < V; ++e) o[e] = S[e] * sg[e];
        } else if constexpr (V == 2) {
          *reinterpret_cast<__nv_bfloat162 *>(o) = __floats2bfloat162_rn(S[0] * sg[0], S[1] * sg[1]);
        } else {
          *o = __float2bfloat16_rn(S[0] * sg[0]);
        }
      }
    }
  }
  ugb_tc::cluster_sync_all();                              // no CTA leaves (or writes the state) while a peer still reads
  if (rank == 0 && threadIdx.x < COLS) {
    const int k = blockIdx.y * COLS + threadIdx.x;
    if (k < ld) state[(size_t)b * ld + k] = carry[threadIdx.x];
  }
}

// ------------------------------------------------- latent attention inputs ---
// pre [n_part][rows][q_ld + c_ld + g_ld]: query latent, key/value latent and head gates of one projection.
//   cq[r] = norm(query latent) * q_gain   cache[b][pos] = norm(kv latent) * c_gain   gate[r] = sigmoid(head gate)
// row r = (b, i) = (r / t, r % t), pos = *pos_p + pos_off + i.  One CTA of up to 512 threads per row, PER groups of 4
// columns per thread (the segments are multiples of 8 wide), U split-K partials in flight.
template <typename T, int PER, int U>
__global__ void __launch_bounds__(512)
latent_inputs_kernel(const float *__restrict__ pre, int n_part, size_t part_stride, const float *__restrict__ q_gain,
                     const float *__restrict__ c_gain, T *__restrict__ cq, T *__restrict__ cache, float *__restrict__ gate,
                     const int *__restrict__ pos_p, int pos_off, int t, int t_max, int q_ld, int c_ld, int g_ld,
                     float inv_q, float inv_c, float eps, ugb_status_word *status) {
  __shared__ float sm[2][16];
  const int r = blockIdx.x, n = q_ld + c_ld + g_ld, tid = threadIdx.x, bd = blockDim.x;
  const int b = r / t, off = pos_off + r % t;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 y[PER], w[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int c = 4 * (tid + i * bd);
    y[i] = w[i] = zero;
    if (c < q_ld) w[i] = __ldg(reinterpret_cast<const float4 *>(q_gain + c));
    else if (c < q_ld + c_ld) w[i] = __ldg(reinterpret_cast<const float4 *>(c_gain + c - q_ld));
  }
  ugb_pdl_wait();
  ugb_pdl_trigger();
  const int pos = *pos_p + off;
  for (int s = 0; s < n_part; s += U) {                    // the partials are added in order
    float4 q[U][PER];
#pragma unroll
    for (int e = 0; e < U; ++e)
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int c = tid + i * bd;
        q[e][i] = zero;
        if (s + e < n_part && c < n >> 2)
          q[e][i] = __ldcs(reinterpret_cast<const float4 *>(pre + (size_t)(s + e) * part_stride + (size_t)r * n) + c);
      }
#pragma unroll
    for (int e = 0; e < U; ++e)
#pragma unroll
      for (int i = 0; i < PER; ++i) { y[i].x += q[e][i].x; y[i].y += q[e][i].y; y[i].z += q[e][i].z; y[i].w += q[e][i].w; }
  }
  float sq = 0.f, sc = 0.f;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int c = 4 * (tid + i * bd);
    if (c < q_ld) sq += sq4(y[i]);
    else if (c < q_ld + c_ld) sc += sq4(y[i]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sc += __shfl_xor_sync(0xffffffffu, sc, o);
  }
  if ((tid & 31) == 0) { sm[0][tid >> 5] = sq; sm[1][tid >> 5] = sc; }
  __syncthreads();
  sq = sc = 0.f;
  for (int i = 0; i < bd >> 5; ++i) { sq += sm[0][i]; sc += sm[1][i]; }
  const float rq = 1.0f / sqrtf(sq * inv_q + eps), rc = 1.0f / sqrtf(sc * inv_c + eps);
  const bool ok = pos >= 0 && pos < t_max;
  if (!ok && tid == 0 && atomicCAS(&status->code, 0u, (unsigned)UGB_ERR_INVALID) == 0u) status->detail = (unsigned)pos;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int c = 4 * (tid + i * bd);
    if (c < q_ld) {
      Act<T>::st4(cq + (size_t)r * q_ld + c, make_float4(y[i].x * rq * w[i].x, y[i].y * rq * w[i].y, y[i].z * rq * w[i].z, y[i].w * rq * w[i].w));
    } else if (c < q_ld + c_ld) {
      if (ok) Act<T>::st4(cache + ((size_t)b * t_max + pos) * c_ld + c - q_ld,
                          make_float4(y[i].x * rc * w[i].x, y[i].y * rc * w[i].y, y[i].z * rc * w[i].z, y[i].w * rc * w[i].w));
    } else if (c < n) {
      *reinterpret_cast<float4 *>(gate + (size_t)r * g_ld + c - q_ld - c_ld) =
          make_float4(sigmoid_f(y[i].x), sigmoid_f(y[i].y), sigmoid_f(y[i].z), sigmoid_f(y[i].w));
    }
  }
}

// max(x, 0)^2 in place, the unfused form of UGB_EPI_RELU2_BF16 for 32-bit activations
static __global__ void relu2_kernel(float *__restrict__ x, size_t n4) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n4; i += (size_t)gridDim.x * blockDim.x) {
    float4 v = reinterpret_cast<float4 *>(x)[i];
    v.x = fmaxf(v.x, 0.f); v.y = fmaxf(v.y, 0.f); v.z = fmaxf(v.z, 0.f); v.w = fmaxf(v.w, 0.f);
    reinterpret_cast<float4 *>(x)[i] = make_float4(v.x * v.x, v.y * v.y, v.z * v.z, v.w * v.w);
  }
}

// ---------------------------------------------------------------- loading ----
// gain[i] = offset + w[i], zero behind n
static __global__ void gain_kernel(const float *__restrict__ w, float *__restrict__ gain, int n, float offset) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) gain[i] = offset + w[i];
}
// conv weights [width][taps] -> [taps][ld]
static __global__ void taps_kernel(const float *__restrict__ w, float *__restrict__ out, int width, int taps, int ld) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < width * taps) out[(size_t)(i % taps) * ld + i / taps] = w[i];
}

}  // namespace ugb_hybrid_k
