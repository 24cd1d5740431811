// Row kernels of the layer-list engine (hybrid_engine.cu): everything between the matrix products of a decoder whose
// layers are recurrent or latent-attention mixers with sandwich norms, input convolutions and a depth average.
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

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
// candidate of the minimal gated recurrent unit: u + 1/2 for u >= 0, sigmoid(u) below
__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.0f ? u + 0.5f : sigmoid_f(u); }

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
//   y   = sum of the projection partials, or the embedding row of token id(r)
//   x   = x + norm(y) * post_gain          (post_gain null: y itself; add_x 0: the stream starts here)
//   bank_out = x;  x = sum_j dwa[j] bank[j] + dwa[n_avg] x        (with a depth average)
//   h   = norm(x) * gain, rounded to T
//   h   = h + sum_j conv[j] h_(-taps+1+j)  (conv set: one new position per sequence; the tail of earlier h's is the
//                                           sequence's state and moves on by one)
template <typename T> struct RowArgs {
  const int *tok = nullptr;            // embedding source: row r = (r / t, r % t) reads tok[(r / t) * tok_stride + tok_off + r % t]
  const T *embed = nullptr;
  int vocab = 0, t = 1, tok_stride = 1, tok_off = 0;
  const float *part = nullptr;         // or projection partials [n_part][rows][ld]
  int n_part = 0;
  size_t part_stride = 0;
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
  const float *conv = nullptr;         // [taps][ld]
  int taps = 0;
  T *tail = nullptr;                   // [rows][taps - 1][ld]
  int ld = 0;
  float inv_width = 0.f, eps = 0.f;
  ugb_status_word *status = nullptr;
};

template <typename T, int VPT>
__global__ void __launch_bounds__(256)
row_update_kernel(RowArgs<T> a) {
  __shared__ float sm[8];
  ugb_pdl_trigger();
  // gains and taps are weights: fetched before the wait for the preceding kernel
  const int r = blockIdx.x, nvec = a.ld >> 2;
  float4 pg[VPT], g2[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    pg[i] = make_float4(1.f, 1.f, 1.f, 1.f);
    g2[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < nvec) {
      if (a.post_gain) pg[i] = __ldg(reinterpret_cast<const float4 *>(a.post_gain) + c);
      g2[i] = __ldg(reinterpret_cast<const float4 *>(a.gain) + c);
    }
  }
  ugb_pdl_wait();
  float4 v[VPT], y[VPT];
  float4 *xr = reinterpret_cast<float4 *>(a.x + (size_t)r * a.ld);
  const T *erow = nullptr;
  if (a.tok) {
    const int id = a.tok[(size_t)(r / a.t) * a.tok_stride + a.tok_off + r % a.t];
    if (id < 0 || id >= a.vocab) {
      if (threadIdx.x == 0 && atomicCAS(&a.status->code, 0u, (unsigned)UGB_ERR_INVALID) == 0u) a.status->detail = r;
      return;
    }
    erow = a.embed + (size_t)id * a.ld;
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    v[i] = y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < nvec) {
      if (a.add_x) v[i] = xr[c];
      if (erow) y[i] = Act<T>::ld4(erow + 4 * c);
      else y[i] = __ldcs(reinterpret_cast<const float4 *>(a.part + (size_t)r * a.ld) + c);
    }
  }
  if (!erow && a.n_part > 1) {
    for (int s = 1; s < a.n_part; s += 4) {               // split-K partials in order, four round trips in flight
      float4 q[4][VPT];
#pragma unroll
      for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int c = threadIdx.x + i * 256;
          q[u][i] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (c < nvec && s + u < a.n_part)
            q[u][i] = __ldcs(reinterpret_cast<const float4 *>(a.part + (size_t)(s + u) * a.part_stride + (size_t)r * a.ld) + c);
        }
#pragma unroll
      for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int i = 0; i < VPT; ++i) { y[i].x += q[u][i].x; y[i].y += q[u][i].y; y[i].z += q[u][i].z; y[i].w += q[u][i].w; }
    }
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
    float4 *bo = reinterpret_cast<float4 *>(a.bank_out + (size_t)r * a.ld);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c < nvec) bo[c] = v[i];
    }
  }
  if (a.dwa) {
    const float own = __ldg(a.dwa + a.n_avg);
    float4 acc[VPT];
#pragma unroll
    for (int i = 0; i < VPT; ++i) acc[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    constexpr int U = VPT <= 2 ? 8 : (VPT <= 4 ? 4 : 2);  // bank rows in flight
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
          q[u][i] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (on && c < nvec) q[u][i] = __ldcg(reinterpret_cast<const float4 *>(a.bank + (size_t)(j + u) * a.bank_stride + (size_t)r * a.ld) + c);
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
    ss += sq4(v[i]);
  }
  const float inv2 = 1.0f / sqrtf(block_sum_256(ss, sm) * a.inv_width + a.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c >= nvec) continue;
    float4 h = make_float4(v[i].x * inv2 * g2[i].x, v[i].y * inv2 * g2[i].y, v[i].z * inv2 * g2[i].z, v[i].w * inv2 * g2[i].w);
    if (a.conv) {
      // what the convolution sees, now and later, is the rounded h
      h = make_float4(Act<T>::round(h.x), Act<T>::round(h.y), Act<T>::round(h.z), Act<T>::round(h.w));
      T *tl = a.tail + (size_t)r * (a.taps - 1) * a.ld + 4 * c;
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int j = 0; j < a.taps; ++j) {
        const float4 w = __ldg(reinterpret_cast<const float4 *>(a.conv + (size_t)j * a.ld) + c);
        const float4 q = j + 1 < a.taps ? Act<T>::ld4(tl + (size_t)j * a.ld) : h;
        if (j > 0) Act<T>::st4(tl + (size_t)(j - 1) * a.ld, q);
        s.x = fmaf(w.x, q.x, s.x); s.y = fmaf(w.y, q.y, s.y); s.z = fmaf(w.z, q.z, s.z); s.w = fmaf(w.w, q.w, s.w);
      }
      h.x += s.x; h.y += s.y; h.z += s.z; h.w += s.w;
    }
    Act<T>::st4(a.h + (size_t)r * a.ld + 4 * c, h);
  }
}

// ------------------------------------------------- causal input convolution ---
// out[b, i] = h[b, i] + sum_j w[j] h[b, i - (taps - 1) + j] over a block of t positions per sequence, rows before the
// block from tail_in [b][taps - 1][ld]; the block's own last taps - 1 rows go to tail_out (a different buffer).
// One thread per 4 channels and CONV_STRIP positions: a row of h is fetched once per tap from L1.
constexpr int CONV_STRIP = 8;

template <typename T>
__global__ void __launch_bounds__(256)
causal_conv_kernel(const T *__restrict__ h, const float *__restrict__ w, const T *__restrict__ tail_in, T *__restrict__ tail_out,
                   T *__restrict__ out, int t, int taps, int ld) {
  const int c = blockIdx.y * blockDim.x + threadIdx.x, b = blockIdx.z;
  if (c >= ld >> 2) return;
  const T *hb = h + (size_t)b * t * ld + 4 * c;
  const T *ti = tail_in + (size_t)b * (taps - 1) * ld + 4 * c;
  T *to = tail_out + (size_t)b * (taps - 1) * ld + 4 * c;
  auto row = [&](int i) { return i >= 0 ? Act<T>::ld4(hb + (size_t)i * ld) : Act<T>::ld4(ti + (size_t)(i + taps - 1) * ld); };
  const int i0 = blockIdx.x * CONV_STRIP, i1 = min(i0 + CONV_STRIP, t);
#pragma unroll 4
  for (int i = i0; i < i1; ++i) {
    float4 own = make_float4(0.f, 0.f, 0.f, 0.f), s = own;
    for (int j = 0; j < taps; ++j) {
      const float4 q = row(i - (taps - 1) + j);
      const float4 wv = __ldg(reinterpret_cast<const float4 *>(w + (size_t)j * ld) + c);
      s.x = fmaf(wv.x, q.x, s.x); s.y = fmaf(wv.y, q.y, s.y); s.z = fmaf(wv.z, q.z, s.z); s.w = fmaf(wv.w, q.w, s.w);
      own = q;                                             // the last tap is position i itself
    }
    Act<T>::st4(out + ((size_t)b * t + i) * ld + 4 * c, make_float4(own.x + s.x, own.y + s.y, own.z + s.z, own.w + s.w));
  }
  if (i1 == t)
    for (int j = 0; j < taps - 1; ++j) Act<T>::st4(to + (size_t)j * ld, row(t - (taps - 1) + j));
}

// ---------------------------------------------------------- minimal GRU -----
// pre [n_part][rows][3 ld]: z, u and gate pre-activations side by side (split-K partials of one projection);
//   S = (1 - z) S + z c(u),  out = S silu(g),  z = sigmoid(pre_z + bz), u = pre_u + bu
// One new position per sequence: one thread per 4 channels, state [rows][ld] in place.
template <typename T>
__global__ void __launch_bounds__(128)
min_gru_step_kernel(const float *__restrict__ pre, int n_part, size_t part_stride, const float *__restrict__ bz,
                    const float *__restrict__ bu, float *__restrict__ state, T *__restrict__ out, int ld) {
  ugb_pdl_trigger();
  const int r = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  const bool on = c < ld >> 2;
  float4 z = make_float4(0.f, 0.f, 0.f, 0.f), u = z, g = z;
  if (on) {
    z = __ldg(reinterpret_cast<const float4 *>(bz) + c);
    u = __ldg(reinterpret_cast<const float4 *>(bu) + c);
  }
  ugb_pdl_wait();
  if (!on) return;
  const float *row = pre + (size_t)r * 3 * ld + 4 * c;
  float4 S = *reinterpret_cast<const float4 *>(state + (size_t)r * ld + 4 * c);
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
    return (1.0f - zz) * S0 + zz * gru_candidate(up);
  };
  S = make_float4(step(S.x, z.x, u.x), step(S.y, z.y, u.y), step(S.z, z.z, u.z), step(S.w, z.w, u.w));
  *reinterpret_cast<float4 *>(state + (size_t)r * ld + 4 * c) = S;
  Act<T>::st4(out + (size_t)r * ld + 4 * c, make_float4(S.x * silu_f(g.x), S.y * silu_f(g.y), S.z * silu_f(g.z), S.w * silu_f(g.w)));
}

// A block of t positions per sequence as a scan over time.  A lane is a channel; a warp takes SCAN_STEPS consecutive
// positions, a CTA SCAN_WARPS warps' worth, a cluster of CTAs (grid.x) consecutive pieces of the sequence.  Each warp
// composes its positions into one affine map S -> A S + B held in registers, the maps meet in shared memory (warps)
// and distributed shared memory (CTAs), and every warp then replays its positions from its own incoming state.  The
// cluster walks the sequence in rounds of SCAN_BLOCK * gridDim.x positions; all CTAs run every round.
constexpr int SCAN_WARPS = 16, SCAN_STEPS = 8, SCAN_BLOCK = SCAN_WARPS * SCAN_STEPS;

template <typename TI> __device__ __forceinline__ float scan_load(const TI *p) { return (float)*p; }

template <typename TI, typename T>
__global__ void __launch_bounds__(SCAN_WARPS * 32)
min_gru_scan_kernel(const TI *__restrict__ pre, const float *__restrict__ bz, const float *__restrict__ bu,
                    float *__restrict__ state, T *__restrict__ out, int t, int ld) {
  __shared__ float agg_a[SCAN_WARPS][32], agg_b[SCAN_WARPS][32];
  __shared__ float tot[2][2][32];                          // [round parity][A, B][channel], read by the cluster
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int rank = blockIdx.x, n_cta = gridDim.x, b = blockIdx.z;
  const int c = blockIdx.y * 32 + lane;
  const bool on = c < ld;
  const float zb = on ? bz[c] : 0.f, ub = on ? bu[c] : 0.f;
  const size_t base = (size_t)b * t;
  float carry = on ? state[(size_t)b * ld + c] : 0.f;      // state before this round (every warp of every CTA keeps it)
  int round = 0;
  for (int t0 = 0; t0 < t; t0 += SCAN_BLOCK * n_cta, ++round) {
    const int i0 = t0 + rank * SCAN_BLOCK + warp * SCAN_STEPS;
    float a[SCAN_STEPS], bb[SCAN_STEPS], sg[SCAN_STEPS];
#pragma unroll
    for (int s = 0; s < SCAN_STEPS; ++s) {
      a[s] = bb[s] = sg[s] = 0.f;
      if (on && i0 + s < t) {
        const TI *row = pre + (base + i0 + s) * (size_t)(3 * ld) + c;
        a[s] = scan_load(row); bb[s] = scan_load(row + ld); sg[s] = scan_load(row + 2 * ld);
      }
    }
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int s = 0; s < SCAN_STEPS; ++s) {
      if (on && i0 + s < t) {
        const float z = sigmoid_f(a[s] + zb);
        a[s] = 1.0f - z;
        bb[s] = z * gru_candidate(bb[s] + ub);
        sg[s] = silu_f(sg[s]);
      } else { a[s] = 1.f; bb[s] = 0.f; sg[s] = 0.f; }
      A *= a[s];
      B = fmaf(a[s], B, bb[s]);
    }
    agg_a[warp][lane] = A; agg_b[warp][lane] = B;
    __syncthreads();
    if (warp == 0) {                                       // this CTA's map
      float TA = 1.f, TB = 0.f;
#pragma unroll
      for (int w = 0; w < SCAN_WARPS; ++w) { TB = fmaf(agg_a[w][lane], TB, agg_b[w][lane]); TA *= agg_a[w][lane]; }
      tot[round & 1][0][lane] = TA; tot[round & 1][1][lane] = TB;
    }
    // the parity of `tot` alternates, so one barrier per round separates a round's writes from the reads of the
    // round before the last
    ugb_tc::cluster_sync_all();
    float in = carry, S = carry;
    for (int q = 0; q < n_cta; ++q) {
      const uint32_t ra = ugb_tc::mapa_u32(ugb_tc::smem_u32(&tot[round & 1][0][lane]), (uint32_t)q);
      const uint32_t rb = ugb_tc::mapa_u32(ugb_tc::smem_u32(&tot[round & 1][1][lane]), (uint32_t)q);
      float va, vb;
      asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(va) : "r"(ra) : "memory");
      asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(vb) : "r"(rb) : "memory");
      if (q == rank) in = S;                               // state entering this CTA's piece
      S = fmaf(va, S, vb);
    }
    carry = S;
    S = in;
    for (int w = 0; w < warp; ++w) S = fmaf(agg_a[w][lane], S, agg_b[w][lane]);
#pragma unroll
    for (int s = 0; s < SCAN_STEPS; ++s) {
      S = fmaf(a[s], S, bb[s]);
      if (on && i0 + s < t) {
        if constexpr (sizeof(T) == 4) out[(base + i0 + s) * (size_t)ld + c] = S * sg[s];
        else out[(base + i0 + s) * (size_t)ld + c] = __float2bfloat16_rn(S * sg[s]);
      }
    }
    __syncthreads();                                       // agg_a / agg_b are free
  }
  ugb_tc::cluster_sync_all();                              // no CTA leaves (or writes the state) while a peer still reads
  if (on && rank == 0 && warp == 0) state[(size_t)b * ld + c] = carry;
}

// ------------------------------------------------- latent attention inputs ---
// pre [n_part][rows][q_ld + c_ld + g_ld]: query latent, key/value latent and head gates of one projection.
//   cq[r] = norm(query latent) * q_gain   cache[b][pos] = norm(kv latent) * c_gain   gate[r] = sigmoid(head gate)
// row r = (b, i) = (r / t, r % t), pos = *pos_p + pos_off + i.  One CTA of 256 threads per row.
template <typename T>
__global__ void __launch_bounds__(256)
latent_inputs_kernel(const float *__restrict__ pre, int n_part, size_t part_stride, const float *__restrict__ q_gain,
                     const float *__restrict__ c_gain, T *__restrict__ cq, T *__restrict__ cache, float *__restrict__ gate,
                     const int *__restrict__ pos_p, int pos_off, int t, int t_max, int q_ld, int c_ld, int g_ld,
                     float inv_q, float inv_c, float eps, ugb_status_word *status) {
  extern __shared__ __align__(16) float row_s[];
  __shared__ float sm[8];
  ugb_pdl_trigger();
  ugb_pdl_wait();
  const int r = blockIdx.x, n = q_ld + c_ld + g_ld, tid = threadIdx.x;
  float sq = 0.f, sc = 0.f;
  for (int c = tid; c < n >> 2; c += 256) {
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < n_part; s += 4) {
      float4 q[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        q[e] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s + e < n_part) q[e] = __ldcs(reinterpret_cast<const float4 *>(pre + (size_t)(s + e) * part_stride + (size_t)r * n) + c);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) { y.x += q[e].x; y.y += q[e].y; y.z += q[e].z; y.w += q[e].w; }
    }
    reinterpret_cast<float4 *>(row_s)[c] = y;
    if (4 * c < q_ld) sq += sq4(y);                        // the segments are multiples of 8 wide
    else if (4 * c < q_ld + c_ld) sc += sq4(y);
  }
  const float rq = 1.0f / sqrtf(block_sum_256(sq, sm) * inv_q + eps);
  const float rc = 1.0f / sqrtf(block_sum_256(sc, sm) * inv_c + eps);   // its barriers also publish row_s
  const int b = r / t, pos = *pos_p + pos_off + r % t;
  const bool ok = pos >= 0 && pos < t_max;
  if (!ok && tid == 0 && atomicCAS(&status->code, 0u, (unsigned)UGB_ERR_INVALID) == 0u) status->detail = (unsigned)pos;
  for (int c = tid; c < n >> 2; c += 256) {
    const float4 y = reinterpret_cast<const float4 *>(row_s)[c];
    if (4 * c < q_ld) {
      const float4 w = __ldg(reinterpret_cast<const float4 *>(q_gain) + c);
      Act<T>::st4(cq + (size_t)r * q_ld + 4 * c, make_float4(y.x * rq * w.x, y.y * rq * w.y, y.z * rq * w.z, y.w * rq * w.w));
    } else if (4 * c < q_ld + c_ld) {
      const int k = 4 * c - q_ld;
      const float4 w = __ldg(reinterpret_cast<const float4 *>(c_gain + k));
      if (ok) Act<T>::st4(cache + ((size_t)b * t_max + pos) * c_ld + k, make_float4(y.x * rc * w.x, y.y * rc * w.y, y.z * rc * w.z, y.w * rc * w.w));
    } else {
      const int k = 4 * c - q_ld - c_ld;
      *reinterpret_cast<float4 *>(gate + (size_t)r * g_ld + k) = make_float4(sigmoid_f(y.x), sigmoid_f(y.y), sigmoid_f(y.z), sigmoid_f(y.w));
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

}  // namespace ugb_hybrid_k
