// Row kernels of layers in the parallel form (hybrid_parallel.cu): what lies between the input projection of a layer and
// its attention, scan and experts, and the token input behind a layer.  T is the activation type; rotations, norms,
// router scores and gates are f32 whatever T is.
#pragma once
#include "hybrid_kernels.cuh"

namespace ugb_hybrid_k {

// ------------------------------------------------------------ mixer inputs ---
// One row of a layer's input projection, columns q heads | k heads | v heads | x | z | router:
//   q, k   rotary positions on the first rot_dims dimensions, then (qk_norm) divided by the root mean square of the
//          head; q -> q_out, k -> key cache          v -> value cache
// and, in a step (one new position per sequence),
//   x      causal convolution over the sequence's last taps inputs, bias, silu -> u; the tail moves on by one
//   router -> choice of experts
// Row r = (b, i) = (r / t, r % t) at position *pos_p + pos_off + i.  The projection is a sum of f32 partials in a step,
// one T row in a block.
constexpr int HEAD_DIM_MAX = 256;      // a lane takes 8 dimensions of a head
constexpr int ROUTER_PER_LANE = 8;     // up to 256 experts

template <typename TI, typename T> struct MixerIn {
  const TI *pre = nullptr;
  int n_part = 1;
  size_t part_stride = 0;
  int ld = 0, t = 1, pos_off = 0, t_max = 0;
  const int *pos_p = nullptr;
  int heads = 0, kv_heads = 0, dim = 0, dp = 0, vp = 0, rot_dims = 0, interleaved = 1, qk_norm = 0;
  float eps = 0.f;
  const float *cos_ = nullptr, *sin_ = nullptr;            // [t_max][rot_dims / 2]
  T *q = nullptr, *kcache = nullptr, *vcache = nullptr;    // [rows][heads][dp], [b][kv_heads][t_max][dp / vp]
  // a step
  const float *conv_w = nullptr, *conv_b = nullptr;        // [taps][ci], [ci]
  int taps = 0, ci = 0;
  T *tail = nullptr, *u = nullptr;                         // [rows][taps - 1][ci], [rows][ci]
  int experts = 0, top = 0;
  float4 *choice = nullptr;                                // [rows][top]
  int *count = nullptr;                                    // [experts]
  ugb_status_word *status = nullptr;
};

// Experts with the `top` largest scores of one row, best first (ties: the lower index): lane l holds the logits of experts
// l, l + 32, ... and every lane returns the pick; `use` is called by all lanes with (k, expert, its logit).
template <typename F>
__device__ __forceinline__ void top_experts(float (&z)[ROUTER_PER_LANE], int experts, int top, F use) {
  const int lane = threadIdx.x & 31;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
#pragma unroll
    for (int j = 0; j < ROUTER_PER_LANE; ++j)
      if (z[j] > best) { best = z[j]; at = lane + 32 * j; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, at, o);
      if (ov > best || (ov == best && oi < at)) { best = ov; at = oi; }
    }
    if (at >= experts) at = k;                             // not-a-number logits: still an expert that exists
#pragma unroll
    for (int j = 0; j < ROUTER_PER_LANE; ++j)
      if (at == lane + 32 * j) z[j] = -INFINITY;
    use(k, at, best);
  }
}

// Lanes of a warp that share a head: 8 dimensions each, rounded up to a power of two.
__host__ __device__ __forceinline__ int head_lanes(int dp) {
  int n = 1;
  while (8 * n < dp) n *= 2;
  return n;
}
// Warps' worth of work in a row: groups of heads, pieces of 256 values, in a step pieces of 128 scan inputs and the router.
struct MixerUnits { int heads, v, x, all; };
template <bool STEP> __host__ __device__ __forceinline__ MixerUnits mixer_units(int heads, int dp, int v, int ci, int experts) {
  MixerUnits n;
  const int per = 32 / head_lanes(dp);
  n.heads = (heads + per - 1) / per;
  n.v = (v + 255) / 256;
  n.x = STEP ? (ci + 127) / 128 : 0;
  n.all = n.heads + n.v + n.x + (STEP && experts > 0 ? 1 : 0);
  return n;
}

template <typename TI, typename T, bool STEP>
__global__ void __launch_bounds__(256)
mixer_inputs_kernel(MixerIn<TI, T> a, int rows) {
  const int n_head = a.heads + a.kv_heads;
  const MixerUnits n = mixer_units<STEP>(n_head, a.dp, a.kv_heads * a.vp, a.ci, a.experts);
  const int id = blockIdx.x * 8 + (threadIdx.x >> 5), r = id / n.all, unit = id - r * n.all, lane = threadIdx.x & 31;
  ugb_pdl_wait();
  ugb_pdl_trigger();
  if (r >= rows) return;
  const int b = r / a.t;
  const TI *row = a.pre + (size_t)r * a.ld;
  auto sum4 = [&](int c) {                                 // the partials are added in order
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int p = 0; p < a.n_part; p += 4) {
      float4 v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = p + e < a.n_part ? Act<TI>::ld4(row + (size_t)(p + e) * a.part_stride + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int e = 0; e < 4; ++e) { s.x += v[e].x; s.y += v[e].y; s.z += v[e].z; s.w += v[e].w; }
    }
    return s;
  };
  auto sum8 = [&](int c) {
    if constexpr (!STEP) return ld8<TI>(row + c);
    Row8<TI> s;
    const float4 x = sum4(c), y = sum4(c + 4);
    s.v[0] = x.x; s.v[1] = x.y; s.v[2] = x.z; s.v[3] = x.w; s.v[4] = y.x; s.v[5] = y.y; s.v[6] = y.z; s.v[7] = y.w;
    return s;
  };
  if (unit < n.heads + n.v) {
    const int pos = *a.pos_p + a.pos_off + r % a.t;
    if (pos < 0 || pos >= a.t_max) {
      if (lane == 0 && atomicCAS(&a.status->code, 0u, (unsigned)UGB_ERR_INVALID) == 0u) a.status->detail = (unsigned)pos;
      return;
    }
    if (unit < n.heads) {
      const int share = head_lanes(a.dp), head = unit * (32 / share) + lane / share, i0 = 8 * (lane % share), half = a.rot_dims >> 1;
      const bool on = head < n_head && i0 < a.dp;          // dp is a multiple of 8
      Row8<TI> x{};
      if (on) x = sum8(head * a.dp + i0);
      if (on && i0 < a.rot_dims) {
        const float *cs = a.cos_ + (size_t)pos * half, *sn = a.sin_ + (size_t)pos * half;
        if (a.interleaved) {
          const int p0 = i0 >> 1;
          float c[4], s[4];
          if ((half & 3) == 0) {                           // four angles at once: all inside, the table's rows aligned
            *reinterpret_cast<float4 *>(c) = __ldg(reinterpret_cast<const float4 *>(cs + p0));
            *reinterpret_cast<float4 *>(s) = __ldg(reinterpret_cast<const float4 *>(sn + p0));
          } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              c[e] = p0 + e < half ? __ldg(cs + p0 + e) : 1.f;
              s[e] = p0 + e < half ? __ldg(sn + p0 + e) : 0.f;
            }
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float u = x.v[2 * e], v = x.v[2 * e + 1];
            x.v[2 * e] = u * c[e] - v * s[e];
            x.v[2 * e + 1] = v * c[e] + u * s[e];
          }
        } else {                                           // the partner of a dimension lies half the rotated part away
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const int i = i0 + e;
            if (i >= a.rot_dims) break;
            const int p = i < half ? i : i - half, other = i < half ? i + half : i - half;
            float y = 0.f;
            for (int q = 0; q < a.n_part; ++q) y += (float)row[(size_t)q * a.part_stride + head * a.dp + other];
            const float c = __ldg(cs + p), s = __ldg(sn + p);
            x.v[e] = i < half ? x.v[e] * c - y * s : x.v[e] * c + y * s;
          }
        }
      }
      if (a.qk_norm) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) ss = fmaf(x.v[e], x.v[e], ss);
        for (int o = share >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.0f / sqrtf(ss / (float)a.dim + a.eps);
#pragma unroll
        for (int e = 0; e < 8; ++e) x.v[e] *= inv;
      }
      if (!on) return;
      T *dst = head < a.heads ? a.q + ((size_t)r * a.heads + head) * a.dp
                              : a.kcache + (((size_t)b * a.kv_heads + head - a.heads) * a.t_max + pos) * a.dp;
      Row8<T> y;
#pragma unroll
      for (int e = 0; e < 8; ++e) y.v[e] = x.v[e];
      st8<T>(dst + i0, y);
    } else {
      const int c = (unit - n.heads) * 256 + 8 * lane;
      if (c >= a.kv_heads * a.vp) return;
      const int h = c / a.vp;                              // vp is a multiple of 8: the 8 values belong to one head
      const Row8<TI> x = sum8(n_head * a.dp + c);
      Row8<T> y;
#pragma unroll
      for (int e = 0; e < 8; ++e) y.v[e] = x.v[e];
      st8<T>(a.vcache + (((size_t)b * a.kv_heads + h) * a.t_max + pos) * a.vp + c - h * a.vp, y);
    }
    return;
  }
  if constexpr (STEP) {
    const int x0 = n_head * a.dp + a.kv_heads * a.vp;
    if (unit < n.heads + n.v + n.x) {
      const int c = (unit - n.heads - n.v) * 128 + 4 * lane;
      if (c >= a.ci) return;
      float4 x = sum4(x0 + c), s = __ldg(reinterpret_cast<const float4 *>(a.conv_b + c));
      // what the convolution sees, now and later, is the rounded input
      x = make_float4(Act<T>::round(x.x), Act<T>::round(x.y), Act<T>::round(x.z), Act<T>::round(x.w));
      T *tp = a.tail + (size_t)r * (a.taps - 1) * a.ci + c;
      for (int j = 0; j < a.taps; ++j) {
        const float4 w = __ldg(reinterpret_cast<const float4 *>(a.conv_w + (size_t)j * a.ci + c));
        const float4 q = j + 1 < a.taps ? Act<T>::ld4(tp + (size_t)j * a.ci) : x;
        if (j > 0) Act<T>::st4(tp + (size_t)(j - 1) * a.ci, q);
        s.x = fmaf(w.x, q.x, s.x); s.y = fmaf(w.y, q.y, s.y); s.z = fmaf(w.z, q.z, s.z); s.w = fmaf(w.w, q.w, s.w);
      }
      constexpr bool EXACT = sizeof(T) == 4;
      Act<T>::st4(a.u + (size_t)r * a.ci + c, make_float4(s.x * sigmoid_t<EXACT>(s.x), s.y * sigmoid_t<EXACT>(s.y),
                                                         s.z * sigmoid_t<EXACT>(s.z), s.w * sigmoid_t<EXACT>(s.w)));
    } else if (a.experts > 0) {
      float z[ROUTER_PER_LANE];
#pragma unroll
      for (int j = 0; j < ROUTER_PER_LANE; ++j) {
        const int e = lane + 32 * j;
        z[j] = e < a.experts ? 0.f : -INFINITY;
        if (e < a.experts)
          for (int p = 0; p < a.n_part; ++p) z[j] += (float)row[(size_t)p * a.part_stride + x0 + 2 * a.ci + e];
      }
      top_experts(z, a.experts, a.top, [&](int k, int e, float zk) {
        if (lane == 0) a.choice[(size_t)r * a.top + k] = make_float4(__int_as_float(e), __int_as_float(atomicAdd(a.count + e, 1)), sigmoid_f(zk), 0.f);
      });
    }
  }
}

// ---------------------------------------------------------------- experts ----
// Router logits [n_part][rows][ld] of a block, to be summed -> choice [rows][top] = {expert, place among the expert's rows, sigmoid score}.  32
// rows per CTA: places are handed out per CTA in shared memory, one global counter update per expert and CTA.  Which place
// a row gets depends on the order of the CTAs; nothing that is computed does.
constexpr int ROUTE_ROWS = 32;
static __global__ void __launch_bounds__(256)
route_kernel(const float *__restrict__ logits, int n_part, int ld, int rows, int experts, int top, float4 *__restrict__ choice, int *__restrict__ count) {
  __shared__ int n[32 * ROUTER_PER_LANE], base[32 * ROUTER_PER_LANE];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r0 = blockIdx.x * ROUTE_ROWS;
  n[threadIdx.x] = 0;
  __syncthreads();
  for (int r = r0 + warp; r < min(rows, r0 + ROUTE_ROWS); r += 8) {
    float z[ROUTER_PER_LANE];
#pragma unroll
    for (int j = 0; j < ROUTER_PER_LANE; ++j) {
      const int e = lane + 32 * j;
      z[j] = e < experts ? 0.f : -INFINITY;
      if (e < experts)
        for (int p = 0; p < n_part; ++p) z[j] += logits[((size_t)p * rows + r) * ld + e];
    }
    top_experts(z, experts, top, [&](int k, int e, float zk) {
      if (lane == 0) choice[(size_t)r * top + k] = make_float4(__int_as_float(e), __int_as_float(atomicAdd(n + e, 1)), sigmoid_f(zk), 0.f);
    });
  }
  __syncthreads();
  if (threadIdx.x < experts && n[threadIdx.x] > 0) base[threadIdx.x] = atomicAdd(count + threadIdx.x, n[threadIdx.x]);
  __syncthreads();
  for (int i = threadIdx.x; i < ROUTE_ROWS * top; i += 256) {
    if (r0 + i / top >= rows) break;
    float4 *c = choice + (size_t)r0 * top + i;
    c->y = __int_as_float(__float_as_int(c->y) + base[__float_as_int(c->x)]);
  }
}

// Lays the chosen rows out by expert: expert e has ceil(count[e] / tile) tiles of `tile` rows, one after the other.
//   x[row of (r, k)] = weight h[r]    slot[r][k] = that row    map[i] = expert of tile i, -1 behind the last
// One CTA per token row.
template <typename T>
__global__ void __launch_bounds__(256)
expert_rows_kernel(const T *__restrict__ h, const float4 *__restrict__ choice, const int *__restrict__ count, int experts, int top,
                   int tile, int tiles, T *__restrict__ x, int *__restrict__ slot, int *__restrict__ map, int ld) {
  __shared__ int first[32 * ROUTER_PER_LANE + 1];          // first tile of every expert
  const int r = blockIdx.x, lane = threadIdx.x & 31;
  ugb_pdl_wait();
  ugb_pdl_trigger();
  if (threadIdx.x < 32) {
    int carry = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      int own = e0 + lane < experts ? (__ldcg(count + e0 + lane) + tile - 1) / tile : 0, sum = own;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += v;
      }
      first[e0 + lane] = carry + sum - own;
      carry += __shfl_sync(0xffffffffu, sum, 31);
    }
    if (lane == 0) first[experts] = carry;
  }
  __syncthreads();
  if (r == 0) {
    for (int i = threadIdx.x; i < tiles; i += 256) {
      int e = -1;
      if (i < first[experts])
        for (e = 0; e + 1 < experts && first[e + 1] <= i;) ++e;
      map[i] = e;
    }
  }
  for (int k = 0; k < top; ++k) {
    const float4 c = choice[(size_t)r * top + k];
    const int e = __float_as_int(c.x), place = __float_as_int(c.y);
    int to = -1;                                           // a row that does not fit is left out, never written elsewhere
    if (e >= 0 && e < experts && place >= 0) to = first[e] * tile + place;
    if (to >= tiles * tile) to = -1;
    if (threadIdx.x == 0) slot[(size_t)r * top + k] = to;
    if (to < 0) continue;
    for (int i = 4 * threadIdx.x; i < ld; i += 1024) {
      const float4 v = Act<T>::ld4(h + (size_t)r * ld + i);
      Act<T>::st4(x + (size_t)to * ld + i, make_float4(c.z * v.x, c.z * v.y, c.z * v.z, c.z * v.w));
    }
  }
}

// (gate, up) pairs [rows][2 n] -> silu(gate) up [rows][n], row strides in elements: the unfused form of
// UGB_EPI_SILU_MUL_BF16 for 32-bit activations
static __global__ void silu_mul_kernel(const float *__restrict__ gu, float *__restrict__ out, size_t rows, int n, size_t in_ld, size_t out_ld) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < rows * n; i += (size_t)gridDim.x * blockDim.x) {
    const size_t r = i / n;
    const int c = (int)(i - r * n);
    const float2 v = *reinterpret_cast<const float2 *>(gu + r * in_ld + 2 * c);
    out[r * out_ld + c] = silu_f(v.x) * v.y;
  }
}

// out = sum of n_part f32 partials, rounded to T; n4 groups of four values
template <typename T>
__global__ void __launch_bounds__(256)
sum_partials_kernel(const float *__restrict__ part, int n_part, size_t part_stride, size_t n4, T *__restrict__ out) {
  ugb_pdl_wait();
  ugb_pdl_trigger();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n4) return;
  float4 v[8], s = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int p = 0; p < n_part; p += 8) {                    // the partials are added in order
#pragma unroll
    for (int k = 0; k < 8; ++k) v[k] = p + k < n_part ? __ldcs(reinterpret_cast<const float4 *>(part + (size_t)(p + k) * part_stride) + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < 8; ++k) { s.x += v[k].x; s.y += v[k].y; s.z += v[k].z; s.w += v[k].w; }
  }
  Act<T>::st4(out + 4 * i, s);
}

// ------------------------------------------------------------- token input ---
// out[r][j] = gelu_tanh(sum of the partials of row r, column j) * table[token(r)][off + j], zero behind n.
// A thread takes 4 columns of a row; n4 = rows * ld / 4.
template <typename T>
__global__ void __launch_bounds__(256)
token_gate_kernel(const float *__restrict__ part, int n_part, size_t part_stride, size_t n4, int ld, int n, const int *__restrict__ tok, int t,
                  int tok_stride, int tok_off, const T *__restrict__ table, size_t table_ld, int off, int vocab, T *__restrict__ out) {
  ugb_pdl_wait();
  ugb_pdl_trigger();
  const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= n4) return;
  const int r = (int)(idx / (ld >> 2)), j = 4 * (int)(idx - (size_t)r * (ld >> 2));
  const int id = tok[(size_t)(r / t) * tok_stride + tok_off + r % t];
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int p = 0; p < n_part; p += 4) {                    // the partials are added in order
    float4 v[4];
#pragma unroll
    for (int k = 0; k < 4; ++k)
      v[k] = p + k < n_part ? *reinterpret_cast<const float4 *>(part + (size_t)(p + k) * part_stride + (size_t)r * ld + j) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < 4; ++k) { s.x += v[k].x; s.y += v[k].y; s.z += v[k].z; s.w += v[k].w; }
  }
  float e[4] = {0.f, 0.f, 0.f, 0.f};
  if (id >= 0 && id < vocab) {
    const T *src = table + (size_t)id * table_ld + off + j;
    if (j + 4 <= n && ((off | n | (int)(table_ld & 3)) & 3) == 0) {
      const float4 q = Act<T>::ld4(src);
      e[0] = q.x; e[1] = q.y; e[2] = q.z; e[3] = q.w;
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (j + k < n) e[k] = (float)src[k];
    }
  }
  auto gelu = [](float x) { return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x))); };
  Act<T>::st4(out + (size_t)r * ld + j, make_float4(gelu(s.x) * e[0], gelu(s.y) * e[1], gelu(s.z) * e[2], gelu(s.w) * e[3]));
}

// ------------------------------------------------------- logits, loading ----
static __global__ void softcap_kernel(float *__restrict__ x, size_t n4, float cap) {
  ugb_pdl_wait();
  ugb_pdl_trigger();
  const float inv = 1.0f / cap;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n4; i += (size_t)gridDim.x * blockDim.x) {
    float4 v = reinterpret_cast<float4 *>(x)[i];
    reinterpret_cast<float4 *>(x)[i] = make_float4(cap * tanhf(v.x * inv), cap * tanhf(v.y * inv), cap * tanhf(v.z * inv), cap * tanhf(v.w * inv));
  }
}

// cos / sin of p * freq[i]; the angle is formed in 64 bits, so that far positions lose nothing
static __global__ void rotation_table_kernel(const double *__restrict__ freq, float *__restrict__ cos_, float *__restrict__ sin_, int positions, int half) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)positions * half) return;
  const double a = (double)(i / half) * freq[i % half];
  cos_[i] = (float)cos(a);
  sin_[i] = (float)sin(a);
}

// a[c][s] = -exp(w[c][s]) * unit, rows of `states` values to rows of np, the padding zero
static __global__ void decay_kernel(const float *__restrict__ w, float *__restrict__ a, int channels, int states, int np, float unit) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < channels * states) a[(size_t)(i / states) * np + i % states] = -expf(w[i]) * unit;
}

// w [rows][cols] f32 -> out[c * ld + r] in T
template <typename T>
__global__ void transpose_kernel(const float *__restrict__ w, T *__restrict__ out, size_t rows, size_t cols, size_t ld) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < rows * cols; i += (size_t)gridDim.x * blockDim.x)
    out[(i % cols) * ld + i / cols] = (T)w[i];
}

}  // namespace ugb_hybrid_k
