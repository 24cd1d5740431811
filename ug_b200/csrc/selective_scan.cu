// Selective scan (see selective_scan.cuh).
//
//   selective_scan_kernel  a block of positions.  A CTA owns a group of channels of one sequence and walks the block in
//                          pieces of TT positions: four warps prepare step sizes (softplus), gates, B and C in shared memory,
//                          the others advance the states, LP lanes per channel pair with NS states of each in registers,
//                          and exchange the sums over the lanes eight positions at a time.
//   selective_step_kernel  one position of several sequences: the step-size projection, the state update and the gate in one
//                          kernel; everything that does not come from the preceding product is fetched ahead of the wait.
#include "selective_scan.cuh"

#include <algorithm>
#include <type_traits>

#include "decode_kernels.cuh"
#include "hybrid_kernels.cuh"

namespace {

using namespace ugb_hybrid_k;

// softplus(x) = log(1 + e^x); fast form: hardware exp2 / log2, a short series where e^x is small
template <bool EXACT> __device__ __forceinline__ float softplus_t(float x) {
  if constexpr (EXACT) return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
  float e, l;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-fabsf(x) * 1.4426950408889634f));
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(l) : "f"(1.0f + e));
  const float tail = e < 0.015625f ? e * (1.0f - e * (0.5f - e * (0.33333333f - 0.25f * e))) : l * 0.6931471805599453f;
  return fmaxf(x, 0.f) + tail;
}
// e^x S + in, or 2^x S + in where A carries log2(e).  In 32 bits as S + ((e^x - 1) S + in): a slow channel's factor differs
// from 1 by less than the factor's own rounding, which would add up over the sequence.
template <bool EXACT> __device__ __forceinline__ float advance(float x, float S, float in) {
  if constexpr (EXACT) return S + fmaf(expm1f(x), S, in);
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return fmaf(y, S, in);
}

template <typename T> struct Pair;
template <> struct Pair<float> {
  using Raw = float2;
  static __device__ __forceinline__ float2 wide(Raw r) { return r; }
  static __device__ __forceinline__ Raw pack(float a, float b) { return make_float2(a, b); }
};
template <> struct Pair<__nv_bfloat16> {
  using Raw = __nv_bfloat162;
  static __device__ __forceinline__ float2 wide(Raw r) { return __bfloat1622float2(r); }
  static __device__ __forceinline__ Raw pack(float a, float b) { return __floats2bfloat162_rn(a, b); }
};
template <typename T> __device__ __forceinline__ typename Pair<T>::Raw ld_pair(const T *p) { return *reinterpret_cast<const typename Pair<T>::Raw *>(p); }

// NS consecutive floats
template <int NS> __device__ __forceinline__ void ld_states(const float *p, float (&v)[NS]) {
  if constexpr (NS % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) {
      const float4 q = *reinterpret_cast<const float4 *>(p + i);
      v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w;
    }
  } else if constexpr (NS % 2 == 0) {
#pragma unroll
    for (int i = 0; i < NS; i += 2) {
      const float2 q = *reinterpret_cast<const float2 *>(p + i);
      v[i] = q.x; v[i + 1] = q.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i) v[i] = p[i];
  }
}
template <int NS> __device__ __forceinline__ void st_states(float *p, const float (&v)[NS]) {
  if constexpr (NS % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) *reinterpret_cast<float4 *>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else if constexpr (NS % 2 == 0) {
#pragma unroll
    for (int i = 0; i < NS; i += 2) *reinterpret_cast<float2 *>(p + i) = make_float2(v[i], v[i + 1]);
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i) p[i] = v[i];
  }
}

// ---------------------------------------------------------------- a block ----
template <typename T> struct Block {
  const T *u, *dt, *xdb, *z;
  const float *a, *skip, *dt_bias;
  float *state;
  T *out;
  size_t z_ld, out_ld;
  float scale;
  int channels, xr, rp, t;
};
constexpr int HELPERS = 128;
template <int LP, int NS> struct ScanCta {
  static constexpr int CC = LP * NS <= 64 ? 32 : 256 / LP, SCANNERS = CC / 2 * LP, ALL = SCANNERS + HELPERS;
};

// two floats at a time (one instruction each on this architecture)
__device__ __forceinline__ uint64_t pack2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float &a, float &b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

// The two halves of the CTA meet here from different places of the code: a barrier that is named, not __syncthreads.
template <int THREADS> __device__ __forceinline__ void piece_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory"); }

// grid (groups of CC channels, sequences).  A scanning thread has NS states of two neighbouring channels, LP lanes share a pair
// of channels; 128 threads help.  Pieces of TT positions lie in two shared buffers: while the scanners advance the states over
// piece i, the helpers turn piece i + 1 -- fetched two pieces ahead -- into step sizes, step size times input, output gate and
// skip term.  Two channels per thread, because shared memory is what bounds this kernel: a 16-byte read takes four passes
// whatever its lanes have in common, and B and C are read once for both.
// CTAS: resident per SM.  Alone on its SM a CTA is bound by its own latencies and takes longer pieces and more registers.
template <typename T, int LP, int NS, int TT, int CTAS>
__global__ void __launch_bounds__(ScanCta<LP, NS>::ALL, CTAS)
selective_scan_kernel(Block<T> p) {
  constexpr bool EXACT = sizeof(T) == 4;
  constexpr int CC = ScanCta<LP, NS>::CC, SCANNERS = ScanCta<LP, NS>::SCANNERS, NP = LP * NS, G = 8;
  constexpr int ROWS = HELPERS / (CC / 2);                           // positions between a helper's channel pairs
  constexpr int PAIRS = (TT + ROWS - 1) / ROWS, BCS = TT * NP / HELPERS;
  static_assert(TT % G == 0 && BCS * HELPERS == TT * NP, "shape");
  using Raw = typename Pair<T>::Raw;
  __shared__ __align__(16) float4 sd[2][TT][CC / 2];                 // of a channel pair: dt, dt, dt x, dt x
  __shared__ __align__(16) float sbc[2][TT][2 * NP];                 // B | C
  __shared__ __align__(16) float4 sg[2][TT][CC / 2 + 1];   // gate, gate, skip x, skip x; the pitch avoids conflicts
  const int tid = threadIdx.x, c0 = blockIdx.x * CC, b = blockIdx.y;
  const size_t row0 = (size_t)b * p.t;
  const int pieces = (p.t + TT - 1) / TT;

  if (tid >= SCANNERS) {
    // channel pair and first position of this helper; addresses outside the block or the model are brought back inside, what is
    // loaded from there is not used
    const int h = tid - SCANNERS, cp = (h % (CC / 2)) * 2, rs = h / (CC / 2), cl = min(c0 + cp, p.channels - 2), last = p.t - 1;
    const float2 bias = *reinterpret_cast<const float2 *>(p.dt_bias + cl), skip = *reinterpret_cast<const float2 *>(p.skip + cl);
    const T *pd = p.dt + row0 * p.channels + cl, *pu = p.u + row0 * p.channels + cl, *pz = p.z + row0 * p.z_ld + cl;
    const T *pb = p.xdb + row0 * p.xr + p.rp;
    struct Fetched { Raw d[PAIRS], u[PAIRS], z[PAIRS], bc[BCS]; } even, odd;
    auto fetch = [&](Fetched &f, int piece) {
      const int t0 = piece * TT;
#pragma unroll
      for (int i = 0; i < PAIRS; ++i) {
        const int t = min(t0 + rs + i * ROWS, last);
        const size_t at = (size_t)t * p.channels;
        f.d[i] = ld_pair(pd + at);
        f.u[i] = ld_pair(pu + at);
        f.z[i] = ld_pair(pz + (size_t)t * p.z_ld);
      }
#pragma unroll
      for (int i = 0; i < BCS; ++i) {
        const int idx = h + i * HELPERS, t = min(t0 + idx / NP, last);
        f.bc[i] = ld_pair(pb + (size_t)t * p.xr + 2 * (idx % NP));
      }
    };
    auto stage = [&](const Fetched &f, int piece) {
      const int q = piece & 1, t0 = piece * TT;
#pragma unroll
      for (int i = 0; i < PAIRS; ++i) {
        const int s = rs + i * ROWS;
        if (TT % ROWS != 0 && s >= TT) continue;
        const bool live = t0 + s <= last;                            // behind the block: leaves the state alone
        const float2 d = Pair<T>::wide(f.d[i]), u = Pair<T>::wide(f.u[i]), z = Pair<T>::wide(f.z[i]);
        const float dx = live ? softplus_t<EXACT>(d.x + bias.x) : 0.f, dy = live ? softplus_t<EXACT>(d.y + bias.y) : 0.f;
        sd[q][s][cp / 2] = make_float4(dx, dy, dx * u.x, dy * u.y);
        sg[q][s][cp / 2] = make_float4(z.x * sigmoid_t<EXACT>(z.x) * p.scale, z.y * sigmoid_t<EXACT>(z.y) * p.scale, skip.x * u.x, skip.y * u.y);
      }
#pragma unroll
      for (int i = 0; i < BCS; ++i) {
        const int idx = h + i * HELPERS;
        *reinterpret_cast<float2 *>(&sbc[q][idx / NP][2 * (idx % NP)]) = Pair<T>::wide(f.bc[i]);
      }
    };
    fetch(even, 0);
    fetch(odd, 1);
    stage(even, 0);
    fetch(even, 2);
    piece_barrier<ScanCta<LP, NS>::ALL>();
    for (int i = 0; i < pieces; i += 2) {                            // pieces i + 1 and i + 2 are prepared; a fetch is used two pieces later
      if (i + 1 < pieces) {
        stage(odd, i + 1);
        fetch(odd, i + 3);
      }
      piece_barrier<ScanCta<LP, NS>::ALL>();
      if (i + 1 >= pieces) break;
      if (i + 2 < pieces) {
        stage(even, i + 2);
        fetch(even, i + 4);
      }
      piece_barrier<ScanCta<LP, NS>::ALL>();
    }
    return;
  }

  const int pair = tid / LP, l = tid % LP, c = c0 + 2 * pair;
  const bool on = c < p.channels;                                    // channels is even
  uint64_t S2[NS], A2[NS];                                           // (this channel, the next)
  float *state = p.state + ((size_t)b * p.channels + c) * NP + l * NS;
  {
    float s0[NS], s1[NS], a0[NS], a1[NS];
#pragma unroll
    for (int n = 0; n < NS; ++n) s0[n] = s1[n] = a0[n] = a1[n] = 0.f;
    if (on) {
      const float *a = p.a + (size_t)c * NP + l * NS;
      ld_states<NS>(state, s0); ld_states<NS>(state + NP, s1); ld_states<NS>(a, a0); ld_states<NS>(a + NP, a1);
    }
#pragma unroll
    for (int n = 0; n < NS; ++n) { S2[n] = pack2(s0[n], s1[n]); A2[n] = pack2(a0[n], a1[n]); }
  }
  T *out = p.out + (row0 + l % G) * p.out_ld + c;
  piece_barrier<ScanCta<LP, NS>::ALL>();
  for (int i = 0; i < pieces; ++i) {
    const int q = i & 1, t0 = i * TT;
    float2 y[TT / G];                                                // stored after the piece: a store would hold up the next reads
#pragma unroll
    for (int s0 = 0; s0 < TT; s0 += G) {
      float v[G], w[G];                                              // sums of the two channels
#pragma unroll
      for (int k = 0; k < G; ++k) {
        const float4 d = sd[q][s0 + k][pair];
        float B[NS], C[NS];
        ld_states<NS>(&sbc[q][s0 + k][l * NS], B);
        ld_states<NS>(&sbc[q][s0 + k][NP + l * NS], C);
        v[k] = w[k] = 0.f;
        const uint64_t dt2 = pack2(d.x, d.y);
#pragma unroll
        for (int n = 0; n < NS; ++n) {
          float x0, x1, s0v, s1v;
          unpack2(mul2(dt2, A2[n]), x0, x1);
          if constexpr (EXACT) {
            unpack2(S2[n], s0v, s1v);
            s0v = advance<true>(x0, s0v, d.z * B[n]);
            s1v = advance<true>(x1, s1v, d.w * B[n]);
            S2[n] = pack2(s0v, s1v);
          } else {
            asm("ex2.approx.ftz.f32 %0, %0;" : "+f"(x0));
            asm("ex2.approx.ftz.f32 %0, %0;" : "+f"(x1));
            S2[n] = fma2(pack2(x0, x1), S2[n], pack2(d.z * B[n], d.w * B[n]));
            unpack2(S2[n], s0v, s1v);
          }
          v[k] = fmaf(s0v, C[n], v[k]);
          w[k] = fmaf(s1v, C[n], w[k]);
        }
      }
      // sums over the lanes of a pair: every exchange halves the positions a lane still holds, lane l ends with position l % G
#pragma unroll
      for (int h = G / 2; h >= 1; h >>= 1) {
        const bool upper = (l & h) != 0;
#pragma unroll
        for (int k = 0; k < h; ++k) {
          const float sv = upper ? v[k] : v[k + h], kv = upper ? v[k + h] : v[k], sw = upper ? w[k] : w[k + h], kw = upper ? w[k + h] : w[k];
          v[k] = kv + __shfl_xor_sync(0xffffffffu, sv, h);
          w[k] = kw + __shfl_xor_sync(0xffffffffu, sw, h);
        }
      }
#pragma unroll
      for (int o = G; o < LP; o <<= 1) {
        v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
        w[0] += __shfl_xor_sync(0xffffffffu, w[0], o);
      }
      y[s0 / G] = make_float2(v[0], w[0]);
    }
    if (l < G && on) {
#pragma unroll
      for (int s0 = 0; s0 < TT; s0 += G) {
        const float4 g = sg[q][s0 + l][pair];
        const float2 v = y[s0 / G];
        if (t0 + s0 + l < p.t) *reinterpret_cast<Raw *>(out + (size_t)(t0 + s0) * p.out_ld) = Pair<T>::pack((v.x + g.z) * g.x, (v.y + g.w) * g.y);
      }
    }
    piece_barrier<ScanCta<LP, NS>::ALL>();
  }
  if (on) {
    float s0[NS], s1[NS];
#pragma unroll
    for (int n = 0; n < NS; ++n) unpack2(S2[n], s0[n], s1[n]);
    st_states<NS>(state, s0);
    st_states<NS>(state + NP, s1);
  }
}

// ----------------------------------------------------------------- a step ----
template <typename T> struct Step {
  const T *u, *w_dt;
  ugb_scan_partials xdb, z;
  const float *a, *skip, *dt_bias;
  float *state;
  T *out;
  size_t out_ld;
  float scale;
  int channels, xr, rp, rows, group, w_shared, early;                // group: sequences of a CTA; w_shared: W_dt columns in shared memory
};
constexpr int THREADS = 256;
constexpr int STEP_J = 4;            // sequences per thread in the projection and the element-wise parts
// sequences of a CTA at most: a thread holds its states of all of them in registers from before the wait
template <int NS> struct StepRows { static constexpr int D = NS <= 4 ? 16 : 8; };

// grid (groups of 256 / LP channels, groups of `group` sequences).  Dynamic shared memory: dt, dt x [group][CC]; low | B | C
// [group][xr]; sums over the states [group][CC]; with w_shared W_dt [rk][CC + 8], and low [16][rk + 8] in T for the tensor cores,
// rk = rp rounded up to 16.
template <typename T, int LP, int NS>
__global__ void __launch_bounds__(THREADS)
selective_step_kernel(Step<T> p) {
  constexpr bool EXACT = sizeof(T) == 4;
  constexpr int CC = THREADS / LP, NP = LP * NS, D = StepRows<NS>::D;
  extern __shared__ __align__(16) float dyn[];
  float2 *sd = reinterpret_cast<float2 *>(dyn);                      // [group][CC]
  float *xs = dyn + 2 * p.group * CC, *sy = xs + p.group * p.xr;
  constexpr int WLD = CC + 8;                                        // pitches that ldmatrix reads without conflicts
  const int rk = (p.rp + 15) / 16 * 16, xld = rk + 8;
  T *ws = reinterpret_cast<T *>(sy + p.group * CC), *xl = ws + rk * WLD;
  const int tid = threadIdx.x, ch = tid / LP, l = tid % LP;
  const int c0 = blockIdx.x * CC, r0 = blockIdx.y * p.group, n_rows = min(p.group, p.rows - r0);
  if (!p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
  const int c = c0 + ch;
  const bool on = c < p.channels;
  float A[NS];
#pragma unroll
  for (int n = 0; n < NS; ++n) A[n] = 0.f;
  if (on) ld_states<NS>(p.a + (size_t)c * NP + l * NS, A);
  float *state = p.state + ((size_t)r0 * p.channels + c) * NP + l * NS;
  const size_t next_row = (size_t)p.channels * NP;
  float S[D][NS];
#pragma unroll
  for (int d = 0; d < D; ++d) {
#pragma unroll
    for (int n = 0; n < NS; ++n) S[d][n] = 0.f;
    if (on && d < n_rows) ld_states<NS>(state + (size_t)d * next_row, S[d]);
  }
  // channel and sequences of this thread in the projection and the element-wise parts
  const int ec = tid % CC, er = tid / CC;
  const bool col = c0 + ec < p.channels;
  float u[STEP_J], z[STEP_J], bias = 0.f, skip = 0.f;
  if (col) { bias = __ldg(p.dt_bias + c0 + ec); skip = __ldg(p.skip + c0 + ec); }
#pragma unroll
  for (int j = 0; j < STEP_J; ++j) {
    const int r = er + LP * j;
    u[j] = z[j] = 0.f;
    if (r < n_rows && col) {
      u[j] = (float)p.u[(size_t)(r0 + r) * p.channels + c0 + ec];
      for (int q = 0; q < p.z.n; ++q) z[j] += p.z.p[q * p.z.stride + (size_t)(r0 + r) * p.z.ld + c0 + ec];
    }
  }
  if (p.w_shared) {
    for (int i = tid; i < rk * (CC / 8); i += THREADS) {             // channels is a multiple of 8
      const int k = i / (CC / 8), w = 8 * (i - k * (CC / 8));
      Row8<T> v{};
      if (k < p.rp && c0 + w < p.channels) v = ld8<T>(p.w_dt + (size_t)k * p.channels + c0 + w);
      st8<T>(ws + k * WLD + w, v);
    }
    if (!EXACT && rk > p.rp && tid < 16) st8<T>(xl + tid * xld + p.rp, Row8<T>{});
  }
  if (p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
  for (int i = tid; i < p.group * (p.xr / 4); i += THREADS) {
    const int r = i / (p.xr / 4), k = 4 * (i - r * (p.xr / 4));
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r < n_rows)
      for (int q = 0; q < p.xdb.n; q += 8) {                         // the partials are added in order
        float4 v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e)
          v[e] = q + e < p.xdb.n ? *reinterpret_cast<const float4 *>(p.xdb.p + (q + e) * p.xdb.stride + (size_t)(r0 + r) * p.xdb.ld + k)
                                 : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int e = 0; e < 8; ++e) { s.x += v[e].x; s.y += v[e].y; s.z += v[e].z; s.w += v[e].w; }
      }
    if (!EXACT && p.w_shared && k < p.rp) Act<T>::st4(xl + r * xld + k, s);
    *reinterpret_cast<float4 *>(xs + r * p.xr + k) = s;
  }
  __syncthreads();
  // step sizes before bias and softplus: on the tensor cores (a 16-row tile of sequences, a warp per 8 channels), or one by one
  float pre[STEP_J];
  bool done = false;
  if constexpr (!EXACT) {
    done = p.w_shared != 0;
    const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    if (done && warp * 8 < CC) {
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      for (int k = 0; k < rk; k += 16) {
        uint32_t a[4], b0, b1;
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                     : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3])
                     : "r"(ugb_tc::smem_u32(xl + (lane & 15) * xld + k + 8 * (lane >> 4))));
        asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];"
                     : "=r"(b0), "=r"(b1) : "r"(ugb_tc::smem_u32(ws + (k + (lane & 15)) * WLD + 8 * warp)));
        ugb_decode::mma_bf16_16x8x16(acc, a[0], a[1], a[2], a[3], b0, b1);
      }
#pragma unroll
      for (int h = 0; h < 2; ++h)
        if (g + 8 * h < p.group) {
          sd[(g + 8 * h) * CC + 8 * warp + 2 * tq].x = acc[2 * h];
          sd[(g + 8 * h) * CC + 8 * warp + 2 * tq + 1].x = acc[2 * h + 1];
        }
    }
    if (done) {
      __syncthreads();
#pragma unroll
      for (int j = 0; j < STEP_J; ++j) pre[j] = er + LP * j < p.group ? sd[(er + LP * j) * CC + ec].x : 0.f;
    }
  }
  if (!done) {
#pragma unroll
    for (int j = 0; j < STEP_J; ++j) pre[j] = 0.f;
    for (int k = 0; k < p.rp; ++k) {
      const float w = p.w_shared ? (float)ws[k * WLD + ec] : (col ? (float)p.w_dt[(size_t)k * p.channels + c0 + ec] : 0.f);
#pragma unroll
      for (int j = 0; j < STEP_J; ++j)
        if (er + LP * j < p.group) pre[j] = fmaf(w, xs[(er + LP * j) * p.xr + k], pre[j]);
    }
  }
#pragma unroll
  for (int j = 0; j < STEP_J; ++j) {
    if (er + LP * j >= p.group) break;
    const float d = softplus_t<EXACT>(pre[j] + bias);
    sd[(er + LP * j) * CC + ec] = make_float2(d, d * u[j]);
  }
  __syncthreads();
#pragma unroll
  for (int d0 = 0; d0 < D; d0 += 4) {                                // the sums of four sequences are exchanged together
    if (d0 >= n_rows) break;                                         // the same for the whole CTA
    float y[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d0 + e;
      y[e] = 0.f;
      if (d >= n_rows) continue;
      const float2 dt = sd[d * CC + ch];
      const float *bc = xs + d * p.xr + p.rp + l * NS;
      float B[NS], C[NS];
      ld_states<NS>(bc, B);
      ld_states<NS>(bc + NP, C);
#pragma unroll
      for (int n = 0; n < NS; ++n) {
        S[d][n] = advance<EXACT>(dt.x * A[n], S[d][n], dt.y * B[n]);
        y[e] = fmaf(S[d][n], C[n], y[e]);
      }
      if (on) st_states<NS>(state + (size_t)d * next_row, S[d]);
    }
#pragma unroll
    for (int o = 1; o < LP; o <<= 1)
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] += __shfl_xor_sync(0xffffffffu, y[e], o);
    if (l == 0) {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (d0 + e < n_rows) sy[(d0 + e) * CC + ch] = y[e];
    }
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < STEP_J; ++j) {
    const int r = er + LP * j;
    if (r < n_rows && col)
      p.out[(size_t)(r0 + r) * p.out_ld + c0 + ec] = (T)(fmaf(skip, u[j], sy[r * CC + ec]) * z[j] * sigmoid_t<EXACT>(z[j]) * p.scale);
  }
}

template <typename T, int LP, int NS>
int32_t block_one(ugb_device *dev, const ugb_scan_args &a, const void *dt, const void *xdb, const void *z, size_t z_ld, int b, int t) {
  using Cta = ScanCta<LP, NS>;
  Block<T> p;
  p.u = (const T *)a.u; p.dt = (const T *)dt; p.xdb = (const T *)xdb; p.z = (const T *)z; p.a = a.a; p.skip = a.skip; p.dt_bias = a.dt_bias;
  p.state = a.state; p.out = (T *)a.out; p.z_ld = z_ld; p.out_ld = a.out_ld; p.scale = a.scale; p.channels = a.channels; p.xr = a.xr;
  p.rp = a.rp; p.t = t;
  const dim3 grid((a.channels + Cta::CC - 1) / Cta::CC, b);
  constexpr int TT = LP * NS <= 64 ? 16 : 8, CTAS = sizeof(T) == 2 && NS <= 4 ? 3 : 1;
  bool alone = false;
  if constexpr (LP * NS <= 16) {
    alone = (long long)grid.x * grid.y <= dev->sm_count;
    if (alone) selective_scan_kernel<T, LP, NS, 2 * TT, 1><<<grid, Cta::ALL, 0, dev->stream>>>(p);
  }
  if (!alone) selective_scan_kernel<T, LP, NS, TT, CTAS><<<grid, Cta::ALL, 0, dev->stream>>>(p);
  return ugb_after_launch(dev, "selective_scan_kernel");
}
template <typename T, int LP, int NS>
int32_t step_one(ugb_device *dev, const ugb_scan_args &a, const void *w_dt, ugb_scan_partials xdb, ugb_scan_partials z, int rows, bool pdl, bool early) {
  constexpr int CC = THREADS / LP;
  Step<T> p;
  p.u = (const T *)a.u; p.w_dt = (const T *)w_dt; p.xdb = xdb; p.z = z; p.a = a.a; p.skip = a.skip; p.dt_bias = a.dt_bias; p.state = a.state;
  p.out = (T *)a.out; p.out_ld = a.out_ld; p.scale = a.scale; p.channels = a.channels; p.xr = a.xr; p.rp = a.rp; p.rows = rows;
  p.early = early && pdl ? 1 : 0;
  // sequences per CTA: two CTAs are resident per SM, so one wave of at least 1.5 per SM; no more than a thread's share and the
  // shared memory allow
  const int groups = (a.channels + CC - 1) / CC, most = std::min(STEP_J * LP, StepRows<NS>::D);
  const int rk = (a.rp + 15) / 16 * 16;
  const size_t w_bytes = ((size_t)rk * (CC + 8) + 16 * (rk + 8)) * sizeof(T), limit = 100 * 1024;   // two CTAs per SM
  p.w_shared = w_bytes <= 64 * 1024;
  const size_t fixed = p.w_shared ? w_bytes : 0, per_row = (size_t)CC * 12 + (size_t)a.xr * 4;
  p.group = most;
  while (p.group > 4 && 2ll * groups * ((rows + p.group - 1) / p.group) < 3 * dev->sm_count) p.group /= 2;
  while (p.group > 1 && fixed + p.group * per_row > limit) p.group /= 2;
  UGB_REQUIRE(dev, fixed + p.group * per_row <= limit, UGB_ERR_UNSUPPORTED, "selective scan: %d columns of step size, B and C", a.xr);
  static size_t allowed[64] = {};                            // by device; a size is met by an eager step before any capture
  size_t &most_smem = allowed[dev->ordinal & 63];
  const size_t smem = fixed + p.group * per_row;
  if (smem > std::max<size_t>(most_smem, 48 * 1024)) {
    UGB_CUDA(dev, cudaFuncSetAttribute(selective_step_kernel<T, LP, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    most_smem = smem;
  }
  const cudaError_t e = ugb_launch(selective_step_kernel<T, LP, NS>, dim3(groups, (rows + p.group - 1) / p.group), dim3(THREADS), smem, dev->stream, pdl, p);
  if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of selective_step_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(dev, "selective_step_kernel");
}

// f(LP, NS) for the step kernel of a shape
template <typename F> int32_t with_shape(ugb_device *dev, const ugb_scan_shape &s, F f) {
#define SHAPE(LP, NS) if (s.lanes == LP && s.per_lane == NS) return f(std::integral_constant<int, LP>(), std::integral_constant<int, NS>())
  SHAPE(4, 2); SHAPE(4, 4); SHAPE(4, 6); SHAPE(4, 8); SHAPE(8, 6); SHAPE(8, 8); SHAPE(16, 8); SHAPE(32, 8);
#undef SHAPE
  return ugb_fail(dev, UGB_ERR_UNSUPPORTED, "selective scan: no kernel for %d states on %d lanes", s.np, s.lanes);
}

int32_t check(ugb_device *dev, const ugb_scan_args &a) {
  UGB_REQUIRE(dev, a.channels > 0 && a.channels % 8 == 0 && a.xr % 8 == 0 && a.rp % 8 == 0 && a.xr >= a.rp + 2 * a.shape.np && a.out_ld % 8 == 0,
              UGB_ERR_SHAPE, "selective scan: %d channels, %d + 2 x %d of %d columns", a.channels, a.rp, a.shape.np, a.xr);
  return UGB_OK;
}

}  // namespace

ugb_scan_shape ugb_scan_shape_of(int states) {
  for (int ns : {2, 4, 6, 8})
    if (states <= 4 * ns) return {4, ns, 4 * ns};
  for (int ns : {6, 8})
    if (states <= 8 * ns) return {8, ns, 8 * ns};
  for (int lanes : {16, 32})
    if (states <= 8 * lanes) return {lanes, 8, 8 * lanes};
  return {0, 0, 0};
}

float ugb_scan_decay_unit(bool f32) { return f32 ? 1.0f : 1.4426950408889634f; }

int32_t ugb_scan_block(ugb_device *dev, const ugb_scan_args &a, const void *dt, const void *xdb, const void *z, size_t z_ld, int b, int t) {
  if (b == 0 || t == 0) return UGB_OK;
  if (int32_t rc = check(dev, a)) return rc;
  UGB_REQUIRE(dev, z_ld % 8 == 0 && b <= 65535, UGB_ERR_SHAPE, "selective scan: %d sequences, gate rows %zu apart", b, z_ld);
#define BLOCK(NP, LP) \
  if (a.shape.np == NP) \
    return a.f32 ? block_one<float, LP, NP / LP>(dev, a, dt, xdb, z, z_ld, b, t) : block_one<__nv_bfloat16, LP, NP / LP>(dev, a, dt, xdb, z, z_ld, b, t)
  BLOCK(8, 8); BLOCK(16, 8); BLOCK(24, 8); BLOCK(32, 8); BLOCK(48, 8); BLOCK(64, 8); BLOCK(128, 16); BLOCK(256, 32);
#undef BLOCK
  return ugb_fail(dev, UGB_ERR_UNSUPPORTED, "selective scan: no kernel for %d states", a.shape.np);
}

int32_t ugb_scan_step(ugb_device *dev, const ugb_scan_args &a, const void *w_dt, ugb_scan_partials xdb, ugb_scan_partials z, int rows, bool pdl, bool early) {
  if (rows == 0) return UGB_OK;
  if (int32_t rc = check(dev, a)) return rc;
  return with_shape(dev, a.shape, [&](auto lp, auto ns) {
    return a.f32 ? step_one<float, lp(), ns()>(dev, a, w_dt, xdb, z, rows, pdl, early) : step_one<__nv_bfloat16, lp(), ns()>(dev, a, w_dt, xdb, z, rows, pdl, early);
  });
}
