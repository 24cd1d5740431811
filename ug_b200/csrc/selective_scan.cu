// Selective scan (see selective_scan.cuh).
//
//   selective_scan_kernel  a block of positions.  A CTA owns 256 / LP channels of one sequence and walks the block in
//                          pieces of TT positions: step sizes (softplus), dt x, B and C go to shared memory, LP lanes per
//                          channel advance NS states each in registers, and the sums over a channel's lanes are exchanged
//                          eight positions at a time.  The next piece is on its way while a piece is worked on.
//   selective_step_kernel  one position of several sequences: the step-size projection, the state update and the gate in one
//                          kernel; everything that does not come from the preceding product is fetched ahead of the wait.
#include "selective_scan.cuh"

#include "hybrid_kernels.cuh"

namespace {

using namespace ugb_hybrid_k;

constexpr int THREADS = 256;

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

template <typename T> struct Block {
  const T *u, *dt, *xdb, *z;
  const float *a, *skip, *dt_bias;
  float *state;
  T *out;
  size_t z_ld, out_ld;
  float scale;
  int channels, xr, rp, t;
};

template <typename T, int LP, int NS>
__global__ void __launch_bounds__(THREADS)
selective_scan_kernel(Block<T> p) {
  constexpr bool EXACT = sizeof(T) == 4;
  constexpr int CC = THREADS / LP, TT = LP == 8 ? 32 : 8, NP = LP * NS;
  constexpr int PAIRS = (TT * CC / 2 + THREADS - 1) / THREADS;       // channel pairs a thread stages per piece
  using Raw = typename Pair<T>::Raw;
  __shared__ float2 sdt[TT][CC];                                     // dt, dt x
  __shared__ __align__(16) float sbc[TT][2 * NP];                    // B | C
  __shared__ float sy[TT][CC + 4];                                   // the pitch keeps the exchange conflict-free
  const int tid = threadIdx.x, ch = tid / LP, l = tid % LP;
  const int c0 = blockIdx.x * CC, b = blockIdx.y, c = c0 + ch;
  const bool on = c < p.channels;
  const size_t row0 = (size_t)b * p.t;
  float S[NS], A[NS];
#pragma unroll
  for (int n = 0; n < NS; ++n) S[n] = A[n] = 0.f;
  float *state = p.state + ((size_t)b * p.channels + c) * NP + l * NS;
  if (on) { ld_states<NS>(state, S); ld_states<NS>(p.a + (size_t)c * NP + l * NS, A); }
  // staging: this thread's channel pair is the same in every row
  const int cp = (tid % (CC / 2)) * 2, rs = tid / (CC / 2);
  constexpr int ROWS = THREADS / (CC / 2);                           // rows between a thread's pairs
  const bool pair_on = c0 + cp < p.channels;
  float2 bias = make_float2(0.f, 0.f), skip = bias;
  if (pair_on) {
    bias = *reinterpret_cast<const float2 *>(p.dt_bias + c0 + cp);
    skip = *reinterpret_cast<const float2 *>(p.skip + c0 + cp);
  }
  const Raw zero = Pair<T>::pack(0.f, 0.f);
  Raw rd[PAIRS], ru[PAIRS], rz[PAIRS], rb[NS];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int s = rs + i * ROWS;
      rd[i] = ru[i] = rz[i] = zero;
      if (s < TT && t0 + s < p.t && pair_on) {
        const size_t r = row0 + t0 + s;
        rd[i] = ld_pair(p.dt + r * p.channels + c0 + cp);
        ru[i] = ld_pair(p.u + r * p.channels + c0 + cp);
        rz[i] = ld_pair(p.z + r * p.z_ld + c0 + cp);
      }
    }
#pragma unroll
    for (int i = 0; i < NS; ++i) {                                   // TT * NP pairs of B and C
      const int idx = tid + i * THREADS, s = idx / NP;
      rb[i] = t0 + s < p.t ? ld_pair(p.xdb + (row0 + t0 + s) * p.xr + p.rp + 2 * (idx % NP)) : zero;
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < p.t; t0 += TT) {
    float2 u[PAIRS], z[PAIRS];
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int s = rs + i * ROWS;
      const float2 d = Pair<T>::wide(rd[i]);
      u[i] = Pair<T>::wide(ru[i]);
      z[i] = Pair<T>::wide(rz[i]);
      if (s < TT) {
        const bool live = t0 + s < p.t;                              // behind the block: leaves the state alone
        const float dx = live ? softplus_t<EXACT>(d.x + bias.x) : 0.f, dy = live ? softplus_t<EXACT>(d.y + bias.y) : 0.f;
        sdt[s][cp] = make_float2(dx, dx * u[i].x);
        sdt[s][cp + 1] = make_float2(dy, dy * u[i].y);
      }
    }
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const int idx = tid + i * THREADS;
      *reinterpret_cast<float2 *>(&sbc[idx / NP][2 * (idx % NP)]) = Pair<T>::wide(rb[i]);
    }
    fetch(t0 + TT);
    __syncthreads();
#pragma unroll 1
    for (int s0 = 0; s0 < TT; s0 += 8) {
      float v[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float2 d = sdt[s0 + k][ch];
        float B[NS], C[NS];
        ld_states<NS>(&sbc[s0 + k][l * NS], B);
        ld_states<NS>(&sbc[s0 + k][NP + l * NS], C);
        v[k] = 0.f;
#pragma unroll
        for (int n = 0; n < NS; ++n) {
          S[n] = advance<EXACT>(d.x * A[n], S[n], d.y * B[n]);
          v[k] = fmaf(S[n], C[n], v[k]);
        }
      }
      // sums over the channel's lanes: every exchange halves the positions a lane still holds, lane l ends with l % 8
#pragma unroll
      for (int w = 4; w >= 1; w >>= 1) {
        const bool upper = (l & w) != 0;
#pragma unroll
        for (int i = 0; i < w; ++i) {
          const float send = upper ? v[i] : v[i + w], keep = upper ? v[i + w] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, w);
        }
      }
#pragma unroll
      for (int o = 8; o < LP; o <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
      if (l < 8) sy[s0 + l][ch] = v[0];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int s = rs + i * ROWS;
      if (s < TT && t0 + s < p.t && pair_on) {
        const float gx = z[i].x * sigmoid_t<EXACT>(z[i].x) * p.scale, gy = z[i].y * sigmoid_t<EXACT>(z[i].y) * p.scale;
        *reinterpret_cast<Raw *>(p.out + (row0 + t0 + s) * p.out_ld + c0 + cp) =
            Pair<T>::pack(fmaf(skip.x, u[i].x, sy[s][cp]) * gx, fmaf(skip.y, u[i].y, sy[s][cp + 1]) * gy);
      }
    }
  }
  if (on) st_states<NS>(state, S);
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
  int channels, xr, rp, rows, early;
};
constexpr int STEP_ROWS = 4;         // sequences of a CTA
constexpr int STEP_W = 16;           // step-size weights a thread holds from before the wait

// grid (groups of 256 / LP channels, groups of STEP_ROWS sequences); dynamic shared memory: low | B | C of the sequences
template <typename T, int LP, int NS>
__global__ void __launch_bounds__(THREADS)
selective_step_kernel(Step<T> p) {
  constexpr bool EXACT = sizeof(T) == 4;
  constexpr int CC = THREADS / LP, NP = LP * NS, KG = THREADS / CC, R = STEP_ROWS;
  extern __shared__ __align__(16) float xs[];                        // [R][xr]
  __shared__ float red[KG][R][CC];
  __shared__ float2 sd[R][CC];                                       // dt, dt x
  __shared__ float sy[R][CC];
  const int tid = threadIdx.x, ch = tid / LP, l = tid % LP;
  const int c0 = blockIdx.x * CC, r0 = blockIdx.y * R, n_rows = min(R, p.rows - r0);
  if (!p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
  const int c = c0 + ch;
  const bool on = c < p.channels;
  float A[NS], S[R][NS];
#pragma unroll
  for (int n = 0; n < NS; ++n) A[n] = 0.f;
  if (on) ld_states<NS>(p.a + (size_t)c * NP + l * NS, A);
#pragma unroll
  for (int r = 0; r < R; ++r) {
#pragma unroll
    for (int n = 0; n < NS; ++n) S[r][n] = 0.f;
    if (on && r < n_rows) ld_states<NS>(p.state + ((size_t)(r0 + r) * p.channels + c) * NP + l * NS, S[r]);
  }
  // (sequence, channel) of this thread in the element-wise parts, and (channel, part of the rank) in the projection
  const int er = tid / CC, ec = tid % CC;
  const bool own = er < n_rows && c0 + ec < p.channels;
  float u = 0.f, z = 0.f, bias = 0.f, skip = 0.f;
  if (own) {
    u = (float)p.u[(size_t)(r0 + er) * p.channels + c0 + ec];
    bias = __ldg(p.dt_bias + c0 + ec);
    skip = __ldg(p.skip + c0 + ec);
    for (int q = 0; q < p.z.n; ++q) z += p.z.p[q * p.z.stride + (size_t)(r0 + er) * p.z.ld + c0 + ec];
  }
  const int kk = tid / CC;
  const bool col = c0 + ec < p.channels;
  float w[STEP_W];
#pragma unroll
  for (int i = 0; i < STEP_W; ++i) w[i] = col && kk + i * KG < p.rp ? (float)p.w_dt[(size_t)(kk + i * KG) * p.channels + c0 + ec] : 0.f;
  if (p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
  for (int i = tid; i < R * (p.xr / 4); i += THREADS) {
    const int r = i / (p.xr / 4), k = 4 * (i - r * (p.xr / 4));
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r < n_rows)
      for (int q = 0; q < p.xdb.n; q += 4) {
        float4 v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
          v[e] = q + e < p.xdb.n ? __ldcs(reinterpret_cast<const float4 *>(p.xdb.p + (q + e) * p.xdb.stride + (size_t)(r0 + r) * p.xdb.ld + k))
                                 : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int e = 0; e < 4; ++e) { s.x += v[e].x; s.y += v[e].y; s.z += v[e].z; s.w += v[e].w; }
      }
    *reinterpret_cast<float4 *>(xs + r * p.xr + k) = s;
  }
  __syncthreads();
  float acc[R];
#pragma unroll
  for (int r = 0; r < R; ++r) acc[r] = 0.f;
#pragma unroll
  for (int i = 0; i < STEP_W; ++i) {
    const int k = kk + i * KG;
    if (k < p.rp) {
#pragma unroll
      for (int r = 0; r < R; ++r) acc[r] = fmaf(w[i], xs[r * p.xr + k], acc[r]);
    }
  }
  for (int k = kk + STEP_W * KG; k < p.rp; k += KG) {                // a rank that does not fit the registers
    const float wk = col ? (float)p.w_dt[(size_t)k * p.channels + c0 + ec] : 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) acc[r] = fmaf(wk, xs[r * p.xr + k], acc[r]);
  }
#pragma unroll
  for (int r = 0; r < R; ++r) red[kk][r][ec] = acc[r];
  __syncthreads();
  if (er < R) {
    float s = bias;
#pragma unroll
    for (int k = 0; k < KG; ++k) s += red[k][er][ec];
    const float d = softplus_t<EXACT>(s);
    sd[er][ec] = make_float2(d, d * u);
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const float2 d = sd[r][ch];
    const float *bc = xs + r * p.xr + p.rp + l * NS;
    float y = 0.f;
#pragma unroll
    for (int n = 0; n < NS; ++n) {
      S[r][n] = advance<EXACT>(d.x * A[n], S[r][n], d.y * bc[n]);
      y = fmaf(S[r][n], bc[NP + n], y);
    }
    if (on && r < n_rows) st_states<NS>(p.state + ((size_t)(r0 + r) * p.channels + c) * NP + l * NS, S[r]);
#pragma unroll
    for (int o = 1; o < LP; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (l == 0) sy[r][ch] = y;
  }
  __syncthreads();
  if (own) p.out[(size_t)(r0 + er) * p.out_ld + c0 + ec] = (T)(fmaf(skip, u, sy[er][ec]) * z * sigmoid_t<EXACT>(z) * p.scale);
}

template <typename T, int LP, int NS>
int32_t block_one(ugb_device *dev, const ugb_scan_args &a, const void *dt, const void *xdb, const void *z, size_t z_ld, int b, int t) {
  constexpr int CC = THREADS / LP;
  Block<T> p;
  p.u = (const T *)a.u; p.dt = (const T *)dt; p.xdb = (const T *)xdb; p.z = (const T *)z; p.a = a.a; p.skip = a.skip; p.dt_bias = a.dt_bias;
  p.state = a.state; p.out = (T *)a.out; p.z_ld = z_ld; p.out_ld = a.out_ld; p.scale = a.scale; p.channels = a.channels; p.xr = a.xr;
  p.rp = a.rp; p.t = t;
  selective_scan_kernel<T, LP, NS><<<dim3((a.channels + CC - 1) / CC, b), THREADS, 0, dev->stream>>>(p);
  return ugb_after_launch(dev, "selective_scan_kernel");
}
template <typename T, int LP, int NS>
int32_t step_one(ugb_device *dev, const ugb_scan_args &a, const void *w_dt, ugb_scan_partials xdb, ugb_scan_partials z, int rows, bool pdl, bool early) {
  constexpr int CC = THREADS / LP;
  Step<T> p;
  p.u = (const T *)a.u; p.w_dt = (const T *)w_dt; p.xdb = xdb; p.z = z; p.a = a.a; p.skip = a.skip; p.dt_bias = a.dt_bias; p.state = a.state;
  p.out = (T *)a.out; p.out_ld = a.out_ld; p.scale = a.scale; p.channels = a.channels; p.xr = a.xr; p.rp = a.rp; p.rows = rows;
  p.early = early && pdl ? 1 : 0;
  const cudaError_t e = ugb_launch(selective_step_kernel<T, LP, NS>, dim3((a.channels + CC - 1) / CC, (rows + STEP_ROWS - 1) / STEP_ROWS),
                                   dim3(THREADS), (size_t)STEP_ROWS * a.xr * 4, dev->stream, pdl, p);
  if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of selective_step_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(dev, "selective_step_kernel");
}

// f(LP, NS) for the kernel of a shape
template <typename F> int32_t with_shape(ugb_device *dev, const ugb_scan_shape &s, F f) {
#define SHAPE(LP, NS) if (s.lanes == LP && s.per_lane == NS) return f(std::integral_constant<int, LP>(), std::integral_constant<int, NS>())
  SHAPE(8, 1); SHAPE(8, 2); SHAPE(8, 3); SHAPE(8, 4); SHAPE(8, 6); SHAPE(8, 8); SHAPE(32, 4); SHAPE(32, 8);
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
  for (int ns : {1, 2, 3, 4, 6, 8})
    if (states <= 8 * ns) return {8, ns, 8 * ns};
  for (int ns : {4, 8})
    if (states <= 32 * ns) return {32, ns, 32 * ns};
  return {0, 0, 0};
}

float ugb_scan_decay_unit(bool f32) { return f32 ? 1.0f : 1.4426950408889634f; }

int32_t ugb_scan_block(ugb_device *dev, const ugb_scan_args &a, const void *dt, const void *xdb, const void *z, size_t z_ld, int b, int t) {
  if (b == 0 || t == 0) return UGB_OK;
  if (int32_t rc = check(dev, a)) return rc;
  UGB_REQUIRE(dev, z_ld % 8 == 0 && b <= 65535, UGB_ERR_SHAPE, "selective scan: %d sequences, gate rows %zu apart", b, z_ld);
  return with_shape(dev, a.shape, [&](auto lp, auto ns) {
    return a.f32 ? block_one<float, lp(), ns()>(dev, a, dt, xdb, z, z_ld, b, t) : block_one<__nv_bfloat16, lp(), ns()>(dev, a, dt, xdb, z, z_ld, b, t);
  });
}

int32_t ugb_scan_step(ugb_device *dev, const ugb_scan_args &a, const void *w_dt, ugb_scan_partials xdb, ugb_scan_partials z, int rows, bool pdl, bool early) {
  if (rows == 0) return UGB_OK;
  if (int32_t rc = check(dev, a)) return rc;
  UGB_REQUIRE(dev, (size_t)STEP_ROWS * a.xr * 4 <= 40 * 1024, UGB_ERR_UNSUPPORTED, "selective scan: %d columns of step size, B and C", a.xr);
  return with_shape(dev, a.shape, [&](auto lp, auto ns) {
    return a.f32 ? step_one<float, lp(), ns()>(dev, a, w_dt, xdb, z, rows, pdl, early) : step_one<__nv_bfloat16, lp(), ns()>(dev, a, w_dt, xdb, z, rows, pdl, early);
  });
}
