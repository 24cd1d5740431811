// Latent attention in the absorbed form (see latent_attention.cuh): used for decode steps, for short blocks of new
// positions, and for every block when the model runs in 32 bits.
//
//   latent_attention_mma_kernel      bf16, mma.sync: 16 heads are the rows of the tile, a CTA streams its slice of the
//                                    cache once through a cp.async ring and uses every tile twice (scores, sums)
//   latent_attention_generic_kernel  f32 (or a row width the fast path has no kernel for): plain FFMA
#include "latent_attention.cuh"

#include <algorithm>

#include "decode_kernels.cuh"

namespace {

using ugb_decode::cp_async16;
using ugb_decode::cp_async_commit;
using ugb_decode::mma_bf16_16x8x16;
using ugb_decode::pack_bf16;
using ugb_tc::cluster_sync_all;
using ugb_tc::mapa_u32;
using ugb_tc::smem_u32;

struct Params {
  const void *q, *cache;
  void *out;
  const float *gate;
  int t, pos_off, heads, ld, t_max, gate_ld, splits, early;
  const int *pos_p;
  float scale;
  ugb_status_word *status;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Number of keys row r attends (position + 1), or 0 with the status word raised when the position is outside the cache.
__device__ __forceinline__ int keys_of(const Params &p, int r) {
  const int T = *p.pos_p + p.pos_off + r % p.t + 1;
  if (T < 1 || T > p.t_max) {
    if (threadIdx.x == 0 && atomicCAS(&p.status->code, 0u, (unsigned)UGB_ERR_INVALID) == 0u) p.status->detail = (unsigned)(T - 1);
    return 0;
  }
  return T;
}

// ---------------------------------------------------------------- bf16 ------
// grid (splits, head groups of 16, rows), 256 threads, cache rows of 64 NT elements.
// A 32-key tile lies in shared memory as rows of NT 128-byte pieces, the 16-byte chunks of a piece XORed with the key
// (the 128-byte swizzle): ldmatrix over 8 keys of one chunk column is conflict-free, plain and transposed.
//   scores   warp w: keys 16 (w & 1) .. + 15 over quarter w >> 1 of the latent; the quarters meet in shared memory
//   softmax  warp w: heads w and w + 8, a lane per key (fp32, online); probabilities to shared memory as bf16
//   sums     warp w: latent columns 8 NT w .. + 8 NT - 1
// The ring matters more than the arithmetic: of STAGES tiles one is worked on, the others are in flight.
constexpr int KT = 32;
constexpr int WARPS = 8;
template <int NT> struct Ring {
  static constexpr int ROW = NT * 128;                     // bytes of a cache row
  static constexpr int TILE = KT * ROW;
  static constexpr int STAGES = NT >= 8 ? 3 : (NT >= 4 ? 4 : 6);
  static constexpr int BYTES = STAGES * TILE;
};

template <int NT>
__global__ void __launch_bounds__(WARPS * 32, 2)
latent_attention_mma_kernel(Params p) {
  using R = Ring<NT>;
  extern __shared__ __align__(128) uint8_t ring[];
  __shared__ float sc[4][16][KT + 8];                      // [latent quarter][head][key]; the pitch keeps 8-byte accesses conflict-free
  __shared__ __align__(16) __nv_bfloat16 pr[16][KT + 8];   // probabilities; pitch of 80 bytes: conflict-free ldmatrix
  __shared__ float al[16];                                 // factor the sums so far take on
  __shared__ float2 ml[16];                                // (max, sum) of this slice per head
  __shared__ float fac[16][UGB_LATENT_MAX_SPLITS];         // weight of a slice's sums, gate and 1 / sum included
  if (!p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
  const int sp = blockIdx.x, hg = blockIdx.y, r = blockIdx.z, b = r / p.t;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  constexpr int LD = NT * 64;
  const int head0 = hg * 16, n_heads = min(16, p.heads - head0);
  const int T = keys_of(p, r);
  if (T == 0) {                                            // the whole cluster leaves
    if (p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
    return;
  }
  const int n_tiles = (T + KT - 1) / KT, per = (n_tiles + p.splits - 1) / p.splits;
  const int tile0 = sp * per, tile1 = min(n_tiles, tile0 + per);
  const __nv_bfloat16 *cache = (const __nv_bfloat16 *)p.cache + (size_t)b * p.t_max * LD;
  const uint32_t ring_u = (uint32_t)__cvta_generic_to_shared(ring);

  auto issue = [&](int tile) {                             // always commits, so the group count stays in step
    if (tile < tile1) {
      const int st = (tile - tile0) % R::STAGES;
      for (int c = threadIdx.x; c < KT * NT * 8; c += WARPS * 32) {
        const int key = c / (NT * 8), ch = c % (NT * 8);
        const uint32_t dst = (uint32_t)st * R::TILE + key * R::ROW + (((ch & ~7) | ((ch ^ key) & 7)) << 4);
        const int pos = tile * KT + key;
        if (pos < p.t_max) cp_async16(ring_u + dst, cache + (size_t)pos * LD + ch * 8);
        else *reinterpret_cast<uint4 *>(ring + dst) = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    cp_async_commit();
  };
  // early: only the newest position's row (in the last tile) comes from a kernel that may still be running
  const int pre = p.early ? max(0, min(R::STAGES - 1, n_tiles - 1 - tile0)) : 0;
#pragma unroll
  for (int s = 0; s < R::STAGES - 1; ++s)
    if (s < pre) issue(tile0 + s);
  if (p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
#pragma unroll
  for (int s = 0; s < R::STAGES - 1; ++s)
    if (s >= pre) issue(tile0 + s);

  // queries of this warp's quarter of the latent: A fragments, rows = heads g and g + 8
  const int quarter = warp >> 1, kp = warp & 1;
  uint32_t qa[NT][4];
  {
    const __nv_bfloat16 *q = (const __nv_bfloat16 *)p.q + ((size_t)r * p.heads + head0) * LD + quarter * (LD / 4);
    auto ld2 = [&](int h, int col) -> uint32_t { return h < n_heads ? *reinterpret_cast<const uint32_t *>(q + (size_t)h * LD + col) : 0u; };
#pragma unroll
    for (int k = 0; k < NT; ++k) {
      qa[k][0] = ld2(g, 16 * k + 2 * tq);
      qa[k][1] = ld2(g + 8, 16 * k + 2 * tq);
      qa[k][2] = ld2(g, 16 * k + 8 + 2 * tq);
      qa[k][3] = ld2(g + 8, 16 * k + 8 + 2 * tq);
    }
  }
  const int mi = lane >> 3, ri = lane & 7;
  auto scores = [&](int tile) {
    const uint32_t base = ring_u + (uint32_t)((tile - tile0) % R::STAGES) * R::TILE;
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
    const int key = 16 * kp + 8 * (mi >> 1) + ri;
    const uint32_t row = base + key * R::ROW;
    constexpr int G = NT < 4 ? NT : 4;                     // operand loads issued ahead of their products
#pragma unroll
    for (int k0 = 0; k0 < NT; k0 += G) {
      uint32_t bf[G][4];
#pragma unroll
      for (int k = 0; k < G; ++k) {
        if (k0 + k >= NT) continue;
        const int ch = quarter * (NT * 2) + 2 * (k0 + k) + (mi & 1);
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                     : "=r"(bf[k][0]), "=r"(bf[k][1]), "=r"(bf[k][2]), "=r"(bf[k][3])
                     : "r"(row + (((ch & ~7) | ((ch ^ key) & 7)) << 4)));
      }
#pragma unroll
      for (int k = 0; k < G; ++k) {
        if (k0 + k >= NT) continue;
        const uint32_t (&a)[4] = qa[k0 + k];
        mma_bf16_16x8x16(s0, a[0], a[1], a[2], a[3], bf[k][0], bf[k][1]);
        mma_bf16_16x8x16(s1, a[0], a[1], a[2], a[3], bf[k][2], bf[k][3]);
      }
    }
    float (*dst)[KT + 8] = sc[quarter];
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      *reinterpret_cast<float2 *>(&dst[g + 8 * rr][16 * kp + 2 * tq]) = make_float2(s0[2 * rr], s0[2 * rr + 1]);
      *reinterpret_cast<float2 *>(&dst[g + 8 * rr][16 * kp + 8 + 2 * tq]) = make_float2(s1[2 * rr], s1[2 * rr + 1]);
    }
  };

  const float scl = p.scale * 1.4426950408889634f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};  // of heads warp and warp + 8; l: this lane's keys
  float o[NT][4];
#pragma unroll
  for (int d = 0; d < NT; ++d) o[d][0] = o[d][1] = o[d][2] = o[d][3] = 0.f;
  const int chunk0 = warp * NT;                            // first 16-byte chunk of this warp's columns

  for (int j = tile0; j < tile1; ++j) {
    // tile j has landed, and nobody works on tile j - 1 any more
    asm volatile("cp.async.wait_group %0;" ::"n"(R::STAGES - 2) : "memory");
    __syncthreads();
    issue(j + R::STAGES - 1);
    scores(j);
    __syncthreads();
    {
      float f[2], mx[2];
      const bool seen = j * KT + lane < T;
#pragma unroll
      for (int rr = 0; rr < 2; ++rr) {
        const int row = warp + 8 * rr;
        f[rr] = seen ? ((sc[0][row][lane] + sc[1][row][lane]) + (sc[2][row][lane] + sc[3][row][lane])) * scl : -INFINITY;
        mx[rr] = f[rr];
      }
#pragma unroll
      for (int s = 16; s > 0; s >>= 1)
#pragma unroll
        for (int rr = 0; rr < 2; ++rr) mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], s));
#pragma unroll
      for (int rr = 0; rr < 2; ++rr) {
        const float mn = fmaxf(m[rr], mx[rr]);             // finite: a tile starts below T
        const float alpha = ex2(m[rr] - mn), pv = ex2(f[rr] - mn);
        m[rr] = mn;
        l[rr] = l[rr] * alpha + pv;
        pr[warp + 8 * rr][lane] = __float2bfloat16_rn(pv);
        if (lane == 0) al[warp + 8 * rr] = alpha;
      }
    }
    __syncthreads();
    const float a0 = al[g], a1 = al[g + 8];
    if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
      for (int d = 0; d < NT; ++d) { o[d][0] *= a0; o[d][1] *= a0; o[d][2] *= a1; o[d][3] *= a1; }
    }
    uint32_t pa[2][4];
#pragma unroll
    for (int kk = 0; kk < 2; ++kk)                         // rows 0-7, 8-15 of keys 16 kk .. + 7, then of + 8 .. + 15
      asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                   : "=r"(pa[kk][0]), "=r"(pa[kk][1]), "=r"(pa[kk][2]), "=r"(pa[kk][3])
                   : "r"(smem_u32(&pr[ri + 8 * (mi & 1)][16 * kk + 8 * (mi >> 1)])));
    const uint32_t base = ring_u + (uint32_t)((j - tile0) % R::STAGES) * R::TILE;
#pragma unroll
    for (int kk = 0; kk < 2; ++kk) {
      const int key = 16 * kk + ri + 8 * (mi & 1);
      if constexpr (NT % 2 == 0) {
        uint32_t bf[NT / 2][4];
#pragma unroll
        for (int d = 0; d < NT / 2; ++d) {
          const int ch = chunk0 + 2 * d + (mi >> 1);
          asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                       : "=r"(bf[d][0]), "=r"(bf[d][1]), "=r"(bf[d][2]), "=r"(bf[d][3])
                       : "r"(base + key * R::ROW + (((ch & ~7) | ((ch ^ key) & 7)) << 4)));
        }
#pragma unroll
        for (int d = 0; d < NT / 2; ++d) {
          mma_bf16_16x8x16(o[2 * d], pa[kk][0], pa[kk][1], pa[kk][2], pa[kk][3], bf[d][0], bf[d][1]);
          mma_bf16_16x8x16(o[2 * d + 1], pa[kk][0], pa[kk][1], pa[kk][2], pa[kk][3], bf[d][2], bf[d][3]);
        }
      } else {
#pragma unroll
        for (int d = 0; d < NT; ++d) {
          const int ch = chunk0 + d;
          uint32_t b0, b1;
          asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];"
                       : "=r"(b0), "=r"(b1) : "r"(base + key * R::ROW + (((ch & ~7) | ((ch ^ key) & 7)) << 4)));
          mma_bf16_16x8x16(o[d], pa[kk][0], pa[kk][1], pa[kk][2], pa[kk][3], b0, b1);
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int rr = 0; rr < 2; ++rr) {
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) l[rr] += __shfl_xor_sync(0xffffffffu, l[rr], s);
    if (lane == 0) ml[warp + 8 * rr] = make_float2(m[rr], l[rr]);
  }
  __nv_bfloat16 *out = (__nv_bfloat16 *)p.out + ((size_t)r * p.heads + head0) * LD;
  if (p.splits == 1) {
    __syncthreads();
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      const int h = g + 8 * rr;
      if (h >= n_heads) continue;
      const float f = (p.gate ? p.gate[(size_t)r * p.gate_ld + head0 + h] : 1.f) / ml[h].y;
#pragma unroll
      for (int d = 0; d < NT; ++d)
        *reinterpret_cast<uint32_t *>(out + (size_t)h * LD + (chunk0 + d) * 8 + 2 * tq) = pack_bf16(o[d][2 * rr] * f, o[d][2 * rr + 1] * f);
    }
    return;
  }
  // The slices of a (row, head group) are the CTAs of one cluster.  Every slice leaves its sums and its (max, sum) in its
  // own shared memory (the ring is idle now); after one cluster barrier each CTA combines its share of the elements,
  // in slice order, reading the peers' shared memory.
  __syncthreads();
  float *os = reinterpret_cast<float *>(ring);             // [16][LD], exactly one ring stage
#pragma unroll
  for (int rr = 0; rr < 2; ++rr) {
    float *po = os + (g + 8 * rr) * LD;
#pragma unroll
    for (int d = 0; d < NT; ++d) *reinterpret_cast<float2 *>(po + (chunk0 + d) * 8 + 2 * tq) = make_float2(o[d][2 * rr], o[d][2 * rr + 1]);
  }
  cluster_sync_all();
  if (threadIdx.x < 16) {
    const int h = threadIdx.x;
    const uint32_t addr = smem_u32(&ml[h]);
    float2 v[UGB_LATENT_MAX_SPLITS];
    float mm = -INFINITY;
#pragma unroll
    for (int s = 0; s < UGB_LATENT_MAX_SPLITS; ++s) {
      v[s] = make_float2(-INFINITY, 0.f);
      if (s < p.splits)
        asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v[s].x), "=f"(v[s].y) : "r"(mapa_u32(addr, (uint32_t)s)) : "memory");
    }
#pragma unroll
    for (int s = 0; s < UGB_LATENT_MAX_SPLITS; ++s) mm = fmaxf(mm, v[s].x);
    float ll = 0.f;
#pragma unroll
    for (int s = 0; s < UGB_LATENT_MAX_SPLITS; ++s) {
      v[s].x = v[s].x == -INFINITY ? 0.f : ex2(v[s].x - mm);
      ll += v[s].x * v[s].y;
    }
    const float k = h < n_heads ? (p.gate ? p.gate[(size_t)r * p.gate_ld + head0 + h] : 1.f) / ll : 0.f;
#pragma unroll
    for (int s = 0; s < UGB_LATENT_MAX_SPLITS; ++s) fac[h][s] = v[s].x * k;
  }
  __syncthreads();
  for (int idx = sp * (WARPS * 32) + threadIdx.x; idx < n_heads * (LD / 4); idx += p.splits * (WARPS * 32)) {
    const int h = idx / (LD / 4), c = (idx % (LD / 4)) * 4;
    const uint32_t addr = smem_u32(os + h * LD + c);
    float4 v[UGB_LATENT_MAX_SPLITS], acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < UGB_LATENT_MAX_SPLITS; ++s) {
      v[s] = acc;
      if (s < p.splits)
        asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];"
                     : "=f"(v[s].x), "=f"(v[s].y), "=f"(v[s].z), "=f"(v[s].w) : "r"(mapa_u32(addr, (uint32_t)s)) : "memory");
    }
#pragma unroll
    for (int s = 0; s < UGB_LATENT_MAX_SPLITS; ++s) {
      const float f = s < p.splits ? fac[h][s] : 0.f;
      acc.x = fmaf(f, v[s].x, acc.x); acc.y = fmaf(f, v[s].y, acc.y); acc.z = fmaf(f, v[s].z, acc.z); acc.w = fmaf(f, v[s].w, acc.w);
    }
    *reinterpret_cast<uint2 *>(out + (size_t)h * LD + c) = make_uint2(pack_bf16(acc.x, acc.y), pack_bf16(acc.z, acc.w));
  }
  cluster_sync_all();                                      // no CTA leaves while a peer may still read its shared memory
}

// ------------------------------------------------------------- generic ------
// grid (rows, groups of 8 heads), 256 threads: warp = head, lane = key of a tile of `kt` keys for the scores, lane =
// latent column (mod 32) for the sums.  Shared memory: queries and sums [8][ld], keys [kt][ld + 1], all f32.
template <typename T>
__global__ void __launch_bounds__(256)
latent_attention_generic_kernel(Params p, int kt) {
  extern __shared__ float gsm[];
  const int ld = p.ld, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float *qs = gsm, *os = qs + 8 * ld, *ks = os + 8 * ld;
  ugb_pdl_wait();
  ugb_pdl_trigger();
  const int r = blockIdx.x, head = blockIdx.y * 8 + warp, b = r / p.t;
  const bool on = head < p.heads;
  const int n = keys_of(p, r);
  if (n == 0) return;
  const T *q = (const T *)p.q + ((size_t)r * p.heads + head) * ld;
  for (int c = lane; c < ld; c += 32) {
    qs[warp * ld + c] = on ? (float)q[c] : 0.f;
    os[warp * ld + c] = 0.f;
  }
  const T *cache = (const T *)p.cache + (size_t)b * p.t_max * ld;
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < n; k0 += kt) {
    __syncthreads();
    for (int i = threadIdx.x; i < kt * ld; i += 256) {
      const int key = i / ld, c = i - key * ld;
      ks[key * (ld + 1) + c] = k0 + key < n ? (float)cache[(size_t)(k0 + key) * ld + c] : 0.f;
    }
    __syncthreads();
    float s = -INFINITY;
    if (lane < kt && k0 + lane < n) {
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      const float *kr = ks + lane * (ld + 1), *qr = qs + warp * ld;
      for (int c = 0; c < ld; c += 4)                      // ld % 8 == 0
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[e] = fmaf(qr[c + e], kr[c + e], acc[e]);
      s = ((acc[0] + acc[1]) + (acc[2] + acc[3])) * p.scale;
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float mn = fmaxf(m, mx), alpha = expf(m - mn), w = s == -INFINITY ? 0.f : expf(s - mn);
    float sum = w;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    l = l * alpha + sum;
    m = mn;
    const int keys = min(kt, n - k0);
    for (int c = lane; c - lane < ld; c += 32) {           // the warp stays together for the shuffles
      float a = c < ld ? os[warp * ld + c] * alpha : 0.f;
      for (int j = 0; j < keys; ++j) {
        const float wj = __shfl_sync(0xffffffffu, w, j);
        if (c < ld) a = fmaf(wj, ks[j * (ld + 1) + c], a);
      }
      if (c < ld) os[warp * ld + c] = a;
    }
  }
  if (!on) return;
  const float f = (p.gate ? p.gate[(size_t)r * p.gate_ld + head] : 1.f) / l;
  T *out = (T *)p.out + ((size_t)r * p.heads + head) * ld;
  for (int c = lane; c < ld; c += 32) out[c] = (T)(os[warp * ld + c] * f);
}

int generic_keys(int ld) {                                 // keys per tile that fit in 200 KiB beside queries and sums
  int kt = 32;
  while (kt > 1 && (size_t)(16 * ld + kt * (ld + 1)) * 4 > 200 * 1024) kt >>= 1;
  return kt;
}

template <int NT> int32_t prepare_one(ugb_device *dev) {
  UGB_CUDA(dev, cudaFuncSetAttribute(latent_attention_mma_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, Ring<NT>::BYTES));
  return UGB_OK;
}
template <int NT> cudaError_t launch_one(dim3 grid, cudaStream_t st, bool pdl, const Params &p) {
  return ugb_launch_cluster(latent_attention_mma_kernel<NT>, grid, dim3(WARPS * 32), Ring<NT>::BYTES, st, pdl, p.splits, p);
}

}  // namespace

int ugb_latent_row_width(int rank) {
  for (int nt : {1, 2, 4, 6, 8})
    if (rank <= nt * 64) return nt * 64;
  return 0;
}

int32_t ugb_latent_attention_prepare(ugb_device *dev) {
  int32_t rc;
  if ((rc = prepare_one<1>(dev)) || (rc = prepare_one<2>(dev)) || (rc = prepare_one<4>(dev)) || (rc = prepare_one<6>(dev)) ||
      (rc = prepare_one<8>(dev)))
    return rc;
  UGB_CUDA(dev, cudaFuncSetAttribute(latent_attention_generic_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
  UGB_CUDA(dev, cudaFuncSetAttribute(latent_attention_generic_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
  return UGB_OK;
}

int32_t ugb_latent_attention(ugb_device *dev, const ugb_latent_attention_args &a) {
  if (a.rows == 0) return UGB_OK;
  Params p;
  p.q = a.q; p.cache = a.cache; p.out = a.out; p.gate = a.gate; p.t = a.t; p.pos_off = a.pos_off; p.heads = a.heads;
  p.ld = a.ld; p.t_max = a.t_max; p.gate_ld = a.gate_ld; p.splits = a.splits; p.pos_p = a.pos_p; p.scale = a.scale;
  p.early = a.early && a.pdl ? 1 : 0; p.status = dev->status_dev;
  cudaError_t e;
  if (!a.f32 && ugb_latent_row_width(a.ld) == a.ld) {
    UGB_REQUIRE(dev, a.splits >= 1 && a.splits <= UGB_LATENT_MAX_SPLITS, UGB_ERR_INVALID, "latent attention: %d slices", a.splits);
    UGB_REQUIRE(dev, a.rows <= 65535, UGB_ERR_UNSUPPORTED, "latent attention: %d rows in one launch", a.rows);
    const dim3 grid((unsigned)a.splits, (unsigned)((a.heads + 15) / 16), (unsigned)a.rows);
    switch (a.ld / 64) {
      case 1: e = launch_one<1>(grid, dev->stream, a.pdl, p); break;
      case 2: e = launch_one<2>(grid, dev->stream, a.pdl, p); break;
      case 4: e = launch_one<4>(grid, dev->stream, a.pdl, p); break;
      case 6: e = launch_one<6>(grid, dev->stream, a.pdl, p); break;
      default: e = launch_one<8>(grid, dev->stream, a.pdl, p); break;
    }
    if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of latent_attention_mma_kernel failed: %s", cudaGetErrorString(e));
    return ugb_after_launch(dev, "latent_attention_mma_kernel");
  }
  const int kt = generic_keys(a.ld);
  const size_t smem = (size_t)(16 * a.ld + kt * (a.ld + 1)) * 4;
  UGB_REQUIRE(dev, smem <= 220 * 1024, UGB_ERR_UNSUPPORTED, "latent attention: a latent of %d values does not fit the kernel", a.ld);
  const dim3 grid((unsigned)a.rows, (unsigned)((a.heads + 7) / 8));
  if (a.f32) e = ugb_launch(latent_attention_generic_kernel<float>, grid, dim3(256), smem, dev->stream, a.pdl, p, kt);
  else e = ugb_launch(latent_attention_generic_kernel<__nv_bfloat16>, grid, dim3(256), smem, dev->stream, a.pdl, p, kt);
  if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of latent_attention_generic_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(dev, "latent_attention_generic_kernel");
}
