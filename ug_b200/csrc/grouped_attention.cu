// Grouped-query attention of single positions (see grouped_attention.cuh).
//
//   grouped_attention_mma_kernel      bf16, heads of 64 or 128: up to 16 query heads of one key / value head are the rows of
//                                     an mma.sync tile; every warp streams its own 16-key pieces through a private cp.async
//                                     ring with its own online softmax; the slices of a row are CTAs of a cluster
//   grouped_attention_generic_kernel  f32, and other head widths: plain FFMA
#include "grouped_attention.cuh"

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
  const void *q, *k, *v;
  void *out;
  size_t out_ld;
  float out_scale, scale;
  int t, pos_off, heads, kv_heads, dq, dv, t_max, splits, early;
  const int *pos_p;
  ugb_status_word *status;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Number of keys row r attends (position + 1), or 0 with the status word raised when the position is outside the cache.
__device__ __forceinline__ int keys_of(const Params &p, int r) {
  const int n = *p.pos_p + p.pos_off + r % p.t + 1;
  if (n < 1 || n > p.t_max) {
    if (threadIdx.x == 0 && atomicCAS(&p.status->code, 0u, (unsigned)UGB_ERR_INVALID) == 0u) p.status->detail = (unsigned)(n - 1);
    return 0;
  }
  return n;
}

// ---------------------------------------------------------------- bf16 ------
// grid (slices, key / value heads x groups of 16 query heads, rows), 128 threads.  A 16-key piece lies in shared memory as
// rows of DQ (DV) values, the 16-byte chunks of a 128-byte part XORed with the key.
constexpr int WARPS = 4, KT = 16, STAGES = 3;
template <int DQ, int DV> struct Ring {
  static constexpr int K_BYTES = KT * DQ * 2, V_BYTES = KT * DV * 2, STAGE = K_BYTES + V_BYTES;
  static constexpr int BYTES = WARPS * STAGES * STAGE;
  // after the last piece the ring holds the sums of the warps f32 [WARPS][16][DV], then those of the CTA [16][DV]
  static_assert((WARPS + 1) * 16 * DV * 4 <= BYTES, "sums fit the ring");
};

template <int DQ, int DV>
__global__ void __launch_bounds__(WARPS * 32)
grouped_attention_mma_kernel(Params p) {
  using R = Ring<DQ, DV>;
  extern __shared__ __align__(128) uint8_t ring[];
  __shared__ float2 wml[WARPS][16];                        // (max, sum) of a warp per head
  __shared__ float2 ml[16];                                // of this slice
  __shared__ float fac[16][UGB_GROUPED_MAX_SPLITS];        // weight of a slice's sums, 1 / sum included
  if (!p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const int share = p.heads / p.kv_heads, per_kv = (share + 15) / 16;
  const int sp = blockIdx.x, kvh = blockIdx.y / per_kv, hg = blockIdx.y % per_kv, r = blockIdx.z, b = r / p.t;
  const int head0 = kvh * share + hg * 16, n_heads = min(16, share - hg * 16);
  const int T = keys_of(p, r);
  if (T == 0) {                                            // the whole cluster leaves
    if (p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }
    return;
  }
  const int n_sub = (T + KT - 1) / KT, per = (n_sub + p.splits - 1) / p.splits;
  const int sub1 = min(n_sub, (sp + 1) * per), first = sp * per + warp;
  const __nv_bfloat16 *kb = (const __nv_bfloat16 *)p.k + ((size_t)b * p.kv_heads + kvh) * p.t_max * DQ;
  const __nv_bfloat16 *vb = (const __nv_bfloat16 *)p.v + ((size_t)b * p.kv_heads + kvh) * p.t_max * DV;
  const uint32_t mine = (uint32_t)__cvta_generic_to_shared(ring) + (uint32_t)warp * (STAGES * R::STAGE);
  auto at = [](int key, int ch, int row) { return (uint32_t)(key * row + (((ch & ~7) | ((ch ^ key) & 7)) << 4)); };
  auto issue = [&](int sub, int stage) {                   // t_max is a multiple of 16: a piece lies inside the cache
    if (sub < sub1) {
      const uint32_t ks = mine + stage * R::STAGE, vs = ks + R::K_BYTES;
      const __nv_bfloat16 *kg = kb + (size_t)sub * KT * DQ, *vg = vb + (size_t)sub * KT * DV;
#pragma unroll
      for (int i = 0; i < KT * DQ / 8 / 32; ++i) {
        const int c = lane + 32 * i;
        cp_async16(ks + at(c / (DQ / 8), c % (DQ / 8), DQ * 2), kg + c * 8);
      }
#pragma unroll
      for (int i = 0; i < KT * DV / 8 / 32; ++i) {
        const int c = lane + 32 * i;
        cp_async16(vs + at(c / (DV / 8), c % (DV / 8), DV * 2), vg + c * 8);
      }
    }
    cp_async_commit();                                     // always, so that the group count stays in step
  };
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) issue(first + s * WARPS, s);
  // queries: A fragments, rows = heads g and g + 8
  uint32_t qa[DQ / 16][4];
  {
    const __nv_bfloat16 *q = (const __nv_bfloat16 *)p.q + ((size_t)r * p.heads + head0) * DQ;
    auto ld2 = [&](int h, int col) -> uint32_t { return h < n_heads ? *reinterpret_cast<const uint32_t *>(q + (size_t)h * DQ + col) : 0u; };
#pragma unroll
    for (int k = 0; k < DQ / 16; ++k) {
      qa[k][0] = ld2(g, 16 * k + 2 * tq);
      qa[k][1] = ld2(g + 8, 16 * k + 2 * tq);
      qa[k][2] = ld2(g, 16 * k + 8 + 2 * tq);
      qa[k][3] = ld2(g + 8, 16 * k + 8 + 2 * tq);
    }
  }
  if (p.early) { ugb_pdl_wait(); ugb_pdl_trigger(); }

  const float scl = p.scale * 1.4426950408889634f;
  const int mi = lane >> 3, ri = lane & 7;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};  // of heads g and g + 8; l: this lane's keys
  float o[DV / 8][4];
#pragma unroll
  for (int d = 0; d < DV / 8; ++d) o[d][0] = o[d][1] = o[d][2] = o[d][3] = 0.f;
  int stage = 0;
  for (int sub = first; sub < sub1; sub += WARPS) {
    issue(sub + (STAGES - 1) * WARPS, (stage + STAGES - 1) % STAGES);
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 1) : "memory");
    __syncwarp();
    const uint32_t ks = mine + stage * R::STAGE, vs = ks + R::K_BYTES;
    float s[2][4];
#pragma unroll
    for (int e = 0; e < 4; ++e) s[0][e] = s[1][e] = 0.f;
#pragma unroll
    for (int k = 0; k < DQ / 16; ++k) {
      uint32_t f[4];
      asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                   : "=r"(f[0]), "=r"(f[1]), "=r"(f[2]), "=r"(f[3]) : "r"(ks + at(8 * (mi >> 1) + ri, 2 * k + (mi & 1), DQ * 2)));
      mma_bf16_16x8x16(s[0], qa[k][0], qa[k][1], qa[k][2], qa[k][3], f[0], f[1]);
      mma_bf16_16x8x16(s[1], qa[k][0], qa[k][1], qa[k][2], qa[k][3], f[2], f[3]);
    }
    const int key0 = sub * KT + 2 * tq;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[j][e] = key0 + 8 * j + (e & 1) < T ? s[j][e] * scl : -INFINITY;
        mx[e >> 1] = fmaxf(mx[e >> 1], s[j][e]);
      }
    float alpha[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
      mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
      const float mn = fmaxf(m[h], mx[h]);                 // finite: a piece starts below T
      alpha[h] = ex2(m[h] - mn);
      m[h] = mn;
      l[h] *= alpha[h];
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[j][e] = ex2(s[j][e] - m[e >> 1]);
        l[e >> 1] += s[j][e];
      }
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int d = 0; d < DV / 8; ++d) { o[d][0] *= alpha[0]; o[d][1] *= alpha[0]; o[d][2] *= alpha[1]; o[d][3] *= alpha[1]; }
    }
    const uint32_t a0 = pack_bf16(s[0][0], s[0][1]), a1 = pack_bf16(s[0][2], s[0][3]);
    const uint32_t a2 = pack_bf16(s[1][0], s[1][1]), a3 = pack_bf16(s[1][2], s[1][3]);
#pragma unroll
    for (int d = 0; d < DV / 8; d += 2) {
      uint32_t f[4];
      asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                   : "=r"(f[0]), "=r"(f[1]), "=r"(f[2]), "=r"(f[3]) : "r"(vs + at(ri + 8 * (mi & 1), d + (mi >> 1), DV * 2)));
      mma_bf16_16x8x16(o[d], a0, a1, a2, a3, f[0], f[1]);
      mma_bf16_16x8x16(o[d + 1], a0, a1, a2, a3, f[2], f[3]);
    }
    __syncwarp();
    stage = (stage + 1) % STAGES;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    if (tq == 0) wml[warp][g + 8 * h] = make_float2(m[h], l[h]);
  }
  __syncthreads();                                         // the ring is idle now
  float *wo = reinterpret_cast<float *>(ring), *co = wo + WARPS * 16 * DV;
#pragma unroll
  for (int d = 0; d < DV / 8; ++d)
#pragma unroll
    for (int h = 0; h < 2; ++h)
      *reinterpret_cast<float2 *>(wo + (warp * 16 + g + 8 * h) * DV + 8 * d + 2 * tq) = make_float2(o[d][2 * h], o[d][2 * h + 1]);
  __syncthreads();
  __nv_bfloat16 *out = (__nv_bfloat16 *)p.out + (size_t)r * p.out_ld + (size_t)head0 * DV;
  for (int idx = threadIdx.x; idx < n_heads * (DV / 4); idx += WARPS * 32) {
    const int h = idx / (DV / 4), c = 4 * (idx % (DV / 4));
    float mm = -INFINITY, ll = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) mm = fmaxf(mm, wml[w][h].x);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float2 s = wml[w][h];
      const float f = s.x == -INFINITY ? 0.f : ex2(s.x - mm);
      const float4 v = *reinterpret_cast<const float4 *>(wo + (w * 16 + h) * DV + c);
      ll = fmaf(f, s.y, ll);
      acc.x = fmaf(f, v.x, acc.x); acc.y = fmaf(f, v.y, acc.y); acc.z = fmaf(f, v.z, acc.z); acc.w = fmaf(f, v.w, acc.w);
    }
    if (p.splits == 1) {
      const float f = p.out_scale / ll;
      *reinterpret_cast<uint2 *>(out + (size_t)h * DV + c) = make_uint2(pack_bf16(acc.x * f, acc.y * f), pack_bf16(acc.z * f, acc.w * f));
    } else {
      *reinterpret_cast<float4 *>(co + h * DV + c) = acc;
      if (c == 0) ml[h] = make_float2(mm, ll);
    }
  }
  if (p.splits == 1) return;
  // The slices of a row are the CTAs of one cluster: after one barrier each combines its share of the elements, in slice
  // order, reading the peers' shared memory.
  cluster_sync_all();
  if (threadIdx.x < n_heads) {
    const int h = threadIdx.x;
    const uint32_t addr = smem_u32(&ml[h]);
    float2 v[UGB_GROUPED_MAX_SPLITS];
    float mm = -INFINITY, ll = 0.f;
#pragma unroll
    for (int s = 0; s < UGB_GROUPED_MAX_SPLITS; ++s) {
      v[s] = make_float2(-INFINITY, 0.f);
      if (s < p.splits)
        asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v[s].x), "=f"(v[s].y) : "r"(mapa_u32(addr, (uint32_t)s)) : "memory");
    }
#pragma unroll
    for (int s = 0; s < UGB_GROUPED_MAX_SPLITS; ++s) mm = fmaxf(mm, v[s].x);
#pragma unroll
    for (int s = 0; s < UGB_GROUPED_MAX_SPLITS; ++s) {
      v[s].x = v[s].x == -INFINITY ? 0.f : ex2(v[s].x - mm);
      ll = fmaf(v[s].x, v[s].y, ll);
    }
#pragma unroll
    for (int s = 0; s < UGB_GROUPED_MAX_SPLITS; ++s) fac[h][s] = v[s].x * (p.out_scale / ll);
  }
  __syncthreads();
  for (int idx = sp * (WARPS * 32) + threadIdx.x; idx < n_heads * (DV / 4); idx += p.splits * (WARPS * 32)) {
    const int h = idx / (DV / 4), c = 4 * (idx % (DV / 4));
    const uint32_t addr = smem_u32(co + h * DV + c);
    float4 v[UGB_GROUPED_MAX_SPLITS], acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < UGB_GROUPED_MAX_SPLITS; ++s) {
      v[s] = acc;
      if (s < p.splits)
        asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];"
                     : "=f"(v[s].x), "=f"(v[s].y), "=f"(v[s].z), "=f"(v[s].w) : "r"(mapa_u32(addr, (uint32_t)s)) : "memory");
    }
#pragma unroll
    for (int s = 0; s < UGB_GROUPED_MAX_SPLITS; ++s) {
      const float f = s < p.splits ? fac[h][s] : 0.f;
      acc.x = fmaf(f, v[s].x, acc.x); acc.y = fmaf(f, v[s].y, acc.y); acc.z = fmaf(f, v[s].z, acc.z); acc.w = fmaf(f, v[s].w, acc.w);
    }
    *reinterpret_cast<uint2 *>(out + (size_t)h * DV + c) = make_uint2(pack_bf16(acc.x, acc.y), pack_bf16(acc.z, acc.w));
  }
  cluster_sync_all();                                      // no CTA leaves while a peer may still read its shared memory
}

// ------------------------------------------------------------- generic ------
// grid (rows, key / value heads x groups of 8 query heads), 256 threads: warp = query head, lane = key of a tile of `kt` keys
// for the scores, lane = column (mod 32) for the sums.  Shared memory, all f32: queries [8][dq], sums [8][dv], keys
// [kt][dq + 1], values [kt][dv].
template <typename T>
__global__ void __launch_bounds__(256)
grouped_attention_generic_kernel(Params p, int kt) {
  extern __shared__ float gsm[];
  const int dq = p.dq, dv = p.dv, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float *qs = gsm, *os = qs + 8 * dq, *ks = os + 8 * dv, *vs = ks + kt * (dq + 1);
  ugb_pdl_wait();
  ugb_pdl_trigger();
  const int share = p.heads / p.kv_heads, per_kv = (share + 7) / 8;
  const int r = blockIdx.x, kvh = blockIdx.y / per_kv, in = (blockIdx.y % per_kv) * 8 + warp, b = r / p.t;
  const bool on = in < share;
  const int head = kvh * share + in, n = keys_of(p, r);
  if (n == 0) return;
  const T *q = (const T *)p.q + ((size_t)r * p.heads + head) * dq;
  for (int c = lane; c < dq; c += 32) qs[warp * dq + c] = on ? (float)q[c] : 0.f;
  for (int c = lane; c < dv; c += 32) os[warp * dv + c] = 0.f;
  const T *kc = (const T *)p.k + ((size_t)b * p.kv_heads + kvh) * p.t_max * dq, *vc = (const T *)p.v + ((size_t)b * p.kv_heads + kvh) * p.t_max * dv;
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < n; k0 += kt) {
    __syncthreads();
    for (int i = threadIdx.x; i < kt * dq; i += 256) {
      const int key = i / dq, c = i - key * dq;
      ks[key * (dq + 1) + c] = k0 + key < n ? (float)kc[(size_t)(k0 + key) * dq + c] : 0.f;
    }
    for (int i = threadIdx.x; i < kt * dv; i += 256) vs[i] = k0 + i / dv < n ? (float)vc[(size_t)k0 * dv + i] : 0.f;
    __syncthreads();
    float s = -INFINITY;
    if (lane < kt && k0 + lane < n) {
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      const float *kr = ks + lane * (dq + 1), *qr = qs + warp * dq;
      for (int c = 0; c < dq; c += 4)                      // dq % 8 == 0
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
    for (int c = lane; c - lane < dv; c += 32) {           // the warp stays together for the shuffles
      float a = c < dv ? os[warp * dv + c] * alpha : 0.f;
      for (int j = 0; j < keys; ++j) {
        const float wj = __shfl_sync(0xffffffffu, w, j);
        if (c < dv) a = fmaf(wj, vs[j * dv + c], a);
      }
      if (c < dv) os[warp * dv + c] = a;
    }
  }
  if (!on) return;
  const float f = p.out_scale / l;
  T *out = (T *)p.out + (size_t)r * p.out_ld + (size_t)head * dv;
  for (int c = lane; c < dv; c += 32) out[c] = (T)(os[warp * dv + c] * f);
}

size_t generic_smem(int dq, int dv, int kt) { return (size_t)(8 * (dq + dv) + kt * (dq + 1 + dv)) * 4; }
int generic_keys(int dq, int dv) {
  int kt = 32;
  while (kt > 1 && generic_smem(dq, dv, kt) > 200 * 1024) kt >>= 1;
  return kt;
}
bool fast(const ugb_grouped_attention_args &a) { return !a.f32 && (a.dq == 64 || a.dq == 128) && (a.dv == 64 || a.dv == 128) && a.t_max % KT == 0; }

template <int DQ, int DV> int32_t prepare_one(ugb_device *dev) {
  UGB_CUDA(dev, cudaFuncSetAttribute(grouped_attention_mma_kernel<DQ, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, Ring<DQ, DV>::BYTES));
  return UGB_OK;
}
template <int DQ, int DV> cudaError_t launch_one(dim3 grid, cudaStream_t st, bool pdl, const Params &p) {
  return ugb_launch_cluster(grouped_attention_mma_kernel<DQ, DV>, grid, dim3(WARPS * 32), Ring<DQ, DV>::BYTES, st, pdl, p.splits, p);
}

}  // namespace

int ugb_grouped_attention_splits(const ugb_grouped_attention_args &a, int sms) {
  const int pairs = a.rows * a.kv_heads * ((a.heads / a.kv_heads + 15) / 16);
  const int slots = a.dq + a.dv <= 128 ? 4 * sms : 2 * sms;    // CTAs that are resident together
  return std::max(1, std::min(UGB_GROUPED_MAX_SPLITS, slots / std::max(1, pairs)));
}

int32_t ugb_grouped_attention_prepare(ugb_device *dev) {
  int32_t rc;
  if ((rc = prepare_one<64, 64>(dev)) || (rc = prepare_one<64, 128>(dev)) || (rc = prepare_one<128, 64>(dev)) || (rc = prepare_one<128, 128>(dev))) return rc;
  UGB_CUDA(dev, cudaFuncSetAttribute(grouped_attention_generic_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
  UGB_CUDA(dev, cudaFuncSetAttribute(grouped_attention_generic_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
  return UGB_OK;
}

int32_t ugb_grouped_attention(ugb_device *dev, const ugb_grouped_attention_args &a) {
  if (a.rows == 0) return UGB_OK;
  UGB_REQUIRE(dev, a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dq % 8 == 0 && a.dv % 8 == 0 && a.dq > 0 && a.dv > 0,
              UGB_ERR_SHAPE, "grouped attention: %d query heads on %d, %d- and %d-wide", a.heads, a.kv_heads, a.dq, a.dv);
  Params p;
  p.q = a.q; p.k = a.k; p.v = a.v; p.out = a.out; p.out_ld = a.out_ld; p.out_scale = a.out_scale; p.scale = a.scale; p.t = a.t;
  p.pos_off = a.pos_off; p.heads = a.heads; p.kv_heads = a.kv_heads; p.dq = a.dq; p.dv = a.dv; p.t_max = a.t_max; p.splits = a.splits;
  p.early = a.early && a.pdl ? 1 : 0; p.pos_p = a.pos_p; p.status = dev->status_dev;
  const int share = a.heads / a.kv_heads;
  cudaError_t e;
  if (fast(a)) {
    UGB_REQUIRE(dev, a.splits >= 1 && a.splits <= UGB_GROUPED_MAX_SPLITS, UGB_ERR_INVALID, "grouped attention: %d slices", a.splits);
    UGB_REQUIRE(dev, a.rows <= 65535 && a.kv_heads * ((share + 15) / 16) <= 65535, UGB_ERR_UNSUPPORTED, "grouped attention: %d rows in one launch", a.rows);
    const dim3 grid((unsigned)a.splits, (unsigned)(a.kv_heads * ((share + 15) / 16)), (unsigned)a.rows);
    if (a.dq == 64) e = a.dv == 64 ? launch_one<64, 64>(grid, dev->stream, a.pdl, p) : launch_one<64, 128>(grid, dev->stream, a.pdl, p);
    else e = a.dv == 64 ? launch_one<128, 64>(grid, dev->stream, a.pdl, p) : launch_one<128, 128>(grid, dev->stream, a.pdl, p);
    if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of grouped_attention_mma_kernel failed: %s", cudaGetErrorString(e));
    return ugb_after_launch(dev, "grouped_attention_mma_kernel");
  }
  const int kt = generic_keys(a.dq, a.dv);
  const size_t smem = generic_smem(a.dq, a.dv, kt);
  UGB_REQUIRE(dev, smem <= 220 * 1024, UGB_ERR_UNSUPPORTED, "grouped attention: heads of %d and %d values do not fit the kernel", a.dq, a.dv);
  const dim3 grid((unsigned)a.rows, (unsigned)(a.kv_heads * ((share + 7) / 8)));
  if (a.f32) e = ugb_launch(grouped_attention_generic_kernel<float>, grid, dim3(256), smem, dev->stream, a.pdl, p, kt);
  else e = ugb_launch(grouped_attention_generic_kernel<__nv_bfloat16>, grid, dim3(256), smem, dev->stream, a.pdl, p, kt);
  if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of grouped_attention_generic_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(dev, "grouped_attention_generic_kernel");
}
