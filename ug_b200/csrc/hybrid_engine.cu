// Decoders described by a list of layers (ugb_hybrid_*).  The step loop, its CUDA graph, the prompt loop and weight upload
// are those of engine_core.cuh; the products run on the tcgen05 GEMM (bf16) or the FP32-pipe kernels (f32).  This file holds
// the model's life cycle and the sandwich form of a layer -- token mixers of several kinds behind one chain of sandwich
// norms, input convolutions and a depth average; the parallel form is in hybrid_parallel.cu.
//
// Launches of a sandwich layer (T = activation type):
//   row_update     stream += norm(previous product); layer bank, depth average; norm -> T   [decode: + convolution]
//   causal_conv    prompts only: the input convolution over the block
//   mingru:        GEMM z|u|g -> f32;  min_gru_step (decode) / min_gru_scan (prompt) -> T;  GEMM out -> f32
//   latent att.:   GEMM query latent | kv latent | gates -> f32;  latent_inputs (both norms, cache append, gates);
//                  GEMM queries;  then either, for decode steps and short blocks, per-head GEMM into the latent space,
//                  attention over the cached latents, per-head GEMM out of it, or, for longer blocks, GEMMs that expand
//                  the cached latents to keys and values and the causal tcgen05 kernel;  GEMM out -> f32
//   row_update     stream += norm(mixer); norm -> T                                          [decode: + convolution]
//   causal_conv    prompts only
//   GEMM up with max(x, 0)^2 in the epilogue;  GEMM down -> f32
// Products with a f32 result are split over k in a decode step; the consumer sums the partials.
//
// Padding: every width is rounded up to 8 (TMA rows of 16 bytes), head widths to 64 or 128 where the tcgen05 attention
// takes them and latents to what latent_attention.cu takes; padded weight rows and columns, gains and biases are zero.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <string>
#include <vector>

#include "attention_tc.cuh"
#include "decode_kernels.cuh"
#include "gemm_tcgen05.cuh"
#include "grouped_attention.cuh"
#include "hybrid_engine.cuh"
#include "latent_attention.cuh"

using namespace ugb_hybrid_k;

using Mat = ugb_hybrid_mat;
using Tiling = ugb_hybrid_tiling;
static size_t up8(size_t n) { return ugb_up8(n); }

int ugb_hybrid::att_splits() const {
  if (att_splits_opt > 0) return std::min(att_splits_opt, (int)UGB_LATENT_MAX_SPLITS);
  // two CTAs per SM over the (row, group of 16 heads) pairs
  int heads = 1;
  for (const ugb_hybrid_weights &L : layers) heads = std::max(heads, L.d.heads);
  const int pairs = batch * ((heads + 15) / 16);
  return std::max(1, std::min((int)UGB_LATENT_MAX_SPLITS, 2 * dev->sm_count / pairs));
}

int32_t ugb_hybrid_alloc(ugb_hybrid *m, void **p, size_t bytes, bool zero) {
  unsigned char *b = nullptr;
  if (int32_t rc = dmalloc(m, &b, bytes, zero)) return rc;
  *p = b;
  return UGB_OK;
}

int32_t ugb_hybrid_matmul(ugb_hybrid *m, const Mat &x) {
  ugb_device *dev = m->dev;
  if (m->f32) {
    if (x.groups)
      return ugb_f32_grouped_gemm(dev, (float *)x.out, (const float *)x.a, (const float *)x.w, x.groups, x.m, x.tile, (int)x.n, (int)x.k);
    int32_t rc = ugb_f32_gemm(dev, (float *)x.out, (const float *)x.a, (const float *)x.w, x.batch, x.m, x.n, x.k,
                              x.a_ld ? x.a_ld : x.k, x.a_batch, x.nk, x.w_batch, x.c_ld ? x.c_ld : x.n,
                              x.c_batch ? x.c_batch : x.m * (x.c_ld ? x.c_ld : x.n));
    if (rc || !(x.relu2 || x.silu_mul)) return rc;
    if (x.silu_mul) return ugb_fail(dev, UGB_ERR_UNSUPPORTED, "f32 product with a fused gate");
    relu2_kernel<<<dev->sm_count * 4, 256, 0, dev->stream>>>((float *)x.out, x.m * x.n / 4);
    return ugb_after_launch(dev, "relu2_kernel");
  }
  ugb_tc_gemm_args g;
  g.out = x.out; g.a = x.a; g.b = x.w;
  g.batch = x.batch; g.m = x.m; g.n = x.n; g.k = x.k;
  g.a_batch = (long long)x.a_batch; g.b_batch = (long long)x.w_batch; g.c_batch = (long long)x.c_batch;
  g.a_ld = x.a_ld == x.k ? 0 : (long long)x.a_ld; g.c_ld = x.c_ld == x.n ? 0 : (long long)x.c_ld;
  g.b_is_nk = x.nk;
  g.epi = x.relu2 ? UGB_EPI_RELU2_BF16 : x.silu_mul ? UGB_EPI_SILU_MUL_BF16 : (x.f32_out ? UGB_EPI_F32 : UGB_EPI_BF16);
  if (x.silu_mul) g.c_ld = x.c_ld == x.n / 2 ? 0 : (long long)x.c_ld;
  g.splits = x.splits; g.bn = x.bn; g.b_static = x.groups == nullptr; g.pdl = m->pdl != 0; g.late_trigger = true;
  g.groups = x.groups; g.n_groups = x.n_groups; g.tile_m = x.tile;
  g.smem_kib = x.m <= 64 || (x.groups && x.tile == 64) ? 144 : 0;
  if (!x.f32_out && !x.groups && x.batch == 1 && x.nk && x.m <= 64 && x.k >= 256) {
    // a T result cannot be split into partials: the two k halves of a tile on a pair of CTAs, with the narrowest tile that fits the SMs
    for (int bn : {64, 96, 128, 160})
      if ((x.n + bn - 1) / bn * 2 <= (size_t)dev->sm_count) {
        g.bn = bn;
        g.pair_k = true;
        const int32_t rc = ugb_tc_gemm(dev, g);
        if (rc != UGB_ERR_UNSUPPORTED) return rc;
        break;
      }
    g.bn = x.bn;
    g.pair_k = false;
  }
  const int32_t rc = ugb_tc_gemm(dev, g);
  if (rc == UGB_ERR_UNSUPPORTED)
    return ugb_fail(dev, rc, "GEMM m=%zu n=%zu k=%zu does not meet the tensor-core kernel's shape rules", x.m, x.n, x.k);
  return rc;
}

// As many CTAs as SMs, no fewer than two k blocks each
Tiling ugb_hybrid_tile(const ugb_hybrid *m, size_t n, size_t k) {
  if (m->f32 || m->batch > 64) return {0, 1};
  // A CTA's time goes with its k blocks and hardly with its tile width (an MMA of 64 rows costs the same up to 160
  // columns), so: the fewest k blocks per CTA over widths and splits that fit one wave, then the fewest partials,
  // then the narrowest tile.
  const int sms = m->dev->sm_count, kb = (int)((k + 63) / 64);
  Tiling best{128, 1};
  int best_kb = kb + 1;
  for (int s = 1; s <= std::min(UGB_HYBRID_MAX_SPLITS, kb); ++s)
    for (int bn : {64, 80, 96, 128, 160}) {
      const int tiles = (int)((n + bn - 1) / bn), per = (kb + s - 1) / s;
      if (tiles * s > sms || per >= best_kb) continue;
      best = {bn, s};
      best_kb = per;
    }
  if (best_kb > kb) return {256, 1};           // more tiles than SMs whatever the width
  return {best.bn, ugb_tc_gemm_effective_splits(k, best.splits)};
}

template <typename T> int32_t ugb_hybrid_rows(ugb_hybrid *m, RowArgs<T> &a, int rows, bool early) {
  if (!m->on(UGB_HYBRID_K_ROWS)) return UGB_OK;
  a.early = early ? 1 : 0;
  a.ld = m->wl; a.inv_width = 1.0f / (float)m->cfg.width; a.eps = m->cfg.eps; a.status = m->dev->status_dev;
  const int nvec = m->wl / 4;
  cudaStream_t st = m->dev->stream;
  const bool pdl = m->pdl != 0;
  const bool step = rows <= m->dev->sm_count;
  auto *k = nvec <= 256    ? (step ? row_update_kernel<T, 1, true> : row_update_kernel<T, 1, false>)
            : nvec <= 512  ? (step ? row_update_kernel<T, 2, true> : row_update_kernel<T, 2, false>)
            : nvec <= 1024 ? (step ? row_update_kernel<T, 4, true> : row_update_kernel<T, 4, false>)
                           : row_update_kernel<T, 8, false>;
  const cudaError_t e = ugb_launch(k, dim3(rows), dim3(256), 0, st, pdl, a);
  if (e != cudaSuccess) return ugb_fail(m->dev, UGB_ERR_CUDA, "launch of row_update_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(m->dev, "row_update_kernel");
}

template int32_t ugb_hybrid_rows<float>(ugb_hybrid *, RowArgs<float> &, int, bool);
template int32_t ugb_hybrid_rows<__nv_bfloat16>(ugb_hybrid *, RowArgs<__nv_bfloat16> &, int, bool);

int32_t ugb_hybrid_keep(ugb_hybrid *m, const ugb_hybrid_work &w, int run, int t_block, int off, int t) {
  if (!m->keep_layers || !m->layer_out) return UGB_OK;     // rows (b, off + i) of [run][batch * t_block][wl]
  const size_t wl = m->wl;
  for (int b = 0; b < m->batch; ++b)
    UGB_CUDA(m->dev, cudaMemcpyAsync(m->layer_out + ((size_t)run * m->batch * t_block + (size_t)b * t_block + off) * wl,
                                     w.x + (size_t)b * t * wl, (size_t)t * wl * 4, cudaMemcpyDeviceToDevice, m->dev->stream));
  return UGB_OK;
}

namespace {

template <typename T>
int32_t launch_conv(ugb_device *dev, const T *h, const float *w, const T *tail_in, T *tail_out, T *out, int b, int t, int taps, int ld) {
  const dim3 grid((unsigned)((t + CONV_STRIP - 1) / CONV_STRIP), (unsigned)((ld / 8 + 127) / 128), (unsigned)b);
  auto *k = causal_conv_kernel<T, 0>;
  if (taps == 2) k = causal_conv_kernel<T, 2>;
  else if (taps == 3) k = causal_conv_kernel<T, 3>;
  else if (taps == 4) k = causal_conv_kernel<T, 4>;
  k<<<grid, 128, 0, dev->stream>>>(h, (size_t)ld, w, nullptr, tail_in, tail_out, out, t, taps, ld);
  return ugb_after_launch(dev, "causal_conv_kernel");
}

template <typename TI, typename T>
int32_t launch_scan(ugb_device *dev, const TI *pre, const float *bz, const float *bu, float *state, T *out, int b, int t, int ld) {
  // CTAs of a cluster: enough pieces of time to fill the SMs twice, no more than the block has
  const int columns = (ld + Scan<TI>::COLUMNS - 1) / Scan<TI>::COLUMNS;
  int c = 1;
  while (c < 8 && c * Scan<TI>::BLOCK < t && 2 * c * b * columns <= 2 * dev->sm_count) c *= 2;
  cudaError_t e = ugb_launch_cluster(min_gru_scan_kernel<TI, T>, dim3((unsigned)c, (unsigned)columns, (unsigned)b),
                                     dim3(SCAN_WARPS * 32), 0, dev->stream, false, c, pre, bz, bu, state, out, t, ld);
  if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of min_gru_scan_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(dev, "min_gru_scan_kernel");
}

// One pass over all layers for rows (b, i), i < t, positions *pos + off + i.  decode: t == 1 and the convolutions and
// recurrent states advance inside the row kernels.  Leaves the final norm's output in w.h.
template <typename T>
int32_t run_layers(ugb_hybrid *m, ugb_hybrid_work &w, const int *tok, int t_block, int off, int t, bool decode) {
  ugb_device *dev = m->dev;
  cudaStream_t st = dev->stream;
  const bool pdl = m->pdl != 0;
  // In a bf16 decode step every kernel lets its successor start only after its own wait, and at least two kernels lie
  // between one row kernel and the next: what earlier row kernels wrote is complete when a row kernel starts.
  const bool early = decode && pdl && !m->f32;
  const int B = m->batch, rows = B * t, wl = m->wl, taps = m->cfg.conv_taps;
  const size_t bank_stride = (size_t)w.rows * wl;
  int32_t rc;
  cudaError_t e;

  // what the products of the layer read: the row kernel's output, in a prompt after the convolution kernel
  auto input_of = [&](const float *conv, int layer, int which, const T **in) -> int32_t {
    *in = (const T *)w.h;
    if (decode || !conv) return UGB_OK;
    const T *ti = (const T *)(m->tails + m->runs[layer].tail[which]);
    T *to = (T *)(m->tails_next + m->runs[layer].tail[which]);
    *in = (const T *)w.hc;
    return m->on(UGB_HYBRID_K_CONV) ? launch_conv<T>(dev, (const T *)w.h, conv, ti, to, (T *)w.hc, B, t, taps, wl) : UGB_OK;
  };
  auto fuse_conv = [&](RowArgs<T> &a, const float *conv, int layer, int which) {
    if (!decode || !conv) return;
    a.conv = conv; a.taps = taps;
    a.tail = (T *)(m->tails + m->runs[layer].tail[which]);
  };

  {
    RowArgs<T> a;
    a.tok = tok; a.embed = (const T *)m->embed; a.vocab = m->cfg.vocab; a.t = t; a.tok_stride = t_block; a.tok_off = off;
    a.post_gain = m->embed_gain; a.x = w.x; a.add_x = 0;
    a.bank_out = m->cfg.depth_average ? w.bank : nullptr;
    a.gain = m->layers.empty() ? m->final_gain : m->layers[0].norm1;
    a.h = (T *)w.h;
    if (!m->layers.empty()) fuse_conv(a, m->layers[0].conv1, 0, 0);
    if ((rc = ugb_hybrid_rows<T>(m, a, rows, early))) return rc;
  }
  const int n_layers = (int)m->layers.size();
  for (int i = 0; i < n_layers; ++i) {
    const ugb_hybrid_weights &L = m->layers[i];
    const ugb_hybrid_run &R = m->runs[i];
    const T *in = nullptr;
    if ((rc = input_of(L.conv1, i, 0, &in))) return rc;
    Tiling out_t{0, 1};
    if (L.d.mixer == UGB_MIXER_MINGRU) {
      const Tiling ti = decode ? ugb_hybrid_tile(m, 3 * (size_t)L.ul, wl) : Tiling{0, 1};
      if (m->on(UGB_HYBRID_K_GRU_IN)) {
        Mat g{w.pre, in, L.w_in, (size_t)rows, 3 * (size_t)L.ul, (size_t)wl};
        g.splits = ti.splits; g.bn = ti.bn;
        g.f32_out = decode || m->f32;            // a block's projection is rounded to T, a step's partials are summed in f32
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
      if (m->on(UGB_HYBRID_K_GRU)) {
        if (decode) {
          e = ugb_launch(min_gru_step_kernel<T>, dim3(rows, (L.ul / 4 + 127) / 128), dim3(128), 0, st, pdl, w.pre, ti.splits,
                         (size_t)rows * 3 * L.ul, L.bz, L.bu, R.state, (T *)w.mid, L.ul);
          if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of min_gru_step_kernel failed: %s", cudaGetErrorString(e));
          if ((rc = ugb_after_launch(dev, "min_gru_step_kernel"))) return rc;
        } else if ((rc = launch_scan<T, T>(dev, (const T *)w.pre, L.bz, L.bu, R.state, (T *)w.mid, B, t, L.ul))) {
          return rc;
        }
      }
      if (decode) out_t = ugb_hybrid_tile(m, wl, L.ul);
      if (m->on(UGB_HYBRID_K_OUT)) {
        Mat g{w.pre, w.mid, L.w_out, (size_t)rows, (size_t)wl, (size_t)L.ul};
        g.splits = out_t.splits; g.bn = out_t.bn;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
    } else {
      const int H = L.d.heads, n_in = L.ql + L.cl + L.gl;
      const Tiling ti = decode ? ugb_hybrid_tile(m, n_in, wl) : Tiling{0, 1};
      if (m->on(UGB_HYBRID_K_LATENT_IN)) {
        Mat g{w.pre, in, L.w_in, (size_t)rows, (size_t)n_in, (size_t)wl};
        g.splits = ti.splits; g.bn = ti.bn;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
      if (m->on(UGB_HYBRID_K_LATENT_ROWS)) {
        const int threads = std::min(512, (n_in / 4 + 31) / 32 * 32), per = (n_in / 4 + threads - 1) / threads;
        auto *k = decode ? (per <= 1 ? latent_inputs_kernel<T, 1, 8> : per <= 2 ? latent_inputs_kernel<T, 2, 8> : latent_inputs_kernel<T, 16, 1>)
                         : (per <= 1 ? latent_inputs_kernel<T, 1, 1> : per <= 2 ? latent_inputs_kernel<T, 2, 1> : per <= 4 ? latent_inputs_kernel<T, 4, 1> : latent_inputs_kernel<T, 16, 1>);
        e = ugb_launch(k, dim3(rows), dim3(threads), 0, st, pdl, w.pre, ti.splits, (size_t)rows * n_in,
                       L.q_gain, L.c_gain, (T *)w.cq, (T *)R.cache, w.gate, m->pos, off, t, m->t_max, L.ql, L.cl, L.gl,
                       1.0f / (float)L.d.q_rank, 1.0f / (float)L.d.kv_rank, m->cfg.eps, dev->status_dev);
        if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of latent_inputs_kernel failed: %s", cudaGetErrorString(e));
        if ((rc = ugb_after_launch(dev, "latent_inputs_kernel"))) return rc;
      }
      const size_t qw = (size_t)H * L.dp, ow = (size_t)H * L.vp, lw = (size_t)H * L.cl;
      if (m->on(UGB_HYBRID_K_UQ)) {
        Mat g{w.q, w.cq, L.w_uq, (size_t)rows, qw, (size_t)L.ql};
        g.f32_out = false;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
      if (!decode && L.expand && t > m->absorb_max) {
        const size_t ctx = (size_t)m->host_pos + off + t;        // positions cached once this block is in
        if (m->on(UGB_HYBRID_K_ABSORB)) {
          Mat g{m->kx, R.cache, L.w_uk, ctx, qw, (size_t)L.cl};
          g.f32_out = false;
          g.batch = B; g.a_batch = (size_t)m->t_max * L.cl; g.c_batch = ctx * qw;
          if ((rc = ugb_hybrid_matmul(m, g))) return rc;
          g.out = m->vx; g.w = L.w_uv; g.n = ow; g.c_batch = ctx * ow;
          if ((rc = ugb_hybrid_matmul(m, g))) return rc;
        }
        if (m->on(UGB_HYBRID_K_ATTENTION)) {
          ugb_prefill_attention_args a;
          a.q = (const __nv_bfloat16 *)w.q; a.k = (const __nv_bfloat16 *)m->kx; a.v = (const __nv_bfloat16 *)m->vx;
          a.out = (__nv_bfloat16 *)w.o; a.batch = B; a.t = t; a.pos0 = m->host_pos + off; a.n_heads = a.n_kv = H;
          a.kv_rows = (int)ctx; a.token_major = 1; a.dq = L.dp; a.dv = L.vp; a.scale = L.d.scale; a.gate = w.gate; a.gate_ld = L.gl;
          if ((rc = ugb_prefill_attention_tc(dev, a))) return rc;
        }
      } else {
        if (m->on(UGB_HYBRID_K_ABSORB)) {
          Mat g{w.ql, w.q, L.w_uk, (size_t)rows, (size_t)L.cl, (size_t)L.dp};   // per head: q W_uk
          g.f32_out = false; g.nk = false;
          g.batch = H; g.a_ld = qw; g.a_batch = L.dp; g.w_batch = (size_t)L.dp * L.cl; g.c_ld = lw; g.c_batch = L.cl;
          if (rows <= 64) g.bn = 64;
          if ((rc = ugb_hybrid_matmul(m, g))) return rc;
        }
        if (m->on(UGB_HYBRID_K_ATTENTION)) {
          ugb_latent_attention_args a{};
          a.q = w.ql; a.cache = R.cache; a.out = w.ol; a.gate = w.gate; a.f32 = m->f32; a.rows = rows; a.t = t;
          a.pos_p = m->pos; a.pos_off = off; a.heads = H; a.ld = L.cl; a.t_max = m->t_max; a.gate_ld = L.gl; a.scale = L.d.scale;
          a.splits = decode ? m->att_splits() : 1;
          a.pdl = pdl; a.early = early;
          if ((rc = ugb_latent_attention(dev, a))) return rc;
        }
        if (m->on(UGB_HYBRID_K_ABSORB)) {
          Mat g{w.o, w.ol, L.w_uv, (size_t)rows, (size_t)L.vp, (size_t)L.cl};   // per head: W_uv o
          g.f32_out = false;
          g.batch = H; g.a_ld = lw; g.a_batch = L.cl; g.w_batch = (size_t)L.vp * L.cl; g.c_ld = ow; g.c_batch = L.vp;
          if (rows <= 64) g.bn = 64;
          if ((rc = ugb_hybrid_matmul(m, g))) return rc;
        }
      }
      if (decode) out_t = ugb_hybrid_tile(m, wl, ow);
      if (m->on(UGB_HYBRID_K_OUT)) {
        Mat g{w.pre, w.o, L.w_out, (size_t)rows, (size_t)wl, ow};
        g.splits = out_t.splits; g.bn = out_t.bn;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
    }
    // stream += norm(mixer output); with a feed-forward its input follows, else the layer ends here
    auto layer_end = [&](RowArgs<T> &a) {
      if (m->cfg.depth_average) {
        if (i + 1 < n_layers) a.bank_out = w.bank + (size_t)(i + 1) * bank_stride;
        a.bank = w.bank; a.bank_stride = bank_stride; a.dwa = L.dwa; a.n_avg = i + 1;
      }
      a.gain = i + 1 < n_layers ? m->layers[i + 1].norm1 : m->final_gain;
      if (i + 1 < n_layers) fuse_conv(a, m->layers[i + 1].conv1, i + 1, 0);
    };
    RowArgs<T> a;
    a.part = w.pre; a.n_part = out_t.splits; a.part_stride = (size_t)rows * wl;
    a.post_gain = L.norm1b; a.x = w.x; a.h = (T *)w.h;
    if (L.d.feed_forward == UGB_FF_NONE) layer_end(a);
    else { a.gain = L.norm2; fuse_conv(a, L.conv2, i, 1); }
    if ((rc = ugb_hybrid_rows<T>(m, a, rows, early))) return rc;
    if (L.d.feed_forward != UGB_FF_NONE) {
      if ((rc = input_of(L.conv2, i, 1, &in))) return rc;
      if (m->on(UGB_HYBRID_K_UP)) {
        Mat g{w.mid, in, L.w_up, (size_t)rows, (size_t)L.fl, (size_t)wl};
        g.f32_out = false; g.relu2 = true;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
      const Tiling td = decode ? ugb_hybrid_tile(m, wl, L.fl) : Tiling{0, 1};
      if (m->on(UGB_HYBRID_K_DOWN)) {
        Mat g{w.pre, w.mid, L.w_down, (size_t)rows, (size_t)wl, (size_t)L.fl};
        g.splits = td.splits; g.bn = td.bn;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
      RowArgs<T> f;
      f.part = w.pre; f.n_part = td.splits; f.part_stride = (size_t)rows * wl;
      f.post_gain = L.norm2b; f.x = w.x; f.h = (T *)w.h;
      layer_end(f);
      if ((rc = ugb_hybrid_rows<T>(m, f, rows, early))) return rc;
    }
    if (!decode && (rc = ugb_hybrid_keep(m, w, i, t_block, off, t))) return rc;
  }
  return UGB_OK;
}

int32_t run_layers_any(ugb_hybrid *m, ugb_hybrid_work &w, const int *tok, int t_block, int off, int t, bool decode) {
  if (m->parallel()) return ugb_parallel_run(m, w, tok, t_block, off, t, decode);
  return m->f32 ? run_layers<float>(m, w, tok, t_block, off, t, decode) : run_layers<__nv_bfloat16>(m, w, tok, t_block, off, t, decode);
}

int32_t alloc_work(ugb_hybrid *m, ugb_hybrid_work &w, int rows, bool decode) {
  if (m->parallel()) return ugb_parallel_work(m, w, rows, decode);
  const size_t R = rows, es = m->es(), wl = m->wl, splits = decode ? UGB_HYBRID_MAX_SPLITS : 1;
  size_t pre = wl, mid = 8, ql = 8, gl = 8, q = 8, lat = 8, o = 8;
  for (const ugb_hybrid_weights &L : m->layers) {
    pre = std::max({pre, (size_t)3 * L.ul, (size_t)(L.ql + L.cl + L.gl)});
    mid = std::max({mid, (size_t)L.ul, (size_t)L.fl});
    ql = std::max(ql, (size_t)L.ql); gl = std::max(gl, (size_t)L.gl);
    q = std::max(q, (size_t)L.d.heads * L.dp); o = std::max(o, (size_t)L.d.heads * L.vp);
    // rows that can run in the latent space: every one, unless the layer expands blocks beyond absorb_max positions
    const size_t lr = decode || !L.expand ? R : std::min(R, (size_t)m->batch * m->absorb_max);
    lat = std::max(lat, (lr * L.d.heads * L.cl + R - 1) / R);
  }
  lat = up8(lat);
  int32_t rc;
  const size_t banks = m->cfg.depth_average ? std::max<size_t>(1, m->layers.size()) : 0;
  if ((rc = dmalloc(m, &w.x, R * wl)) || (rc = dmalloc(m, &w.pre, splits * R * pre)) || (rc = dmalloc(m, &w.gate, R * gl)) ||
      (rc = dmalloc(m, &w.bank, banks * R * wl)) || (rc = ugb_hybrid_alloc(m, &w.h, R * wl * es, true)) ||
      (rc = ugb_hybrid_alloc(m, &w.hc, decode ? 16 : R * wl * es, false)) || (rc = ugb_hybrid_alloc(m, &w.mid, R * mid * es, false)) ||
      (rc = ugb_hybrid_alloc(m, &w.cq, R * ql * es, false)) || (rc = ugb_hybrid_alloc(m, &w.q, R * q * es, false)) ||
      (rc = ugb_hybrid_alloc(m, &w.ql, R * lat * es, false)) || (rc = ugb_hybrid_alloc(m, &w.ol, R * lat * es, false)) ||
      (rc = ugb_hybrid_alloc(m, &w.o, R * o * es, false)))
    return rc;
  w.rows = rows;
  return UGB_OK;
}

}  // namespace

int32_t ugb_hybrid::enqueue_step(const int *tok) {
  if (int32_t rc = run_layers_any(this, dec, tok, 1, 0, 1, true)) return rc;
  return enqueue_head(true);
}

int32_t ugb_hybrid::ensure_prefill_workspace() {
  if (pf_rows) return UGB_OK;
  const int chunk = std::max(1, std::min(pf_rows_max / batch, t_max));
  int32_t rc;
  if ((rc = alloc_work(this, pf, batch * chunk, false))) return rc;
  size_t k = 0, v = 0;
  for (const ugb_hybrid_weights &L : layers)
    if (L.expand && !parallel()) { k = std::max(k, (size_t)L.d.heads * L.dp); v = std::max(v, (size_t)L.d.heads * L.vp); }
  if ((rc = ugb_hybrid_alloc(this, &kx, (size_t)batch * t_max * k * es(), false)) || (rc = ugb_hybrid_alloc(this, &vx, (size_t)batch * t_max * v * es(), false)))
    return rc;
  pf_chunk = chunk;
  pf_rows = batch * chunk;
  return UGB_OK;
}

int32_t ugb_hybrid::enqueue_prefill_chunk(const int *tok, int t, int c0, int tc, bool all_logits) {
  if (keep_layers && c0 == 0) {
    const size_t need = runs.size() * (size_t)batch * t * wl;
    if (need > layer_cap) {
      float *p = nullptr;
      if (int32_t rc = dmalloc(this, &p, need)) return rc;    // freed with the model
      layer_out = p;
      layer_cap = need;
    }
    layer_rows = batch * t;
  }
  int32_t rc;
  if ((rc = run_layers_any(this, pf, tok, t, c0, tc, false))) return rc;
  if (tail_bytes && only == UGB_HYBRID_K_ALL)
    UGB_CUDA(dev, cudaMemcpyAsync(tails, tails_next, tail_bytes, cudaMemcpyDeviceToDevice, dev->stream));
  if (all_logits) {
    Mat g{pf_logits + (size_t)c0 * logits_ld, pf.h, head, (size_t)tc, (size_t)logits_ld, (size_t)wl};
    g.batch = batch; g.a_batch = (size_t)tc * wl; g.c_batch = (size_t)t * logits_ld;
    if ((rc = ugb_hybrid_matmul(this, g))) return rc;
    if (cfg.logit_softcap > 0.f)
      for (int b = 0; b < batch; ++b)
        if ((rc = ugb_parallel_softcap(this, pf_logits + ((size_t)b * t + c0) * logits_ld, (size_t)tc * logits_ld))) return rc;
  }
  return UGB_OK;
}

int32_t ugb_hybrid::enqueue_prefill_tail(int tc) {
  const size_t hb = (size_t)wl * es(), xb = (size_t)wl * 4;
  UGB_CUDA(dev, cudaMemcpy2DAsync(dec.h, hb, (const char *)pf.h + (size_t)(tc - 1) * hb, (size_t)tc * hb, hb, batch,
                                  cudaMemcpyDeviceToDevice, dev->stream));
  UGB_CUDA(dev, cudaMemcpy2DAsync(dec.x, xb, (const char *)pf.x + (size_t)(tc - 1) * xb, (size_t)tc * xb, xb, batch,
                                  cudaMemcpyDeviceToDevice, dev->stream));
  return UGB_OK;
}

int32_t ugb_hybrid::enqueue_head(bool) {
  if (!on(UGB_HYBRID_K_HEAD)) return UGB_OK;
  Mat g{logits, dec.h, head, (size_t)batch, (size_t)logits_ld, (size_t)wl};
  if (!f32 && batch <= 64) g.bn = logits_ld > 128 * dev->sm_count ? 256 : 128;
  int32_t rc;
  if ((rc = ugb_hybrid_matmul(this, g))) return rc;
  if (only != UGB_HYBRID_K_ALL) return UGB_OK;
  if (cfg.logit_softcap > 0.f && (rc = ugb_parallel_softcap(this, logits, (size_t)batch * logits_ld))) return rc;
  cudaError_t e = ugb_launch(ugb_decode::argmax_rows_kernel, dim3(batch), dim3(1024), 0, dev->stream, pdl != 0, logits, vl, logits_ld, next, pos);
  if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of argmax_rows_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(dev, "argmax_rows_kernel");
}

extern "C" {

int32_t ugb_hybrid_create(ugb_device *dev, const ugb_hybrid_config *cfg, const ugb_hybrid_layer *layers, int32_t batch,
                          int32_t t_max, ugb_hybrid **out) {
  if (!dev) return UGB_ERR_INVALID;
  UGB_REQUIRE(dev, cfg && out && (layers || cfg->layers == 0), UGB_ERR_INVALID, "ugb_hybrid_create: null argument");
  *out = nullptr;
  UGB_REQUIRE(dev, cfg->width > 0 && cfg->vocab > 0 && cfg->layers >= 0 && cfg->conv_taps >= 0, UGB_ERR_INVALID,
              "ugb_hybrid_create: non-positive dimension");
  UGB_REQUIRE(dev, cfg->width <= 8192 && cfg->conv_taps <= 64, UGB_ERR_UNSUPPORTED, "width %d (at most 8192), %d taps (at most 64)",
              cfg->width, cfg->conv_taps);
  UGB_REQUIRE(dev, cfg->dtype == UGB_BF16 || cfg->dtype == UGB_F32, UGB_ERR_DTYPE, "ugb_hybrid_create: dtype must be BF16 or F32");
  UGB_REQUIRE(dev, batch >= 1 && batch <= 128, UGB_ERR_UNSUPPORTED, "batch %d: 1..128 sequences", batch);
  UGB_REQUIRE(dev, t_max >= 1, UGB_ERR_INVALID, "t_max %d", t_max);
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  ugb_hybrid *m = new ugb_hybrid();
  m->dev = dev; m->cfg = *cfg; m->batch = batch; m->t_max = (t_max + 31) / 32 * 32;
  m->f32 = cfg->dtype == UGB_F32;
  m->wl = (int)up8(cfg->width);
  m->vl = cfg->vocab; m->logits_ld = (int)up8(cfg->vocab);
  const size_t es = m->es(), wl = m->wl;
  int32_t rc = UGB_OK;
#define TRY(e) do { if ((rc = (e)) != UGB_OK) { engine_free(m); delete m; return rc; } } while (0)
#define CHECK(cond, code, ...) do { if (!(cond)) { rc = ugb_fail(dev, code, __VA_ARGS__); engine_free(m); delete m; return rc; } } while (0)
  m->layers.resize(cfg->layers);
  CHECK(cfg->form == UGB_FORM_SANDWICH || cfg->form == UGB_FORM_PARALLEL, UGB_ERR_UNSUPPORTED, "form %d of the layers", cfg->form);
  for (int i = 0; i < cfg->layers; ++i) m->layers[i].d = layers[i];
  if (m->parallel()) TRY(ugb_parallel_model(m));
  else m->runs.resize(cfg->layers);
  for (int i = 0; i < cfg->layers && !m->parallel(); ++i) {
    ugb_hybrid_weights &L = m->layers[i];
    ugb_hybrid_run &R = m->runs[i];
    R.layer = i;
    const ugb_hybrid_layer &d = L.d;
    for (int k = 0; k < 2 && cfg->conv_taps > 1; ++k) {
      R.tail[k] = m->tail_bytes;
      m->tail_bytes += (size_t)batch * (cfg->conv_taps - 1) * wl * es;
    }
    TRY(dmalloc(m, &L.norm1, wl, true));
    TRY(dmalloc(m, &L.norm1b, wl, true));
    if (cfg->conv_taps) TRY(dmalloc(m, &L.conv1, cfg->conv_taps * wl, true));
    if (cfg->depth_average) TRY(dmalloc(m, &L.dwa, i + 2, true));
    CHECK(d.feed_forward == UGB_FF_NONE || d.feed_forward == UGB_FF_RELU2, UGB_ERR_UNSUPPORTED, "layer %d: feed-forward kind %d", i, d.feed_forward);
    if (d.feed_forward != UGB_FF_NONE) {
      CHECK(d.ff > 0, UGB_ERR_INVALID, "layer %d: ff %d", i, d.ff);
      L.fl = (int)up8(d.ff);
      TRY(dmalloc(m, &L.norm2, wl, true));
      TRY(dmalloc(m, &L.norm2b, wl, true));
      if (cfg->conv_taps) TRY(dmalloc(m, &L.conv2, cfg->conv_taps * wl, true));
      TRY(ugb_hybrid_alloc(m, &L.w_up, L.fl * wl * es, true));
      TRY(ugb_hybrid_alloc(m, &L.w_down, wl * L.fl * es, true));
    }
    if (d.mixer == UGB_MIXER_MINGRU) {
      CHECK(d.width > 0, UGB_ERR_INVALID, "layer %d: %d recurrent channels", i, d.width);
      L.d.heads = 0;
      L.ul = (int)up8(d.width);
      TRY(ugb_hybrid_alloc(m, &L.w_in, 3 * (size_t)L.ul * wl * es, true));
      TRY(ugb_hybrid_alloc(m, &L.w_out, wl * L.ul * es, true));
      TRY(dmalloc(m, &L.bz, L.ul, true));
      TRY(dmalloc(m, &L.bu, L.ul, true));
      R.state_len = (size_t)batch * L.ul;
      TRY(dmalloc(m, &R.state, R.state_len, true));
    } else {
      CHECK(d.mixer == UGB_MIXER_LATENT_ATTENTION, UGB_ERR_UNSUPPORTED, "layer %d: mixer kind %d", i, d.mixer);
      CHECK(d.heads > 0 && d.dim > 0 && d.vdim > 0 && d.q_rank > 0 && d.kv_rank > 0, UGB_ERR_INVALID, "layer %d: non-positive attention dimension", i);
      L.ql = (int)up8(d.q_rank);
      L.gl = (int)up8(d.heads);
      const int wide = m->f32 ? 0 : ugb_latent_row_width(d.kv_rank);
      L.cl = wide ? wide : (int)up8(d.kv_rank);
      const int dp = ugb_prefill_attention_width(d.dim), vp = ugb_prefill_attention_width(d.vdim);
      L.expand = !m->f32 && dp && vp && d.scale > 0.f;
      L.dp = L.expand ? dp : (int)up8(d.dim);
      L.vp = L.expand ? vp : (int)up8(d.vdim);
      CHECK(L.ql + L.cl + L.gl <= 16 * 4 * 512, UGB_ERR_UNSUPPORTED, "layer %d: latents of %d + %d values", i, d.q_rank, d.kv_rank);
      TRY(ugb_hybrid_alloc(m, &L.w_in, (size_t)(L.ql + L.cl + L.gl) * wl * es, true));
      TRY(ugb_hybrid_alloc(m, &L.w_uq, (size_t)d.heads * L.dp * L.ql * es, true));
      TRY(ugb_hybrid_alloc(m, &L.w_uk, (size_t)d.heads * L.dp * L.cl * es, true));
      TRY(ugb_hybrid_alloc(m, &L.w_uv, (size_t)d.heads * L.vp * L.cl * es, true));
      TRY(ugb_hybrid_alloc(m, &L.w_out, wl * d.heads * L.vp * es, true));
      TRY(dmalloc(m, &L.q_gain, L.ql, true));
      TRY(dmalloc(m, &L.c_gain, L.cl, true));
      TRY(ugb_hybrid_alloc(m, &R.cache, (size_t)batch * m->t_max * L.cl * es, true));
    }
  }
  TRY(ugb_hybrid_alloc(m, &m->embed, (size_t)cfg->vocab * wl * es, true));
  TRY(ugb_hybrid_alloc(m, &m->head, (size_t)m->logits_ld * wl * es, true));
  TRY(dmalloc(m, &m->embed_gain, wl, true));
  TRY(dmalloc(m, &m->final_gain, wl, true));
  TRY(dmalloc(m, &m->tails, m->tail_bytes, true));
  TRY(dmalloc(m, &m->tails_next, m->tail_bytes, true));
  TRY(dmalloc(m, &m->logits, (size_t)batch * m->logits_ld, true));
  TRY(dmalloc(m, &m->next, batch, true));
  TRY(dmalloc(m, &m->pos, 1, true));
  TRY(alloc_work(m, m->dec, batch, true));
  TRY(ugb_latent_attention_prepare(dev));
  TRY(ugb_grouped_attention_prepare(dev));
#undef TRY
#undef CHECK
  *out = m;
  return UGB_OK;
}

int32_t ugb_hybrid_destroy(ugb_hybrid *m) {
  if (!m) return UGB_ERR_INVALID;
  engine_free(m);
  delete m;
  return UGB_OK;
}

int32_t ugb_hybrid_load_weight(ugb_hybrid *m, const char *name, const ugb_slice *w) {
  if (!m) return UGB_ERR_INVALID;
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, name && w, UGB_ERR_INVALID, "ugb_hybrid_load_weight: null argument");
  UGB_REQUIRE(dev, w->dev == dev, UGB_ERR_INVALID, "%s: slice belongs to another device", name);
  const ugb_hybrid_config &c = m->cfg;
  const size_t W = c.width, wl = m->wl, es = m->es();
  const int32_t dt = m->f32 ? UGB_F32 : UGB_BF16;
  const std::string s(name);
  auto at = [&](void *base, size_t elems) { return (void *)((char *)base + elems * es); };
  // rows x cols matrix into rows of `pitch` elements
  auto put = [&](void *dst, size_t rows, size_t cols, size_t pitch) {
    return engine_put_matrix(m, w, dst, dt, rows, cols, 0, rows, 0, cols, pitch, name);
  };
  auto put_heads = [&](void *dst, size_t heads, size_t d, size_t dp, size_t cols, size_t pitch) -> int32_t {   // d rows per head
    if (d == dp) return put(dst, heads * d, cols, pitch);
    for (size_t h = 0; h < heads; ++h)
      if (int32_t rc = engine_put_matrix(m, w, at(dst, h * dp * pitch), dt, heads * d, cols, h * d, d, 0, cols, pitch, name)) return rc;
    return UGB_OK;
  };
  auto vec = [&](float *dst, size_t n) { return engine_put_matrix(m, w, dst, UGB_F32, 1, n, 0, 1, 0, n, n, name); };
  auto conv = [&](float *dst) {
    UGB_REQUIRE(dev, dst != nullptr, UGB_ERR_INVALID, "%s: the model has no input convolution there", name);
    return ugb_hybrid_f32(m, w, W * c.conv_taps, name, [&](const float *src) {
      taps_kernel<<<((int)W * c.conv_taps + 255) / 256, 256, 0, dev->stream>>>(src, dst, (int)W, c.conv_taps, (int)wl);
      return ugb_after_launch(dev, "taps_kernel");
    });
  };
  auto gain = [&](float *dst) {
    UGB_REQUIRE(dev, dst != nullptr, UGB_ERR_INVALID, "%s: the layer has no such norm", name);
    return ugb_hybrid_gain(m, w, dst, (int)W, c.gain_offset, name);
  };
  m->loaded++;
  if (s == "embed") return put(m->embed, c.vocab, W, wl);
  if (s == "head") return put(m->head, c.vocab, W, wl);
  if (s == "embed.norm" && !m->parallel()) return gain(m->embed_gain);
  if (s == "final.norm") return gain(m->final_gain);
  if (m->parallel()) {
    bool known = true;
    const int32_t rc = ugb_parallel_load(m, name, w, &known);
    if (known) return rc;
    m->loaded--;
    return ugb_fail(dev, UGB_ERR_INVALID, "unknown weight name %s", name);
  }
  const size_t dot = s.find('.');
  if (s.size() > 1 && s[0] == 'l' && dot != std::string::npos && dot > 1 &&
      s.find_first_not_of("0123456789", 1) == dot && dot < 10) {
    const int i = atoi(s.c_str() + 1);
    UGB_REQUIRE(dev, i < c.layers, UGB_ERR_INVALID, "%s: layer index out of range", name);
    ugb_hybrid_weights &L = m->layers[i];
    const ugb_hybrid_layer &d = L.d;
    const std::string k = s.substr(dot + 1);
    if (k == "norm1") return gain(L.norm1);
    if (k == "norm1b") return gain(L.norm1b);
    if (k == "norm2") return gain(L.norm2);
    if (k == "norm2b") return gain(L.norm2b);
    if (k == "canon1") return conv(L.conv1);
    if (k == "canon2") return conv(L.conv2);
    if (k == "dwa" && c.depth_average) return vec(L.dwa, (size_t)i + 2);
    if (d.feed_forward != UGB_FF_NONE) {
      if (k == "mlp.up") return put(L.w_up, d.ff, W, wl);
      if (k == "mlp.down") return put(L.w_down, W, d.ff, L.fl);
    }
    if (d.mixer == UGB_MIXER_MINGRU) {
      const size_t n = d.width, ul = L.ul;
      if (k == "mix.z") return put(L.w_in, n, W, wl);
      if (k == "mix.x") return put(at(L.w_in, ul * wl), n, W, wl);
      if (k == "mix.g") return put(at(L.w_in, 2 * ul * wl), n, W, wl);
      if (k == "mix.z.b") return vec(L.bz, n);
      if (k == "mix.x.b") return vec(L.bu, n);
      if (k == "mix.o") return put(L.w_out, W, n, ul);
    } else {
      const size_t H = d.heads;
      if (k == "mix.dq") return put(L.w_in, d.q_rank, W, wl);
      if (k == "mix.dkv") return put(at(L.w_in, (size_t)L.ql * wl), d.kv_rank, W, wl);
      if (k == "mix.g") return put(at(L.w_in, (size_t)(L.ql + L.cl) * wl), H, W, wl);
      if (k == "mix.dq.norm") return vec(L.q_gain, d.q_rank);
      if (k == "mix.dkv.norm") return vec(L.c_gain, d.kv_rank);
      if (k == "mix.uq") return put_heads(L.w_uq, H, d.dim, L.dp, d.q_rank, L.ql);
      if (k == "mix.uk") return put_heads(L.w_uk, H, d.dim, L.dp, d.kv_rank, L.cl);
      if (k == "mix.uv") return put_heads(L.w_uv, H, d.vdim, L.vp, d.kv_rank, L.cl);
      if (k == "mix.o") {                                  // columns head by head
        for (size_t h = 0; h < H; ++h)
          if (int32_t rc = engine_put_matrix(m, w, at(L.w_out, h * L.vp), dt, W, H * d.vdim, 0, W, h * d.vdim, d.vdim, H * L.vp, name)) return rc;
        return UGB_OK;
      }
    }
  }
  m->loaded--;
  return ugb_fail(dev, UGB_ERR_INVALID, "unknown weight name %s", name);
}

int32_t ugb_hybrid_set_option(ugb_hybrid *m, const char *key, int32_t value) {
  if (!m || !key) return UGB_ERR_INVALID;
  ugb_device *dev = m->dev;
  const std::string k(key);
  if (k == "pdl") m->pdl = value != 0;
  else if (k == "att_splits") {
    UGB_REQUIRE(dev, value >= 0 && value <= UGB_LATENT_MAX_SPLITS, UGB_ERR_INVALID, "option att_splits: %d outside 0..%d", value, UGB_LATENT_MAX_SPLITS);
    m->att_splits_opt = value;
  } else if (k == "keep_layers") m->keep_layers = value != 0;
  else if (k == "absorb_max" || k == "prefill_rows") {
    UGB_REQUIRE(dev, m->pf_rows == 0, UGB_ERR_INVALID, "option %s must be set before the first prompt", key);
    if (k == "absorb_max") {
      UGB_REQUIRE(dev, value >= 0 && value <= 65536, UGB_ERR_INVALID, "option absorb_max: %d outside 0..65536", value);
      m->absorb_max = value;
    } else {
      UGB_REQUIRE(dev, value >= 16 && value <= 65535, UGB_ERR_INVALID, "option prefill_rows: %d outside 16..65535", value);
      m->pf_rows_max = value;
    }
  } else return ugb_fail(dev, UGB_ERR_INVALID, "unknown option %s", key);
  engine_drop_graph(m);
  return UGB_OK;
}

int32_t ugb_hybrid_reset(ugb_hybrid *m, int32_t pos) {
  if (!m) return UGB_ERR_INVALID;
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, pos == 0 || pos == m->host_pos, UGB_ERR_UNSUPPORTED,
              "a recurrent model cannot go from position %d to %d: it restarts at 0", m->host_pos, pos);
  if (pos == 0) {
    UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
    if (m->tail_bytes) UGB_CUDA(dev, cudaMemsetAsync(m->tails, 0, m->tail_bytes, dev->stream));
    for (const ugb_hybrid_run &R : m->runs)
      if (R.state) UGB_CUDA(dev, cudaMemsetAsync(R.state, 0, R.state_len * 4, dev->stream));
  }
  return engine_reset(m, pos);
}

int32_t ugb_hybrid_position(const ugb_hybrid *m) { return m ? m->host_pos : -1; }

int32_t ugb_hybrid_decode(ugb_hybrid *m, const ugb_slice *tokens, int32_t n_steps) {
  return m ? engine_decode(m, tokens, n_steps) : UGB_ERR_INVALID;
}

int32_t ugb_hybrid_prefill(ugb_hybrid *m, const ugb_slice *tokens, int32_t t, int32_t all_logits) {
  return m ? engine_prefill(m, tokens, t, all_logits) : UGB_ERR_INVALID;
}

int32_t ugb_hybrid_read(ugb_hybrid *m, int32_t what, void *host_dst, size_t len) {
  if (!m) return UGB_ERR_INVALID;
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, host_dst != nullptr, UGB_ERR_INVALID, "ugb_hybrid_read: null destination");
  switch (what) {
    case UGB_HYBRID_LOGITS: return engine_read_rows(m, m->logits, m->batch, m->vl, m->logits_ld, host_dst, len);
    case UGB_HYBRID_NEXT_TOKENS: return engine_read_rows(m, m->next, m->batch, 1, 1, host_dst, len);
    case UGB_HYBRID_HIDDEN: return engine_read_rows(m, m->dec.x, m->batch, m->cfg.width, m->wl, host_dst, len);
    case UGB_HYBRID_PREFILL_LOGITS:
      UGB_REQUIRE(dev, m->pf_logits && m->pf_logits_t > 0, UGB_ERR_INVALID, "no all-position logits: run ugb_hybrid_prefill with all_logits first");
      return engine_read_rows(m, m->pf_logits, (size_t)m->batch * m->pf_logits_t, m->vl, m->logits_ld, host_dst, len);
    case UGB_HYBRID_LAYERS:
      UGB_REQUIRE(dev, m->layer_out, UGB_ERR_INVALID, "no layer outputs: set option keep_layers and run ugb_hybrid_prefill first");
      return engine_read_rows(m, m->layer_out, m->runs.size() * (size_t)m->layer_rows, m->cfg.width, m->wl, host_dst, len);
    default: return ugb_fail(dev, UGB_ERR_INVALID, "ugb_hybrid_read: unknown selector %d", what);
  }
}

uint64_t ugb_hybrid_state_bytes(const ugb_hybrid *m, int32_t positions) {
  if (!m) return 0;
  uint64_t n = m->tail_bytes / m->batch;
  for (const ugb_hybrid_run &R : m->runs) {
    const ugb_hybrid_weights &L = m->layers[R.layer];
    if (R.state) n += R.state_len / m->batch * 4;
    if (R.vcache) n += (uint64_t)positions * L.d.kv_heads * (L.dp + L.vp) * m->es();
    else if (R.cache) n += (uint64_t)positions * L.cl * m->es();
  }
  return n;
}

int32_t ugb_hybrid_time_kernel(ugb_hybrid *m, int32_t which, int32_t t, int32_t iters, float *ms_per_pass) {
  if (!m) return UGB_ERR_INVALID;
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, ms_per_pass && iters >= 1 && t >= 1 && which >= 0 && which <= UGB_HYBRID_K_ALL, UGB_ERR_INVALID, "ugb_hybrid_time_kernel: bad argument");
  UGB_REQUIRE(dev, m->warmed, UGB_ERR_INVALID, "ugb_hybrid_time_kernel: run one decode step first");
  int32_t rc;
  const int saved = m->host_pos;
  if (t > 1) {
    if ((rc = m->ensure_prefill_workspace())) return rc;
    UGB_REQUIRE(dev, t <= m->pf_chunk && saved + t <= m->t_max, UGB_ERR_SHAPE, "ugb_hybrid_time_kernel: a block of %d positions does not fit", t);
  } else {
    UGB_REQUIRE(dev, saved < m->t_max, UGB_ERR_SHAPE, "ugb_hybrid_time_kernel: the cache is full");
  }
  void *tok = nullptr;
  UGB_CUDA(dev, cudaMalloc(&tok, (size_t)m->batch * t * 4));
  UGB_CUDA(dev, cudaMemsetAsync(tok, 0, (size_t)m->batch * t * 4, dev->stream));
  cudaGraph_t g = nullptr;
  cudaGraphExec_t ge = nullptr;
  cudaError_t e = cudaStreamBeginCapture(dev->stream, cudaStreamCaptureModeThreadLocal);
  m->only = which;
  if (t > 1) rc = run_layers_any(m, m->pf, (const int *)tok, t, 0, t, false);
  else rc = run_layers_any(m, m->dec, (const int *)tok, 1, 0, 1, true);
  if (!rc && which == UGB_HYBRID_K_HEAD) rc = m->enqueue_head(true);
  m->only = UGB_HYBRID_K_ALL;
  const cudaError_t ee = cudaStreamEndCapture(dev->stream, &g);
  if (e == cudaSuccess) e = ee;
  if (!rc && e == cudaSuccess) e = cudaGraphInstantiate(&ge, g, 0);
  if (g) cudaGraphDestroy(g);
  float ms = 0.f;
  if (!rc && e == cudaSuccess) {
    for (int it = -2; it < iters && e == cudaSuccess; ++it) {     // two untimed passes
      if (it == 0) e = cudaEventRecord(dev->ev_begin, dev->stream);
      if (e == cudaSuccess) e = cudaGraphLaunch(ge, dev->stream);
    }
    if (e == cudaSuccess) e = cudaEventRecord(dev->ev_end, dev->stream);
    if (e == cudaSuccess) e = cudaEventSynchronize(dev->ev_end);
    if (e == cudaSuccess) e = cudaEventElapsedTime(&ms, dev->ev_begin, dev->ev_end);
  }
  cudaStreamSynchronize(dev->stream);
  if (ge) cudaGraphExecDestroy(ge);
  cudaFree(tok);
  if (rc) return rc;
  if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "ugb_hybrid_time_kernel: %s", cudaGetErrorString(e));
  *ms_per_pass = ms / (float)iters;
  return UGB_OK;
}

// ------------------------------------------------------- mechanisms alone ----
static int32_t act_dtype(ugb_device *dev, const ugb_slice *a, const ugb_slice *b, const char *what) {
  UGB_REQUIRE(dev, a && b, UGB_ERR_INVALID, "%s: null slice", what);
  UGB_REQUIRE(dev, a->dtype == b->dtype && (a->dtype == UGB_BF16 || a->dtype == UGB_F32), UGB_ERR_DTYPE,
              "%s: activations must be BF16 or F32 alike", what);
  return UGB_OK;
}

int32_t ugb_causal_conv(ugb_device *dev, const ugb_slice *h, const ugb_slice *w, ugb_slice *tail, ugb_slice *out, size_t b,
                        size_t t, size_t width, size_t taps) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, h, out, "causal_conv")) return rc;
  UGB_REQUIRE(dev, width % 8 == 0 && taps >= 1 && taps <= 64 && b <= 65535 && b * t * width < (1ull << 31), UGB_ERR_SHAPE, "causal_conv: unsupported shape");
  UGB_SLICE(dev, h, h->dtype, b * t * width);
  UGB_SLICE(dev, out, h->dtype, b * t * width);
  UGB_SLICE(dev, tail, h->dtype, b * (taps - 1) * width);
  UGB_SLICE(dev, w, UGB_F32, taps * width);
  UGB_REQUIRE(dev, out->ptr != h->ptr, UGB_ERR_INVALID, "causal_conv: in place");
  if (b == 0 || t == 0 || width == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  const size_t bytes = b * (taps - 1) * width * ugb_dtype_size(h->dtype);
  void *tmp = nullptr;
  UGB_CUDA(dev, ugb_malloc_async(dev, &tmp, bytes + 16));
  int32_t rc = h->dtype == UGB_F32
      ? launch_conv<float>(dev, (const float *)h->ptr, (const float *)w->ptr, (const float *)tail->ptr, (float *)tmp, (float *)out->ptr, (int)b, (int)t, (int)taps, (int)width)
      : launch_conv<__nv_bfloat16>(dev, (const __nv_bfloat16 *)h->ptr, (const float *)w->ptr, (const __nv_bfloat16 *)tail->ptr, (__nv_bfloat16 *)tmp, (__nv_bfloat16 *)out->ptr, (int)b, (int)t, (int)taps, (int)width);
  if (!rc && bytes) UGB_CUDA(dev, cudaMemcpyAsync(tail->ptr, tmp, bytes, cudaMemcpyDeviceToDevice, dev->stream));
  cudaFreeAsync(tmp, dev->stream);
  return rc;
}

int32_t ugb_min_gru(ugb_device *dev, const ugb_slice *pre, const ugb_slice *bias_z, const ugb_slice *bias_x, ugb_slice *state,
                    ugb_slice *out, size_t b, size_t t, size_t width) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, out, out, "min_gru")) return rc;
  UGB_REQUIRE(dev, width % 8 == 0 && b <= 65535 && 3 * b * t * width < (1ull << 31), UGB_ERR_SHAPE, "min_gru: unsupported shape");
  if (int32_t rc = act_dtype(dev, pre, pre, "min_gru")) return rc;
  const bool half = pre->dtype == UGB_BF16;
  UGB_REQUIRE(dev, !half || (t > 1 && out->dtype == UGB_BF16), UGB_ERR_DTYPE, "min_gru: bf16 pre-activations want a block and a bf16 result");
  UGB_SLICE(dev, pre, pre->dtype, 3 * b * t * width);
  UGB_SLICE(dev, bias_z, UGB_F32, width);
  UGB_SLICE(dev, bias_x, UGB_F32, width);
  UGB_SLICE(dev, state, UGB_F32, b * width);
  UGB_SLICE(dev, out, out->dtype, b * t * width);
  if (b == 0 || t == 0 || width == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  const float *p = (const float *)pre->ptr, *bz = (const float *)bias_z->ptr, *bx = (const float *)bias_x->ptr;
  float *s = (float *)state->ptr;
  const dim3 grid((unsigned)b, (unsigned)((width / 4 + 127) / 128));
  if (out->dtype == UGB_F32) {
    if (t > 1) return launch_scan<float, float>(dev, p, bz, bx, s, (float *)out->ptr, (int)b, (int)t, (int)width);
    min_gru_step_kernel<float><<<grid, 128, 0, dev->stream>>>(p, 1, 0, bz, bx, s, (float *)out->ptr, (int)width);
  } else {
    if (half) return launch_scan<__nv_bfloat16, __nv_bfloat16>(dev, (const __nv_bfloat16 *)p, bz, bx, s, (__nv_bfloat16 *)out->ptr, (int)b, (int)t, (int)width);
    if (t > 1) return launch_scan<float, __nv_bfloat16>(dev, p, bz, bx, s, (__nv_bfloat16 *)out->ptr, (int)b, (int)t, (int)width);
    min_gru_step_kernel<__nv_bfloat16><<<grid, 128, 0, dev->stream>>>(p, 1, 0, bz, bx, s, (__nv_bfloat16 *)out->ptr, (int)width);
  }
  return ugb_after_launch(dev, "min_gru_step_kernel");
}

int32_t ugb_latent_attend(ugb_device *dev, const ugb_slice *q, const ugb_slice *cache, const ugb_slice *gate, const ugb_slice *pos,
                          ugb_slice *out, size_t b, size_t t, size_t heads, size_t rank, size_t t_max, float scale, int32_t n_slices) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, q, cache, "latent_attend")) return rc;
  UGB_REQUIRE(dev, rank % 8 == 0 && rank > 0 && heads > 0 && b * t <= 65535 && heads <= 65535 && t_max <= (1u << 30), UGB_ERR_SHAPE, "latent_attend: unsupported shape");
  UGB_REQUIRE(dev, n_slices >= 1 && n_slices <= UGB_LATENT_MAX_SPLITS, UGB_ERR_INVALID, "latent_attend: %d slices", n_slices);
  UGB_SLICE(dev, q, q->dtype, b * t * heads * rank);
  UGB_SLICE(dev, out, q->dtype, b * t * heads * rank);
  UGB_SLICE(dev, cache, q->dtype, b * t_max * rank);
  UGB_SLICE(dev, pos, UGB_I32, 1);
  if (gate) UGB_SLICE(dev, gate, UGB_F32, b * t * heads);
  if (b == 0 || t == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  int32_t rc = ugb_latent_attention_prepare(dev);
  if (rc) return rc;
  ugb_latent_attention_args a{};
  a.q = q->ptr; a.cache = cache->ptr; a.out = out->ptr; a.gate = gate ? (const float *)gate->ptr : nullptr; a.f32 = q->dtype == UGB_F32;
  a.rows = (int)(b * t); a.t = (int)t; a.pos_p = (const int *)pos->ptr; a.heads = (int)heads; a.ld = (int)rank; a.t_max = (int)t_max;
  a.gate_ld = (int)heads; a.scale = scale; a.splits = n_slices;
  return ugb_latent_attention(dev, a);
}

int32_t ugb_causal_attention_wide(ugb_device *dev, const ugb_slice *q, const ugb_slice *k, const ugb_slice *v, const ugb_slice *gate,
                                  ugb_slice *out, size_t b, size_t t, size_t pos0, size_t heads, size_t dq, size_t dv, float scale) {
  if (!dev) return UGB_ERR_INVALID;
  UGB_REQUIRE(dev, heads > 0 && b <= 65535 && heads <= 65535 && pos0 + t <= (1u << 30) && ((t + 127) / 128) * heads * b <= (size_t)INT32_MAX,
              UGB_ERR_SHAPE, "causal_attention_wide: a dimension exceeds the kernel's index range");
  UGB_REQUIRE(dev, scale > 0.f, UGB_ERR_UNSUPPORTED, "causal_attention_wide: the scale must be positive");
  UGB_SLICE(dev, q, UGB_BF16, b * t * heads * dq);
  UGB_SLICE(dev, k, UGB_BF16, b * (pos0 + t) * heads * dq);
  UGB_SLICE(dev, v, UGB_BF16, b * (pos0 + t) * heads * dv);
  UGB_SLICE(dev, out, UGB_BF16, b * t * heads * dv);
  if (gate) UGB_SLICE(dev, gate, UGB_F32, b * t * heads);
  if (b == 0 || t == 0) return UGB_OK;
  UGB_REQUIRE(dev, (((uintptr_t)q->ptr | (uintptr_t)k->ptr | (uintptr_t)v->ptr | (uintptr_t)out->ptr) & 15) == 0,
              UGB_ERR_UNSUPPORTED, "causal_attention_wide: buffers must be 16-byte aligned");
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  ugb_prefill_attention_args a;
  a.q = (const __nv_bfloat16 *)q->ptr; a.k = (const __nv_bfloat16 *)k->ptr; a.v = (const __nv_bfloat16 *)v->ptr;
  a.out = (__nv_bfloat16 *)out->ptr; a.batch = (int)b; a.t = (int)t; a.pos0 = (int)pos0; a.n_heads = a.n_kv = (int)heads;
  a.kv_rows = (int)(pos0 + t); a.token_major = 1; a.dq = (int)dq; a.dv = (int)dv; a.scale = scale;
  a.gate = gate ? (const float *)gate->ptr : nullptr; a.gate_ld = (int)heads;
  return ugb_prefill_attention_tc(dev, a);
}

int32_t ugb_residual_update(ugb_device *dev, ugb_slice *x, const ugb_slice *y, const ugb_slice *post_gain, ugb_slice *bank,
                            const ugb_slice *dwa, size_t n, const ugb_slice *gain, ugb_slice *h, size_t rows, size_t width, float eps) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, h, h, "residual_update")) return rc;
  UGB_REQUIRE(dev, width % 8 == 0 && width > 0 && width <= 8192 && rows <= (1u << 30) && n <= 65535, UGB_ERR_SHAPE, "residual_update: unsupported shape");
  UGB_REQUIRE(dev, (bank == nullptr) == (dwa == nullptr), UGB_ERR_INVALID, "residual_update: bank and dwa go together");
  UGB_SLICE(dev, x, UGB_F32, rows * width);
  UGB_SLICE(dev, y, UGB_F32, rows * width);
  UGB_SLICE(dev, post_gain, UGB_F32, width);
  UGB_SLICE(dev, gain, UGB_F32, width);
  UGB_SLICE(dev, h, h->dtype, rows * width);
  if (bank) { UGB_SLICE(dev, bank, UGB_F32, (n + 1) * rows * width); UGB_SLICE(dev, dwa, UGB_F32, n + 1); }
  if (rows == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  ugb_hybrid m;                                            // the launcher reads device, width and eps only
  m.dev = dev; m.wl = (int)width; m.cfg.width = (int)width; m.cfg.eps = eps; m.pdl = 0;
  auto fill = [&](auto &a) {
    a.part = (const float *)y->ptr; a.n_part = 1; a.post_gain = (const float *)post_gain->ptr; a.x = (float *)x->ptr;
    a.gain = (const float *)gain->ptr;
    if (bank) {
      a.bank = (const float *)bank->ptr; a.bank_out = (float *)bank->ptr + n * rows * width; a.bank_stride = rows * width;
      a.dwa = (const float *)dwa->ptr; a.n_avg = (int)n;
    }
  };
  if (h->dtype == UGB_F32) {
    RowArgs<float> a;
    fill(a);
    a.h = (float *)h->ptr;
    return ugb_hybrid_rows<float>(&m, a, (int)rows, false);
  }
  RowArgs<__nv_bfloat16> a;
  fill(a);
  a.h = (__nv_bfloat16 *)h->ptr;
  return ugb_hybrid_rows<__nv_bfloat16>(&m, a, (int)rows, false);
}

}  // extern "C"
