// Layers in the parallel form: attention and selective scan side by side and the feed-forward read one norm, their sum joins
// the residual stream, and an input of the token follows (see ugb200.h).  Life cycle and options are hybrid_engine.cu's.
//
// Launches of a layer (T = activation type; h = the norm's output, left by the row kernel before):
//   [loop]  GEMM stream | embedding output -> f32;  row_update  stream = product + step;  norm -> h
//   GEMM h -> q | k | v | x | z [| router]              f32 partials in a step, T in a block
//   mixer_inputs    rotation and norm of q and k, cache append          [step: + convolution, choice of experts]
//   causal_conv     blocks only: convolution, bias, silu -> u
//   GEMM u -> low | B | C;  blocks: GEMM low -> dt
//   selective_scan  scan, gate -> cat                                   [step: + step-size projection]
//   attention       -> cat                              tcgen05 for blocks, grouped_attention for steps
//   GEMM h -> (gate, up) pairs with silu(gate) up in the epilogue -> cat       dense or shared feed-forward
//   [experts]  blocks: GEMM router, route;  expert_rows (rows by expert, times their weight);  grouped GEMMs up and down
//   GEMM cat -> f32                                     output projections of mixer and feed-forward as one product
//   row_update      stream += product + experts' rows;  copy -> T (token input or loop) or norm -> h
//   [token input]  GEMM gate;  token_gate;  GEMM proj -> f32;  row_update  stream += norm(product);  copy or norm
// The factors of attention and scan are applied where their f32 results are rounded to T.  Products with a f32 result are
// split over k in a step; the consumer sums the partials.
//
// Padding: every width is rounded up to 8, head widths to 64 or 128 where the tensor-core attention kernels take them, states
// of a channel to what selective_scan.cu takes; padded weight rows and columns, gains and biases are zero.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <string>

#include "attention_tc.cuh"
#include "gemm_tcgen05.cuh"
#include "grouped_attention.cuh"
#include "hybrid_engine.cuh"
#include "parallel_kernels.cuh"
#include "selective_scan.cuh"

using namespace ugb_hybrid_k;

using Mat = ugb_hybrid_mat;
using Tiling = ugb_hybrid_tiling;
using Weights = ugb_hybrid_weights;
static size_t up8(size_t n) { return ugb_up8(n); }

namespace {

// Narrow products of a block have few tiles and a long k loop that one CTA walks in order: k splits that fill the SMs with
// 128 x 256 tiles, four k blocks or more each.  Their f32 partials take at most narrow_rows() rows.
int narrow_splits(const ugb_hybrid *m, int rows, size_t n, size_t k) {
  if (m->f32) return 1;
  const int tiles = (rows + 127) / 128 * (int)((n + 255) / 256), kb = (int)((k + 63) / 64);
  const int s = std::min({UGB_HYBRID_MAX_SPLITS, m->dev->sm_count / tiles, kb / 4});
  return s > 1 ? ugb_tc_gemm_effective_splits(k, s) : 1;
}
size_t narrow_rows(const ugb_hybrid *m, size_t rows) {
  return m->f32 ? rows : std::max(rows, std::min(rows * UGB_HYBRID_MAX_SPLITS, (size_t)m->dev->sm_count * 128));
}

// tiles of `tile` rows that hold `rows` rows grouped into `groups`
int group_tiles(size_t rows, int groups, int tile) { return (int)(rows / tile) + groups; }

template <typename T>
int32_t launch_gated_conv(ugb_device *dev, const T *h, size_t h_ld, const float *w, const float *bias, const T *tail_in, T *tail_out, T *out,
                          int b, int t, int taps, int ld) {
  const dim3 grid((unsigned)((t + CONV_STRIP - 1) / CONV_STRIP), (unsigned)((ld / 8 + 127) / 128), (unsigned)b);
  auto *k = causal_conv_kernel<T, 0, true>;
  if (taps == 2) k = causal_conv_kernel<T, 2, true>;
  else if (taps == 3) k = causal_conv_kernel<T, 3, true>;
  else if (taps == 4) k = causal_conv_kernel<T, 4, true>;
  k<<<grid, 128, 0, dev->stream>>>(h, h_ld, w, bias, tail_in, tail_out, out, t, taps, ld);
  return ugb_after_launch(dev, "causal_conv_kernel");
}

template <typename TI, typename T, bool STEP>
int32_t launch_mixer_inputs(ugb_device *dev, const MixerIn<TI, T> &a, int rows, bool pdl) {
  const MixerUnits n = mixer_units<STEP>(a.heads + a.kv_heads, a.dp, a.kv_heads * a.vp, a.ci, a.experts);
  const long long warps = (long long)rows * n.all;
  UGB_REQUIRE(dev, warps < (1ll << 31), UGB_ERR_UNSUPPORTED, "mixer inputs: %d rows of %d units", rows, n.all);
  const cudaError_t e = ugb_launch(mixer_inputs_kernel<TI, T, STEP>, dim3((unsigned)((warps + 7) / 8)), dim3(256), 0, dev->stream, pdl, a, rows);
  if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of mixer_inputs_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(dev, "mixer_inputs_kernel");
}

// T result of (gate, up) pairs: fused in bf16, two launches in f32
int32_t gated_product(ugb_hybrid *m, ugb_hybrid_work &w, Mat g) {
  if (!m->f32) {
    g.silu_mul = true; g.f32_out = false;
    return ugb_hybrid_matmul(m, g);
  }
  float *out = (float *)g.out;
  const size_t out_ld = g.c_ld ? g.c_ld : g.n / 2;
  g.out = w.gu; g.c_ld = 0;
  if (int32_t rc = ugb_hybrid_matmul(m, g)) return rc;
  silu_mul_kernel<<<m->dev->sm_count * 4, 256, 0, m->dev->stream>>>(w.gu, out, g.m, (int)(g.n / 2), g.n, out_ld);
  return ugb_after_launch(m->dev, "silu_mul_kernel");
}

template <typename T>
int32_t run(ugb_hybrid *m, ugb_hybrid_work &w, const int *tok, int t_block, int off, int t, bool decode) {
  ugb_device *dev = m->dev;
  const bool pdl = m->pdl != 0;
  // In a bf16 decode step every kernel lets its successor start only after its own wait: when a kernel starts, everything up
  // to its predecessor's predecessor is complete (see row_update_kernel).
  const bool early = decode && pdl && !m->f32;
  const int B = m->batch, rows = B * t, wl = m->wl, n_runs = (int)m->runs.size();
  const bool whole = m->only == UGB_HYBRID_K_ALL;            // kernels timed alone leave the counts of the last whole pass as they are
  const bool looped = m->cfg.loop_times > 0, side = m->cfg.side_dim > 0;
  int32_t rc;
  cudaError_t e;

  // what the row kernel that completes the stream ahead of run i leaves for it
  auto prepare = [&](RowArgs<T> &a, int i) {
    a.copy_ld = wl;
    if (i < n_runs && m->runs[i].enter >= 0) {
      a.copy = (T *)w.xx; a.copy_ld = 2 * (size_t)wl;
      return;
    }
    a.h = (T *)w.h;
    a.gain = i < n_runs ? m->layers[m->runs[i].layer].norm1 : m->final_gain;
    if (whole && i < n_runs && m->layers[m->runs[i].layer].d.feed_forward == UGB_FF_EXPERTS) { a.zero = w.count; a.n_zero = m->layers[m->runs[i].layer].d.experts; }
  };
  {
    RowArgs<T> a;
    a.tok = tok; a.embed = (const T *)m->embed; a.vocab = m->cfg.vocab; a.t = t; a.tok_stride = t_block; a.tok_off = off;
    a.x = w.x; a.add_x = 0;
    prepare(a, 0);
    if (looped) { a.copy2 = (T *)w.xx + wl; a.copy_ld = 2 * (size_t)wl; }
    if ((rc = ugb_hybrid_rows<T>(m, a, rows, early))) return rc;
  }
  for (int i = 0; i < n_runs; ++i) {
    const ugb_hybrid_run &R = m->runs[i];
    const Weights &L = m->layers[R.layer];
    const ugb_hybrid_layer &d = L.d;
    const bool experts = d.feed_forward == UGB_FF_EXPERTS;
    if (R.enter >= 0) {
      const Tiling ti = decode ? ugb_hybrid_tile(m, wl, 2 * (size_t)wl) : Tiling{0, 1};
      if (m->on(UGB_HYBRID_K_LOOP)) {
        Mat g{w.prod, w.xx, m->loop_in, (size_t)rows, (size_t)wl, 2 * (size_t)wl};
        g.splits = ti.splits; g.bn = ti.bn;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
      RowArgs<T> a;
      a.part = w.prod; a.n_part = ti.splits; a.part_stride = (size_t)rows * wl;
      a.bias = m->loop_step + (size_t)R.enter * wl;
      a.x = w.x; a.add_x = 0; a.h = (T *)w.h; a.gain = L.norm1;
      if (experts && whole) { a.zero = w.count; a.n_zero = d.experts; }
      if ((rc = ugb_hybrid_rows<T>(m, a, rows, early))) return rc;
    }

    // ---- input projections
    const size_t n_in = L.n_in(), n_pre = n_in + (decode ? L.ep : 0);
    const Tiling in_t = decode ? ugb_hybrid_tile(m, n_pre, wl) : Tiling{0, 1};
    if (m->on(UGB_HYBRID_K_MIX_IN)) {
      Mat g{w.pre, w.h, L.w_in, (size_t)rows, n_pre, (size_t)wl};
      g.splits = in_t.splits; g.bn = in_t.bn; g.f32_out = decode || m->f32;
      if ((rc = ugb_hybrid_matmul(m, g))) return rc;
    }
    const size_t x0 = L.n_heads_in(), z0 = x0 + L.ci, pre_part = (size_t)rows * n_pre;
    auto heads = [&](auto &a) {
      a.ld = (int)n_pre; a.t = t; a.pos_off = off; a.t_max = m->t_max; a.pos_p = m->pos;
      a.heads = d.heads; a.kv_heads = d.kv_heads; a.dim = d.dim; a.dp = L.dp; a.vp = L.vp; a.rot_dims = d.rot_dims;
      a.interleaved = d.rot_interleaved; a.qk_norm = d.qk_norm; a.eps = m->cfg.eps;
      if (L.rot >= 0) { a.cos_ = m->rot[L.rot].cos_; a.sin_ = m->rot[L.rot].sin_; }
      a.q = (T *)w.q; a.kcache = (T *)R.cache; a.vcache = (T *)R.vcache; a.status = dev->status_dev;
    };
    T *tail = (T *)(m->tails + R.tail[0]);
    if (decode) {
      if (m->on(UGB_HYBRID_K_MIX_ROWS)) {
        MixerIn<float, T> a;
        heads(a);
        a.pre = w.pre; a.n_part = in_t.splits; a.part_stride = pre_part;
        a.conv_w = L.conv_w; a.conv_b = L.conv_b; a.taps = d.conv; a.ci = L.ci; a.tail = tail; a.u = (T *)w.hc;
        if (experts && whole) { a.experts = d.experts; a.top = d.top; a.choice = w.choice; a.count = w.count; }
        if ((rc = launch_mixer_inputs<float, T, true>(dev, a, rows, pdl))) return rc;
      }
    } else {
      if (m->on(UGB_HYBRID_K_MIX_ROWS)) {
        MixerIn<T, T> a;
        heads(a);
        a.pre = (const T *)w.pre;
        if ((rc = launch_mixer_inputs<T, T, false>(dev, a, rows, pdl))) return rc;
      }
      if (m->on(UGB_HYBRID_K_CONV) &&
          (rc = launch_gated_conv<T>(dev, (const T *)w.pre + x0, n_in, L.conv_w, L.conv_b, tail, (T *)(m->tails_next + R.tail[0]), (T *)w.hc, B, t,
                                     d.conv, L.ci)))
        return rc;
    }

    // ---- scan
    const size_t n_cat = L.n_cat(), cat_s = (size_t)d.heads * L.vp, cat_f = cat_s + L.ci;
    const int xr = L.rp + 2 * L.np;
    const Tiling x_t = decode ? ugb_hybrid_tile(m, xr, L.ci) : Tiling{0, narrow_splits(m, rows, xr, L.ci)};
    if (m->on(UGB_HYBRID_K_SCAN_IN)) {
      const bool sum = !decode && x_t.splits > 1;            // a block's split product is summed and rounded to T
      Mat g{sum ? (void *)w.part : w.xdb, w.hc, L.w_x, (size_t)rows, (size_t)xr, (size_t)L.ci};
      g.splits = x_t.splits; g.bn = sum ? 256 : x_t.bn; g.f32_out = decode || m->f32 || sum;
      if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      if (sum) {
        const size_t n4 = (size_t)rows * xr / 4;
        e = ugb_launch(sum_partials_kernel<T>, dim3((unsigned)((n4 + 255) / 256)), dim3(256), 0, dev->stream, pdl, w.part, x_t.splits, (size_t)rows * xr, n4, (T *)w.xdb);
        if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of sum_partials_kernel failed: %s", cudaGetErrorString(e));
        if ((rc = ugb_after_launch(dev, "sum_partials_kernel"))) return rc;
      }
      if (!decode) {
        Mat h{w.dt, w.xdb, L.w_dt, (size_t)rows, (size_t)L.ci, (size_t)L.rp};
        h.a_ld = xr; h.nk = false; h.f32_out = m->f32;
        h.bn = 128;                                          // few k blocks: the epilogues are the work, and small ones overlap better
        if ((rc = ugb_hybrid_matmul(m, h))) return rc;
      }
    }
    if (m->on(UGB_HYBRID_K_SCAN)) {
      ugb_scan_args a{};
      a.f32 = m->f32; a.shape = {L.lanes, L.per_lane, L.np}; a.channels = L.ci; a.u = w.hc; a.a = L.a; a.skip = L.skip; a.dt_bias = L.dt_b;
      a.state = R.state; a.out = (T *)w.cat + cat_s; a.out_ld = n_cat; a.scale = d.scan_scale; a.xr = xr; a.rp = L.rp;
      if (decode) rc = ugb_scan_step(dev, a, L.w_dt, {(const float *)w.xdb, x_t.splits, (size_t)rows * xr, (size_t)xr},
                                     {w.pre + z0, in_t.splits, pre_part, n_pre}, rows, pdl, early);
      else rc = ugb_scan_block(dev, a, w.dt, w.xdb, (const T *)w.pre + z0, n_in, B, t);
      if (rc) return rc;
    }

    // ---- attention
    if (m->on(UGB_HYBRID_K_ATTENTION)) {
      if (!decode && L.expand && t > m->absorb_max) {
        ugb_prefill_attention_args a;
        a.q = (const __nv_bfloat16 *)w.q; a.k = (const __nv_bfloat16 *)R.cache; a.v = (const __nv_bfloat16 *)R.vcache;
        a.out = (__nv_bfloat16 *)w.cat; a.out_ld = (long long)n_cat; a.out_scale = d.attention_scale;
        a.batch = B; a.t = t; a.pos0 = m->host_pos + off; a.n_heads = d.heads; a.n_kv = d.kv_heads; a.kv_rows = m->t_max;
        a.dq = L.dp; a.dv = L.vp; a.scale = d.scale;
        if ((rc = ugb_prefill_attention_tc(dev, a))) return rc;
      } else {
        ugb_grouped_attention_args a{};
        a.f32 = m->f32; a.q = w.q; a.k = R.cache; a.v = R.vcache; a.out = w.cat; a.out_ld = n_cat; a.out_scale = d.attention_scale;
        a.rows = rows; a.t = t; a.pos_p = m->pos; a.pos_off = off; a.heads = d.heads; a.kv_heads = d.kv_heads; a.dq = L.dp; a.dv = L.vp;
        a.t_max = m->t_max; a.scale = d.scale; a.pdl = pdl; a.early = early;
        a.splits = m->att_splits_opt > 0 ? std::min(m->att_splits_opt, UGB_GROUPED_MAX_SPLITS) : ugb_grouped_attention_splits(a, dev->sm_count);
        if ((rc = ugb_grouped_attention(dev, a))) return rc;
      }
    }

    // ---- feed-forward
    if (L.fl && m->on(UGB_HYBRID_K_UP)) {
      Mat g{(T *)w.cat + cat_f, w.h, L.w_up, (size_t)rows, 2 * (size_t)L.fl, (size_t)wl};
      g.c_ld = n_cat;
      if ((rc = gated_product(m, w, g))) return rc;
    }
    if (experts) {
      const int tile = w.tile, tiles = group_tiles((size_t)rows * d.top, d.experts, tile);
      const size_t xrows = (size_t)tiles * tile;
      if (m->on(UGB_HYBRID_K_ROUTE)) {
        if (!decode) {
          const size_t es = m->es();
          Mat g{w.part, w.h, (const char *)L.w_in + n_in * wl * es, (size_t)rows, (size_t)L.ep, (size_t)wl};
          g.splits = narrow_splits(m, rows, L.ep, wl); g.bn = g.splits > 1 ? 256 : 0;
          if ((rc = ugb_hybrid_matmul(m, g))) return rc;
          if (!whole) UGB_CUDA(dev, cudaMemsetAsync(w.count, 0, d.experts * sizeof(int), dev->stream));
          route_kernel<<<(rows + ROUTE_ROWS - 1) / ROUTE_ROWS, 256, 0, dev->stream>>>(w.part, g.splits, L.ep, rows, d.experts, d.top, w.choice, w.count);
          if ((rc = ugb_after_launch(dev, "route_kernel"))) return rc;
        }
        e = ugb_launch(expert_rows_kernel<T>, dim3(rows), dim3(256), 0, dev->stream, pdl, (const T *)w.h, w.choice, w.count, d.experts, d.top, tile, tiles,
                       (T *)w.xin, w.slot, w.map, wl);
        if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of expert_rows_kernel failed: %s", cudaGetErrorString(e));
        if ((rc = ugb_after_launch(dev, "expert_rows_kernel"))) return rc;
      }
      Mat g{w.xmid, w.xin, L.x_up, xrows, 2 * (size_t)L.ef, (size_t)wl};
      g.groups = w.map; g.n_groups = d.experts; g.tile = tile;
      g.bn = tile == 64 ? 128 : 256;
      if (m->on(UGB_HYBRID_K_EXPERT_UP) && (rc = gated_product(m, w, g))) return rc;
      g.out = w.xout; g.a = w.xmid; g.w = L.x_down; g.n = wl; g.k = L.ef;
      if (m->on(UGB_HYBRID_K_EXPERT_DOWN) && (rc = ugb_hybrid_matmul(m, g))) return rc;
    }

    // ---- output projections, residual
    const Tiling out_t = decode ? ugb_hybrid_tile(m, wl, n_cat) : Tiling{0, 1};
    if (m->on(UGB_HYBRID_K_OUT)) {
      Mat g{w.prod, w.cat, L.w_out, (size_t)rows, (size_t)wl, n_cat};
      g.splits = out_t.splits; g.bn = out_t.bn;
      if ((rc = ugb_hybrid_matmul(m, g))) return rc;
    }
    RowArgs<T> a;
    a.part = w.prod; a.n_part = out_t.splits; a.part_stride = (size_t)rows * wl; a.x = w.x;
    if (experts) { a.routed = w.xout; a.slot = w.slot; a.top = d.top; }
    if (side) { a.copy = (T *)w.xs; a.copy_ld = wl; }
    else prepare(a, i + 1);
    if ((rc = ugb_hybrid_rows<T>(m, a, rows, early))) return rc;

    // ---- input of the token
    if (side) {
      const Tiling g_t = decode ? ugb_hybrid_tile(m, m->sl, wl) : Tiling{0, narrow_splits(m, rows, m->sl, wl)}, p_t = decode ? ugb_hybrid_tile(m, wl, m->sl) : Tiling{0, 1};
      if (m->on(UGB_HYBRID_K_SIDE)) {
        Mat g{w.side, w.xs, L.side_gate, (size_t)rows, (size_t)m->sl, (size_t)wl};
        g.splits = g_t.splits; g.bn = !decode && g_t.splits > 1 ? 256 : g_t.bn;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
      if (m->on(UGB_HYBRID_K_SIDE_GATE)) {
        e = ugb_launch(token_gate_kernel<T>, dim3((unsigned)(((size_t)rows * m->sl / 4 + 255) / 256)), dim3(256), 0, dev->stream, pdl, w.side, g_t.splits,
                       (size_t)rows * m->sl, (size_t)rows * m->sl / 4, m->sl, m->cfg.side_dim, tok, t, t_block, off, (const T *)m->side_embed, (size_t)m->cfg.layers * m->cfg.side_dim,
                       R.layer * m->cfg.side_dim, m->cfg.vocab, (T *)w.side_h);
        if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "launch of token_gate_kernel failed: %s", cudaGetErrorString(e));
        if ((rc = ugb_after_launch(dev, "token_gate_kernel"))) return rc;
      }
      if (m->on(UGB_HYBRID_K_SIDE)) {
        Mat g{w.prod, w.side_h, L.side_proj, (size_t)rows, (size_t)wl, (size_t)m->sl};
        g.splits = p_t.splits; g.bn = p_t.bn;
        if ((rc = ugb_hybrid_matmul(m, g))) return rc;
      }
      RowArgs<T> s;
      s.part = w.prod; s.n_part = p_t.splits; s.part_stride = (size_t)rows * wl; s.x = w.x; s.post_gain = L.side_gain;
      prepare(s, i + 1);
      if ((rc = ugb_hybrid_rows<T>(m, s, rows, early))) return rc;
    }
    if (!decode && (rc = ugb_hybrid_keep(m, w, i, t_block, off, t))) return rc;
  }
  return UGB_OK;
}

}  // namespace

int32_t ugb_parallel_run(ugb_hybrid *m, ugb_hybrid_work &w, const int *tok, int t_block, int off, int t, bool decode) {
  return m->f32 ? run<float>(m, w, tok, t_block, off, t, decode) : run<__nv_bfloat16>(m, w, tok, t_block, off, t, decode);
}

int32_t ugb_parallel_softcap(ugb_hybrid *m, float *logits, size_t n) {
  const cudaError_t e = ugb_launch(softcap_kernel, dim3((unsigned)std::min<size_t>((n / 4 + 255) / 256, (size_t)m->dev->sm_count * 8)), dim3(256), 0,
                                   m->dev->stream, m->pdl != 0, logits, n / 4, m->cfg.logit_softcap);
  if (e != cudaSuccess) return ugb_fail(m->dev, UGB_ERR_CUDA, "launch of softcap_kernel failed: %s", cudaGetErrorString(e));
  return ugb_after_launch(m->dev, "softcap_kernel");
}

// ------------------------------------------------------------ life cycle ----
int32_t ugb_parallel_layer(ugb_hybrid *m, int i) {
  ugb_device *dev = m->dev;
  Weights &L = m->layers[i];
  const ugb_hybrid_layer &d = L.d;
  const size_t es = m->es(), wl = m->wl;
  int32_t rc;
  UGB_REQUIRE(dev, d.mixer == UGB_MIXER_ATTENTION_SCAN, UGB_ERR_UNSUPPORTED, "layer %d: mixer kind %d in the parallel form", i, d.mixer);
  UGB_REQUIRE(dev, d.heads > 0 && d.kv_heads > 0 && d.heads % d.kv_heads == 0 && d.dim > 0 && d.vdim > 0, UGB_ERR_INVALID,
              "layer %d: %d heads on %d, %d- and %d-wide", i, d.heads, d.kv_heads, d.dim, d.vdim);
  UGB_REQUIRE(dev, d.dim <= HEAD_DIM_MAX && d.vdim <= 512, UGB_ERR_UNSUPPORTED, "layer %d: heads of %d and %d values", i, d.dim, d.vdim);
  UGB_REQUIRE(dev, d.rot_dims >= 0 && d.rot_dims <= d.dim && d.rot_dims % 2 == 0, UGB_ERR_INVALID, "layer %d: %d rotated dimensions of %d", i, d.rot_dims, d.dim);
  UGB_REQUIRE(dev, d.inner > 0 && d.state > 0 && d.conv > 0 && d.conv <= 64 && d.dt_rank > 0, UGB_ERR_INVALID,
              "layer %d: scan of %d channels, %d states, %d taps, rank %d", i, d.inner, d.state, d.conv, d.dt_rank);
  const int dp = ugb_prefill_attention_width(d.dim), vp = ugb_prefill_attention_width(d.vdim);
  const bool padded = !m->f32 && dp && vp;                   // heads that the tensor-core kernels take
  L.expand = padded && d.scale > 0.f;
  L.dp = padded ? dp : (int)up8(d.dim);
  L.vp = padded ? vp : (int)up8(d.vdim);
  L.nq = d.heads * L.dp; L.nk = d.kv_heads * L.dp; L.nv = d.kv_heads * L.vp;
  const ugb_scan_shape sh = ugb_scan_shape_of(d.state);
  UGB_REQUIRE(dev, sh.lanes > 0, UGB_ERR_UNSUPPORTED, "layer %d: %d states per channel", i, d.state);
  L.lanes = sh.lanes; L.per_lane = sh.per_lane; L.np = sh.np;
  L.ci = (int)up8(d.inner); L.rp = (int)up8(d.dt_rank);
  if (d.feed_forward == UGB_FF_GATED) UGB_REQUIRE(dev, d.ff > 0, UGB_ERR_INVALID, "layer %d: ff %d", i, d.ff);
  else if (d.feed_forward == UGB_FF_EXPERTS)
    UGB_REQUIRE(dev, d.ff >= 0 && d.experts > 0 && d.experts <= 32 * ROUTER_PER_LANE && d.top > 0 && d.top <= d.experts && d.expert_ff > 0, UGB_ERR_UNSUPPORTED,
                "layer %d: %d of %d experts, %d columns (shared %d)", i, d.top, d.experts, d.expert_ff, d.ff);
  else UGB_REQUIRE(dev, d.feed_forward == UGB_FF_NONE, UGB_ERR_UNSUPPORTED, "layer %d: feed-forward kind %d", i, d.feed_forward);
  const bool experts = d.feed_forward == UGB_FF_EXPERTS;
  L.fl = d.feed_forward == UGB_FF_NONE ? 0 : (int)up8(d.ff);
  L.ep = experts ? (int)up8(d.experts) : 0;
  L.ef = experts ? (int)up8(d.expert_ff) : 0;
  const size_t E = experts ? d.experts : 0;
  if ((rc = dmalloc(m, &L.norm1, wl, true)) || (rc = ugb_hybrid_alloc(m, &L.w_in, (size_t)(L.n_in() + L.ep) * wl * es, true)) ||
      (rc = ugb_hybrid_alloc(m, &L.w_out, wl * L.n_cat() * es, true)) || (rc = ugb_hybrid_alloc(m, &L.w_up, 2 * (size_t)L.fl * wl * es, true)) ||
      (rc = ugb_hybrid_alloc(m, &L.x_up, E * 2 * L.ef * wl * es, true)) || (rc = ugb_hybrid_alloc(m, &L.x_down, E * wl * L.ef * es, true)) ||
      (rc = ugb_hybrid_alloc(m, &L.w_x, (size_t)(L.rp + 2 * L.np) * L.ci * es, true)) || (rc = ugb_hybrid_alloc(m, &L.w_dt, (size_t)L.rp * L.ci * es, true)) ||
      (rc = dmalloc(m, &L.conv_w, (size_t)d.conv * L.ci, true)) || (rc = dmalloc(m, &L.conv_b, L.ci, true)) ||
      (rc = dmalloc(m, &L.a, (size_t)L.ci * L.np, true)) || (rc = dmalloc(m, &L.skip, L.ci, true)) || (rc = dmalloc(m, &L.dt_b, L.ci, true)))
    return rc;
  if (m->sl && ((rc = ugb_hybrid_alloc(m, &L.side_gate, m->sl * wl * es, true)) || (rc = ugb_hybrid_alloc(m, &L.side_proj, wl * m->sl * es, true)) ||
                (rc = dmalloc(m, &L.side_gain, wl, true))))
    return rc;
  if (d.rot_dims > 0) {
    for (size_t k = 0; k < m->rot.size(); ++k)
      if (m->rot[k].base == d.rot_base && m->rot[k].dims == d.rot_dims) L.rot = (int)k;
    if (L.rot < 0) {
      ugb_hybrid::Rotation R{d.rot_base, d.rot_dims, nullptr, nullptr};
      const int half = d.rot_dims / 2;
      std::vector<double> freq(half);
      for (int k = 0; k < half; ++k) freq[k] = std::pow((double)d.rot_base, -2.0 * k / d.rot_dims);
      double *dev_freq = nullptr;
      if ((rc = dmalloc(m, &R.cos_, (size_t)m->t_max * half)) || (rc = dmalloc(m, &R.sin_, (size_t)m->t_max * half)) || (rc = dmalloc(m, &dev_freq, half))) return rc;
      UGB_CUDA(dev, cudaMemcpyAsync(dev_freq, freq.data(), half * sizeof(double), cudaMemcpyHostToDevice, dev->stream));
      rotation_table_kernel<<<(unsigned)(((size_t)m->t_max * half + 255) / 256), 256, 0, dev->stream>>>(dev_freq, R.cos_, R.sin_, m->t_max, half);
      if ((rc = ugb_after_launch(dev, "rotation_table_kernel"))) return rc;
      UGB_CUDA(dev, cudaStreamSynchronize(dev->stream));     // freq is the copy's source
      L.rot = (int)m->rot.size();
      m->rot.push_back(R);
    }
  }
  return UGB_OK;
}

int32_t ugb_parallel_model(ugb_hybrid *m) {
  ugb_device *dev = m->dev;
  const ugb_hybrid_config &c = m->cfg;
  const size_t es = m->es(), wl = m->wl;
  int32_t rc;
  UGB_REQUIRE(dev, c.conv_taps == 0 && c.depth_average == 0, UGB_ERR_UNSUPPORTED, "the parallel form has no input convolution and no depth average");
  UGB_REQUIRE(dev, c.loop_times >= 0 && c.side_dim >= 0 && c.logit_softcap >= 0.f, UGB_ERR_INVALID, "negative loop count, token input or soft cap");
  UGB_REQUIRE(dev, c.loop_times == 0 || (c.loop_start >= 0 && c.loop_start < c.loop_stop && c.loop_stop <= c.layers), UGB_ERR_INVALID,
              "a loop over layers %d .. %d of %d", c.loop_start, c.loop_stop, c.layers);
  m->sl = (int)up8(c.side_dim);
  for (int i = 0; i < c.layers; ++i)
    if ((rc = ugb_parallel_layer(m, i))) return rc;
  auto add = [&](int layer, int enter) { ugb_hybrid_run R; R.layer = layer; R.enter = enter; m->runs.push_back(R); };
  const int lo = c.loop_times ? c.loop_start : c.layers, hi = c.loop_times ? c.loop_stop : c.layers;
  for (int i = 0; i < lo; ++i) add(i, -1);
  for (int p = 0; p < c.loop_times; ++p)
    for (int i = lo; i < hi; ++i) add(i, i == lo ? p : -1);
  for (int i = hi; i < c.layers; ++i) add(i, -1);
  for (ugb_hybrid_run &R : m->runs) {
    const Weights &L = m->layers[R.layer];
    R.tail[0] = m->tail_bytes;
    m->tail_bytes += (size_t)m->batch * (L.d.conv - 1) * L.ci * es;
    R.state_len = (size_t)m->batch * L.ci * L.np;
    const size_t keys = (size_t)m->batch * L.d.kv_heads * m->t_max;
    if ((rc = dmalloc(m, &R.state, R.state_len, true)) || (rc = ugb_hybrid_alloc(m, &R.cache, keys * L.dp * es, true)) ||
        (rc = ugb_hybrid_alloc(m, &R.vcache, keys * L.vp * es, true)))
      return rc;
  }
  if (c.loop_times && ((rc = ugb_hybrid_alloc(m, &m->loop_in, wl * 2 * wl * es, true)) || (rc = dmalloc(m, &m->loop_step, (size_t)c.loop_times * wl, true)))) return rc;
  if (c.side_dim && (rc = ugb_hybrid_alloc(m, &m->side_embed, (size_t)c.vocab * c.layers * c.side_dim * es, true))) return rc;
  return UGB_OK;
}

int32_t ugb_parallel_work(ugb_hybrid *m, ugb_hybrid_work &w, int rows, bool decode) {
  const size_t R = rows, es = m->es(), wl = m->wl, parts = decode ? UGB_HYBRID_MAX_SPLITS : 1;
  size_t pre = 8, q = 8, ci = 8, cat = 8, xr = 8, gu = 8, ep = 8, top = 0, E = 0, xrows = 0, ef = 8;
  w.tile = decode ? 64 : 128;
  for (const Weights &L : m->layers) {
    pre = std::max<size_t>(pre, L.n_in() + L.ep); q = std::max<size_t>(q, L.nq); ci = std::max<size_t>(ci, L.ci);
    cat = std::max<size_t>(cat, L.n_cat()); xr = std::max<size_t>(xr, L.rp + 2 * L.np); ep = std::max<size_t>(ep, L.ep);
    size_t xl = 0;
    if (L.d.feed_forward == UGB_FF_EXPERTS) {
      top = std::max<size_t>(top, L.d.top); E = std::max<size_t>(E, L.d.experts); ef = std::max<size_t>(ef, L.ef);
      w.tiles = std::max(w.tiles, group_tiles(R * L.d.top, L.d.experts, w.tile));
      xl = (size_t)group_tiles(R * L.d.top, L.d.experts, w.tile) * w.tile;
    }
    xrows = std::max(xrows, xl);
    if (m->f32) gu = std::max({gu, R * 2 * L.fl, xl * 2 * L.ef});
  }
  int32_t rc;
  void *pre_p = nullptr;
  if ((rc = dmalloc(m, &w.x, R * wl)) || (rc = ugb_hybrid_alloc(m, &pre_p, parts * R * pre * (decode ? 4 : es), false)) || (rc = dmalloc(m, &w.prod, parts * R * wl)) ||
      (rc = ugb_hybrid_alloc(m, &w.h, R * wl * es, true)) || (rc = ugb_hybrid_alloc(m, &w.hc, R * ci * es, false)) || (rc = ugb_hybrid_alloc(m, &w.q, R * q * es, false)) ||
      (rc = ugb_hybrid_alloc(m, &w.cat, R * cat * es, false)) || (rc = ugb_hybrid_alloc(m, &w.xs, R * wl * es, false)) ||
      (rc = ugb_hybrid_alloc(m, &w.xx, m->cfg.loop_times ? R * 2 * wl * es : 0, false)) ||
      (rc = ugb_hybrid_alloc(m, &w.xdb, parts * R * xr * (decode ? 4 : es), false)) || (rc = ugb_hybrid_alloc(m, &w.dt, decode ? 0 : R * ci * es, false)) ||
      (rc = dmalloc(m, &w.gu, gu)) || (rc = dmalloc(m, &w.side, (decode ? parts * R : narrow_rows(m, R)) * m->sl)) || (rc = ugb_hybrid_alloc(m, &w.side_h, R * m->sl * es, false)) ||
      (rc = dmalloc(m, &w.part, decode ? 0 : narrow_rows(m, R) * std::max(xr, ep))) || (rc = dmalloc(m, &w.choice, R * top, true)) || (rc = dmalloc(m, &w.slot, R * top, true)) ||
      (rc = dmalloc(m, &w.count, E, true)) || (rc = dmalloc(m, &w.map, w.tiles)) || (rc = ugb_hybrid_alloc(m, &w.xin, xrows * wl * es, true)) ||
      (rc = ugb_hybrid_alloc(m, &w.xmid, xrows * ef * es, true)) || (rc = dmalloc(m, &w.xout, xrows * wl)))
    return rc;
  w.pre = (float *)pre_p;
  if (w.tiles) UGB_CUDA(m->dev, cudaMemsetAsync(w.map, 0xff, (size_t)w.tiles * sizeof(int), m->dev->stream));
  w.rows = rows;
  return UGB_OK;
}

int32_t ugb_parallel_load(ugb_hybrid *m, const char *name, const ugb_slice *w, bool *known) {
  ugb_device *dev = m->dev;
  const ugb_hybrid_config &c = m->cfg;
  const size_t W = c.width, wl = m->wl, es = m->es();
  const int32_t dt = m->f32 ? UGB_F32 : UGB_BF16;
  const std::string s(name);
  auto at = [&](void *base, size_t elems) { return (void *)((char *)base + elems * es); };
  // rows [row0, row0 + n) x columns [col0, col0 + nc) of a [rows, cols] tensor into rows of `pitch` elements
  auto part = [&](void *dst, size_t rows, size_t cols, size_t row0, size_t n, size_t col0, size_t nc, size_t pitch) {
    return engine_put_matrix(m, w, dst, dt, rows, cols, row0, n, col0, nc, pitch, name);
  };
  auto put = [&](void *dst, size_t rows, size_t cols, size_t pitch) { return part(dst, rows, cols, 0, rows, 0, cols, pitch); };
  auto put_heads = [&](void *dst, size_t heads, size_t d, size_t dp) -> int32_t {      // d rows per head
    for (size_t h = 0; h < heads; ++h)
      if (int32_t rc = part(at(dst, h * dp * wl), heads * d, W, h * d, d, 0, W, wl)) return rc;
    return UGB_OK;
  };
  auto vec = [&](float *dst, size_t n) { return engine_put_matrix(m, w, dst, UGB_F32, 1, n, 0, 1, 0, n, n, name); };
  auto gain = [&](float *dst) { return ugb_hybrid_gain(m, w, dst, (int)W, c.gain_offset, name); };
  if (s == "loop.in" && c.loop_times) {
    if (int32_t rc = part(m->loop_in, W, 2 * W, 0, W, 0, W, 2 * wl)) return rc;
    return part(at(m->loop_in, wl), W, 2 * W, 0, W, W, W, 2 * wl);
  }
  if (s == "loop.step" && c.loop_times) return engine_put_matrix(m, w, m->loop_step, UGB_F32, c.loop_times, W, 0, c.loop_times, 0, W, wl, name);
  if (s == "side.embed" && c.side_dim) return put(m->side_embed, c.vocab, (size_t)c.layers * c.side_dim, (size_t)c.layers * c.side_dim);
  const size_t dot = s.find('.');
  *known = s.size() > 1 && s[0] == 'l' && dot != std::string::npos && dot > 1 && dot < 10 && s.find_first_not_of("0123456789", 1) == dot;
  if (!*known) return UGB_OK;
  const int i = atoi(s.c_str() + 1);
  UGB_REQUIRE(dev, i < c.layers, UGB_ERR_INVALID, "%s: layer index out of range", name);
  Weights &L = m->layers[i];
  const ugb_hybrid_layer &d = L.d;
  const std::string k = s.substr(dot + 1);
  const size_t n_cat = L.n_cat(), cat_s = (size_t)d.heads * L.vp, cat_f = cat_s + L.ci, I = d.inner;
  if (k == "norm1") return gain(L.norm1);
  if (c.side_dim) {
    if (k == "side.gate") return put(L.side_gate, c.side_dim, W, wl);
    if (k == "side.proj") return put(L.side_proj, W, c.side_dim, m->sl);
    if (k == "side.norm") return ugb_hybrid_gain(m, w, L.side_gain, (int)W, 0.f, name);
  }
  if (k == "mix.left.q") return put_heads(L.w_in, d.heads, d.dim, L.dp);
  if (k == "mix.left.k") return put_heads(at(L.w_in, (size_t)L.nq * wl), d.kv_heads, d.dim, L.dp);
  if (k == "mix.left.v") return put_heads(at(L.w_in, (size_t)(L.nq + L.nk) * wl), d.kv_heads, d.vdim, L.vp);
  if (k == "mix.left.o") {                                   // columns head by head
    for (size_t h = 0; h < (size_t)d.heads; ++h)
      if (int32_t rc = part(at(L.w_out, h * L.vp), W, (size_t)d.heads * d.vdim, 0, W, h * d.vdim, d.vdim, n_cat)) return rc;
    return UGB_OK;
  }
  if (k == "mix.right.in") {
    void *x = at(L.w_in, (size_t)L.n_heads_in() * wl);
    if (int32_t rc = part(x, 2 * I, W, 0, I, 0, W, wl)) return rc;
    return part(at(x, (size_t)L.ci * wl), 2 * I, W, I, I, 0, W, wl);
  }
  if (k == "mix.right.conv")
    return ugb_hybrid_f32(m, w, I * d.conv, name, [&](const float *src) {
      taps_kernel<<<((int)I * d.conv + 255) / 256, 256, 0, dev->stream>>>(src, L.conv_w, (int)I, d.conv, L.ci);
      return ugb_after_launch(dev, "taps_kernel");
    });
  if (k == "mix.right.conv.b") return vec(L.conv_b, I);
  if (k == "mix.right.x") {
    const size_t n = d.state, r = d.dt_rank, all = r + 2 * n, ci = L.ci;
    if (int32_t rc = part(L.w_x, all, I, 0, r, 0, I, ci)) return rc;
    if (int32_t rc = part(at(L.w_x, L.rp * ci), all, I, r, n, 0, I, ci)) return rc;
    return part(at(L.w_x, (L.rp + L.np) * ci), all, I, r + n, n, 0, I, ci);
  }
  if (k == "mix.right.dt")
    return ugb_hybrid_f32(m, w, I * d.dt_rank, name, [&](const float *src) {
      const int grid = dev->sm_count * 4;
      if (m->f32) transpose_kernel<float><<<grid, 256, 0, dev->stream>>>(src, (float *)L.w_dt, I, (size_t)d.dt_rank, (size_t)L.ci);
      else transpose_kernel<__nv_bfloat16><<<grid, 256, 0, dev->stream>>>(src, (__nv_bfloat16 *)L.w_dt, I, (size_t)d.dt_rank, (size_t)L.ci);
      return ugb_after_launch(dev, "transpose_kernel");
    });
  if (k == "mix.right.dt.b") return vec(L.dt_b, I);
  if (k == "mix.right.A_log")
    return ugb_hybrid_f32(m, w, I * d.state, name, [&](const float *src) {
      decay_kernel<<<((int)I * d.state + 255) / 256, 256, 0, dev->stream>>>(src, L.a, (int)I, d.state, L.np, ugb_scan_decay_unit(m->f32));
      return ugb_after_launch(dev, "decay_kernel");
    });
  if (k == "mix.right.D") return vec(L.skip, I);
  if (k == "mix.right.o") return put(at(L.w_out, cat_s), W, I, n_cat);
  // gated feed-forwards: gate and up rows alternate
  if (d.feed_forward == UGB_FF_GATED || (d.feed_forward == UGB_FF_EXPERTS && d.ff > 0)) {
    const std::string p = d.feed_forward == UGB_FF_GATED ? "mlp." : "mlp.shared.";
    if (k == p + "gate") return put(L.w_up, d.ff, W, 2 * wl);
    if (k == p + "up") return put(at(L.w_up, wl), d.ff, W, 2 * wl);
    if (k == p + "down") return put(at(L.w_out, cat_f), W, d.ff, n_cat);
  }
  if (d.feed_forward == UGB_FF_EXPERTS) {
    if (k == "mlp.router") return put(at(L.w_in, (size_t)L.n_in() * wl), d.experts, W, wl);
    int e = -1, n = 0;
    if (sscanf(k.c_str(), "mlp.e%d.%n", &e, &n) == 1 && n > 0 && e >= 0 && e < d.experts) {
      const std::string what = k.substr(n);
      void *up = at(L.x_up, (size_t)e * 2 * L.ef * wl);
      if (what == "gate") return put(up, d.expert_ff, W, 2 * wl);
      if (what == "up") return put(at(up, wl), d.expert_ff, W, 2 * wl);
      if (what == "down") return put(at(L.x_down, (size_t)e * wl * L.ef), W, d.expert_ff, L.ef);
    }
  }
  *known = false;
  return UGB_OK;
}

// ------------------------------------------------------- mechanisms alone ----
extern "C" {

static int32_t act_dtype(ugb_device *dev, const ugb_slice *a, const ugb_slice *b, const char *what) {
  UGB_REQUIRE(dev, a && b, UGB_ERR_INVALID, "%s: null slice", what);
  UGB_REQUIRE(dev, a->dtype == b->dtype && (a->dtype == UGB_BF16 || a->dtype == UGB_F32), UGB_ERR_DTYPE,
              "%s: activations must be BF16 or F32 alike", what);
  return UGB_OK;
}

int32_t ugb_gated_conv(ugb_device *dev, const ugb_slice *h, const ugb_slice *w, const ugb_slice *bias, ugb_slice *tail, ugb_slice *out,
                       size_t b, size_t t, size_t width, size_t taps) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, h, out, "gated_conv")) return rc;
  UGB_REQUIRE(dev, width % 8 == 0 && taps >= 1 && taps <= 64 && b <= 65535 && b * t * width < (1ull << 31), UGB_ERR_SHAPE, "gated_conv: unsupported shape");
  UGB_SLICE(dev, h, h->dtype, b * t * width);
  UGB_SLICE(dev, out, h->dtype, b * t * width);
  UGB_SLICE(dev, tail, h->dtype, b * (taps - 1) * width);
  UGB_SLICE(dev, w, UGB_F32, taps * width);
  UGB_SLICE(dev, bias, UGB_F32, width);
  UGB_REQUIRE(dev, out->ptr != h->ptr, UGB_ERR_INVALID, "gated_conv: in place");
  if (b == 0 || t == 0 || width == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  const size_t bytes = b * (taps - 1) * width * ugb_dtype_size(h->dtype);
  void *tmp = nullptr;
  UGB_CUDA(dev, ugb_malloc_async(dev, &tmp, bytes + 16));
  const float *wp = (const float *)w->ptr, *bp = (const float *)bias->ptr;
  int32_t rc;
  if (h->dtype == UGB_F32)
    rc = launch_gated_conv<float>(dev, (const float *)h->ptr, width, wp, bp, (const float *)tail->ptr, (float *)tmp, (float *)out->ptr, (int)b, (int)t, (int)taps, (int)width);
  else
    rc = launch_gated_conv<__nv_bfloat16>(dev, (const __nv_bfloat16 *)h->ptr, width, wp, bp, (const __nv_bfloat16 *)tail->ptr, (__nv_bfloat16 *)tmp,
                                          (__nv_bfloat16 *)out->ptr, (int)b, (int)t, (int)taps, (int)width);
  if (!rc && bytes) UGB_CUDA(dev, cudaMemcpyAsync(tail->ptr, tmp, bytes, cudaMemcpyDeviceToDevice, dev->stream));
  cudaFreeAsync(tmp, dev->stream);
  return rc;
}

int32_t ugb_head_inputs(ugb_device *dev, const ugb_slice *pre, const ugb_slice *cos_, const ugb_slice *sin_, const ugb_slice *pos, ugb_slice *q,
                        ugb_slice *kcache, ugb_slice *vcache, size_t b, size_t t, size_t heads, size_t kv_heads, size_t dim, size_t vdim, size_t rot_dims,
                        int32_t interleaved, int32_t qk_norm, float eps, size_t t_max) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, pre, q, "head_inputs")) return rc;
  UGB_REQUIRE(dev, dim % 8 == 0 && vdim % 8 == 0 && dim > 0 && vdim > 0 && dim <= HEAD_DIM_MAX && rot_dims <= dim && rot_dims % 2 == 0 && heads > 0 &&
                       kv_heads > 0 && b * t <= (1u << 30) && t_max <= (1u << 30) && heads + kv_heads * (1 + vdim) <= 65535, UGB_ERR_SHAPE, "head_inputs: unsupported shape");
  const size_t ld = (heads + kv_heads) * dim + kv_heads * vdim;
  UGB_SLICE(dev, pre, q->dtype, b * t * ld);
  UGB_SLICE(dev, q, q->dtype, b * t * heads * dim);
  UGB_SLICE(dev, kcache, q->dtype, b * kv_heads * t_max * dim);
  UGB_SLICE(dev, vcache, q->dtype, b * kv_heads * t_max * vdim);
  UGB_SLICE(dev, cos_, UGB_F32, t_max * rot_dims / 2);
  UGB_SLICE(dev, sin_, UGB_F32, t_max * rot_dims / 2);
  UGB_SLICE(dev, pos, UGB_I32, 1);
  if (b == 0 || t == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  auto fill = [&](auto &a) {
    a.ld = (int)ld; a.t = (int)t; a.t_max = (int)t_max; a.pos_p = (const int *)pos->ptr; a.heads = (int)heads; a.kv_heads = (int)kv_heads;
    a.dim = a.dp = (int)dim; a.vp = (int)vdim; a.rot_dims = (int)rot_dims; a.interleaved = interleaved; a.qk_norm = qk_norm; a.eps = eps;
    a.cos_ = (const float *)cos_->ptr; a.sin_ = (const float *)sin_->ptr; a.status = dev->status_dev;
  };
  if (q->dtype == UGB_F32) {
    MixerIn<float, float> a;
    fill(a);
    a.pre = (const float *)pre->ptr; a.q = (float *)q->ptr; a.kcache = (float *)kcache->ptr; a.vcache = (float *)vcache->ptr;
    return launch_mixer_inputs<float, float, false>(dev, a, (int)(b * t), false);
  }
  MixerIn<__nv_bfloat16, __nv_bfloat16> a;
  fill(a);
  a.pre = (const __nv_bfloat16 *)pre->ptr; a.q = (__nv_bfloat16 *)q->ptr; a.kcache = (__nv_bfloat16 *)kcache->ptr; a.vcache = (__nv_bfloat16 *)vcache->ptr;
  return launch_mixer_inputs<__nv_bfloat16, __nv_bfloat16, false>(dev, a, (int)(b * t), false);
}

int32_t ugb_grouped_attend(ugb_device *dev, const ugb_slice *q, const ugb_slice *k, const ugb_slice *v, const ugb_slice *pos, ugb_slice *out, size_t b,
                           size_t t, size_t heads, size_t kv_heads, size_t dq, size_t dv, size_t t_max, float scale, float out_scale, int32_t n_slices) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, q, out, "grouped_attend")) return rc;
  UGB_REQUIRE(dev, kv_heads > 0 && heads > 0 && heads % kv_heads == 0 && dq % 8 == 0 && dv % 8 == 0 && dq > 0 && dv > 0 && dq <= 4096 && dv <= 4096 && heads <= 65535 &&
                       b * t <= 65535 && t_max <= (1u << 30), UGB_ERR_SHAPE, "grouped_attend: unsupported shape");
  UGB_REQUIRE(dev, n_slices >= 1 && n_slices <= UGB_GROUPED_MAX_SPLITS, UGB_ERR_INVALID, "grouped_attend: %d slices", n_slices);
  UGB_SLICE(dev, q, q->dtype, b * t * heads * dq);
  UGB_SLICE(dev, out, q->dtype, b * t * heads * dv);
  UGB_SLICE(dev, k, q->dtype, b * kv_heads * t_max * dq);
  UGB_SLICE(dev, v, q->dtype, b * kv_heads * t_max * dv);
  UGB_SLICE(dev, pos, UGB_I32, 1);
  if (b == 0 || t == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  if (int32_t rc = ugb_grouped_attention_prepare(dev)) return rc;
  ugb_grouped_attention_args a{};
  a.f32 = q->dtype == UGB_F32; a.q = q->ptr; a.k = k->ptr; a.v = v->ptr; a.out = out->ptr; a.out_ld = heads * dv; a.out_scale = out_scale;
  a.rows = (int)(b * t); a.t = (int)t; a.pos_p = (const int *)pos->ptr; a.heads = (int)heads; a.kv_heads = (int)kv_heads; a.dq = (int)dq; a.dv = (int)dv;
  a.t_max = (int)t_max; a.scale = scale; a.splits = n_slices;
  return ugb_grouped_attention(dev, a);
}

int32_t ugb_grouped_attend_block(ugb_device *dev, const ugb_slice *q, const ugb_slice *k, const ugb_slice *v, ugb_slice *out, size_t b, size_t t,
                                 size_t pos0, size_t heads, size_t kv_heads, size_t dq, size_t dv, size_t t_max, float scale, float out_scale) {
  if (!dev) return UGB_ERR_INVALID;
  UGB_REQUIRE(dev, kv_heads > 0 && heads > 0 && heads % kv_heads == 0 && b <= 65535 && heads <= 65535 && pos0 + t <= t_max && t_max <= (1u << 30) &&
                       ((t + 127) / 128) * heads * b <= (size_t)INT32_MAX, UGB_ERR_SHAPE, "grouped_attend_block: unsupported shape");
  UGB_REQUIRE(dev, scale > 0.f, UGB_ERR_UNSUPPORTED, "grouped_attend_block: the scale must be positive");
  UGB_SLICE(dev, q, UGB_BF16, b * t * heads * dq);
  UGB_SLICE(dev, k, UGB_BF16, b * kv_heads * t_max * dq);
  UGB_SLICE(dev, v, UGB_BF16, b * kv_heads * t_max * dv);
  UGB_SLICE(dev, out, UGB_BF16, b * t * heads * dv);
  if (b == 0 || t == 0) return UGB_OK;
  UGB_REQUIRE(dev, (((uintptr_t)q->ptr | (uintptr_t)k->ptr | (uintptr_t)v->ptr | (uintptr_t)out->ptr) & 15) == 0, UGB_ERR_UNSUPPORTED,
              "grouped_attend_block: buffers must be 16-byte aligned");
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  ugb_prefill_attention_args a;
  a.q = (const __nv_bfloat16 *)q->ptr; a.k = (const __nv_bfloat16 *)k->ptr; a.v = (const __nv_bfloat16 *)v->ptr; a.out = (__nv_bfloat16 *)out->ptr;
  a.batch = (int)b; a.t = (int)t; a.pos0 = (int)pos0; a.n_heads = (int)heads; a.n_kv = (int)kv_heads; a.kv_rows = (int)t_max; a.dq = (int)dq; a.dv = (int)dv;
  a.scale = scale; a.out_scale = out_scale;
  return ugb_prefill_attention_tc(dev, a);
}

// the op's decay: A = -exp(A_log) in stream-ordered scratch
static int32_t with_decay(ugb_device *dev, const ugb_slice *a_log, size_t channels, size_t states, bool f32, ugb_scan_args &a, float **scratch) {
  a.shape = ugb_scan_shape_of((int)std::min<size_t>(states, 4096));
  UGB_REQUIRE(dev, a.shape.lanes > 0 && (size_t)a.shape.np == states, UGB_ERR_UNSUPPORTED, "selective scan: %zu states per channel", states);
  UGB_SLICE(dev, a_log, UGB_F32, channels * states);
  void *p = nullptr;
  UGB_CUDA(dev, ugb_malloc_async(dev, &p, channels * states * 4));
  *scratch = (float *)p;
  decay_kernel<<<(unsigned)((channels * states + 255) / 256), 256, 0, dev->stream>>>((const float *)a_log->ptr, *scratch, (int)channels, (int)states, (int)states, ugb_scan_decay_unit(f32));
  a.a = *scratch;
  return ugb_after_launch(dev, "decay_kernel");
}

int32_t ugb_selective_scan(ugb_device *dev, const ugb_slice *x, const ugb_slice *dt, const ugb_slice *bc, const ugb_slice *z, const ugb_slice *a_log,
                           const ugb_slice *skip, const ugb_slice *dt_bias, ugb_slice *state, ugb_slice *out, size_t b, size_t t, size_t channels,
                           size_t states, float scale) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, x, out, "selective_scan")) return rc;
  UGB_REQUIRE(dev, channels % 8 == 0 && channels > 0 && b <= 65535 && b * t * channels < (1ull << 31) && channels * states < (1ull << 31), UGB_ERR_SHAPE, "selective_scan: unsupported shape");
  UGB_SLICE(dev, x, x->dtype, b * t * channels);
  UGB_SLICE(dev, dt, x->dtype, b * t * channels);
  UGB_SLICE(dev, z, x->dtype, b * t * channels);
  UGB_SLICE(dev, bc, x->dtype, b * t * 2 * states);
  UGB_SLICE(dev, out, x->dtype, b * t * channels);
  UGB_SLICE(dev, skip, UGB_F32, channels);
  UGB_SLICE(dev, dt_bias, UGB_F32, channels);
  UGB_SLICE(dev, state, UGB_F32, b * channels * states);
  if (b == 0 || t == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  ugb_scan_args a{};
  float *scratch = nullptr;
  int32_t rc = with_decay(dev, a_log, channels, states, x->dtype == UGB_F32, a, &scratch);
  if (!rc) {
    a.f32 = x->dtype == UGB_F32; a.channels = (int)channels; a.u = x->ptr; a.skip = (const float *)skip->ptr; a.dt_bias = (const float *)dt_bias->ptr;
    a.state = (float *)state->ptr; a.out = out->ptr; a.out_ld = channels; a.scale = scale; a.xr = 2 * (int)states; a.rp = 0;
    rc = ugb_scan_block(dev, a, dt->ptr, bc->ptr, z->ptr, channels, (int)b, (int)t);
  }
  if (scratch) cudaFreeAsync(scratch, dev->stream);
  return rc;
}

int32_t ugb_selective_step(ugb_device *dev, const ugb_slice *x, const ugb_slice *low_bc, const ugb_slice *w_dt, const ugb_slice *z, const ugb_slice *a_log,
                           const ugb_slice *skip, const ugb_slice *dt_bias, ugb_slice *state, ugb_slice *out, size_t rows, size_t channels, size_t rank,
                           size_t states, float scale) {
  if (!dev) return UGB_ERR_INVALID;
  if (int32_t rc = act_dtype(dev, x, out, "selective_step")) return rc;
  if (int32_t rc = act_dtype(dev, x, w_dt, "selective_step")) return rc;
  UGB_REQUIRE(dev, channels % 8 == 0 && channels > 0 && rank % 8 == 0 && rank > 0 && rank <= 4096 && rows <= 65535 && rows * channels * states < (1ull << 31), UGB_ERR_SHAPE,
              "selective_step: unsupported shape");
  UGB_SLICE(dev, x, x->dtype, rows * channels);
  UGB_SLICE(dev, out, x->dtype, rows * channels);
  UGB_SLICE(dev, w_dt, x->dtype, rank * channels);
  UGB_SLICE(dev, low_bc, UGB_F32, rows * (rank + 2 * states));
  UGB_SLICE(dev, z, UGB_F32, rows * channels);
  UGB_SLICE(dev, skip, UGB_F32, channels);
  UGB_SLICE(dev, dt_bias, UGB_F32, channels);
  UGB_SLICE(dev, state, UGB_F32, rows * channels * states);
  if (rows == 0) return UGB_OK;
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  ugb_scan_args a{};
  float *scratch = nullptr;
  int32_t rc = with_decay(dev, a_log, channels, states, x->dtype == UGB_F32, a, &scratch);
  if (!rc) {
    a.f32 = x->dtype == UGB_F32; a.channels = (int)channels; a.u = x->ptr; a.skip = (const float *)skip->ptr; a.dt_bias = (const float *)dt_bias->ptr;
    a.state = (float *)state->ptr; a.out = out->ptr; a.out_ld = channels; a.scale = scale; a.rp = (int)rank; a.xr = (int)(rank + 2 * states);
    rc = ugb_scan_step(dev, a, w_dt->ptr, {(const float *)low_bc->ptr, 1, 0, (size_t)a.xr}, {(const float *)z->ptr, 1, 0, channels}, (int)rows, false, false);
  }
  if (scratch) cudaFreeAsync(scratch, dev->stream);
  return rc;
}

}  // extern "C"
