// State of a decoder described by a list of layers, shared by the two forms a layer can have: hybrid_engine.cu (weights,
// options, the sandwich form) and hybrid_parallel.cu (the parallel form).
#pragma once
#include <vector>

#include "engine_core.cuh"
#include "hybrid_kernels.cuh"

// Weights of one layer.
struct ugb_hybrid_weights {
  ugb_hybrid_layer d{};
  float *norm1 = nullptr;
  // sandwich form
  int ul = 0, fl = 0;                         // padded recurrent channels, feed-forward columns
  int ql = 0, cl = 0, gl = 0;                 // latent attention: query latent, cache row, gates
  bool expand = false;                        // blocks may run on the tcgen05 attention kernel
  float *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *conv1 = nullptr, *conv2 = nullptr, *dwa = nullptr;
  void *w_in = nullptr, *w_out = nullptr;     // input projections of the layer side by side, output projections
  float *bz = nullptr, *bu = nullptr;
  float *q_gain = nullptr, *c_gain = nullptr;
  void *w_uq = nullptr, *w_uk = nullptr, *w_uv = nullptr;
  void *w_up = nullptr, *w_down = nullptr;    // parallel form: w_up holds (gate, up) row pairs
  int dp = 0, vp = 0;                         // padded widths of an attention head's queries / keys and values
  // parallel form: w_in rows are q | k | v | x | z | router, w_out columns attention | scan | feed-forward
  int nq = 0, nk = 0, nv = 0;                 // columns of all heads
  int ci = 0, np = 0, rp = 0;                 // scan channels, states per channel, step-size rank
  int ep = 0, ef = 0;                         // router columns, columns of an expert
  int lanes = 0, per_lane = 0;                // of the scan kernels: lanes per channel x states per lane = np
  int rot = -1;                               // index into ugb_hybrid::rot
  float *conv_w = nullptr, *conv_b = nullptr, *a = nullptr, *skip = nullptr, *dt_b = nullptr;
  void *w_x = nullptr, *w_dt = nullptr;       // W_dt transposed: [rp][ci]
  void *x_up = nullptr, *x_down = nullptr;    // experts: [experts][2 ef][width] in (gate, up) row pairs, [experts][width][ef]
  void *side_gate = nullptr, *side_proj = nullptr;
  float *side_gain = nullptr;
  int n_heads_in() const { return nq + nk + nv; }
  int n_in() const { return nq + nk + nv + 2 * ci; }       // without the router
  int n_cat() const { return d.heads * vp + ci + fl; }     // inputs of the output projection
};

// One pass over a layer: a layer inside a loop is run several times, each time with its own state.
struct ugb_hybrid_run {
  int layer = 0, enter = -1;                  // enter: number of the pass that begins here, -1 = none
  size_t tail[2] = {0, 0};                    // byte offsets of the convolution tails in ugb_hybrid::tails
  float *state = nullptr;                     // recurrent state [batch][channels (x states)]
  size_t state_len = 0;                       // of all sequences
  void *cache = nullptr, *vcache = nullptr;   // latents [batch][t_max][cl], or keys and values [batch][kv_heads][t_max][dp / vp]
};

// Activations of up to `rows` rows.
struct ugb_hybrid_work {
  int rows = 0;
  float *x = nullptr, *bank = nullptr, *gate = nullptr;
  float *pre = nullptr;                                    // projections: f32 partials in a step, T in a block
  void *h = nullptr, *hc = nullptr, *mid = nullptr;        // norm output, convolved, mixer / feed-forward inner
  void *cq = nullptr, *q = nullptr, *ql = nullptr, *ol = nullptr, *o = nullptr;
  // parallel form
  float *prod = nullptr;                                   // products that go to the residual stream
  void *cat = nullptr;                                     // inputs of the output projection, side by side
  void *xs = nullptr, *xx = nullptr;                       // the stream in T; stream | embedding output for a loop's input
  void *xdb = nullptr, *dt = nullptr;                      // step-size latent | B | C; step sizes before their bias
  float *gu = nullptr;                                     // f32 model: (gate, up) products
  float *side = nullptr, *part = nullptr;                  // part: narrow products of a block, before they are summed
  void *side_h = nullptr;
  // mixture of experts: token rows grouped by expert in tiles of `tile` rows
  int tile = 0, tiles = 0;
  float *xout = nullptr;
  void *xin = nullptr, *xmid = nullptr;
  int *count = nullptr, *map = nullptr, *slot = nullptr;   // rows per expert, expert of a tile, row of (token, choice)
  float4 *choice = nullptr;                                // {expert, place, weight}
};

struct ugb_hybrid_mat {            // out[b, m, n] = a . w
  void *out; const void *a, *w;
  size_t m, n, k, batch = 1, a_ld = 0, a_batch = 0, w_batch = 0, c_ld = 0, c_batch = 0;
  bool nk = true;
  bool f32_out = true;             // f32 result (split over k when splits > 1), else T
  bool relu2 = false;
  bool silu_mul = false;           // columns are (gate, up) pairs; T result of n / 2 columns
  const int *groups = nullptr;     // rows in tiles of `tile`, tile i against weights groups[i]
  int tile = 0, n_groups = 0;
  int splits = 1, bn = 0;
};

struct ugb_hybrid_tiling { int bn, splits; };

struct ugb_hybrid : ugb_engine {
  ugb_hybrid_config cfg{};
  std::vector<ugb_hybrid_weights> layers;
  std::vector<ugb_hybrid_run> runs;
  bool f32 = false;
  int wl = 0;                      // padded width
  void *embed = nullptr, *head = nullptr;
  float *embed_gain = nullptr, *final_gain = nullptr;
  unsigned char *tails = nullptr, *tails_next = nullptr;   // a block writes the second
  size_t tail_bytes = 0;
  ugb_hybrid_work dec, pf;
  void *kx = nullptr, *vx = nullptr;                       // expanded keys / values of one layer
  int att_splits_opt = 0, absorb_max = 16, keep_layers = 0;
  float *layer_out = nullptr;
  size_t layer_cap = 0;
  int layer_rows = 0;
  int only = UGB_HYBRID_K_ALL;     // measurement aid: the kernel kind that is launched
  // parallel form
  struct Rotation { float base; int dims; float *cos_, *sin_; };
  std::vector<Rotation> rot;       // [t_max][dims / 2] tables, one per (base, dims)
  void *loop_in = nullptr, *side_embed = nullptr;
  float *loop_step = nullptr;
  int sl = 0;                      // padded columns of the token input

  bool parallel() const { return cfg.form == UGB_FORM_PARALLEL; }
  size_t es() const { return f32 ? 4 : 2; }
  bool on(int kind) const { return only == UGB_HYBRID_K_ALL || only == kind; }
  int att_splits() const;
  int32_t enqueue_step(const int *tok) override;
  int32_t ensure_prefill_workspace() override;
  int32_t enqueue_prefill_chunk(const int *tok, int t, int c0, int tc, bool all_logits) override;
  int32_t enqueue_prefill_tail(int tc) override;
  int32_t enqueue_head(bool after_step) override;
};

inline size_t ugb_up8(size_t n) { return (n + 7) / 8 * 8; }
constexpr int UGB_HYBRID_MAX_SPLITS = 8;

int32_t ugb_hybrid_alloc(ugb_hybrid *m, void **p, size_t bytes, bool zero);
int32_t ugb_hybrid_matmul(ugb_hybrid *m, const ugb_hybrid_mat &x);
// k splits of a decode product with a f32 result
ugb_hybrid_tiling ugb_hybrid_tile(const ugb_hybrid *m, size_t n, size_t k);
template <typename T> int32_t ugb_hybrid_rows(ugb_hybrid *m, ugb_hybrid_k::RowArgs<T> &a, int rows, bool early);
extern template int32_t ugb_hybrid_rows<float>(ugb_hybrid *, ugb_hybrid_k::RowArgs<float> &, int, bool);
extern template int32_t ugb_hybrid_rows<__nv_bfloat16>(ugb_hybrid *, ugb_hybrid_k::RowArgs<__nv_bfloat16> &, int, bool);
// The stream behind run `run` of a block's positions, kept for UGB_HYBRID_LAYERS.
int32_t ugb_hybrid_keep(ugb_hybrid *m, const ugb_hybrid_work &w, int run, int t_block, int off, int t);

// The tensor as f32 in stream-ordered scratch, handed to `use`.
template <typename F>
int32_t ugb_hybrid_f32(ugb_hybrid *m, const ugb_slice *w, size_t n, const char *name, F use) {
  ugb_device *dev = m->dev;
  void *tmp = nullptr;
  UGB_CUDA(dev, ugb_malloc_async(dev, &tmp, n * 4));
  int32_t rc = engine_put_matrix(m, w, tmp, UGB_F32, 1, n, 0, 1, 0, n, n, name);
  if (!rc) rc = use((const float *)tmp);
  cudaFreeAsync(tmp, dev->stream);
  return rc;
}
inline int32_t ugb_hybrid_gain(ugb_hybrid *m, const ugb_slice *w, float *dst, int n, float offset, const char *name) {
  return ugb_hybrid_f32(m, w, n, name, [&](const float *s) {
    ugb_hybrid_k::gain_kernel<<<(n + 255) / 256, 256, 0, m->dev->stream>>>(s, dst, n, offset);
    return ugb_after_launch(m->dev, "gain_kernel");
  });
}

// hybrid_parallel.cu: shapes, weights and state of layer / run i, activations, loading, and one pass over all runs for
// rows (b, i), i < t, positions *pos + off + i, which leaves the final norm's output in w.h.
int32_t ugb_parallel_layer(ugb_hybrid *m, int i);
int32_t ugb_parallel_model(ugb_hybrid *m);
int32_t ugb_parallel_work(ugb_hybrid *m, ugb_hybrid_work &w, int rows, bool decode);
int32_t ugb_parallel_load(ugb_hybrid *m, const char *name, const ugb_slice *w, bool *known);
int32_t ugb_parallel_run(ugb_hybrid *m, ugb_hybrid_work &w, const int *tok, int t_block, int off, int t, bool decode);
// Logits <- cap tanh(logits / cap), n (a multiple of 4) values.
int32_t ugb_parallel_softcap(ugb_hybrid *m, float *logits, size_t n);
