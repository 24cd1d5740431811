// What every fused decoder engine of this library shares, whatever its layers are: the device-side token / position
// state of a batch of sequences, weight upload, the greedy step loop with its CUDA graph, and the chunked prompt
// loop.  llama_engine.cu and hybrid_engine.cu derive from it and supply the layers.
#pragma once
#include <cuda_bf16.h>

#include <cstddef>
#include <vector>

#include "ugb_internal.h"

struct ugb_engine {
  ugb_device *dev = nullptr;
  int batch = 0, t_max = 0;       // sequences and cached positions per sequence
  int *next = nullptr, *pos = nullptr;   // device: input token of the next step per sequence, shared position
  int host_pos = 0;
  float *logits = nullptr;        // [batch, logits_ld], the first `vl` columns are vocabulary entries
  int vl = 0, logits_ld = 0;
  int pdl = 1;                    // programmatic dependent launch between the kernels of a step
  // graph of one step that reads `next` as its input tokens
  cudaGraphExec_t graph = nullptr;
  int graph_nodes = 0;
  bool warmed = false;
  std::vector<void *> allocs;
  size_t loaded = 0;
  // prompts are processed in chunks of pf_chunk positions of every sequence (pf_rows = batch * pf_chunk rows);
  // the workspace is allocated by the first prompt
  int pf_rows_max = 8192;         // option prefill_rows: upper bound on rows per chunk
  int pf_rows = 0, pf_chunk = 0;
  float *pf_logits = nullptr;     // [batch, pf_logits_t, logits_ld] when all-position logits were requested
  int pf_logits_t = 0;
  size_t pf_logits_cap = 0;

  virtual ~ugb_engine() {}
  virtual int position_limit() const { return t_max; }              // positions a sequence may reach
  virtual int32_t before_step() { return UGB_OK; }                  // refuses or prepares a decode call
  virtual int32_t before_prefill() { return UGB_OK; }
  // Enqueues one step of one position per sequence on the device stream: `tok` -> next, position + 1.
  virtual int32_t enqueue_step(const int *tok) = 0;
  virtual int32_t ensure_prefill_workspace() = 0;
  // Positions c0 .. c0 + tc - 1 of a block of t per sequence, cache positions host_pos + c0 onwards.
  virtual int32_t enqueue_prefill_chunk(const int *tok, int t, int c0, int tc, bool all_logits) = 0;
  // The last position of every sequence (row tc - 1 of the last chunk) -> normalised rows for the output head.
  virtual int32_t enqueue_prefill_tail(int tc) = 0;
  // Output head over those rows, greedy choice, device position + 1.
  virtual int32_t enqueue_head(bool after_step) = 0;
};

template <typename T>
int32_t dmalloc(ugb_engine *m, T **p, size_t n, bool zero = false) {
  ugb_device *dev = m->dev;
  void *v = nullptr;
  UGB_CUDA(dev, cudaMalloc(&v, n * sizeof(T) ? n * sizeof(T) : 16));
  if (zero) UGB_CUDA(dev, cudaMemsetAsync(v, 0, n * sizeof(T), dev->stream));
  m->allocs.push_back(v);
  *p = (T *)v;
  return UGB_OK;
}

// Any change of shapes, options or buffers that a captured step holds.
inline void engine_drop_graph(ugb_engine *m) {
  if (m->graph) { cudaGraphExecDestroy(m->graph); m->graph = nullptr; }
}
// Frees everything the engine owns on the device (the stream must be idle or is synchronised here).
void engine_free(ugb_engine *m);

// Copies rows [row0, row0 + nrows) x columns [col0, col0 + ncols) of a [rows, cols] matrix (BF16 or F32) into `dst`
// of type `dst_dtype` (BF16 or F32; f32 -> bf16 rounds to nearest even, bf16 -> f32 is exact) with a destination row
// pitch in elements.  The shape check is on the whole tensor.
int32_t engine_put_matrix(ugb_engine *m, const ugb_slice *w, void *dst, int32_t dst_dtype, size_t rows, size_t cols,
                          size_t row0, size_t nrows, size_t col0, size_t ncols, size_t dst_pitch, const char *name);

int32_t engine_reset(ugb_engine *m, int32_t pos);
int32_t engine_decode(ugb_engine *m, const ugb_slice *tokens, int32_t n_steps);
int32_t engine_prefill(ugb_engine *m, const ugb_slice *tokens, int32_t t, int32_t all_logits);
// Blocking host copy of `rows` x `cols` 4-byte elements with a source pitch in elements.
int32_t engine_read_rows(ugb_engine *m, const void *src, size_t rows, size_t cols, size_t src_ld, void *host_dst, size_t len);
