// Shared part of the fused decoder engines, see engine_core.cuh.
#include "engine_core.cuh"

#include <algorithm>

namespace {

template <typename S, typename D>
__global__ void convert_rows_kernel(const S *__restrict__ s, D *__restrict__ d, size_t n, size_t row_len,
                                    size_t dst_pitch, size_t src_pitch) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    d[(i / row_len) * dst_pitch + i % row_len] = (D)(float)s[(i / row_len) * src_pitch + i % row_len];
}

}  // namespace

void engine_free(ugb_engine *m) {
  cudaSetDevice(m->dev->ordinal);
  cudaStreamSynchronize(m->dev->stream);
  engine_drop_graph(m);
  for (void *p : m->allocs) cudaFree(p);
  m->allocs.clear();
  if (m->pf_logits) cudaFree(m->pf_logits);
  m->pf_logits = nullptr;
}

int32_t engine_put_matrix(ugb_engine *m, const ugb_slice *w, void *dst, int32_t dst_dtype, size_t rows, size_t cols,
                          size_t row0, size_t nrows, size_t col0, size_t ncols, size_t dst_pitch, const char *name) {
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, w->len == rows * cols, UGB_ERR_SHAPE, "unexpected shape for %s: %zu elements, expected (%zu, %zu)",
              name, w->len, rows, cols);
  UGB_REQUIRE(dev, w->dtype == UGB_BF16 || w->dtype == UGB_F32, UGB_ERR_DTYPE, "%s: weights must be BF16 or F32", name);
  if (nrows * ncols == 0) return UGB_OK;
  const size_t off = row0 * cols + col0, es = ugb_dtype_size(w->dtype);
  if (w->dtype == dst_dtype) {
    UGB_CUDA(dev, cudaMemcpy2DAsync(dst, dst_pitch * es, (const char *)w->ptr + off * es, cols * es, ncols * es, nrows,
                                    cudaMemcpyDeviceToDevice, dev->stream));
    return UGB_OK;
  }
  const int grid = dev->sm_count * 8;
  if (w->dtype == UGB_F32)
    convert_rows_kernel<float, __nv_bfloat16><<<grid, 256, 0, dev->stream>>>((const float *)w->ptr + off, (__nv_bfloat16 *)dst,
                                                                             nrows * ncols, ncols, dst_pitch, cols);
  else
    convert_rows_kernel<__nv_bfloat16, float><<<grid, 256, 0, dev->stream>>>((const __nv_bfloat16 *)w->ptr + off, (float *)dst,
                                                                             nrows * ncols, ncols, dst_pitch, cols);
  return ugb_after_launch(dev, "convert_rows_kernel");
}

int32_t engine_reset(ugb_engine *m, int32_t pos) {
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, pos >= 0 && pos < m->t_max, UGB_ERR_INVALID, "reset position %d outside 0..%d", pos, m->t_max - 1);
  UGB_CUDA(dev, cudaMemcpyAsync(m->pos, &pos, 4, cudaMemcpyHostToDevice, dev->stream));
  UGB_CUDA(dev, cudaStreamSynchronize(dev->stream));
  m->host_pos = pos;
  return UGB_OK;
}

int32_t engine_decode(ugb_engine *m, const ugb_slice *tokens, int32_t n_steps) {
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, n_steps >= 1, UGB_ERR_INVALID, "n_steps must be >= 1");
  UGB_REQUIRE(dev, tokens == nullptr || n_steps == 1, UGB_ERR_INVALID, "explicit tokens feed exactly one step");
  UGB_REQUIRE(dev, m->host_pos + n_steps <= m->position_limit(), UGB_ERR_SHAPE,
              "decode of %d steps from position %d exceeds the cache (%d positions)", n_steps, m->host_pos, m->t_max);
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  int32_t rc;
  if ((rc = m->before_step())) return rc;
  if (tokens) {
    UGB_SLICE(dev, tokens, UGB_I32, (size_t)m->batch);
    UGB_CUDA(dev, cudaMemcpyAsync(m->next, tokens->ptr, (size_t)m->batch * 4, cudaMemcpyDeviceToDevice, dev->stream));
  }
  for (int s = 0; s < n_steps; ++s) {
    if (!m->warmed) {
      // first step runs eagerly: it sets kernel attributes, which must not happen inside a capture
      if ((rc = m->enqueue_step(m->next))) return rc;
      m->warmed = true;
    } else {
      if (!m->graph) {
        cudaGraph_t g = nullptr;
        const uint64_t before = dev->launches;
        UGB_CUDA(dev, cudaStreamBeginCapture(dev->stream, cudaStreamCaptureModeThreadLocal));
        rc = m->enqueue_step(m->next);
        cudaError_t e = cudaStreamEndCapture(dev->stream, &g);
        m->graph_nodes = (int)(dev->launches - before);
        dev->launches = before;
        if (rc) { if (g) cudaGraphDestroy(g); return rc; }
        if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "stream capture failed: %s", cudaGetErrorString(e));
        e = cudaGraphInstantiate(&m->graph, g, 0);
        cudaGraphDestroy(g);
        if (e != cudaSuccess) return ugb_fail(dev, UGB_ERR_CUDA, "cudaGraphInstantiate failed: %s", cudaGetErrorString(e));
      }
      UGB_CUDA(dev, cudaGraphLaunch(m->graph, dev->stream));
      dev->launches += (uint64_t)m->graph_nodes;
    }
    m->host_pos++;
  }
  return UGB_OK;
}

int32_t engine_prefill(ugb_engine *m, const ugb_slice *tokens, int32_t t, int32_t all_logits) {
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, t >= 1, UGB_ERR_INVALID, "prefill of %d positions", t);
  UGB_REQUIRE(dev, tokens != nullptr, UGB_ERR_INVALID, "prefill: null tokens");
  UGB_SLICE(dev, tokens, UGB_I32, (size_t)m->batch * t);
  UGB_REQUIRE(dev, m->host_pos + t <= m->position_limit(), UGB_ERR_SHAPE,
              "prefill of %d positions from position %d exceeds the cache (%d positions)", t, m->host_pos, m->t_max);
  UGB_CUDA(dev, cudaSetDevice(dev->ordinal));
  int32_t rc;
  if ((rc = m->before_prefill())) return rc;
  if ((rc = m->ensure_prefill_workspace())) return rc;
  if (all_logits) {
    const size_t need = (size_t)m->batch * t * m->logits_ld;
    if (need > m->pf_logits_cap) {
      UGB_CUDA(dev, cudaStreamSynchronize(dev->stream));
      if (m->pf_logits) { cudaFree(m->pf_logits); m->pf_logits = nullptr; m->pf_logits_cap = 0; }
      void *v = nullptr;
      UGB_CUDA(dev, cudaMalloc(&v, need * sizeof(float)));
      m->pf_logits = (float *)v;
      m->pf_logits_cap = need;
    }
    m->pf_logits_t = t;
  }
  const int *tok = (const int *)tokens->ptr;
  int tc = 0;
  for (int c0 = 0; c0 < t; c0 += tc) {
    tc = std::min(m->pf_chunk, t - c0);
    if ((rc = m->enqueue_prefill_chunk(tok, t, c0, tc, all_logits != 0))) return rc;
  }
  // last position of every sequence: final norm, output head, greedy choice
  if ((rc = m->enqueue_prefill_tail(tc))) return rc;
  const int last = m->host_pos + t - 1;     // the argmax kernel advances the device-side position by one
  UGB_CUDA(dev, cudaMemcpyAsync(m->pos, &last, 4, cudaMemcpyHostToDevice, dev->stream));
  if ((rc = m->enqueue_head(false))) return rc;
  m->host_pos += t;
  return UGB_OK;
}

int32_t engine_read_rows(ugb_engine *m, const void *src, size_t rows, size_t cols, size_t src_ld, void *host_dst, size_t len) {
  ugb_device *dev = m->dev;
  UGB_REQUIRE(dev, len == rows * cols, UGB_ERR_SHAPE, "read: destination holds %zu elements, %zu expected", len, rows * cols);
  if (len == 0) return UGB_OK;
  if (src_ld == cols) UGB_CUDA(dev, cudaMemcpyAsync(host_dst, src, len * 4, cudaMemcpyDeviceToHost, dev->stream));
  else UGB_CUDA(dev, cudaMemcpy2DAsync(host_dst, cols * 4, src, src_ld * 4, cols * 4, rows, cudaMemcpyDeviceToHost, dev->stream));
  UGB_CUDA(dev, cudaStreamSynchronize(dev->stream));
  return UGB_OK;
}
