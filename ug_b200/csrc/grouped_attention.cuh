// Grouped-query attention over cached keys and values: H query heads share G key / value heads, query head h reads head
// h / (H / G).  Heads of any width; for decode steps and short blocks (longer ones: attention_tc.cuh) and for 32 bits.
#pragma once
#include <cuda_bf16.h>

#include "ugb_internal.h"

struct ugb_grouped_attention_args {
  bool f32;                  // T = f32, else bf16 with fp32 scores, softmax and sums
  const void *q;             // T [rows][heads][dq], rotated and normalised
  const void *k, *v;         // T [b][kv_heads][t_max][dq / dv]; rows behind the newest position hold finite values
  void *out;                 // T [rows], out_ld apart: [heads][dv] times out_scale
  size_t out_ld;
  float out_scale;
  int rows, t;               // row r = (sequence r / t, position *pos_p + pos_off + r % t)
  const int *pos_p;          // device
  int pos_off;
  int heads, kv_heads, dq, dv, t_max;
  float scale;
  int splits;                // slices of the cached positions per row that run as separate CTAs (bf16 fast path)
  bool pdl;
  bool early;                // with pdl: q and the cache were written by kernels before the predecessor of this one
};

constexpr int UGB_GROUPED_MAX_SPLITS = 8;    // CTAs of a cluster
// Slices that fill `sms` SMs.
int ugb_grouped_attention_splits(const ugb_grouped_attention_args &a, int sms);
// Sets the kernels' shared-memory attributes (must not happen inside a stream capture).
int32_t ugb_grouped_attention_prepare(ugb_device *dev);
int32_t ugb_grouped_attention(ugb_device *dev, const ugb_grouped_attention_args &a);
