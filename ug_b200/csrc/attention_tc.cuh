// Interface of the tcgen05 / TMEM causal prefill attention translation unit.
#pragma once
#include <cuda_bf16.h>

#include "ugb_internal.h"

// out[b, i, head, :] = out_scale gate softmax_j(scale * q[b, i, head, :] . k[b, kvh, j, :]) v[b, kvh, j, :] over the cached
// positions j <= pos0 + i, for i in [0, t).  All base pointers 16-byte aligned.
struct ugb_prefill_attention_args {
  const __nv_bfloat16 *q;          // [batch, t, n_heads, dq]
  const __nv_bfloat16 *k, *v;      // [batch, n_kv, kv_rows, dq / dv], or token_major: [batch, kv_rows, n_kv, dq / dv]
  __nv_bfloat16 *out;              // [batch, t, n_heads * dv]
  int batch, t, pos0, n_heads, n_kv;
  int kv_rows;                     // positions the k / v buffers hold per sequence (>= pos0 + t)
  int token_major = 0;
  int dq = 64, dv = 64;            // 64 or 128 each
  float scale;
  const float *gate = nullptr;     // f32 [batch * t][gate_ld]: factor per query and head
  int gate_ld = 0;
  long long out_ld = 0;            // output elements between positions (a multiple of 8), 0 = n_heads * dv
  float out_scale = 1.0f;          // factor of every output
  int dynamic = 1;                 // the persistent CTAs draw their work items from the device's counter (longest
                                   // first); 0: the items are dealt round-robin
};
// Padded head width the kernel wants for `dim` values per head, 0 when it has none.
int ugb_prefill_attention_width(int dim);
int32_t ugb_prefill_attention_tc(ugb_device *dev, const ugb_prefill_attention_args &a);
