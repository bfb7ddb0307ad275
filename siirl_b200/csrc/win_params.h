// Arguments of attention over a paged cache with a sliding window, kept first tokens and a linear distance bias
// (fmha_window.cu for prompts, fmha_decode_split.cu for single tokens), mirrored by a ctypes structure in
// ops/window_attention.py.
//
// One layer's cache is [num_blocks, block_elems]; a block holds 64 tokens as K [Hkv, 64, dk] then V [Hkv, 64, dv].
// Query position i sees key position j when j <= i and (window == 0 or i - j < window or j < keep_first);
// score = q . k * scale - slope_h * (i - j), slope_h = 2^(-bias_exp (h + 1) / Hq) (bias_exp == 0: no bias), or with a
// soft cap and / or a table of distances cap * tanh(q . k * scale / cap) + rel[h, min(i - j, rel_n - 1)].  With a sink the
// soft-max sum has one more term, of score 0 (or sink_w[h]) and without a value.
// pool = P > 0 (with a window): i also sees the whole runs of P tokens before its window, run b when (b + 1) P - 1 <= i -
// window, as one key and one value each, entry b at row b % 64 of cache block pool_table[slot, b / 64].
#pragma once
#include "common.cuh"

namespace sb {

struct WinParams {
  const void* x;            // projected rows [T, row_stride]: queries at q_off, keys at k_off, values at v_off
  long long row_stride;
  int q_off, k_off, v_off, T;
  const int* seq_ids;       // [T] cache slot of every row (-1: none)
  const int* positions;     // [T]
  const int* block_table;   // [slots, max_blocks]
  void* cache;
  long long num_blocks, block_elems;
  int max_blocks, Hq, Hkv, dk, dv, window, keep_first;
  float scale, bias_exp, out_scale;
  void* out;                // [T, out_stride], heads at column out_off
  long long out_stride;
  int out_off;
  int kv_mode;              // where keys and values are, see below
  const void* gain;         // one number that multiplies the queries and the gate, or null
  const void* gate;         // columns like out's: the result is multiplied by sigmoid(gain * gate) (prompts); null: none
  long long gate_stride;
  float softcap;            // 0: none
  int sink;
  const float* rel;         // [Hq, rel_n] bias by distance, or null (bias_exp must be 0 then)
  long long rel_n;
  const float* head_gate;   // [T, Hq]: the result is multiplied by it, or null
  int pool, pool_blocks;    // 0: none; columns of pool_table
  const int* pool_table;    // [slots, pool_blocks]
  const void* sink_w;       // [Hq] scores of the sink in the activation format, or null
};
// kPaged: as described above.  kPackedRows (prompts): `cache` is [num_blocks, block_elems], one row per KEY, keys of all
// heads before values, and a tile's slot is the row of its sequence's first key.  kLatent (general kernel): keys and
// values are the same dk-wide rows, [num_blocks, 64, dk].
enum { kPaged = 0, kPackedRows = 1, kLatent = 2 };
static_assert(sizeof(WinParams) == 224, "WinParams is mirrored from Python");

// pooled entries a query at position i sees
__host__ __device__ __forceinline__ int pooled_entries(int i, int window, int pool) {
  const int n = i - window + 1;      // tokens before the window
  return pool > 0 && n > 0 ? n / pool : 0;
}

// soft cap in units of log 2 of a raw product x: 2 * log2(e) * scale / cap * x is the exponent's argument
struct ScoreCap {
  float in, out;            // cap * tanh(scale * x / cap) * log2(e) = out - 2 out / (1 + 2^(in x))
  __device__ __forceinline__ ScoreCap(float cap, float scale)
      : in(2.f * 1.4426950408889634f * scale / cap), out(cap * 1.4426950408889634f) {}
  __device__ __forceinline__ float operator()(float x) const {
    return fmaf(-2.f * out, fast_rcp(1.f + fast_exp2(in * x)), out);
  }
};

}  // namespace sb
