// Arguments of attention over a paged cache with a sliding window, kept first tokens and a linear distance bias
// (fmha_window.cu for prompts, fmha_decode_split.cu for single tokens), mirrored by a ctypes structure in
// ops/window_attention.py.
//
// One layer's cache is [num_blocks, block_elems]; a block holds 64 tokens as K [Hkv, 64, dk] then V [Hkv, 64, dv].
// Query position i sees key position j when j <= i and (window == 0 or i - j < window or j < keep_first);
// score = q . k * scale - slope_h * (i - j), slope_h = 2^(-bias_exp (h + 1) / Hq) (bias_exp == 0: no bias).
#pragma once

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
};
// kPaged: as described above.  kPackedRows (prompts): `cache` is [num_blocks, block_elems], one row per KEY, keys of all
// heads before values, and a tile's slot is the row of its sequence's first key.  kLatent (general kernel): keys and
// values are the same dk-wide rows, [num_blocks, 64, dk].
enum { kPaged = 0, kPackedRows = 1, kLatent = 2 };
static_assert(sizeof(WinParams) == 168, "WinParams is mirrored from Python");

}  // namespace sb
