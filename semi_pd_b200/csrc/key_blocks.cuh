// Pooled key / value blocks beside a sliding window: block b of a request stands for its positions b size .. b size +
// size - 1 through one row (the mean of their cache rows) that the query at position i sees once the whole block lies
// before its window, b size + size - 1 <= i - window.  The rows live behind the token rows of the same pool: a cache
// whose slots come in runs of `run_len` (slot 0 unused, run q = slots 1 + q run_len ...) keeps per run the blocks that
// END in it, per_run = ceil(run_len / size) rows each, so the row of a block follows from the slot of its last token
// and a block comes and goes with its run.
// Kept first tokens beside a sliding window: positions 0 .. keep - 1 of a request stay visible when the window has moved
// past them.  Either kind of entry stands in front of the window's tokens in a query's list of keys.
#pragma once
#include <stdint.h>

namespace spd {

struct KeyBlocks {
  int size;      // tokens per block; 0: no blocks
  int run_len;   // slots per run of the cache
  int per_run;   // block rows per run
  int64_t base;  // first block row of the pool
  int keep;      // first tokens that stay visible (0: none; not together with blocks)
};

// entries in front of the window of the query at `pos`: the blocks it sees (they are 0 .. n - 1), or the kept tokens that
// the window no longer covers (positions 0 .. n - 1)
__device__ __forceinline__ int64_t key_blocks_seen(const KeyBlocks& kb, int64_t pos, int window) {
  const int64_t before = window > 0 ? pos - window + 1 : 0;  // tokens that lie before the window
  if (before <= 0) return 0;
  return kb.size > 0 ? before / kb.size : (before < kb.keep ? before : kb.keep);
}
// pool row of the block whose last token sits in `slot`
__device__ __forceinline__ int64_t key_block_row(const KeyBlocks& kb, int slot) {
  const int s = slot - 1, run = s / kb.run_len;
  return kb.base + (int64_t)run * kb.per_run + (s - run * kb.run_len) / kb.size;
}
// A query's keys in one list: its nb front entries, then its tokens from position j_lo on.  Pool row of entry e.
__device__ __forceinline__ int key_row(const KeyBlocks& kb, const int32_t* __restrict__ page, int64_t e, int64_t nb,
                                       int64_t j_lo) {
  if (e >= nb) return page[j_lo + e - nb];
  if (kb.size == 0) return page[e];
  return (int)key_block_row(kb, page[e * kb.size + kb.size - 1]);
}

// distance from the query at `pos` to entry e of its list of n_keys (blocks have none: their value is not used)
__device__ __forceinline__ int64_t key_distance(int64_t e, int64_t nb, int64_t pos, int64_t n_keys) {
  return e >= nb ? n_keys - 1 - e : pos - e;
}

// A bias per head and distance that joins the scores: table [heads, len] fp32, distances from len - 1 on share the last
// entry (table null: no bias).
struct DistanceBias {
  const float* table;
  int len;
};
__device__ __forceinline__ float distance_bias(const float* __restrict__ row, int len, int64_t dist) {
  return row[dist < len ? dist : len - 1];
}

}  // namespace spd
