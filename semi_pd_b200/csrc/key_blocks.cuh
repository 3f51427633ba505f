// Pooled key / value blocks beside a sliding window: block b of a request stands for its positions b size .. b size +
// size - 1 through one row (the mean of their cache rows) that the query at position i sees once the whole block lies
// before its window, b size + size - 1 <= i - window.  The rows live behind the token rows of the same pool: a cache
// whose slots come in runs of `run_len` (slot 0 unused, run q = slots 1 + q run_len ...) keeps per run the blocks that
// END in it, per_run = ceil(run_len / size) rows each, so the row of a block follows from the slot of its last token
// and a block comes and goes with its run.
#pragma once
#include <stdint.h>

namespace spd {

struct KeyBlocks {
  int size;      // tokens per block; 0: no blocks
  int run_len;   // slots per run of the cache
  int per_run;   // block rows per run
  int64_t base;  // first block row of the pool
};

// blocks the query at `pos` sees (they are 0 .. n - 1)
__device__ __forceinline__ int64_t key_blocks_seen(const KeyBlocks& kb, int64_t pos, int window) {
  const int64_t before = pos - window + 1;  // tokens that lie before the window
  return kb.size > 0 && before > 0 ? before / kb.size : 0;
}
// pool row of the block whose last token sits in `slot`
__device__ __forceinline__ int64_t key_block_row(const KeyBlocks& kb, int slot) {
  const int s = slot - 1, run = s / kb.run_len;
  return kb.base + (int64_t)run * kb.per_run + (s - run * kb.run_len) / kb.size;
}
// A query's keys in one list: its nb blocks, then its tokens from position j_lo on.  Pool row of entry e.
__device__ __forceinline__ int key_row(const KeyBlocks& kb, const int32_t* __restrict__ page, int64_t e, int64_t nb,
                                       int64_t j_lo) {
  if (e >= nb) return page[j_lo + e - nb];
  return (int)key_block_row(kb, page[e * kb.size + kb.size - 1]);
}

}  // namespace spd
