// The key tiles that a block of queries with a sliding window, kept first keys and pooled blocks reads.
#pragma once

#include "common.cuh"

// Which key tiles of a query block are read: tiles 0 .. pooled - 1 of the pooled blocks, then [0, kept) and [from, end) of the
// tokens, walked as one list of `count`.
struct ZbTileList {
  int kept, from, count, pooled;
  ZB_DEVICE bool is_pooled(int i) const { return i < pooled; }
  ZB_DEVICE int at(int i) const {
    if (i < pooled) return i;
    i -= pooled;
    return i < kept ? i : from + i - kept;
  }
};
ZB_DEVICE ZbTileList zb_visible_tiles(int first_key, int keep, int end_tile, int tile_keys, int pooled_blocks = 0) {
  ZbTileList l;
  l.from = first_key / tile_keys;
  l.kept = min((keep + tile_keys - 1) / tile_keys, l.from);
  l.pooled = (pooled_blocks + tile_keys - 1) / tile_keys;
  l.count = l.pooled + l.kept + end_tile - l.from;
  return l;
}

// Pooled blocks that position `pos` sees: those that lie wholly in front of its window.
ZB_DEVICE int zb_pooled_visible(int pos, int window, int pool) {
  const int left = pos - window + 1;
  return left > 0 ? left / pool : 0;
}

// Row of pooled block b: a page holds the blocks whose last position lies in it, `rows` at most.
ZB_DEVICE int zb_pool_page_index(int b, int pool, int page_size) { return (b * pool + pool - 1) / page_size; }
ZB_DEVICE long long zb_pool_row(int page, int page_index, int b, int pool, int page_size, int rows) {
  return static_cast<long long>(page) * rows + b - page_index * page_size / pool;
}
