// The key tiles that a block of queries with a sliding window and kept first keys reads.
#pragma once

#include "common.cuh"

// Which key tiles of a query block are read: [0, kept) and [from, end), walked as one list of `count`.
struct ZbTileList {
  int kept, from, count;
  ZB_DEVICE int at(int i) const { return i < kept ? i : from + i - kept; }
};
ZB_DEVICE ZbTileList zb_visible_tiles(int first_key, int keep, int end_tile, int tile_keys) {
  ZbTileList l;
  l.from = first_key / tile_keys;
  l.kept = min((keep + tile_keys - 1) / tile_keys, l.from);
  l.count = l.kept + end_tile - l.from;
  return l;
}
