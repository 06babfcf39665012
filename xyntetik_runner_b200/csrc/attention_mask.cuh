// What the attention kernels share beyond plain causal attention: which keys a query sees, and a bias by distance.
//
// Visible keys.  The query at position p sees key j if j <= p and (p - j < window or j < keep_first); window 0: no window.  A
// request's first keep_first keys stay visible from anywhere (and their pages stay held, csrc/host/page_cache.cpp).  A
// kernel that walks keys in tiles of T visits the tiles of the window, t_lo = lo / T .. t_hi, and ahead of them the tiles
// below t_lo that hold kept keys, in ascending order: xr_kept_tiles of them.  In those, rows behind the kept keys are
// masked (their page may be the kept keys' own, or not be held at all).
//
// Bias.  score = (q . k) * scale + b[head][min(p - j, bias_len - 1)]: a table per query head over distances, constant from
// its last entry on.  The kernels take it divided by the scale ([H][bias_len] float32), so that it is added to the raw
// product: a matrix instruction's accumulator starts there instead of at zero.
#pragma once

struct XrBias {
    const float* table;          // [H][len], already divided by the score scale; null: no bias
    int len;
};

__host__ __device__ __forceinline__ int xr_kept_tiles(int keep_first, int lo, int tile) {
    const int kept = (keep_first + tile - 1) / tile, first = lo / tile;
    return kept < first ? kept : first;
}
// the tile at place i of a walk whose window begins with tile t_lo
__device__ __forceinline__ int xr_walk_tile(int i, int kept_tiles, int t_lo) { return i < kept_tiles ? i : t_lo + i - kept_tiles; }
// lo: the first key of the query's window
__device__ __forceinline__ bool xr_sees(int key, int pos, int lo, int keep_first) { return key <= pos && (key >= lo || key < keep_first); }
// row: the head's row of the table (any memory); distances below zero belong to keys that are masked anyway
__device__ __forceinline__ float xr_bias_at(const float* row, int len, int distance) { return row[min(max(distance, 0), len - 1)]; }
