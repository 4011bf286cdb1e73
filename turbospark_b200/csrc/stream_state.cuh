// What a stream keeps of its last rows, and how the rows of a pass are cut into tiles.
#pragma once
#include "attention_window.cuh"

// A per-position quantity of every stream: [stream][ring_rows][width] f32, position p in slot p & (ring_rows - 1), ring_rows a power
// of two.  A row needs the `keep` rows before it.  A pass whose portions overwrite rows that its first rows need reads them from
// `before` instead: [stream][keep][width], entry i is the row of position base - keep + i.
struct RowRing {
    float *ring = nullptr, *before = nullptr;
    int width = 0, ring_rows = 0, keep = 0, n_streams = 0;
};

// Tiles of consecutive rows of one stream: listed on the device, or (tiles null) per_tile rows each of portions that all have
// rows_per_seq rows.
struct RowTiles {
    const AttnTile* tiles = nullptr;
    int n = 0, rows_per_seq = 1, per_tile = 1, tiles_per_seq = 1;
    int longest = 0;  // rows of the longest tile
    static RowTiles uniform(int rows, int rows_per_seq, int per_tile) {
        RowTiles t;
        t.rows_per_seq = rows_per_seq, t.per_tile = per_tile, t.tiles_per_seq = (rows_per_seq + per_tile - 1) / per_tile;
        t.n = rows / rows_per_seq * t.tiles_per_seq, t.longest = per_tile < rows_per_seq ? per_tile : rows_per_seq;
        return t;
    }
    static RowTiles list(const AttnTile* dev, int n) {
        RowTiles t;
        t.tiles = dev, t.n = n;
        return t;
    }
};

#ifdef __CUDACC__
__device__ __forceinline__ AttnTile row_tile(const RowTiles& t, int i) {
    if (t.tiles) return t.tiles[i];
    const int in_seq = (i % t.tiles_per_seq) * t.per_tile;
    return AttnTile{(i / t.tiles_per_seq) * t.rows_per_seq + in_seq, min(t.per_tile, t.rows_per_seq - in_seq)};
}
// row of position `pos` of stream `seq` before a portion that starts at `base`
__device__ __forceinline__ const float* ring_row_before(const RowRing& r, int seq, int base, int pos, bool use_before) {
    return use_before ? r.before + ((int64_t)seq * r.keep + (pos - (base - r.keep))) * r.width
                      : r.ring + ((int64_t)seq * r.ring_rows + (pos & (r.ring_rows - 1))) * r.width;
}
__device__ __forceinline__ float* ring_row(const RowRing& r, int seq, int pos) {
    return r.ring + ((int64_t)seq * r.ring_rows + (pos & (r.ring_rows - 1))) * r.width;
}
// is row r of a pass among the last ring_rows of its portion?  (a stream's rows are consecutive, and it comes once per pass)
__device__ __forceinline__ bool ring_keeps(const RowRing& ring, const tsb_row_desc* rows, int n_rows, int r, int seq) {
    return r + ring.ring_rows >= n_rows || rows[r + ring.ring_rows].seq != seq;
}
#endif
