// Which rows of a flat batch a thread block of a fixed-shape grid works on, found on the device: request s owns the tokens
// q_start[s] .. q_start[s + 1] - 1, every token `per_token` consecutive rows, and a request's rows are cut in tiles of
// `tile_rows` (the last one part empty).  Requests without tokens and padding (tok_seq < 0) have no tiles.
#pragma once
#include "common.cuh"

struct RowTile {
    int seq;   // the request's index in the step (-1: the grid has more blocks than there are tiles)
    int row0;  // the tile's first row in the flat batch
    int rows;
};

// Tile b, counted from the first request's first tile or (from_end) from the last one's last.  Called by one whole warp;
// the lanes look at 32 requests at a time, so that their loads are in flight together.
__device__ __forceinline__ RowTile find_row_tile(int b, bool from_end, const int* __restrict__ q_start, const int* __restrict__ tok_seq,
                                                 int S, int per_token, int tile_rows) {
    const int lane = threadIdx.x & 31;
    auto tiles_of = [&](int s, int& first) {
        if (s >= S) return 0;
        first = q_start[s];
        const int len = q_start[s + 1] - first;
        return len > 0 && tok_seq[first] >= 0 ? (len * per_token + tile_rows - 1) / tile_rows : 0;
    };
    if (from_end) {
        int total = 0, first = 0;
        for (int s0 = 0; s0 < S; s0 += 32) total += tiles_of(s0 + lane, first);
        for (int o = 16; o > 0; o >>= 1) total += __shfl_xor_sync(0xffffffffu, total, o);
        b = total - 1 - b;
    }
    RowTile out = {-1, 0, 0};
    if (b < 0) return out;
    for (int s0 = 0; s0 < S; s0 += 32) {
        int first = 0;
        const int s = s0 + lane, mine = tiles_of(s, first);
        int upto = mine;  // tiles of requests s0 .. s
        for (int o = 1; o < 32; o <<= 1) {
            const int other = __shfl_up_sync(0xffffffffu, upto, o);
            if (lane >= o) upto += other;
        }
        const unsigned here = __ballot_sync(0xffffffffu, b >= upto - mine && b < upto);
        if (here != 0) {  // (one lane at most)
            const int src = __ffs(here) - 1, at = b - (upto - mine);
            if (lane == src) {
                out.seq = tok_seq[first];
                out.row0 = first * per_token + tile_rows * at;
                out.rows = min(tile_rows, q_start[s + 1] * per_token - out.row0);
            }
            out.seq = __shfl_sync(0xffffffffu, out.seq, src);
            out.row0 = __shfl_sync(0xffffffffu, out.row0, src);
            out.rows = __shfl_sync(0xffffffffu, out.rows, src);
            return out;
        }
        b -= __shfl_sync(0xffffffffu, upto, 31);
    }
    return out;
}
