// A learned bias on an attention score that depends on the query's head and on how far the key lies behind the query:
// score <- score + bias[h][min(distance, len - 1)], after the scale and the soft cap, before the mask.
// The parameter is spread out over the distances (buckets of distances repeat their value), so that a kernel needs one
// index and no logarithm; every distance from len - 1 on has the last entry's value, so a block of keys that lies at
// least that far behind all its queries takes one constant.  A head's row of the table is DIST_BIAS_PAD copies of the first
// entry, the len entries, and DIST_BIAS_PAD copies of the last one: inside a block of queries and keys of which at least
// one pair is nearer than the last entry no distance leaves the row, so the kernels index it without clamping.
#pragma once

#define DIST_BIAS_PAD 192       // a tile of 128 queries and a block of 64 keys: distances from -190 to len + 189

struct DistBias {
    const float* table;          // [H, DIST_BIAS_PAD + len + DIST_BIAS_PAD]; null: no bias
    int len;
};

__host__ __device__ __forceinline__ int ri_bias_pitch(int len) { return len + 2 * DIST_BIAS_PAD; }
// entry d of the returned row belongs to distance d, -DIST_BIAS_PAD <= d < len + DIST_BIAS_PAD
__device__ __forceinline__ const float* ri_bias_row(const DistBias& b, int h) { return b.table + (size_t)h * ri_bias_pitch(b.len) + DIST_BIAS_PAD; }
// any distance from 0 on
__device__ __forceinline__ float ri_bias_at(const float* row, int len, int distance) { return __ldg(row + min(distance, len - 1)); }
