// A learned bias on an attention score that depends on the query's head and on how far the key lies behind the query:
// score <- score + table[h][min(distance, len - 1)], after the scale and the soft cap, before the mask.
// `table` [H, len] float32 is a parameter spread out over the distances (buckets of distances repeat their value), so
// that a kernel needs one index and no logarithm; every distance from len - 1 on has the last entry's value, so a block
// of keys that lies at least that far behind all its queries takes one constant.
#pragma once

struct DistBias {
    const float* table;          // null: no bias
    int len;
};

__device__ __forceinline__ const float* ri_bias_row(const DistBias& b, int h) { return b.table + (size_t)h * b.len; }
// (a key past the query, which the mask takes out anyway, reads the entry of distance 0)
__device__ __forceinline__ float ri_bias_at(const float* row, int len, int distance) {
    return __ldg(row + max(0, min(distance, len - 1)));
}
