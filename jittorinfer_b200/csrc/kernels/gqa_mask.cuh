// First key position a query at position p can see: a sliding window holds the last `window` positions (p itself included), a chunk
// the positions with the same p / chunk; 0 turns either off.  Non-decreasing in p.
#pragma once

__host__ __device__ __forceinline__ int gqa_first_key(int p, int window, int chunk) {
    int lo = 0;
    if (window > 0 && p - window + 1 > lo) lo = p - window + 1;
    if (chunk > 0 && p / chunk * chunk > lo) lo = p / chunk * chunk;
    return lo;
}

// Blocks of `pool` positions that a query at position p sees as one key each: blocks 0 .. n - 1, those that lie wholly before its window.
// Non-decreasing in p.
__host__ __device__ __forceinline__ int gqa_blocks_seen(int p, int window, int pool) {
    return pool > 0 && p - window + 1 >= pool ? (p - window + 1) / pool : 0;
}

// Gathered for a prompt, the pooled rows fill whole tiles of 128 rows (the last is padded with zeros), so that a window of whole tiles stays so.
__host__ __device__ __forceinline__ int gqa_pool_gathered(int blocks) { return (blocks + 127) / 128 * 128; }

// Row of pooled block b: the pooled blocks that end in a cache block go with it, `rows` places for each.
__device__ __forceinline__ long long gqa_pool_row(const int * block_table, int b, int pool, int rows, int block_size) {
    const int page = ((b + 1) * pool - 1) / block_size;
    return (long long) block_table[page] * rows + b - page * block_size / pool;
}
