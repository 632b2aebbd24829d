// First key position a query at position p can see: a sliding window holds the last `window` positions (p itself included), a chunk
// the positions with the same p / chunk; 0 turns either off.  Non-decreasing in p.
#pragma once

__host__ __device__ __forceinline__ int gqa_first_key(int p, int window, int chunk) {
    int lo = 0;
    if (window > 0 && p - window + 1 > lo) lo = p - window + 1;
    if (chunk > 0 && p / chunk * chunk > lo) lo = p / chunk * chunk;
    return lo;
}
