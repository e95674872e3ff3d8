// A step's tokens in chunks: every sequence's new tokens are cut into pieces of CHUNK_TOKENS, counted from its first new one.
#pragma once
#include "common.cuh"

#define CHUNK_TOKENS 64

// The tokens [t0, t0 + count) of chunk `c` of the step: false beyond the last one. Every warp looks at 32 sequences at once.
__device__ __forceinline__ bool chunk_of(const int* cu_seqlens, int B, int c, int& t0, int& count) {
    const int lane = threadIdx.x & 31;
    for (int b0 = 0; b0 < B; b0 += 32) {
        const int b = b0 + lane;
        const int lo = b < B ? __ldcg(cu_seqlens + b) : 0, len = b < B ? __ldcg(cu_seqlens + b + 1) - lo : 0;
        const int chunks = (len + CHUNK_TOKENS - 1) / CHUNK_TOKENS;
        int upto = chunks;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int p = __shfl_up_sync(0xffffffffu, upto, o);
            if (lane >= o) upto += p;
        }
        const unsigned after = __ballot_sync(0xffffffffu, c < upto);
        if (after != 0) {
            const int owner = __ffs(after) - 1;
            const int k = c - __shfl_sync(0xffffffffu, upto - chunks, owner);
            t0 = __shfl_sync(0xffffffffu, lo, owner) + k * CHUNK_TOKENS;
            count = min(CHUNK_TOKENS, __shfl_sync(0xffffffffu, len, owner) - k * CHUNK_TOKENS);
            return true;
        }
        c -= __shfl_sync(0xffffffffu, upto, 31);
    }
    return false;
}

// Chunks of the sequences before sequence b; every lane of the warp gets the sum.
__device__ __forceinline__ int chunks_before(const int* cu_seqlens, int b) {
    int first = 0;
    for (int i = threadIdx.x & 31; i < b; i += 32) first += (__ldcg(cu_seqlens + i + 1) - __ldcg(cu_seqlens + i) + CHUNK_TOKENS - 1) / CHUNK_TOKENS;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) first += __shfl_xor_sync(0xffffffffu, first, o);
    return first;
}
