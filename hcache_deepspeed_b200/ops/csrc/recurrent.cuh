// Shared pieces of recurrences whose inputs are plain projections (minGRU, gated linear attention): chunks of a ragged batch.
#pragma once
#include "ssm.cuh"

namespace hds {

struct ChunkPlace {
    SsmSpan span;
    int seq, chunk;     // chunk inside its sequence
};

// Sequences with one token have no chunks (they are stepped).
__device__ __forceinline__ int span_chunks(const SsmSpan& s, int tokens) { return s.n > 1 ? (s.n + tokens - 1) / tokens : 0; }

// Which chunk is number `index` of the batch (counted over all sequences in order)? By warp 0; *place is shared memory, all threads
// of the block return its validity.
__device__ __forceinline__ bool find_chunk(const SsmSpan* spans, int n_seqs, int tokens, int index, ChunkPlace* place) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        int base = 0, seq = -1, chunk = 0;
        for (int s0 = 0; s0 < n_seqs && seq < 0; s0 += 32) {
            const int s = s0 + lane;
            const int mine = s < n_seqs ? span_chunks(spans[s], tokens) : 0;
            int incl = mine;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, incl, o);
                if (lane >= o) incl += up;
            }
            const unsigned hit = __ballot_sync(0xffffffffu, index < base + incl);
            if (hit) {
                const int l = __ffs(hit) - 1;
                seq = s0 + l;
                chunk = index - base - __shfl_sync(0xffffffffu, incl - mine, l);
            }
            base += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (lane == 0) {
            place->seq = seq;
            place->chunk = chunk;
            if (seq >= 0) place->span = spans[seq];
        }
    }
    __syncthreads();
    return place->seq >= 0;
}

// Number of the first chunk of sequence `seq` (uniform; a few sequences at most have chunks).
__device__ __forceinline__ int first_chunk(const SsmSpan* spans, int seq, int tokens) {
    int n = 0;
    for (int s = 0; s < seq; ++s) n += span_chunks(spans[s], tokens);
    return n;
}

}  // namespace hds
