// The pooled key/value entry of one block of tokens: the mean of the block's keys and of its values, as the cache holds
// them.  Sums in 32-bit in the order of the positions, one rounding into the storage type.
//
// tokens:  pages [pages, 2, G, page_size, D] behind the request's block table `bt`; the block's tokens are all there.
// entries: pages of the same shape, one entry where the others hold a token.  The entries' group counts tokens,
//          page_size * pool to a page, so the entry of the block whose last token has slot `slot` is slot / pool.
#pragma once
#include "common.cuh"

// How a kernel that has just written tokens finds where their blocks' entries go (pool 0: there are none).
struct PooledWrite {
    int pool;
    const int* table;
    int max_blocks;
    const int* req_of_token;
    const int* slots;
    void* entries;
};

// All threads of the block take part; `pos` is the position of the block of tokens' last one.
template <typename A>
__device__ __forceinline__ void pool_one_block(const A* kv, const int* __restrict__ bt, A* __restrict__ entries, int slot,
                                               int pos, int G, int page_size, int D, int pool) {
    if (slot < 0) return;
    const int entry = slot / pool, page_out = entry / page_size, off_out = entry - page_out * page_size;
    const size_t page_elems = (size_t)2 * G * page_size * D;
    const float inv = 1.f / (float)pool;
    for (int e = threadIdx.x; e < 2 * G * D; e += blockDim.x) {
        const int hh = e / D, i = e - hh * D;                       // keys of head 0 .. G - 1, then values
        const A* src = kv + (size_t)hh * page_size * D + i;
        float sum = 0.f;
#pragma unroll 4
        for (int j = 0; j < pool; ++j) {
            const int p = pos - pool + 1 + j, page = p / page_size;
            sum += to_f32(src[(size_t)bt[page] * page_elems + (size_t)(p - page * page_size) * D]);
        }
        entries[(size_t)page_out * page_elems + ((size_t)hh * page_size + off_out) * D + i] = from_f32<A>(sum * inv);
    }
}
