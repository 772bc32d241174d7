// Pooled key/value entries (attention_pool.cuh) of all blocks of tokens that a step completes, after the kernel that
// wrote the step's keys and values: steps with portions of prompts, where a block's tokens may come from several thread
// blocks of that kernel (single-token steps pool inside it).
#include "attention_pool.cuh"

template <typename A>
__global__ void pool_blocks_kernel(const A* __restrict__ kv, const int* __restrict__ table, int max_blocks,
                                   const int* __restrict__ req_of_token, const int* __restrict__ positions,
                                   const int* __restrict__ slots, A* __restrict__ entries, int T, int G, int page_size,
                                   int D, int pool, int span) {
    pdl_wait();
    pdl_trigger();
    const int t1 = min(T, (int)(blockIdx.x + 1) * span);
    for (int t = blockIdx.x * span; t < t1; ++t) {
        const int pos = positions[t];
        if ((pos + 1) % pool == 0)
            pool_one_block(kv, table + (size_t)req_of_token[t] * max_blocks, entries, slots[t], pos, G, page_size, D, pool);
    }
}

extern "C" int rg_pool_blocks(const void* kv, int dtype, const int* table, int max_blocks, const int* req_of_token,
                              const int* positions, const int* slots, void* entries, int T, int G, int page_size, int D,
                              int pool, void* stream) {
    if (T <= 0) return 0;
    if (G < 1 || page_size < 1 || D < 1 || pool < 1) return RG_ERR_UNSUPPORTED;
    const int threads = 2 * G * D >= 512 ? 512 : 128;
    const int span = pool < 16 ? pool : 16;                         // tokens per thread block: about one ends a block
    cudaStream_t s = (cudaStream_t)stream;
#define POOL_LAUNCH(A) return rg_launch(pool_blocks_kernel<A>, dim3((T + span - 1) / span), dim3(threads), 0, s, 1, \
        (const A*)kv, table, max_blocks, req_of_token, positions, slots, (A*)entries, T, G, page_size, D, pool, span)
    if (dtype == RG_DTYPE_BF16) POOL_LAUNCH(bf16);
    if (dtype == RG_DTYPE_F32) POOL_LAUNCH(float);
#undef POOL_LAUNCH
    return RG_ERR_UNSUPPORTED;
}
