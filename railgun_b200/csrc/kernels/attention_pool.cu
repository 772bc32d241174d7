// Pooled key/value entries: the mean of the keys and the mean of the values of every block of `pool` consecutive tokens
// of a request, as the cache holds them, written once, by the step that brings the block's last token.
//
// tokens:  pages [pages, 2, G, page_size, D] and the requests' block tables; the block's earlier tokens were written in
//          earlier steps or by this step's kernel before this one.
// entries: pages of the same shape, one entry where the others hold a token.  slots: the entries' group counts tokens,
//          page_size * pool to a page, so the entry of the block that ends at token t is slots[t] / pool.
// Sums in 32-bit in the order of the positions, one rounding into the storage type.
#include "common.cuh"

template <typename A>
__global__ void pool_blocks_kernel(const A* __restrict__ kv, const int* __restrict__ table, int max_blocks,
                                   const int* __restrict__ req_of_token, const int* __restrict__ positions,
                                   const int* __restrict__ slots, A* __restrict__ entries, int G, int page_size, int D,
                                   int pool) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x;
    const int pos = positions[t], slot = slots[t];
    if (slot < 0 || (pos + 1) % pool) return;
    const int* bt = table + (size_t)req_of_token[t] * max_blocks;
    const int entry = slot / pool, page_out = entry / page_size, off_out = entry - page_out * page_size;
    const size_t page_elems = (size_t)2 * G * page_size * D;
    const float inv = 1.f / (float)pool;
    for (int e = threadIdx.x; e < 2 * G * D; e += blockDim.x) {
        const int hh = e / D, i = e - hh * D;                       // keys of head 0 .. G - 1, then values
        float sum = 0.f;
        for (int j = 0; j < pool; ++j) {
            const int p = pos - pool + 1 + j;
            sum += to_f32(kv[(size_t)bt[p / page_size] * page_elems + ((size_t)hh * page_size + p % page_size) * D + i]);
        }
        entries[(size_t)page_out * page_elems + ((size_t)hh * page_size + off_out) * D + i] = from_f32<A>(sum * inv);
    }
}

extern "C" int rg_pool_blocks(const void* kv, int dtype, const int* table, int max_blocks, const int* req_of_token,
                              const int* positions, const int* slots, void* entries, int T, int G, int page_size, int D,
                              int pool, void* stream) {
    if (T <= 0) return 0;
    if (G < 1 || page_size < 1 || D < 1 || pool < 1) return RG_ERR_UNSUPPORTED;
    const int threads = 2 * G * D >= 512 ? 512 : 128;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == RG_DTYPE_BF16)
        return rg_launch(pool_blocks_kernel<bf16>, dim3(T), dim3(threads), 0, s, 1, (const bf16*)kv, table, max_blocks,
                         req_of_token, positions, slots, (bf16*)entries, G, page_size, D, pool);
    if (dtype == RG_DTYPE_F32)
        return rg_launch(pool_blocks_kernel<float>, dim3(T), dim3(threads), 0, s, 1, (const float*)kv, table, max_blocks,
                         req_of_token, positions, slots, (float*)entries, G, page_size, D, pool);
    return RG_ERR_UNSUPPORTED;
}
