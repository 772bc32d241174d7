// General paged attention: one thread block per (query token, head), any head
// size up to 256, any page size, 32-bit or bfloat16 storage, all arithmetic in
// 32-bit.  It serves the true 32-bit path and every shape the fast kernels
// refuse.  A query at absolute position p of request r attends the keys of r
// at positions [max(0, p - window + 1), p] (window < 0: those of its own chunk
// of -window positions up to its own) and, with keep_first, also the first
// keep_first positions of r whatever the window (kept tokens keep their own
// positions), read from the paged cache through r's block table (the step's
// own keys are written before it runs).  Optional: `sink` [nh], one more term
// exp(sink[h]) in head h's denominator that has neither key nor value and is
// not scaled; `gate`, rows gate_ld apart, head h's output at token t is
// multiplied by sigmoid(gate[t, h]); with a window and `pool` > 0, blocks of
// `pool` tokens that lie wholly before the window are seen as one entry each
// of a second set of pages (block b stands for positions b pool ..
// (b + 1) pool - 1 and is seen if (b + 1) pool - 1 <= p - window); output rows
// out_ld apart, times out_scale.
//
// Formulas: kv_head = head / (nh / nkv); s_j = scale * q.k_j; running max m,
// p_j = exp(s_j - m), out = sum p_j v_j / sum p_j
// (crates/vllm-cuda/src/kernels/paged_attention.cu:40,66-69,103-107;
// single-pass online form crates/vllm-cuda/src/kernels/paged_attention_v1_plus.cu:56-100).
// The reference masks only j < context_len; the mask by the query's own
// position (causal inside a portion of a prompt) is added here.
#include "common.cuh"

#define ATT_THREADS 128

// q: rows of stride q_stride elements, head h at offset h*d.  out: [T, nh*d].
// kv_cache: [NP, 2, nkv, ps, d].  block_table: [R, max_blocks].
template <typename A>
__global__ void paged_attention_general_kernel(
        const A* __restrict__ q, int q_stride, A* __restrict__ out, const A* __restrict__ kv_cache,
        const int* __restrict__ block_table, int max_blocks, const int* __restrict__ req_of_token,
        const int* __restrict__ positions, int nh, int nkv, int d, int page_size, int window, float scale, int keep_first,
        const float* __restrict__ sink, const A* __restrict__ gate, int gate_ld,
        const A* __restrict__ pool_kv, const int* __restrict__ pool_table, int pool_blocks, int pool, int out_ld,
        float out_scale) {
    extern __shared__ float smem[];
    float* qs = smem;                    // [d]
    float* ps = qs + d;                  // [ATT_THREADS]
    float* scratch = ps + ATT_THREADS;   // [33]
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, h = blockIdx.y;
    const int kvh = h / (nh / nkv);
    const int r = req_of_token[t];
    const int pos = positions[t];
    const int lo = first_seen(pos, window);
    const int* bt = block_table + (size_t)r * max_blocks;
    const A* qrow = q + (size_t)t * q_stride + (size_t)h * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) qs[i] = to_f32(qrow[i]) * scale;
    __syncthreads();

    float m = -INFINITY, l = 0.f;
    float acc0 = 0.f, acc1 = 0.f;        // output dims threadIdx.x and threadIdx.x + 128
    const size_t page_elems = (size_t)2 * nkv * page_size * d;
    // the keys a query sees, numbered 0 .. n_sink + (pos - lo): the kept first tokens that the window has passed, then the window
    // (pooled entries are numbered the same way, before the window)
    const int n_sink = pool > 0 ? (pos - window + 1 >= pool ? (pos - window + 1) / pool : 0) : (window > 0 ? min(keep_first, lo) : 0);
    const int* pbt = pool > 0 ? pool_table + (size_t)r * pool_blocks : bt;
    const A* first_kv = pool > 0 ? pool_kv : kv_cache;
    const int n_seen = n_sink + pos - lo + 1;
    for (int base = 0; base < n_seen; base += ATT_THREADS) {
        const int e = base + threadIdx.x;
        const int j = e < n_sink ? e : lo + (e - n_sink);
        float s = -INFINITY;
        if (e < n_seen) {
            const int page = (e < n_sink ? pbt : bt)[j / page_size], off = j % page_size;
            const A* krow = (e < n_sink ? first_kv : kv_cache) + (size_t)page * page_elems + ((size_t)kvh * page_size + off) * d;
            float dot = 0.f;
            for (int i = 0; i < d; ++i) dot += qs[i] * to_f32(krow[i]);
            s = dot;
        }
        const float cmax = block_max(s, scratch);
        const float m_new = fmaxf(m, cmax);
        const float p = (e < n_seen) ? expf(s - m_new) : 0.f;
        const float alpha = expf(m - m_new);           // 0 when m = -inf
        const float csum = block_sum(p, scratch);
        l = l * alpha + csum;
        m = m_new;
        ps[threadIdx.x] = p;
        __syncthreads();
        acc0 *= alpha;
        acc1 *= alpha;
        const int n = min(ATT_THREADS, n_seen - base);
        for (int k = 0; k < n; ++k) {
            const int jj = base + k < n_sink ? base + k : lo + (base + k - n_sink);
            const bool before = base + k < n_sink;
            const int page = (before ? pbt : bt)[jj / page_size], off = jj % page_size;
            const A* vrow = (before ? first_kv : kv_cache) + (size_t)page * page_elems
                            + ((size_t)(nkv + kvh) * page_size + off) * d;
            const float pk = ps[k];
            if (threadIdx.x < d) acc0 += pk * to_f32(vrow[threadIdx.x]);
            if (threadIdx.x + ATT_THREADS < d) acc1 += pk * to_f32(vrow[threadIdx.x + ATT_THREADS]);
        }
        __syncthreads();
    }
    A* orow = out + (size_t)t * out_ld + (size_t)h * d;
    if (sink) {
        const float m_new = fmaxf(m, sink[h]);
        const float alpha = expf(m - m_new);
        l = l * alpha + expf(sink[h] - m_new);
        acc0 *= alpha;
        acc1 *= alpha;
    }
    float inv = l > 0.f ? 1.f / l : 0.f;
    inv *= out_scale;
    if (gate) inv *= 1.f / (1.f + expf(-to_f32(gate[(size_t)t * gate_ld + h])));
    if (threadIdx.x < d) orow[threadIdx.x] = from_f32<A>(acc0 * inv);
    if (threadIdx.x + ATT_THREADS < d) orow[threadIdx.x + ATT_THREADS] = from_f32<A>(acc1 * inv);
}

extern "C" int rg_paged_attention_general(
        const void* q, int q_stride, void* out, const void* kv_cache, int dtype,
        const int* block_table, int max_blocks, const int* req_of_token, const int* positions,
        int T, int nh, int nkv, int d, int page_size, int window, float scale, int keep_first, const float* sink,
        const void* gate, int gate_ld, const void* pool_kv, const int* pool_table, int pool_blocks, int pool, int out_ld,
        float out_scale, void* stream) {
    if (T <= 0) return 0;
    if (pool < 0 || (pool > 0 && (!pool_kv || !pool_table || window <= 0 || keep_first > 0)) || out_ld < nh * d)
        return RG_ERR_UNSUPPORTED;
    if (d > 2 * ATT_THREADS || d < 1 || nkv < 1 || nh < nkv || nh % nkv || keep_first < 0) return RG_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid(T, nh);
    const size_t smem = (size_t)(d + ATT_THREADS + 33) * sizeof(float);
    if (dtype == RG_DTYPE_BF16)
        return rg_launch(paged_attention_general_kernel<bf16>, grid, dim3(ATT_THREADS), smem, s, 1,
                         (const bf16*)q, q_stride, (bf16*)out, (const bf16*)kv_cache, block_table, max_blocks,
                         req_of_token, positions, nh, nkv, d, page_size, window, scale, keep_first, sink, (const bf16*)gate,
                         gate_ld, (const bf16*)pool_kv, pool_table, pool_blocks, pool, out_ld, out_scale);
    if (dtype == RG_DTYPE_F32)
        return rg_launch(paged_attention_general_kernel<float>, grid, dim3(ATT_THREADS), smem, s, 1,
                         (const float*)q, q_stride, (float*)out, (const float*)kv_cache, block_table, max_blocks,
                         req_of_token, positions, nh, nkv, d, page_size, window, scale, keep_first, sink, (const float*)gate,
                         gate_ld, (const float*)pool_kv, pool_table, pool_blocks, pool, out_ld, out_scale);
    return RG_ERR_UNSUPPORTED;
}
