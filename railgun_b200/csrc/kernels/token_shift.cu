// Mixing a token with the token before it, and what RWKV-style time mixing computes around its scan.
//
//   postnorm_shift   x_t <- x_t + w unit(y_t) (y: the last part's output; unit: divided by its root mean square; without
//                    w: x_t + y_t), and h_t = x_t + (x_(t-1) - x_t) shift: the residual addition with the norm on a
//                    part's output, and the token shift of the part that reads the sum next, in one pass
//   shift_mixes      h_t + (h_(t-1) - h_t) mu_s for five vectors mu_s: four in the products' type, the fifth in 32-bit
//                    (for bfloat16 products: as the two halves hi | lo of a 32-bit number)
//   lowrank_decay    exp(-exp(W tanh(a_t) + w0)), the decay per token and channel, in 32-bit
//
// A request's row before the step's first one is kept in its state slot (32-bit, zeros at position 0).  The block that
// works on a request's first row is the one that reads the slot, and it also writes it (the step's last row), so that
// no other block can see the slot half way; a slot of -1 (padding of a static batch) is neither read nor written.
#include "common.cuh"

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = raw;
}
// One number at a time, for rows whose size is no multiple of four.
template <int V> struct Vec;
template <> struct Vec<4> {
    float4 v;
    template <typename T> __device__ __forceinline__ static Vec load(const T* p) { return {load4(p)}; }
    template <typename T> __device__ __forceinline__ void store(T* p) const { store4(p, v); }
    __device__ __forceinline__ static Vec zero() { return {make_float4(0.f, 0.f, 0.f, 0.f)}; }
    template <typename F> __device__ __forceinline__ static Vec map(Vec a, Vec b, Vec c, F f) {
        return {make_float4(f(a.v.x, b.v.x, c.v.x), f(a.v.y, b.v.y, c.v.y), f(a.v.z, b.v.z, c.v.z), f(a.v.w, b.v.w, c.v.w))};
    }
    __device__ __forceinline__ float squares() const { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
};
template <> struct Vec<1> {
    float v;
    template <typename T> __device__ __forceinline__ static Vec load(const T* p) { return {to_f32(*p)}; }
    template <typename T> __device__ __forceinline__ void store(T* p) const { *p = from_f32<T>(v); }
    __device__ __forceinline__ static Vec zero() { return {0.f}; }
    template <typename F> __device__ __forceinline__ static Vec map(Vec a, Vec b, Vec c, F f) { return {f(a.v, b.v, c.v)}; }
    __device__ __forceinline__ float squares() const { return v * v; }
};

// x [T, H] float and y [T, H] (or null) in; x_out [T, H] float: the new rows, another buffer than x where rows are
// shifted (a block reads the old row before its own first one); out [T, H] (type O).  shift [H] or null (out = the new
// rows); state [slots, H].  A block takes rows_per_block rows.  y_norm: post_w [H] and eps, or post_w null.
template <int V, typename P, typename O>
__global__ void postnorm_shift_kernel(const float* __restrict__ x, const P* __restrict__ y,
                                      const float* __restrict__ post_w, float eps, const float* __restrict__ shift,
                                      float* __restrict__ state, const int* __restrict__ cu_seqlens,
                                      const int* __restrict__ req_of_token, const int* __restrict__ start_pos,
                                      const int* __restrict__ slots, float* __restrict__ x_out, O* __restrict__ out,
                                      int T, int H, int rows_per_block) {
    extern __shared__ __align__(16) float prev[];     // [H]: the row before; every thread touches its own numbers only
    __shared__ float scratch[33];
    pdl_wait();
    pdl_trigger();
    const int t0 = blockIdx.x * rows_per_block, t1 = min(T, t0 + rows_per_block);
    auto unit = [&](int t) {                           // 1 / rms of y's row t (every thread of the block takes part)
        if (!y || !post_w) return 1.f;
        const P* p = y + (size_t)t * H;
        float ss = 0.f;
        for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) ss += Vec<V>::load(p + i).squares();
        return rsqrtf(block_sum(ss, scratch) / (float)H + eps);
    };
    auto value = [&](int t, int i, float inv) {        // numbers i .. i + V - 1 of the new row t
        Vec<V> v = Vec<V>::load(x + (size_t)t * H + i);
        if (y) {
            const Vec<V> p = Vec<V>::load(y + (size_t)t * H + i);
            if (post_w)
                v = Vec<V>::map(v, p, Vec<V>::load(post_w + i), [&](float a, float b, float w) { return a + b * inv * w; });
            else
                v = Vec<V>::map(v, p, p, [](float a, float b, float) { return a + b; });
        }
        return v;
    };
    int r = req_of_token ? req_of_token[t0] : 0;
    if (shift && t0 > cu_seqlens[r]) {                 // the block starts inside a request: its row before the first one
        const float inv = unit(t0 - 1);
        for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) value(t0 - 1, i, inv).store(prev + i);
    }
    for (int t = t0; t < t1; ++t) {
        const float inv = unit(t);
        if (!shift) {
            for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
                const Vec<V> v = value(t, i, inv);
                v.store(x_out + (size_t)t * H + i);
                v.store(out + (size_t)t * H + i);
            }
            continue;
        }
        r = req_of_token[t];
        const bool first = t == cu_seqlens[r];
        const int slot = slots[r];
        const bool has_past = first && slot >= 0 && start_pos[r] > 0;
        float* st = state + (size_t)(slot >= 0 ? slot : 0) * H;
        const int last = cu_seqlens[r + 1] - 1;
        for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
            const Vec<V> v = value(t, i, inv);
            const Vec<V> before = !first ? Vec<V>::load(prev + i) : (has_past ? Vec<V>::load(st + i) : Vec<V>::zero());
            v.store(x_out + (size_t)t * H + i);
            Vec<V>::map(v, before, Vec<V>::load(shift + i), [](float a, float b, float s) { return a + (b - a) * s; })
                .store(out + (size_t)t * H + i);
            v.store(prev + i);
            if (first && last == t && slot >= 0) v.store(st + i);
        }
        if (first && last > t && slot >= 0) {          // the slot gets the step's last row
            const float inv_last = unit(last);
            for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) value(last, i, inv_last).store(st + i);
        }
    }
}

extern "C" int rg_postnorm_shift(const float* x, const void* y, int y_dtype, const float* post_w, float eps,
                                 const float* shift, float* state, const int* cu_seqlens, const int* req_of_token,
                                 const int* start_pos, const int* slots, float* x_out, void* out, int out_dtype, int T,
                                 int H, int rows_per_block, void* stream) {
    if (T <= 0 || H <= 0) return 0;
    if (rows_per_block < 1 || (shift && (!state || !cu_seqlens || !req_of_token || !start_pos || !slots || x == x_out)))
        return RG_ERR_UNSUPPORTED;
    const size_t smem = shift ? (size_t)H * sizeof(float) : 0;
    if (smem > 48 * 1024) return RG_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const uintptr_t all = (uintptr_t)x | (uintptr_t)y | (uintptr_t)post_w | (uintptr_t)shift | (uintptr_t)state |
                          (uintptr_t)x_out | (uintptr_t)out;
    const bool vec = H % 4 == 0 && (all & 15) == 0;
    const int work = vec ? H / 4 : H;
    const int threads = work >= 512 ? 512 : (work >= 256 ? 256 : 128);
    dim3 grid((T + rows_per_block - 1) / rows_per_block);
    if (!y) y_dtype = RG_DTYPE_F32;
#define TS_LAUNCH(V, P, O) return rg_launch(postnorm_shift_kernel<V, P, O>, grid, dim3(threads), smem, s, 1, x, (const P*)y, \
        post_w, eps, shift, state, cu_seqlens, req_of_token, start_pos, slots, x_out, (O*)out, T, H, rows_per_block)
#define TS_TYPES(P, O) { if (vec) TS_LAUNCH(4, P, O); TS_LAUNCH(1, P, O); }
    if (y_dtype == RG_DTYPE_BF16 && out_dtype == RG_DTYPE_BF16) TS_TYPES(bf16, bf16)
    if (y_dtype == RG_DTYPE_F32 && out_dtype == RG_DTYPE_BF16) TS_TYPES(float, bf16)
    if (y_dtype == RG_DTYPE_F32 && out_dtype == RG_DTYPE_F32) TS_TYPES(float, float)
    if (y_dtype == RG_DTYPE_BF16 && out_dtype == RG_DTYPE_F32) TS_TYPES(bf16, float)
#undef TS_TYPES
#undef TS_LAUNCH
    return RG_ERR_UNSUPPORTED;
}

// h [T, H] (type A).  mu [5, H].  mixes [4, T, H] (type A): mu 0 .. 3.  last: mu 4, [T, H] float for float rows; for
// bfloat16 rows [T, 2 H] bfloat16, hi | lo with hi + lo the 32-bit number to 2^-17.  One block per row.
template <int V, typename A>
__global__ void shift_mixes_kernel(const A* __restrict__ h, const float* __restrict__ mu, float* __restrict__ state,
                                   const int* __restrict__ cu_seqlens, const int* __restrict__ req_of_token,
                                   const int* __restrict__ start_pos, const int* __restrict__ slots,
                                   A* __restrict__ mixes, A* __restrict__ last, int T, int H) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x;
    const int r = req_of_token[t];
    const int lo = cu_seqlens[r];
    const bool first = t == lo;
    const int slot = slots[r];
    const bool has_past = first && slot >= 0 && start_pos[r] > 0;
    float* st = state + (size_t)(slot >= 0 ? slot : 0) * H;
    const int end = cu_seqlens[r + 1] - 1;
    for (int i = (blockIdx.y * blockDim.x + threadIdx.x) * V; i < H; i += gridDim.y * blockDim.x * V) {
        const Vec<V> v = Vec<V>::load(h + (size_t)t * H + i);
        const Vec<V> before = !first ? Vec<V>::load(h + (size_t)(t - 1) * H + i)
                                     : (has_past ? Vec<V>::load(st + i) : Vec<V>::zero());
        auto mix = [](float a, float b, float s) { return a + (b - a) * s; };
#pragma unroll
        for (int m = 0; m < 4; ++m)
            Vec<V>::map(v, before, Vec<V>::load(mu + (size_t)m * H + i), mix).store(mixes + ((size_t)m * T + t) * H + i);
        const Vec<V> w = Vec<V>::map(v, before, Vec<V>::load(mu + (size_t)4 * H + i), mix);
        if (sizeof(A) == 4) {
            w.store(last + (size_t)t * H + i);
        } else {
            auto rounded = [](float a, float, float) { return __bfloat162float(__float2bfloat16_rn(a)); };
            const Vec<V> hi = Vec<V>::map(w, w, w, rounded);
            hi.store(last + (size_t)t * 2 * H + i);
            Vec<V>::map(w, hi, hi, [](float a, float b, float) { return a - b; }).store(last + (size_t)t * 2 * H + H + i);
        }
        if (first && slot >= 0) Vec<V>::load(h + (size_t)end * H + i).store(st + i);
    }
}

extern "C" int rg_shift_mixes(const void* h, int dtype, const float* mu, float* state, const int* cu_seqlens,
                              const int* req_of_token, const int* start_pos, const int* slots, void* mixes, void* last,
                              int T, int H, void* stream) {
    if (T <= 0 || H <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const uintptr_t all = (uintptr_t)h | (uintptr_t)mu | (uintptr_t)state | (uintptr_t)mixes | (uintptr_t)last;
    const bool vec = H % 4 == 0 && (all & 15) == 0;
    const int work = vec ? (H + 3) / 4 : H;
    const int threads = work >= 256 ? 256 : 128;
    // few rows: a row is spread over blocks
    int spread = (work + threads - 1) / threads;
    if (T >= 592) spread = 1;
    if (spread > 65535) return RG_ERR_UNSUPPORTED;
    dim3 grid(T, spread);
#define TS_MIX(V, A) return rg_launch(shift_mixes_kernel<V, A>, grid, dim3(threads), 0, s, 1, (const A*)h, mu, state, \
        cu_seqlens, req_of_token, start_pos, slots, (A*)mixes, (A*)last, T, H)
    if (dtype == RG_DTYPE_BF16) { if (vec) TS_MIX(4, bf16); TS_MIX(1, bf16); }
    if (dtype == RG_DTYPE_F32) { if (vec) TS_MIX(4, float); TS_MIX(1, float); }
#undef TS_MIX
    return RG_ERR_UNSUPPORTED;
}

// a [T, rank] float; w [N, rank] (type A), w0 [N]; out [T, N] float = exp(-exp(w . tanh(a) + w0)).  A block takes TT
// tokens and CC channels, the rank in pieces of 64 through shared memory; a thread has TT / 16 tokens x CC / 16 channels
// (few tokens: 16 x 16, so that a step of single tokens has blocks enough; portions: 64 x 64).
#define LD_RANK 64
template <int TT, int CC, typename A>
__global__ void __launch_bounds__(256)
lowrank_decay_kernel(const float* __restrict__ a, const A* __restrict__ w, const float* __restrict__ w0,
                     float* __restrict__ out, int T, int N, int rank) {
    constexpr int NT = TT / 16, NC = CC / 16;
    __shared__ __align__(16) float sa[LD_RANK][TT + 4];
    __shared__ __align__(16) float sw[LD_RANK][CC + 4];
    pdl_wait();
    pdl_trigger();
    const int t0 = blockIdx.x * TT, n0 = blockIdx.y * CC;
    const int tc = threadIdx.x & 15, tr = threadIdx.x >> 4;     // channels NC tc .. + NC - 1, tokens tr NT .. + NT - 1
    float acc[NT][NC];
#pragma unroll
    for (int x = 0; x < NT; ++x)
#pragma unroll
        for (int y = 0; y < NC; ++y) acc[x][y] = 0.f;
    for (int k0 = 0; k0 < rank; k0 += LD_RANK) {
        const int n = min(LD_RANK, rank - k0);
        // 8 neighbouring k of 4 rows at a time: whole sectors in, different banks out
#pragma unroll 4
        for (int e = threadIdx.x; e < TT * LD_RANK; e += 256) {
            const int k = (e & 7) + ((e >> 5) & 7) * 8, t = ((e >> 3) & 3) + (e >> 8) * 4;
            sa[k][t] = (k < n && t0 + t < T) ? tanhf(a[(size_t)(t0 + t) * rank + k0 + k]) : 0.f;
        }
#pragma unroll 4
        for (int e = threadIdx.x; e < CC * LD_RANK; e += 256) {
            const int k = (e & 7) + ((e >> 5) & 7) * 8, c = ((e >> 3) & 3) + (e >> 8) * 4;
            sw[k][c] = (k < n && n0 + c < N) ? to_f32(w[(size_t)(n0 + c) * rank + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll 4
        for (int k = 0; k < n; ++k) {
            float av[NT], wv[NC];
#pragma unroll
            for (int x = 0; x < NT; ++x) av[x] = sa[k][tr * NT + x];
#pragma unroll
            for (int y = 0; y < NC; ++y) wv[y] = sw[k][tc * NC + y];
#pragma unroll
            for (int x = 0; x < NT; ++x)
#pragma unroll
                for (int y = 0; y < NC; ++y) acc[x][y] += av[x] * wv[y];
        }
        __syncthreads();
    }
#pragma unroll
    for (int x = 0; x < NT; ++x) {
        const int t = t0 + tr * NT + x;
        if (t >= T) continue;
#pragma unroll
        for (int y = 0; y < NC; ++y) {
            const int c = n0 + NC * tc + y;
            if (c < N) out[(size_t)t * N + c] = expf(-expf(acc[x][y] + w0[c]));
        }
    }
}

extern "C" int rg_lowrank_decay(const float* a, const void* w, int dtype, const float* w0, float* out, int T, int N,
                                int rank, void* stream) {
    if (T <= 0 || N <= 0) return 0;
    if (rank < 1) return RG_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const int tt = T > 64 ? 64 : 16;
    dim3 grid((T + tt - 1) / tt, (N + tt - 1) / tt);
    if (grid.y > 65535) return RG_ERR_UNSUPPORTED;
#define TS_DECAY(TT, A) return rg_launch(lowrank_decay_kernel<TT, TT, A>, grid, dim3(256), 0, s, 1, a, (const A*)w, w0, out, T, N, rank)
    if (dtype == RG_DTYPE_BF16) { if (tt == 64) TS_DECAY(64, bf16); TS_DECAY(16, bf16); }
    if (dtype == RG_DTYPE_F32) { if (tt == 64) TS_DECAY(64, float); TS_DECAY(16, float); }
#undef TS_DECAY
    return RG_ERR_UNSUPPORTED;
}
