// The residual step of blocks whose norms may be layer norms:
//
//   u   = post(y)                     the part's output y, normed: not at all, by its root mean square, or centred first
//                                     (kind 0: y; 1: w y / sqrt(mean(y^2) + eps); 2: w (y - m) / sqrt(mean((y - m)^2) + eps) + b
//                                     with m = mean(y))
//   r   = residual[row] + u           32-bit, written back (not with `rows`)
//   out = pre(r)                      the next part's input: r in the activation type, or r normed in one of the ways above
//
// Sums, means, roots and the addition are 32-bit; the deviations' squares are summed after the mean is known (the row
// waits in registers), so a row far from zero loses nothing.  With `rows` given, output row i is computed from residual
// row rows[i].  One block per row.
#include "common.cuh"

struct RowNorm {
    int kind;                 // 0: none, 1: root mean square, 2: layer norm
    const float* w;
    const float* b;           // kind 2
    float eps;
};

// The row's numbers of this thread: piece j holds numbers V (threadIdx.x + j blockDim.x) .. + V - 1.
template <int NV, int V>
__device__ __forceinline__ void norm_row(float (&x)[NV][V], const RowNorm& n, int H, float* scratch) {
    if (n.kind == 0) return;
    float mean = 0.f;
    if (n.kind == 2) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) s += x[j][e];
        mean = block_sum(s, scratch) / (float)H;
    }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        if (V * (int)(threadIdx.x + j * blockDim.x) < H) {
#pragma unroll
            for (int e = 0; e < V; ++e) { x[j][e] -= mean; ss += x[j][e] * x[j][e]; }
        }
    }
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)H + n.eps);
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = V * (threadIdx.x + j * blockDim.x);
        if (i < H) {
            __align__(16) float w[V], b[V];
            if (V == 4) {
                *reinterpret_cast<float4*>(w) = *reinterpret_cast<const float4*>(n.w + i);
                if (n.kind == 2) *reinterpret_cast<float4*>(b) = *reinterpret_cast<const float4*>(n.b + i);
            } else {
                w[0] = n.w[i];
                if (n.kind == 2) b[0] = n.b[i];
            }
#pragma unroll
            for (int e = 0; e < V; ++e) x[j][e] = n.kind == 2 ? x[j][e] * inv * w[e] + b[e] : x[j][e] * inv * w[e];
        }
    }
}

template <int V, typename P>
__device__ __forceinline__ void load_piece(const P* p, float (&x)[V]) {
    if (V == 4 && sizeof(P) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        x[0] = a.x; x[1 % V] = a.y; x[2 % V] = b.x; x[3 % V] = b.y;
    } else if (V == 4) {
        *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(p);
    } else {
        x[0] = to_f32(p[0]);
    }
}
template <int V, typename P>
__device__ __forceinline__ void store_piece(P* p, const float (&x)[V]) {
    if (V == 4 && sizeof(P) == 2) {
        uint2 o;
        *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(x[0], x[1 % V]);
        *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(x[2 % V], x[3 % V]);
        *reinterpret_cast<uint2*>(p) = o;
    } else if (V == 4) {
        *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(x);
    } else {
        p[0] = from_f32<P>(x[0]);
    }
}

template <int NV, int V, typename P, typename O>
__global__ void __launch_bounds__(512)
stream_norm_kernel(float* __restrict__ resid, const P* __restrict__ y, RowNorm post, RowNorm pre, O* __restrict__ out,
                   const int* __restrict__ rows, int H) {
    __shared__ float scratch[33];
    pdl_wait();
    pdl_trigger();
    const int orow = blockIdx.x;
    const int srow = rows ? rows[orow] : orow;
    float* r = resid + (size_t)srow * H;
    __align__(16) float x[NV][V];
    if (y) {
        const P* p = y + (size_t)srow * H;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = V * (threadIdx.x + j * blockDim.x);
            if (i < H) {
                load_piece<V>(p + i, x[j]);
            } else {
#pragma unroll
                for (int e = 0; e < V; ++e) x[j][e] = 0.f;
            }
        }
        norm_row<NV, V>(x, post, H, scratch);
    } else {
#pragma unroll
        for (int j = 0; j < NV; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) x[j][e] = 0.f;
    }
    const bool write_back = rows == nullptr && y != nullptr;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = V * (threadIdx.x + j * blockDim.x);
        if (i < H) {
            __align__(16) float v[V];
            load_piece<V>(r + i, v);
#pragma unroll
            for (int e = 0; e < V; ++e) x[j][e] += v[e];
            if (write_back) store_piece<V>(r + i, x[j]);
        }
    }
    if (out == nullptr) return;
    norm_row<NV, V>(x, pre, H, scratch);
    O* o = out + (size_t)orow * H;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = V * (threadIdx.x + j * blockDim.x);
        if (i < H) store_piece<V>(o + i, x[j]);
    }
}

// y (rows of H, y_dtype) may be null; out may be null.
extern "C" int rg_stream_norm(float* resid, const void* y, int y_dtype, int post_kind, const float* post_w, const float* post_b,
                              float post_eps, int pre_kind, const float* pre_w, const float* pre_b, float pre_eps, void* out,
                              int out_dtype, const int* rows, int n_out_rows, int H, void* stream) {
    if (n_out_rows <= 0) return 0;
    auto bad = [](int kind, const float* w, const float* b) {
        return kind < 0 || kind > 2 || (kind > 0 && !w) || (kind == 2 && !b);
    };
    if (H < 1 || bad(post_kind, post_w, post_b) || bad(pre_kind, pre_w, pre_b)) return RG_ERR_UNSUPPORTED;
    const RowNorm post = {post_kind, post_w, post_b, post_eps}, pre = {pre_kind, pre_w, pre_b, pre_eps};
    cudaStream_t s = (cudaStream_t)stream;
    if (y == nullptr) y_dtype = RG_DTYPE_F32;
    if (out == nullptr) out_dtype = RG_DTYPE_F32;
    const uintptr_t wide = (uintptr_t)resid | (uintptr_t)post_w | (uintptr_t)post_b | (uintptr_t)pre_w | (uintptr_t)pre_b;
    auto aligned = [](const void* p, int dtype) { return ((uintptr_t)p & (dtype == RG_DTYPE_BF16 ? 7 : 15)) == 0; };
    const bool vec = H % 4 == 0 && (wide & 15) == 0 && aligned(y, y_dtype) && aligned(out, out_dtype);
    const int pieces = vec ? H / 4 : H;
    int nv = 1;
    while (nv < 16 && pieces > nv * (nv == 1 ? 256 : 512)) nv <<= 1;
    int threads = ((pieces + nv - 1) / nv + 31) / 32 * 32;
    if (threads > 512) return RG_ERR_UNSUPPORTED;
#define SN_ROW(NV, V, P, O) return rg_launch(stream_norm_kernel<NV, V, P, O>, dim3(n_out_rows), dim3(threads), 0, s, 1, resid, \
        (const P*)y, post, pre, (O*)out, rows, H)
#define SN_TYPES(NV, V) { \
        if (y_dtype == RG_DTYPE_BF16 && out_dtype == RG_DTYPE_BF16) SN_ROW(NV, V, bf16, bf16); \
        if (y_dtype == RG_DTYPE_F32 && out_dtype == RG_DTYPE_BF16) SN_ROW(NV, V, float, bf16); \
        if (y_dtype == RG_DTYPE_BF16 && out_dtype == RG_DTYPE_F32) SN_ROW(NV, V, bf16, float); \
        if (y_dtype == RG_DTYPE_F32 && out_dtype == RG_DTYPE_F32) SN_ROW(NV, V, float, float); \
        return RG_ERR_UNSUPPORTED; }
#define SN_COUNT(V) switch (nv) { case 1: SN_TYPES(1, V) case 2: SN_TYPES(2, V) case 4: SN_TYPES(4, V) case 8: SN_TYPES(8, V) \
        default: SN_TYPES(16, V) }
    if (vec) SN_COUNT(4)
    SN_COUNT(1)
#undef SN_COUNT
#undef SN_TYPES
#undef SN_ROW
}
