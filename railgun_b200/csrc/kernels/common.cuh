// Shared helpers of the sm_100a kernels: element conversion, reductions and
// the launchers' error convention (every extern "C" launcher returns a
// cudaError_t as int; 0 is success, the Python side raises on anything else).
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>

#define RG_DTYPE_F32 0
#define RG_DTYPE_BF16 1
// An argument the launcher refuses (bad size, unsupported combination).
#define RG_ERR_UNSUPPORTED 10001

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Block-wide sum; every thread gets the result.  scratch: >= 33 floats of
// shared memory.  blockDim.x must be a multiple of 32.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < nwarp ? scratch[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}
__device__ __forceinline__ float block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    v = warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < nwarp ? scratch[lane] : -INFINITY;
        t = warp_max(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}

// cos and sin of pos * freq for rotary angles.  The product and its reduction to [-pi, pi] are 64-bit (three
// operations: the angle of a far position keeps all its digits), the functions themselves 32-bit on the small
// remainder, where they are good to a few 1e-8.
__device__ __forceinline__ void rotary_cos_sin(double pos, double freq, float* c, float* s) {
    const double a = pos * freq;
    const double n = rint(a * 0.15915494309189535);                  // a / (2 pi)
    const double r = fma(-n, 2.4492935982947064e-16, fma(-n, 6.283185307179586, a));
    sincosf((float)r, s, c);
}

// The gated activations of feed-forwards, act(gate) * up in 32-bit.  kind 0: silu(g) u; 1: gelu (tanh form) of g, times u;
// 2: the clamped form g' sigmoid(1.702 g') (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit).
#define RG_GATED_SILU 0
#define RG_GATED_GELU_TANH 1
#define RG_GATED_CLAMPED_SWISH 2
__device__ __forceinline__ float gated_act(float g, float u, int kind, float limit) {
    if (kind == RG_GATED_SILU) return g / (1.f + expf(-g)) * u;
    if (kind == RG_GATED_GELU_TANH)
        return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}

// Activations without a gate, in 32-bit.  kind 0: the square of relu; 1: relu; 2: gelu (tanh form); 3: silu; 4: gelu
// (exact, by the error function).
__device__ __forceinline__ float plain_act(float v, int kind) {
    if (kind == 0) { const float r = fmaxf(v, 0.f); return r * r; }
    if (kind == 1) return fmaxf(v, 0.f);
    if (kind == 2) return 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    if (kind == 4) return 0.5f * v * (1.f + erff(v * 0.70710678118654752f));
    return v / (1.f + expf(-v));
}

// The first position that the query at position p sees.  window > 0: a sliding window, p and the window - 1 positions
// before it; window < 0: chunks of -window positions counted from position 0, the query's own chunk; 0: everything.
// Never decreases with p.
__device__ __forceinline__ int first_seen(int p, int window) {
    return window > 0 ? max(0, p - window + 1) : (window < 0 ? p - p % -window : 0);
}

#define RG_LAUNCH_RESULT() ((int)cudaGetLastError())

// Programmatic dependent launch.  A kernel launched with the attribute may start while the kernel before it
// in the stream is still running; it must not touch anything that kernel (or an earlier one) reads or writes
// before pdl_wait(), which returns once the previous kernel has completed and its writes are visible.  Only
// constants (weights) may be read earlier.  pdl_trigger() lets the next kernel start launching.  Without the
// attribute both are no-ops.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

static int rg_pdl_enabled = 0;
extern "C" void rg_set_pdl(int on) { rg_pdl_enabled = on; }

// While one of these lives (constructed with true), launches are in plain stream order.
struct RgStreamOrder {
    int saved;
    explicit RgStreamOrder(bool on) : saved(rg_pdl_enabled) { if (on) rg_pdl_enabled = 0; }
    ~RgStreamOrder() { rg_pdl_enabled = saved; }
};

// Launch through cudaLaunchKernelEx so that the launch can carry attributes (dependent launch, clusters).
template <typename... KArgs, typename... Args>
static int rg_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, int cluster_x,
                     Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (rg_pdl_enabled) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    if (cluster_x > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = cluster_x;
        attr[n].val.clusterDim.y = 1;
        attr[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
    if (e != cudaSuccess) return (int)e;
    return (int)cudaGetLastError();
}
