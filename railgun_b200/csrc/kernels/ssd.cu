// The mixer of Mamba-2 around its scan (Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms
// Through Structured State Space Duality").
//
//   ssd_prepare      dt = softplus(raw + bias), g = exp(-exp(A_log) dt), per token and head
//   ssd_step         single tokens: the causal convolution with its activation on x, B and C, dt and g, one step of
//                      S <- g S + dt B x^T;  o = S^T C + D x
//                    and the output, in one kernel; the convolution's state is read here and moved on by the kernel
//                    behind it (gate_group_norm), since the heads of a group share their B and C channels
//   gate_group_norm  (o silu(z)) / rms, each of `groups` equal parts by its own root mean square, times a weight: the
//                    gate comes before the norm; rounded once for the output product
//
// A request whose start position is 0 begins from zeros whatever its slot holds; a slot of -1 (padding of a static
// batch) is neither read nor written.  All arithmetic is 32-bit.
#include "common.cuh"

__device__ __forceinline__ float ssd_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float ssd_softplus(float z) { return log1pf(expf(-fabsf(z))) + fmaxf(z, 0.f); }

// raw: rows raw_ld apart, H numbers each.  dt, g [T, H].
__global__ void ssd_prepare_kernel(const float* __restrict__ raw, int raw_ld, const float* __restrict__ dt_bias,
                                   const float* __restrict__ A_log, float* __restrict__ dt, float* __restrict__ g, int T,
                                   int H) {
    pdl_wait();
    pdl_trigger();
    const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= (long long)T * H) return;
    const int t = (int)(e / H), h = (int)(e - (long long)t * H);
    const float v = ssd_softplus(raw[(size_t)t * raw_ld + h] + dt_bias[h]);
    dt[e] = v;
    g[e] = expf(-expf(A_log[h]) * v);
}

extern "C" int rg_ssd_prepare(const float* raw, int raw_ld, const float* dt_bias, const float* A_log, float* dt, float* g,
                              int T, int H, void* stream) {
    if (T <= 0) return 0;
    if (H < 1) return RG_ERR_UNSUPPORTED;
    const long long n = (long long)T * H;
    return rg_launch(ssd_prepare_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, 1, raw,
                     raw_ld, dt_bias, A_log, dt, g, T, H);
}

// One block per (token, head, block of columns of S).  proj: rows ld apart, [.. x: H dv at x_off | B: G N | C: G N .. ]
// side by side, raw dt at dt_off (32-bit rows).  conv_state [slots, K - 1, C] (C = H dv + 2 G N), taps [K, C], bias [C].
// state [slots, H, dv, N]: S transposed.  o [T, H, dv].  A warp takes one column of S at a time: N numbers side by side.
#define SSD_THREADS 256
template <bool VEC>
__global__ void __launch_bounds__(SSD_THREADS)
ssd_step_kernel(const float* __restrict__ proj, int ld, int x_off, int dt_off, const float* __restrict__ taps,
                const float* __restrict__ bias, const float* __restrict__ conv_state, const float* __restrict__ dt_bias,
                const float* __restrict__ A_log, const float* __restrict__ D, float* __restrict__ state,
                const int* __restrict__ req_of_token, const int* __restrict__ start_pos, const int* __restrict__ slots,
                float* __restrict__ o, int H, int G, int N, int dv, int K, int cols) {
    extern __shared__ __align__(16) float sm[];       // B [N], C [N] (padded to 4), x [cols]
    const int NP = (N + 3) & ~3;
    float *sB = sm, *sC = sm + NP, *sx = sm + 2 * NP;
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * cols;
    const int n = min(cols, dv - j0);
    const int r = req_of_token[t];
    const int slot = slots[r];
    const bool has_past = slot >= 0 && start_pos[r] > 0;
    const int grp = h / (H / G), C = H * dv + 2 * G * N;
    const float* row = proj + (size_t)t * ld;
    const float* past = conv_state + (size_t)(slot >= 0 ? slot : 0) * (K - 1) * C;
    for (int e = threadIdx.x; e < 2 * N + n; e += blockDim.x) {
        const int c = e < N ? H * dv + grp * N + e : (e < 2 * N ? H * dv + G * N + grp * N + (e - N) : h * dv + j0 + (e - 2 * N));
        float acc = bias ? bias[c] : 0.f;
        if (has_past)
            for (int j = 0; j < K - 1; ++j) acc += taps[(size_t)j * C + c] * past[(size_t)j * C + c];
        acc += taps[(size_t)(K - 1) * C + c] * row[x_off + c];
        acc = ssd_silu(acc);
        if (e < N) sB[e] = acc;
        else if (e < 2 * N) sC[e - N] = acc;
        else sx[e - 2 * N] = acc;
    }
    const float dt = ssd_softplus(row[dt_off + h] + dt_bias[h]);
    const float g = expf(-expf(A_log[h]) * dt);
    const float skip = D[h];
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* st = state + (((size_t)(slot >= 0 ? slot : 0) * H + h) * dv + j0) * N;
    for (int j = warp; j < n; j += SSD_THREADS / 32) {
        float* col = st + (size_t)j * N;
        const float u = dt * sx[j];
        float acc = 0.f;
        if (VEC) {
            for (int i = lane * 4; i < N; i += 128) {
                float4 S = has_past ? *reinterpret_cast<const float4*>(col + i) : make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 b = *reinterpret_cast<const float4*>(sB + i), c = *reinterpret_cast<const float4*>(sC + i);
                S.x = S.x * g + b.x * u; S.y = S.y * g + b.y * u; S.z = S.z * g + b.z * u; S.w = S.w * g + b.w * u;
                acc += S.x * c.x + S.y * c.y + S.z * c.z + S.w * c.w;
                if (slot >= 0) *reinterpret_cast<float4*>(col + i) = S;
            }
        } else {
            for (int i = lane; i < N; i += 32) {
                const float S = (has_past ? col[i] : 0.f) * g + sB[i] * u;
                acc += S * sC[i];
                if (slot >= 0) col[i] = S;
            }
        }
        acc = warp_sum(acc);
        if (lane == 0) o[((size_t)t * H + h) * dv + j0 + j] = acc + skip * sx[j];
    }
}

extern "C" int rg_ssd_step(const float* proj, int ld, int x_off, int dt_off, const float* taps, const float* bias,
                           const float* conv_state, const float* dt_bias, const float* A_log, const float* D, float* state,
                           const int* req_of_token, const int* start_pos, const int* slots, float* o, int T, int H, int G,
                           int N, int dv, int K, void* stream) {
    if (T <= 0) return 0;
    if (H < 1 || G < 1 || H % G || N < 1 || dv < 1 || K < 1 || (K > 1 && !conv_state) || H > 65535) return RG_ERR_UNSUPPORTED;
    // while there are few (token, head) pairs a head's columns are spread over blocks, 8 (one per warp) at the least
    int cols = dv;
    while ((long long)T * H * ((dv + cols - 1) / cols) < 592 && cols > 8) cols = (cols + 1) / 2;
    const size_t smem = (size_t)(2 * ((N + 3) & ~3) + cols) * sizeof(float);
    if (smem > 48 * 1024) return RG_ERR_UNSUPPORTED;
    dim3 grid(T, H, (dv + cols - 1) / cols);
    if (grid.z > 65535) return RG_ERR_UNSUPPORTED;
    const bool vec = N % 4 == 0 && ((uintptr_t)state & 15) == 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (vec)
        return rg_launch(ssd_step_kernel<true>, grid, dim3(SSD_THREADS), smem, s, 1, proj, ld, x_off, dt_off, taps, bias,
                         conv_state, dt_bias, A_log, D, state, req_of_token, start_pos, slots, o, H, G, N, dv, K, cols);
    return rg_launch(ssd_step_kernel<false>, grid, dim3(SSD_THREADS), smem, s, 1, proj, ld, x_off, dt_off, taps, bias,
                     conv_state, dt_bias, A_log, D, state, req_of_token, start_pos, slots, o, H, G, N, dv, K, cols);
}

// o [T, n] float; z: rows z_ld apart (type Z).  One block per (token, group of n / groups numbers); the gated numbers
// wait in shared memory for the group's root mean square.  With `raw` (rows raw_ld apart, C numbers) further blocks of
// the same launch move the convolution state of the token's request on by that one token (single-token steps).
template <typename Z, typename O>
__global__ void gate_group_norm_kernel(const float* __restrict__ o, const Z* __restrict__ z, int z_ld,
                                       const float* __restrict__ weight, float eps, O* __restrict__ out, int n, int gs,
                                       int groups, const float* __restrict__ raw, int raw_ld,
                                       float* __restrict__ conv_state, const int* __restrict__ req_of_token,
                                       const int* __restrict__ start_pos, const int* __restrict__ slots, int C, int K) {
    extern __shared__ __align__(16) float y[];        // [gs]
    __shared__ float scratch[33];
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x;
    if ((int)blockIdx.y >= groups) {
        const int c = (blockIdx.y - groups) * blockDim.x + threadIdx.x;
        const int r = req_of_token[t], slot = slots[r];
        if (slot < 0 || c >= C) return;
        const bool has_past = start_pos[r] > 0;
        float* st = conv_state + (size_t)slot * (K - 1) * C + c;
        const float now = raw[(size_t)t * raw_ld + c];
        for (int j0 = 0; j0 < K - 2; j0 += 4) {       // four rows at a time, each read before the one above it is written
            float v[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) v[j] = has_past && j0 + j < K - 2 ? st[(size_t)(j0 + j + 1) * C] : 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (j0 + j < K - 2) st[(size_t)(j0 + j) * C] = v[j];
        }
        st[(size_t)(K - 2) * C] = now;
        return;
    }
    const int base = blockIdx.y * gs;
    const float* src = o + (size_t)t * n + base;
    const Z* zr = z + (size_t)t * z_ld + base;
    float ss = 0.f;
    for (int i = threadIdx.x; i < gs; i += blockDim.x) {
        const float v = src[i] * ssd_silu(to_f32(zr[i]));
        y[i] = v;
        ss += v * v;
    }
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)gs + eps);
    for (int i = threadIdx.x; i < gs; i += blockDim.x)
        out[(size_t)t * n + base + i] = from_f32<O>(y[i] * inv * weight[base + i]);
}

extern "C" int rg_gate_group_norm(const float* o, const void* z, int z_dtype, int z_ld, const float* weight, float eps,
                                  void* out, int out_dtype, int T, int n, int groups, const float* raw, int raw_ld,
                                  float* conv_state, const int* req_of_token, const int* start_pos, const int* slots, int C,
                                  int K, void* stream) {
    if (T <= 0) return 0;
    if (n < 1 || groups < 1 || n % groups || groups > 65535 || (raw && K > 1 && !conv_state)) return RG_ERR_UNSUPPORTED;
    const int gs = n / groups;
    const size_t smem = (size_t)gs * sizeof(float);
    if (smem > 200 * 1024) return RG_ERR_UNSUPPORTED;
    int threads = 64;
    while (threads < 512 && threads * 4 < gs) threads <<= 1;
    const int conv_blocks = raw && K > 1 ? (C + threads - 1) / threads : 0;
    if (groups + conv_blocks > 65535) return RG_ERR_UNSUPPORTED;
    dim3 grid(T, groups + conv_blocks);
    cudaStream_t s = (cudaStream_t)stream;
#define SSD_GGN(Z, O) { if (smem > 47 * 1024) { \
            const int e = (int)cudaFuncSetAttribute(gate_group_norm_kernel<Z, O>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e) return e; } \
        return rg_launch(gate_group_norm_kernel<Z, O>, grid, dim3(threads), smem, s, 1, o, (const Z*)z, z_ld, weight, eps, \
                         (O*)out, n, gs, groups, raw, raw_ld, conv_state, req_of_token, start_pos, slots, C, K); }
    if (z_dtype == RG_DTYPE_BF16 && out_dtype == RG_DTYPE_BF16) SSD_GGN(bf16, bf16)
    if (z_dtype == RG_DTYPE_F32 && out_dtype == RG_DTYPE_BF16) SSD_GGN(float, bf16)
    if (z_dtype == RG_DTYPE_F32 && out_dtype == RG_DTYPE_F32) SSD_GGN(float, float)
#undef SSD_GGN
    return RG_ERR_UNSUPPORTED;
}
