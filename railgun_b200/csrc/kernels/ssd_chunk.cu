// The recurrence of Mamba-2 over portions of prompts, in chunks of 64 tokens side by side instead of token by token:
//
//   S <- g_t S + dt_t B_t x_t^T,  o_t = S^T C_t + D x_t,   g_t = exp(a_t),  a_t = -exp(A_log) dt_t
//
// With c_i = a_1 + .. + a_i inside a chunk of L tokens and S the state before it,
//   o_i   = exp(c_i) S^T C_i + sum_(j <= i) exp(c_i - c_j) dt_j (B_j . C_i) x_j + D x_i
//   S_end = exp(c_L) S + sum_j exp(c_L - c_j) dt_j B_j x_j^T
// so that everything but the pass from chunk to chunk is products.  Three kernels:
//   chunk_states   per (chunk, head): the sum in S_end, and exp(c_L); per (chunk, group): all B_j . C_i
//   chunk_pass     per (request, head, number of S): S before every chunk, and the last one into the request's slot
//   chunk_outputs  per (chunk, head): o
// (the block decomposition of Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through
// Structured State Space Duality").  The products are 32-bit fused multiply-adds; the exponents' sums are 64-bit, since
// their differences are small beside them where a head forgets fast.
//
// The same recurrence with the logarithm of every token's decay given instead of A_log and dt (then dt holds the weights of
// the new terms only), without D, and with n, the sum of the B's with the same decays and weights, carried as one more
// row of the state ("ones": the column of a value that is always 1), for memories that divide by n . C.  n and n . C are
// sums that the light blocks of the launches work out.
//
// The step's tokens are packed request by request (cu_seqlens); a request's chunks start at its first token of the step.
#include "chunk_scan.cuh"

// c_i of the chunk's tokens for head h (64-bit), by the block's first warp; dt of the tokens into sdt.  a_t is loga's
// number, or without loga -exp(A_log) dt_t.
__device__ __forceinline__ void chunk_sums(const float* __restrict__ dt, const float* __restrict__ loga,
                                           const float* __restrict__ A_log, int lo, int n, int H, int h,
                                           double* __restrict__ cum, float* __restrict__ sdt) {
    if (threadIdx.x < 32) {
        const int i0 = 2 * threadIdx.x, i1 = i0 + 1;
        const float d0 = i0 < n ? dt[(size_t)(lo + i0) * H + h] : 0.f, d1 = i1 < n ? dt[(size_t)(lo + i1) * H + h] : 0.f;
        double a0, a1;
        if (loga) {
            a0 = i0 < n ? (double)loga[(size_t)(lo + i0) * H + h] : 0.0;
            a1 = i1 < n ? (double)loga[(size_t)(lo + i1) * H + h] : 0.0;
        } else {
            const float rate = -expf(A_log[h]);
            a0 = (double)(rate * d0);
            a1 = (double)(rate * d1);
        }
        double s = a0 + a1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, s, o);
            if ((int)threadIdx.x >= o) s += up;
        }
        cum[i0] = s - a1;
        cum[i1] = s;
        sdt[i0] = d0;
        sdt[i1] = d1;
    }
}

// x, B, C: rows ld apart (head h's x at column h dv, group g's B and C at column g N).  sums [chunks, H, dv + ones, N],
// decays [chunks, H], dots [chunks, G, 64, 64] = B_j . C_i at [j][i].  grid: chunks, H (tiles of S: z) and then G (z = 0).
template <int W>
__global__ void __launch_bounds__(NTH)
chunk_states_kernel(const float* __restrict__ x, const float* __restrict__ B, const float* __restrict__ C, int ld,
                    const float* __restrict__ dt, const float* __restrict__ loga, const float* __restrict__ A_log,
                    const int* __restrict__ cu, int R, float* __restrict__ sums, float* __restrict__ decays,
                    float* __restrict__ dots, int H, int G, int N, int dv, int ntiles, int ones) {
    extern __shared__ __align__(16) float sm[];
    float (*sA)[PITCH] = reinterpret_cast<float (*)[PITCH]>(sm);                            // [CH][PITCH]
    float (*sB)[TILE * W + 4] = reinterpret_cast<float (*)[TILE * W + 4]>(sm + CH * PITCH);     // [CH][TILE W + 4]
    __shared__ double cum[CH];
    __shared__ float sdt[CH];
    pdl_wait();
    pdl_trigger();
    int r, lo, n;
    if (!find_chunk(cu, R, blockIdx.x, r, lo, n)) return;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float acc[4][4 * W];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4 * W; ++j) acc[i][j] = 0.f;
    if ((int)blockIdx.y >= H) {
        if (blockIdx.z > 0) return;
        const int g = blockIdx.y - H;
        float (*sC)[PITCH] = reinterpret_cast<float (*)[PITCH]>(sm + CH * PITCH);
        float a1[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) a1[i][j] = 0.f;
        for (int k0 = 0; k0 < N; k0 += TILE) {
            load_transposed(sA, B + (size_t)lo * ld + (size_t)g * N, ld, n, N, k0, nullptr);
            load_transposed(sC, C + (size_t)lo * ld + (size_t)g * N, ld, n, N, k0, nullptr);
            __syncthreads();
            multiply<1>(a1, sA, sC, min(TILE, N - k0), ty, tx);
            __syncthreads();
        }
        float* out = dots + ((size_t)blockIdx.x * G + g) * CH * CH;
#pragma unroll
        for (int i = 0; i < 4; ++i)
            *reinterpret_cast<float4*>(out + (4 * ty + i) * CH + 4 * tx) = make_float4(a1[i][0], a1[i][1], a1[i][2], a1[i][3]);
        if (!ones) return;
        for (int h = g * (H / G); h < (g + 1) * (H / G); ++h) {         // the row of n: every head of the group
            __syncthreads();
            chunk_sums(dt, loga, A_log, lo, n, H, h, cum, sdt);
            __syncthreads();
            const double last = cum[CH - 1];
            __syncthreads();
            if (threadIdx.x < n) sdt[threadIdx.x] *= expf((float)(last - cum[threadIdx.x]));
            __syncthreads();
            for (int k = threadIdx.x; k < N; k += NTH) {
                float s = 0.f;
#pragma unroll 8
                for (int t = 0; t < n; ++t) s += B[(size_t)(lo + t) * ld + (size_t)g * N + k] * sdt[t];
                sums[(((size_t)blockIdx.x * H + h) * (dv + 1) + dv) * N + k] = s;
            }
        }
        return;
    }
    const int h = blockIdx.y, grp = h / (H / G);
    const int j0 = (blockIdx.z / ntiles) * TILE, n0 = (blockIdx.z % ntiles) * TILE * W;      // columns of S, rows of S
    chunk_sums(dt, loga, A_log, lo, n, H, h, cum, sdt);
    __syncthreads();
    const double end = cum[CH - 1];
    for (int e = threadIdx.x; e < CH * TILE; e += NTH) {
        const int t = e / TILE, j = e - t * TILE;
        sA[t][j] = t < n && j0 + j < dv
                       ? x[(size_t)(lo + t) * ld + (size_t)h * dv + j0 + j] * sdt[t] * expf((float)(end - cum[t])) : 0.f;
    }
    for (int e = threadIdx.x; e < CH * TILE * W; e += NTH) {
        const int t = e / (TILE * W), k = e - t * TILE * W;
        sB[t][k] = t < n && n0 + k < N ? B[(size_t)(lo + t) * ld + (size_t)grp * N + n0 + k] : 0.f;
    }
    __syncthreads();
    multiply<W>(acc, sA, sB, n, ty, tx);
    float* out = sums + ((size_t)blockIdx.x * H + h) * (dv + ones) * N;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int j = j0 + 4 * ty + i;
        if (j >= dv) continue;
#pragma unroll
        for (int w = 0; w < W; ++w) {
            const int k = n0 + TILE * w + 4 * tx;
            if (N % 4 == 0) {
                if (k < N) *reinterpret_cast<float4*>(out + (size_t)j * N + k) =
                    make_float4(acc[i][4 * w], acc[i][4 * w + 1], acc[i][4 * w + 2], acc[i][4 * w + 3]);
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (k + q < N) out[(size_t)j * N + k + q] = acc[i][4 * w + q];
            }
        }
    }
    if (blockIdx.z == 0 && threadIdx.x == 0) decays[(size_t)blockIdx.x * H + h] = expf((float)end);
}

// before [chunks, H, dv + ones, N]: the state before every chunk.  o [T, H, dv + ones].  grid: chunks, H, tiles of 64
// columns, and with `ones` a light block for n . C.
__global__ void __launch_bounds__(NTH)
chunk_outputs_kernel(const float* __restrict__ x, const float* __restrict__ C, int ld, const float* __restrict__ dt,
                     const float* __restrict__ loga, const float* __restrict__ A_log, const float* __restrict__ D,
                     const int* __restrict__ cu, int R, const float* __restrict__ before, const float* __restrict__ dots,
                     float* __restrict__ o, int H, int G, int N, int dv, int ones) {
    __shared__ __align__(16) float sA[CH][PITCH];
    __shared__ __align__(16) float sB[CH][PITCH];
    __shared__ double cum[CH];
    __shared__ float sdt[CH], grown[CH];
    pdl_wait();
    pdl_trigger();
    int r, lo, n;
    if (!find_chunk(cu, R, blockIdx.x, r, lo, n)) return;
    const int h = blockIdx.y, grp = h / (H / G), j0 = blockIdx.z * TILE;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    chunk_sums(dt, loga, A_log, lo, n, H, h, cum, sdt);
    __syncthreads();
    if (j0 >= dv) {
        // n . C_i: four threads a token (neighbouring lanes) share its sums over the chunk's tokens and over n's numbers
        const float* dd = dots + ((size_t)blockIdx.x * G + grp) * CH * CH;
        const float* nb = before + (((size_t)blockIdx.x * H + h) * (dv + 1) + dv) * N;
        const int i = threadIdx.x >> 2, part = threadIdx.x & 3;
        float s = 0.f, b = 0.f;
        if (i < n) {
            const float* c = C + (size_t)(lo + i) * ld + (size_t)grp * N;
            for (int j = part; j <= i; j += 4) s += dd[j * CH + i] * sdt[j] * expf((float)(cum[i] - cum[j]));
            for (int k = part; k < N; k += 4) b += nb[k] * c[k];
            s += b * expf((float)cum[i]);
        }
        s += __shfl_xor_sync(0xffffffffu, s, 1);
        s += __shfl_xor_sync(0xffffffffu, s, 2);
        if (i < n && part == 0) o[((size_t)(lo + i) * H + h) * (dv + 1) + dv] = s;
        return;
    }
    if (threadIdx.x < CH) grown[threadIdx.x] = expf((float)cum[threadIdx.x]);
    // within the chunk
    const float* d = dots + ((size_t)blockIdx.x * G + grp) * CH * CH;
    for (int e = threadIdx.x; e < CH * CH; e += NTH) {
        const int j = e / CH, i = e - j * CH;
        sA[j][i] = j <= i && i < n ? d[e] * sdt[j] * expf((float)(cum[i] - cum[j])) : 0.f;
    }
    for (int e = threadIdx.x; e < CH * TILE; e += NTH) {
        const int t = e / TILE, j = e - t * TILE;
        sB[t][j] = t < n && j0 + j < dv ? x[(size_t)(lo + t) * ld + (size_t)h * dv + j0 + j] : 0.f;
    }
    __syncthreads();
    float acc[4][4];
    const float skip = D ? D[h] : 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = skip * sB[4 * ty + i][4 * tx + j];
    multiply<1>(acc, sA, sB, min(n, 4 * (ty | 1) + 4), ty, tx);     // token j counts for the tokens from j on only
    // from the state before it
    const float* S = before + (((size_t)blockIdx.x * H + h) * (dv + ones) + j0) * N;
    for (int k0 = 0; k0 < N; k0 += TILE) {
        __syncthreads();
        load_transposed(sA, C + (size_t)lo * ld + (size_t)grp * N, ld, n, N, k0, grown);
        load_transposed(sB, S, N, min(TILE, dv - j0), N, k0, nullptr);
        __syncthreads();
        multiply<1>(acc, sA, sB, min(TILE, N - k0), ty, tx);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        if (t >= n) continue;
        float* out = o + ((size_t)(lo + t) * H + h) * (dv + ones) + j0 + 4 * tx;
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (j0 + 4 * tx + j < dv) out[j] = acc[i][j];
    }
}

// loga [T, H] or null (then A_log [H]); D [H] or null.  state [slots, H, dv + ones, N].
// Scratch of the caller: sums [chunks, H, dv + ones, N], decays [chunks, H], dots [chunks, G, 64, 64], with chunks at least
// T / 64 + R (rounded down).
extern "C" int rg_ssd_chunk_scan(const float* x, const float* B, const float* C, int ld, const float* dt, const float* loga,
                                 const float* A_log, const float* D, float* state, const int* cu_seqlens, const int* start_pos,
                                 const int* slots, float* sums, float* decays, float* dots, float* o, int T, int R, int H,
                                 int G, int N, int dv, int ones, void* stream) {
    if (T <= 0 || R <= 0) return 0;
    if ((!loga && !A_log) || ones < 0 || ones > 1) return RG_ERR_UNSUPPORTED;
    if (H < 1 || G < 1 || H % G || N < 1 || dv < 1 || H + G > 65535 || R > 65535) return RG_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const int chunks = T / CH + R;
    const int wide = N > TILE ? 2 : 1;
    const int jt = (dv + TILE - 1) / TILE, nt = (N + TILE * wide - 1) / (TILE * wide);
    if (jt * nt > 65535) return RG_ERR_UNSUPPORTED;
    dim3 g1(chunks, H + G, jt * nt);
    const size_t smem = (size_t)CH * (PITCH + TILE * wide + 4) * sizeof(float);
    int e = 0;
#define SSD_STATES(W) { \
        if (smem > 46 * 1024) e = (int)cudaFuncSetAttribute(chunk_states_kernel<W>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e == 0) e = rg_launch(chunk_states_kernel<W>, g1, dim3(NTH), smem, s, 1, x, B, C, ld, dt, loga, A_log, \
                                  cu_seqlens, R, sums, decays, dots, H, G, N, dv, nt, ones); }
    if (wide == 2) SSD_STATES(2) else SSD_STATES(1)
#undef SSD_STATES
    if (e) return e;
    const int M = (dv + ones) * N;
    const bool vec = M % 4 == 0 && ((uintptr_t)state & 15) == 0;
    const long long work = vec ? (long long)H * M / 4 : (long long)H * M;
    dim3 g2((unsigned)((work + 255) / 256), R);
    e = vec ? rg_launch(chunk_pass_kernel<4, false>, g2, dim3(256), 0, s, 1, sums, (const float*)decays, state, cu_seqlens, start_pos, slots, H, M, N)
            : rg_launch(chunk_pass_kernel<1, false>, g2, dim3(256), 0, s, 1, sums, (const float*)decays, state, cu_seqlens, start_pos, slots, H, M, N);
    if (e) return e;
    dim3 g3(chunks, H, jt + ones);
    return rg_launch(chunk_outputs_kernel, g3, dim3(NTH), 0, s, 1, x, C, ld, dt, loga, A_log, D, cu_seqlens, R,
                     (const float*)sums, (const float*)dots, o, H, G, N, dv, ones);
}
