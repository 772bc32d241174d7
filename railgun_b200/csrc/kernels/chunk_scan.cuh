// What the chunked forms of the matrix-state recurrences share: a step's tokens, packed request by request (cu_seqlens),
// cut into chunks of 64 that start at each request's first token of the step; 64 x 64 (x 128) products in 32-bit fused
// multiply-adds; and the pass from chunk to chunk.
#pragma once
#include "common.cuh"

#define CH 64                 // tokens per chunk
#define TILE 64               // rows and columns of a block's output (columns: 64 or 128)
#define PITCH (TILE + 4)
#define NTH 256

// Chunk number c of the step: its request, first token and number of tokens; false beyond the last one.
__device__ __forceinline__ bool find_chunk(const int* __restrict__ cu, int R, int c, int& r, int& lo, int& n) {
    for (r = 0; r < R; ++r) {
        const int len = cu[r + 1] - cu[r], k = (len + CH - 1) / CH;
        if (c < k) {
            lo = cu[r] + c * CH;
            n = min(CH, len - c * CH);
            return true;
        }
        c -= k;
    }
    return false;
}

// dst[k][i] = src row i, number k0 + k (rows ld apart, n rows of N numbers; zeros elsewhere), for 64 x 64, times scale[i].
// A warp reads 4 rows x 8 neighbouring numbers at a time and writes 32 different banks.
__device__ __forceinline__ void load_transposed(float (*__restrict__ dst)[PITCH], const float* __restrict__ src, size_t ld,
                                                int n, int N, int k0, const float* __restrict__ scale) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int kl = lane & 7, il = lane >> 3;
#pragma unroll 4
    for (int p = warp; p < (TILE / 8) * (TILE / 4); p += NTH / 32) {
        const int k = (p & 7) * 8 + kl, i = (p >> 3) * 4 + il;
        float v = i < n && k0 + k < N ? src[(size_t)i * ld + k0 + k] : 0.f;
        if (scale) v *= scale[i];
        dst[k][i] = v;
    }
}

// acc[4][4 W] += A[k][4 rows]^T B[k][4 W columns] over kn values of k.  Thread (ty, tx): rows 4 ty .., columns 4 tx .. (+ 64)
template <int W>
__device__ __forceinline__ void multiply(float (&acc)[4][4 * W], const float (*__restrict__ A)[PITCH],
                                         const float (*__restrict__ B)[TILE * W + 4], int kn, int ty, int tx) {
#pragma unroll 4
    for (int k = 0; k < kn; ++k) {
        const float4 a = *reinterpret_cast<const float4*>(&A[k][4 * ty]);
#pragma unroll
        for (int w = 0; w < W; ++w) {
            const float4 b = *reinterpret_cast<const float4*>(&B[k][TILE * w + 4 * tx]);
            acc[0][4 * w] += a.x * b.x; acc[0][4 * w + 1] += a.x * b.y; acc[0][4 * w + 2] += a.x * b.z; acc[0][4 * w + 3] += a.x * b.w;
            acc[1][4 * w] += a.y * b.x; acc[1][4 * w + 1] += a.y * b.y; acc[1][4 * w + 2] += a.y * b.z; acc[1][4 * w + 3] += a.y * b.w;
            acc[2][4 * w] += a.z * b.x; acc[2][4 * w + 1] += a.z * b.y; acc[2][4 * w + 2] += a.z * b.z; acc[2][4 * w + 3] += a.z * b.w;
            acc[3][4 * w] += a.w * b.x; acc[3][4 * w + 1] += a.w * b.y; acc[3][4 * w + 2] += a.w * b.z; acc[3][4 * w + 3] += a.w * b.w;
        }
    }
}

// sums [chunks, H, M]: each chunk's sum becomes the state before the chunk, and the state after the last one goes into the
// request's slot (M = dv d numbers per head, S transposed).  decays [chunks, H], or with CHANNEL [chunks, H, d]: one per
// row of S.  V numbers per thread (with CHANNEL neighbours in a column of S: d % V == 0).
template <int V, bool CHANNEL>
__global__ void chunk_pass_kernel(float* __restrict__ sums, const float* __restrict__ decays, float* __restrict__ state,
                                  const int* __restrict__ cu, const int* __restrict__ start_pos,
                                  const int* __restrict__ slots, int H, int M, int d) {
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.y;
    const long long e = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (e >= (long long)H * M) return;
    const int h = (int)(e / M);
    int c0 = 0;
    for (int q = 0; q < r; ++q) c0 += (cu[q + 1] - cu[q] + CH - 1) / CH;
    const int nc = (cu[r + 1] - cu[r] + CH - 1) / CH;
    const int slot = slots[r];
    float S[V];
#pragma unroll
    for (int i = 0; i < V; ++i) S[i] = 0.f;
    float* st = state + (size_t)(slot >= 0 ? slot : 0) * H * M + e;
    if (slot >= 0 && start_pos[r] > 0) {
#pragma unroll
        for (int i = 0; i < V; ++i) S[i] = st[i];
    }
    float* p = sums + (size_t)c0 * H * M + e;
    const float* dec = CHANNEL ? decays + (size_t)c0 * H * d + (size_t)h * d + (e - (long long)h * M) % d
                               : decays + (size_t)c0 * H + h;
    const size_t dec_step = CHANNEL ? (size_t)H * d : (size_t)H;
    const size_t step = (size_t)H * M;
    constexpr int U = 4;                              // chunks in flight
    for (int c = 0; c < nc; c += U) {
        float u[U][V], g[U][V];
#pragma unroll
        for (int k = 0; k < U; ++k) {
            if (c + k < nc) {
#pragma unroll
                for (int i = 0; i < V; ++i) g[k][i] = dec[(c + k) * dec_step + (CHANNEL ? i : 0)];
                if (V == 4) {
                    const float4 q = *reinterpret_cast<const float4*>(p + (c + k) * step);
                    u[k][0] = q.x; u[k][1 % V] = q.y; u[k][2 % V] = q.z; u[k][3 % V] = q.w;
                } else {
                    u[k][0] = p[(c + k) * step];
                }
            }
        }
#pragma unroll
        for (int k = 0; k < U; ++k) {
            if (c + k < nc) {
                if (V == 4) *reinterpret_cast<float4*>(p + (c + k) * step) = make_float4(S[0], S[1 % V], S[2 % V], S[3 % V]);
                else p[(c + k) * step] = S[0];
#pragma unroll
                for (int i = 0; i < V; ++i) S[i] = S[i] * g[k][i] + u[k][i];
            }
        }
    }
    if (slot >= 0) {
#pragma unroll
        for (int i = 0; i < V; ++i) st[i] = S[i];
    }
}
