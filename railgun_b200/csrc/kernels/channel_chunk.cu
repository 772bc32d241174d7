// The recurrence with a decay per token and key channel over portions of prompts, in chunks of 64 tokens side by side:
//
//   o_t = (S + diag(u) k_t v_t^T)^T r_t;   S <- diag(w_t) S + k_t v_t^T
//
// Inside a chunk of L tokens, with S the state before it and W(a, b) the product of w_s over a < s < b, channel by channel,
//   o_i   = S^T (W(0, i) r_i) + sum_(j < i) (r_i . W(j, i) k_j) v_j + (r_i . u k_i) v_i
//   S_end = diag(W(0, L + 1)) S + sum_j (W(j, L + 1) k_j) v_j^T
// All W are products of at most 63 decays between 0 and 1, formed by multiplication alone (a quotient of two of them, or
// a difference of their logarithms, would fail where a channel forgets at once).  Five kernels:
//   channel_rows     per (chunk, channel): W(0, i) r_i, W(j, L + 1) k_j and W(0, L + 1)
//   channel_dots     per (chunk, head): the numbers r_i . W(j, i) k_j and r_i . u k_i
//   channel_states   per (chunk, head): the sum in S_end
//   chunk_pass       S before every chunk, and the last one into the request's slot
//   channel_outputs  per (chunk, head): o
#include "chunk_scan.cuh"

// r, k, w: rows r_ld, k_ld, w_ld apart, n = H d channels.  q_out, k_out [T, n]; decays [chunks, n].  One thread per channel.
__global__ void channel_rows_kernel(const float* __restrict__ r, int r_ld, const float* __restrict__ k, int k_ld,
                                    const float* __restrict__ w, int w_ld, const int* __restrict__ cu, int R,
                                    float* __restrict__ q_out, float* __restrict__ k_out, float* __restrict__ decays, int n) {
    pdl_wait();
    pdl_trigger();
    int rq, lo, len;
    if (!find_chunk(cu, R, blockIdx.x, rq, lo, len)) return;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= n) return;
    float p = 1.f;
#pragma unroll 8
    for (int i = 0; i < len; ++i) {
        const size_t t = lo + i;
        q_out[t * n + c] = r[t * r_ld + c] * p;
        p *= w[t * w_ld + c];
    }
    decays[(size_t)blockIdx.x * n + c] = p;
    p = 1.f;
#pragma unroll 8
    for (int i = len - 1; i >= 0; --i) {
        const size_t t = lo + i;
        k_out[t * n + c] = k[t * k_ld + c] * p;
        p *= w[t * w_ld + c];
    }
}

// Sums of four numbers over a warp with six shuffles: lane 8 x holds the sum of s[x].
__device__ __forceinline__ float warp_sum4(const float (&s)[4], int lane) {
    const bool hi = lane & 16, odd = lane & 8;
    float a = hi ? s[2] : s[0], b = hi ? s[3] : s[1];
    a += __shfl_xor_sync(0xffffffffu, hi ? s[0] : s[2], 16);
    b += __shfl_xor_sync(0xffffffffu, hi ? s[1] : s[3], 16);
    float c = odd ? b : a;
    c += __shfl_xor_sync(0xffffffffu, odd ? a : b, 8);
    c += __shfl_xor_sync(0xffffffffu, c, 4);
    c += __shfl_xor_sync(0xffffffffu, c, 2);
    return c + __shfl_xor_sync(0xffffffffu, c, 1);
}

// dots [chunks, H, 64, 64] at [j][i], j <= i.  A warp takes four tokens j at a time (from both ends of the chunk in turn:
// equal work together), their keys decayed on the way in registers (channel q of a lane: lane + 32 q), against every later r_i.
// grid: chunks, H, 2 halves of 4 warps.
#define DOT_THREADS 128
template <int NQ>
__global__ void __launch_bounds__(DOT_THREADS)
channel_dots_kernel(const float* __restrict__ r, int r_ld, const float* __restrict__ k, int k_ld, const float* __restrict__ w,
                    int w_ld, const float* __restrict__ bonus, const int* __restrict__ cu, int R, float* __restrict__ dots,
                    int H, int d) {
    pdl_wait();
    pdl_trigger();
    int rq, lo, n;
    if (!find_chunk(cu, R, blockIdx.x, rq, lo, n)) return;
    const int h = blockIdx.y, lane = threadIdx.x & 31, first = blockIdx.z * (DOT_THREADS / 32) + (threadIdx.x >> 5);
    float* out = dots + ((size_t)blockIdx.x * H + h) * CH * CH + (lane >> 3) * CH;
    const bool writes = (lane & 7) == 0;
    const float *rh = r + (size_t)lo * r_ld + (size_t)h * d, *kh = k + (size_t)lo * k_ld + (size_t)h * d,
                *wh = w + (size_t)lo * w_ld + (size_t)h * d, *uh = bonus + (size_t)h * d;
    auto row = [&](const float* p, int ld, int i, float (&x)[NQ]) {
#pragma unroll
        for (int q = 0; q < NQ; ++q) x[q] = lane + 32 * q < d ? p[(size_t)i * ld + lane + 32 * q] : 0.f;
    };
    for (int half = 0; half < 2; ++half) {
        const int j0 = 4 * (half ? CH / 4 - 1 - first : first);
        if (j0 >= n) continue;
        float kp[4][NQ];
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int q = 0; q < NQ; ++q) kp[x][q] = 0.f;
        // the four tokens themselves: a token's own number has the bonus, and its key joins undecayed
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            const int i = j0 + a;
            if (i >= n) break;
            float rv[NQ], wv[NQ], kv[NQ], s[4] = {0.f, 0.f, 0.f, 0.f};
            row(rh, r_ld, i, rv);
            row(wh, w_ld, i, wv);
            row(kh, k_ld, i, kv);
#pragma unroll
            for (int q = 0; q < NQ; ++q) {
#pragma unroll
                for (int x = 0; x < a; ++x) {
                    s[x] += rv[q] * kp[x][q];
                    kp[x][q] *= wv[q];
                }
                s[a] += rv[q] * (lane + 32 * q < d ? uh[lane + 32 * q] : 0.f) * kv[q];
                kp[a][q] = kv[q];
            }
            const float c = warp_sum4(s, lane);
            if (writes && (lane >> 3) <= a) out[j0 * CH + i] = c;
        }
#pragma unroll 2
        for (int i = j0 + 4; i < n; ++i) {
            float rv[NQ], wv[NQ], s[4] = {0.f, 0.f, 0.f, 0.f};
            row(rh, r_ld, i, rv);
            row(wh, w_ld, i, wv);
#pragma unroll
            for (int q = 0; q < NQ; ++q)
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    s[x] += rv[q] * kp[x][q];
                    kp[x][q] *= wv[q];
                }
            const float c = warp_sum4(s, lane);
            if (writes) out[j0 * CH + i] = c;
        }
    }
}

// kd [T, H d]: the decayed keys.  v: rows v_ld apart, head h at column h dv.  sums [chunks, H, dv, d].  grid: chunks, H,
// tiles of S.
template <int W>
__global__ void __launch_bounds__(NTH)
channel_states_kernel(const float* __restrict__ kd, const float* __restrict__ v, int v_ld, const int* __restrict__ cu, int R,
                      float* __restrict__ sums, int H, int d, int dv, int ntiles) {
    extern __shared__ __align__(16) float sm[];
    float (*sA)[PITCH] = reinterpret_cast<float (*)[PITCH]>(sm);
    float (*sB)[TILE * W + 4] = reinterpret_cast<float (*)[TILE * W + 4]>(sm + CH * PITCH);
    pdl_wait();
    pdl_trigger();
    int rq, lo, n;
    if (!find_chunk(cu, R, blockIdx.x, rq, lo, n)) return;
    const int h = blockIdx.y;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const int j0 = (blockIdx.z / ntiles) * TILE, n0 = (blockIdx.z % ntiles) * TILE * W;
    float acc[4][4 * W];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4 * W; ++j) acc[i][j] = 0.f;
    for (int e = threadIdx.x; e < CH * TILE; e += NTH) {
        const int t = e / TILE, j = e - t * TILE;
        sA[t][j] = t < n && j0 + j < dv ? v[(size_t)(lo + t) * v_ld + (size_t)h * dv + j0 + j] : 0.f;
    }
    for (int e = threadIdx.x; e < CH * TILE * W; e += NTH) {
        const int t = e / (TILE * W), c = e - t * TILE * W;
        sB[t][c] = t < n && n0 + c < d ? kd[((size_t)(lo + t) * H + h) * d + n0 + c] : 0.f;
    }
    __syncthreads();
    multiply<W>(acc, sA, sB, n, ty, tx);
    float* out = sums + ((size_t)blockIdx.x * H + h) * dv * d;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int j = j0 + 4 * ty + i;
        if (j >= dv) continue;
#pragma unroll
        for (int x = 0; x < W; ++x) {
            const int c = n0 + TILE * x + 4 * tx;
            if (d % 4 == 0) {
                if (c < d) *reinterpret_cast<float4*>(out + (size_t)j * d + c) =
                    make_float4(acc[i][4 * x], acc[i][4 * x + 1], acc[i][4 * x + 2], acc[i][4 * x + 3]);
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (c + q < d) out[(size_t)j * d + c + q] = acc[i][4 * x + q];
            }
        }
    }
}

// qd [T, H d]: the decayed queries; before [chunks, H, dv, d].  o [T, H, dv].  grid: chunks, H, tiles of 64 columns.
__global__ void __launch_bounds__(NTH)
channel_outputs_kernel(const float* __restrict__ qd, const float* __restrict__ v, int v_ld, const int* __restrict__ cu, int R,
                       const float* __restrict__ before, const float* __restrict__ dots, float* __restrict__ o, int H, int d,
                       int dv) {
    __shared__ __align__(16) float sA[CH][PITCH];
    __shared__ __align__(16) float sB[CH][PITCH];
    pdl_wait();
    pdl_trigger();
    int rq, lo, n;
    if (!find_chunk(cu, R, blockIdx.x, rq, lo, n)) return;
    const int h = blockIdx.y, j0 = blockIdx.z * TILE;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const float* m = dots + ((size_t)blockIdx.x * H + h) * CH * CH;
    for (int e = threadIdx.x; e < CH * CH; e += NTH) {
        const int j = e / CH, i = e - j * CH;
        sA[j][i] = j <= i && i < n ? m[e] : 0.f;
    }
    for (int e = threadIdx.x; e < CH * TILE; e += NTH) {
        const int t = e / TILE, j = e - t * TILE;
        sB[t][j] = t < n && j0 + j < dv ? v[(size_t)(lo + t) * v_ld + (size_t)h * dv + j0 + j] : 0.f;
    }
    __syncthreads();
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    multiply<1>(acc, sA, sB, min(n, 4 * (ty | 1) + 4), ty, tx);     // token j counts for the tokens from j on only
    const float* S = before + (((size_t)blockIdx.x * H + h) * dv + j0) * d;
    for (int k0 = 0; k0 < d; k0 += TILE) {
        __syncthreads();
        load_transposed(sA, qd + ((size_t)lo * H + h) * d, (size_t)H * d, n, d, k0, nullptr);
        load_transposed(sB, S, d, min(TILE, dv - j0), d, k0, nullptr);
        __syncthreads();
        multiply<1>(acc, sA, sB, min(TILE, d - k0), ty, tx);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        if (t >= n) continue;
        float* out = o + ((size_t)(lo + t) * H + h) * dv + j0 + 4 * tx;
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (j0 + 4 * tx + j < dv) out[j] = acc[i][j];
    }
}

// Scratch of the caller: qd, kd [T, H d], sums [chunks, H, dv, d], decays [chunks, H d], dots [chunks, H, 64, 64], with chunks
// at least T / 64 + R (rounded down).
extern "C" int rg_channel_chunk_scan(const float* r, int r_ld, const float* k, int k_ld, const float* v, int v_ld,
                                     const float* w, int w_ld, const float* bonus, float* state, const int* cu_seqlens,
                                     const int* start_pos, const int* slots, float* qd, float* kd, float* sums, float* decays,
                                     float* dots, float* o, int T, int R, int H, int d, int dv, void* stream) {
    if (T <= 0 || R <= 0) return 0;
    if (H < 1 || d < 1 || d > 256 || dv < 1 || H > 65535 || R > 65535) return RG_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const int chunks = T / CH + R, n = H * d;
    dim3 g0(chunks, (n + 127) / 128);
    if (g0.y > 65535) return RG_ERR_UNSUPPORTED;
    int e = rg_launch(channel_rows_kernel, g0, dim3(128), 0, s, 1, r, r_ld, k, k_ld, w, w_ld, cu_seqlens, R, qd, kd, decays, n);
    if (e) return e;
    dim3 gd(chunks, H, CH / 4 / 2 / (DOT_THREADS / 32));
#define CH_DOTS(NQ) e = rg_launch(channel_dots_kernel<NQ>, gd, dim3(DOT_THREADS), 0, s, 1, r, r_ld, k, k_ld, w, w_ld, bonus, \
                                  cu_seqlens, R, dots, H, d)
    if (d <= 32) CH_DOTS(1); else if (d <= 64) CH_DOTS(2); else if (d <= 128) CH_DOTS(4); else CH_DOTS(8);
#undef CH_DOTS
    if (e) return e;
    const int wide = d > TILE ? 2 : 1;
    const int jt = (dv + TILE - 1) / TILE, nt = (d + TILE * wide - 1) / (TILE * wide);
    if (jt * nt > 65535) return RG_ERR_UNSUPPORTED;
    dim3 g1(chunks, H, jt * nt);
    const size_t smem = (size_t)CH * (PITCH + TILE * wide + 4) * sizeof(float);
#define CH_STATES(W) { \
        if (smem > 46 * 1024) e = (int)cudaFuncSetAttribute(channel_states_kernel<W>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e == 0) e = rg_launch(channel_states_kernel<W>, g1, dim3(NTH), smem, s, 1, (const float*)kd, v, v_ld, cu_seqlens, \
                                  R, sums, H, d, dv, nt); }
    if (wide == 2) CH_STATES(2) else CH_STATES(1)
#undef CH_STATES
    if (e) return e;
    const int M = dv * d;
    const bool vec = d % 4 == 0 && ((uintptr_t)state & 15) == 0;
    const long long work = vec ? (long long)H * M / 4 : (long long)H * M;
    dim3 g2((unsigned)((work + 255) / 256), R);
    e = vec ? rg_launch(chunk_pass_kernel<4, true>, g2, dim3(256), 0, s, 1, sums, (const float*)decays, state, cu_seqlens,
                        start_pos, slots, H, M, d)
            : rg_launch(chunk_pass_kernel<1, true>, g2, dim3(256), 0, s, 1, sums, (const float*)decays, state, cu_seqlens,
                        start_pos, slots, H, M, d);
    if (e) return e;
    dim3 g3(chunks, H, jt);
    return rg_launch(channel_outputs_kernel, g3, dim3(NTH), 0, s, 1, (const float*)qd, v, v_ld, cu_seqlens, R,
                     (const float*)sums, (const float*)dots, o, H, d, dv);
}
