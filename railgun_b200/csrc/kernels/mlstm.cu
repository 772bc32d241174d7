// The matrix memory of xLSTM (Beck et al., "xLSTM: Extended Long Short-Term Memory") around its scan:
//
//   a = c(z_in), b = log sigmoid(c(z_forget)),  c(z) = cap tanh(z / cap)               per head
//   m' = max(m + b, a)                                                                 m = 0 where a sequence begins
//   [S | n] <- e^(m + b - m') [S | n] + e^(a - m') k [v | 1]^T
//   [y | y_n] = q^T [S | n],  out = y / (max(|y_n|, e^(-m')) + 1e-6)
//
// n is one more column of S: the column of a value that is always 1.  The state of a request is S transposed with n
// behind it, [H, dv + 1, d], and m, [H], all in 32-bit; a request whose start position is 0 begins from zeros whatever
// its slot holds.
//   mlstm_gates   portions: a, b and m of every token and head, and from them the factors of the two terms
//   mlstm_step    steps of single tokens: gates, S, n and S^T q, n . q in one kernel
//   mlstm_out     the division, the heads' norm with a weight of all heads' size, the sigmoid gate, one rounding
// The scan itself of portions is state_scan (state_mixers.cu) or ssd_chunk_scan (ssd_chunk.cu) with a column of ones.
#include "common.cuh"

__device__ __forceinline__ float ml_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_forget_gate(float z, float cap) {
    const float x = cap * tanhf(z / cap);
    return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

// raw: rows ld apart, the H raw input gates at i_off, the forget gates at f_off.  keep [T, H] (its logarithm with
// log_keep), put [T, H], m_out [T, H].  m [slots, H].  One block per (request, head), MG_SPAN tokens at a time: the gates'
// logarithms go into shared memory, every thread takes a run of tokens, the runs' composed steps m -> max(m + A, B) are
// scanned over the block, then every run is gone through again from its own first m.
#define MG_THREADS 256
#define MG_SPAN 4096
__global__ void __launch_bounds__(MG_THREADS)
mlstm_gates_kernel(const float* __restrict__ raw, int ld, int i_off, int f_off, const float* __restrict__ ib,
                   const float* __restrict__ fb, float cap, float* __restrict__ m, const int* __restrict__ cu_seqlens,
                   const int* __restrict__ start_pos, const int* __restrict__ slots, float* __restrict__ keep,
                   float* __restrict__ put, float* __restrict__ m_out, int H, int log_keep) {
    __shared__ float si[MG_SPAN + MG_SPAN / 32], sf[MG_SPAN + MG_SPAN / 32];   // a place unused after every 32: runs of 16 hit all banks
    __shared__ float wa[MG_THREADS / 32], wb[MG_THREADS / 32], carry;
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.x, h = blockIdx.y;
    const int lo = cu_seqlens[r], n = cu_seqlens[r + 1] - lo;
    if (n <= 0) return;
    const int slot = slots[r];
    const float bi = ib[h], bf = fb[h];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    auto at = [](int t) { return t + (t >> 5); };
    if (threadIdx.x == 0) carry = slot >= 0 && start_pos[r] > 0 ? m[(size_t)slot * H + h] : 0.f;
    for (int s0 = 0; s0 < n; s0 += MG_SPAN) {
        const int ns = min(MG_SPAN, n - s0);
        const float* row = raw + (size_t)(lo + s0) * ld + h;
#pragma unroll 4
        for (int t = threadIdx.x; t < ns; t += MG_THREADS) {
            const float zi = row[(size_t)t * ld + i_off], zf = row[(size_t)t * ld + f_off];
            si[at(t)] = ml_input_gate(zi + bi, cap);
            sf[at(t)] = ml_forget_gate(zf + bf, cap);
        }
        __syncthreads();
        const int run = (ns + MG_THREADS - 1) / MG_THREADS;
        const int t0 = min(ns, (int)threadIdx.x * run), t1 = min(ns, t0 + run);
        float a = 0.f, b = -INFINITY;
        for (int t = t0; t < t1; ++t) {
            const float f = sf[at(t)];
            a += f;
            b = fmaxf(b + f, si[at(t)]);
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float ua = __shfl_up_sync(0xffffffffu, a, o), ub = __shfl_up_sync(0xffffffffu, b, o);
            if (lane >= o) { b = fmaxf(ub + a, b); a += ua; }
        }
        if (lane == 31) { wa[warp] = a; wb[warp] = b; }
        __syncthreads();
        float mt = carry;                                  // m before this warp's runs
        for (int w = 0; w < warp; ++w) mt = fmaxf(wa[w] + mt, wb[w]);
        const float pa = __shfl_up_sync(0xffffffffu, a, 1), pb = __shfl_up_sync(0xffffffffu, b, 1);
        if (lane > 0) mt = fmaxf(pa + mt, pb);
        __syncthreads();                                   // carry has been read
        for (int t = t0; t < t1; ++t) {
            const float f = sf[at(t)], i = si[at(t)];
            const float now = fmaxf(f + mt, i);
            const float k = f + mt - now;
            const size_t to = (size_t)(lo + s0 + t) * H + h;
            keep[to] = log_keep ? k : expf(k);
            put[to] = expf(i - now);
            m_out[to] = now;
            mt = now;
        }
        if (t1 == ns && t0 < ns) carry = mt;
        __syncthreads();
    }
    if (slot >= 0 && threadIdx.x == 0) m[(size_t)slot * H + h] = carry;        // read at the start by this block only
}

extern "C" int rg_mlstm_gates(const float* raw, int ld, int i_off, int f_off, const float* ib, const float* fb, float cap,
                              float* m, const int* cu_seqlens, const int* start_pos, const int* slots, float* keep, float* put,
                              float* m_out, int R, int H, int log_keep, void* stream) {
    if (R <= 0) return 0;
    if (H < 1 || H > 65535 || !(cap > 0.f)) return RG_ERR_UNSUPPORTED;
    return rg_launch(mlstm_gates_kernel, dim3(R, H), dim3(MG_THREADS), 0, (cudaStream_t)stream, 1, raw, ld, i_off, f_off, ib,
                     fb, cap, m, cu_seqlens, start_pos, slots, keep, put, m_out, H, log_keep);
}

// One block per (token, head, block of columns of S; column dv is n).  proj: 32-bit rows ld apart, q, k [H d], v [H dv],
// raw gates [H].  state [slots, H, dv + 1, d].  o [T, H, dv + 1]: S^T q and n . q.  A warp takes MS_COLS columns at a time.
#define MS_THREADS 128
#define MS_COLS 4
template <bool VEC>
__global__ void __launch_bounds__(MS_THREADS)
mlstm_step_kernel(const float* __restrict__ proj, int ld, int q_off, int k_off, int v_off, int i_off, int f_off,
                  const float* __restrict__ ib, const float* __restrict__ fb, float cap, float* __restrict__ state,
                  const float* __restrict__ m, const int* __restrict__ req_of_token, const int* __restrict__ start_pos,
                  const int* __restrict__ slots, float* __restrict__ o, int H, int d, int dv, int cols) {
    extern __shared__ __align__(16) float sm[];        // q [d], k [d] (padded to 4)
    const int DP = (d + 3) & ~3;
    float *sq = sm, *sk = sm + DP;
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * cols, C = dv + 1;
    const int n = min(cols, C - j0);
    const int r = req_of_token[t];
    const int slot = slots[r];
    const bool has_past = slot >= 0 && start_pos[r] > 0;
    const float* row = proj + (size_t)t * ld;
    for (int e = threadIdx.x; e < 2 * d; e += MS_THREADS) {
        if (e < d) sq[e] = row[q_off + (size_t)h * d + e];
        else sk[e - d] = row[k_off + (size_t)h * d + (e - d)];
    }
    const float m0 = has_past ? m[(size_t)slot * H + h] : 0.f;
    const float i = ml_input_gate(row[i_off + h] + ib[h], cap), f = ml_forget_gate(row[f_off + h] + fb[h], cap);
    const float now = fmaxf(f + m0, i);
    const float keep = expf(f + m0 - now), put = expf(i - now);
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* st = state + (((size_t)(slot >= 0 ? slot : 0) * H + h) * C + j0) * d;
    const float* vrow = row + v_off + (size_t)h * dv + j0;
    for (int jb = warp * MS_COLS; jb < n; jb += MS_COLS * (MS_THREADS / 32)) {
        float u[MS_COLS], acc[MS_COLS];
#pragma unroll
        for (int c = 0; c < MS_COLS; ++c) {
            const int j = jb + c;
            u[c] = j < n ? put * (j0 + j < dv ? vrow[j] : 1.f) : 0.f;
            acc[c] = 0.f;
        }
        if (VEC) {
            for (int x = lane * 4; x < d; x += 128) {
                float4 S[MS_COLS];
#pragma unroll
                for (int c = 0; c < MS_COLS; ++c)
                    S[c] = has_past && jb + c < n ? *reinterpret_cast<const float4*>(st + (size_t)(jb + c) * d + x)
                                                  : make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 k = *reinterpret_cast<const float4*>(sk + x), q = *reinterpret_cast<const float4*>(sq + x);
#pragma unroll
                for (int c = 0; c < MS_COLS; ++c) {
                    S[c].x = S[c].x * keep + k.x * u[c]; S[c].y = S[c].y * keep + k.y * u[c];
                    S[c].z = S[c].z * keep + k.z * u[c]; S[c].w = S[c].w * keep + k.w * u[c];
                    acc[c] += S[c].x * q.x + S[c].y * q.y + S[c].z * q.z + S[c].w * q.w;
                    if (slot >= 0 && jb + c < n) *reinterpret_cast<float4*>(st + (size_t)(jb + c) * d + x) = S[c];
                }
            }
        } else {
            for (int x = lane; x < d; x += 32) {
#pragma unroll
                for (int c = 0; c < MS_COLS; ++c) {
                    if (jb + c >= n) break;
                    float* p = st + (size_t)(jb + c) * d + x;
                    const float S = (has_past ? *p : 0.f) * keep + sk[x] * u[c];
                    acc[c] += S * sq[x];
                    if (slot >= 0) *p = S;
                }
            }
        }
#pragma unroll
        for (int c = 0; c < MS_COLS; ++c) {
            const float s = warp_sum(acc[c]);
            if (lane == 0 && jb + c < n) o[((size_t)t * H + h) * C + j0 + jb + c] = s;
        }
    }
}

extern "C" int rg_mlstm_step(const float* proj, int ld, int q_off, int k_off, int v_off, int i_off, int f_off,
                             const float* ib, const float* fb, float cap, float* state, const float* m,
                             const int* req_of_token, const int* start_pos, const int* slots, float* o, int T, int H, int d,
                             int dv, void* stream) {
    if (T <= 0) return 0;
    if (H < 1 || H > 65535 || d < 1 || dv < 1 || !(cap > 0.f)) return RG_ERR_UNSUPPORTED;
    // while there are few (token, head) pairs a head's columns are spread over blocks, 16 (a round of the warps) at the least
    int cols = ((dv + 1) + 15) / 16 * 16;
    while ((long long)T * H * ((dv + cols) / cols) < 1184 && cols > 16) cols = ((cols + 1) / 2 + 15) / 16 * 16;
    const size_t smem = (size_t)2 * ((d + 3) & ~3) * sizeof(float);
    if (smem > 48 * 1024) return RG_ERR_UNSUPPORTED;
    dim3 grid(T, H, (dv + cols) / cols);               // dv + 1 columns, rounded up
    if (grid.z > 65535) return RG_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    if (d % 4 == 0 && ((uintptr_t)state & 15) == 0)
        return rg_launch(mlstm_step_kernel<true>, grid, dim3(MS_THREADS), smem, s, 1, proj, ld, q_off, k_off, v_off, i_off,
                         f_off, ib, fb, cap, state, m, req_of_token, start_pos, slots, o, H, d, dv, cols);
    return rg_launch(mlstm_step_kernel<false>, grid, dim3(MS_THREADS), smem, s, 1, proj, ld, q_off, k_off, v_off, i_off,
                     f_off, ib, fb, cap, state, m, req_of_token, start_pos, slots, o, H, d, dv, cols);
}

// o [T, H, dv + 1] (S^T q and n . q without q's factor q_scale); gate: 32-bit rows gate_ld apart, head h at column h dv.
// x = q_scale o / (max(|q_scale n . q|, exp(-m)) + 1e-6); out = x / sqrt(mean(x^2) + eps) * weight[h dv + ..] * sigmoid(gate).
// m_rows [T, H], or null in steps of single tokens: then m is worked out from the raw gates and the request's m, and left
// there.  One warp per (token, head).
template <typename O>
__global__ void mlstm_out_kernel(const float* __restrict__ o, const float* __restrict__ gate, int gate_ld,
                                 const float* __restrict__ weight, float eps, float q_scale, const float* __restrict__ m_rows,
                                 const float* __restrict__ raw, int raw_ld, int i_off, int f_off, const float* __restrict__ ib,
                                 const float* __restrict__ fb, float cap, float* __restrict__ m,
                                 const int* __restrict__ req_of_token, const int* __restrict__ start_pos,
                                 const int* __restrict__ slots, O* __restrict__ out, int T, int H, int dv) {
    pdl_wait();
    pdl_trigger();
    const int lane = threadIdx.x & 31;
    const long long idx = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (idx >= (long long)T * H) return;
    const int t = (int)(idx / H), h = (int)(idx - (long long)t * H);
    float now;
    if (m_rows) {
        now = m_rows[idx];
    } else {
        const int r = req_of_token[t], slot = slots[r];
        float* mp = m + (size_t)(slot >= 0 ? slot : 0) * H + h;
        const float m0 = slot >= 0 && start_pos[r] > 0 ? *mp : 0.f;
        const float* row = raw + (size_t)t * raw_ld;
        now = fmaxf(ml_forget_gate(row[f_off + h] + fb[h], cap) + m0, ml_input_gate(row[i_off + h] + ib[h], cap));
        __syncwarp();
        if (slot >= 0 && lane == 0) *mp = now;
    }
    const float* src = o + (size_t)idx * (dv + 1);
    const float inv_den = 1.f / (fmaxf(fabsf(q_scale * src[dv]), expf(-now)) + 1e-6f);
    const float f = q_scale * inv_den;
    float ss = 0.f;
    for (int i = lane; i < dv; i += 32) { const float v = src[i] * f; ss += v * v; }
    ss = warp_sum(ss);
    const float inv = rsqrtf(ss / (float)dv + eps);
    const float* grow = gate + (size_t)t * gate_ld + (size_t)h * dv;
    const float* wrow = weight + (size_t)h * dv;
    O* dst = out + (size_t)idx * dv;
    for (int i = lane; i < dv; i += 32) dst[i] = from_f32<O>(src[i] * f * inv * wrow[i] / (1.f + expf(-grow[i])));
}

extern "C" int rg_mlstm_out(const float* o, const float* gate, int gate_ld, const float* weight, float eps, float q_scale,
                            const float* m_rows, const float* raw, int raw_ld, int i_off, int f_off, const float* ib,
                            const float* fb, float cap, float* m, const int* req_of_token, const int* start_pos,
                            const int* slots, void* out, int out_dtype, int T, int H, int dv, void* stream) {
    if (T <= 0) return 0;
    if (H < 1 || dv < 1 || !(cap > 0.f) || (!m_rows && !m)) return RG_ERR_UNSUPPORTED;
    const long long n = (long long)T * H;
    dim3 grid((unsigned)((n + 3) / 4));
    cudaStream_t s = (cudaStream_t)stream;
#define ML_OUT(O) return rg_launch(mlstm_out_kernel<O>, grid, dim3(128), 0, s, 1, o, gate, gate_ld, weight, eps, q_scale, \
        m_rows, raw, raw_ld, i_off, f_off, ib, fb, cap, m, req_of_token, start_pos, slots, (O*)out, T, H, dv)
    if (out_dtype == RG_DTYPE_BF16) ML_OUT(bf16);
    if (out_dtype == RG_DTYPE_F32) ML_OUT(float);
#undef ML_OUT
    return RG_ERR_UNSUPPORTED;
}
