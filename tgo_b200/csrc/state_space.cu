// A selective state-space mixer's recurrent part (the form known as Mamba-2): a short causal
// convolution per channel with its last inputs kept per request, and the scan
//
//   dt_t = softplus(raw_t + dt_bias_h)                      per head h, float32
//   S_t  = exp(-exp(A_log_h) dt_t) S_(t-1) + dt_t B_t x_t^T      S is [N, P], float32
//   y_t  = S_t^T C_t + D_h x_t
//
// over each request's tokens of the step, from and into the request's float32 state. Head h
// reads B and C of group floor(h / (H / G)). Everything after the convolution's input is
// float32 whatever the storage type of the projections.
//
// A second scan (the form known as Mamba-1) has a decay of its own for every channel and state,
// and B and C shared by all channels:
//
//   dt_t    = softplus(raw_t + dt_bias)                     per channel c
//   S[c, n] = exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n       S is [channels, N], float32
//   y_c     = (sum_n S[c, n] C_n + D_c x_c) * silu(z_c)
//
// A request's state row (float32, `state_stride` floats apart) holds the scan's state
// [H][N][P] (or [channels][N]) at `ssm_offset` and the convolution's last taps - 1 inputs [taps - 1][C] (oldest
// first) at `conv_offset`.
#include "common.cuh"

// ------------------------------------------------------------------------- convolution
// y[t][c] = silu(bias[c] + sum_j w[c][j] x[t - (taps - 1 - j)][c]); inputs before the step's
// first token come from the request's kept inputs, zeros before the request's start (a fresh
// state row is zero). x is a column view [T, C] in the storage type; y [T, C] float32 or in the
// storage type (TY).
template <typename T, typename TY>
__global__ void __launch_bounds__(256)
causal_conv_act_kernel(const T* __restrict__ x, long long x_stride, const float* __restrict__ w,
                       const float* __restrict__ bias, TY* __restrict__ y, int C, int taps,
                       const int* __restrict__ seq_ids, const int* __restrict__ q_start,
                       const int* __restrict__ state_slots, const float* __restrict__ state,
                       long long state_stride, long long conv_offset) {
    pdl_wait();
    const int t = blockIdx.x;
    const int b = seq_ids[t];
    const int r = t - q_start[b];                       // place among the request's tokens
    const float* kept = state + (size_t)state_slots[b] * state_stride + conv_offset;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        float a = bias ? bias[c] : 0.f;
        for (int j = 0; j < taps; ++j) {
            const int back = taps - 1 - j;               // how many tokens before this one
            float v;
            if (back <= r) v = to_f32(x[(size_t)(t - back) * x_stride + c]);
            else v = kept[(size_t)(taps - 1 - (back - r)) * C + c];
            a = fmaf(w[(size_t)c * taps + j], v, a);
        }
        y[(size_t)t * C + c] = from_f32<TY>(a / (1.f + expf(-a)));
    }
}

// The same with eight channels a thread (16-byte loads of x) and TOK consecutive tokens, whose
// rows are asked for before the first is used, the window of inputs in registers: for up to four
// taps, C, the row stride and x's address as multiples of eight elements. `kept4`: the kept rows
// can be read 16 bytes at a time. One token a thread where the step has only single tokens.
#define CV_TOK 8
__device__ __forceinline__ void cv_widen(float* v, uint4 q) {
    const uint32_t* w = (const uint32_t*)&q;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const float2 f = __bfloat1622float2(*(const __nv_bfloat162*)(w + k));
        v[2 * k] = f.x;
        v[2 * k + 1] = f.y;
    }
}
__device__ __forceinline__ void cv_load8(float* v, const float* p) {
    const float4 a = *(const float4*)p, b = *(const float4*)(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void cv_store(bf16* p, const float* v) {
    uint4 q;
    uint32_t* w = (uint32_t*)&q;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
        w[k] = *(const uint32_t*)&b;
    }
    *(uint4*)p = q;
}
__device__ __forceinline__ void cv_store(float* p, const float* v) {
    *(float4*)p = make_float4(v[0], v[1], v[2], v[3]);
    *(float4*)(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

template <typename TY, int TAPS, int TOK>
__global__ void __launch_bounds__(128)
causal_conv_act_x8_kernel(const bf16* __restrict__ x, long long x_stride, const float* __restrict__ w,
                          const float* __restrict__ bias, TY* __restrict__ y, int Tn, int C,
                          const int* __restrict__ seq_ids, const int* __restrict__ q_start,
                          const int* __restrict__ state_slots, const float* __restrict__ state,
                          long long state_stride, long long conv_offset, int kept4) {
    pdl_wait();
    const int c = 8 * (blockIdx.y * blockDim.x + threadIdx.x), t_lo = blockIdx.x * TOK;
    if (c >= C) return;
    uint4 rows[TOK];
#pragma unroll
    for (int u = 0; u < TOK; ++u)
        rows[u] = *(const uint4*)(x + (size_t)(t_lo + u < Tn ? t_lo + u : Tn - 1) * x_stride + c);
    float wt[8 * TAPS], bs[8], win[TAPS][8];             // win[j] meets tap j; the last is the token's own
#pragma unroll
    for (int q = 0; q < TAPS; ++q) cv_load8(wt + 8 * q, w + (size_t)c * TAPS + 8 * q);    // [channel][tap]
    if (bias) {
        cv_load8(bs, bias + c);
    } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) bs[i] = 0.f;
    }
    int q_at = -1, first = 0;
#pragma unroll
    for (int u = 0; u < TOK; ++u) {
        const int t = t_lo + u;
        if (t >= Tn) break;
        const int b = seq_ids[t];
        if (u == 0 || b != q_at) {                       // a window from the start: rows of the step, then kept ones
            q_at = b;
            first = q_start[b];
            const float* kept = state + (size_t)state_slots[b] * state_stride + conv_offset;
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) {
                const int back = TAPS - 1 - j, r = t - first;
                if (back <= r) {
                    cv_widen(win[j], *(const uint4*)(x + (size_t)(t - back) * x_stride + c));
                } else {
                    const float* k = kept + (size_t)(TAPS - 1 - (back - r)) * C + c;
                    if (kept4) {
                        cv_load8(win[j], k);
                    } else {
#pragma unroll
                        for (int i = 0; i < 8; ++i) win[j][i] = k[i];
                    }
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
                for (int i = 0; i < 8; ++i) win[j][i] = win[j + 1][i];
        }
        cv_widen(win[TAPS - 1], rows[u]);
        float o[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            float a = bs[i];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) a = fmaf(wt[i * TAPS + j], win[j][i], a);
            o[i] = __fdividef(a, 1.f + __expf(-a));
        }
        cv_store(y + (size_t)t * C + c, o);
    }
}

// After the convolution has run: the kept inputs of every request become the last taps - 1
// of (kept inputs, then the step's inputs). A thread per (request, channel).
template <typename T>
__global__ void __launch_bounds__(256)
causal_conv_keep_kernel(const T* __restrict__ x, long long x_stride, int C, int taps,
                        const int* __restrict__ q_start, const int* __restrict__ state_slots,
                        float* __restrict__ state, long long state_stride, long long conv_offset) {
    pdl_wait();
    const int b = blockIdx.x;
    const int t0 = q_start[b], n = q_start[b + 1] - t0;
    float* kept = state + (size_t)state_slots[b] * state_stride + conv_offset;
    const int keep = taps - 1;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        // ascending i reads kept[n + i] before any later write could reach it (n + i >= i)
        for (int i = 0; i < keep; ++i) {
            const int at = n + i;                        // place in (kept, then new)
            const float v = at < keep ? kept[(size_t)at * C + c]
                                      : to_f32(x[(size_t)(t0 + at - keep) * x_stride + c]);
            kept[(size_t)i * C + c] = v;
        }
    }
}

// y_dtype: float32, or the storage type. `keep` 0 leaves the kept inputs where they are (the
// channel scan below moves them on itself).
TGO_API int tgo_causal_conv_act(const void* x, long long x_stride, int dtype, const float* w,
                                const float* bias, void* y, int y_dtype, int T, int B, int C, int taps,
                                const int* seq_ids, const int* q_start, const int* state_slots,
                                float* state, long long state_stride, long long conv_offset, int keep,
                                cudaStream_t stream) {
    if (T <= 0 || B <= 0) return 0;
    if (C <= 0 || taps <= 0 || taps > 64 || state_stride < conv_offset + (long long)(taps - 1) * C)
        return TGO_E_BAD_ARG;
    const int cy = (C + 255) / 256 > 64 ? 64 : (C + 255) / 256;
    int rc;
#define CONV_GO(TT, TY)                                                                                    \
    tgo_launch_pdl(causal_conv_act_kernel<TT, TY>, dim3(T, cy), dim3(256), 0, stream, (const TT*)x, x_stride, w, \
                   bias, (TY*)y, C, taps, seq_ids, q_start, state_slots, (const float*)state, state_stride, \
                   conv_offset)
    const int kept4 = state_stride % 4 == 0 && conv_offset % 4 == 0 && (uintptr_t)state % 16 == 0;
#define CONV_X8_AT(TY, TAPS, TOK)                                                                          \
    tgo_launch_pdl(causal_conv_act_x8_kernel<TY, TAPS, TOK>, dim3((T + TOK - 1) / TOK, (C / 8 + 127) / 128),       \
                   dim3(128), 0, stream, (const bf16*)x, x_stride, w, bias, (TY*)y, T, C, seq_ids, q_start,      \
                   state_slots, (const float*)state, state_stride, conv_offset, kept4)
#define CONV_X8(TY, TAPS) (T == B ? CONV_X8_AT(TY, TAPS, 1) : CONV_X8_AT(TY, TAPS, CV_TOK))
#define CONV_TAPS(TY) (taps == 1 ? CONV_X8(TY, 1) : taps == 2 ? CONV_X8(TY, 2) : taps == 3 ? CONV_X8(TY, 3) : CONV_X8(TY, 4))
    if (dtype == TGO_BF16 && (y_dtype == TGO_F32 || y_dtype == TGO_BF16) && taps <= 4 && C % 8 == 0 &&
        x_stride % 8 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)w % 16 == 0 &&
        (uintptr_t)bias % 16 == 0)
        rc = y_dtype == TGO_F32 ? CONV_TAPS(float) : CONV_TAPS(bf16);
    else if (dtype == TGO_BF16 && y_dtype == TGO_F32) rc = CONV_GO(bf16, float);
    else if (dtype == TGO_BF16 && y_dtype == TGO_BF16) rc = CONV_GO(bf16, bf16);
    else if (dtype == TGO_F32 && y_dtype == TGO_F32) rc = CONV_GO(float, float);
    else return TGO_E_BAD_ARG;
#undef CONV_GO
#undef CONV_X8
#undef CONV_X8_AT
#undef CONV_TAPS
    if (rc || taps == 1 || !keep) return rc;
    if (dtype == TGO_BF16)
        return tgo_launch_pdl(causal_conv_keep_kernel<bf16>, dim3(B, cy), dim3(256), 0, stream, (const bf16*)x,
                              x_stride, C, taps, q_start, state_slots, state, state_stride, conv_offset);
    return tgo_launch_pdl(causal_conv_keep_kernel<float>, dim3(B, cy), dim3(256), 0, stream, (const float*)x,
                          x_stride, C, taps, q_start, state_slots, state, state_stride, conv_offset);
}

// -------------------------------------------------------------------------------- scan
// A block per (request, head, 32 columns of P). 256 threads: thread (column c = tid / 8,
// slice s = tid % 8) keeps rows n = 32 i + 4 s + j (j = 0..3) of its column of S in registers
// for the whole walk over the request's tokens; a token's y[c] is the sum of the eight
// slices' partial sums (three shuffles, the same order for every token). The tokens' B, C, x
// and dt come through shared memory SS_TOK at a time, two buffers: the next tokens load while
// these are walked; B and C are read four rows at a time. The order of every sum depends on
// the sizes alone, so a token's result does not depend on how the tokens were cut or batched
// beyond the state's own history, which is the same sequence of updates whatever the cut.
#define SS_TOK 16
#define SS_COLS 32

// a 4-byte asynchronous copy into shared memory (zeros when !valid)
__device__ __forceinline__ void ss_copy4(float* dst, const float* src, bool valid) {
    const int n = valid ? 4 : 0;
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(
                     (uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(n));
}

template <typename T, int NI>
__global__ void __launch_bounds__(256)
selective_scan_kernel(const float* __restrict__ xbc, int C, const T* __restrict__ dt_raw,
                      long long dt_stride, const float* __restrict__ dt_bias,
                      const float* __restrict__ A_log, const float* __restrict__ D,
                      float* __restrict__ y, int H, int G, int N, int P,
                      const int* __restrict__ q_start, const int* __restrict__ state_slots,
                      float* __restrict__ state, long long state_stride, long long ssm_offset) {
    constexpr int NP = NI * 8;                           // N rounded up to whole rounds of 32
    extern __shared__ __align__(16) float smem[];
    // per buffer: B [SS_TOK][NP], C [SS_TOK][NP], x [SS_TOK][SS_COLS], dt [SS_TOK], decay [SS_TOK]
    constexpr int BUF = 2 * SS_TOK * NP + SS_TOK * SS_COLS + 2 * SS_TOK;
    pdl_wait();
    const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * SS_COLS;
    const int g = h / (H / G);
    const int inner = H * P;
    const int col = threadIdx.x >> 3, s = threadIdx.x & 7;
    const int c = c0 + col;
    const bool live = c < P;
    const int t0 = q_start[b], n_tok = q_start[b + 1] - t0;
    float* Sg = state + (size_t)state_slots[b] * state_stride + ssm_offset + (size_t)h * N * P;
    // the state comes and goes through shared memory, so that global memory sees whole rows
    // of 32 columns (the staging buffers are idle then; [N][33] floats fit in them)
    float S[NI];
    for (int i = threadIdx.x; i < N * SS_COLS; i += 256) {
        const int n = i / SS_COLS, cc = i % SS_COLS;
        smem[n * (SS_COLS + 1) + cc] = c0 + cc < P ? Sg[(size_t)n * P + c0 + cc] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = 32 * (i >> 2) + 4 * s + (i & 3);
        S[i] = n < N ? smem[n * (SS_COLS + 1) + col] : 0.f;
    }
    __syncthreads();
    const float A = expf(A_log[h]);
    const float Dh = D ? D[h] : 0.f;
    const float bias = dt_bias ? dt_bias[h] : 0.f;
    auto stage = [&](int base, int buf) {
        float* Bs = smem + buf * BUF;
        float* Cs = Bs + SS_TOK * NP;
        float* xs = Cs + SS_TOK * NP;
        float* dts = xs + SS_TOK * SS_COLS;
        float* das = dts + SS_TOK;
        const int nt = n_tok - base < SS_TOK ? n_tok - base : SS_TOK;
        for (int i = threadIdx.x; i < nt * NP; i += 256) {
            const int r = i / NP, n = i % NP;
            const float* row = xbc + (size_t)(t0 + base + r) * C + inner + (size_t)g * N;
            ss_copy4(Bs + i, n < N ? row + n : xbc, n < N);
            ss_copy4(Cs + i, n < N ? row + (size_t)G * N + n : xbc, n < N);
        }
        for (int i = threadIdx.x; i < nt * SS_COLS; i += 256) {
            const int r = i / SS_COLS, cc = i % SS_COLS;
            const bool ok = c0 + cc < P;
            ss_copy4(xs + i, ok ? xbc + (size_t)(t0 + base + r) * C + (size_t)h * P + c0 + cc : xbc, ok);
        }
        asm volatile("cp.async.commit_group;\n" ::);
        if (threadIdx.x < nt) {
            const float z = to_f32(dt_raw[(size_t)(t0 + base + threadIdx.x) * dt_stride + h]) + bias;
            const float dt = z > 20.f ? z : log1pf(expf(z));
            dts[threadIdx.x] = dt;
            das[threadIdx.x] = expf(-A * dt);
        }
    };
    stage(0, 0);
    for (int base = 0, buf = 0; base < n_tok; base += SS_TOK, buf ^= 1) {
        const int nt = n_tok - base < SS_TOK ? n_tok - base : SS_TOK;
        if (base + SS_TOK < n_tok) {
            stage(base + SS_TOK, buf ^ 1);                // the buffer the last pass left
            asm volatile("cp.async.wait_group 1;\n" ::);
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::);
        }
        __syncthreads();
        const float* Bs = smem + buf * BUF;
        const float* Cs = Bs + SS_TOK * NP;
        const float* xs = Cs + SS_TOK * NP;
        const float* dts = xs + SS_TOK * SS_COLS;
        const float* das = dts + SS_TOK;
        for (int r = 0; r < nt; ++r) {
            const float x = xs[r * SS_COLS + col];
            const float dx = dts[r] * x, da = das[r];
            float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i4 = 0; i4 < NI / 4; ++i4) {
                const float4 bq = *(const float4*)(Bs + r * NP + 32 * i4 + 4 * s);
                const float4 cq = *(const float4*)(Cs + r * NP + 32 * i4 + 4 * s);
                S[4 * i4 + 0] = fmaf(da, S[4 * i4 + 0], dx * bq.x);
                S[4 * i4 + 1] = fmaf(da, S[4 * i4 + 1], dx * bq.y);
                S[4 * i4 + 2] = fmaf(da, S[4 * i4 + 2], dx * bq.z);
                S[4 * i4 + 3] = fmaf(da, S[4 * i4 + 3], dx * bq.w);
                part[0] = fmaf(S[4 * i4 + 0], cq.x, part[0]);
                part[1] = fmaf(S[4 * i4 + 1], cq.y, part[1]);
                part[2] = fmaf(S[4 * i4 + 2], cq.z, part[2]);
                part[3] = fmaf(S[4 * i4 + 3], cq.w, part[3]);
            }
            float sum = (part[0] + part[1]) + (part[2] + part[3]);
            sum += __shfl_xor_sync(0xffffffffu, sum, 1);
            sum += __shfl_xor_sync(0xffffffffu, sum, 2);
            sum += __shfl_xor_sync(0xffffffffu, sum, 4);
            if (s == 0 && live) y[(size_t)(t0 + base + r) * inner + (size_t)h * P + c] = sum + Dh * x;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = 32 * (i >> 2) + 4 * s + (i & 3);
        if (n < N) smem[n * (SS_COLS + 1) + col] = S[i];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < N * SS_COLS; i += 256) {
        const int n = i / SS_COLS, cc = i % SS_COLS;
        if (c0 + cc < P) Sg[(size_t)n * P + c0 + cc] = smem[n * (SS_COLS + 1) + cc];
    }
}

template <typename T, int NI>
static int launch_scan(const float* xbc, int C, const T* dt_raw, long long dt_stride,
                       const float* dt_bias, const float* A_log, const float* D, float* y, int B,
                       int H, int G, int N, int P, const int* q_start, const int* state_slots,
                       float* state, long long state_stride, long long ssm_offset,
                       cudaStream_t stream) {
    const size_t smem = 2 * ((size_t)2 * SS_TOK * NI * 8 + SS_TOK * SS_COLS + 2 * SS_TOK) * sizeof(float);
    auto kernel = selective_scan_kernel<T, NI>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return tgo_launch_pdl(kernel, dim3(B, H, (P + SS_COLS - 1) / SS_COLS), dim3(256),
                          smem, stream, xbc, C, dt_raw, dt_stride, dt_bias, A_log, D, y, H, G, N, P,
                          q_start, state_slots, state, state_stride, ssm_offset);
}

template <typename T>
static int scan_by_size(const float* xbc, int C, const T* dt_raw, long long dt_stride,
                        const float* dt_bias, const float* A_log, const float* D, float* y, int B,
                        int H, int G, int N, int P, const int* q_start, const int* state_slots,
                        float* state, long long state_stride, long long ssm_offset,
                        cudaStream_t stream) {
#define SS_GO(NI) launch_scan<T, NI>(xbc, C, dt_raw, dt_stride, dt_bias, A_log, D, y, B, H, G, N, P, \
                                     q_start, state_slots, state, state_stride, ssm_offset, stream)
    const int ni = (N + 7) / 8;
    if (ni <= 4) return SS_GO(4);
    if (ni <= 8) return SS_GO(8);
    if (ni <= 16) return SS_GO(16);
    return SS_GO(32);
#undef SS_GO
}

// xbc float32 [T, C], C = H P + 2 G N: the convolution's output (x, then B, then C of every
// group); dt_raw a column view [T, H] in the storage type; y float32 [T, H P].
TGO_API int tgo_selective_scan(const float* xbc, int C, const void* dt_raw, long long dt_stride,
                               int dtype, const float* dt_bias, const float* A_log, const float* D,
                               float* y, int B, int H, int G, int N, int P, const int* q_start,
                               const int* state_slots, float* state, long long state_stride,
                               long long ssm_offset, cudaStream_t stream) {
    if (B <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || N <= 0 || N > 256 || P <= 0 || H > 65535 ||
        C != H * P + 2 * G * N || state_stride < ssm_offset + (long long)H * N * P)
        return TGO_E_BAD_ARG;
    if (dtype == TGO_BF16)
        return scan_by_size<bf16>(xbc, C, (const bf16*)dt_raw, dt_stride, dt_bias, A_log, D, y, B, H, G, N,
                                  P, q_start, state_slots, state, state_stride, ssm_offset, stream);
    if (dtype == TGO_F32)
        return scan_by_size<float>(xbc, C, (const float*)dt_raw, dt_stride, dt_bias, A_log, D, y, B, H, G, N,
                                   P, q_start, state_slots, state, state_stride, ssm_offset, stream);
    return TGO_E_BAD_ARG;
}

// ---------------------------------------------------------------------- scan per channel
// A block per (request, CS_WALK / L channels) whose threads have two roles and work on different
// tiles of TOK tokens at the same time. The walking warps: L lanes share a channel and lane l keeps states
// l * NS .. l * NS + NS - 1 of it in registers for the whole walk over the request's tokens. Four
// tokens are taken together: their decays do not depend on the state, so only one FMA per state
// and token is a chain, and the four sums over n are joined by a transposing exchange in the
// quad (three shuffles for four tokens) and, for L > 4, by shuffles over the quads, the same
// order for every token. Tokens past the end of a tile have dt = 0 and leave the state as it is.
// The serving warps: while tile k is walked it puts tile k + 1 into shared memory (dt through
// softplus once per (token, channel), beside dt * x; B and C as float32 rows), asks for tile
// k + 2's inputs, and finishes tile k - 1 (D x added, times silu(z), stored). `a2` is A log2(e).
//
// The walk ends with the convolution's kept inputs: the last taps - 1 of (kept, then the
// step's raw inputs `conv_in`), which the convolution has read before this kernel starts.
#define CS_WALK 128              // walking threads
// serving threads: 256 where a tile has a (token, channel) pair for each, else 128
#define CS_SERVE(TOK, L) ((TOK) * (CS_WALK / (L)) % 256 == 0 ? 256 : 128)

// One step of one state: 2^e S + add. A state that decays slowly is multiplied by nearly 1
// thousands of times, and an exponential that is off by the same fraction of a unit in the last
// place each time adds up; the float32 engine therefore takes the change S (2^e - 1), whose
// rounding is relative to the change, while the decay is slow.
template <typename T> __device__ __forceinline__ float cs_step(float S, float e, float add);
template <> __device__ __forceinline__ float cs_step<bf16>(float S, float e, float add) {
    float d;                                             // a decay below 2^-126 is none
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(d) : "f"(e));
    return fmaf(d, S, add);
}
template <> __device__ __forceinline__ float cs_step<float>(float S, float e, float add) {
    if (e < -0.5f) return fmaf(exp2f(e), S, add);
    return S + fmaf(expm1f(e * 0.69314718055994531f), S, add);
}

// softplus and silu: the library's functions in the float32 engine; in the bfloat16 engine the
// special-function unit's exponential, logarithm and reciprocal (float32, a few units in the
// last place), with log(1 + e) by its series where e is small.
template <typename T> __device__ __forceinline__ float cs_softplus(float v);
template <> __device__ __forceinline__ float cs_softplus<float>(float v) { return v > 20.f ? v : log1pf(expf(v)); }
template <> __device__ __forceinline__ float cs_softplus<bf16>(float v) {
    const float e = __expf(v);
    const float small = e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 0.33333334f), -0.5f), 1.f);
    return v > 20.f ? v : e < 0.03f ? small : __logf(1.f + e);
}
template <typename T> __device__ __forceinline__ float cs_silu(float z);
template <> __device__ __forceinline__ float cs_silu<float>(float z) { return z / (1.f + expf(-z)); }
template <> __device__ __forceinline__ float cs_silu<bf16>(float z) { return __fdividef(z, 1.f + __expf(-z)); }

// The kept inputs of one channel of one request.
template <typename T>
__device__ __forceinline__ void cs_keep(float* kept, const T* __restrict__ conv_in, long long conv_in_stride,
                                        int c, int C, int taps, int t0, int n_tok) {
    const int keep = taps - 1;
    // ascending i reads kept[n_tok + i] before any later write could reach it
    for (int i = 0; i < keep; ++i) {
        const int at = n_tok + i;                        // place in (kept, then new)
        kept[(size_t)i * C + c] = at < keep ? kept[(size_t)at * C + c]
                                            : to_f32(conv_in[(size_t)(t0 + at - keep) * conv_in_stride + c]);
    }
}

template <typename T, int L, int NS, int TOK>
__global__ void __launch_bounds__(CS_WALK + CS_SERVE(TOK, L))
channel_scan_kernel(const T* __restrict__ x, long long x_stride, const T* __restrict__ z, long long z_stride,
                    const float* __restrict__ dt_raw, long long dt_stride, const float* __restrict__ dt_bias,
                    const float* __restrict__ a2, const T* __restrict__ bm, const T* __restrict__ cm,
                    long long bc_stride, const float* __restrict__ D, T* __restrict__ y, int C, int N,
                    const int* __restrict__ q_start, const int* __restrict__ state_slots,
                    float* __restrict__ state, long long state_stride, long long ssm_offset,
                    const T* __restrict__ conv_in, long long conv_in_stride, int taps, long long conv_offset) {
    constexpr int CH = CS_WALK / L;                      // channels of this block
    constexpr int NP = L * NS;                           // N rounded up
    constexpr int SERVE = CS_SERVE(TOK, L);
    constexpr int PER = TOK * CH / SERVE;                // (token, channel) pairs a serving thread loads
    constexpr int RSTEP = SERVE / CH;                 // tokens between a thread's pairs
    constexpr int PBC = TOK * NP / SERVE;
    static_assert(TOK * CH % SERVE == 0 && TOK * NP % SERVE == 0, "tile");
    extern __shared__ __align__(16) float cs_smem[];
    float* s_b = cs_smem;                                // [2][TOK][NP]
    float* s_c = s_b + 2 * TOK * NP;                  // [2][TOK][NP]
    float2* s_dt = (float2*)(s_c + 2 * TOK * NP);     // [2][TOK][CH + 1]: dt, dt x
    float* s_y = (float*)(s_dt + 2 * TOK * (CH + 1)); // [2][TOK][CH + 1]
    pdl_wait();
    const int b = blockIdx.x, c0 = blockIdx.y * CH;
    const int t0 = q_start[b], n_tok = q_start[b + 1] - t0;
    const int n_tiles = (n_tok + TOK - 1) / TOK;
    float* row = state + (size_t)state_slots[b] * state_stride;
    if (threadIdx.x < CS_WALK) {
        // ---- walking
        const int tid = threadIdx.x;
        const int lane_l = tid % L, wch = tid / L, wc = c0 + wch, n0 = lane_l * NS;
        const bool live = wc < C;
        float S[NS], A[NS];
#pragma unroll
        for (int i = 0; i < NS; ++i) {
            const bool ok = live && n0 + i < N;
            S[i] = ok ? row[ssm_offset + (size_t)wc * N + n0 + i] : 0.f;
            A[i] = ok ? a2[(size_t)wc * N + n0 + i] : 0.f;
        }
        const bool odd = tid & 1, high = tid & 2;
        __syncthreads();                                 // tile 0 is in shared memory
        for (int k = 0; k < n_tiles; ++k) {
            const int nt = n_tok - k * TOK < TOK ? n_tok - k * TOK : TOK;
            const float2* dts = s_dt + (k & 1) * TOK * (CH + 1) + wch;
            const float* bs = s_b + (k & 1) * TOK * NP + n0;
            const float* cs = s_c + (k & 1) * TOK * NP + n0;
            float* ys = s_y + (k & 1) * TOK * (CH + 1) + wch;
            for (int r = 0; r < nt; r += 4) {
                float part[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const float2 dd = dts[(r + u) * (CH + 1)];
                    const float* br = bs + (r + u) * NP;
                    const float* cr = cs + (r + u) * NP;
                    float p = 0.f, p2 = 0.f;
#pragma unroll
                    for (int i = 0; i < NS; i += 4) {
                        const float4 bq = *(const float4*)(br + i), cq = *(const float4*)(cr + i);
                        S[i] = cs_step<T>(S[i], dd.x * A[i], dd.y * bq.x);
                        S[i + 1] = cs_step<T>(S[i + 1], dd.x * A[i + 1], dd.y * bq.y);
                        S[i + 2] = cs_step<T>(S[i + 2], dd.x * A[i + 2], dd.y * bq.z);
                        S[i + 3] = cs_step<T>(S[i + 3], dd.x * A[i + 3], dd.y * bq.w);
                        p = fmaf(S[i], cq.x, p);
                        p2 = fmaf(S[i + 1], cq.y, p2);
                        p = fmaf(S[i + 2], cq.z, p);
                        p2 = fmaf(S[i + 3], cq.w, p2);
                    }
                    part[u] = p + p2;
                }
                // four sums over the quad, transposed: lane q of a quad ends with token r + q
                const float s0 = odd ? part[0] : part[1], s1 = odd ? part[2] : part[3];
                float k0 = odd ? part[1] : part[0], k1 = odd ? part[3] : part[2];
                k0 += __shfl_xor_sync(0xffffffffu, s0, 1);
                k1 += __shfl_xor_sync(0xffffffffu, s1, 1);
                const float s2 = high ? k0 : k1;
                float sum = high ? k1 : k0;
                sum += __shfl_xor_sync(0xffffffffu, s2, 2);
#pragma unroll
                for (int o = 4; o < L; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
                if (lane_l < 4) ys[(r + (tid & 3)) * (CH + 1)] = sum;
            }
            __syncthreads();
        }
#pragma unroll
        for (int i = 0; i < NS; ++i)
            if (live && n0 + i < N) row[ssm_offset + (size_t)wc * N + n0 + i] = S[i];
        return;
    }
    // ---- serving: channel lc, tokens lt + RSTEP i of a tile
    const int tid = threadIdx.x - CS_WALK;
    const int lcl = tid % CH, lc = c0 + lcl, lt = tid / CH;
    const bool lok = lc < C;
    const float bias = (lok && dt_bias) ? dt_bias[lc] : 0.f;
    const float skip = (lok && D) ? D[lc] : 0.f;
    const T zero = from_f32<T>(0.f);
    T xn[PER], bn[PBC], cn[PBC];                         // raw, so that nothing waits for them here
    float dn[PER];
    auto fetch = [&](int k) {
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = k * TOK + lt + RSTEP * i;
            const bool ok = lok && r < n_tok;
            const size_t t = (size_t)(t0 + r);
            xn[i] = ok ? x[t * x_stride + lc] : zero;
            dn[i] = ok ? dt_raw[t * dt_stride + lc] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < PBC; ++i) {
            const int q = tid + SERVE * i;
            const int r = k * TOK + q / NP, n = q % NP;
            const bool ok = n < N && r < n_tok;
            bn[i] = ok ? bm[(size_t)(t0 + r) * bc_stride + n] : zero;
            cn[i] = ok ? cm[(size_t)(t0 + r) * bc_stride + n] : zero;
        }
    };
    auto stage = [&](int k) {                            // what fetch(k) has brought
        float2* dts = s_dt + (k & 1) * TOK * (CH + 1);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = lt + RSTEP * i;
            const float dt = k * TOK + r < n_tok ? cs_softplus<T>(dn[i] + bias) : 0.f;
            dts[r * (CH + 1) + lcl] = make_float2(dt, dt * to_f32(xn[i]));
        }
#pragma unroll
        for (int i = 0; i < PBC; ++i) {
            s_b[(k & 1) * TOK * NP + tid + SERVE * i] = to_f32(bn[i]);
            s_c[(k & 1) * TOK * NP + tid + SERVE * i] = to_f32(cn[i]);
        }
    };
    T xr[PER], zr[PER];
    auto recall = [&](int k) {                           // x and z of a walked tile, ahead of their use
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = k * TOK + lt + RSTEP * i;
            const bool ok = lok && r < n_tok;
            xr[i] = ok ? x[(size_t)(t0 + r) * x_stride + lc] : zero;
            zr[i] = ok ? z[(size_t)(t0 + r) * z_stride + lc] : zero;
        }
    };
    auto finish = [&](int k) {                           // the walked tile k: gate and store
        const float* ys = s_y + (k & 1) * TOK * (CH + 1);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = lt + RSTEP * i;
            if (lok && k * TOK + r < n_tok)
                y[(size_t)(t0 + k * TOK + r) * C + lc] =
                    from_f32<T>(fmaf(skip, to_f32(xr[i]), ys[r * (CH + 1) + lcl]) * cs_silu<T>(to_f32(zr[i])));
        }
    };
    fetch(0);
    stage(0);
    if (n_tiles > 1) fetch(1);
    __syncthreads();
    for (int k = 0; k < n_tiles; ++k) {
        if (k > 0) recall(k - 1);
        if (k + 1 < n_tiles) stage(k + 1);
        if (k + 2 < n_tiles) fetch(k + 2);
        if (k > 0) finish(k - 1);
        __syncthreads();
    }
    if (n_tiles > 0) {
        recall(n_tiles - 1);
        finish(n_tiles - 1);
    }
    if (conv_in && tid < CH && c0 + tid < C)
        cs_keep(row + conv_offset, conv_in, conv_in_stride, c0 + tid, C, taps, t0, n_tok);
}

// A step in which every request brings one token: nothing to stage, a thread takes NS states of
// one channel of one request (L lanes a channel, four states a 16-byte access where they lie
// that way), the lanes join their sums and the first of them gates and stores.
template <typename T, int L, int NS, bool VEC>
__global__ void __launch_bounds__(128)
channel_scan_single_kernel(const T* __restrict__ x, long long x_stride, const T* __restrict__ z, long long z_stride,
                           const float* __restrict__ dt_raw, long long dt_stride, const float* __restrict__ dt_bias,
                           const float* __restrict__ a2, const T* __restrict__ bm, const T* __restrict__ cm,
                           long long bc_stride, const float* __restrict__ D, T* __restrict__ y, int C, int N,
                           const int* __restrict__ q_start, const int* __restrict__ state_slots,
                           float* __restrict__ state, long long state_stride, long long ssm_offset,
                           const T* __restrict__ conv_in, long long conv_in_stride, int taps, long long conv_offset) {
    constexpr int CH = 128 / L;
    pdl_wait();
    const int b = blockIdx.x, lane_l = threadIdx.x % L, n0 = lane_l * NS;
    const int c = blockIdx.y * CH + threadIdx.x / L;
    const bool live = c < C;
    const int t = q_start[b];
    float* row = state + (size_t)state_slots[b] * state_stride;
    float* Sg = row + ssm_offset + (size_t)(live ? c : 0) * N + n0;
    const float* Ag = a2 + (size_t)(live ? c : 0) * N + n0;
    float S[NS], A[NS];
    if (VEC) {
#pragma unroll
        for (int i = 0; i < NS; i += 4) {
            const bool ok = live && n0 + i < N;          // N % 4 == 0: the four are in or out together
            const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 s4 = ok ? *(const float4*)(Sg + i) : zero4, a4 = ok ? *(const float4*)(Ag + i) : zero4;
            S[i] = s4.x; S[i + 1] = s4.y; S[i + 2] = s4.z; S[i + 3] = s4.w;
            A[i] = a4.x; A[i + 1] = a4.y; A[i + 2] = a4.z; A[i + 3] = a4.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < NS; ++i) {
            const bool ok = live && n0 + i < N;
            S[i] = ok ? Sg[i] : 0.f;
            A[i] = ok ? Ag[i] : 0.f;
        }
    }
    const float xv = live ? to_f32(x[(size_t)t * x_stride + c]) : 0.f;
    const float zv = live ? to_f32(z[(size_t)t * z_stride + c]) : 0.f;
    const float dv = live ? dt_raw[(size_t)t * dt_stride + c] + (dt_bias ? dt_bias[c] : 0.f) : 0.f;
    const float dt = cs_softplus<T>(dv), dx = dt * xv;
    float p = 0.f, p2 = 0.f;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const bool in = n0 + i < N;
        const float bv = in ? to_f32(bm[(size_t)t * bc_stride + n0 + i]) : 0.f;
        const float cv = in ? to_f32(cm[(size_t)t * bc_stride + n0 + i]) : 0.f;
        S[i] = cs_step<T>(S[i], dt * A[i], dx * bv);
        if (i & 1) p2 = fmaf(S[i], cv, p2); else p = fmaf(S[i], cv, p);
    }
    if (VEC) {
#pragma unroll
        for (int i = 0; i < NS; i += 4)
            if (live && n0 + i < N) *(float4*)(Sg + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
    } else {
#pragma unroll
        for (int i = 0; i < NS; ++i)
            if (live && n0 + i < N) Sg[i] = S[i];
    }
    float sum = p + p2;
#pragma unroll
    for (int o = 1; o < L; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (lane_l || !live) return;
    const float skip = D ? D[c] : 0.f;
    y[(size_t)t * C + c] = from_f32<T>(fmaf(skip, xv, sum) * cs_silu<T>(zv));
    if (conv_in) cs_keep(row + conv_offset, conv_in, conv_in_stride, c, C, taps, t, 1);
}

template <typename T, int L, int NS>
static int launch_channel_scan(const void* x, long long x_stride, const void* z, long long z_stride,
                               const float* dt_raw, long long dt_stride, const float* dt_bias, const float* a2,
                               const void* bm, const void* cm, long long bc_stride, const float* D, void* y, int Tn,
                               int B, int C, int N, const int* q_start, const int* state_slots, float* state,
                               long long state_stride, long long ssm_offset, const void* conv_in,
                               long long conv_in_stride, int taps, long long conv_offset, cudaStream_t stream) {
    constexpr int CH = CS_WALK / L, NP = L * NS;
#define CS_LAUNCH(KERNEL, GRID, BLOCK, SMEM)                                                                  \
    tgo_launch_pdl(KERNEL, GRID, dim3(BLOCK), SMEM, stream, (const T*)x, x_stride, (const T*)z, z_stride,     \
                   dt_raw, dt_stride, dt_bias, a2, (const T*)bm, (const T*)cm, bc_stride, D, (T*)y, C, N, q_start, \
                   state_slots, state, state_stride, ssm_offset, (const T*)conv_in, conv_in_stride, taps, conv_offset)
    if (Tn == B) {                                       // every request brings one token
        const dim3 grid(B, (C + 128 / L - 1) / (128 / L));
        const bool vec = N % 4 == 0 && state_stride % 4 == 0 && ssm_offset % 4 == 0 && (uintptr_t)state % 16 == 0 &&
                         (uintptr_t)a2 % 16 == 0;
        if (vec) return CS_LAUNCH((channel_scan_single_kernel<T, L, NS, true>), grid, 128, 0);
        return CS_LAUNCH((channel_scan_single_kernel<T, L, NS, false>), grid, 128, 0);
    }
    constexpr int TOK = NP <= 32 ? 64 : 32;              // tokens a tile: what shared memory has room for
    const size_t smem = (size_t)2 * TOK * (2 * NP + 3 * (CH + 1)) * sizeof(float);
    auto kernel = channel_scan_kernel<T, L, NS, TOK>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return CS_LAUNCH(kernel, dim3(B, (C + CH - 1) / CH), CS_WALK + CS_SERVE(TOK, L), smem);
#undef CS_LAUNCH
}

// x, z column views [T, C], bm, cm column views [T, N] (row stride bc_stride) and conv_in a
// column view [T, C] (null: no kept inputs to move on), all in the storage type; dt_raw float32
// [T, C] (strided); a2 float32 [C, N]; y [T, C] in the storage type. A request's state [C][N] lies
// at `ssm_offset` of its state row, its kept inputs [taps - 1][C] at `conv_offset`.
TGO_API int tgo_channel_scan(const void* x, long long x_stride, const void* z, long long z_stride, int dtype,
                             const float* dt_raw, long long dt_stride, const float* dt_bias, const float* a2,
                             const void* bm, const void* cm, long long bc_stride, const float* D, void* y, int T,
                             int B, int C, int N, const int* q_start, const int* state_slots, float* state,
                             long long state_stride, long long ssm_offset, const void* conv_in,
                             long long conv_in_stride, int taps, long long conv_offset, cudaStream_t stream) {
    if (B <= 0 || T <= 0) return 0;
    if (C <= 0 || N <= 0 || N > 256 || T < B || (dtype != TGO_BF16 && dtype != TGO_F32) ||
        state_stride < ssm_offset + (long long)C * N || (C + 3) / 4 > 65535 ||
        (conv_in && (taps < 1 || state_stride < conv_offset + (long long)(taps - 1) * C)))
        return TGO_E_BAD_ARG;
#define CS_GO(L, NS)                                                                                          \
    (dtype == TGO_BF16                                                                                        \
         ? launch_channel_scan<bf16, L, NS>(x, x_stride, z, z_stride, dt_raw, dt_stride, dt_bias, a2, bm, cm,  \
                                            bc_stride, D, y, T, B, C, N, q_start, state_slots, state, state_stride, \
                                            ssm_offset, conv_in, conv_in_stride, taps, conv_offset, stream)   \
         : launch_channel_scan<float, L, NS>(x, x_stride, z, z_stride, dt_raw, dt_stride, dt_bias, a2, bm, cm, \
                                             bc_stride, D, y, T, B, C, N, q_start, state_slots, state, state_stride, \
                                             ssm_offset, conv_in, conv_in_stride, taps, conv_offset, stream))
    if (N <= 16) return CS_GO(4, 4);
    if (N <= 32) return CS_GO(4, 8);
    if (N <= 64) return CS_GO(8, 8);
    if (N <= 128) return CS_GO(16, 8);
    return CS_GO(32, 8);
#undef CS_GO
}
