// The gated delta rule: a matrix memory per head that is corrected by the error of its own recall,
//
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q          S is [dk, dv], float32
//
// over each request's tokens of the step, from and into the request's float32 state. Before the
// rule q, k and v pass a short causal convolution over time per channel and SiLU; q and k of a head
// are then divided by sqrt(sum of squares + 1e-6), q also by sqrt(dk); g = exp(-A softplus(a +
// dt_bias)) and beta = sigmoid(b) are one number per head and token. Head h uses the q and k of head
// floor(h / (H / G)). Everything after the projections is float32 whatever their storage type.
//
// Tokens are taken in pairs (0 1)(2 3).. from a request's first token of the step, so that the two
// reads of the memory by k and the two by q meet the same S. With c = k0.k1, d_ij = k_i.q_j:
//
//   u0 = b0 (v0 - g0 S^T k0)                   o0 = g0 S^T q0 + d00 u0
//   u1 = b1 (v1 - g1 (g0 S^T k1 + c u0))       o1 = g1 (g0 S^T q1 + d01 u0) + d11 u1
//   S' = g1 g0 S + k0 (g1 u0)^T + k1 u1^T
//
//   prepare   rows [T, G, 2, DKP] float32 (q, then k, unit vectors, padded with zeros to DKP = dk
//             rounded up to 32), values [T, H, dv] float32, gates [T, H] (g, g - 1, beta, 0) and
//             pairs [T, G] (k.q of the token; k and q of a pair's second token with the first's k)
//   scan      the rule over requests of any number of tokens; y [T, H dv] float32
//   step      the rule for requests of one token each, with the norm and the gate behind it
//
// A request's state row (float32, `state_stride` floats apart) holds S [H][dk][dv] at `mem_offset`
// and the convolution's last taps - 1 inputs [taps - 1][C] (oldest first) at `conv_offset`, C = 2 G
// dk + H dv channels in the order q, k, v. The prepare kernel reads the kept inputs, the kernel
// after it moves them on.
#include "common.cuh"

template <typename T> __device__ __forceinline__ float dl_exp(float x);
template <> __device__ __forceinline__ float dl_exp<float>(float x) { return expf(x); }
template <> __device__ __forceinline__ float dl_exp<bf16>(float x) { return __expf(x); }
template <typename T> __device__ __forceinline__ float dl_sigmoid(float x) { return 1.f / (1.f + dl_exp<T>(-x)); }
template <typename T> __device__ __forceinline__ float dl_silu(float x);
template <> __device__ __forceinline__ float dl_silu<float>(float x) { return x / (1.f + expf(-x)); }
template <> __device__ __forceinline__ float dl_silu<bf16>(float x) { return __fdividef(x, 1.f + __expf(-x)); }

template <typename T, int VEC> __device__ __forceinline__ void dl_load(float* v, const T* p) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = to_f32(p[i]);
}
template <> __device__ __forceinline__ void dl_load<float, 4>(float* v, const float* p) {
    const float4 q = *(const float4*)p;
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
}
template <> __device__ __forceinline__ void dl_load<bf16, 4>(float* v, const bf16* p) {
    const uint2 q = *(const uint2*)p;
    const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&q.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&q.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <int VEC> __device__ __forceinline__ void dl_store(float* p, const float* v) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) p[i] = v[i];
}
template <> __device__ __forceinline__ void dl_store<4>(float* p, const float* v) {
    *(float4*)p = make_float4(v[0], v[1], v[2], v[3]);
}

// --------------------------------------------------------------------------------- prepare
// The convolution and SiLU of VEC channels from c on for a pair: token t0 (place r0 of its portion)
// and the next one. Rows before the portion are the request's kept inputs. w [taps][C].
template <typename T, int VEC>
__device__ __forceinline__ void dl_conv_pair(float* y0, float* y1, bool two, const T* __restrict__ x,
                                             long long x_stride, const float* __restrict__ w, int C, int c,
                                             int taps, int t0, int r0, const float* __restrict__ kept) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) y0[i] = y1[i] = 0.f;
    for (int j = 0; j <= taps; ++j) {
        const int back = taps - 1 - j;                   // tokens before t0; -1: the pair's second token
        if (back < 0 && !two) break;
        float v[VEC], wj[VEC];
        if (back <= r0) dl_load<T, VEC>(v, x + (long long)(t0 - back) * x_stride + c);
        else dl_load<float, VEC>(v, kept + (size_t)(taps - 1 - (back - r0)) * C + c);
        if (j < taps) {
            dl_load<float, VEC>(wj, w + (size_t)j * C + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) y0[i] = fmaf(wj[i], v[i], y0[i]);
        }
        if (j > 0) {
            dl_load<float, VEC>(wj, w + (size_t)(j - 1) * C + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) y1[i] = fmaf(wj[i], v[i], y1[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        y0[i] = dl_silu<T>(y0[i]);
        y1[i] = dl_silu<T>(y1[i]);                       // of no use without a second token
    }
}

// A warp takes a pair and a unit: unit u < G is q and k of head u, the next `v_units` are runs of
// 32 VEC value channels, the rest 32 heads' gates each. NV rounds of 32 VEC channels cover DKP.
#define DP_WARPS 8
template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(32 * DP_WARPS)
delta_prepare_kernel(const T* __restrict__ x, long long x_stride, const float* __restrict__ w,
                     const T* __restrict__ b_raw, const T* __restrict__ a_raw, long long gate_stride,
                     const float* __restrict__ dt_bias, const float* __restrict__ A, float* __restrict__ qk,
                     float* __restrict__ v_out, float4* __restrict__ gates, float4* __restrict__ pairs, int Tn,
                     int H, int G, int dk, int dv, int dkp, int taps, float q_scale, int v_units,
                     const int* __restrict__ seq_ids, const int* __restrict__ q_start,
                     const int* __restrict__ state_slots, const float* __restrict__ state,
                     long long state_stride, long long conv_offset) {
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * DP_WARPS + warp;
    if (t >= Tn) return;
    const int b = seq_ids[t], r = t - q_start[b];
    if (r & 1) return;                                   // the second of a pair
    const bool two = t + 1 < q_start[b + 1];
    const int C = 2 * G * dk + H * dv;
    const float* kept = state + (size_t)state_slots[b] * state_stride + conv_offset;
    const int unit = blockIdx.y;
    if (unit >= G + v_units) {                           // gates
        const int h = (unit - G - v_units) * 32 + lane;
        if (h >= H) return;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            if (j && !two) break;
            const float z = to_f32(a_raw[(size_t)(t + j) * gate_stride + h]) + dt_bias[h];
            const float sp = z > 20.f ? z : log1pf(expf(z));
            const float l = -A[h] * sp;
            gates[(size_t)(t + j) * H + h] =
                make_float4(expf(l), expm1f(l), dl_sigmoid<float>(to_f32(b_raw[(size_t)(t + j) * gate_stride + h])), 0.f);
        }
        return;
    }
    if (unit >= G) {                                     // values
        const int c = ((unit - G) * 32 + lane) * VEC;
        if (c >= H * dv) return;
        float y0[VEC], y1[VEC];
        dl_conv_pair<T, VEC>(y0, y1, two, x, x_stride, w, C, 2 * G * dk + c, taps, t, r, kept);
        dl_store<VEC>(v_out + (size_t)t * H * dv + c, y0);
        if (two) dl_store<VEC>(v_out + (size_t)(t + 1) * H * dv + c, y1);
        return;
    }
    float q[2][NV * VEC], k[2][NV * VEC];
    float s[8];                                          // q0q0 q1q1 k0k0 k1k1 k0q0 k1q1 k0k1 k0q1
#pragma unroll
    for (int i = 0; i < 8; ++i) s[i] = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = (n * 32 + lane) * VEC;
        float* q0 = q[0] + n * VEC;
        float* q1 = q[1] + n * VEC;
        float* k0 = k[0] + n * VEC;
        float* k1 = k[1] + n * VEC;
        if (c < dk) {
            dl_conv_pair<T, VEC>(q0, q1, two, x, x_stride, w, C, unit * dk + c, taps, t, r, kept);
            dl_conv_pair<T, VEC>(k0, k1, two, x, x_stride, w, C, (G + unit) * dk + c, taps, t, r, kept);
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) q0[i] = q1[i] = k0[i] = k1[i] = 0.f;
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            s[0] = fmaf(q0[i], q0[i], s[0]);
            s[1] = fmaf(q1[i], q1[i], s[1]);
            s[2] = fmaf(k0[i], k0[i], s[2]);
            s[3] = fmaf(k1[i], k1[i], s[3]);
            s[4] = fmaf(k0[i], q0[i], s[4]);
            s[5] = fmaf(k1[i], q1[i], s[5]);
            s[6] = fmaf(k0[i], k1[i], s[6]);
            s[7] = fmaf(k0[i], q1[i], s[7]);
        }
    }
    // eight sums over 32 lanes: with each of the first rounds a lane keeps half of its values; sum i
    // ends in the lanes whose bits 4, 3, 2 spell i
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
        const bool up = lane & (o * 4);
#pragma unroll
        for (int i = 0; i < o; ++i) {
            const float give = up ? s[i] : s[i + o], have = up ? s[i + o] : s[i];
            s[i] = have + __shfl_xor_sync(0xffffffffu, give, o * 4);
        }
    }
    float sum = s[0];
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    float f[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = __shfl_sync(0xffffffffu, sum, 4 * i);
    const float rq0 = q_scale / sqrtf(f[0] + 1e-6f), rq1 = q_scale / sqrtf(f[1] + 1e-6f);
    const float rk0 = 1.f / sqrtf(f[2] + 1e-6f), rk1 = 1.f / sqrtf(f[3] + 1e-6f);
    float* row = qk + ((size_t)t * G + unit) * 2 * dkp;
    const size_t next = (size_t)G * 2 * dkp;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = (n * 32 + lane) * VEC;
        if (c >= dkp) break;
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            q[0][n * VEC + i] *= rq0;
            q[1][n * VEC + i] *= rq1;
            k[0][n * VEC + i] *= rk0;
            k[1][n * VEC + i] *= rk1;
        }
        dl_store<VEC>(row + c, q[0] + n * VEC);
        dl_store<VEC>(row + dkp + c, k[0] + n * VEC);
        if (two) {
            dl_store<VEC>(row + next + c, q[1] + n * VEC);
            dl_store<VEC>(row + next + dkp + c, k[1] + n * VEC);
        }
    }
    if (lane == 0) {
        pairs[(size_t)t * G + unit] = make_float4(f[4] * rk0 * rq0, 0.f, 0.f, 0.f);
        if (two) pairs[(size_t)(t + 1) * G + unit] = make_float4(f[5] * rk1 * rq1, f[6] * rk0 * rk1, f[7] * rk0 * rq1, 0.f);
    }
}

// x [T, C] a column view in the storage type (q, k, v side by side), b_raw and a_raw [T, H] column
// views with one stride; w float32 [taps][C], dt_bias and A = exp(A_log) float32 [H].
TGO_API int tgo_delta_prepare(const void* x, long long x_stride, int dtype, const float* w, const void* b_raw,
                              const void* a_raw, long long gate_stride, const float* dt_bias, const float* A,
                              float* qk, float* v_out, float* gates, float* pairs, int T, int B, int H, int G,
                              int dk, int dv, int taps, const int* seq_ids, const int* q_start,
                              const int* state_slots, const float* state, long long state_stride,
                              long long conv_offset, cudaStream_t stream) {
    if (T <= 0 || B <= 0) return 0;
    const int C = 2 * G * dk + H * dv, dkp = (dk + 31) / 32 * 32;
    if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > 256 || dv <= 0 || taps <= 0 || taps > 64 ||
        state_stride < conv_offset + (long long)(taps - 1) * C || (uintptr_t)qk % 16 || (uintptr_t)gates % 16 ||
        (uintptr_t)pairs % 16 || (dtype != TGO_BF16 && dtype != TGO_F32))
        return TGO_E_BAD_ARG;
    const uintptr_t width = dtype == TGO_BF16 ? 8 : 16;  // bytes of four elements
    const bool quads = dk % 4 == 0 && dv % 4 == 0 && x_stride % 4 == 0 && (uintptr_t)x % width == 0 &&
                       (uintptr_t)w % 16 == 0 && (uintptr_t)v_out % 16 == 0 && (uintptr_t)state % 16 == 0 &&
                       state_stride % 4 == 0 && conv_offset % 4 == 0;
    const int per = quads ? 128 : 32, v_units = (H * dv + per - 1) / per;
    const long long units = (long long)G + v_units + (H + 31) / 32;
    if (units > 65535) return TGO_E_BAD_ARG;
    const dim3 grid((T + DP_WARPS - 1) / DP_WARPS, (unsigned)units);
    const float q_scale = 1.f / sqrtf((float)dk);
#define DP_GO(TT, VEC, NV)                                                                                 \
    tgo_launch_pdl(delta_prepare_kernel<TT, VEC, NV>, grid, dim3(32 * DP_WARPS), 0, stream, (const TT*)x, x_stride, \
                   w, (const TT*)b_raw, (const TT*)a_raw, gate_stride, dt_bias, A, qk, v_out, (float4*)gates, \
                   (float4*)pairs, T, H, G, dk, dv, dkp, taps, q_scale, v_units, seq_ids, q_start, state_slots, \
                   state, state_stride, conv_offset)
#define DP_SIZE(TT) (quads ? (dkp <= 128 ? DP_GO(TT, 4, 1) : DP_GO(TT, 4, 2))                              \
                           : (dkp <= 64 ? DP_GO(TT, 1, 2) : dkp <= 128 ? DP_GO(TT, 1, 4) : DP_GO(TT, 1, 8)))
    return dtype == TGO_BF16 ? DP_SIZE(bf16) : DP_SIZE(float);
#undef DP_SIZE
#undef DP_GO
}

// ------------------------------------------------------------------------ kept inputs
// The kept inputs of channel c become the last taps - 1 of (kept, then the step's). Ascending i
// reads kept[n_tok + i] before any later write could reach it.
template <typename T>
__device__ __forceinline__ void dl_keep(float* kept, const T* __restrict__ x, long long x_stride, int c, int C,
                                        int taps, int t0, int n_tok) {
    const int keep = taps - 1;
    for (int i = 0; i < keep; ++i) {
        const int at = n_tok + i;
        kept[(size_t)i * C + c] = at < keep ? kept[(size_t)at * C + c]
                                            : to_f32(x[(size_t)(t0 + at - keep) * x_stride + c]);
    }
}
// The channels that the block of head h (value columns c0 .. c0 + n - 1) moves on: those columns,
// and for the first block of the first head of a group the group's q and k.
template <typename T>
__device__ __forceinline__ void dl_keep_block(float* kept, const T* __restrict__ x, long long x_stride, int H, int G,
                                              int dk, int dv, int h, int c0, int n, int taps, int t0, int n_tok) {
    const int C = 2 * G * dk + H * dv, per = H / G, g = h / per;
    for (int i = threadIdx.x; i < n; i += blockDim.x)
        if (c0 + i < dv) dl_keep(kept, x, x_stride, 2 * G * dk + h * dv + c0 + i, C, taps, t0, n_tok);
    if (c0 == 0 && h % per == 0)
        for (int i = threadIdx.x; i < 2 * dk; i += blockDim.x)
            dl_keep(kept, x, x_stride, i < dk ? g * dk + i : (G + g) * dk + i - dk, C, taps, t0, n_tok);
}

// ----------------------------------------------------------------------------------- scan
// A block per (request, head, 16 columns of dv). A warp holds four columns, lane = 4 slice + column:
// slice s keeps rows 32 i + 4 s + j (j = 0..3) of its column of S in registers for the whole walk
// over the request's tokens. A pair costs four products with S, one exchange over the slices that
// leaves a sum in each quarter of the warp, two broadcasts of the reads by k, and one update of S.
// DS_TOK tokens at a time come through shared memory by asynchronous copies, two buffers. The order
// of every sum depends on the sizes alone.
#define DS_TOK 16
#define DS_COLS 16
#define DS_THREADS (8 * DS_COLS)

__device__ __forceinline__ void ds_copy4(float* dst, const float* src, bool valid) {
    const int n = valid ? 4 : 0;
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(
                     (uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(n));
}
__device__ __forceinline__ void ds_copy16(float* dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(
                     (uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(n));
}

// g x. A memory that decays slowly is multiplied by nearly 1 a thousand times, and a factor rounded
// to the same side each time adds up: the float32 engine adds (g - 1) x while the decay is slow,
// whose rounding is relative to the change.
template <typename T> __device__ __forceinline__ float dl_decay(float x, float g, float gm1);
template <> __device__ __forceinline__ float dl_decay<bf16>(float x, float g, float gm1) { return g * x; }
template <> __device__ __forceinline__ float dl_decay<float>(float x, float g, float gm1) {
    return gm1 > -0.3f ? fmaf(gm1, x, x) : g * x;
}

template <typename T, int NI>
__global__ void __launch_bounds__(DS_THREADS)
delta_scan_kernel(const float* __restrict__ qk, const float* __restrict__ v, const float4* __restrict__ gates,
                  const float4* __restrict__ pairs, float* __restrict__ y, int H, int G, int dk, int dv,
                  const int* __restrict__ q_start, const int* __restrict__ state_slots, float* __restrict__ state,
                  long long state_stride, long long mem_offset, const T* __restrict__ conv_in,
                  long long conv_in_stride, int taps, long long conv_offset) {
    constexpr int DKP = NI * 8;
    constexpr int BUF = DS_TOK * (2 * DKP + DS_COLS + 8);
    extern __shared__ __align__(16) float smem[];        // 2 x { qk [TOK][2 DKP], gates [TOK][4], pairs [TOK][4], v }
    pdl_wait();
    const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * DS_COLS;
    const int t0 = q_start[b], n_tok = q_start[b + 1] - t0;
    if (n_tok <= 0) return;
    const int g = h / (H / G);
    const int lane = threadIdx.x & 31, col = (threadIdx.x >> 5) * 4 + (lane & 3), s = lane >> 2;
    const int c = c0 + col;
    float* row = state + (size_t)state_slots[b] * state_stride;
    float* Sg = row + mem_offset + (size_t)h * dk * dv;
    // the memory comes and goes through shared memory ([dk][COLS + 1] floats fit in the buffers)
    for (int i = threadIdx.x; i < dk * DS_COLS; i += DS_THREADS) {
        const int n = i / DS_COLS, cc = i % DS_COLS;
        smem[n * (DS_COLS + 1) + cc] = c0 + cc < dv ? Sg[(size_t)n * dv + c0 + cc] : 0.f;
    }
    __syncthreads();
    float S[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = 32 * (i >> 2) + 4 * s + (i & 3);
        S[i] = n < dk ? smem[n * (DS_COLS + 1) + col] : 0.f;
    }
    __syncthreads();
    auto stage = [&](int base, int buf) {
        float* qks = smem + buf * BUF;
        float* gs = qks + DS_TOK * 2 * DKP;
        float* ps = gs + DS_TOK * 4;
        float* vs = ps + DS_TOK * 4;
        const int nt = n_tok - base < DS_TOK ? n_tok - base : DS_TOK, ne = (nt + 1) & ~1;
        for (int i = threadIdx.x; i < ne * (2 * DKP / 4); i += DS_THREADS) {
            const int r = i / (2 * DKP / 4), q = i % (2 * DKP / 4);
            const bool ok = r < nt;
            ds_copy16(qks + 4 * i, ok ? qk + ((size_t)(t0 + base + r) * G + g) * 2 * DKP + 4 * q : qk, ok);
        }
        for (int i = threadIdx.x; i < ne * DS_COLS; i += DS_THREADS) {
            const int r = i / DS_COLS, cc = i % DS_COLS;
            const bool ok = r < nt && c0 + cc < dv;
            ds_copy4(vs + i, ok ? v + ((size_t)(t0 + base + r) * H + h) * dv + c0 + cc : v, ok);
        }
        if (threadIdx.x < ne) {
            const bool ok = threadIdx.x < nt;
            const size_t at = t0 + base + threadIdx.x;
            ds_copy16(gs + 4 * threadIdx.x, ok ? (const void*)(gates + at * H + h) : (const void*)gates, ok);
            ds_copy16(ps + 4 * threadIdx.x, ok ? (const void*)(pairs + at * G + g) : (const void*)pairs, ok);
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    const bool upper = lane & 16, second = lane & 8;     // this lane's sum: by q (else k), of token 1 (else 0)
    stage(0, 0);
    for (int base = 0, buf = 0; base < n_tok; base += DS_TOK, buf ^= 1) {
        const int nt = n_tok - base < DS_TOK ? n_tok - base : DS_TOK;
        if (base + DS_TOK < n_tok) {
            stage(base + DS_TOK, buf ^ 1);                // the buffer the last pass left
            asm volatile("cp.async.wait_group 1;\n" ::);
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::);
        }
        __syncthreads();
        const float* qks = smem + buf * BUF;
        const float* gs = qks + DS_TOK * 2 * DKP;
        const float* ps = gs + DS_TOK * 4;
        const float* vs = ps + DS_TOK * 4;
        for (int r = 0; r < nt; r += 2) {
            const float* q0 = qks + r * 2 * DKP + 4 * s;
            const float* k0 = q0 + DKP;
            const float* q1 = q0 + 2 * DKP;
            const float* k1 = q1 + DKP;
            const float4 ga = *(const float4*)(gs + 4 * r), pa = *(const float4*)(ps + 4 * r);
            float4 gb = *(const float4*)(gs + 4 * r + 4), pb = *(const float4*)(ps + 4 * r + 4);
            if (r + 1 >= nt) gb.x = 1.f;                 // no second token: it neither decays nor writes
            const float va = vs[r * DS_COLS + col], vb = vs[(r + 1) * DS_COLS + col];
            float4 ka[NI / 4], kb[NI / 4];
            float sk0 = 0.f, sk1 = 0.f, sq0 = 0.f, sq1 = 0.f, tk0 = 0.f, tk1 = 0.f, tq0 = 0.f, tq1 = 0.f;
#pragma unroll
            for (int i = 0; i < NI / 4; ++i) {
                ka[i] = *(const float4*)(k0 + 32 * i);
                kb[i] = *(const float4*)(k1 + 32 * i);
                const float4 qa = *(const float4*)(q0 + 32 * i), qb = *(const float4*)(q1 + 32 * i);
                const float x = S[4 * i], yy = S[4 * i + 1], z = S[4 * i + 2], w = S[4 * i + 3];
                sk0 = fmaf(ka[i].x, x, sk0); tk0 = fmaf(ka[i].y, yy, tk0);
                sk1 = fmaf(kb[i].x, x, sk1); tk1 = fmaf(kb[i].y, yy, tk1);
                sq0 = fmaf(qa.x, x, sq0);    tq0 = fmaf(qa.y, yy, tq0);
                sq1 = fmaf(qb.x, x, sq1);    tq1 = fmaf(qb.y, yy, tq1);
                sk0 = fmaf(ka[i].z, z, sk0); tk0 = fmaf(ka[i].w, w, tk0);
                sk1 = fmaf(kb[i].z, z, sk1); tk1 = fmaf(kb[i].w, w, tk1);
                sq0 = fmaf(qa.z, z, sq0);    tq0 = fmaf(qa.w, w, tq0);
                sq1 = fmaf(qb.z, z, sq1);    tq1 = fmaf(qb.w, w, tq1);
            }
            sk0 += tk0; sk1 += tk1; sq0 += tq0; sq1 += tq1;
            float a0 = upper ? sq0 : sk0, a1 = upper ? sq1 : sk1;
            a0 += __shfl_xor_sync(0xffffffffu, upper ? sk0 : sq0, 16);
            a1 += __shfl_xor_sync(0xffffffffu, upper ? sk1 : sq1, 16);
            float m = second ? a1 : a0;
            m += __shfl_xor_sync(0xffffffffu, second ? a0 : a1, 8);
            m += __shfl_xor_sync(0xffffffffu, m, 4);
            const float rk0 = __shfl_sync(0xffffffffu, m, lane & 3), rk1 = __shfl_sync(0xffffffffu, m, 8 + (lane & 3));
            const float u0 = ga.z * (va - dl_decay<T>(rk0, ga.x, ga.y));
            const float u1 = gb.z * (vb - dl_decay<T>(fmaf(pb.y, u0, dl_decay<T>(rk1, ga.x, ga.y)), gb.x, gb.y));
            const float w0 = dl_decay<T>(u0, gb.x, gb.y);
            const float gm = fmaf(ga.y, gb.y, ga.y + gb.y), gg = ga.x * gb.x;
            if (sizeof(T) == 4 && gm > -0.3f) {
#pragma unroll
                for (int i = 0; i < NI / 4; ++i) {
                    S[4 * i] += fmaf(gm, S[4 * i], fmaf(kb[i].x, u1, ka[i].x * w0));
                    S[4 * i + 1] += fmaf(gm, S[4 * i + 1], fmaf(kb[i].y, u1, ka[i].y * w0));
                    S[4 * i + 2] += fmaf(gm, S[4 * i + 2], fmaf(kb[i].z, u1, ka[i].z * w0));
                    S[4 * i + 3] += fmaf(gm, S[4 * i + 3], fmaf(kb[i].w, u1, ka[i].w * w0));
                }
            } else {
#pragma unroll
                for (int i = 0; i < NI / 4; ++i) {
                    S[4 * i] = fmaf(kb[i].x, u1, fmaf(ka[i].x, w0, gg * S[4 * i]));
                    S[4 * i + 1] = fmaf(kb[i].y, u1, fmaf(ka[i].y, w0, gg * S[4 * i + 1]));
                    S[4 * i + 2] = fmaf(kb[i].z, u1, fmaf(ka[i].z, w0, gg * S[4 * i + 2]));
                    S[4 * i + 3] = fmaf(kb[i].w, u1, fmaf(ka[i].w, w0, gg * S[4 * i + 3]));
                }
            }
            if (upper && !(lane & 4) && c < dv && r + (second ? 1 : 0) < nt) {
                const float first = dl_decay<T>(m, ga.x, ga.y);
                const float o = second ? fmaf(pb.x, u1, dl_decay<T>(fmaf(pb.z, u0, first), gb.x, gb.y))
                                       : fmaf(pa.x, u0, first);
                y[((size_t)(t0 + base + r + (second ? 1 : 0)) * H + h) * dv + c] = o;
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = 32 * (i >> 2) + 4 * s + (i & 3);
        if (n < dk) smem[n * (DS_COLS + 1) + col] = S[i];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < dk * DS_COLS; i += DS_THREADS) {
        const int n = i / DS_COLS, cc = i % DS_COLS;
        if (c0 + cc < dv) Sg[(size_t)n * dv + c0 + cc] = smem[n * (DS_COLS + 1) + cc];
    }
    dl_keep_block(row + conv_offset, conv_in, conv_in_stride, H, G, dk, dv, h, c0, DS_COLS, taps, t0, n_tok);
}

template <typename T, int NI>
static int launch_delta_scan(const float* qk, const float* v, const float* gates, const float* pairs, float* y,
                             int B, int H, int G, int dk, int dv, const int* q_start, const int* state_slots,
                             float* state, long long state_stride, long long mem_offset, const T* conv_in,
                             long long conv_in_stride, int taps, long long conv_offset, cudaStream_t stream) {
    const size_t smem = 2 * (size_t)DS_TOK * (2 * NI * 8 + DS_COLS + 8) * sizeof(float);
    auto kernel = delta_scan_kernel<T, NI>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return tgo_launch_pdl(kernel, dim3(B, H, (dv + DS_COLS - 1) / DS_COLS), dim3(DS_THREADS), smem, stream, qk, v,
                          (const float4*)gates, (const float4*)pairs, y, H, G, dk, dv, q_start, state_slots, state,
                          state_stride, mem_offset, conv_in, conv_in_stride, taps, conv_offset);
}

static bool delta_sizes_ok(int H, int G, int dk, int dv, int taps, long long state_stride, long long mem_offset,
                           long long conv_offset) {
    return H > 0 && G > 0 && H % G == 0 && H <= 65535 && dk > 0 && dk <= 256 && dv > 0 && dv <= 65535 * DS_COLS &&
           taps > 0 && taps <= 64 && state_stride >= mem_offset + (long long)H * dk * dv &&
           state_stride >= conv_offset + (long long)(taps - 1) * (2 * G * dk + H * dv);
}

TGO_API int tgo_delta_scan(const float* qk, const float* v, const float* gates, const float* pairs, float* y, int B,
                           int H, int G, int dk, int dv, const int* q_start, const int* state_slots, float* state,
                           long long state_stride, long long mem_offset, const void* conv_in,
                           long long conv_in_stride, int dtype, int taps, long long conv_offset,
                           cudaStream_t stream) {
    if (B <= 0) return 0;
    if (!delta_sizes_ok(H, G, dk, dv, taps, state_stride, mem_offset, conv_offset) || (uintptr_t)qk % 16 ||
        (uintptr_t)gates % 16 || (uintptr_t)pairs % 16 || (dtype != TGO_BF16 && dtype != TGO_F32))
        return TGO_E_BAD_ARG;
#define DS_GO(TT, NI)                                                                                      \
    launch_delta_scan<TT, NI>(qk, v, gates, pairs, y, B, H, G, dk, dv, q_start, state_slots, state, state_stride, \
                              mem_offset, (const TT*)conv_in, conv_in_stride, taps, conv_offset, stream)
#define DS_CASE(n) case n: return dtype == TGO_BF16 ? DS_GO(bf16, 4 * n) : DS_GO(float, 4 * n);
    switch ((dk + 31) / 32) {                            // the rows are DKP = 32 n wide
        DS_CASE(1) DS_CASE(2) DS_CASE(3) DS_CASE(4) DS_CASE(5) DS_CASE(6) DS_CASE(7) DS_CASE(8)
    }
#undef DS_CASE
#undef DS_GO
    return TGO_E_BAD_ARG;
}

// ----------------------------------------------------------------------------------- step
// Requests of one token each. A block per (request, head): thread (row group q, column quad) holds
// rows q, q + R, .. of four columns of S in registers between the reads and the update, so the memory
// is read and written once, in whole rows. The reads by k and q are joined over the row groups
// through shared memory, in order. Then, in the same block, the head's output is divided by its root
// mean square over dv, multiplied by the gain [dv] and by SiLU of the gate.
#define DT_THREADS 512
template <typename T, int NR>
__global__ void __launch_bounds__(DT_THREADS)
delta_step_kernel(const float* __restrict__ qk, const float* __restrict__ v, const float4* __restrict__ gates,
                  const float4* __restrict__ pairs, const T* __restrict__ z, long long z_stride,
                  const float* __restrict__ gain, float eps, T* __restrict__ out, int H, int G, int dk, int dv,
                  int dkp, const int* __restrict__ q_start, const int* __restrict__ state_slots,
                  float* __restrict__ state, long long state_stride, long long mem_offset,
                  const T* __restrict__ conv_in, long long conv_in_stride, int taps, long long conv_offset) {
    extern __shared__ __align__(16) float smem[];        // qk [2 dkp], u [dv], parts [2][R][dv]
    __shared__ float scratch[33];
    pdl_wait();
    const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int t = q_start[b];
    if (q_start[b + 1] - t <= 0) return;
    const int QN = dv / 4, R = DT_THREADS / QN, g = h / (H / G);
    const int rg = tid / QN, quad = tid % QN;
    const bool works = rg < R;
    float* qs = smem;
    float* us = qs + 2 * dkp;
    float* part = us + dv;
    float* row = state + (size_t)state_slots[b] * state_stride;
    float* Sg = row + mem_offset + (size_t)h * dk * dv + 4 * quad;
    float4 S[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int n = rg + i * R;
        S[i] = (works && n < dk) ? *(const float4*)(Sg + (size_t)n * dv) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float4 gt = gates[(size_t)t * H + h], pr = pairs[(size_t)t * G + g];
    for (int i = tid; i < 2 * dkp; i += DT_THREADS) qs[i] = qk[((size_t)t * G + g) * 2 * dkp + i];
    __syncthreads();
    if (works) {
        float4 sk = make_float4(0.f, 0.f, 0.f, 0.f), sq = sk;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int n = rg + i * R;
            if (n < dk) {
                const float kn = qs[dkp + n], qn = qs[n];
                sk.x = fmaf(kn, S[i].x, sk.x); sk.y = fmaf(kn, S[i].y, sk.y);
                sk.z = fmaf(kn, S[i].z, sk.z); sk.w = fmaf(kn, S[i].w, sk.w);
                sq.x = fmaf(qn, S[i].x, sq.x); sq.y = fmaf(qn, S[i].y, sq.y);
                sq.z = fmaf(qn, S[i].z, sq.z); sq.w = fmaf(qn, S[i].w, sq.w);
            }
        }
        *(float4*)(part + (size_t)rg * dv + 4 * quad) = sk;
        *(float4*)(part + (size_t)(R + rg) * dv + 4 * quad) = sq;
    }
    __syncthreads();
    float o = 0.f;
    if (tid < dv) {
        float sk = 0.f, sq = 0.f;
        for (int i = 0; i < R; ++i) {
            sk += part[(size_t)i * dv + tid];
            sq += part[(size_t)(R + i) * dv + tid];
        }
        const float u = gt.z * (v[((size_t)t * H + h) * dv + tid] - dl_decay<T>(sk, gt.x, gt.y));
        us[tid] = u;
        o = fmaf(pr.x, u, dl_decay<T>(sq, gt.x, gt.y));
    }
    const float ss = block_sum(o * o, scratch);          // its barriers make `us` visible too
    if (works) {
        const float4 u = *(const float4*)(us + 4 * quad);
        const bool slow = sizeof(T) == 4 && gt.y > -0.3f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int n = rg + i * R;
            if (n < dk) {
                const float kn = qs[dkp + n];
                float4 r;
                if (slow) {
                    r.x = S[i].x + fmaf(gt.y, S[i].x, kn * u.x); r.y = S[i].y + fmaf(gt.y, S[i].y, kn * u.y);
                    r.z = S[i].z + fmaf(gt.y, S[i].z, kn * u.z); r.w = S[i].w + fmaf(gt.y, S[i].w, kn * u.w);
                } else {
                    r.x = fmaf(kn, u.x, gt.x * S[i].x); r.y = fmaf(kn, u.y, gt.x * S[i].y);
                    r.z = fmaf(kn, u.z, gt.x * S[i].z); r.w = fmaf(kn, u.w, gt.x * S[i].w);
                }
                *(float4*)(Sg + (size_t)n * dv) = r;
            }
        }
    }
    if (tid < dv) {
        const float a = (o * rsqrtf(ss / (float)dv + eps)) * gain[tid];
        out[((size_t)t * H + h) * dv + tid] =
            from_f32<T>(a * dl_silu<T>(to_f32(z[(size_t)t * z_stride + (size_t)h * dv + tid])));
    }
    dl_keep_block(row + conv_offset, conv_in, conv_in_stride, H, G, dk, dv, h, 0, dv, taps, t, 1);
}

TGO_API int tgo_delta_step_supports(int H, int G, int dk, int dv, long long state_stride, long long mem_offset) {
    if (H <= 0 || G <= 0 || H % G || H > 65535 || dk <= 0 || dk > 256 || dv <= 0 || dv > DT_THREADS || dv % 4 ||
        state_stride % 4 || mem_offset % 4)
        return 0;
    const int R = DT_THREADS / (dv / 4);
    return (dk + R - 1) / R <= 16 ? 1 : 0;
}

TGO_API int tgo_delta_step(const float* qk, const float* v, const float* gates, const float* pairs, const void* z,
                           long long z_stride, const float* gain, float eps, void* out, int B, int H, int G, int dk,
                           int dv, const int* q_start, const int* state_slots, float* state, long long state_stride,
                           long long mem_offset, const void* conv_in, long long conv_in_stride, int dtype, int taps,
                           long long conv_offset, cudaStream_t stream) {
    if (B <= 0) return 0;
    if (!tgo_delta_step_supports(H, G, dk, dv, state_stride, mem_offset) ||
        !delta_sizes_ok(H, G, dk, dv, taps, state_stride, mem_offset, conv_offset) || (uintptr_t)state % 16 ||
        (uintptr_t)gates % 16 || (uintptr_t)pairs % 16 || (dtype != TGO_BF16 && dtype != TGO_F32))
        return TGO_E_BAD_ARG;
    const int R = DT_THREADS / (dv / 4), nr = (dk + R - 1) / R, dkp = (dk + 31) / 32 * 32;
    const size_t smem = ((size_t)2 * dkp + dv + (size_t)2 * R * dv) * sizeof(float);    // at most 20 KB
#define DT_GO(TT, NR)                                                                                      \
    tgo_launch_pdl(delta_step_kernel<TT, NR>, dim3(B, H), dim3(DT_THREADS), smem, stream, qk, v, (const float4*)gates, \
                   (const float4*)pairs, (const TT*)z, z_stride, gain, eps, (TT*)out, H, G, dk, dv, dkp, q_start, \
                   state_slots, state, state_stride, mem_offset, (const TT*)conv_in, conv_in_stride, taps, conv_offset)
#define DT_SIZE(TT) (nr <= 1 ? DT_GO(TT, 1) : nr <= 2 ? DT_GO(TT, 2) : nr <= 4 ? DT_GO(TT, 4) : nr <= 8 ? DT_GO(TT, 8) \
                                                                                 : DT_GO(TT, 16))
    return dtype == TGO_BF16 ? DT_SIZE(bf16) : DT_SIZE(float);
#undef DT_SIZE
#undef DT_GO
}
