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
// Tokens are taken four at a time, (0 1 2 3)(4 5 6 7).. from a request's first token of the step, so
// that the reads of the memory by four k and four q meet the same S and the exchanges between
// threads are paid once. With P_j = g_0 .. g_j, E_j = g_j+1 .. g_last and S as it was before the four:
//
//   u_j = b_j v_j - b_j P_j S^T k_j - sum_(m<j) b_j (P_j / P_m) (k_m.k_j) u_m
//   o_j = P_j S^T q_j + sum_(m<=j) (P_j / P_m) (k_m.q_j) u_m
//   S'  = P_last S + sum_j k_j (E_j u_j)^T
//
// where the ratios are exponentials of sums of the tokens' log decays, and every factor that does not
// depend on S is made ahead:
//
//   prepare   rows [T, G, 2, DKP] float32 (q, then k, unit vectors, padded with zeros to DKP = 32, 64,
//             128 or 256), values b v [T, H, dv] float32 and records [T, H, 12]: for token j of a four
//             (b P_j, b x the three k_m.k_j terms; the four k_m.q_j terms; P_j, E_j, P_last, P_last - 1)
//   scan      the rule over requests of any number of tokens; y [T, H dv] float32
//   step      the rule for requests of one token each, with the norm and the gate behind it
//
// A request's state row (float32, `state_stride` floats apart) holds S [H][dk][dv] at `mem_offset`
// and the convolution's last taps - 1 inputs [taps - 1][C] (oldest first) at `conv_offset`, C = 2 G
// dk + H dv channels in the order q, k, v. The prepare kernel reads the kept inputs, the kernel
// after it moves them on.
#include "common.cuh"

static int delta_row_width(int dk) { return dk <= 32 ? 32 : dk <= 64 ? 64 : dk <= 128 ? 128 : 256; }

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
// The convolution and SiLU of VEC channels from c on for up to four tokens: t0 (place r0 of its
// portion) and the `count - 1` after it. Rows before the portion are the request's kept inputs. w
// [taps][C]. Tokens past `count` come out as zeros.
#define DP_GROUP 4
template <typename T, int VEC, int TAPS>
__device__ __forceinline__ void dl_conv(float (*y)[VEC], int count, const T* __restrict__ x, long long x_stride,
                                        const float* __restrict__ w, int C, int c, int taps, int t0, int r0,
                                        const float* __restrict__ kept) {
#pragma unroll
    for (int u = 0; u < DP_GROUP; ++u)
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[u][i] = 0.f;
    auto input = [&](float* v, int back) {               // `back` tokens before t0; negative: after it
        if (back <= r0) dl_load<T, VEC>(v, x + (long long)(t0 - back) * x_stride + c);
        else dl_load<float, VEC>(v, kept + (size_t)(taps - 1 - (back - r0)) * C + c);
    };
    if (TAPS > 0) {                                      // every load ahead of the sums
        float v[TAPS + DP_GROUP - 1][VEC], wt[TAPS > 0 ? TAPS : 1][VEC];
#pragma unroll
        for (int j = 0; j < TAPS + DP_GROUP - 1; ++j) {
            if (j - (TAPS - 1) < count) {
                input(v[j], TAPS - 1 - j);
            } else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) v[j][i] = 0.f;
            }
        }
#pragma unroll
        for (int q = 0; q < TAPS; ++q) dl_load<float, VEC>(wt[q], w + (size_t)q * C + c);
#pragma unroll
        for (int u = 0; u < DP_GROUP; ++u)
#pragma unroll
            for (int q = 0; q < TAPS; ++q)
#pragma unroll
                for (int i = 0; i < VEC; ++i) y[u][i] = fmaf(wt[q][i], v[u + q][i], y[u][i]);
    } else {
        for (int j = 0; j < taps + DP_GROUP - 1 && j - (taps - 1) < count; ++j) {
            float v[VEC];
            input(v, taps - 1 - j);
#pragma unroll
            for (int u = 0; u < DP_GROUP; ++u) {         // this input meets tap j - u of token u
                if (j < u || j - u >= taps) continue;
                float wj[VEC];
                dl_load<float, VEC>(wj, w + (size_t)(j - u) * C + c);
#pragma unroll
                for (int i = 0; i < VEC; ++i) y[u][i] = fmaf(wj[i], v[i], y[u][i]);
            }
        }
    }
#pragma unroll
    for (int u = 0; u < DP_GROUP; ++u)
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[u][i] = u < count ? dl_silu<T>(y[u][i]) : 0.f;
}

// A warp takes four tokens and a unit: unit u < G is q and k of head u and the records of
// its group's heads, the others are runs of 32 VEC value channels. NV rounds of 32 VEC channels cover DKP.
// A warp looks for the first tokens of fours among `per` consecutive ones: 4 in prompts, 1 in steps of
// single tokens.
#define DP_WARPS 4
template <typename T, int VEC, int NV, int TAPS>
__device__ __forceinline__ void
delta_prepare_four(int t, int b, int r, const T* __restrict__ x, long long x_stride, const float* __restrict__ w,
                   const T* __restrict__ b_raw, const T* __restrict__ a_raw, long long gate_stride,
                   const float* __restrict__ dt_bias, const float* __restrict__ A, float* __restrict__ qk,
                   float* __restrict__ v_out, float4* __restrict__ records,
                   int H, int G, int dk, int dv, int dkp, int taps, float q_scale,
                   const int* __restrict__ q_start, const int* __restrict__ state_slots,
                   const float* __restrict__ state, long long state_stride, long long conv_offset) {
    const int lane = threadIdx.x & 31;
    const int left = q_start[b + 1] - t, count = left < DP_GROUP ? left : DP_GROUP;
    const int C = 2 * G * dk + H * dv;
    const float* kept = state + (size_t)state_slots[b] * state_stride + conv_offset;
    const int unit = blockIdx.y;
    if (unit >= G) {                                     // values, times their steps
        const int c = ((unit - G) * 32 + lane) * VEC;
        if (c >= H * dv) return;
        float y[DP_GROUP][VEC];
        dl_conv<T, VEC, TAPS>(y, count, x, x_stride, w, C, 2 * G * dk + c, taps, t, r, kept);
#pragma unroll
        for (int u = 0; u < DP_GROUP; ++u)
            if (u < count) {
                const float beta = dl_sigmoid<T>(to_f32(b_raw[(size_t)(t + u) * gate_stride + c / dv]));
#pragma unroll
                for (int i = 0; i < VEC; ++i) y[u][i] *= beta;
                dl_store<VEC>(v_out + (size_t)(t + u) * H * dv + c, y[u]);
            }
        return;
    }
    float q[NV][DP_GROUP][VEC], k[NV][DP_GROUP][VEC];
    // sums 0-3 q_j.q_j, 4-7 k_j.k_j, 8-11 k_j.q_j, 12-17 c_ij, 18-23 d_ij for ij = 01 02 12 03 13 23
    float s[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) s[i] = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = (n * 32 + lane) * VEC;
        if (c < dk) {
            dl_conv<T, VEC, TAPS>(q[n], count, x, x_stride, w, C, unit * dk + c, taps, t, r, kept);
            dl_conv<T, VEC, TAPS>(k[n], count, x, x_stride, w, C, (G + unit) * dk + c, taps, t, r, kept);
        } else {
#pragma unroll
            for (int u = 0; u < DP_GROUP; ++u)
#pragma unroll
                for (int i = 0; i < VEC; ++i) q[n][u][i] = k[n][u][i] = 0.f;
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            int at = 0;
#pragma unroll
            for (int u = 0; u < DP_GROUP; ++u) {
                s[u] = fmaf(q[n][u][i], q[n][u][i], s[u]);
                s[4 + u] = fmaf(k[n][u][i], k[n][u][i], s[4 + u]);
                s[8 + u] = fmaf(k[n][u][i], q[n][u][i], s[8 + u]);
#pragma unroll
                for (int m = 0; m < u; ++m, ++at) {
                    s[12 + at] = fmaf(k[n][m][i], k[n][u][i], s[12 + at]);
                    s[18 + at] = fmaf(k[n][m][i], q[n][u][i], s[18 + at]);
                }
            }
        }
    }
    // 32 sums over 32 lanes: with each round a lane keeps half of its values, lane i ends with sum i
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int i = 0; i < o; ++i) {
            const float give = up ? s[i] : s[i + o], have = up ? s[i + o] : s[i];
            s[i] = have + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
    const float inv = 1.f / sqrtf(s[0] + 1e-6f);         // lanes 0-7: one over the lengths of q_j, k_j
    float rq[DP_GROUP], rk[DP_GROUP];
#pragma unroll
    for (int u = 0; u < DP_GROUP; ++u) {
        rq[u] = __shfl_sync(0xffffffffu, inv, u) * q_scale;
        rk[u] = __shfl_sync(0xffffffffu, inv, 4 + u);
    }
    const size_t next = (size_t)G * 2 * dkp;
    float* row = qk + ((size_t)t * G + unit) * 2 * dkp;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = (n * 32 + lane) * VEC;
        if (c >= dkp) break;
#pragma unroll
        for (int u = 0; u < DP_GROUP; ++u) {
            if (u >= count) break;
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                q[n][u][i] *= rq[u];
                k[n][u][i] *= rk[u];
            }
            dl_store<VEC>(row + u * next + c, q[n][u]);
            dl_store<VEC>(row + u * next + dkp + c, k[n][u]);
        }
    }
    // The records of the group's heads: lane 4 i + u is token u of the i-th of eight heads. Lanes 8 + j
    // have k_j.q_j, lanes 12 + p and 18 + p the products of tokens m < j, p = j (j - 1) / 2 + m.
    const int u = lane & 3, per_group = H / G;
    const float rku = u == 0 ? rk[0] : u == 1 ? rk[1] : u == 2 ? rk[2] : rk[3];
    const float rqu = u == 0 ? rq[0] : u == 1 ? rq[1] : u == 2 ? rq[2] : rq[3];
    const float own = __shfl_sync(0xffffffffu, s[0], 8 + u) * rku * rqu;
    float ck[3], cq[3];
#pragma unroll
    for (int m = 0; m < 3; ++m) {
        const int at = u > m ? u * (u - 1) / 2 + m : 0;
        ck[m] = __shfl_sync(0xffffffffu, s[0], 12 + at) * rk[m] * rku;
        cq[m] = __shfl_sync(0xffffffffu, s[0], 18 + at) * rk[m] * rqu;
    }
    for (int h0 = 0; h0 < per_group; h0 += 8) {
        const int hh = h0 + lane / 4, h = unit * per_group + (hh < per_group ? hh : per_group - 1);
        float l = 0.f, beta = 0.f;
        if (u < count) {
            const float zz = to_f32(a_raw[(size_t)(t + u) * gate_stride + h]) + dt_bias[h];
            l = -A[h] * (zz > 20.f ? zz : log1pf(expf(zz)));
            beta = dl_sigmoid<T>(to_f32(b_raw[(size_t)(t + u) * gate_stride + h]));
        }
        // log decays: of the tokens up to this one, of those between m and this one, of those after it
        float at[4], ratio[3];
#pragma unroll
        for (int m = 0; m < 4; ++m) at[m] = __shfl_sync(0xffffffffu, l, (lane & ~3) + m);
        const float upto = at[0] + (u > 0 ? at[1] : 0.f) + (u > 1 ? at[2] : 0.f) + (u > 2 ? at[3] : 0.f);
        const float all = at[0] + at[1] + at[2] + at[3];
        const float later = (u < 1 ? at[1] : 0.f) + (u < 2 ? at[2] : 0.f) + (u < 3 ? at[3] : 0.f);
        ratio[0] = (u > 0 ? at[1] : 0.f) + (u > 1 ? at[2] : 0.f) + (u > 2 ? at[3] : 0.f);
        ratio[1] = (u > 1 ? at[2] : 0.f) + (u > 2 ? at[3] : 0.f);
        ratio[2] = u > 2 ? at[3] : 0.f;
        float pk[3], pq[4];
#pragma unroll
        for (int m = 0; m < 3; ++m) {
            const float e = m < u ? expf(ratio[m]) : 0.f;
            pk[m] = beta * e * ck[m];
            pq[m] = e * cq[m];
        }
        pq[3] = 0.f;
#pragma unroll
        for (int m = 0; m < 4; ++m)
            if (m == u) pq[m] = own;
        if (u < count && hh < per_group) {
            float4* rec = records + ((size_t)(t + u) * H + h) * 3;
            const float p = expf(upto);
            rec[0] = make_float4(beta * p, pk[0], pk[1], pk[2]);
            rec[1] = make_float4(pq[0], pq[1], pq[2], pq[3]);
            rec[2] = make_float4(p, expf(later), expf(all), expm1f(all));
        }
    }
}

template <typename T, int VEC, int NV, int TAPS>
__global__ void __launch_bounds__(32 * DP_WARPS, VEC * NV <= 4 ? 6 : 4)
delta_prepare_kernel(const T* __restrict__ x, long long x_stride, const float* __restrict__ w,
                     const T* __restrict__ b_raw, const T* __restrict__ a_raw, long long gate_stride,
                     const float* __restrict__ dt_bias, const float* __restrict__ A, float* __restrict__ qk,
                     float* __restrict__ v_out, float4* __restrict__ records, int Tn,
                     int per, int H, int G, int dk, int dv, int dkp, int taps, float q_scale,
                     const int* __restrict__ seq_ids, const int* __restrict__ q_start,
                     const int* __restrict__ state_slots, const float* __restrict__ state,
                     long long state_stride, long long conv_offset) {
    pdl_wait();
    const int first = (blockIdx.x * DP_WARPS + (threadIdx.x >> 5)) * per, lane = threadIdx.x & 31;
    // the tokens of this warp that begin a four, looked up side by side
    int b = 0, r = 1;
    if (lane < per && first + lane < Tn) {
        b = seq_ids[first + lane];
        r = first + lane - q_start[b];
    }
    unsigned begins = __ballot_sync(0xffffffffu, r % DP_GROUP == 0);
    while (begins) {
        const int at = __ffs(begins) - 1;
        begins &= begins - 1;
        delta_prepare_four<T, VEC, NV, TAPS>(
            first + at, __shfl_sync(0xffffffffu, b, at), __shfl_sync(0xffffffffu, r, at), x, x_stride, w, b_raw, a_raw,
            gate_stride, dt_bias, A, qk, v_out, records, H, G, dk, dv, dkp, taps, q_scale, q_start, state_slots, state,
            state_stride, conv_offset);
    }
}

// x [T, C] a column view in the storage type (q, k, v side by side), b_raw and a_raw [T, H] column
// views with one stride; w float32 [taps][C], dt_bias and A = exp(A_log) float32 [H].
TGO_API int tgo_delta_prepare(const void* x, long long x_stride, int dtype, const float* w, const void* b_raw,
                              const void* a_raw, long long gate_stride, const float* dt_bias, const float* A,
                              float* qk, float* v_out, float* records, int T, int B, int H, int G,
                              int dk, int dv, int taps, const int* seq_ids, const int* q_start,
                              const int* state_slots, const float* state, long long state_stride,
                              long long conv_offset, cudaStream_t stream) {
    if (T <= 0 || B <= 0) return 0;
    const int C = 2 * G * dk + H * dv, dkp = delta_row_width(dk);
    if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > 256 || dv <= 0 || taps <= 0 || taps > 64 ||
        state_stride < conv_offset + (long long)(taps - 1) * C || (uintptr_t)qk % 16 || (uintptr_t)records % 16 ||
         (dtype != TGO_BF16 && dtype != TGO_F32))
        return TGO_E_BAD_ARG;
    const uintptr_t width = dtype == TGO_BF16 ? 8 : 16;  // bytes of four elements
    const bool quads = dk % 4 == 0 && dv % 4 == 0 && x_stride % 4 == 0 && (uintptr_t)x % width == 0 &&
                       (uintptr_t)w % 16 == 0 && (uintptr_t)v_out % 16 == 0 && (uintptr_t)state % 16 == 0 &&
                       state_stride % 4 == 0 && conv_offset % 4 == 0;
    const int per = quads ? 128 : 32, v_units = (H * dv + per - 1) / per;
    const long long units = (long long)G + v_units;
    if (units > 65535) return TGO_E_BAD_ARG;
    const int each = T == B ? 1 : DP_GROUP;
    const dim3 grid((T + DP_WARPS * each - 1) / (DP_WARPS * each), (unsigned)units);
    const float q_scale = 1.f / sqrtf((float)dk);
#define DP_GO(TT, VEC, NV, TAPS)                                                                           \
    tgo_launch_pdl(delta_prepare_kernel<TT, VEC, NV, TAPS>, grid, dim3(32 * DP_WARPS), 0, stream, (const TT*)x, x_stride, \
                   w, (const TT*)b_raw, (const TT*)a_raw, gate_stride, dt_bias, A, qk, v_out, (float4*)records, T, \
                   each, H, G, dk, dv, dkp, taps, q_scale, seq_ids, q_start, state_slots, \
                   state, state_stride, conv_offset)
#define DP_TAPS(TT, NV)                                                                                    \
    (taps == 4 ? DP_GO(TT, 4, NV, 4) : taps == 3 ? DP_GO(TT, 4, NV, 3) : taps == 2 ? DP_GO(TT, 4, NV, 2)    \
                                                                       : DP_GO(TT, 4, NV, 0))
#define DP_SIZE(TT) (quads ? (dkp <= 128 ? DP_TAPS(TT, 1) : DP_TAPS(TT, 2)) : DP_GO(TT, 1, 8, 0))
    return dtype == TGO_BF16 ? DP_SIZE(bf16) : DP_SIZE(float);
#undef DP_SIZE
#undef DP_TAPS
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
// A block per (request, head, 16 or 32 columns of dv). L lanes of a warp share a column (the column in
// the low bits of the lane): slice s keeps its rows 4 s + 4 L i + (0..3) in registers for the whole walk
// over the request's tokens. Four tokens cost eight products of a vector with S, one transposing
// exchange over the slices that leaves one of the eight sums in each, four broadcasts of the reads by
// k, ten multiply-adds for the four u, and one update of S. DS_TOK tokens at a time come through shared
// memory by asynchronous copies, two buffers. The order of every sum depends on the sizes alone.
#define DS_TOK 16
#define DS_THREADS 256

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

// A memory that decays slowly is multiplied by nearly 1 a thousand times, and a factor rounded to the
// same side each time adds up: the float32 engine adds (P - 1) S while the decay is slow, whose rounding
// is relative to the change.
template <typename T> __device__ __forceinline__ bool dl_slow(float pm1) { return false; }
template <> __device__ __forceinline__ bool dl_slow<float>(float pm1) { return pm1 > -0.3f; }

template <typename T, int L, int NQ>
__global__ void __launch_bounds__(DS_THREADS)
delta_scan_kernel(const float* __restrict__ qk, const float* __restrict__ v, const float4* __restrict__ records,
                  float* __restrict__ y, int H, int G, int dk, int dv,
                  const int* __restrict__ q_start, const int* __restrict__ state_slots, float* __restrict__ state,
                  long long state_stride, long long mem_offset, const T* __restrict__ conv_in,
                  long long conv_in_stride, int taps, long long conv_offset) {
    constexpr int NI = 4 * NQ, DKP = L * NI, CG = 32 / L, COLS = DS_THREADS / L;
    constexpr int BUF = DS_TOK * (2 * DKP + COLS + 12);
    extern __shared__ __align__(16) float smem[];        // 2 x { qk [TOK][2 DKP], records [TOK][12], v [TOK][COLS] }
    pdl_wait();
    const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS;
    const int t0 = q_start[b], n_tok = q_start[b + 1] - t0;
    if (n_tok <= 0) return;
    const int g = h / (H / G);
    const int lane = threadIdx.x & 31, cg = lane % CG, s = lane / CG;
    const int col = (threadIdx.x >> 5) * CG + cg, c = c0 + col;
    float* row = state + (size_t)state_slots[b] * state_stride;
    float* Sg = row + mem_offset + (size_t)h * dk * dv;
    // the memory comes and goes through shared memory ([dk][COLS + 1] floats fit in the buffers)
    for (int i = threadIdx.x; i < dk * COLS; i += DS_THREADS) {
        const int n = i / COLS, cc = i % COLS;
        smem[n * (COLS + 1) + cc] = c0 + cc < dv ? Sg[(size_t)n * dv + c0 + cc] : 0.f;
    }
    __syncthreads();
    float S[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = 4 * s + 4 * L * (i >> 2) + (i & 3);
        S[i] = n < dk ? smem[n * (COLS + 1) + col] : 0.f;
    }
    __syncthreads();
    auto stage = [&](int base, int buf) {
        float* qks = smem + buf * BUF;
        float* rs = qks + DS_TOK * 2 * DKP;
        float* vs = rs + DS_TOK * 12;
        const int nt = n_tok - base < DS_TOK ? n_tok - base : DS_TOK, ne = (nt + 3) & ~3;
        for (int i = threadIdx.x; i < ne * (2 * DKP / 4); i += DS_THREADS) {
            const int r = i / (2 * DKP / 4), q = i % (2 * DKP / 4);
            const bool ok = r < nt;
            ds_copy16(qks + 4 * i, ok ? qk + ((size_t)(t0 + base + r) * G + g) * 2 * DKP + 4 * q : qk, ok);
        }
        for (int i = threadIdx.x; i < ne * COLS; i += DS_THREADS) {
            const int r = i / COLS, cc = i % COLS;
            const bool ok = r < nt && c0 + cc < dv;
            ds_copy4(vs + i, ok ? v + ((size_t)(t0 + base + r) * H + h) * dv + c0 + cc : v, ok);
        }
        if (threadIdx.x < 3 * ne) {
            const int r = threadIdx.x / 3, part = threadIdx.x % 3;
            const bool ok = r < nt;
            ds_copy16(rs + 4 * threadIdx.x, ok ? records + ((size_t)(t0 + base + r) * H + h) * 3 + part : records, ok);
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    // the sum this slice ends with: the read by k of token `mine` of the four, or (by_q) by its q
    const int vec = s / (L / 8), mine = vec & 3;
    const bool stores = vec >= 4 && (s % (L / 8)) == 0 && c < dv;
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
        const float* rs = qks + DS_TOK * 2 * DKP;
        const float* vs = rs + DS_TOK * 12;
        float* yt = y + ((size_t)(t0 + base + mine) * H + h) * dv + c;
        auto four = [&](int r) {
            const float* q0 = qks + r * 2 * DKP + 4 * s;
            float4 ka[NQ][4];
            float sum[8];                                // four reads by k, four by q
#pragma unroll
            for (int j = 0; j < 8; ++j) sum[j] = 0.f;
#pragma unroll
            for (int i = 0; i < NQ; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float4 kk = *(const float4*)(q0 + j * 2 * DKP + DKP + 4 * L * i);
                    const float4 qq = *(const float4*)(q0 + j * 2 * DKP + 4 * L * i);
                    ka[i][j] = kk;
                    sum[j] = fmaf(kk.x, S[4 * i], sum[j]);
                    sum[4 + j] = fmaf(qq.x, S[4 * i], sum[4 + j]);
                    sum[j] = fmaf(kk.y, S[4 * i + 1], sum[j]);
                    sum[4 + j] = fmaf(qq.y, S[4 * i + 1], sum[4 + j]);
                    sum[j] = fmaf(kk.z, S[4 * i + 2], sum[j]);
                    sum[4 + j] = fmaf(qq.z, S[4 * i + 2], sum[4 + j]);
                    sum[j] = fmaf(kk.w, S[4 * i + 3], sum[j]);
                    sum[4 + j] = fmaf(qq.w, S[4 * i + 3], sum[4 + j]);
                }
            float4 ra[4];                                // (b P_j, the three k_m.k_j terms); zeros past the end
            float2 rc[4];                                // P_j, E_j
            float vj[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                ra[j] = *(const float4*)(rs + 12 * (r + j));
                rc[j] = *(const float2*)(rs + 12 * (r + j) + 8);
                vj[j] = vs[(r + j) * COLS + col];
            }
            const float2 total = *(const float2*)(rs + 12 * r + 10);         // P_last, P_last - 1
            const float4 rd = *(const float4*)(rs + 12 * (r + mine) + 4);
            const float p_mine = rs[12 * (r + mine) + 8];
#pragma unroll
            for (int half = 4; half > 0; half >>= 1) {   // a slice keeps half of its sums
                const int o = half * (L / 8);
                const bool up = s & o;
#pragma unroll
                for (int i = 0; i < half; ++i) {
                    const float give = up ? sum[i] : sum[i + half], have = up ? sum[i + half] : sum[i];
                    sum[i] = have + __shfl_xor_sync(0xffffffffu, give, CG * o);
                }
            }
#pragma unroll
            for (int o = L / 16; o > 0; o >>= 1) sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], CG * o);
            float u[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float x = __shfl_sync(0xffffffffu, sum[0], j * (L / 8) * CG + cg);
                u[j] = fmaf(-ra[j].x, x, vj[j]);
            }
            u[1] = fmaf(-ra[1].y, u[0], u[1]);
            u[2] = fmaf(-ra[2].y, u[0], u[2]);
            u[3] = fmaf(-ra[3].y, u[0], u[3]);
            u[2] = fmaf(-ra[2].z, u[1], u[2]);
            u[3] = fmaf(-ra[3].z, u[1], u[3]);
            u[3] = fmaf(-ra[3].w, u[2], u[3]);
            const float o0 = fmaf(rd.y, u[1], fmaf(rd.x, u[0], p_mine * sum[0]));
            const float o1 = fmaf(rd.w, u[3], rd.z * u[2]);
            if (stores && r + mine < nt) *yt = o0 + o1;
            yt += (size_t)4 * H * dv;
#pragma unroll
            for (int j = 0; j < 4; ++j) u[j] *= rc[j].y;                      // decayed by the later ones
            const bool slow = dl_slow<T>(total.y);
            const float f = slow ? total.y : total.x;
#pragma unroll
            for (int i = 0; i < NQ; ++i) {
                float4 a = make_float4(f * S[4 * i], f * S[4 * i + 1], f * S[4 * i + 2], f * S[4 * i + 3]);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    a.x = fmaf(ka[i][j].x, u[j], a.x);
                    a.y = fmaf(ka[i][j].y, u[j], a.y);
                    a.z = fmaf(ka[i][j].z, u[j], a.z);
                    a.w = fmaf(ka[i][j].w, u[j], a.w);
                }
                S[4 * i] = slow ? S[4 * i] + a.x : a.x;
                S[4 * i + 1] = slow ? S[4 * i + 1] + a.y : a.y;
                S[4 * i + 2] = slow ? S[4 * i + 2] + a.z : a.z;
                S[4 * i + 3] = slow ? S[4 * i + 3] + a.w : a.w;
            }
        };
        if (nt == DS_TOK) {                              // unrolled: the next four's rows load while these are joined
#pragma unroll
            for (int r = 0; r < DS_TOK; r += 4) four(r);
        } else {
            for (int r = 0; r < nt; r += 4) four(r);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = 4 * s + 4 * L * (i >> 2) + (i & 3);
        if (n < dk) smem[n * (COLS + 1) + col] = S[i];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < dk * COLS; i += DS_THREADS) {
        const int n = i / COLS, cc = i % COLS;
        if (c0 + cc < dv) Sg[(size_t)n * dv + c0 + cc] = smem[n * (COLS + 1) + cc];
    }
    dl_keep_block(row + conv_offset, conv_in, conv_in_stride, H, G, dk, dv, h, c0, COLS, taps, t0, n_tok);
}

template <typename T, int L, int NQ>
static int launch_delta_scan(const float* qk, const float* v, const float* records, float* y,
                             int B, int H, int G, int dk, int dv, const int* q_start, const int* state_slots,
                             float* state, long long state_stride, long long mem_offset, const T* conv_in,
                             long long conv_in_stride, int taps, long long conv_offset, cudaStream_t stream) {
    constexpr int DKP = 4 * L * NQ, COLS = DS_THREADS / L;
    const size_t smem = 2 * (size_t)DS_TOK * (2 * DKP + COLS + 12) * sizeof(float);
    auto kernel = delta_scan_kernel<T, L, NQ>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return tgo_launch_pdl(kernel, dim3(B, H, (dv + COLS - 1) / COLS), dim3(DS_THREADS), smem, stream, qk, v,
                          (const float4*)records, y, H, G, dk, dv, q_start, state_slots, state,
                          state_stride, mem_offset, conv_in, conv_in_stride, taps, conv_offset);
}

static bool delta_sizes_ok(int H, int G, int dk, int dv, int taps, long long state_stride, long long mem_offset,
                           long long conv_offset) {
    return H > 0 && G > 0 && H % G == 0 && H <= 65535 && dk > 0 && dk <= 256 && dv > 0 && dv <= 1 << 20 &&
           taps > 0 && taps <= 64 && state_stride >= mem_offset + (long long)H * dk * dv &&
           state_stride >= conv_offset + (long long)(taps - 1) * (2 * G * dk + H * dv);
}

TGO_API int tgo_delta_scan(const float* qk, const float* v, const float* records, float* y, int B,
                           int H, int G, int dk, int dv, const int* q_start, const int* state_slots, float* state,
                           long long state_stride, long long mem_offset, const void* conv_in,
                           long long conv_in_stride, int dtype, int taps, long long conv_offset,
                           cudaStream_t stream) {
    if (B <= 0) return 0;
    if (!delta_sizes_ok(H, G, dk, dv, taps, state_stride, mem_offset, conv_offset) || (uintptr_t)qk % 16 ||
        (uintptr_t)records % 16 || (dtype != TGO_BF16 && dtype != TGO_F32))
        return TGO_E_BAD_ARG;
#define DS_GO(TT, L, NQ)                                                                                   \
    launch_delta_scan<TT, L, NQ>(qk, v, records, y, B, H, G, dk, dv, q_start, state_slots, state, state_stride, \
                                 mem_offset, (const TT*)conv_in, conv_in_stride, taps, conv_offset, stream)
#define DS_SIZE(TT)                                                                                        \
    (width == 32 ? DS_GO(TT, 8, 1) : width == 64 ? DS_GO(TT, 16, 1) : width == 128 ? DS_GO(TT, 16, 2) : DS_GO(TT, 16, 4))
    const int width = delta_row_width(dk);
    return dtype == TGO_BF16 ? DS_SIZE(bf16) : DS_SIZE(float);
#undef DS_SIZE
#undef DS_GO
}

// ----------------------------------------------------------------------------------- step
// Requests of one token each. A block per (request, head): the head's memory comes into shared memory
// whole by asynchronous copies, as many blocks to a multiprocessor as fit, and goes out once. Thread
// (row group, column quad) takes rows q, q + R, .. of four columns; the reads by k and q are joined
// over the row groups through shared memory, in order. Then, in the same block, the head's output is
// divided by its root mean square over dv, multiplied by the gain [dv] and by SiLU of the gate.
#define DT_THREADS 256
#define DT_SMEM (200 * 1024)
static size_t delta_step_smem(int dk, int dv) {
    const int R = DT_THREADS / (dv / 4), dkp = delta_row_width(dk);
    return ((size_t)dk * dv + 2 * dkp + 2 * dv + (size_t)2 * R * dv) * sizeof(float);
}

template <typename T>
__global__ void __launch_bounds__(DT_THREADS)
delta_step_kernel(const float* __restrict__ qk, const float* __restrict__ v, const float4* __restrict__ records,
                  const T* __restrict__ z, long long z_stride,
                  const float* __restrict__ gain, float eps, T* __restrict__ out, int H, int G, int dk, int dv,
                  int dkp, const int* __restrict__ q_start, const int* __restrict__ state_slots,
                  float* __restrict__ state, long long state_stride, long long mem_offset,
                  const T* __restrict__ conv_in, long long conv_in_stride, int taps, long long conv_offset) {
    extern __shared__ __align__(16) float smem[];        // S [dk][dv], qk [2 dkp], u [dv], o [dv], parts [2][R][dv]
    __shared__ float scratch[33];
    pdl_wait();
    const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int t = q_start[b];
    if (q_start[b + 1] - t <= 0) return;
    const int QN = dv / 4, R = DT_THREADS / QN, g = h / (H / G);
    const int rg = tid / QN, quad = tid % QN;
    const bool works = rg < R;
    float* qs = smem + (size_t)dk * dv;
    float* us = qs + 2 * dkp;
    float* os = us + dv;
    float* part = os + dv;
    float* row = state + (size_t)state_slots[b] * state_stride;
    float* Sg = row + mem_offset + (size_t)h * dk * dv;
    for (int i = tid; i < dk * QN; i += DT_THREADS) ds_copy16(smem + 4 * i, Sg + 4 * i, true);
    asm volatile("cp.async.commit_group;\n" ::);
    const float4* rec = records + ((size_t)t * H + h) * 3;
    const float bp = rec[0].x, kq = rec[1].x, decay = rec[2].x, decay_m1 = rec[2].w;
    for (int i = tid; i < 2 * dkp; i += DT_THREADS) qs[i] = qk[((size_t)t * G + g) * 2 * dkp + i];
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();
    if (works) {
        float4 sk = make_float4(0.f, 0.f, 0.f, 0.f), sq = sk;
#pragma unroll 4
        for (int n = rg; n < dk; n += R) {
            const float kn = qs[dkp + n], qn = qs[n];
            const float4 S = *(const float4*)(smem + (size_t)n * dv + 4 * quad);
            sk.x = fmaf(kn, S.x, sk.x); sk.y = fmaf(kn, S.y, sk.y);
            sk.z = fmaf(kn, S.z, sk.z); sk.w = fmaf(kn, S.w, sk.w);
            sq.x = fmaf(qn, S.x, sq.x); sq.y = fmaf(qn, S.y, sq.y);
            sq.z = fmaf(qn, S.z, sq.z); sq.w = fmaf(qn, S.w, sq.w);
        }
        *(float4*)(part + (size_t)rg * dv + 4 * quad) = sk;
        *(float4*)(part + (size_t)(R + rg) * dv + 4 * quad) = sq;
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < dv; c += DT_THREADS) {
        float sk = 0.f, sq = 0.f;
        for (int i = 0; i < R; ++i) {
            sk += part[(size_t)i * dv + c];
            sq += part[(size_t)(R + i) * dv + c];
        }
        const float u = fmaf(-bp, sk, v[((size_t)t * H + h) * dv + c]);
        const float o = fmaf(kq, u, decay * sq);
        us[c] = u;
        os[c] = o;
        ss += o * o;
    }
    ss = block_sum(ss, scratch);                         // its barriers make `us` visible too
    if (works) {
        const float4 u = *(const float4*)(us + 4 * quad);
        const bool slow = dl_slow<T>(decay_m1);
#pragma unroll 4
        for (int n = rg; n < dk; n += R) {
            const float kn = qs[dkp + n];
            const float4 S = *(const float4*)(smem + (size_t)n * dv + 4 * quad);
            float4 r;
            if (slow) {
                r.x = S.x + fmaf(decay_m1, S.x, kn * u.x); r.y = S.y + fmaf(decay_m1, S.y, kn * u.y);
                r.z = S.z + fmaf(decay_m1, S.z, kn * u.z); r.w = S.w + fmaf(decay_m1, S.w, kn * u.w);
            } else {
                r.x = fmaf(kn, u.x, decay * S.x); r.y = fmaf(kn, u.y, decay * S.y);
                r.z = fmaf(kn, u.z, decay * S.z); r.w = fmaf(kn, u.w, decay * S.w);
            }
            *(float4*)(Sg + (size_t)n * dv + 4 * quad) = r;
        }
    }
    for (int c = tid; c < dv; c += DT_THREADS) {
        const float a = (os[c] * rsqrtf(ss / (float)dv + eps)) * gain[c];
        out[((size_t)t * H + h) * dv + c] =
            from_f32<T>(a * dl_silu<T>(to_f32(z[(size_t)t * z_stride + (size_t)h * dv + c])));
    }
    dl_keep_block(row + conv_offset, conv_in, conv_in_stride, H, G, dk, dv, h, 0, dv, taps, t, 1);
}

TGO_API int tgo_delta_step_supports(int H, int G, int dk, int dv, long long state_stride, long long mem_offset) {
    return (H > 0 && G > 0 && H % G == 0 && H <= 65535 && dk > 0 && dk <= 256 && dv > 0 && dv <= 4 * DT_THREADS &&
            dv % 4 == 0 && state_stride % 4 == 0 && mem_offset % 4 == 0 && delta_step_smem(dk, dv) <= DT_SMEM) ? 1 : 0;
}

TGO_API int tgo_delta_step(const float* qk, const float* v, const float* records, const void* z,
                           long long z_stride, const float* gain, float eps, void* out, int B, int H, int G, int dk,
                           int dv, const int* q_start, const int* state_slots, float* state, long long state_stride,
                           long long mem_offset, const void* conv_in, long long conv_in_stride, int dtype, int taps,
                           long long conv_offset, cudaStream_t stream) {
    if (B <= 0) return 0;
    if (!tgo_delta_step_supports(H, G, dk, dv, state_stride, mem_offset) ||
        !delta_sizes_ok(H, G, dk, dv, taps, state_stride, mem_offset, conv_offset) || (uintptr_t)state % 16 ||
        (uintptr_t)records % 16 || (dtype != TGO_BF16 && dtype != TGO_F32))
        return TGO_E_BAD_ARG;
    const int dkp = delta_row_width(dk);
    const size_t smem = delta_step_smem(dk, dv);
#define DT_GO(TT)                                                                                          \
    do {                                                                                                   \
        auto kernel = delta_step_kernel<TT>;                                                               \
        if (smem > 48 * 1024)                                                                              \
            cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);          \
        return tgo_launch_pdl(kernel, dim3(B, H), dim3(DT_THREADS), smem, stream, qk, v, (const float4*)records, \
                              (const TT*)z, z_stride, gain, eps, (TT*)out, H, G, dk, dv, dkp, q_start, state_slots, \
                              state, state_stride, mem_offset, (const TT*)conv_in, conv_in_stride, taps, conv_offset); \
    } while (0)
    if (dtype == TGO_BF16) DT_GO(bf16);
    DT_GO(float);
#undef DT_GO
}
