// A routed feed-forward (mixture of experts): every token goes to the `top` experts with the
// largest router logits, weighted by the softmax over those logits alone.
//
//   logits     Wr x + br in float32 (Wr, br float32; x in the storage type)
//   pick       the top experts (ties: the lower index), their weights, and a count per expert
//   plan       expert e's (token, choice) pairs get places offsets[e] .. offsets[e+1]-1; the
//              places are cut into row tiles of one expert each
//              (steps of few tokens: pick, plan and scatter are one block's work)
//   scatter    pair -> place (within an expert the order is whatever the atomics give; a
//              pair's result does not depend on its place)
//   up         hidden[place] = act(x Wg_e^T) * (x Wu_e^T) for the token of the pair at `place`
//   down       y[pair] = hidden[place] Wd_e^T, float32
//   combine    out[t] = sum_j weight[t][j] y[t top + j] (+ extra[t]), j in order, all float32
//
// The products are tiled: float32 storage takes plain-FMA tiles with float32 sums over k in
// order; bfloat16 storage takes mma.sync m16n8k16 tiles (float32 accumulators) fed by cp.async
// through two shared-memory buffers, when the widths are multiples of 8 (16-byte chunks), and
// the plain tiles otherwise. Either way a row's result does not depend on which tile or batch
// it falls in.
//
// Variants, each a parameter: `score_mode` 1 takes the softmax over ALL router logits; the choice
// is by that score plus a per-expert `correction`, the weights are the chosen experts' scores
// (without the correction) divided by their sum (+ 1e-20). The last router outputs past the
// `E_real` experts that have matrices are identity experts: their output is the token's input
// row itself; they get no place and no tile, the combine adds weight * x for them.
// `score_mode` 2 takes the logistic function of each logit as its score; with `groups` > 1 the
// experts are that many equal runs of neighbours, a run's strength is the sum of its two largest
// choice scores (`run_best` 2) or its largest alone (`run_best` 1), and only experts of the `keep`
// strongest runs can be chosen; without `renorm` the weights are the chosen scores themselves; `route_scale` multiplies the weights. One more
// router row after all experts (`gate_out`) gives a logistic gate per token that multiplies
// `extra` in the combine. Experts without a gate matrix (wg null) are W_down act(W_up x);
// activation 3 is the square of relu.
#include "mma_sync.cuh"

#define MOE_TM 64
#define MOE_TN 64
#define MOE_TK 16

// ------------------------------------------------------------------------------ logits
// A block takes ML_TOK tokens and ML_EXP router rows (experts); its eight warps share the width,
// four channels a thread and 1024 a round, so that the loads of a few tokens are all in flight
// at once. A warp's 32 sums are joined by a transposing exchange (lane i ends with pair i), the
// warps' through shared memory in warp order: the order of a sum depends on the width alone.
// out [T, rows]; the last row may have no bias (the gate of a shared expert). Block 0 also zeroes
// the experts' counts.
#define ML_TOK 8
#define ML_EXP 4
template <typename T> struct Load4;
template <> struct Load4<bf16> {
    static __device__ __forceinline__ float4 get(const bf16* p) {
        const uint2 v = *(const uint2*)p;
        const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&v.x);
        const float2 b = __bfloat1622float2(*(const __nv_bfloat162*)&v.y);
        return make_float4(a.x, a.y, b.x, b.y);
    }
};
template <> struct Load4<float> {
    static __device__ __forceinline__ float4 get(const float* p) { return *(const float4*)p; }
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
moe_logits_kernel(const T* __restrict__ x, long long x_stride, const float* __restrict__ wr,
                  const float* __restrict__ br, int Tn, int d, int rows, int E, float* __restrict__ out,
                  int* __restrict__ counts, int E_real) {
    __shared__ float s_part[8][32];
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (blockIdx.x == 0 && blockIdx.y == 0)
        for (int i = threadIdx.x; i < E_real; i += 256) counts[i] = 0;
    const int e0 = blockIdx.y * ML_EXP, t0 = blockIdx.x * ML_TOK;
    // tokens and rows past the end repeat the last one: their sums are not stored
    const T* xr[ML_TOK];
    const float* w[ML_EXP];
#pragma unroll
    for (int j = 0; j < ML_TOK; ++j) xr[j] = x + (size_t)(t0 + j < Tn ? t0 + j : Tn - 1) * x_stride;
#pragma unroll
    for (int k = 0; k < ML_EXP; ++k) w[k] = wr + (size_t)(e0 + k < rows ? e0 + k : rows - 1) * d;
    float a[32];                                         // a[4 j + k]: token j, row k
#pragma unroll
    for (int q = 0; q < 32; ++q) a[q] = 0.f;
    if (VEC) {
        for (int i = 4 * threadIdx.x; i < d; i += 1024) {
            float4 wv[ML_EXP], xv[ML_TOK];
#pragma unroll
            for (int k = 0; k < ML_EXP; ++k) wv[k] = *(const float4*)(w[k] + i);
#pragma unroll
            for (int j = 0; j < ML_TOK; ++j) xv[j] = Load4<T>::get(xr[j] + i);
#pragma unroll
            for (int j = 0; j < ML_TOK; ++j)
#pragma unroll
                for (int k = 0; k < ML_EXP; ++k) {
                    float v = a[4 * j + k];
                    v = fmaf(wv[k].x, xv[j].x, v);
                    v = fmaf(wv[k].y, xv[j].y, v);
                    v = fmaf(wv[k].z, xv[j].z, v);
                    a[4 * j + k] = fmaf(wv[k].w, xv[j].w, v);
                }
        }
    } else {
        for (int i = threadIdx.x; i < d; i += 256) {
            float wv[ML_EXP];
#pragma unroll
            for (int k = 0; k < ML_EXP; ++k) wv[k] = w[k][i];
#pragma unroll
            for (int j = 0; j < ML_TOK; ++j) {
                const float v = to_f32(xr[j][i]);
#pragma unroll
                for (int k = 0; k < ML_EXP; ++k) a[4 * j + k] = fmaf(wv[k], v, a[4 * j + k]);
            }
        }
    }
    // 32 sums over 32 lanes: with each round a lane keeps half of its values, lane i ends with sum i
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int q = 0; q < o; ++q) {
            const float give = up ? a[q] : a[q + o], have = up ? a[q + o] : a[q];
            a[q] = have + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
    s_part[warp][lane] = a[0];
    __syncthreads();
    if (warp == 0) {
        float v = 0.f;
#pragma unroll
        for (int q = 0; q < 8; ++q) v += s_part[q][lane];
        const int t = t0 + lane / 4, e = e0 + lane % 4;
        if (t < Tn && e < rows) out[(size_t)t * rows + e] = v + ((br && e < E) ? br[e] : 0.f);
    }
}

// -------------------------------------------------------------------------------- pick
// One warp picks one token's experts. lg [E + 1], sc [E] and gs [groups] are the warp's own
// shared memory; `z` the token's logits.
__device__ __forceinline__ void moe_pick(const float* __restrict__ z, float* lg, float* sc, float* gs,
                                         int t, int E, int top, int* __restrict__ ids,
                                         float* __restrict__ wts, int* counts, int score_mode,
                                         const float* __restrict__ correction, int E_real,
                                         float* __restrict__ gate_out, int groups, int keep, int renorm,
                                         float route_scale, int run_best) {
    const int lane = threadIdx.x & 31;
    for (int e = lane; e < E + (gate_out ? 1 : 0); e += 32) lg[e] = z[e];
    __syncwarp();
    if (gate_out && lane == 0) gate_out[t] = 1.f / (1.f + expf(-lg[E]));
    float first = 0.f, sum = 0.f, mine = 0.f;
    int mine_e = 0;
    // the largest of n values in shared memory below `limit` and its index (ties: the lower index),
    // the same in every lane; with nothing above -inf the index is `fallback`
    auto largest = [&](const float* v, int n, int fallback, float limit, float& best) {
        float mine_v = -INFINITY;
        int be = 0x7fffffff;
        for (int e = lane; e < n; e += 32) {
            const float x = v[e];
            if (x > mine_v && x < limit) { mine_v = x; be = e; }
        }
        // a float's bits, reordered so that they compare as integers
        const unsigned raw = __float_as_uint(mine_v);
        const unsigned key = (raw & 0x80000000u) ? ~raw : raw | 0x80000000u;
        const unsigned top_key = __reduce_max_sync(0xffffffffu, key);
        best = __uint_as_float((top_key & 0x80000000u) ? top_key & 0x7fffffffu : ~top_key);
        const unsigned bi = __reduce_min_sync(0xffffffffu, key == top_key ? (unsigned)be : 0x7fffffffu);
        return (int)bi < n ? (int)bi : fallback;
    };
    if (score_mode != 0) {
        // scores: the softmax over every logit, or each logit's logistic; the choice adds the correction
        float mx = 0.f, den = 1.f;
        if (score_mode == 1) {
            mx = -INFINITY;
            for (int e = lane; e < E; e += 32) mx = fmaxf(mx, lg[e]);
            mx = warp_max(mx);
            den = 0.f;
            for (int e = lane; e < E; e += 32) {
                const float w = expf(lg[e] - mx);
                sc[e] = w;
                den += w;
            }
            den = warp_sum(den);
        }
        for (int e = lane; e < E; e += 32) {
            const float sv = score_mode == 1 ? sc[e] / den : 1.f / (1.f + expf(-lg[e]));
            sc[e] = sv;
            lg[e] = sv + (correction ? correction[e] : 0.f);
        }
        __syncwarp();
        if (groups > 1) {
            const int size = E / groups;
            for (int g = lane; g < groups; g += 32) {
                float a = -INFINITY, c = -INFINITY;      // the two largest of the run
                for (int e = g * size; e < (g + 1) * size; ++e) {
                    const float v = lg[e];
                    if (v > a) { c = a; a = v; } else if (v > c) { c = v; }
                }
                gs[g] = size > 1 && run_best > 1 ? a + c : a;
            }
            __syncwarp();
            // the weakest groups - keep runs go: mark the strongest with +inf, then close the others
            for (int j = 0; j < keep; ++j) {
                float best;
                const int bg = largest(gs, groups, groups, INFINITY, best);
                __syncwarp();                            // every lane has read gs
                if (lane == 0 && bg < groups) gs[bg] = INFINITY;
                __syncwarp();
            }
            for (int e = lane; e < E; e += 32)
                if (gs[e / size] != INFINITY) lg[e] = -INFINITY;
            __syncwarp();
        }
        for (int j = 0; j < top; ++j) {
            float best;
            const int be = largest(lg, E, j, INFINITY, best);
            const float w = sc[be];
            sum += w;
            if (lane == j) { mine = w; mine_e = be; }
            __syncwarp();                                // every lane has read lg
            if (lane == 0) lg[be] = -INFINITY;
            __syncwarp();
        }
        if (lane < top) {
            ids[(size_t)t * top + lane] = mine_e;
            wts[(size_t)t * top + lane] = (renorm ? mine / (sum + 1e-20f) : mine) * route_scale;
            if (mine_e < E_real) atomicAdd(&counts[mine_e], 1);
        }
        return;
    }
    for (int j = 0; j < top; ++j) {
        float best;
        const int be = largest(lg, E, j, INFINITY, best);
        if (j == 0) first = best;
        const float w = expf(best - first);
        sum += w;
        if (lane == j) { mine = w; mine_e = be; }
        __syncwarp();
        if (lane == 0) lg[be] = -INFINITY;
        __syncwarp();
    }
    if (lane < top) {
        ids[(size_t)t * top + lane] = mine_e;
        wts[(size_t)t * top + lane] = mine / sum * route_scale;
        if (mine_e < E_real) atomicAdd(&counts[mine_e], 1);
    }
}

#define MOE_PW 4
__global__ void __launch_bounds__(32 * MOE_PW)
moe_pick_kernel(const float* __restrict__ logits, int rows, int Tn, int E, int top, int* __restrict__ ids,
                float* __restrict__ wts, int* __restrict__ counts, int score_mode,
                const float* __restrict__ correction, int E_real, float* __restrict__ gate_out, int groups,
                int keep, int renorm, float route_scale, int run_best) {
    extern __shared__ float smem[];                      // [MOE_PW][2 E + 1 + groups]
    pdl_wait();
    const int warp = threadIdx.x >> 5, t = blockIdx.x * MOE_PW + warp;
    if (t >= Tn) return;
    float* lg = smem + (size_t)warp * (2 * E + 1 + groups);
    moe_pick(logits + (size_t)t * rows, lg, lg + E + 1, lg + 2 * E + 1, t, E, top, ids, wts, counts, score_mode,
             correction, E_real, gate_out, groups, keep, renorm, route_scale, run_best);
}

// -------------------------------------------------------------------------------- plan
// One warp: offsets [E + 1], tiles (expert, first place, rows) and their count in tile_info[0]; the
// fill counters go back to zero. A lane takes a run of experts, the places and tiles before it by
// a running sum over the lanes.
__device__ __forceinline__ void moe_plan(const int* counts, int E, int* __restrict__ offsets, int* fill,
                                         int* __restrict__ tile_info, int* __restrict__ tiles, int max_tiles) {
    const int lane = threadIdx.x & 31, per = (E + 31) / 32;
    const int e_lo = lane * per < E ? lane * per : E, e_hi = e_lo + per < E ? e_lo + per : E;
    int c = 0, nt = 0;
    for (int e = e_lo; e < e_hi; ++e) {
        c += counts[e];
        nt += (counts[e] + MOE_TM - 1) / MOE_TM;
    }
    int at = c, tile = nt;                               // inclusive sums over the lanes
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, at, o), b = __shfl_up_sync(0xffffffffu, tile, o);
        if (lane >= o) { at += a; tile += b; }
    }
    if (lane == 31) {
        offsets[E] = at;
        tile_info[0] = tile < max_tiles ? tile : max_tiles;
    }
    at -= c;
    tile -= nt;
    for (int e = e_lo; e < e_hi; ++e) {
        const int n = counts[e];
        offsets[e] = at;
        fill[e] = 0;
        for (int r = 0; r < n; r += MOE_TM, ++tile) {
            if (tile >= max_tiles) break;
            tiles[3 * tile] = e;
            tiles[3 * tile + 1] = at + r;
            tiles[3 * tile + 2] = n - r < MOE_TM ? n - r : MOE_TM;
        }
        at += n;
    }
}

__global__ void __launch_bounds__(32)
moe_plan_kernel(const int* __restrict__ counts, int E, int* __restrict__ offsets, int* __restrict__ fill,
                int* __restrict__ tile_info, int* __restrict__ tiles, int max_tiles) {
    pdl_wait();
    moe_plan(counts, E, offsets, fill, tile_info, tiles, max_tiles);
}

// A step of few tokens: pick, plan and scatter by one block, the counts and fill counters in
// shared memory.
#define MOE_FEW_WARPS 32
__global__ void __launch_bounds__(32 * MOE_FEW_WARPS)
moe_route_few_kernel(const float* __restrict__ logits, int rows, int Tn, int E, int top, int* __restrict__ ids,
                     float* __restrict__ wts, int score_mode, const float* __restrict__ correction, int E_real,
                     float* __restrict__ gate_out, int groups, int keep, int renorm, float route_scale,
                     int run_best, int* __restrict__ offsets, int* __restrict__ perm, int* __restrict__ place,
                     int* __restrict__ tile_info, int* __restrict__ tiles, int max_tiles) {
    extern __shared__ float smem[];                      // [warps][2 E + 1 + groups], counts, fill
    const int per = 2 * E + 1 + groups;
    int* counts = (int*)(smem + (size_t)MOE_FEW_WARPS * per);
    int* fill = counts + E_real;
    const int warp = threadIdx.x >> 5, n = 32 * MOE_FEW_WARPS;
    for (int i = threadIdx.x; i < E_real; i += n) counts[i] = 0;
    pdl_wait();
    __syncthreads();
    float* lg = smem + (size_t)warp * per;
    for (int t = warp; t < Tn; t += MOE_FEW_WARPS) {
        moe_pick(logits + (size_t)t * rows, lg, lg + E + 1, lg + 2 * E + 1, t, E, top, ids, wts, counts, score_mode,
                 correction, E_real, gate_out, groups, keep, renorm, route_scale, run_best);
        __syncwarp();
    }
    __syncthreads();                                     // ids are in memory for the whole block
    if (warp == 0) moe_plan(counts, E_real, offsets, fill, tile_info, tiles, max_tiles);
    __syncthreads();
    for (int p = threadIdx.x; p < Tn * top; p += n) {
        const int e = ids[p];
        if (e >= E_real) { place[p] = -1; continue; }
        const int at = offsets[e] + atomicAdd(&fill[e], 1);
        perm[at] = p;
        place[p] = at;
    }
}

__global__ void moe_scatter_kernel(const int* __restrict__ ids, int pairs,
                                   const int* __restrict__ offsets, int* __restrict__ fill,
                                   int* __restrict__ perm, int* __restrict__ place, int E_real) {
    pdl_wait();
    const int p = blockIdx.x * blockDim.x + threadIdx.x;
    if (p >= pairs) return;
    const int e = ids[p];
    if (e >= E_real) { place[p] = -1; return; }          // an identity expert: no matrices, no place
    const int at = offsets[e] + atomicAdd(&fill[e], 1);
    perm[at] = p;
    place[p] = at;
}

// ----------------------------------------------------------------------------- products
__device__ __forceinline__ float moe_act(float z, int act) {
    if (act == 1) return z > 0.f ? z : 0.f;
    if (act == 3) return z > 0.f ? z * z : 0.f;
    if (act == 2) return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    return z / (1.f + expf(-z));
}

// hidden[place][f] = act(x_tok . Wg[e][f]) * (x_tok . Wu[e][f]); Wg, Wu [E, ff, d]. Without a
// gate matrix (wg null): act(x_tok . Wu[e][f]).
template <typename T>
__global__ void __launch_bounds__(256)
moe_up_kernel(const T* __restrict__ x, long long x_stride, const T* __restrict__ wg,
              const T* __restrict__ wu, T* __restrict__ hidden, int d, int ff, int top, int act,
              const int* __restrict__ perm, const int* __restrict__ tile_info,
              const int* __restrict__ tiles) {
    __shared__ float xs[MOE_TK][MOE_TM + 4];
    __shared__ float gs[MOE_TK][MOE_TN + 4];
    __shared__ float us[MOE_TK][MOE_TN + 4];
    __shared__ int toks[MOE_TM];
    pdl_wait();
    if ((int)blockIdx.y >= tile_info[0]) return;
    const int e = tiles[3 * blockIdx.y], r0 = tiles[3 * blockIdx.y + 1], rows = tiles[3 * blockIdx.y + 2];
    const int n0 = blockIdx.x * MOE_TN;
    if (threadIdx.x < MOE_TM) toks[threadIdx.x] = threadIdx.x < rows ? perm[r0 + threadIdx.x] / top : -1;
    __syncthreads();
    const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    const T* wge = wg + (size_t)e * ff * d;
    const T* wue = wu + (size_t)e * ff * d;
    float ag[4][4], au[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) ag[i][j] = au[i][j] = 0.f;
    for (int k0 = 0; k0 < d; k0 += MOE_TK) {
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int idx = threadIdx.x + r * 256;
            const int row = idx / MOE_TK, kk = idx % MOE_TK;
            const int gk = k0 + kk, gn = n0 + row;
            const int tok = toks[row];
            xs[kk][row] = (tok >= 0 && gk < d) ? to_f32(x[(size_t)tok * x_stride + gk]) : 0.f;
            const bool in = gn < ff && gk < d;
            gs[kk][row] = (in && wg) ? to_f32(wge[(size_t)gn * d + gk]) : 0.f;
            us[kk][row] = in ? to_f32(wue[(size_t)gn * d + gk]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < MOE_TK; ++kk) {
            float a[4], g[4], u[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = xs[kk][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) { g[j] = gs[kk][tx * 4 + j]; u[j] = us[kk][tx * 4 + j]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    ag[i][j] = fmaf(a[i], g[j], ag[i][j]);
                    au[i][j] = fmaf(a[i], u[j], au[i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int row = ty * 4 + i;
        if (row >= rows) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int gn = n0 + tx * 4 + j;
            if (gn < ff)
                hidden[(size_t)(r0 + row) * ff + gn] =
                    from_f32<T>(wg ? moe_act(ag[i][j], act) * au[i][j] : moe_act(au[i][j], act));
        }
    }
}

// y[pair][n] = hidden[place] . Wd[e][n]; Wd [E, d, ff]; y float32 [pairs, d].
template <typename T>
__global__ void __launch_bounds__(256)
moe_down_kernel(const T* __restrict__ hidden, const T* __restrict__ wd, float* __restrict__ y, int d,
                int ff, const int* __restrict__ perm, const int* __restrict__ tile_info,
                const int* __restrict__ tiles) {
    __shared__ float hs[MOE_TK][MOE_TM + 4];
    __shared__ float ws[MOE_TK][MOE_TN + 4];
    pdl_wait();
    if ((int)blockIdx.y >= tile_info[0]) return;
    const int e = tiles[3 * blockIdx.y], r0 = tiles[3 * blockIdx.y + 1], rows = tiles[3 * blockIdx.y + 2];
    const int n0 = blockIdx.x * MOE_TN;
    const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    const T* wde = wd + (size_t)e * d * ff;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < ff; k0 += MOE_TK) {
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int idx = threadIdx.x + r * 256;
            const int row = idx / MOE_TK, kk = idx % MOE_TK;
            const int gk = k0 + kk, gn = n0 + row;
            hs[kk][row] = (row < rows && gk < ff) ? to_f32(hidden[(size_t)(r0 + row) * ff + gk]) : 0.f;
            ws[kk][row] = (gn < d && gk < ff) ? to_f32(wde[(size_t)gn * ff + gk]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < MOE_TK; ++kk) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = hs[kk][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = ws[kk][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int row = ty * 4 + i;
        if (row >= rows) continue;
        const int pair = perm[r0 + row];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int gn = n0 + tx * 4 + j;
            if (gn < d) y[(size_t)pair * d + gn] = acc[i][j];
        }
    }
}

// ------------------------------------------------------------- products on the tensor cores
// A tile of up to 64 rows of one expert by 64 columns; four warps, warp w owns rows 16w..16w+15
// and all 64 columns. UP: A rows are x rows gathered by token, B is Wg[e] and Wu[e] ([N, K]
// each), the result act(gate) * up goes to hidden[place] in bfloat16. MODE 1 is that; MODE 2
// is the form without a gate, B is Wu[e] alone and the result act(up). MODE 0: A rows are
// hidden[place], B is Wd[e], the result goes to y[pair] in float32.
#define MT_BK 64
#define MT_LD (MT_BK + 8)
#define MT_STAGES 3

template <int MODE>
__global__ void __launch_bounds__(128)
moe_tc_kernel(const bf16* __restrict__ a, long long a_stride, const bf16* __restrict__ w0,
              const bf16* __restrict__ w1, bf16* __restrict__ hidden, float* __restrict__ y, int N,
              int K, int top, int act, const int* __restrict__ perm,
              const int* __restrict__ tile_info, const int* __restrict__ tiles) {
    extern __shared__ __align__(16) unsigned char moe_smem[];
    typedef bf16 (*Tile)[MOE_TM][MT_LD];
    Tile As = (Tile)moe_smem;                                        // [MT_STAGES][64][MT_LD]
    Tile B0 = (Tile)(moe_smem + sizeof(bf16) * MT_STAGES * MOE_TM * MT_LD);
    Tile B1 = (Tile)(moe_smem + sizeof(bf16) * 2 * MT_STAGES * MOE_TM * MT_LD);   // UP only
    __shared__ int src_row[MOE_TM];
    constexpr bool UP = MODE != 0, GATED = MODE == 1;
    pdl_wait();
    if ((int)blockIdx.y >= tile_info[0]) return;
    const int e = tiles[3 * blockIdx.y], r0 = tiles[3 * blockIdx.y + 1], rows = tiles[3 * blockIdx.y + 2];
    const int n0 = blockIdx.x * MOE_TN;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid < MOE_TM) src_row[tid] = tid < rows ? (UP ? perm[r0 + tid] / top : r0 + tid) : -1;
    __syncthreads();
    const bf16* w0e = w0 + (size_t)e * N * K;
    const bf16* w1e = GATED ? w1 + (size_t)e * N * K : nullptr;
    auto load = [&](int k0, int buf) {
        // 64 rows x 8 chunks of 8 per operand
        for (int i = tid; i < MOE_TM * (MT_BK / 8); i += 128) {
            const int r = i >> 3, c = i & 7;
            const int k = k0 + c * 8;
            const int sr = src_row[r];
            const bool oka = sr >= 0 && k < K;
            cp_async16(&As[buf][r][c * 8], oka ? a + (size_t)sr * a_stride + k : a, oka);
            const bool okb = n0 + r < N && k < K;
            cp_async16(&B0[buf][r][c * 8], okb ? w0e + (size_t)(n0 + r) * K + k : w0, okb);
            if (GATED) cp_async16(&B1[buf][r][c * 8], okb ? w1e + (size_t)(n0 + r) * K + k : w0, okb);
        }
    };
    float c0[MOE_TN / 8][4], c1[GATED ? MOE_TN / 8 : 1][4];
#pragma unroll
    for (int i = 0; i < MOE_TN / 8; ++i) c0[i][0] = c0[i][1] = c0[i][2] = c0[i][3] = 0.f;
#pragma unroll
    for (int i = 0; i < (GATED ? MOE_TN / 8 : 1); ++i) c1[i][0] = c1[i][1] = c1[i][2] = c1[i][3] = 0.f;
    const int steps = (K + MT_BK - 1) / MT_BK;
#pragma unroll
    for (int p = 0; p < MT_STAGES - 1; ++p) {
        if (p < steps) load(p * MT_BK, p);
        cp_async_commit();
    }
    const bool warp_active = warp * 16 < rows;
    for (int st = 0; st < steps; ++st) {
        const int buf = st % MT_STAGES;
        cp_async_wait<MT_STAGES - 2>();                   // this step's tiles have landed
        __syncthreads();                                  // and the buffer of step st - 1 is free
        if (st + MT_STAGES - 1 < steps) load((st + MT_STAGES - 1) * MT_BK, (st + MT_STAGES - 1) % MT_STAGES);
        cp_async_commit();
        if (warp_active) {
#pragma unroll
            for (int ks = 0; ks < MT_BK / 16; ++ks) {
                uint32_t fa[4];
                ldmatrix_x4(fa, &As[buf][warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8][ks * 16 + (lane >> 4) * 8]);
#pragma unroll
                for (int np = 0; np < MOE_TN / 16; ++np) {
                    uint32_t fb[4];
                    ldmatrix_x4(fb, &B0[buf][np * 16 + (lane & 7) + (lane >> 4) * 8][ks * 16 + ((lane >> 3) & 1) * 8]);
                    mma_bf16(c0[2 * np], fa, fb[0], fb[1]);
                    mma_bf16(c0[2 * np + 1], fa, fb[2], fb[3]);
                    if (GATED) {
                        ldmatrix_x4(fb, &B1[buf][np * 16 + (lane & 7) + (lane >> 4) * 8][ks * 16 + ((lane >> 3) & 1) * 8]);
                        mma_bf16(c1[2 * np], fa, fb[0], fb[1]);
                        mma_bf16(c1[2 * np + 1], fa, fb[2], fb[3]);
                    }
                }
            }
        }
    }
    cp_async_wait<0>();
    if (!warp_active) return;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int row = warp * 16 + (lane >> 2) + 8 * h;
        if (row >= rows) continue;
        const int pair = UP ? 0 : perm[r0 + row];
#pragma unroll
        for (int i = 0; i < MOE_TN / 8; ++i) {
            const int col = n0 + i * 8 + (lane & 3) * 2;
            if (col >= N) continue;                       // N is even: col + 1 < N too
            if (UP) {
                const float v0 = moe_act(c0[i][2 * h], act) * (GATED ? c1[GATED ? i : 0][2 * h] : 1.f);
                const float v1 = moe_act(c0[i][2 * h + 1], act) * (GATED ? c1[GATED ? i : 0][2 * h + 1] : 1.f);
                *(uint32_t*)(hidden + (size_t)(r0 + row) * N + col) = pack_bf16(v0, v1);
            } else {
                *(float2*)(y + (size_t)pair * N + col) = make_float2(c0[i][2 * h], c0[i][2 * h + 1]);
            }
        }
    }
}

// out[t][c] = sum_j wts[t][j] y[t top + j][c] + extra_gate[t] * extra[t][c]; a pair whose
// expert is an identity expert (ids >= E_real; `ids` null: there are none) contributes
// wts * x[t][c] instead. `beside` [T, d] (TB: float32 or bfloat16; null: none) is added too, and
// with `accumulate` the whole is added to out: a block whose mixer and feed-forward read the
// same rows has both results put into the stream by this one pass.
template <typename T, typename TB>
__global__ void moe_combine_kernel(const float* __restrict__ y, const float* __restrict__ wts,
                                   const float* __restrict__ extra, float* __restrict__ out, int d,
                                   int top, const int* __restrict__ ids, int E_real,
                                   const T* __restrict__ x, long long x_stride,
                                   const float* __restrict__ extra_gate,
                                   const TB* __restrict__ beside, int accumulate, int vec) {
    pdl_wait();
    const int t = blockIdx.x;
    const float eg = extra_gate ? extra_gate[t] : 1.f;
    if (vec) {                                           // four columns a thread
        for (int c = 4 * (blockIdx.y * blockDim.x + threadIdx.x); c < d; c += 4 * blockDim.x * gridDim.y) {
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 ex = extra ? *(const float4*)(extra + (size_t)t * d + c) : a;
            const float4 bs = beside ? Load4<TB>::get(beside + (size_t)t * d + c) : a;
            const float4 o = accumulate ? *(const float4*)(out + (size_t)t * d + c) : a;
#pragma unroll 4
            for (int j = 0; j < top; ++j) {
                const size_t pair = (size_t)t * top + j;
                const float w = wts[pair];
                const float4 v = (ids && ids[pair] >= E_real) ? Load4<T>::get(x + (size_t)t * x_stride + c)
                                                              : *(const float4*)(y + pair * d + c);
                a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y);
                a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
            }
            if (extra) {
                a.x = fmaf(eg, ex.x, a.x); a.y = fmaf(eg, ex.y, a.y);
                a.z = fmaf(eg, ex.z, a.z); a.w = fmaf(eg, ex.w, a.w);
            }
            if (beside) { a.x += bs.x; a.y += bs.y; a.z += bs.z; a.w += bs.w; }
            if (accumulate) { a.x += o.x; a.y += o.y; a.z += o.z; a.w += o.w; }
            *(float4*)(out + (size_t)t * d + c) = a;
        }
        return;
    }
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < d; c += blockDim.x * gridDim.y) {
        float a = 0.f;
        for (int j = 0; j < top; ++j) {
            const size_t pair = (size_t)t * top + j;
            const float v = (ids && ids[pair] >= E_real) ? to_f32(x[(size_t)t * x_stride + c]) : y[pair * d + c];
            a = fmaf(wts[pair], v, a);
        }
        if (extra) a = fmaf(eg, extra[(size_t)t * d + c], a);
        if (beside) a += to_f32(beside[(size_t)t * d + c]);
        if (accumulate) a += out[(size_t)t * d + c];
        out[(size_t)t * d + c] = a;
    }
}

TGO_API int tgo_moe_tile_rows() { return MOE_TM; }

// ids, place int32 [T top]; wts float32 [T top]; logits float32 [T, router rows]; counts, fill
// int32 [E]; offsets int32 [E + 1]; perm int32 [T top]; tile_info int32 [1]; tiles int32
// [3 max_tiles].
#define MOE_FEW_TOKENS 128
TGO_API int tgo_moe_route(const void* x, long long x_stride, int dtype, const float* wr,
                          const float* br, int T, int d, int E, int top, float* logits, int* ids, float* wts,
                          int* counts, int* fill, int* offsets, int* perm, int* place,
                          int* tile_info, int* tiles, int max_tiles, int score_mode,
                          const float* correction, int E_real, float* gate_out, int groups, int keep,
                          int renorm, float route_scale, int run_best, int* launches, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (d <= 0 || E <= 0 || E > 2048 || top <= 0 || top > 32 || top > E || max_tiles <= 0 ||
        E_real < 0 || E_real > E || score_mode < 0 || score_mode > 2 || groups < 1 || E % groups ||
        keep < 1 || keep > groups || (long long)keep * (E / groups) < top || (groups > 1 && score_mode == 0) ||
        run_best < 1 || run_best > 2 || (dtype != TGO_BF16 && dtype != TGO_F32))
        return TGO_E_BAD_ARG;
    const int rows = E + (gate_out ? 1 : 0);
    const dim3 lgrid((T + ML_TOK - 1) / ML_TOK, (rows + ML_EXP - 1) / ML_EXP);
    const bool vec = d % 4 == 0 && x_stride % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)wr % 16 == 0;
#define LOGITS_GO(TT, V)                                                                                    \
    tgo_launch_pdl(moe_logits_kernel<TT, V>, lgrid, dim3(256), 0, stream, (const TT*)x, x_stride, wr, br, T, d, \
                   rows, E, logits, counts, E_real)
    int rc = dtype == TGO_BF16 ? (vec ? LOGITS_GO(bf16, true) : LOGITS_GO(bf16, false))
                               : (vec ? LOGITS_GO(float, true) : LOGITS_GO(float, false));
#undef LOGITS_GO
    if (rc) return rc;
    const size_t per = (size_t)(2 * E + 1 + groups) * sizeof(float);
    const size_t few = MOE_FEW_WARPS * per + (size_t)2 * E_real * sizeof(int);
    if (T <= MOE_FEW_TOKENS && few <= 200 * 1024) {
        if (few > 48 * 1024)
            cudaFuncSetAttribute(moe_route_few_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)few);
        *launches = 2;
        return tgo_launch_pdl(moe_route_few_kernel, dim3(1), dim3(32 * MOE_FEW_WARPS), few, stream,
                              (const float*)logits, rows, T, E, top, ids, wts, score_mode, correction, E_real,
                              gate_out, groups, keep, renorm, route_scale, run_best, offsets, perm, place, tile_info,
                              tiles, max_tiles);
    }
    *launches = 4;
    const size_t smem = MOE_PW * per;
    if (smem > 48 * 1024)                                // more than about 1000 router outputs
        cudaFuncSetAttribute(moe_pick_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    rc = tgo_launch_pdl(moe_pick_kernel, dim3((T + MOE_PW - 1) / MOE_PW), dim3(32 * MOE_PW), smem, stream,
                        (const float*)logits, rows, T, E, top, ids, wts, counts, score_mode, correction, E_real,
                        gate_out, groups, keep, renorm, route_scale, run_best);
    if (rc) return rc;
    rc = tgo_launch_pdl(moe_plan_kernel, dim3(1), dim3(32), 0, stream, (const int*)counts, E_real, offsets, fill,
                        tile_info, tiles, max_tiles);
    if (rc) return rc;
    const int pairs = T * top;
    return tgo_launch_pdl(moe_scatter_kernel, dim3((pairs + 255) / 256), dim3(256), 0, stream,
                          (const int*)ids, pairs, (const int*)offsets, fill, perm, place, E_real);
}

// x [T, d] rows (stride x_stride); wg, wu [E, ff, d]; wd [E, d, ff]; hidden [T top, ff] in the
// storage type; y float32 [T top, d]; extra float32 [T, d] or null; out float32 [T, d].
TGO_API int tgo_moe_experts(const void* x, long long x_stride, int dtype, const void* wg,
                            const void* wu, const void* wd, void* hidden, float* y,
                            const float* wts, const float* extra, float* out, int T, int d, int ff,
                            int top, int act, const int* perm, const int* tile_info,
                            const int* tiles, int max_tiles, const int* ids, int E_real,
                            const float* extra_gate, const void* beside, int beside_dtype,
                            int accumulate, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (d <= 0 || ff <= 0 || top <= 0 || max_tiles <= 0 || max_tiles > 65535 || act < 0 || act > 3)
        return TGO_E_BAD_ARG;
    const int comb_vec = d % 4 == 0 && x_stride % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)y % 16 == 0 &&
                         (uintptr_t)extra % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)beside % 16 == 0;
    const int comb_y = comb_vec && d > 512 ? (d / 512 < 16 ? d / 512 : 16) : 1;
    if (beside && beside_dtype != TGO_F32 && beside_dtype != TGO_BF16) return TGO_E_BAD_ARG;
#define MOE_COMBINE_OF(TT, TB)                                                                             \
    tgo_launch_pdl(moe_combine_kernel<TT, TB>, dim3(T, comb_y), dim3(128), 0, stream, (const float*)y, wts, extra,  \
                   out, d, top, ids, E_real, (const TT*)x, x_stride, extra_gate, (const TB*)beside, accumulate,     \
                   comb_vec)
#define MOE_COMBINE(TT) (beside && beside_dtype == TGO_BF16 ? MOE_COMBINE_OF(TT, bf16) : MOE_COMBINE_OF(TT, float))
    const dim3 g1((ff + MOE_TN - 1) / MOE_TN, max_tiles), g2((d + MOE_TN - 1) / MOE_TN, max_tiles);
    int rc;
    const bool chunks = d % 8 == 0 && ff % 8 == 0 && x_stride % 8 == 0 && (uintptr_t)x % 16 == 0 &&
                        (uintptr_t)wg % 16 == 0 && (uintptr_t)wu % 16 == 0 && (uintptr_t)wd % 16 == 0 &&
                        (uintptr_t)hidden % 16 == 0 && (uintptr_t)y % 8 == 0;
    if (dtype == TGO_BF16 && chunks) {
        const size_t tile = sizeof(bf16) * MT_STAGES * MOE_TM * MT_LD;
        static bool asked = false;
        if (!asked) {
            cudaFuncSetAttribute(moe_tc_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(3 * tile));
            cudaFuncSetAttribute(moe_tc_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(2 * tile));
            cudaFuncSetAttribute(moe_tc_kernel<0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(2 * tile));
            asked = true;
        }
        if (wg)
            rc = tgo_launch_pdl(moe_tc_kernel<1>, g1, dim3(128), 3 * tile, stream, (const bf16*)x, x_stride,
                                (const bf16*)wg, (const bf16*)wu, (bf16*)hidden, (float*)nullptr, ff, d, top, act,
                                perm, tile_info, tiles);
        else
            rc = tgo_launch_pdl(moe_tc_kernel<2>, g1, dim3(128), 2 * tile, stream, (const bf16*)x, x_stride,
                                (const bf16*)wu, (const bf16*)nullptr, (bf16*)hidden, (float*)nullptr, ff, d, top,
                                act, perm, tile_info, tiles);
        if (rc) return rc;
        rc = tgo_launch_pdl(moe_tc_kernel<0>, g2, dim3(128), 2 * tile, stream, (const bf16*)hidden, (long long)ff,
                            (const bf16*)wd, (const bf16*)nullptr, (bf16*)nullptr, y, d, ff, top, act, perm,
                            tile_info, tiles);
        if (rc) return rc;
        return MOE_COMBINE(bf16);
    }
    if (dtype == TGO_BF16) {
        rc = tgo_launch_pdl(moe_up_kernel<bf16>, g1, dim3(256), 0, stream, (const bf16*)x, x_stride,
                            (const bf16*)wg, (const bf16*)wu, (bf16*)hidden, d, ff, top, act, perm, tile_info,
                            tiles);
        if (rc) return rc;
        rc = tgo_launch_pdl(moe_down_kernel<bf16>, g2, dim3(256), 0, stream, (const bf16*)hidden,
                            (const bf16*)wd, y, d, ff, perm, tile_info, tiles);
        if (rc) return rc;
        return MOE_COMBINE(bf16);
    }
    if (dtype != TGO_F32) return TGO_E_BAD_ARG;
    rc = tgo_launch_pdl(moe_up_kernel<float>, g1, dim3(256), 0, stream, (const float*)x, x_stride,
                        (const float*)wg, (const float*)wu, (float*)hidden, d, ff, top, act, perm, tile_info,
                        tiles);
    if (rc) return rc;
    rc = tgo_launch_pdl(moe_down_kernel<float>, g2, dim3(256), 0, stream, (const float*)hidden,
                        (const float*)wd, y, d, ff, perm, tile_info, tiles);
    if (rc) return rc;
    return MOE_COMBINE(float);
#undef MOE_COMBINE
#undef MOE_COMBINE_OF
}
