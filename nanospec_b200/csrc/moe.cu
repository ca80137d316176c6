// Routed experts: scoring and choice per token, the bookkeeping that brings each expert's tokens together, and
// the experts' products for steps of a few tokens.
//
//   ns_cast_f32        rows of the compute type as float (the router's input: its logits are a float product)
//   ns_router_logits   the router's float product with an optional bias (the largest steps and routers: ns_cast_f32 and the float GEMM)
//   ns_moe_route       scores = sigmoid(logits) (or softmax); consecutive experts form `groups` groups of equal size, ranked by
//                      the top-2 sum of their scores; all but the `keep` highest-ranked groups are barred; then the `top`
//                      highest-scoring experts that are not barred; weights = score / (sum of the chosen + 1e-20) * scale,
//                      or score * scale; or the logits rank and choose, and the weights are their softmax over the chosen alone,
//                      times scale.  An optional correction per expert is added to the scores that choose (groups
//                      and experts) and not to the weights.  Ties go to the lower index.
//   ns_moe_plan        counts per expert, their running offsets, and for every (token, choice) its row in the
//                      order that has each expert's tokens side by side; a choice beyond the experts that have weights (an
//                      expert that returns its input) has no row: -1
//   ns_moe_route_plan  both in one launch, for steps of a few tokens
//   ns_moe_pad_rows    the same rows in a layout where every expert owns a fixed number of rows (for one batched product)
//   ns_moe_gather      x rows into that order
//   ns_moe_combine     out[n] = sum_k weight[n, k] * y[row(n, k)] in float (x[n] in place of y for a choice without a row),
//                      or the same sum added to a float stream
//   ns_moe_expert_rows the experts themselves for a few tokens, no host round trip: one block row per (token,
//                      choice) streams the chosen expert's gate and up rows, then its down rows
//   ns_activation      out = act(x) elementwise: exact (erf) gelu, tanh gelu, silu, squared relu, xielu
#include "common.cuh"

namespace {

template <typename T>
__global__ void cast_f32_kernel(const T* __restrict__ x, long long ldx, float* __restrict__ out, int cols, size_t total) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t row = i / cols;
    out[i] = ns_ld(x, row * ldx + (i - row * cols));
}

constexpr int kMaxExperts = 1024;

// logits[n, e] = x[n] . w[e] (+ bias[e]) in float: a block takes TOK tokens (their rows in shared memory) and eight experts, a warp per expert,
// so a row of w is read once for TOK tokens.  The sum over a row runs in the same order whatever TOK is.
template <typename T, int TOK>
__global__ void __launch_bounds__(256)
router_logits_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ w, const float* __restrict__ bias,
                     float* __restrict__ logits, int n_tokens, int E, int K) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    extern __shared__ __align__(16) float xrow[];  // [TOK][K4]
    const int K4 = (K + 3) / 4 * 4;
    const int n0 = blockIdx.x * TOK, lane = threadIdx.x & 31, e = blockIdx.y * 8 + (threadIdx.x >> 5);
    const int cnt = min(TOK, n_tokens - n0);
    const bool vec = K % 8 == 0 && ldx % 8 == 0 && (((uintptr_t)w | (uintptr_t)x) % 16 == 0);
    if (vec) {
        const int per_row = K / 8;
        for (int i = threadIdx.x; i < TOK * per_row; i += blockDim.x) {
            const int t = i / per_row, k = (i - t * per_row) * 8;
            float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if (t < cnt) ld8(x + (size_t)(n0 + t) * ldx + k, v);
            st8(xrow + (size_t)t * K4 + k, v);
        }
    } else {
        for (int i = threadIdx.x; i < TOK * K; i += blockDim.x) {
            const int t = i / K, k = i - t * K;
            xrow[(size_t)t * K4 + k] = t < cnt ? ns_ld(x, (size_t)(n0 + t) * ldx + k) : 0.f;
        }
    }
    __syncthreads();
    if (e >= E) return;
    const float* wr = w + (size_t)e * K;
    float a[TOK];
#pragma unroll
    for (int t = 0; t < TOK; ++t) a[t] = 0.f;
    if (vec) {
#pragma unroll 4
        for (int k = lane * 4; k < K; k += 128) {
            const float4 v = *reinterpret_cast<const float4*>(wr + k);
#pragma unroll
            for (int t = 0; t < TOK; ++t) {
                const float4 u = *reinterpret_cast<const float4*>(xrow + (size_t)t * K4 + k);
                a[t] = fmaf(v.x, u.x, a[t]); a[t] = fmaf(v.y, u.y, a[t]); a[t] = fmaf(v.z, u.z, a[t]); a[t] = fmaf(v.w, u.w, a[t]);
            }
        }
    } else {
        for (int k = lane; k < K; k += 32) {
            const float v = wr[k];
#pragma unroll
            for (int t = 0; t < TOK; ++t) a[t] = fmaf(v, xrow[(size_t)t * K4 + k], a[t]);
        }
    }
#pragma unroll
    for (int t = 0; t < TOK; ++t) {
        const float v = ns_warp_sum(a[t]) + (bias ? bias[e] : 0.f);
        if (lane == 0 && t < cnt) logits[(size_t)(n0 + t) * E + e] = v;
    }
}

struct RouteRule {
    int E, groups, keep, top;
    float scale;
    int softmax;  // 0: sigmoid scores, 1: a softmax over all, 2: a softmax over the chosen alone (the logits choose)
    const float* correction;
    int renormalize;
};

// one token by one warp: z [E] its logits, sc [3 E] scratch in shared memory, ids and weights [top] its results
__device__ __forceinline__ void route_token(const float* __restrict__ z, const RouteRule& r, float* sc, int* __restrict__ ids,
                                            float* __restrict__ weights, int lane) {
    const int E = r.E, groups = r.groups, top = r.top;
    float* cs = sc + E;  // scores, the scores that choose, then group scores (at most E of them)
    float* gs = cs + E;
    if (r.softmax) {
        float mx = -INFINITY;
        for (int e = lane; e < E; e += 32) mx = fmaxf(mx, z[e]);
        mx = ns_warp_max(mx);
        float sum = 0.f;
        for (int e = lane; e < E; e += 32) {
            const float v = expf(z[e] - mx);
            sc[e] = v;
            sum += v;
        }
        if (r.softmax == 1) {
            sum = ns_warp_sum(sum);
            for (int e = lane; e < E; e += 32) sc[e] /= sum;
        }
    } else {
        for (int e = lane; e < E; e += 32) sc[e] = 1.f / (1.f + expf(-z[e]));
    }
    for (int e = lane; e < E; e += 32) cs[e] = (r.softmax == 2 ? z[e] : sc[e]) + (r.correction ? r.correction[e] : 0.f);
    __syncwarp();
    const float taken = -INFINITY;  // a taken or barred entry
    if (groups > 1) {
        const int per = E / groups;
        for (int g = lane; g < groups; g += 32) {
            float a = -INFINITY, b = -INFINITY;  // the two largest
            for (int e = g * per; e < (g + 1) * per; ++e) {
                const float v = cs[e];
                if (v > a) { b = a; a = v; } else if (v > b) { b = v; }
            }
            gs[g] = per > 1 ? a + b : a;
        }
        __syncwarp();
        // the best `keep` groups stay; the others' experts are barred
        for (int round = 0; round < groups - r.keep; ++round) {  // bar the worst, one a round (the higher index at a tie)
            float worst = INFINITY;
            int wi = -1;
            for (int g = lane; g < groups; g += 32) {
                const float v = gs[g];
                if (v > taken && (v < worst || (v == worst && g > wi))) { worst = v; wi = g; }
            }
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, worst, o);
                const int oi = __shfl_xor_sync(0xffffffffu, wi, o);
                if (oi >= 0 && (wi < 0 || ov < worst || (ov == worst && oi > wi))) { worst = ov; wi = oi; }
            }
            if (lane == 0 && wi >= 0) gs[wi] = taken;
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (gs[e / per] == taken) cs[e] = taken;
        __syncwarp();
    }
    float total = 0.f, mine = 0.f;
    int mine_id = 0;
    for (int k = 0; k < top; ++k) {
        float best = taken;
        int bi = -1;
        for (int e = lane; e < E; e += 32) {
            const float v = cs[e];
            if (v > best) { best = v; bi = e; }  // ascending e: the lower index wins a tie
        }
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (oi >= 0 && (bi < 0 || ov > best || (ov == best && oi < bi))) { best = ov; bi = oi; }
        }
        bi = max(bi, 0);  // (no score above the marker is left only when the logits are not numbers)
        const float w = sc[bi];
        total += w;
        if (lane == k % 32 && k < 32) { mine = w; mine_id = bi; }
        if (k >= 32 && lane == 0) {  // more than 32 choices: written unnormalised, fixed up below
            ids[k] = bi;
            weights[k] = w;
        }
        if (lane == 0) cs[bi] = taken;
        __syncwarp();
    }
    // (a softmax over the chosen: the largest logit is among them, so the total is 1 or more)
    const float f = r.renormalize || r.softmax == 2 ? r.scale / (total + 1e-20f) : r.scale;
    if (lane < top && lane < 32) {
        ids[lane] = mine_id;
        weights[lane] = mine * f;
    }
    __syncwarp();
    for (int k = 32 + lane; k < top; k += 32) weights[k] *= f;
}

// one warp per token
__global__ void __launch_bounds__(128)
moe_route_kernel(const float* __restrict__ logits, int n_tokens, RouteRule r, int* __restrict__ ids, float* __restrict__ weights) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    extern __shared__ float rs[];
    const int wib = threadIdx.x >> 5;
    const int n = blockIdx.x * 4 + wib;
    if (n >= n_tokens) return;
    route_token(logits + (size_t)n * r.E, r, rs + (size_t)wib * 3 * r.E, ids + (size_t)n * r.top, weights + (size_t)n * r.top, threadIdx.x & 31);
}

// one block: counts, offsets, rows
__device__ __forceinline__ void plan_pairs(const int* ids, int n_pairs, int E, int* __restrict__ offsets, int* __restrict__ row_of,
                                           int* __restrict__ pair_of, int* count, int* cursor) {
    const int tid = threadIdx.x;
    for (int e = tid; e < E; e += blockDim.x) count[e] = 0;
    __syncthreads();
    for (int i = tid; i < n_pairs; i += blockDim.x)
        if (ids[i] < E) atomicAdd(&count[ids[i]], 1);
    __syncthreads();
    if (tid < 32) {  // running sums, 32 experts at a time
        int at = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + tid, c = e < E ? count[e] : 0;
            int sum = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, sum, o);
                if (tid >= o) sum += v;
            }
            if (e < E) {
                offsets[e] = at + sum - c;
                cursor[e] = at + sum - c;
            }
            at += __shfl_sync(0xffffffffu, sum, 31);
        }
        if (tid == 0) offsets[E] = at;
    }
    __syncthreads();
    // which row of its expert's run a pair gets does not matter to any result: rows are computed alone
    for (int i = tid; i < n_pairs; i += blockDim.x) {
        const int e = ids[i];
        const int row = e < E ? atomicAdd(&cursor[e], 1) : -1;
        row_of[i] = row;
        if (pair_of && row >= 0) pair_of[row] = i;
    }
}

__global__ void __launch_bounds__(1024)
moe_plan_kernel(const int* __restrict__ ids, int n_pairs, int E, int* __restrict__ offsets, int* __restrict__ row_of,
                int* __restrict__ pair_of) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    __shared__ int count[kMaxExperts], cursor[kMaxExperts];
    plan_pairs(ids, n_pairs, E, offsets, row_of, pair_of, count, cursor);
}

// both for a step of a few tokens: one block, its warps take the tokens in turn, then the plan over what they chose
__global__ void __launch_bounds__(1024)
moe_route_plan_kernel(const float* __restrict__ logits, int n_tokens, RouteRule r, int* ids, float* __restrict__ weights, int E,
                      int* __restrict__ offsets, int* __restrict__ row_of, int* __restrict__ pair_of) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    __shared__ int count[kMaxExperts], cursor[kMaxExperts];
    extern __shared__ float rs[];
    const int warp = threadIdx.x >> 5;
    for (int n = warp; n < n_tokens; n += blockDim.x >> 5)
        route_token(logits + (size_t)n * r.E, r, rs + (size_t)warp * 3 * r.E, ids + (size_t)n * r.top, weights + (size_t)n * r.top, threadIdx.x & 31);
    __syncthreads();  // (a block's own writes to global memory are visible to it after the barrier)
    plan_pairs(ids, n_tokens * r.top, E, offsets, row_of, pair_of, count, cursor);
}

// rows of the plan moved to a layout in which every expert owns `capacity` rows: row = expert * capacity + rank in the expert
__global__ void moe_pad_rows_kernel(const int* __restrict__ ids, const int* __restrict__ offsets, int* __restrict__ row_of, int n_pairs,
                                    int capacity) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n_pairs) return;
    if (row_of[i] < 0) return;  // a choice without a row
    const int e = ids[i];
    row_of[i] = e * capacity + (row_of[i] - offsets[e]);
}

template <typename T, int VEC>
__global__ void moe_gather_kernel(const T* __restrict__ x, const int* __restrict__ row_of, T* __restrict__ xs, int top,
                                  int width) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const int pair = blockIdx.x;
    if (row_of[pair] < 0) return;
    const T* src = x + (size_t)(pair / top) * width;
    T* dst = xs + (size_t)row_of[pair] * width;
    if constexpr (VEC == 1) {
        for (int h = threadIdx.x; h < width; h += blockDim.x) dst[h] = src[h];
    } else {
        for (int h = threadIdx.x * VEC; h < width; h += blockDim.x * VEC)  // 16-byte pieces
            *reinterpret_cast<uint4*>(dst + h) = *reinterpret_cast<const uint4*>(src + h);
    }
}

// out[n] = sum_k weight[n, k] * (row >= 0 ? ys[row] : x[n]), float sums in the order of the choice, rounded once; with `resid`
// the sum is added to that float row instead.  VEC = 8: eight features to a thread with 16-byte accesses.
template <typename T, int VEC>
__global__ void moe_combine_kernel(const T* __restrict__ ys, const int* __restrict__ row_of, const float* __restrict__ weights,
                                   const T* __restrict__ x, T* __restrict__ out, float* __restrict__ resid, int top, int width) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const int n = blockIdx.x;
    const int* rows = row_of + (size_t)n * top;
    const float* w = weights + (size_t)n * top;
    for (int h = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; h < width; h += gridDim.y * blockDim.x * VEC) {
        const size_t at = (size_t)n * width + h;
        if constexpr (VEC == 8) {
            float a[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) a[i] = 0.f;
            for (int k = 0; k < top; ++k) {
                const int row = rows[k];
                const float wk = w[k];
                float v[8];
                ld8(row >= 0 ? ys + (size_t)row * width + h : x + at, v);
#pragma unroll
                for (int i = 0; i < 8; ++i) a[i] = fmaf(wk, v[i], a[i]);
            }
            if (resid) {
                float v[8];
                ld8(resid + at, v);
#pragma unroll
                for (int i = 0; i < 8; ++i) a[i] += v[i];
                st8(resid + at, a);
            } else {
                st8(out + at, a);
            }
        } else {
            float a = 0.f;
            for (int k = 0; k < top; ++k) a = fmaf(w[k], rows[k] >= 0 ? ns_ld(ys, (size_t)rows[k] * width + h) : ns_ld(x, at), a);
            if (resid) resid[at] += a;
            else ns_st(out, at, a);
        }
    }
}

template <typename T>
__device__ __forceinline__ float dot_row(const T* __restrict__ w, const float* __restrict__ xs, int K, int lane, bool vec) {
    float a = 0.f;
    if (vec) {
        for (int k = lane * 8; k < K; k += 256) {
            float v[8];
            ld8(w + k, v);
#pragma unroll
            for (int i = 0; i < 8; ++i) a = fmaf(v[i], xs[k + i], a);
        }
    } else {
        for (int k = lane; k < K; k += 32) a = fmaf(ns_ld(w, k), xs[k], a);
    }
    return ns_warp_sum(a);
}

// act[pair, j] = silu(gate_e[j] . x) * (up_e[j] . x), or another unit of that form; grid (pairs, feature chunks), a warp per feature
template <typename T>
__global__ void __launch_bounds__(256)
moe_gate_up_rows_kernel(const T* __restrict__ x, const int* __restrict__ ids, const T* __restrict__ w_gate,
                        const T* __restrict__ w_up, T* __restrict__ act, int E, int top, int width, int ff, int per_block, NsGate unit) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    extern __shared__ float xs[];
    const int pair = blockIdx.x, lane = threadIdx.x & 31, wib = threadIdx.x >> 5;
    const int e = ids[pair];
    if (e >= E) return;  // returns its input: nothing to compute here
    const T* xr = x + (size_t)(pair / top) * width;
    for (int k = threadIdx.x; k < width; k += blockDim.x) xs[k] = ns_ld(xr, k);
    __syncthreads();
    const bool vec = width % 8 == 0 && (((uintptr_t)w_gate | (uintptr_t)w_up) % 16 == 0);
    const int j0 = blockIdx.y * per_block, j1 = min(ff, j0 + per_block);
    for (int j = j0 + wib; j < j1; j += 8) {
        const size_t off = ((size_t)e * ff + j) * width;
        const float g = dot_row(w_gate + off, xs, width, lane, vec);
        const float u = dot_row(w_up + off, xs, width, lane, vec);
        if (lane == 0) ns_st(act, (size_t)pair * ff + j, ns_gate_mul<false>(unit, g, u));
    }
}

// out[n, i] = sum_k weight[n, k] * (down_e(k)[i] . act[n, k]), x[n, i] in place of the product for e(k) >= E; grid (tokens, feature chunks)
template <typename T>
__global__ void __launch_bounds__(256)
moe_down_rows_kernel(const T* __restrict__ act, const int* __restrict__ ids, const float* __restrict__ weights,
                     const T* __restrict__ w_down, const T* __restrict__ x, T* __restrict__ out, int E, int top, int width, int ff,
                     int per_block) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    extern __shared__ float as[];  // [top][ff]
    const int n = blockIdx.x, lane = threadIdx.x & 31, wib = threadIdx.x >> 5;
    for (int i = threadIdx.x; i < top * ff; i += blockDim.x)
        as[i] = ids[(size_t)n * top + i / ff] < E ? ns_ld(act, (size_t)n * top * ff + i) : 0.f;
    __syncthreads();
    const bool vec = ff % 8 == 0 && ((uintptr_t)w_down % 16 == 0);
    const int i0 = blockIdx.y * per_block, i1 = min(width, i0 + per_block);
    for (int i = i0 + wib; i < i1; i += 8) {
        float a = 0.f;
        for (int k = 0; k < top; ++k) {
            const int e = ids[(size_t)n * top + k];
            if (e >= E) {
                a = fmaf(weights[(size_t)n * top + k], ns_ld(x, (size_t)n * width + i), a);
                continue;
            }
            a = fmaf(weights[(size_t)n * top + k], dot_row(w_down + ((size_t)e * width + i) * ff, as + (size_t)k * ff, ff, lane, vec), a);
        }
        if (lane == 0) ns_st(out, (size_t)n * width + i, a);
    }
}

// xielu's coefficients, taken by the kinds that have none as well: a of the quadratic branch, b of the exponential one
struct ActCoef { float a, b; };
__device__ __forceinline__ ActCoef act_coef(const float* coef) { return coef ? ActCoef{coef[0], coef[1]} : ActCoef{0.f, 0.f}; }

__device__ __forceinline__ float act_value(float z, int kind, ActCoef c) {
    if (kind == 0) return 0.5f * z * (1.f + erff(z * 0.70710678118654752440f));
    if (kind == 1) return 0.5f * z * (1.f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
    if (kind == 3) { const float p = fmaxf(z, 0.f); return p * p; }
    if (kind == 4) return (z > 0.f ? c.a * z * z : c.b * (expm1f(z) - z)) + 0.5f * z;
    return z / (1.f + expf(-z));
}

template <typename T>
__global__ void activation_vec_kernel(const T* __restrict__ x, T* __restrict__ out, int kind, const float* __restrict__ coef, size_t total8) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total8) return;
    float v[8];
    ld8(x + i * 8, v);
    const ActCoef c = act_coef(coef);
#pragma unroll
    for (int k = 0; k < 8; ++k) v[k] = act_value(v[k], kind, c);
    st8(out + i * 8, v);
}

// rows of `cols` features with strides of their own (column ranges of wider buffers); VEC = 8 needs both rows on 16 bytes
template <typename T, int VEC>
__global__ void activation_rows_kernel(const T* __restrict__ x, long long ldx, T* __restrict__ out, long long ldo, int cols, int kind,
                                       const float* __restrict__ coef, size_t total) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int per_row = cols / VEC;
    const size_t row = i / per_row;
    const int c = (int)(i - row * per_row) * VEC;
    const ActCoef co = act_coef(coef);
    if constexpr (VEC == 8) {
        float v[8];
        ld8(x + row * ldx + c, v);
#pragma unroll
        for (int k = 0; k < 8; ++k) v[k] = act_value(v[k], kind, co);
        st8(out + row * ldo + c, v);
    } else {
        ns_st(out, row * ldo + c, act_value(ns_ld(x, row * ldx + c), kind, co));
    }
}

template <typename T>
__global__ void activation_kernel(const T* __restrict__ x, T* __restrict__ out, int kind, const float* __restrict__ coef, size_t total) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    ns_st(out, i, act_value(ns_ld(x, i), kind, act_coef(coef)));
}

}  // namespace

NS_API int ns_cast_f32(const void* x, long long ldx, float* out, int n_rows, int cols, int dtype, cudaStream_t stream) {
    const size_t total = (size_t)n_rows * cols;
    if (total == 0) return NS_OK;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == NS_F32) NS_LAUNCH((cast_f32_kernel<float>), blocks, 256, 0, stream, (const float*)x, ldx, out, cols, total);
    else if (dtype == NS_BF16) NS_LAUNCH((cast_f32_kernel<__nv_bfloat16>), blocks, 256, 0, stream, (const __nv_bfloat16*)x, ldx, out, cols, total);
    else NS_FAIL(NS_ERR_ARGUMENT, "ns_cast_f32: unknown dtype %d", dtype);
    NS_CHECK_LAUNCH("ns_cast_f32");
    return NS_OK;
}

// x [n, K] (row stride ldx) in the compute type, w [E, K] and bias [E] (or null) float, logits [n, E] float
NS_API int ns_router_logits(const void* x, long long ldx, const float* w, const float* bias, float* logits, int n_tokens, int E, int K, int dtype,
                            cudaStream_t stream) {
    if (n_tokens <= 0) return NS_OK;
    const size_t row = (size_t)(K + 3) / 4 * 4 * sizeof(float);
    if (row > 200 * 1024) NS_FAIL(NS_ERR_UNSUPPORTED, "ns_router_logits: a row of %d floats does not fit shared memory", K);
    if (dtype != NS_F32 && dtype != NS_BF16) NS_FAIL(NS_ERR_ARGUMENT, "ns_router_logits: unknown dtype %d", dtype);
    // tokens to a block: one while that gives few blocks, more as the step grows (two blocks of 100 KB an SM)
    int tok = n_tokens <= 32 ? 1 : n_tokens <= 128 ? 2 : n_tokens <= 512 ? 4 : 8;
    while (tok > 1 && tok * row > 100 * 1024) tok /= 2;
    const size_t smem = tok * row;
    const dim3 grid((n_tokens + tok - 1) / tok, (E + 7) / 8);
#define NS_ROUTER(T, TK)                                                                                                              \
    {                                                                                                                                 \
        if (smem > 48 * 1024) NS_CUDA(cudaFuncSetAttribute(router_logits_kernel<T, TK>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); \
        NS_LAUNCH((router_logits_kernel<T, TK>), grid, 256, smem, stream, (const T*)x, ldx, w, bias, logits, n_tokens, E, K);         \
    }
#define NS_ROUTER_T(T) { if (tok == 1) NS_ROUTER(T, 1) else if (tok == 2) NS_ROUTER(T, 2) else if (tok == 4) NS_ROUTER(T, 4) else NS_ROUTER(T, 8) }
    if (dtype == NS_F32) NS_ROUTER_T(float)
    else NS_ROUTER_T(__nv_bfloat16)
#undef NS_ROUTER_T
#undef NS_ROUTER
    NS_CHECK_LAUNCH("ns_router_logits");
    return NS_OK;
}

namespace {
int check_rule(const RouteRule& r) {
    if (r.E < 1 || r.E > kMaxExperts || r.top < 1 || r.top > r.E)
        NS_FAIL(NS_ERR_UNSUPPORTED, "ns_moe_route: %d experts, %d chosen (at most %d experts)", r.E, r.top, kMaxExperts);
    if (r.groups > 1 && (r.E % r.groups || r.keep < 1 || r.keep > r.groups || r.keep * (r.E / r.groups) < r.top))
        NS_FAIL(NS_ERR_ARGUMENT, "ns_moe_route: %d groups over %d experts, %d kept, %d chosen", r.groups, r.E, r.keep, r.top);
    return NS_OK;
}
}  // namespace

NS_API int ns_moe_route(const float* logits, int n_tokens, int E, int groups, int keep, int top, float scale, int softmax,
                        const float* correction, int renormalize, int* ids, float* weights, cudaStream_t stream) {
    if (n_tokens <= 0) return NS_OK;
    const RouteRule r{E, groups, keep, top, scale, softmax, correction, renormalize};
    if (const int rc = check_rule(r)) return rc;
    const size_t smem = (size_t)4 * 3 * E * sizeof(float);
    NS_LAUNCH(moe_route_kernel, (n_tokens + 3) / 4, 128, smem, stream, logits, n_tokens, r, ids, weights);
    NS_CHECK_LAUNCH("ns_moe_route");
    return NS_OK;
}

// ns_moe_route and ns_moe_plan in one launch of one block: E router outputs, n_experts of them with rows in the plan (at most 512 outputs)
NS_API int ns_moe_route_plan(const float* logits, int n_tokens, int E, int groups, int keep, int top, float scale, int softmax,
                             const float* correction, int renormalize, int* ids, float* weights, int n_experts, int* offsets, int* row_of,
                             int* pair_of, cudaStream_t stream) {
    if (n_tokens <= 0) return NS_OK;
    const RouteRule r{E, groups, keep, top, scale, softmax, correction, renormalize};
    if (const int rc = check_rule(r)) return rc;
    const int warps = n_tokens < 32 ? (n_tokens < 4 ? 4 : n_tokens) : 32;
    const size_t smem = (size_t)warps * 3 * E * sizeof(float);
    if (E > 512 || n_experts < 1 || n_experts > E) NS_FAIL(NS_ERR_UNSUPPORTED, "ns_moe_route_plan: %d of %d experts (at most 512)", n_experts, E);
    if (smem > 40 * 1024) NS_CUDA(cudaFuncSetAttribute(moe_route_plan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    NS_LAUNCH(moe_route_plan_kernel, 1, warps * 32, smem, stream, logits, n_tokens, r, ids, weights, n_experts, offsets, row_of, pair_of);
    NS_CHECK_LAUNCH("ns_moe_route_plan");
    return NS_OK;
}

// pair_of (optional): the inverse of row_of
NS_API int ns_moe_plan(const int* ids, int n_pairs, int E, int* offsets, int* row_of, int* pair_of, cudaStream_t stream) {
    if (E < 1 || E > kMaxExperts) NS_FAIL(NS_ERR_UNSUPPORTED, "ns_moe_plan: %d experts (at most %d)", E, kMaxExperts);
    NS_LAUNCH(moe_plan_kernel, 1, 1024, 0, stream, ids, n_pairs, E, offsets, row_of, pair_of);
    NS_CHECK_LAUNCH("ns_moe_plan");
    return NS_OK;
}

NS_API int ns_moe_pad_rows(const int* ids, const int* offsets, int* row_of, int n_pairs, int capacity, cudaStream_t stream) {
    if (n_pairs <= 0) return NS_OK;
    NS_LAUNCH(moe_pad_rows_kernel, (n_pairs + 255) / 256, 256, 0, stream, ids, offsets, row_of, n_pairs, capacity);
    NS_CHECK_LAUNCH("ns_moe_pad_rows");
    return NS_OK;
}

NS_API int ns_moe_gather(const void* x, const int* row_of, void* xs, int n_tokens, int top, int width, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return NS_OK;
    const bool vec = width % 8 == 0 && (((uintptr_t)x | (uintptr_t)xs) % 16 == 0);
    if (dtype == NS_F32 && vec) NS_LAUNCH((moe_gather_kernel<float, 4>), n_tokens * top, 128, 0, stream, (const float*)x, row_of, (float*)xs, top, width);
    else if (dtype == NS_F32) NS_LAUNCH((moe_gather_kernel<float, 1>), n_tokens * top, 128, 0, stream, (const float*)x, row_of, (float*)xs, top, width);
    else if (dtype == NS_BF16 && vec) NS_LAUNCH((moe_gather_kernel<__nv_bfloat16, 8>), n_tokens * top, 128, 0, stream, (const __nv_bfloat16*)x, row_of, (__nv_bfloat16*)xs, top, width);
    else if (dtype == NS_BF16) NS_LAUNCH((moe_gather_kernel<__nv_bfloat16, 1>), n_tokens * top, 128, 0, stream, (const __nv_bfloat16*)x, row_of, (__nv_bfloat16*)xs, top, width);
    else NS_FAIL(NS_ERR_ARGUMENT, "ns_moe_gather: unknown dtype %d", dtype);
    NS_CHECK_LAUNCH("ns_moe_gather");
    return NS_OK;
}

// x [n, width] (only read for choices without a row); resid (float) or out receives the sum
NS_API int ns_moe_combine(const void* ys, const int* row_of, const float* weights, const void* x, void* out, float* resid, int n_tokens,
                          int top, int width, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return NS_OK;
    if (dtype != NS_F32 && dtype != NS_BF16) NS_FAIL(NS_ERR_ARGUMENT, "ns_moe_combine: unknown dtype %d", dtype);
    if (!out && !resid) NS_FAIL(NS_ERR_ARGUMENT, "ns_moe_combine: nowhere to put the sum");
    const bool vec = width % 8 == 0 && (((uintptr_t)ys | (uintptr_t)x | (uintptr_t)out | (uintptr_t)resid) % 16 == 0);
    const int per_row = vec ? width / 8 : width;
    const int threads = per_row >= 256 ? 256 : (per_row + 31) / 32 * 32;
    const dim3 grid(n_tokens, vec ? (per_row + threads - 1) / threads : 1);
#define NS_COMBINE(T, V) NS_LAUNCH((moe_combine_kernel<T, V>), grid, threads, 0, stream, (const T*)ys, row_of, weights, (const T*)x, (T*)out, resid, top, width)
    if (dtype == NS_F32) { if (vec) NS_COMBINE(float, 8); else NS_COMBINE(float, 1); }
    else { if (vec) NS_COMBINE(__nv_bfloat16, 8); else NS_COMBINE(__nv_bfloat16, 1); }
#undef NS_COMBINE
    NS_CHECK_LAUNCH("ns_moe_combine");
    return NS_OK;
}

// x [n, width]; ids, weights [n, top]; w_gate, w_up [E, ff, width]; w_down [E, width, ff]; act [n * top, ff] scratch;
// out [n, width]; ids from n_experts on return their input; alpha, shift, limit: NsGate
NS_API int ns_moe_expert_rows(const void* x, const int* ids, const float* weights, const void* w_gate, const void* w_up,
                              const void* w_down, void* act, void* out, int n_experts, int n_tokens, int top, int width,
                              int ff, float alpha, float shift, float limit, int dtype, cudaStream_t stream) {
    const NsGate unit{alpha, shift, limit};
    if (n_tokens <= 0) return NS_OK;
    const size_t smem_a = (size_t)width * sizeof(float), smem_b = (size_t)top * ff * sizeof(float);
    if (smem_a > 200 * 1024 || smem_b > 200 * 1024)
        NS_FAIL(NS_ERR_UNSUPPORTED, "ns_moe_expert_rows: a row of %d or %d x %d floats does not fit shared memory", width, top, ff);
    const int per_a = 64, per_b = 64;
    dim3 grid_a(n_tokens * top, (ff + per_a - 1) / per_a), grid_b(n_tokens, (width + per_b - 1) / per_b);
#define NS_MOE_ROWS(T)                                                                                                        \
    {                                                                                                                         \
        if (smem_a > 48 * 1024) NS_CUDA(cudaFuncSetAttribute(moe_gate_up_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); \
        if (smem_b > 48 * 1024) NS_CUDA(cudaFuncSetAttribute(moe_down_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));    \
        NS_LAUNCH((moe_gate_up_rows_kernel<T>), grid_a, 256, smem_a, stream, (const T*)x, ids, (const T*)w_gate, (const T*)w_up,      \
                  (T*)act, n_experts, top, width, ff, per_a, unit);                                                                          \
        NS_CHECK_LAUNCH("ns_moe_expert_rows");                                                                                \
        NS_LAUNCH((moe_down_rows_kernel<T>), grid_b, 256, smem_b, stream, (const T*)act, ids, weights, (const T*)w_down, (const T*)x, (T*)out,     \
                  n_experts, top, width, ff, per_b);                                                                                     \
    }
    if (dtype == NS_F32) NS_MOE_ROWS(float)
    else if (dtype == NS_BF16) NS_MOE_ROWS(__nv_bfloat16)
    else NS_FAIL(NS_ERR_ARGUMENT, "ns_moe_expert_rows: unknown dtype %d", dtype);
#undef NS_MOE_ROWS
    NS_CHECK_LAUNCH("ns_moe_expert_rows");
    return NS_OK;
}

// the same over rows that lie in wider buffers: x[r * ldx + c] -> out[r * ldo + c], c < cols
NS_API int ns_activation_rows(const void* x, long long ldx, void* out, long long ldo, int n_rows, int cols, int kind,
                              const float* coef, int dtype, cudaStream_t stream) {
    if (n_rows <= 0 || cols <= 0) return NS_OK;
    if (kind < 0 || kind > 4 || (kind == 4 && !coef)) NS_FAIL(NS_ERR_ARGUMENT, "ns_activation_rows: unknown kind %d", kind);
    if (dtype != NS_F32 && dtype != NS_BF16) NS_FAIL(NS_ERR_ARGUMENT, "ns_activation_rows: unknown dtype %d", dtype);
    const size_t esz = dtype == NS_F32 ? 4 : 2;
    const bool vec = cols % 8 == 0 && (((uintptr_t)x | (uintptr_t)out) % 16 == 0) && (ldx * esz) % 16 == 0 && (ldo * esz) % 16 == 0;
    const size_t total = (size_t)n_rows * (vec ? cols / 8 : cols);
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == NS_F32) {
        if (vec) NS_LAUNCH((activation_rows_kernel<float, 8>), blocks, 256, 0, stream, (const float*)x, ldx, (float*)out, ldo, cols, kind, coef, total);
        else NS_LAUNCH((activation_rows_kernel<float, 1>), blocks, 256, 0, stream, (const float*)x, ldx, (float*)out, ldo, cols, kind, coef, total);
    } else {
        if (vec) NS_LAUNCH((activation_rows_kernel<__nv_bfloat16, 8>), blocks, 256, 0, stream, (const __nv_bfloat16*)x, ldx, (__nv_bfloat16*)out, ldo, cols, kind, coef, total);
        else NS_LAUNCH((activation_rows_kernel<__nv_bfloat16, 1>), blocks, 256, 0, stream, (const __nv_bfloat16*)x, ldx, (__nv_bfloat16*)out, ldo, cols, kind, coef, total);
    }
    NS_CHECK_LAUNCH("ns_activation_rows");
    return NS_OK;
}

// kind 0: 0.5 z (1 + erf(z / sqrt 2));  1: 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3)));  2: z sigmoid(z);  3: max(z, 0)^2;
// 4: (z > 0 ? a z^2 : b (exp(z) - 1 - z)) + z / 2 with a, b = coef[0], coef[1] (float, on the device)
NS_API int ns_activation(const void* x, void* out, long long total, int kind, const float* coef, int dtype, cudaStream_t stream) {
    if (total <= 0) return NS_OK;
    if (kind < 0 || kind > 4 || (kind == 4 && !coef)) NS_FAIL(NS_ERR_ARGUMENT, "ns_activation: unknown kind %d", kind);
    if (total % 8 == 0 && (((uintptr_t)x | (uintptr_t)out) % 16 == 0)) {  // eight elements to a thread
        const size_t total8 = (size_t)total / 8;
        const unsigned vblocks = (unsigned)((total8 + 255) / 256);
        if (dtype == NS_F32) NS_LAUNCH((activation_vec_kernel<float>), vblocks, 256, 0, stream, (const float*)x, (float*)out, kind, coef, total8);
        else if (dtype == NS_BF16) NS_LAUNCH((activation_vec_kernel<__nv_bfloat16>), vblocks, 256, 0, stream, (const __nv_bfloat16*)x, (__nv_bfloat16*)out, kind, coef, total8);
        else NS_FAIL(NS_ERR_ARGUMENT, "ns_activation: unknown dtype %d", dtype);
        NS_CHECK_LAUNCH("ns_activation");
        return NS_OK;
    }
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == NS_F32) NS_LAUNCH((activation_kernel<float>), blocks, 256, 0, stream, (const float*)x, (float*)out, kind, coef, (size_t)total);
    else if (dtype == NS_BF16) NS_LAUNCH((activation_kernel<__nv_bfloat16>), blocks, 256, 0, stream, (const __nv_bfloat16*)x, (__nv_bfloat16*)out, kind, coef, (size_t)total);
    else NS_FAIL(NS_ERR_ARGUMENT, "ns_activation: unknown dtype %d", dtype);
    NS_CHECK_LAUNCH("ns_activation");
    return NS_OK;
}
