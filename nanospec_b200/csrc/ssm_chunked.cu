// The state space of Mamba-2 over long portions of prompts, a chunk of 64 tokens at a time instead of a token at a time.
//
// Per head, with step sizes a_t and l_t = -exp(A_log) a_t (the logarithm of the decay), L_t the sum of l over a chunk up to t and S_in the
// state before the chunk:
//     y_t   = exp(L_t) S_in^T C_t + sum_{s <= t} exp(L_t - L_s) a_s (C_t . B_s) x_s
//     S_out = exp(L_end) S_in + sum_s exp(L_end - L_s) a_s B_s x_s^T
// which is the recurrence S = exp(l) S + a B x^T, y = S^T C written out over the chunk.  Three kernels:
//     chunk_states   the sum over a chunk (a product over its tokens), every chunk and head at once, and the chunk's decay exp(L_end)
//     chunk_pass     the chunks of a request in order, element by element of the state: S_in of every chunk, and the request's state
//     chunk_outputs  y of a chunk: C B^T masked and weighted, times x, plus C S_in scaled
// Everything is float (the same operands as the token walk's: csrc/recurrent.cu), L and its differences double, so that a difference of
// two large sums keeps its digits.  A request's chunks start at its first token of the step; requests of fewer than min_len
// tokens are left to the token walk.  Blocks find their (request, chunk) from the step's token offsets on the device.
#include "common.cuh"

namespace {

constexpr int kQ = 64;         // tokens of a chunk
constexpr int kThreads = 128;  // 8 x 16 threads on a 64 x 64 tile, 8 x 4 results each
constexpr int kLd = 68;        // floats of a staged row: 16-byte aligned, rows in different banks

struct Chunk {
    int request, start, count, slot;  // count 0: no such chunk
};

// the chunk that slot number `slot` stands for; called by a whole warp
__device__ __forceinline__ Chunk find_chunk(int slot, const int* __restrict__ qo_indptr, int n_requests, int min_len) {
    const int lane = threadIdx.x & 31;
    int before = 0;
    for (int b0 = 0; b0 < n_requests; b0 += 32) {
        const int b = b0 + lane;
        const int start = b < n_requests ? qo_indptr[b] : 0, len = b < n_requests ? qo_indptr[b + 1] - start : 0;
        const int chunks = len >= min_len ? (len + kQ - 1) / kQ : 0;
        int sum = chunks;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int v = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += v;
        }
        const int c = slot - (before + sum - chunks);
        const unsigned who = __ballot_sync(0xffffffffu, c >= 0 && c < chunks);
        if (who) {
            const int src = __ffs(who) - 1;
            return {__shfl_sync(0xffffffffu, b, src), __shfl_sync(0xffffffffu, start + c * kQ, src),
                    __shfl_sync(0xffffffffu, min(kQ, len - c * kQ), src), slot};
        }
        before += __shfl_sync(0xffffffffu, sum, 31);
    }
    return {0, 0, 0, slot};
}

// running sums of l over the chunk (double) and the step sizes, by one warp, two tokens to a lane; tokens beyond the chunk have step 0
__device__ __forceinline__ void chunk_logs(const float* __restrict__ step, int ld, int start, int count, float a, double* L, float* dt) {
    const int lane = threadIdx.x & 31;
    const int t0 = 2 * lane, t1 = t0 + 1;
    const float d0 = t0 < count ? step[(size_t)(start + t0) * ld] : 0.f, d1 = t1 < count ? step[(size_t)(start + t1) * ld] : 0.f;
    const double l0 = -(double)(a * d0), l1 = -(double)(a * d1);
    double sum = l0 + l1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double v = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += v;
    }
    L[t0] = sum - l1;
    L[t1] = sum;
    dt[t0] = d0;
    dt[t1] = d1;
}

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }

// acc[8][4] += a[8] b[4]^T
__device__ __forceinline__ void outer(float (&acc)[8][4], const float4& a0, const float4& a1, const float4& b) {
    const float av[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
}

// rows of a staged tile: dst[r][c] = src[(row0 + r) * ld + c] for r < rows, c < cols, zeros elsewhere, 64 x 64; `scale` (or null) per row
__device__ __forceinline__ void stage_rows(float* dst, const float* __restrict__ src, int ld, int rows, int cols, const float* scale, bool vec) {
    if (vec) {
        for (int i = threadIdx.x; i < kQ * 16; i += kThreads) {
            const int r = i >> 4, c = (i & 15) * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < rows && c < cols) v = ld4(src + (size_t)r * ld + c);
            if (scale) { const float s = scale[r]; v.x *= s; v.y *= s; v.z *= s; v.w *= s; }
            *reinterpret_cast<float4*>(dst + r * kLd + c) = v;
        }
    } else {
        for (int i = threadIdx.x; i < kQ * kQ; i += kThreads) {
            const int r = i >> 6, c = i & 63;
            const float v = r < rows && c < cols ? src[(size_t)r * ld + c] : 0.f;
            dst[r * kLd + c] = scale ? v * scale[r] : v;
        }
    }
}

// grid (chunk slots, heads, tiles of 64 x 64 of the state)
__global__ void __launch_bounds__(kThreads)
chunk_states_kernel(const float* __restrict__ B, const float* __restrict__ x, const float* __restrict__ step, int ld,
                    const float* __restrict__ a_log, const int* __restrict__ qo_indptr, int n_requests, int min_len,
                    float* __restrict__ states, float* __restrict__ decays, int H, int G, int N, int Np, int V) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    __shared__ __align__(16) float Bs[kQ * kLd], xs[kQ * kLd];
    __shared__ double L[kQ];
    __shared__ float dt[kQ], w[kQ];
    __shared__ Chunk chunk;
    const int tid = threadIdx.x, h = blockIdx.y, g = h / (H / G);
    if (tid < 32) {
        const Chunk c = find_chunk(blockIdx.x, qo_indptr, n_requests, min_len);
        if (tid == 0) chunk = c;
        if (c.count > 0) chunk_logs(step + h, ld, c.start, c.count, expf(a_log[h]), L, dt);
    }
    __syncthreads();
    const Chunk c = chunk;
    if (c.count == 0) return;
    if (tid < kQ) w[tid] = expf((float)(L[kQ - 1] - L[tid])) * dt[tid];  // (tokens beyond the chunk: step 0)
    if (tid == 0 && blockIdx.z == 0) decays[(size_t)c.slot * H + h] = expf((float)L[kQ - 1]);
    __syncthreads();
    const int v_tiles = (V + 63) / 64, n0 = (blockIdx.z / v_tiles) * 64, v0 = (blockIdx.z % v_tiles) * 64;
    stage_rows(Bs, B + (size_t)c.start * ld + (size_t)g * Np + n0, ld, c.count, N - n0, nullptr, N % 4 == 0);
    stage_rows(xs, x + (size_t)c.start * ld + (size_t)h * V + v0, ld, c.count, V - v0, w, V % 4 == 0);
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;
    float acc[8][4] = {};
#pragma unroll 4
    for (int s = 0; s < c.count; ++s)
        outer(acc, ld4(Bs + s * kLd + ty * 8), ld4(Bs + s * kLd + ty * 8 + 4), ld4(xs + s * kLd + tx * 4));
    float* dst = states + ((size_t)c.slot * H + h) * N * V;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int n = n0 + ty * 8 + i, v = v0 + tx * 4;
        if (n >= N) break;
        if (V % 4 == 0) {
            if (v < V) *reinterpret_cast<float4*>(dst + (size_t)n * V + v) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (v + j < V) dst[(size_t)n * V + v + j] = acc[i][j];
        }
    }
}

// grid (requests, elements of the state / (256 * VEC)); states[slot] becomes the state before the chunk
template <int VEC>
__global__ void __launch_bounds__(256)
chunk_pass_kernel(float* __restrict__ states, const float* __restrict__ decays, float* __restrict__ state, long long state_floats,
                  const int* __restrict__ qo_indptr, const int* __restrict__ state_slot, int min_len, int H, int per_head) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    __shared__ int first_slot;
    const int b = blockIdx.x, len = qo_indptr[b + 1] - qo_indptr[b];
    if (len < min_len) return;
    if (threadIdx.x < 32) {  // the chunks of the requests before this one
        int sum = 0;
        for (int r = threadIdx.x; r < b; r += 32) {
            const int n = qo_indptr[r + 1] - qo_indptr[r];
            if (n >= min_len) sum += (n + kQ - 1) / kQ;
        }
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if (threadIdx.x == 0) first_slot = sum;
    }
    __syncthreads();
    const long long total = (long long)H * per_head, e = ((long long)blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    if (e >= total) return;
    const int h = (int)(e / per_head), chunks = (len + kQ - 1) / kQ;  // (VEC elements lie in one head)
    float* S_mem = state + (long long)state_slot[b] * state_floats + e;
    float* at = states + (size_t)first_slot * total + e;
    const float* dec = decays + (size_t)first_slot * H + h;
    float S[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) S[k] = S_mem[k];
    for (int c0 = 0; c0 < chunks; c0 += 4) {  // four chunks' loads are in flight together
        float add[4][VEC], d[4];
        const int cnt = min(4, chunks - c0);
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (u < cnt) {
                d[u] = dec[(size_t)(c0 + u) * H];
                if constexpr (VEC == 4) {
                    const float4 v = ld4(at + (size_t)(c0 + u) * total);
                    add[u][0] = v.x; add[u][1] = v.y; add[u][2] = v.z; add[u][3] = v.w;
                } else {
                    add[u][0] = at[(size_t)(c0 + u) * total];
                }
            }
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (u < cnt) {
                if constexpr (VEC == 4) *reinterpret_cast<float4*>(at + (size_t)(c0 + u) * total) = make_float4(S[0], S[1], S[2], S[3]);
                else at[(size_t)(c0 + u) * total] = S[0];
#pragma unroll
                for (int k = 0; k < VEC; ++k) S[k] = fmaf(d[u], S[k], add[u][k]);
            }
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) S_mem[k] = S[k];
}

// grid (chunk slots, heads, tiles of 64 of a head's features)
__global__ void __launch_bounds__(kThreads, 4)
chunk_outputs_kernel(const float* __restrict__ C, const float* __restrict__ B, const float* __restrict__ x, const float* __restrict__ step,
                     int ld, const float* __restrict__ a_log, const int* __restrict__ qo_indptr, int n_requests, int min_len,
                     const float* __restrict__ states, float* __restrict__ out, int ld_out, int H, int G, int N, int Np, int V) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    constexpr int kK = 32;  // rows of the state to a pass
    __shared__ __align__(16) float slices[3 * kK * kLd];  // C and B of the pass transposed [k][token], S_in [k][feature]; then x [token][feature]
    __shared__ __align__(16) float Mt[kQ * kLd];          // the weights of x, [s][t]
    __shared__ double L[kQ];
    __shared__ float dt[kQ];
    __shared__ Chunk chunk;
    static_assert(3 * kK >= kQ, "x takes the place of the slices");
    const int tid = threadIdx.x, h = blockIdx.y, g = h / (H / G), v0 = blockIdx.z * 64;
    if (tid < 32) {
        const Chunk c = find_chunk(blockIdx.x, qo_indptr, n_requests, min_len);
        if (tid == 0) chunk = c;
        if (c.count > 0) chunk_logs(step + h, ld, c.start, c.count, expf(a_log[h]), L, dt);
    }
    __syncthreads();
    const Chunk c = chunk;
    if (c.count == 0) return;
    const int ty = tid >> 4, tx = tid & 15;
    float *Ct = slices, *Bt = slices + kK * kLd, *Ss = slices + 2 * kK * kLd;
    const float* C0 = C + (size_t)c.start * ld + (size_t)g * Np;
    const float* B0 = B + (size_t)c.start * ld + (size_t)g * Np;
    const float* S0 = states + ((size_t)c.slot * H + h) * N * V;
    const bool vec = V % 4 == 0;
    float scores[8][4] = {}, y[8][4] = {};
    for (int k0 = 0; k0 < N; k0 += kK) {
        __syncthreads();  // the pass before has been read
        for (int i = tid; i < kQ * kK; i += kThreads) {
            const int t = i >> 5, k = i & 31;
            const bool in = t < c.count && k0 + k < N;
            Ct[k * kLd + t] = in ? C0[(size_t)t * ld + k0 + k] : 0.f;
            Bt[k * kLd + t] = in ? B0[(size_t)t * ld + k0 + k] : 0.f;
        }
        if (vec) {
            for (int i = tid; i < kK * 16; i += kThreads) {
                const int k = i >> 4, v = (i & 15) * 4;
                float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
                if (k0 + k < N && v0 + v < V) s = ld4(S0 + (size_t)(k0 + k) * V + v0 + v);
                *reinterpret_cast<float4*>(Ss + k * kLd + v) = s;
            }
        } else {
            for (int i = tid; i < kK * 64; i += kThreads) {
                const int k = i >> 6, v = i & 63;
                Ss[k * kLd + v] = k0 + k < N && v0 + v < V ? S0[(size_t)(k0 + k) * V + v0 + v] : 0.f;
            }
        }
        __syncthreads();
        const int k_end = min(kK, N - k0);
#pragma unroll 4
        for (int k = 0; k < k_end; ++k) {
            const float4 a0 = ld4(Ct + k * kLd + ty * 8), a1 = ld4(Ct + k * kLd + ty * 8 + 4);
            outer(scores, a0, a1, ld4(Bt + k * kLd + tx * 4));
            outer(y, a0, a1, ld4(Ss + k * kLd + tx * 4));
        }
    }
    // the weights of x: this thread's tokens t = 8 ty + i against s = 4 tx + j
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int s = tx * 4 + j;
        float m[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int t = ty * 8 + i;
            m[i] = s <= t ? scores[i][j] * (expf((float)(L[t] - L[s])) * dt[s]) : 0.f;
        }
        *reinterpret_cast<float4*>(Mt + s * kLd + ty * 8) = make_float4(m[0], m[1], m[2], m[3]);
        *reinterpret_cast<float4*>(Mt + s * kLd + ty * 8 + 4) = make_float4(m[4], m[5], m[6], m[7]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const float f = expf((float)L[ty * 8 + i]);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[i][j] *= f;
    }
    __syncthreads();  // the last pass has been read; the weights are complete
    stage_rows(slices, x + (size_t)c.start * ld + (size_t)h * V + v0, ld, c.count, V - v0, nullptr, vec);
    __syncthreads();
    const int s_end = min(c.count, ((ty | 1) + 1) * 8);  // no weight of this warp's tokens lies beyond
#pragma unroll 4
    for (int s = 0; s < s_end; ++s)
        outer(y, ld4(Mt + s * kLd + ty * 8), ld4(Mt + s * kLd + ty * 8 + 4), ld4(slices + s * kLd + tx * 4));
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = ty * 8 + i, v = v0 + tx * 4;
        if (t >= c.count) break;
        float* dst = out + (size_t)(c.start + t) * ld_out + (size_t)h * V + v;
        if (vec && ld_out % 4 == 0) {
            if (v < V) *reinterpret_cast<float4*>(dst) = make_float4(y[i][0], y[i][1], y[i][2], y[i][3]);
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (v + j < V) dst[j] = y[i][j];
        }
    }
}

}  // namespace

// C, B, x, step: the columns of the preparation's rows (row stride ld floats; groups of C and B Np apart, heads of x V, one step size
// per head); a_log [H]; state [slots, state_floats] with S [H, N, V] at the start of a row; states: scratch for `chunks` chunks of
// H * N * V floats, decays: H floats each, where `chunks` is at least the number of chunks of all requests of min_len tokens or more.
// Requests of fewer tokens are not touched.
NS_API int ns_ssm_chunked(const float* C, const float* B, const float* x, const float* step, int ld, const float* a_log, float* state,
                          long long state_floats, const int* qo_indptr, const int* state_slot, float* out, int ld_out, int n_requests,
                          int min_len, int chunks, float* states, float* decays, int H, int G, int N, int Np, int V, cudaStream_t stream) {
    if (n_requests <= 0 || chunks <= 0) return NS_OK;
    if (G < 1 || H % G || N < 1 || V < 1 || Np < N) NS_FAIL(NS_ERR_ARGUMENT, "ns_ssm_chunked: %d heads in %d groups, state %d (%d), features %d", H, G, N, Np, V);
    if (ld % 4 || Np % 4 || (((uintptr_t)C | (uintptr_t)B | (uintptr_t)x | (uintptr_t)states) % 16) || (V % 4 == 0 && (uintptr_t)out % 16))
        NS_FAIL(NS_ERR_ARGUMENT, "ns_ssm_chunked: rows must start on 16 bytes");
    const int n_tiles = (N + 63) / 64, v_tiles = (V + 63) / 64;
    if (H > 65535 || n_tiles * v_tiles > 65535) NS_FAIL(NS_ERR_UNSUPPORTED, "ns_ssm_chunked: %d heads, state of %d x %d exceed the grid", H, N, V);
    NS_LAUNCH(chunk_states_kernel, dim3(chunks, H, n_tiles * v_tiles), kThreads, 0, stream, B, x, step, ld, a_log, qo_indptr, n_requests, min_len,
              states, decays, H, G, N, Np, V);
    NS_CHECK_LAUNCH("ns_ssm_chunked");
    const long long total = (long long)H * N * V;
    const bool vec = (N * V) % 4 == 0 && state_floats % 4 == 0 && (uintptr_t)state % 16 == 0;
    const long long blocks = (total + 256 * (vec ? 4 : 1) - 1) / (256 * (vec ? 4 : 1));
    if (blocks > 65535) NS_FAIL(NS_ERR_UNSUPPORTED, "ns_ssm_chunked: a state of %lld floats exceeds the grid", total);
    if (vec)
        NS_LAUNCH((chunk_pass_kernel<4>), dim3(n_requests, (unsigned)blocks), 256, 0, stream, states, decays, state, state_floats, qo_indptr, state_slot,
                  min_len, H, N * V);
    else
        NS_LAUNCH((chunk_pass_kernel<1>), dim3(n_requests, (unsigned)blocks), 256, 0, stream, states, decays, state, state_floats, qo_indptr, state_slot,
                  min_len, H, N * V);
    NS_CHECK_LAUNCH("ns_ssm_chunked");
    NS_LAUNCH(chunk_outputs_kernel, dim3(chunks, H, v_tiles), kThreads, 0, stream, C, B, x, step, ld, a_log, qo_indptr, n_requests, min_len,
              states, out, ld_out, H, G, N, Np, V);
    NS_CHECK_LAUNCH("ns_ssm_chunked");
    return NS_OK;
}
