// Embedding gather, RMSNorm with the residual sum fused in, and the SwiGLU gate.
//
// The residual stream is float in every precision mode: the sum of branch outputs is kept
// in 32-bit and only the normalised activations that feed a matrix product are rounded to
// the compute type.
#include "common.cuh"

thread_local char ns_error_text[512] = "";
NS_API const char* ns_last_error() { return ns_error_text; }

int ns_pdl_enabled = 1, ns_pdl_skip_one = 0;

// The next kernel launch (on whatever stream) starts only when everything before it is complete.
NS_API int ns_full_launch_next() {
    ns_pdl_skip_one = 1;
    return NS_OK;
}
// 1 (default): kernels are launched so that they may overlap the tail of their predecessor
// (programmatic dependent launch); 0: plain stream order.
NS_API int ns_set_pdl(int enabled) {
    ns_pdl_enabled = enabled ? 1 : 0;
    return NS_OK;
}

// ---------------------------------------------------------------------------------------
// embedding: out[n, :] = float(table[ids[n], :]); a negative id (padding row) gives zeros
// ---------------------------------------------------------------------------------------
template <typename T>
__global__ void embed_kernel(const T* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out,
                             int hidden, int vocab) {
    ns_pdl_launch_dependents();  // the next kernel may be scheduled now; it waits for this one before it reads
    ns_pdl_wait();               // everything below sees the previous kernel's results
    const int n = blockIdx.x;
    const int id = ids[n];
    float* o = out + (size_t)n * hidden;
    if (id < 0 || id >= vocab) {
        for (int h = threadIdx.x; h < hidden; h += blockDim.x) o[h] = 0.f;
        return;
    }
    const T* row = table + (size_t)id * hidden;
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) o[h] = ns_ld(row, h);
}

NS_API int ns_embed(const void* table, const int* ids, float* out, int n_tokens, int hidden, int vocab, int dtype,
                    cudaStream_t stream) {
    if (n_tokens <= 0) return NS_OK;
    const int threads = hidden >= 1024 ? 256 : (hidden >= 256 ? 128 : 64);
    if (dtype == NS_F32)
        NS_LAUNCH((embed_kernel<float>), n_tokens, threads, 0, stream, (const float*)table, ids, out, hidden, vocab);
    else if (dtype == NS_BF16)
        NS_LAUNCH((embed_kernel<__nv_bfloat16>), n_tokens, threads, 0, stream, (const __nv_bfloat16*)table, ids, out, hidden, vocab);
    else
        NS_FAIL(NS_ERR_ARGUMENT, "ns_embed: unknown dtype %d", dtype);
    NS_CHECK_LAUNCH("ns_embed");
    return NS_OK;
}

// ---------------------------------------------------------------------------------------
// token ids that an earlier step sampled and the host has not seen yet: ids[dst_rows[i]] = src[src_rows[i]]
// ---------------------------------------------------------------------------------------
__global__ void take_ids_kernel(int* __restrict__ ids, const int* __restrict__ dst_rows, const int* __restrict__ src,
                                const int* __restrict__ src_rows, int n) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) ids[dst_rows[i]] = src[src_rows[i]];
}

NS_API int ns_take_ids(int* ids, const int* dst_rows, const int* src, const int* src_rows, int n, cudaStream_t stream) {
    if (n <= 0) return NS_OK;
    NS_LAUNCH(take_ids_kernel, (n + 127) / 128, 128, 0, stream, ids, dst_rows, src, src_rows, n);
    NS_CHECK_LAUNCH("ns_take_ids");
    return NS_OK;
}

// ---------------------------------------------------------------------------------------
// RMSNorm over the residual stream, with the pending branch output added first:
//   r = resid[row] + branch[row]        (branch may be absent)
//   resid[row] = r                      (when write_resid)
//   out[j]  = r * rsqrt(mean(r^2) + eps) * gain          all in float, rounded once to T
// `rows` (optional) selects the input rows: output row j reads input row rows[j]; then the
// residual is not written back (used for the final norm at the wanted positions).
// ---------------------------------------------------------------------------------------
template <typename T, int THREADS, int PER_THREAD>
__global__ void __launch_bounds__(THREADS)
add_rmsnorm_kernel(float* __restrict__ resid, const T* __restrict__ branch, const float* __restrict__ gain,
                   T* __restrict__ out, const int* __restrict__ rows, int hidden, float eps, int write_resid) {
    ns_pdl_launch_dependents();  // the next kernel may be scheduled now; it waits for this one before it reads
    ns_pdl_wait();               // everything below sees the previous kernel's results
    __shared__ float scratch[32];
    const int j = blockIdx.x;
    const int row = rows ? rows[j] : j;
    float* r = resid + (size_t)row * hidden;
    const T* b = branch ? branch + (size_t)row * hidden : nullptr;
    T* o = out + (size_t)j * hidden;

    float v[PER_THREAD];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < PER_THREAD; ++i) {
        const int h = threadIdx.x + i * THREADS;
        float x = 0.f;
        if (h < hidden) {
            x = r[h];
            if (b) x += ns_ld(b, h);
            if (write_resid && b) r[h] = x;
        }
        v[i] = x;
        ss += x * x;
    }
    // elements beyond PER_THREAD * THREADS (very wide rows) are handled from memory
    for (int h = threadIdx.x + PER_THREAD * THREADS; h < hidden; h += THREADS) {
        float x = r[h];
        if (b) x += ns_ld(b, h);
        if (write_resid && b) r[h] = x;
        ss += x * x;
    }
    const float total = ns_block_sum(ss, scratch);
    const float inv = rsqrtf(total / (float)hidden + eps);
#pragma unroll
    for (int i = 0; i < PER_THREAD; ++i) {
        const int h = threadIdx.x + i * THREADS;
        if (h < hidden) ns_st(o, h, v[i] * inv * gain[h]);
    }
    for (int h = threadIdx.x + PER_THREAD * THREADS; h < hidden; h += THREADS) {
        float x = r[h];
        if (b && !write_resid) x += ns_ld(b, h);
        ns_st(o, h, x * inv * gain[h]);
    }
}

// Vector variant for widths that are a multiple of 8 with 16-byte aligned rows: every thread owns
// CHUNKS groups of 8 consecutive elements, read and written with 16-byte accesses.
// CENTERED: the layer norm without bias instead - the mean is taken off first and the variance is the mean of the
// squared deviations (a second sum over the values, which are in registers).
template <typename T, int THREADS, int CHUNKS, bool CENTERED = false>
__global__ void __launch_bounds__(THREADS)
add_rmsnorm_vec_kernel(float* __restrict__ resid, const T* __restrict__ branch, const float* __restrict__ gain,
                       T* __restrict__ out, const int* __restrict__ rows, int hidden, float eps, int write_resid) {
    ns_pdl_launch_dependents();  // the next kernel may be scheduled now; it waits for this one before it reads
    __shared__ float scratch[32];
    // the gain is a weight: it is fetched while the previous kernel is still running
    float g[CHUNKS][8];
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int h = (threadIdx.x + c * THREADS) * 8;
        if (h < hidden) ld8(gain + h, g[c]);
    }
    ns_pdl_wait();               // everything below sees the previous kernel's results
    const int j = blockIdx.x;
    const int row = rows ? rows[j] : j;
    float* r = resid + (size_t)row * hidden;
    const T* b = branch ? branch + (size_t)row * hidden : nullptr;
    T* o = out + (size_t)j * hidden;
    float v[CHUNKS][8];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int h = (threadIdx.x + c * THREADS) * 8;
        if (h < hidden) {
            ld8(r + h, v[c]);
            if (b) {
                float t[8];
                ld8(b + h, t);
#pragma unroll
                for (int i = 0; i < 8; ++i) v[c][i] += t[i];
                if (write_resid) st8(r + h, v[c]);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) ss += CENTERED ? v[c][i] : v[c][i] * v[c][i];
        }
    }
    if (CENTERED) {
        const float mean = ns_block_sum(ss, scratch) / (float)hidden;
        ss = 0.f;
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int h = (threadIdx.x + c * THREADS) * 8;
            if (h < hidden) {
#pragma unroll
                for (int i = 0; i < 8; ++i) { v[c][i] -= mean; ss += v[c][i] * v[c][i]; }
            }
        }
    }
    const float inv = rsqrtf(ns_block_sum(ss, scratch) / (float)hidden + eps);
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int h = (threadIdx.x + c * THREADS) * 8;
        if (h < hidden) {
            float y[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) y[i] = v[c][i] * inv * g[c][i];
            st8(o + h, y);
        }
    }
}

template <typename T>
static int launch_add_rmsnorm(float* resid, const void* branch, const float* gain, void* out, const int* rows,
                              int n_rows, int hidden, float eps, int write_resid, cudaStream_t stream) {
    const T* b = (const T*)branch;
    T* o = (T*)out;
    const bool aligned = hidden % 8 == 0 && (((uintptr_t)resid | (uintptr_t)branch | (uintptr_t)gain | (uintptr_t)out) % 16 == 0);
    if (aligned && hidden >= 1024 && hidden <= 16384) {
        // the sum of squares runs over the same elements in another grouping than the scalar kernel;
        // which kernel runs depends on the width and alignment only, never on the batch
        if (hidden <= 2048)
            NS_LAUNCH((add_rmsnorm_vec_kernel<T, 128, 2>), n_rows, 128, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
        else if (hidden <= 4096)
            NS_LAUNCH((add_rmsnorm_vec_kernel<T, 256, 2>), n_rows, 256, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
        else if (hidden <= 8192)
            NS_LAUNCH((add_rmsnorm_vec_kernel<T, 512, 2>), n_rows, 512, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
        else
            NS_LAUNCH((add_rmsnorm_vec_kernel<T, 1024, 2>), n_rows, 1024, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
        NS_CHECK_LAUNCH("ns_add_rmsnorm");
        return NS_OK;
    }
    if (hidden <= 256)
        NS_LAUNCH((add_rmsnorm_kernel<T, 64, 4>), n_rows, 64, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
    else if (hidden <= 1024)
        NS_LAUNCH((add_rmsnorm_kernel<T, 128, 8>), n_rows, 128, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
    else if (hidden <= 4096)
        NS_LAUNCH((add_rmsnorm_kernel<T, 512, 8>), n_rows, 512, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
    else
        NS_LAUNCH((add_rmsnorm_kernel<T, 1024, 8>), n_rows, 1024, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
    NS_CHECK_LAUNCH("ns_add_rmsnorm");
    return NS_OK;
}

NS_API int ns_add_rmsnorm(float* resid, const void* branch, const float* gain, void* out, const int* rows, int n_rows,
                          int hidden, float eps, int write_resid, int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return NS_OK;
    if (hidden <= 0) NS_FAIL(NS_ERR_ARGUMENT, "ns_add_rmsnorm: hidden=%d", hidden);
    if (rows && write_resid) NS_FAIL(NS_ERR_ARGUMENT, "ns_add_rmsnorm: a row selection cannot write the residual back");
    if (dtype == NS_F32)
        return launch_add_rmsnorm<float>(resid, branch, gain, out, rows, n_rows, hidden, eps, write_resid, stream);
    if (dtype == NS_BF16)
        return launch_add_rmsnorm<__nv_bfloat16>(resid, branch, gain, out, rows, n_rows, hidden, eps, write_resid, stream);
    NS_FAIL(NS_ERR_ARGUMENT, "ns_add_rmsnorm: unknown dtype %d", dtype);
}

// ---------------------------------------------------------------------------------------
// residual sum alone: resid[row] += branch[row]  (used when no norm follows)
// ---------------------------------------------------------------------------------------
template <typename T>
__global__ void residual_add_kernel(float* __restrict__ resid, const T* __restrict__ branch, size_t n) {
    ns_pdl_launch_dependents();  // the next kernel may be scheduled now; it waits for this one before it reads
    ns_pdl_wait();               // everything below sees the previous kernel's results
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) resid[i] += ns_ld(branch, i);
}

NS_API int ns_residual_add(float* resid, const void* branch, int n_rows, int hidden, int dtype, cudaStream_t stream) {
    const size_t n = (size_t)n_rows * hidden;
    if (n == 0) return NS_OK;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (dtype == NS_F32)
        NS_LAUNCH((residual_add_kernel<float>), blocks, 256, 0, stream, resid, (const float*)branch, n);
    else if (dtype == NS_BF16)
        NS_LAUNCH((residual_add_kernel<__nv_bfloat16>), blocks, 256, 0, stream, resid, (const __nv_bfloat16*)branch, n);
    else
        NS_FAIL(NS_ERR_ARGUMENT, "ns_residual_add: unknown dtype %d", dtype);
    NS_CHECK_LAUNCH("ns_residual_add");
    return NS_OK;
}

// ---------------------------------------------------------------------------------------
// SwiGLU gate on the packed [gate | up] projection, and gated units of the same form (NsGate, common.cuh):
//   out[n, j] = silu(gu[n, j]) * gu[n, inter + j],  silu(a) = a / (1 + exp(-a)),  in float
// ---------------------------------------------------------------------------------------
// The float kernels use the accurate exponential and division; the bfloat16 ones the hardware approximations.

template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gu, long long ldg, T* __restrict__ out, long long ldo, int inter, int block, size_t total, NsGate act) {
    ns_pdl_launch_dependents();  // the next kernel may be scheduled now; it waits for this one before it reads
    ns_pdl_wait();               // everything below sees the previous kernel's results
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t n = i / inter;
    const int j = (int)(i - n * inter);
    // block == 0: [gate | up]; otherwise gate and up alternate in runs of `block` features
    const size_t gi = block ? (size_t)(j / block) * 2 * block + j % block : (size_t)j;
    const float g = ns_ld(gu, n * ldg + gi);
    const float u = ns_ld(gu, n * ldg + gi + (block ? block : inter));
    ns_st(out, n * ldo + j, ns_gate_mul<sizeof(T) == 2>(act, g, u));
}

template <typename T>
__global__ void swiglu_vec_kernel(const T* __restrict__ gu, long long ldg, T* __restrict__ out, long long ldo, int inter, int block, size_t total8, NsGate act) {
    ns_pdl_launch_dependents();  // the next kernel may be scheduled now; it waits for this one before it reads
    ns_pdl_wait();               // everything below sees the previous kernel's results
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total8) return;
    const int per_row = inter / 8;
    const size_t n = i / per_row;
    const int j = (int)(i - n * per_row) * 8;
    float g[8], u[8], y[8];
    const size_t gi = block ? (size_t)(j / block) * 2 * block + j % block : (size_t)j;  // block is a multiple of 8
    ld8(gu + n * ldg + gi, g);
    ld8(gu + n * ldg + gi + (block ? block : inter), u);
#pragma unroll
    for (int k = 0; k < 8; ++k) y[k] = ns_gate_mul<sizeof(T) == 2>(act, g[k], u[k]);
    st8(out + n * ldo + j, y);
}

// out[n, j] = silu(g) * u with g, u = gate_up[n, j], gate_up[n, inter + j] (block == 0), or, when gate and up
// alternate in runs of `block` features (a multiple of 8 that divides inter), gate_up[n, (j / block) * 2 * block +
// j % block] and the element `block` further.  Rows of gate_up start ldg elements apart, rows of out ldo.  alpha, shift, limit: NsGate.
NS_API int ns_gate_mul_rows(const void* gate_up, long long ldg, void* out, long long ldo, int n_rows, int inter, int block, float alpha, float shift,
                            float limit, int dtype, cudaStream_t stream) {
    const NsGate act{alpha, shift, limit};
    const size_t total = (size_t)n_rows * inter;
    if (total == 0) return NS_OK;
    if (block < 0 || (block && (block % 8 || inter % block)))
        NS_FAIL(NS_ERR_ARGUMENT, "ns_swiglu: block=%d must be 0 or a multiple of 8 that divides %d", block, inter);
    if (dtype != NS_F32 && dtype != NS_BF16) NS_FAIL(NS_ERR_ARGUMENT, "ns_swiglu: unknown dtype %d", dtype);
    const size_t esz = dtype == NS_F32 ? 4 : 2;
    if (inter % 8 == 0 && (((uintptr_t)gate_up | (uintptr_t)out) % 16 == 0) && (ldg * esz) % 16 == 0 && (ldo * esz) % 16 == 0) {
        const size_t total8 = total / 8;
        const unsigned vblocks = (unsigned)((total8 + 255) / 256);
        if (dtype == NS_F32)
            NS_LAUNCH((swiglu_vec_kernel<float>), vblocks, 256, 0, stream, (const float*)gate_up, ldg, (float*)out, ldo, inter, block, total8, act);
        else
            NS_LAUNCH((swiglu_vec_kernel<__nv_bfloat16>), vblocks, 256, 0, stream, (const __nv_bfloat16*)gate_up, ldg, (__nv_bfloat16*)out, ldo, inter, block, total8, act);
    } else {
        const unsigned blocks = (unsigned)((total + 255) / 256);
        if (dtype == NS_F32)
            NS_LAUNCH((swiglu_kernel<float>), blocks, 256, 0, stream, (const float*)gate_up, ldg, (float*)out, ldo, inter, block, total, act);
        else
            NS_LAUNCH((swiglu_kernel<__nv_bfloat16>), blocks, 256, 0, stream, (const __nv_bfloat16*)gate_up, ldg, (__nv_bfloat16*)out, ldo, inter, block, total, act);
    }
    NS_CHECK_LAUNCH("ns_swiglu");
    return NS_OK;
}

// silu(gate) * up
NS_API int ns_swiglu_rows(const void* gate_up, long long ldg, void* out, long long ldo, int n_rows, int inter, int block, int dtype,
                          cudaStream_t stream) {
    return ns_gate_mul_rows(gate_up, ldg, out, ldo, n_rows, inter, block, 1.f, 0.f, 0.f, dtype, stream);
}

// the same over contiguous rows
NS_API int ns_swiglu(const void* gate_up, void* out, int n_rows, int inter, int block, int dtype, cudaStream_t stream) {
    return ns_swiglu_rows(gate_up, 2ll * inter, out, inter, n_rows, inter, block, dtype, stream);
}

// ---------------------------------------------------------------------------------------
// Layer norm without a bias over the residual stream, with the pending branch output added first:
//   r = resid[row] + branch[row];  mean = sum(r) / H;  var = sum((r - mean)^2) / H  (two passes over the
//   row, which lies in shared memory);  out = (r - mean) * rsqrt(var + eps) * gain,  all in float.
// `rows` and `write_resid` as in add_rmsnorm.
// ---------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
add_layernorm_kernel(float* __restrict__ resid, const T* __restrict__ branch, const float* __restrict__ gain,
                     T* __restrict__ out, const int* __restrict__ rows, int hidden, float eps, int write_resid) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    extern __shared__ float ln_row[];
    __shared__ float scratch[32];
    const int j = blockIdx.x;
    const int row = rows ? rows[j] : j;
    float* r = resid + (size_t)row * hidden;
    const T* b = branch ? branch + (size_t)row * hidden : nullptr;
    T* o = out + (size_t)j * hidden;
    float s = 0.f;
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
        float x = r[h];
        if (b) {
            x += ns_ld(b, h);
            if (write_resid) r[h] = x;
        }
        ln_row[h] = x;
        s += x;
    }
    const float mean = ns_block_sum(s, scratch) / (float)hidden;
    float ss = 0.f;
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
        const float dlt = ln_row[h] - mean;
        ss += dlt * dlt;
    }
    const float inv = rsqrtf(ns_block_sum(ss, scratch) / (float)hidden + eps);
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) ns_st(o, h, (ln_row[h] - mean) * inv * gain[h]);
}

template <typename T>
static int launch_add_layernorm(float* resid, const void* branch, const float* gain, void* out, const int* rows, int n_rows,
                                int hidden, float eps, int write_resid, cudaStream_t stream) {
    const size_t smem = (size_t)hidden * sizeof(float);
    if (smem > 200 * 1024) NS_FAIL(NS_ERR_UNSUPPORTED, "ns_add_layernorm: a row of %d floats does not fit shared memory", hidden);
    if (smem > 48 * 1024) {
        static int raised = 0;  // per instantiation
        if (raised < (int)smem) {
            NS_CUDA(cudaFuncSetAttribute(add_layernorm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
            raised = 200 * 1024;
        }
    }
    const bool aligned = hidden % 8 == 0 && (((uintptr_t)resid | (uintptr_t)branch | (uintptr_t)gain | (uintptr_t)out) % 16 == 0);
    if (aligned && hidden >= 1024 && hidden <= 16384) {  // which kernel runs depends on the width and alignment only, never on the batch
        const T* b = (const T*)branch;
        T* o = (T*)out;
        if (hidden <= 2048)
            NS_LAUNCH((add_rmsnorm_vec_kernel<T, 128, 2, true>), n_rows, 128, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
        else if (hidden <= 4096)
            NS_LAUNCH((add_rmsnorm_vec_kernel<T, 256, 2, true>), n_rows, 256, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
        else if (hidden <= 8192)
            NS_LAUNCH((add_rmsnorm_vec_kernel<T, 512, 2, true>), n_rows, 512, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
        else
            NS_LAUNCH((add_rmsnorm_vec_kernel<T, 1024, 2, true>), n_rows, 1024, 0, stream, resid, b, gain, o, rows, hidden, eps, write_resid);
        NS_CHECK_LAUNCH("ns_add_layernorm");
        return NS_OK;
    }
    NS_LAUNCH((add_layernorm_kernel<T>), n_rows, 256, smem, stream, resid, (const T*)branch, gain, (T*)out, rows, hidden, eps,
              write_resid);
    NS_CHECK_LAUNCH("ns_add_layernorm");
    return NS_OK;
}

NS_API int ns_add_layernorm(float* resid, const void* branch, const float* gain, void* out, const int* rows, int n_rows,
                            int hidden, float eps, int write_resid, int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return NS_OK;
    if (hidden <= 0) NS_FAIL(NS_ERR_ARGUMENT, "ns_add_layernorm: hidden=%d", hidden);
    if (rows && write_resid) NS_FAIL(NS_ERR_ARGUMENT, "ns_add_layernorm: a row selection cannot write the residual back");
    if (dtype == NS_F32) return launch_add_layernorm<float>(resid, branch, gain, out, rows, n_rows, hidden, eps, write_resid, stream);
    if (dtype == NS_BF16)
        return launch_add_layernorm<__nv_bfloat16>(resid, branch, gain, out, rows, n_rows, hidden, eps, write_resid, stream);
    NS_FAIL(NS_ERR_ARGUMENT, "ns_add_layernorm: unknown dtype %d", dtype);
}

// ---------------------------------------------------------------------------------------
// logits in place: x = x * scale, then x = cap * tanh(x / cap) when cap > 0
// ---------------------------------------------------------------------------------------
__global__ void scale_softcap_kernel(float* __restrict__ x, int cols, long long stride, float scale, float cap, size_t total) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    float* p = x + (i / cols) * stride + (i % cols);
    float v = *p * scale;
    if (cap > 0.f) v = cap * tanhf(v / cap);
    *p = v;
}

NS_API int ns_scale_softcap(float* x, int n_rows, int cols, long long stride, float scale, float cap, cudaStream_t stream) {
    const size_t total = (size_t)n_rows * cols;
    if (total == 0) return NS_OK;
    NS_LAUNCH(scale_softcap_kernel, (unsigned)((total + 255) / 256), 256, 0, stream, x, cols, stride, scale, cap, total);
    NS_CHECK_LAUNCH("ns_scale_softcap");
    return NS_OK;
}

// ---------------------------------------------------------------------------------------
// The norm that takes no statistics (a "dynamic tanh"): out = tanh(alpha * x) * gain + bias, with one scalar alpha.
// Fused with the residual sum like the norms above: x = resid (+ a) (+ b), the two optional branches in the output's
// type; the sum is written back to the float stream unless rows are selected.  Everything is elementwise, so the grid is
// (pieces of a row, rows) and a thread takes eight neighbouring features where the rows start on 16 bytes.
// `alpha` is read from device memory (it is a weight).
// ---------------------------------------------------------------------------------------
namespace {

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
add_dyt_kernel(float* __restrict__ resid, const T* __restrict__ a, const T* __restrict__ b, const float* __restrict__ gain,
               const float* __restrict__ bias, const float* __restrict__ alpha, T* __restrict__ out,
               const int* __restrict__ rows, int hidden, int write_resid) {
    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const int r = blockIdx.y;
    const size_t src = (size_t)(rows ? rows[r] : r) * hidden;
    const int e0 = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (e0 >= hidden) return;
    const float al = *alpha;
    T* o = out + (size_t)r * hidden + e0;
    if constexpr (VEC == 8) {  // eight neighbouring features with 16-byte accesses
        float x[8], t[8], g[8];
        ld8(resid + src + e0, x);
        if (a) {
            ld8(a + src + e0, t);
#pragma unroll
            for (int i = 0; i < 8; ++i) x[i] += t[i];
        }
        if (b) {
            ld8(b + src + e0, t);
#pragma unroll
            for (int i = 0; i < 8; ++i) x[i] += t[i];
        }
        if (write_resid && (a || b)) st8(resid + src + e0, x);
        ld8(gain + e0, g);
        if (bias) ld8(bias + e0, t);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = fmaf(ns_tanh<sizeof(T) == 2>(al * x[i]), g[i], bias ? t[i] : 0.f);
        st8(o, x);
    } else {
        float x = resid[src + e0];
        if (a) x += ns_ld(a, src + e0);
        if (b) x += ns_ld(b, src + e0);
        if (write_resid && (a || b)) resid[src + e0] = x;
        ns_st(o, 0, fmaf(ns_tanh<sizeof(T) == 2>(al * x), gain[e0], bias ? bias[e0] : 0.f));
    }
}

template <typename T>
int launch_add_dyt(float* resid, const void* a, const void* b, const float* gain, const float* bias, const float* alpha, void* out,
                   const int* rows, int n_rows, int hidden, int write_resid, cudaStream_t stream) {
    const bool vec = hidden % 8 == 0 && (((uintptr_t)resid | (uintptr_t)a | (uintptr_t)b | (uintptr_t)gain | (uintptr_t)bias | (uintptr_t)out) % 16 == 0);
    const int per = vec ? 8 : 1;
    const int threads = hidden / per >= 256 ? 256 : hidden / per > 64 ? 128 : 64;
    const unsigned bx = (unsigned)((hidden + threads * per - 1) / (threads * per));
    // the grid's y extent holds 65,535 rows: longer steps go in slices
    for (int r0 = 0; r0 < n_rows; r0 += 65535) {
        const int nr = n_rows - r0 < 65535 ? n_rows - r0 : 65535;
        float* rs = rows ? resid : resid + (size_t)r0 * hidden;
        const T* as = a && !rows ? (const T*)a + (size_t)r0 * hidden : (const T*)a;
        const T* bs = b && !rows ? (const T*)b + (size_t)r0 * hidden : (const T*)b;
        T* os = (T*)out + (size_t)r0 * hidden;
        const int* rw = rows ? rows + r0 : nullptr;
        if (vec) NS_LAUNCH((add_dyt_kernel<T, 8>), dim3(bx, nr), threads, 0, stream, rs, as, bs, gain, bias, alpha, os, rw, hidden, write_resid);
        else NS_LAUNCH((add_dyt_kernel<T, 1>), dim3(bx, nr), threads, 0, stream, rs, as, bs, gain, bias, alpha, os, rw, hidden, write_resid);
    }
    NS_CHECK_LAUNCH("ns_add_dyt");
    return NS_OK;
}

}  // namespace

NS_API int ns_add_dyt(float* resid, const void* a, const void* b, const float* gain, const float* bias, const float* alpha, void* out,
                      const int* rows, int n_rows, int hidden, int write_resid, int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return NS_OK;
    if (hidden <= 0 || !gain || !alpha) NS_FAIL(NS_ERR_ARGUMENT, "ns_add_dyt: hidden=%d, a gain and alpha are needed", hidden);
    if (rows && write_resid) NS_FAIL(NS_ERR_ARGUMENT, "ns_add_dyt: a row selection cannot write the residual back");
    if (dtype == NS_F32) return launch_add_dyt<float>(resid, a, b, gain, bias, alpha, out, rows, n_rows, hidden, write_resid, stream);
    if (dtype == NS_BF16) return launch_add_dyt<__nv_bfloat16>(resid, a, b, gain, bias, alpha, out, rows, n_rows, hidden, write_resid, stream);
    NS_FAIL(NS_ERR_ARGUMENT, "ns_add_dyt: unknown dtype %d", dtype);
}

// ---------------------------------------------------------------------------------------
// The same norm on what a sublayer returns, joined to the stream, and the next sublayer's norm after it, in one pass:
//   y = a + b + sum_k weights[row, k] * ys[row_of[row, k]]      each optional; the last term is a routed sum (see moe.cu)
//   x = resid + tanh(post.alpha y) post.gain + post.bias        written back unless rows are selected
//   out = tanh(alpha x) gain + bias                              skipped without `out`
// All in float; y is never rounded.  One thread takes eight neighbouring features where the rows start on 16 bytes.
// ---------------------------------------------------------------------------------------
namespace {

struct TanhNorm { const float *gain, *bias, *alpha; };

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
dyt_join_kernel(float* __restrict__ resid, const T* __restrict__ a, const T* __restrict__ b, const T* __restrict__ ys,
                const int* __restrict__ row_of, const float* __restrict__ weights, int top, const TanhNorm post, const TanhNorm next,
                T* __restrict__ out, const int* __restrict__ rows, int hidden, int write_resid) {
    ns_pdl_launch_dependents();
    const int e0 = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    ns_pdl_wait();
    if (e0 >= hidden) return;
    const int r = blockIdx.x;
    const size_t row = rows ? rows[r] : r, src = row * hidden + e0;
    float y[VEC], t[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) y[i] = 0.f;
    auto load = [&](const auto* p, float (&v)[VEC]) {
        if constexpr (VEC == 8) ld8(p, v);
        else v[0] = ns_ld(p, 0);
    };
    auto store = [&](auto* p, const float (&v)[VEC]) {
        if constexpr (VEC == 8) st8(p, v);
        else ns_st(p, 0, v[0]);
    };
    if (ys) {
        for (int k = 0; k < top; ++k) {
            const int at = row_of[row * top + k];
            const float w = weights[row * top + k];
            load(ys + (size_t)at * hidden + e0, t);
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] = fmaf(w, t[i], y[i]);
        }
    }
    if (a) {
        load(a + src, t);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] += t[i];
    }
    if (b) {
        load(b + src, t);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] += t[i];
    }
    auto norm = [&](const TanhNorm& n, float (&v)[VEC]) {
        float g[VEC];
        const float al = *n.alpha;
        load(n.gain + e0, g);
        if (n.bias) load(n.bias + e0, t);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = fmaf(ns_tanh<sizeof(T) == 2>(al * v[i]), g[i], n.bias ? t[i] : 0.f);
    };
    norm(post, y);
    load(resid + src, t);
#pragma unroll
    for (int i = 0; i < VEC; ++i) y[i] += t[i];
    if (write_resid) store(resid + src, y);
    if (!out) return;
    norm(next, y);
    store(out + (size_t)r * hidden + e0, y);
}

template <typename T>
int launch_dyt_join(float* resid, const void* a, const void* b, const void* ys, const int* row_of, const float* weights, int top,
                    const TanhNorm& post, const TanhNorm& next, void* out, const int* rows, int n_rows, int hidden, int write_resid,
                    cudaStream_t stream) {
    const uintptr_t all = (uintptr_t)resid | (uintptr_t)a | (uintptr_t)b | (uintptr_t)ys | (uintptr_t)post.gain | (uintptr_t)post.bias |
                          (uintptr_t)next.gain | (uintptr_t)next.bias | (uintptr_t)out;
    const bool vec = hidden % 8 == 0 && all % 16 == 0;
    const int per = vec ? 8 : 1;
    const int threads = hidden / per >= 256 ? 256 : hidden / per > 64 ? 128 : 64;
    const unsigned bx = (unsigned)((hidden + threads * per - 1) / (threads * per));
    if (vec)
        NS_LAUNCH((dyt_join_kernel<T, 8>), dim3(n_rows, bx), threads, 0, stream, resid, (const T*)a, (const T*)b, (const T*)ys, row_of, weights,
                  top, post, next, (T*)out, rows, hidden, write_resid);
    else
        NS_LAUNCH((dyt_join_kernel<T, 1>), dim3(n_rows, bx), threads, 0, stream, resid, (const T*)a, (const T*)b, (const T*)ys, row_of, weights,
                  top, post, next, (T*)out, rows, hidden, write_resid);
    NS_CHECK_LAUNCH("ns_dyt_join");
    return NS_OK;
}

}  // namespace

// a, b [n, hidden] and ys [pairs, hidden] in the compute type (row_of, weights [n, top] with ys; every row_of entry >= 0); out may be null.
NS_API int ns_dyt_join(float* resid, const void* a, const void* b, const void* ys, const int* row_of, const float* weights, int top,
                       const float* post_gain, const float* post_bias, const float* post_alpha, const float* gain, const float* bias,
                       const float* alpha, void* out, const int* rows, int n_rows, int hidden, int write_resid, int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return NS_OK;
    if (hidden <= 0 || !post_gain || !post_alpha || (out && (!gain || !alpha))) NS_FAIL(NS_ERR_ARGUMENT, "ns_dyt_join: hidden=%d, gains and alphas are needed", hidden);
    if (ys && (!row_of || !weights || top < 1)) NS_FAIL(NS_ERR_ARGUMENT, "ns_dyt_join: a routed sum needs its rows and weights");
    if (rows && write_resid) NS_FAIL(NS_ERR_ARGUMENT, "ns_dyt_join: a row selection cannot write the stream back");
    const TanhNorm post{post_gain, post_bias, post_alpha}, next{gain, bias, alpha};
    if (dtype == NS_F32) return launch_dyt_join<float>(resid, a, b, ys, row_of, weights, top, post, next, out, rows, n_rows, hidden, write_resid, stream);
    if (dtype == NS_BF16) return launch_dyt_join<__nv_bfloat16>(resid, a, b, ys, row_of, weights, top, post, next, out, rows, n_rows, hidden, write_resid, stream);
    NS_FAIL(NS_ERR_ARGUMENT, "ns_dyt_join: unknown dtype %d", dtype);
}
