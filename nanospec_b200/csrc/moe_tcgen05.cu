// Routed experts on the 5th-generation tensor cores, without a host round trip.
//
// ns_moe_plan has laid the (token, choice) pairs out so that every expert's pairs are neighbours and ns_moe_gather has brought
// their rows of x into that order: expert e owns rows offsets[e] .. offsets[e + 1] of xs, read on the device.  Two products,
// one kernel: the experts' packed gate/up projection (runs of 64 gate features and the 64 matching up features alternate, so a
// tile of 128 weight rows holds both halves of 64 outputs) with silu(gate) * up, or another unit of that form (NsGate), in the
// epilogue, and the down projection.
//
// The layout of a product is gemm_tcgen05.cu's: 128 weight rows are the M side of tcgen05.mma, BN rows of xs its N side; one lane
// of warp 0 loads tiles of 64 along k with TMA (128-byte swizzle) into a ring of stages, one lane of warp 1 issues the products
// into TMEM, warps 2-5 read the accumulator into shared memory (the ring is free by then), and the whole block writes rows of
// 16-byte pieces.  blockIdx.y counts (expert, BN rows) tiles: a warp finds which one from the offsets; the grid holds the most
// tiles that the step's pairs can make, and blocks beyond the tiles there are leave.  A tile's last rows may belong to the next
// expert: they are multiplied and not stored.
#include "tcgen05_utils.cuh"

namespace {

constexpr int BM = 128, BK = 64, UMMA_K = 16, kThreads = 192;
constexpr int kPadM = BM + 4;  // floats of a staged row

enum GroupedError { kErrProducerWait = 41, kErrMmaWait = 42, kErrEpilogueWait = 43, kErrDrainWait = 44 };

template <int BN>
struct Cfg {
    static constexpr int kStages = BN == 256 ? 4 : BN == 128 ? 3 : 5;
    static constexpr int kMinBlocks = BN == 256 ? 1 : 2;
    static constexpr int kABytes = BM * BK * 2, kBBytes = BN * BK * 2, kStageBytes = kABytes + kBBytes;
    static constexpr size_t kSmemBytes = (size_t)kStages * kStageBytes + 1024 /* alignment slack */ + 128 /* barriers */;
    static_assert(BN * kPadM * 4 <= kStages * kStageBytes, "the accumulator is staged where the ring was");
};

template <int BN>
__global__ void __launch_bounds__(kThreads, Cfg<BN>::kMinBlocks)
moe_grouped_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x,
                      __nv_bfloat16* __restrict__ out, long long ldo, const int* __restrict__ offsets, int E, int rows_w, int k_blocks,
                      int gated, NsGate act, int* __restrict__ error_flag) {
    using C = Cfg<BN>;
    extern __shared__ unsigned char smem_dyn[];
    const uint32_t base = (smem_u32(smem_dyn) + 1023u) & ~1023u;
    const uint32_t bar_base = base + C::kStages * C::kStageBytes;
    auto full_bar = [&](int s) { return bar_base + 8u * s; };
    auto empty_bar = [&](int s) { return bar_base + 8u * (C::kStages + s); };
    const uint32_t accum_bar = bar_base + 8u * (2 * C::kStages);
    const uint32_t holder = accum_bar + 8u;
    __shared__ int failed, tile_expert, tile_row, tile_rows;
    float* stage_f32 = reinterpret_cast<float*>(smem_dyn + (base - smem_u32(smem_dyn)));

    ns_pdl_launch_dependents();
    ns_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n0 = blockIdx.x * BM;
    if (warp == 0) {  // which expert's rows this block takes
        int before = 0, found = -1, row = 0, count = 0;
        for (int e0 = 0; e0 < E && found < 0; e0 += 32) {
            const int e = e0 + lane;
            const int lo = e < E ? offsets[e] : 0, cnt = e < E ? offsets[e + 1] - lo : 0;
            const int tiles = (cnt + BN - 1) / BN;
            int sum = tiles;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += v;
            }
            const int first = before + sum - tiles;
            const bool mine = (int)blockIdx.y >= first && (int)blockIdx.y < first + tiles;
            const unsigned who = __ballot_sync(0xffffffffu, mine);
            if (who) {
                const int src = __ffs(who) - 1;
                const int t0 = ((int)blockIdx.y - first) * BN;
                found = __shfl_sync(0xffffffffu, e, src);
                row = __shfl_sync(0xffffffffu, lo + t0, src);
                count = __shfl_sync(0xffffffffu, min(BN, cnt - t0), src);
            }
            before += __shfl_sync(0xffffffffu, sum, 31);
        }
        if (lane == 0) { tile_expert = found; tile_row = row; tile_rows = count; failed = 0; }
    }
    __syncthreads();
    const int expert = tile_expert, row0 = tile_row, rows = tile_rows;
    if (expert < 0) return;

    if (threadIdx.x == 0) {
        for (int s = 0; s < C::kStages; ++s) {
            mbar_init(full_bar(s), 1);
            mbar_init(empty_bar(s), 1);
        }
        mbar_init(accum_bar, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(holder, BN);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    uint32_t tmem_base;
    asm volatile("ld.shared.b32 %0, [%1];" : "=r"(tmem_base) : "r"(holder));

    if (warp == 0) {
        int issued = 0;
        bool ok = true;
        for (int i = 0; i < k_blocks; ++i) {
            const int s = i % C::kStages;
            if (i >= C::kStages && !mbar_wait_warp(empty_bar(s), (uint32_t)(i / C::kStages - 1) & 1u)) {
                ok = false;
                if (lane == 0) atomicExch(error_flag, kErrProducerWait);
                break;
            }
            if (elect_one()) {
                mbar_expect_tx(full_bar(s), C::kStageBytes);
                const uint32_t a = base + s * C::kStageBytes;
                tma_load_2d(a, &map_w, i * BK, expert * rows_w + n0, full_bar(s));
                tma_load_2d(a + C::kABytes, &map_x, i * BK, row0, full_bar(s));
            }
            ++issued;
        }
        if (!ok) {  // wait, bounded, for the copies that are still in flight before the block may exit
            if (lane == 0) failed = 1;
            for (int i = max(0, issued - C::kStages); i < issued; ++i)
                if (!mbar_wait_warp(full_bar(i % C::kStages), (uint32_t)(i / C::kStages) & 1u)) {
                    if (lane == 0) atomicExch(error_flag, kErrDrainWait);
                    break;
                }
        }
    } else if (warp == 1) {
        // D = float, A = B = bf16, both K-major, M = 128, N = BN
        constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(BM >> 4) << 24);
        for (int i = 0; i < k_blocks; ++i) {
            const int s = i % C::kStages;
            if (!mbar_wait_warp(full_bar(s), (uint32_t)(i / C::kStages) & 1u)) {
                if (lane == 0) { failed = 1; atomicExch(error_flag, kErrMmaWait); }
                break;
            }
            tc_fence_after();
            const uint32_t a = base + s * C::kStageBytes, b = a + C::kABytes;
            if (elect_one()) {
#pragma unroll
                for (int k = 0; k < BK / UMMA_K; ++k)
                    umma_bf16(tmem_base, smem_desc(a + k * UMMA_K * 2), smem_desc(b + k * UMMA_K * 2), idesc, (i > 0 || k > 0) ? 1u : 0u);
                umma_commit(empty_bar(s));
            }
        }
        if (elect_one()) umma_commit(accum_bar);
    } else {
        const int q = warp & 3;  // the TMEM lane quarter this warp may read
        if (!mbar_wait_warp(accum_bar, 0)) {
            if (lane == 0) { failed = 1; atomicExch(error_flag, kErrEpilogueWait); }
        } else {
            tc_fence_after();
            const uint32_t taddr = tmem_base + ((uint32_t)(q * 32) << 16);
#pragma unroll 1
            for (int c0 = 0; c0 < BN; c0 += 32) {
                if (c0 >= rows) break;  // uniform across the warp
                uint32_t r[32];
                tmem_ld32(taddr + c0, r);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; ++j) stage_f32[(c0 + j) * kPadM + q * 32 + lane] = __uint_as_float(r[j]);
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, BN);
    }
    if (failed) return;
    // rows of 16-byte pieces: eight outputs to a thread and turn
    const int pieces = gated ? 8 : 16;
    for (int i = threadIdx.x; i < rows * pieces; i += kThreads) {
        const int j = i / pieces, p = (i - j * pieces) * 8;
        const float* src = stage_f32 + j * kPadM + p;
        float v[8];
#pragma unroll
        for (int k = 0; k < 8; k += 4) *reinterpret_cast<float4*>(v + k) = *reinterpret_cast<const float4*>(src + k);
        if (gated) {
            float u[8];
#pragma unroll
            for (int k = 0; k < 8; k += 4) *reinterpret_cast<float4*>(u + k) = *reinterpret_cast<const float4*>(src + 64 + k);
#pragma unroll
            for (int k = 0; k < 8; ++k) v[k] = ns_gate_mul<true>(act, v[k], u[k]);
            st8(out + (size_t)(row0 + j) * ldo + n0 / 2 + p, v);
        } else if (n0 + p < rows_w) {  // (rows beyond the expert's belong to the next one)
            st8(out + (size_t)(row0 + j) * ldo + n0 + p, v);
        }
    }
}

template <int BN>
int launch_grouped(const void* x, const void* w, void* out, long long ldo, const int* offsets, int E, int n_pairs, int rows_w, int K,
                   int gated, NsGate act, int* error_flag, cudaStream_t stream) {
    using C = Cfg<BN>;
    static bool configured = false;
    if (!configured) {
        NS_CUDA(cudaFuncSetAttribute(moe_grouped_tc_kernel<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::kSmemBytes));
        configured = true;
    }
    CUtensorMap mw, mx;
    if (const int rc = ns_make_map_bf16(&mw, w, (unsigned long long)E * rows_w, K, K, BM, "ns_moe_grouped_tc")) return rc;
    if (const int rc = ns_make_map_bf16(&mx, x, (unsigned long long)n_pairs, K, K, BN, "ns_moe_grouped_tc")) return rc;
    const int most = min(n_pairs, n_pairs / BN + E);  // tiles that n_pairs rows of E experts can make
    if (most > 65535) NS_FAIL(NS_ERR_UNSUPPORTED, "ns_moe_grouped_tc: %d pairs over %d experts exceed the grid", n_pairs, E);
    NS_LAUNCH((moe_grouped_tc_kernel<BN>), dim3((rows_w + BM - 1) / BM, most), kThreads, C::kSmemBytes, stream, mw, mx, (__nv_bfloat16*)out,
              ldo, offsets, E, rows_w, (K + BK - 1) / BK, gated, act, error_flag);
    NS_CHECK_LAUNCH("ns_moe_grouped_tc");
    return NS_OK;
}

}  // namespace

// xs [n_pairs, width]: the pairs' rows in the plan's order; offsets [E + 1] of that plan; w_gate_up [E, 2 * ff, width] (runs of 64 gate and
// 64 up rows alternate); w_down [E, width, ff]; act [n_pairs, ff] and ys [n_pairs, width] in the plan's order; everything bfloat16,
// width a multiple of 8, ff of 64; alpha, shift, limit: NsGate.  tile: 32, 128 or 256 rows of xs to a block.  error_flag: a device int that a timed-out wait sets.
NS_API int ns_moe_grouped_tc(const void* xs, const int* offsets, const void* w_gate_up, const void* w_down, void* act, void* ys,
                             int n_experts, int n_pairs, int width, int ff, int tile, float alpha, float shift, float limit, int* error_flag,
                             cudaStream_t stream) {
    if (n_pairs <= 0) return NS_OK;
    if (width % 8 || ff % 64 || n_experts < 1) NS_FAIL(NS_ERR_UNSUPPORTED, "ns_moe_grouped_tc: width %d (a multiple of 8), expert width %d (of 64)", width, ff);
    if (((uintptr_t)xs | (uintptr_t)w_gate_up | (uintptr_t)w_down | (uintptr_t)act | (uintptr_t)ys) % 16)
        NS_FAIL(NS_ERR_ARGUMENT, "ns_moe_grouped_tc: operands must start on 16 bytes");
    if (tile != 32 && tile != 128 && tile != 256) NS_FAIL(NS_ERR_ARGUMENT, "ns_moe_grouped_tc: tiles of %d rows", tile);
    auto run = [&](const void* x, const void* w, void* out, int rows_w, int K, int gated) {
        auto* launch = tile == 256 ? launch_grouped<256> : tile == 128 ? launch_grouped<128> : launch_grouped<32>;
        return launch(x, w, out, gated ? rows_w / 2 : rows_w, offsets, n_experts, n_pairs, rows_w, K, gated, NsGate{alpha, shift, limit}, error_flag, stream);
    };
    if (const int rc = run(xs, w_gate_up, act, 2 * ff, width, 1)) return rc;
    return run(act, w_down, ys, width, ff, 0);
}
