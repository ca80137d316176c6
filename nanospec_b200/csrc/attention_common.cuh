// Pieces shared by the bfloat16 attention kernels: tile sizes and the loader that brings 64
// keys and values of one kv head from scattered cache pages into padded shared-memory tiles.
#pragma once

#include "mma_utils.cuh"

namespace {

constexpr int kTileKeys = 64;
constexpr int kThreads = 128;
constexpr float kLog2e = 1.4426950408889634f;

// Rows key0 .. key0+63 of one kv head: cache[page, hk, offset, :] with page = bt[key / page_size].
// Rows before key_lo (their pages may already have been given back behind a window) and rows at or
// beyond key_end are not read but zero-filled (a masked weight of zero must not meet a NaN).
// Kept first keys behind a window: the caller counts keys in a virtual range in which the kept keys lie
// directly before the window; a virtual key below key_split is the real key (virtual - gap).  With
// gap == 0 virtual and real keys are the same.
// Keys of dk and values of dv features (multiples of 8, at most D) lie in the cache at their own widths; the tile's columns
// beyond them are zero-filled, so that the products over D features are those over dk and dv.  Values wider than a tile are taken a
// slice at a time: v_cache points at the slice's first feature, dv is its width and dv_row the width of a whole value (0: dv).
template <int D, int THREADS = kThreads>
__device__ __forceinline__ void load_kv_tile(__nv_bfloat16* ks, __nv_bfloat16* vs, const __nv_bfloat16* k_cache,
                                             const __nv_bfloat16* v_cache, const int* bt, int key0, int key_lo, int key_end,
                                             int hk, int nkv, int page_size, int page_shift, int key_split = 0, int gap = 0,
                                             int dk = D, int dv = D, int dv_row = 0) {
    if (dv_row == 0) dv_row = dv;
    constexpr int kChunks = D / 8;
    constexpr int kItems = (kTileKeys * kChunks + THREADS - 1) / THREADS;  // 16-byte pieces per thread and tensor
    // When the threads divide evenly over the pieces of a row, a thread keeps the same piece of
    // the row for every item and its rows advance by a constant: no division per item.
    constexpr bool kRegular = THREADS % kChunks == 0;
    constexpr int kRowStep = kRegular ? THREADS / kChunks : 0;
    const int ch0 = kRegular ? threadIdx.x % kChunks : 0;
    const int row0 = kRegular ? threadIdx.x / kChunks : 0;
    // first the block-table entries of all of this thread's rows (independent loads), then the copies:
    // the copies are ordered against other memory operations, and a table lookup between two of them
    // would cost a full load latency each time
    int page[kItems];
#pragma unroll
    for (int i = 0; i < kItems; ++i) {
        const int c = threadIdx.x + i * THREADS;
        const int row = kRegular ? row0 + i * kRowStep : c / kChunks;
        const int vkey = key0 + row;
        const int key = vkey >= key_split ? vkey : vkey - gap;
        const bool valid = c < kTileKeys * kChunks && vkey >= key_lo && vkey < key_end;
        // page_shift >= 0: the page size is a power of two (no integer division per row)
        page[i] = valid ? __ldg(bt + (page_shift >= 0 ? key >> page_shift : key / page_size)) : -1;
    }
#pragma unroll
    for (int i = 0; i < kItems; ++i) {
        const int c = threadIdx.x + i * THREADS;
        if (c >= kTileKeys * kChunks) break;
        const int row = kRegular ? row0 + i * kRowStep : c / kChunks;
        const int ch = kRegular ? ch0 : c - row * kChunks;
        const int vkey = key0 + row;
        const int key = vkey >= key_split ? vkey : vkey - gap;
        const bool valid = page[i] >= 0;
        size_t slot = 0;
        if (valid) {
            const int within = page_shift >= 0 ? key & (page_size - 1) : key % page_size;
            slot = ((size_t)page[i] * nkv + hk) * page_size + within;
        }
        const bool in_k = valid && ch * 8 < dk, in_v = valid && ch * 8 < dv;
        ns_cp_async16(NsTile<D>::at(ks, row, ch * 8), k_cache + (in_k ? slot * dk + ch * 8 : 0), in_k);
        ns_cp_async16(NsTile<D>::at(vs, row, ch * 8), v_cache + (in_v ? slot * dv_row + ch * 8 : 0), in_v);
    }
}

// How values of dv features meet keys of dk in an instance of at most 128: in slices of equal width (a multiple of 8, the last may be
// narrower), one block each - the scores are computed once per slice - and the instance (a multiple of 16) that runs.
struct ValueSlices { int count, width, instance; };
inline ValueSlices value_slices(int dk, int dv) {
    const int count = (dv + 127) / 128;
    const int width = ((dv + count - 1) / count + 7) / 8 * 8;
    return {count, width, ((dk > width ? dk : width) + 15) / 16 * 16};
}

// The factor of an output feature: the sigmoid of the head's gate (per_feature 0) or of the feature's own, times out_scale.
struct OutGate { const __nv_bfloat16* gate; int stride, per_feature; float out_scale; };
__device__ __forceinline__ float gate_factor(const OutGate& g, size_t token, int h, int feature) {
    if (!g.gate) return g.out_scale;
    const float z = __bfloat162float(g.gate[token * g.stride + (g.per_feature ? feature : h)]);
    return __fdividef(g.out_scale, 1.f + __expf(-z));
}

}  // namespace
