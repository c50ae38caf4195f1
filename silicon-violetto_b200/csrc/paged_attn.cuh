// What the attention kernels over paged keys share: asynchronous copies, a cluster's barrier and addresses, what a token sees, and the
// score's soft cap.
#pragma once
#include "kernels.h"
#include "mma.cuh"

namespace vlt {

namespace paged {

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void cluster_sync() { asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ uint32_t cluster_addr(uint32_t addr, uint32_t rank) {
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
    return r;
}
__device__ __forceinline__ float gated(float y, float gate) { return y / (1.0f + __expf(-gate)); }

constexpr uint32_t PAGE_SHIFT = 6, PAGE = 1u << PAGE_SHIFT;

// What token t sees: cached keys [0, keep) and [lo, first) and, of its tile of 8 rows (token `tile` on) that starts at cache position
// `first`, those `mask` names (its `vis`, less the rows of an earlier chunk or out of the window: the rows of a draft tree may lie on
// both sides of an edge).
struct View {
    uint32_t slot, pos, lo, keep, first, mask, tile;
};
__device__ __forceinline__ View view_of(const ChunkedAttnArgs& a, uint32_t t) {
    const uint32_t pos = a.meta[2 * t + 1], row = a.tin[2 * t + 1], i = row % 8;
    View v;
    v.slot = a.meta[2 * t];
    v.pos = pos;
    v.keep = a.keep;
    v.tile = t - i;
    v.first = a.meta[2 * (t - row) + 1] + row - i;
    v.lo = a.chunk ? pos / a.chunk * a.chunk : a.window && pos + 1 > a.window ? pos + 1 - a.window : 0;
    v.mask = a.vis[t];
    if (v.lo) {
        uint32_t seen = 0;
        for (uint32_t m = v.mask; m;) {
            const uint32_t j = __ffs(m) - 1;
            m &= m - 1;
            const uint32_t at = a.meta[2 * (v.tile + j) + 1];
            if (at >= v.lo || at < v.keep) seen |= 1u << j;
        }
        v.mask = seen;
    }
    return v;
}
__device__ __forceinline__ bool sees(const View& v, uint32_t key) {
    return key < v.first ? key >= v.lo || key < v.keep : key - v.first < 32 && ((v.mask >> (key - v.first)) & 1u);
}
// How far a seen key lies back. (A draft tree's rows lie in the cache one after the other, but at positions of their own.)
__device__ __forceinline__ float distance(const ChunkedAttnArgs& a, const View& v, uint32_t key) {
    return float(int(v.pos) - int(key < v.first ? key : a.meta[2 * (v.tile + key - v.first) + 1]));
}
// The tiles of SIZE positions that hold keys seen, of rows whose lowest `lo` is `low`: the first `head` ones with keys kept, then from
// low's on. Walked by number.
template <uint32_t SIZE>
struct Tiles {
    uint32_t head, skip;
    __device__ __forceinline__ Tiles(uint32_t low, uint32_t keep) {
        head = min((keep + SIZE - 1) / SIZE, low / SIZE);
        skip = low / SIZE - head;
    }
    __device__ __forceinline__ uint32_t count(uint32_t end) const { return (end + SIZE - 1) / SIZE - skip; }
    __device__ __forceinline__ uint32_t at(uint32_t i) const { return i < head ? i : i + skip; }
};
// A score times log2(e), soft-capped: cap tanh(s / cap) as cap - 2 cap / (e^(2 s / cap) + 1), whose error is one of the exponential's and
// the quotient's last bits of the cap. cap: the constant times log2(e); inv: 2 / the constant.
__device__ __forceinline__ float capped(float s, float cap, float inv) { return cap - __fdividef(2.0f * cap, fast_exp2(s * inv) + 1.0f); }

}  // namespace paged

}  // namespace vlt
