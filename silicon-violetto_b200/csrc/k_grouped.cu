// Grouped linear layers on the 5th-generation tensor cores: the experts' matrices of a mixture, each against the tokens that
// chose it, or a matrix per head against that head's part of every token. A block takes one (expert, rows <= N) tile of the sorted pairs (k_moe.cu's table) and 128 of the expert's output
// rows: the weights are the MMA's M side, so an expert's matrix crosses HBM once for its tile of tokens, from one token on;
// the tokens are its N side, N rounded to 16 per tile. Weights come by TMA into 128-byte-swizzled stages; four warps fetch
// the tokens' rows -- gathered through the pair -> token table, or in place -- by 16-byte asynchronous copies into the same
// swizzle; one elected lane issues tcgen05.mma with the accumulator in tensor memory; the four warps then read it back and
// apply the epilogue. Two blocks share an SM, so that one's fill and epilogue run under the other's main loop. Every wait is
// bounded: on a time-out the kernel sets the error word, frees its tensor memory and returns.
#include <cuda.h>

#include <algorithm>
#include <map>
#include <tuple>

#include "kernels.h"
#include "tcgen05.cuh"

namespace vlt {

namespace grouped {

using namespace gemm;

constexpr uint32_t BM = 128, BK = 64, LOADERS = 4, THREADS = 32 * (2 + LOADERS);

struct Map {
    alignas(64) uint8_t a[128];
};

struct Args {
    LinearArgs l;
    uint32_t stages, n_max, tmem_cols;  // n_max: a tile's rows at most, rounded to 16
    uint32_t* err_flag;
};

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }

// grid (m / 128, tiles). warp 0: weights by TMA; warp 1: MMA; warps 2..5: the tokens' rows, then the epilogue.
template <uint32_t EPI>
__global__ void __launch_bounds__(THREADS, 2) grouped_kernel(const __grid_constant__ Map map, const Args a) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");  // which expert a block works for is the kernel before's result
    if (blockIdx.y >= *a.l.n_tiles) return;
    const uint32_t group = a.l.tiles[3 * blockIdx.y], p0 = a.l.tiles[3 * blockIdx.y + 1], count = a.l.tiles[3 * blockIdx.y + 2];
    const uint32_t S = a.stages, n = (count + 15) / 16 * 16, a_bytes = BM * BK * 2, b_bytes = a.n_max * BK * 2, stage = a_bytes + b_bytes;
    const uint32_t base = smem_u32(smem), tid = threadIdx.x, warp = tid / 32, lane = tid % 32, nkb = a.l.k / BK;
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + S * stage);  // full[S], empty[S], accumulator
    const uint32_t bar_full = smem_u32(bars), bar_empty = bar_full + 8 * S, bar_accum = bar_empty + 8 * S;
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(bars + 2 * S + 1);
    volatile uint32_t* abort_flag = tmem_slot + 1;
    if (tid == 0) {
        for (uint32_t c = 0; c < S; c++) {
            mbar_init(bar_full + 8 * c, 1 + LOADERS);  // the TMA's expect_tx and the loader warps
            mbar_init(bar_empty + 8 * c, 1);
        }
        mbar_init(bar_accum, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(const_cast<uint32_t*>(tmem_slot))), "r"(a.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;
    const uint32_t row0 = blockIdx.x * BM;
    bool ok = true;
    if (warp == 0) {
        if (lane == 0) {
            uint32_t st = 0, ph = 1;
            for (uint32_t i = 0; i < nkb; i++) {
                ok = wait_or_abort(bar_empty + 8 * st, ph, abort_flag);
                if (!ok) break;
                mbar_expect_tx(bar_full + 8 * st, a_bytes);
                tma_load_2d(base + st * stage, &map, int(i * BK), int(group * a.l.m + row0), bar_full + 8 * st);
                if (++st == S) { st = 0; ph ^= 1; }
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        const uint32_t leader = elect_one(), idesc = instr_desc(BM, n);
        const uint64_t da0 = smem_desc(base), db0 = smem_desc(base + a_bytes);
        const uint32_t hi_a = uint32_t(da0 >> 32), hi_b = uint32_t(db0 >> 32), lo_a0 = uint32_t(da0), lo_b0 = uint32_t(db0);
        uint32_t st = 0, ph = 0;
        for (uint32_t i = 0; i < nkb; i++) {
            ok = wait_or_abort(bar_full + 8 * st, ph, abort_flag);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t lo_a = lo_a0 + st * (stage >> 4), lo_b = lo_b0 + st * (stage >> 4);
            if (leader) {
#pragma unroll
                for (uint32_t k4 = 0; k4 < BK / 16; k4++)
                    mma_f16(tmem, (uint64_t(hi_a) << 32) | (lo_a + 2 * k4), (uint64_t(hi_b) << 32) | (lo_b + 2 * k4), idesc, (i | k4) != 0 ? 1u : 0u);
                mma_commit(bar_empty + 8 * st);
            }
            __syncwarp();
            if (++st == S) { st = 0; ph ^= 1; }
        }
        if (ok && leader) mma_commit(bar_accum);
        __syncwarp();
    } else {
        // The tokens' rows: chunk c of a stage is 16-byte piece c % 8 of row c / 8, at piece ^ (row & 7) of that row (the
        // swizzle the MMA's descriptor names). A row past the tile's count repeats its first: its column is not read.
        const uint32_t me = (warp - 2) * 32 + lane, piece = me % 8, r_first = me / 8, per = n / 16;  // 128 threads: 16 rows at a time
        const uint16_t* X = static_cast<const uint16_t*>(a.l.X);
        constexpr uint32_t MAX_PER = 8;  // (n <= 128)
        const uint16_t* src[MAX_PER];
#pragma unroll
        for (uint32_t j = 0; j < MAX_PER; j++) {
            const uint32_t r = r_first + 16 * j, p = p0 + (r < count ? r : 0);
            const size_t from = j >= per ? 0 : a.l.src ? a.l.src[p] : a.l.by_head ? size_t(p - group * a.l.by_head) * a.l.heads + group : p;
            src[j] = X + from * a.l.k + piece * 8;
        }
        const uint32_t dst0 = base + a_bytes + r_first * 128 + ((piece ^ (r_first & 7)) << 4);
        constexpr uint32_t LAG = 2;  // stages requested ahead of the one reported full
        uint32_t st = 0, ph = 1, rst = 0;
        for (uint32_t i = 0; i < nkb + LAG; i++) {
            if (i < nkb && ok) {
                ok = wait_or_abort(bar_empty + 8 * st, ph, abort_flag);
                if (ok) {
                    const uint32_t dst = dst0 + st * stage;
#pragma unroll
                    for (uint32_t j = 0; j < MAX_PER; j++)
                        if (j < per) cp_async16(dst + j * 16 * 128, src[j] + size_t(i) * BK);
                }
                if (++st == S) { st = 0; ph ^= 1; }
            }
            asm volatile("cp.async.commit_group;" ::: "memory");  // (empty groups at the end, so that the count below holds)
            if (i >= LAG) {
                asm volatile("cp.async.wait_group %0;" ::"n"(LAG) : "memory");
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
                __syncwarp();
                if (lane == 0) mbar_arrive(bar_full + 8 * rst);
                if (++rst == S) rst = 0;
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        if (ok) ok = wait_or_abort(bar_accum, 0, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t quarter = warp & 3, row = row0 + quarter * 32 + lane;
            for (uint32_t c0 = 0; c0 < n; c0 += 16) {
                float acc[16];
                float gate[16];
                if (EPI == EPI_RAW && a.l.by_head && a.l.gate) {  // (their loads go out together)
                    const float* from = a.l.gate + size_t(p0 + c0 - group * a.l.by_head) * a.l.ldg + (a.l.gate_w == 1 ? group : size_t(group) * a.l.m + row);
#pragma unroll
                    for (uint32_t j = 0; j < 16; j++) gate[j] = c0 + j < count ? from[size_t(j) * a.l.ldg] : 0.0f;
                }
                tmem_ld16(tmem + ((quarter * 32) << 16) + c0, acc);
#pragma unroll
                for (uint32_t j = 0; j < 16; j++) {
                    if (c0 + j >= count) break;
                    float y = acc[j];
                    size_t o = size_t(p0 + c0 + j) * a.l.m + row;
                    if (EPI == EPI_RELU2) y = y > 0.0f ? y * y : 0.0f;
                    if (EPI == EPI_GLU_CLAMP) {
                        if (a.l.row_scale) y *= a.l.row_scale[p0 + c0 + j];
                        const float u = __shfl_xor_sync(0xffffffffu, y, 1);
                        if (lane & 1) continue;  // (a pair's even row has its output)
                        y = clamped_glu(y, u, a.l.limit);
                        o = size_t(p0 + c0 + j) * (a.l.m / 2) + row / 2;
                    } else if (EPI == EPI_RAW && a.l.by_head) {
                        const size_t t = p0 + c0 + j - group * a.l.by_head;
                        if (a.l.gate) y *= __fdividef(1.0f, 1.0f + __expf(-gate[j]));
                        o = (t * a.l.heads + group) * a.l.ldy + row;
                    }
                    if (a.l.Y) a.l.Y[o] = y;
                    if (a.l.Yb) a.l.Yb[o] = f32_to_bf16(y);
                }
            }
        }
    }
    if (!ok) {
        *abort_flag = 1;
        atomicExch(a.err_flag, 5u);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(a.tmem_cols) : "memory");
    }
}

}  // namespace grouped

bool grouped_fits(uint32_t m, uint32_t k) { return m % grouped::BM == 0 && k % grouped::BK == 0; }

// n_groups: the matrices stacked at a.W; tile: the most rows a tile of the table has (16 .. 128).
void launch_grouped(const LinearArgs& a, uint32_t n_groups, uint32_t tile, uint32_t* err_flag, cudaStream_t s) {
    static thread_local std::map<std::tuple<const void*, uint32_t, uint32_t, uint32_t>, grouped::Map> maps;
    static PerDevice configured;
    if (!a.max_tiles) return;
    if (!grouped_fits(a.m, a.k) || tile < 16 || tile > 128 || tile % 16 || (a.epi != EPI_RAW && a.epi != EPI_RELU2 && a.epi != EPI_GLU_CLAMP) || (a.row_scale && a.epi != EPI_GLU_CLAMP) || a.bias) throw Error("internal: a grouped GEMM of an unsupported shape");
    auto key = std::make_tuple(static_cast<const void*>(a.W), a.m, a.k, n_groups);
    auto it = maps.find(key);
    if (it == maps.end()) {
        grouped::Map m;
        make_tensor_map_2d(m.a, a.W, a.k, uint64_t(n_groups) * a.m, grouped::BK, grouped::BM, 2, true);
        it = maps.emplace(key, m).first;
    }
    constexpr uint32_t SMEM = 112 * 1024;  // two blocks an SM
    configured.once([] {
        for (auto f : {grouped::grouped_kernel<EPI_RAW>, grouped::grouped_kernel<EPI_RELU2>, grouped::grouped_kernel<EPI_GLU_CLAMP>}) VLT_CUDA(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, int(SMEM)));
    });
    grouped::Args g;
    g.l = a;
    g.n_max = tile;
    const uint32_t stage = grouped::BM * grouped::BK * 2 + tile * grouped::BK * 2;
    g.stages = std::min(6u, (SMEM - 2048) / stage);
    g.tmem_cols = std::max(32u, tile <= 32 ? 32u : tile <= 64 ? 64u : 128u);
    g.err_flag = err_flag;
    // (at least 78 KiB, so that no third block, whose tensor memory might not be there, comes onto the SM)
    const size_t smem = std::max<size_t>(size_t(g.stages) * stage + 1024 + (2 * g.stages + 1) * 8 + 16, 78 * 1024);
    const dim3 grid(a.m / grouped::BM, a.max_tiles);
    if (a.epi == EPI_GLU_CLAMP) launch_pdl(grouped::grouped_kernel<EPI_GLU_CLAMP>, grid, grouped::THREADS, smem, s, it->second, g);
    else if (a.epi == EPI_RELU2) launch_pdl(grouped::grouped_kernel<EPI_RELU2>, grid, grouped::THREADS, smem, s, it->second, g);
    else launch_pdl(grouped::grouped_kernel<EPI_RAW>, grid, grouped::THREADS, smem, s, it->second, g);
}

}  // namespace vlt
