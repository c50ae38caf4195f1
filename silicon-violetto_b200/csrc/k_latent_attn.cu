// Latent attention over paged rows (c ; r) on the 5th-generation tensor cores (sizes it does not take and fp32 caches: k_mixer.cu's
// scalar kernel). All query heads read one row per position, whose first part is the value as well, so a block's (token, head) rows
// share the rows it fetches:
//
//   S[row][position] = Q (c ; r)^T          the rows are the MMA's M side (64, as many of them as a block has meaning something)
//   O^T[column][row] += c^T P^T             128 columns of c a time are its M side, the rows its N side
//
// so that O takes rows x columns / 128 of tensor memory's columns, and c is read as it lies: its positions are the second product's
// k side, 64 neighbouring columns a swizzled line. A block has 16, 32 or 64 (token, head) rows of one run -- decoding, a token's
// heads; a prompt's portion, the heads of several neighbouring tokens -- and goes through its share of the run's positions a tile
// at a time:
//
//   warp 0       tiles of 64 positions by TMA, 64 columns a box: the columns of c in pairs of boxes, each pair a slot of a ring, the boxes
//                behind them (of r) in a ring of their own
//   warp 1       the scores' MMAs, a pair of boxes at a time as they come
//   warp 2       the sums' MMAs (a warp of their own: neither kind waits in front of the other's barriers)
//   warps 3..6   softmax in fp32 (a warp has 16 rows: 64 MMA rows lie on the first 16 lanes of each quarter of tensor memory), P in bf16
//                through shared memory; the running maximum moves when a score exceeds it by more than 8, and only then does O come
//                through registers; in the end O
//
// A row's positions may be split over a cluster of blocks, each of which finishes a span of the columns from what the others store
// into its shared memory. Every wait is bounded: when one runs out, the kernel sets the error word, goes on without waiting for more of
// the kind, and leaves by the way it always does.
//
// It takes q with scale * log2(e) folded in, rounded to bf16, and leaves the sums in bf16 for the per-head product after it.
#include <algorithm>
#include <map>
#include <tuple>

#include "paged_attn.cuh"
#include "tcgen05.cuh"

namespace vlt {

namespace latent {

using gemm::elect_one;
using gemm::instr_desc;
using gemm::mbar_arrive;
using gemm::mbar_expect_tx;
using gemm::mbar_init;
using gemm::mma_commit;
using gemm::mma_f16;
using gemm::tma_load_2d;
using gemm::tmem_ld16;
using gemm::wait_or_abort;
using namespace paged;

constexpr uint32_t THREADS = 224, SOFTMAX = 128, MAX_SPLITS = 16, KT = 64, BOX = KT * 128;  // KT: positions of a tile (a page)
constexpr uint32_t MAX_SLOTS = 16, REST_SLOTS = 3, MISC = 2048;
constexpr uint32_t SMEM = 227 * 1024, SMEM_MIN = 116 * 1024;  // (at least half an SM's: one block an SM, which never waits for another's tensor memory)

struct Map {
    alignas(64) uint8_t a[128];
};
struct Args {
    ChunkedAttnArgs c;
    uint32_t groups, sub, toks;                      // see latent_kernel
    uint32_t boxes, mtiles, rest;                    // of a row: boxes of 64 columns; pairs of them that hold c; those behind the pairs
    uint32_t slots, rest_slots, tmem_cols;
    uint32_t* err_flag;
};

// Four times 8 columns of this warp's first 16 lanes: thread (g, tq) has row g's columns 8 j + 2 tq, + 1 and row g + 8's, for each j.
__device__ __forceinline__ void ld_scores(uint32_t taddr, float (&s)[4][4]) {
    uint32_t r[16];
    asm volatile("tcgen05.ld.sync.aligned.16x256b.x4.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]),
                   "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                 : "r"(taddr));
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 16; i++) s[i / 4][i % 4] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const float (&v)[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr), "f"(v[0]), "f"(v[1]), "f"(v[2]),
                 "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]), "f"(v[7]), "f"(v[8]), "f"(v[9]), "f"(v[10]), "f"(v[11]), "f"(v[12]), "f"(v[13]), "f"(v[14]), "f"(v[15])
                 : "memory");
}
__device__ __forceinline__ bool softmax_any(bool mine) {
    uint32_t any;
    asm volatile("{\n.reg .pred p, q;\nsetp.ne.u32 p, %1, 0;\nbar.red.or.pred q, 1, %2, p;\nselp.u32 %0, 1, 0, q;\n}" : "=r"(any) : "r"(uint32_t(mine)), "n"(SOFTMAX) : "memory");
    return any != 0;
}
__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, %0;" ::"n"(SOFTMAX) : "memory"); }
// As gemm::smem_desc, of an operand whose lines are its k: 64 entries of the M side a line, the next 64 `next` bytes on.
__device__ __forceinline__ uint64_t mn_major_desc(uint32_t addr, uint32_t next) {
    return uint64_t((addr & 0x3FFFFu) >> 4) | (uint64_t(next >> 4) << 16) | (uint64_t(1024 >> 4) << 32) | (uint64_t(1) << 46) | (uint64_t(2) << 61);
}

// grid (tiles, 1, key splits). Prompts (sub > 0): tile = (chunk tile, one of its `sub` spans of `toks` tokens, group of ROWS heads); else
// (token, group).
template <uint32_t ROWS>
__global__ void __launch_bounds__(THREADS, 1) latent_kernel(const __grid_constant__ Map map, const Args p) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    constexpr uint32_t QB = ROWS * 128, ACTIVE = ROWS / 16;
    extern __shared__ uint8_t smem_raw[];
    const ChunkedAttnArgs& a = p.c;
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const uint32_t tid = threadIdx.x, warp = tid / 32, lane = tid % 32, grp = blockIdx.x % p.groups, unit = blockIdx.x / p.groups, sp = blockIdx.z, splits = gridDim.z;
    uint32_t t0 = unit, n_tok = 1;
    if (p.sub) {  // (the step's inputs: uploaded before its first kernel)
        const uint32_t tile = unit / p.sub, at = unit % p.sub * p.toks, rows = a.ctiles[2 * tile + 1];
        if (at >= rows) return;  // (all of a cluster's blocks together)
        t0 = a.ctiles[2 * tile] + at;
        n_tok = min(p.toks, rows - at);
    }
    const uint32_t dk = a.kv.dk, rank = a.kv.dv, NP = p.slots, NR = p.rest_slots;
    // Q | the pairs' ring | the ring behind them | P | what follows
    const uint32_t base = smem_u32(smem), ring = base + p.boxes * QB, rest = ring + NP * 2 * BOX, probs = rest + NR * p.rest * BOX;
    uint8_t* misc = smem + (probs - base) + QB;
    const uint32_t bar_full = smem_u32(misc), bar_empty = bar_full + 8 * MAX_SLOTS, bar_rest = bar_empty + 8 * MAX_SLOTS, bar_free = bar_rest + 8 * REST_SLOTS, bar_scores = bar_free + 8 * REST_SLOTS,
                   bar_p = bar_scores + 16, bar_sums = bar_p + 16, bar_merge = bar_sums + 8;
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(misc + 8 * (2 * MAX_SLOTS + 2 * REST_SLOTS + 6));
    volatile uint32_t* abort_flag = tmem_slot + 1;
    volatile uint32_t* end_s = tmem_slot + 2;
    volatile uint32_t* low_s = tmem_slot + 3;
    int* from = reinterpret_cast<int*>(misc + 512);  // a row's place among the queries and the outputs, -1: none
    float* corr_s = reinterpret_cast<float*>(from + ROWS);
    float2* ml_s = reinterpret_cast<float2*>(corr_s + ROWS);  // a row's maximum and the sum under it
    if (tid == 0) {
        for (uint32_t i = 0; i < 2 * MAX_SLOTS + 2 * REST_SLOTS; i++) mbar_init(bar_full + 8 * i, 1);
        mbar_init(bar_scores, 1);
        mbar_init(bar_scores + 8, 1);
        mbar_init(bar_p, ACTIVE);
        mbar_init(bar_p + 8, ACTIVE);
        mbar_init(bar_sums, 1);
        mbar_init(bar_merge, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map) : "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(const_cast<uint32_t*>(tmem_slot))), "r"(p.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    const uint32_t hpt = min(a.heads, ROWS);
    auto row_at = [&](uint32_t r, uint32_t& tok) {
        tok = t0 + r / hpt;
        const uint32_t head = grp * ROWS + r % hpt;
        return r / hpt < n_tok && head < a.heads ? int(tok * a.heads + head) : -1;
    };
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const uint32_t* pages = a.kv.page_table + size_t(a.meta[2 * t0]) * a.kv.max_pages;
    uint32_t begin = 0, n = 0, head = 0, skip = 0, st = 0, ph = 1, rs = 0, rph = 1;
    auto load = [&](uint32_t page) {  // a tile's boxes, into slots that are free; false: they did not become so
        const int row = int(page << PAGE_SHIFT);
        for (uint32_t m = 0; m < p.mtiles; m++) {
            const bool two = 2 * m + 1 < p.boxes;
            if (!wait_or_abort(bar_empty + 8 * st, ph, abort_flag)) return false;
            mbar_expect_tx(bar_full + 8 * st, two ? 2 * BOX : BOX);
            tma_load_2d(ring + st * 2 * BOX, &map, int(m * 128), row, bar_full + 8 * st);
            if (two) tma_load_2d(ring + st * 2 * BOX + BOX, &map, int(m * 128 + 64), row, bar_full + 8 * st);
            if (++st == NP) { st = 0; ph ^= 1; }
        }
        if (!p.rest) return true;
        if (!wait_or_abort(bar_free + 8 * rs, rph, abort_flag)) return false;
        mbar_expect_tx(bar_rest + 8 * rs, p.rest * BOX);
        for (uint32_t b = 0; b < p.rest; b++) tma_load_2d(rest + (rs * p.rest + b) * BOX, &map, int((2 * p.mtiles + b) * 64), row, bar_rest + 8 * rs);
        if (++rs == NR) { rs = 0; rph ^= 1; }
        return true;
    };
    auto share_of = [&](uint32_t low, uint32_t end) {  // this block's tiles: `n` from number `begin` on (see Tiles)
        const Tiles<KT> walk(low, a.keep);
        const uint32_t tiles = walk.count(end), share = (tiles + splits - 1) / splits;
        begin = min(sp * share, tiles);
        n = min(share, tiles - begin);
        head = walk.head;
        skip = walk.skip;
    };
    auto tile_at = [&](uint32_t i) { return begin + i < head ? begin + i : begin + i + skip; };
    // Splits: what the cluster's blocks send of their sums arrives as [source][column of this block's span][row], (m, l) per (source, row)
    // behind it, in the room of Q and the rings; there, too, this block's own, to be copied from.
    constexpr uint32_t RP = ROWS + 4;     // a column's pitch
    constexpr bool BULK = ROWS < 64;      // (64 rows: no room for both; stored one by one)
    const uint32_t span = p.mtiles * 128 / splits, stats = splits * span * RP * 4, own = stats + splits * ROWS * 8;
    bool ok = true;
    if (warp == 0) {  // how far the rows see, and the first two tiles on their way while the others fetch the queries
        uint32_t end = 0, low = 0xffffffffu;
        for (uint32_t i = lane; i < n_tok; i += 32) {
            const View v = view_of(a, t0 + i);
            end = max(end, v.first + 32 - __clz(v.mask));
            low = min(low, v.lo);
        }
        end = __reduce_max_sync(0xffffffffu, end);
        low = __reduce_min_sync(0xffffffffu, low);
        share_of(low, end);
        if (lane == 0) {
            *end_s = end;
            *low_s = low;
            for (uint32_t i = 0; i < min(n, 2u) && ok; i++) ok = load(pages[tile_at(i)]);
        }
    } else {
        if (tid - 32 < ROWS) {
            uint32_t tok;
            from[tid - 32] = row_at(tid - 32, tok);
        }
        // Q in the MMA's swizzle, zeros where there are no rows or columns: a row a warp, three of them at a time, 16 bytes a lane and load.
        constexpr uint32_t WARPS = THREADS / 32 - 1, AT_ONCE = 3;
        for (uint32_t r0 = warp - 1; r0 < ROWS; r0 += AT_ONCE * WARPS) {
            uint4 x[AT_ONCE][3];
#pragma unroll
            for (uint32_t u = 0; u < AT_ONCE; u++) {
                uint32_t tok;
                const uint32_t r = r0 + u * WARPS;
                const int at = r < ROWS ? row_at(r, tok) : -1;
                const uint4* src = reinterpret_cast<const uint4*>(a.q_b + size_t(max(at, 0)) * dk);
#pragma unroll
                for (uint32_t y = 0; y < 3; y++) x[u][y] = at >= 0 && (lane + 32 * y) * 8 < dk ? src[lane + 32 * y] : make_uint4(0, 0, 0, 0);
            }
#pragma unroll
            for (uint32_t u = 0; u < AT_ONCE; u++) {
                const uint32_t r = r0 + u * WARPS;
#pragma unroll
                for (uint32_t y = 0; y < 3; y++) {
                    const uint32_t c = lane + 32 * y;
                    if (r < ROWS && c < p.boxes * 8) *reinterpret_cast<uint4*>(smem + c / 8 * QB + r * 128 + ((c % 8 ^ (r & 7)) << 4)) = x[u][y];
                }
            }
        }
    }
    __syncwarp();
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot, tmem_o = tmem + 2 * KT;
    share_of(*low_s, *end_s);
    auto lo = [](uint32_t addr) { return (addr & 0x3FFFFu) >> 4; };  // (an address in a cluster has the block's rank above these bits)
    const uint64_t k_major = gemm::smem_desc(0);
    if (warp == 0) {
        if (lane == 0) {
            uint32_t page = n > 2 ? pages[tile_at(2)] : 0;
            for (uint32_t i = 2; i < n && ok; i++) {
                const uint32_t now = page;
                if (i + 1 < n) page = pages[tile_at(i + 1)];
                ok = load(now);
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        if (elect_one()) {
            constexpr uint32_t idesc = instr_desc(64, KT);
            const uint32_t q0 = lo(base), ring0 = lo(ring), rest0 = lo(rest);
            uint32_t fs = 0, fph = 0, frs = 0, frph = 0;
            for (uint32_t i = 0; i < n && ok; i++) {
                const uint32_t d = tmem + (i & 1) * KT;
                auto box = [&](uint32_t b, uint32_t at) {  // box b of the tile, which lies at `at`: four steps of 16 columns
#pragma unroll
                    for (uint32_t x = 0; x < 4; x++) mma_f16(d, k_major + (q0 + b * (QB >> 4) + 2 * x), k_major + (at + 2 * x), idesc, (b | x) != 0 ? 1u : 0u);
                };
                if (i >= 2) {  // the softmax has read the scores that lie there
                    ok = wait_or_abort(bar_p + 8 * (i & 1), (i / 2 - 1) & 1, abort_flag);
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                }
                for (uint32_t m = 0; m < p.mtiles && ok; m++) {
                    ok = wait_or_abort(bar_full + 8 * fs, fph, abort_flag);
                    if (!ok) break;
                    box(2 * m, ring0 + fs * (2 * BOX >> 4));
                    if (2 * m + 1 < p.boxes) box(2 * m + 1, ring0 + fs * (2 * BOX >> 4) + (BOX >> 4));
                    if (++fs == NP) { fs = 0; fph ^= 1; }
                }
                if (p.rest && ok) {
                    ok = wait_or_abort(bar_rest + 8 * frs, frph, abort_flag);
                    for (uint32_t b = 0; b < p.rest && ok; b++) box(2 * p.mtiles + b, rest0 + (frs * p.rest + b) * (BOX >> 4));
                    if (ok) mma_commit(bar_free + 8 * frs);
                    if (++frs == NR) { frs = 0; frph ^= 1; }
                }
                if (ok) mma_commit(bar_scores + 8 * (i & 1));
            }
        }
        __syncwarp();
    } else if (warp == 2) {
        if (elect_one()) {
            constexpr uint32_t idesc = instr_desc(128, ROWS) | (1u << 15);  // (bit 15: A's lines are its k)
            const uint64_t mn_major = mn_major_desc(0, BOX);
            const uint32_t ring0 = lo(ring), p0 = lo(probs);
            uint32_t fs = 0;
            for (uint32_t i = 0; i < n && ok; i++) {
                ok = wait_or_abort(bar_p + 8 * (i & 1), (i >> 1) & 1, abort_flag);  // (P comes of the scores, and they of the whole tile)
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                for (uint32_t m = 0; m < p.mtiles; m++) {
#pragma unroll
                    for (uint32_t kk = 0; kk < KT / 16; kk++)
                        mma_f16(tmem_o + m * ROWS, mn_major + (ring0 + fs * (2 * BOX >> 4) + kk * (2048 >> 4)), k_major + (p0 + kk * 2), idesc, (i | kk) != 0 ? 1u : 0u);
                    mma_commit(bar_empty + 8 * fs);
                    if (++fs == NP) fs = 0;
                }
                mma_commit(bar_sums);
            }
        }
        __syncwarp();
    } else {
        const uint32_t quarter = warp & 3, g = lane >> 2, tq = lane & 3, o_addr = tmem_o + ((quarter * 32) << 16);
        const bool active = quarter < ACTIVE;
        const float cap = a.softcap * LOG2E, cap_inv = 2.0f / a.softcap;
        View v[2];
        bool live[2];
        float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
#pragma unroll
        for (uint32_t r = 0; r < 2; r++) {
            uint32_t tok;
            live[r] = active && row_at(quarter * 16 + g + 8 * r, tok) >= 0;
            v[r] = view_of(a, live[r] ? tok : t0);
        }
        const uint32_t first = min(v[0].first, v[1].first), lo_max = max(v[0].lo, v[1].lo);
        for (uint32_t i = 0; i < n; i++) {
            float s[KT / 8][4], m_new[2] = {m_run[0], m_run[1]};
            bool need = false;
            if (active) {
                ok = ok && wait_or_abort(bar_scores + 8 * (i & 1), (i >> 1) & 1, abort_flag);
                ok = __all_sync(0xffffffffu, ok);
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
                for (uint32_t x = 0; x < KT / 32; x++) ld_scores(tmem + (i & 1) * KT + 32 * x + ((quarter * 32) << 16), *reinterpret_cast<float(*)[4][4]>(&s[4 * x]));
                asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                if (a.softcap > 0) {
#pragma unroll
                    for (uint32_t j = 0; j < KT / 8; j++)
#pragma unroll
                        for (uint32_t e = 0; e < 4; e++) s[j][e] = capped(s[j][e], cap, cap_inv);
                }
                const uint32_t key0 = tile_at(i) * KT;
                if (key0 < lo_max || key0 + KT > first || !live[0] || !live[1]) {
#pragma unroll
                    for (uint32_t j = 0; j < KT / 8; j++)
#pragma unroll
                        for (uint32_t e = 0; e < 4; e++)
                            if (!live[e >> 1] || !sees(v[e >> 1], key0 + 8 * j + 2 * tq + (e & 1))) s[j][e] = -INFINITY;
                }
#pragma unroll
                for (uint32_t r = 0; r < 2; r++) {
                    float mx = -INFINITY;
#pragma unroll
                    for (uint32_t j = 0; j < KT / 8; j++) mx = fmaxf(mx, fmaxf(s[j][2 * r], s[j][2 * r + 1]));
                    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                    if (mx > m_run[r] + 8.0f) {
                        need = true;
                        m_new[r] = mx;
                    }
                }
            }
            if (softmax_any(need)) {  // some row's maximum moves (the first tile's do)
                if (active) {
#pragma unroll
                    for (uint32_t r = 0; r < 2; r++) {
                        const float corr = m_new[r] == m_run[r] ? 1.0f : fast_exp2(m_run[r] - m_new[r]);  // (0 from -infinity)
                        m_run[r] = m_new[r];
                        l_run[r] *= corr;
                        if (tq == 0) corr_s[quarter * 16 + g + 8 * r] = corr;
                    }
                }
                softmax_sync();
                if (i) {
                    ok = ok && wait_or_abort(bar_sums, (i - 1) & 1, abort_flag);
                    ok = __all_sync(0xffffffffu, ok);
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    for (uint32_t c = 0; c < p.mtiles * ROWS; c += 16) {
                        float o[16];
                        tmem_ld16(o_addr + c, o);
#pragma unroll
                        for (uint32_t j = 0; j < 16; j++) o[j] *= corr_s[c % ROWS + j];
                        tmem_st16(o_addr + c, o);
                    }
                    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
                    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                }
                softmax_sync();
            }
            if (!active) continue;
            if (i) ok = ok && wait_or_abort(bar_sums, (i - 1) & 1, abort_flag);  // P has been read
            ok = __all_sync(0xffffffffu, ok);
#pragma unroll
            for (uint32_t r = 0; r < 2; r++) {
                const float m = m_run[r] == -INFINITY ? 0.0f : m_run[r];
                const uint32_t row = quarter * 16 + g + 8 * r;
                uint8_t* dst = smem + (probs - base) + row * 128 + tq * 4;
#pragma unroll
                for (uint32_t j = 0; j < KT / 8; j++) {
                    const float e0 = fast_exp2(s[j][2 * r] - m), e1 = fast_exp2(s[j][2 * r + 1] - m);
                    l_run[r] += e0 + e1;
                    *reinterpret_cast<uint32_t*>(dst + ((j ^ (row & 7)) << 4)) = pack_bf16(e0, e1);
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_p + 8 * (i & 1));
        }
        if (active) {
#pragma unroll
            for (uint32_t r = 0; r < 2; r++) {
                l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
                l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
                if (splits == 1 && a.sink && live[r]) l_run[r] += fast_exp2(bf16_to_f32(a.sink[grp * ROWS + (quarter * 16 + g + 8 * r) % hpt]) * LOG2E - m_run[r]);
                if (tq == 0) ml_s[quarter * 16 + g + 8 * r] = make_float2(m_run[r], l_run[r]);
            }
        }
        if (n) ok = ok && wait_or_abort(bar_sums, (n - 1) & 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        softmax_sync();
        if (splits > 1 && BULK) {  // O as the cluster's blocks will take it, a column's rows together
            for (uint32_t c = 0; c < p.mtiles * ROWS; c += 16) {
                float o[16];
                tmem_ld16(o_addr + c, o);
                float4* dst = reinterpret_cast<float4*>(smem + own + ((c / ROWS * 128 + quarter * 32 + lane) * RP + c % ROWS) * 4);
#pragma unroll
                for (uint32_t j = 0; j < 4; j++) dst[j] = n ? make_float4(o[4 * j], o[4 * j + 1], o[4 * j + 2], o[4 * j + 3]) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
        } else if (splits == 1) {
            for (uint32_t c = 0; c < p.mtiles * ROWS; c += 16) {
                float o[16];
                tmem_ld16(o_addr + c, o);
                const uint32_t x = c / ROWS * 128 + quarter * 32 + lane, r0 = c % ROWS;
#pragma unroll
                for (uint32_t j = 0; j < 16; j++)
                    if (from[r0 + j] >= 0 && x < rank) a.out_b[size_t(from[r0 + j]) * rank + x] = f32_to_bf16(__fdividef(o[j], ml_s[r0 + j].y));
            }
        }
    }
    if (!ok) {
        *abort_flag = 1;
        atomicExch(p.err_flag, 6u);
    }
    __syncwarp();
    if (splits > 1) {
        // The cluster: block b finishes columns b span on.
        if (BULK) {
            if (tid == 0) mbar_expect_tx(bar_merge, splits * (span * RP * 4 + ROWS * 8));
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            cluster_sync();  // every block is done with its ring, has laid out its sums and expects the others'
            if (tid < splits) {
                auto copy = [&](uint32_t to, uint32_t src, uint32_t bytes) {
                    asm volatile("cp.async.bulk.shared::cluster.shared::cta.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(cluster_addr(base + to, tid)), "r"(src), "r"(bytes),
                                 "r"(cluster_addr(bar_merge, tid))
                                 : "memory");
                };
                copy(sp * span * RP * 4, base + own + tid * span * RP * 4, span * RP * 4);
                copy(stats + sp * ROWS * 8, smem_u32(ml_s), ROWS * 8);
            }
            ok = gemm::mbar_wait(bar_merge, 0);  // (they come whatever went wrong before)
            if (!ok) atomicExch(p.err_flag, 6u);
            __syncwarp();
            // (No block leaves before every copy, its own among them, has arrived.)
            asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        } else {
            cluster_sync();  // every block is done with its ring
            if (warp >= 3) {
                const uint32_t quarter = warp & 3, me = tid - 96;
                for (uint32_t c = 0; c < p.mtiles * ROWS; c += 16) {
                    float o[16];
                    tmem_ld16(tmem_o + ((quarter * 32) << 16) + c, o);
                    const uint32_t x = c / ROWS * 128 + quarter * 32 + lane;
                    const uint32_t dst = cluster_addr(base + ((sp * span + x % span) * RP + c % ROWS) * 4, x / span);
#pragma unroll
                    for (uint32_t j = 0; j < 16; j += 4) {
                        if (!n) o[j] = o[j + 1] = o[j + 2] = o[j + 3] = 0.0f;
                        asm volatile("st.shared::cluster.v4.f32 [%0], {%1, %2, %3, %4};" ::"r"(dst + j * 4), "f"(o[j]), "f"(o[j + 1]), "f"(o[j + 2]), "f"(o[j + 3]) : "memory");
                    }
                }
                if (me < ROWS)
                    for (uint32_t b = 0; b < splits; b++)
                        asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(cluster_addr(base + stats + (sp * ROWS + me) * 8, b)), "f"(ml_s[me].x), "f"(ml_s[me].y) : "memory");
            }
            __syncwarp();
            cluster_sync();  // every partial has arrived
            asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        }
        const float* recv = reinterpret_cast<const float*>(smem);
        float* stat = reinterpret_cast<float*>(smem + stats);
        // (Code that runs once a block: rolled loops, as its instructions have to be fetched.)
        if (tid < ROWS) {  // what each source's sums of the row are worth
            float m = -INFINITY, l = 0.0f;
#pragma unroll 1
            for (uint32_t k = 0; k < splits; k++) {
                const float2 ml = *reinterpret_cast<const float2*>(stat + (k * ROWS + tid) * 2);
                const float top = fmaxf(m, ml.x);
                if (top != -INFINITY) l = l * fast_exp2(m - top) + ml.y * fast_exp2(ml.x - top);
                m = top;
            }
            if (a.sink && from[tid] >= 0) l += fast_exp2(bf16_to_f32(a.sink[from[tid] % a.heads]) * LOG2E - m);
#pragma unroll 1
            for (uint32_t k = 0; k < splits; k++) {
                float* w = stat + (k * ROWS + tid) * 2;
                *w = *w == -INFINITY ? 0.0f : __fdividef(fast_exp2(*w - m), l);
            }
        }
        __syncthreads();
#pragma unroll 1
        for (uint32_t u = warp, per = (span + 31) / 32; u < ROWS / 4 * per; u += THREADS / 32) {  // 32 neighbouring columns of four rows
            const uint32_t r0 = u / per * 4, c = u % per * 32 + lane, x = sp * span + c;
            if (c >= span || x >= rank) continue;
            float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 2
            for (uint32_t k = 0; k < splits; k++) {
                const float4 v = *reinterpret_cast<const float4*>(recv + (k * span + c) * RP + r0);
                const float* w = stat + (k * ROWS + r0) * 2;
                y.x = fmaf(w[0], v.x, y.x);
                y.y = fmaf(w[2], v.y, y.y);
                y.z = fmaf(w[4], v.z, y.z);
                y.w = fmaf(w[6], v.w, y.w);
            }
            const float ys[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
            for (uint32_t j = 0; j < 4; j++)
                if (from[r0 + j] >= 0) a.out_b[size_t(from[r0 + j]) * rank + x] = f32_to_bf16(ys[j]);
        }
        __syncwarp();
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
    }
}

template <uint32_t ROWS>
void launch(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t max_keys, uint32_t sm_count, uint32_t keys_per_block, uint32_t* err_flag, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] {
        VLT_CUDA(cudaFuncSetAttribute(latent_kernel<ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(SMEM)));
        VLT_CUDA(cudaFuncSetAttribute(latent_kernel<ROWS>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    });
    static thread_local std::map<std::tuple<const void*, uint32_t, uint32_t>, Map> maps;
    auto key = std::make_tuple(static_cast<const void*>(a.kv.k), a.kv.dk, a.kv.n_pages);
    auto it = maps.find(key);
    if (it == maps.end()) {
        Map m;
        make_tensor_map_2d(m.a, a.kv.k, a.kv.dk, uint64_t(a.kv.n_pages) * PAGE, 64, KT, 2, true);
        it = maps.emplace(key, m).first;
    }
    Args p;
    p.c = a;
    p.err_flag = err_flag;
    p.groups = (a.heads + ROWS - 1) / ROWS;
    p.toks = n_ctiles ? std::max(1u, ROWS / a.heads) : 1;
    p.sub = n_ctiles ? (64 + p.toks - 1) / p.toks : 0;
    p.mtiles = (a.kv.dv + 127) / 128;
    p.boxes = (a.kv.dk + 63) / 64;
    p.rest = p.boxes > 2 * p.mtiles ? p.boxes - 2 * p.mtiles : 0;
    // Room for two tiles at least (the sums of one wait for their P while the scores of the next come in).
    const uint32_t fixed = 1024 + (p.boxes + 1) * ROWS * 128 + MISC;
    p.rest_slots = fixed + (p.rest * REST_SLOTS + 4 * p.mtiles) * BOX <= SMEM ? REST_SLOTS : 2;
    p.slots = std::min(MAX_SLOTS, (SMEM - fixed - p.rest * p.rest_slots * BOX) / (2 * BOX));
    if (p.slots < 2 * p.mtiles) throw Error("internal: latent attention over " + std::to_string(a.kv.dk) + " columns");
    p.tmem_cols = 32;
    while (p.tmem_cols < 2 * KT + p.mtiles * ROWS) p.tmem_cols *= 2;
    // A tile's positions over 1, 2, 4, 8 or 16 blocks: the count that makes waves of clusters times a block's positions, plus what a block and
    // a cluster's exchange cost besides (as much as some hundred positions), least.
    const uint32_t units = std::max(1u, (n + p.toks - 1) / p.toks * p.groups), smem = std::max(SMEM_MIN, fixed + (p.rest * p.rest_slots + 2 * p.slots) * BOX);
    static thread_local std::map<std::pair<uint32_t, uint32_t>, uint32_t> wave;  // (shared memory, cluster size) -> clusters that run at once
    auto at_once = [&](uint32_t c) {
        if (c == 1) return sm_count;
        auto w = wave.find({smem, c});
        if (w != wave.end()) return w->second;
        cudaLaunchConfig_t q = {};
        q.gridDim = dim3(sm_count, 1, c);
        q.blockDim = dim3(THREADS);
        q.dynamicSmemBytes = smem;
        cudaLaunchAttribute qa[1];
        qa[0].id = cudaLaunchAttributeClusterDimension;
        qa[0].val.clusterDim.x = qa[0].val.clusterDim.y = 1;
        qa[0].val.clusterDim.z = c;
        q.attrs = qa;
        q.numAttrs = 1;
        int clusters = 0;
        const cudaError_t e = cudaOccupancyMaxActiveClusters(&clusters, latent_kernel<ROWS>, &q);
        return wave.emplace(std::make_pair(smem, c), e == cudaSuccess ? uint32_t(clusters) : 0u).first->second;
    };
    uint32_t splits = 1;
    uint64_t best = ~0ull;
    for (uint32_t c = 1; c <= MAX_SPLITS && (c == 1 || max_keys / c >= KT); c *= 2) {
        const uint32_t w = at_once(c);
        if (!w) continue;
        const uint64_t cost = uint64_t((units + w - 1) / w) * ((max_keys + c - 1) / c + (c > 1 ? 550 : 300));
        if (cost < best) { best = cost; splits = c; }
    }
    if (keys_per_block)
        for (splits = 1; splits < MAX_SPLITS && splits * keys_per_block < max_keys && at_once(2 * splits);) splits *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((p.sub ? n_ctiles * p.sub : n) * p.groups, 1, splits);
    cfg.blockDim = dim3(THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = splits;
    cfg.attrs = attr;
    cfg.numAttrs = splits > 1 ? 2 : 1;
    VLT_CUDA(cudaLaunchKernelEx(&cfg, latent_kernel<ROWS>, it->second, p));
    launch_counter()++;
}

}  // namespace latent

bool latent_attn_fits(uint32_t kv_rank, uint32_t rot_dim, uint32_t page) {
    return page == paged::PAGE && kv_rank <= 512 && kv_rank % 8 == 0 && rot_dim % 8 == 0 && kv_rank + rot_dim <= 576;
}
void launch_attn_latent(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t max_keys, uint32_t sm_count, uint32_t keys_per_block, uint32_t* err_flag, cudaStream_t s) {
    if (a.slopes) throw Error("internal: latent attention has no slopes");
    if (n_ctiles || a.heads > 32) latent::launch<64>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, err_flag, s);
    else if (a.heads > 16) latent::launch<32>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, err_flag, s);
    else latent::launch<16>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, err_flag, s);
}

}  // namespace vlt
