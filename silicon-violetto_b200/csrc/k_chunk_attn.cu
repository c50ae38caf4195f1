// Attention over paged keys on the tensor cores, chunked, windowed or over everything before, for head sizes that are instantiated
// below (other sizes and fp32 caches: k_mixer.cu's scalar kernel). What a row walks begins wherever its chunk or window does, in
// the middle of a page or not, and is bounded by it; in front of a window come the tiles of the first positions, if some are kept.
// Scores may be capped, and lowered by a head's slope times the distance.
//
//   chunk_decode_kernel   a row (token) and up to 8 query heads of one kv head per block: the keys are the MMAs' M side, the
//                         heads its columns; four warps take tiles of 16 keys in turn, each with its own ring of asynchronous
//                         copies; a row's keys may be split over a cluster of blocks, whose first adds up what the others
//                         store into its shared memory.
//   chunk_prefill_kernel  64 rows of a run and one query head per block: the rows are the M side, the keys come a page at a
//                         time, every other page to each of two groups of four warps, which meet at the end (a prompt's portion
//                         has few blocks for its SMs); the softmax stays in registers.
//
// Both take q rotated, scaled by scale * log2(e) and rounded to bf16, keep scores and softmax in fp32, and finish the mixer:
// the output times sigmoid(gate) where there is a gate, bf16 for the projection after it.
#include <algorithm>

#include "paged_attn.cuh"

namespace vlt {

namespace chunked {

using namespace paged;

constexpr uint32_t TILE = 16, WARPS = 4, STAGES = 2, MAX_SPLITS = 16;
template <uint32_t DK, uint32_t DV>
constexpr uint32_t decode_smem() {
    const uint32_t ring = WARPS * STAGES * TILE * (DK + DV) * 2, own = WARPS * 8 * (DV + 6) * 4, cluster = MAX_SPLITS * 8 * (DV + 4) * 4;
    return std::max(ring, std::max(own, cluster));
}

// grid (tokens, kv heads x groups of 8 query heads, key splits); the splits of a (token, kv head) are one cluster.
template <uint32_t DK, uint32_t DV>
__global__ void __launch_bounds__(WARPS * 32, 3) chunk_decode_kernel(const ChunkedAttnArgs a) {
    pdl_start();
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr uint32_t KB = TILE * DK * 2, VB = TILE * DV * 2, KS = DK / 16, DM = DV / 16, KC = DK / 8, VC = DV / 8;
    const uint32_t t = blockIdx.x, kvh = blockIdx.y % a.kv.n_kv, sp = blockIdx.z, warp = threadIdx.x / 32, lane = threadIdx.x % 32, g = lane >> 2, tq = lane & 3;
    const uint32_t G = a.heads / a.kv.n_kv, h0 = kvh * G + blockIdx.y / a.kv.n_kv * 8, cols = min(8u, kvh * G + G - h0);
    const View v = view_of(a, t);
    const float cap = a.softcap * LOG2E, cap_inv = 2.0f / a.softcap;
    float slope[2] = {0.0f, 0.0f};
    if (a.slopes)
#pragma unroll
        for (uint32_t e = 0; e < 2; e++) slope[e] = a.slopes[h0 + min(2 * tq + e, cols - 1)] * LOG2E;
    // Tiles of 16 positions up to the last key seen (pages hold whole tiles): an even share.
    const Tiles<TILE> walk(v.lo, v.keep);
    const uint32_t tiles = walk.count(v.first + 32 - __clz(v.mask)), share = (tiles + gridDim.z - 1) / gridDim.z;
    const uint32_t begin = min(sp * share, tiles), n = min(share, tiles - begin), my = warp < n ? (n - warp + WARPS - 1) / WARPS : 0;

    uint32_t q[KS][2];
    {
        const uint32_t* qp = reinterpret_cast<const uint32_t*>(a.q_b + (size_t(t) * a.heads + h0 + min(g, cols - 1)) * DK);
#pragma unroll
        for (uint32_t ks = 0; ks < KS; ks++) {
            q[ks][0] = g < cols ? qp[8 * ks + tq] : 0u;
            q[ks][1] = g < cols ? qp[8 * ks + 4 + tq] : 0u;
        }
    }
    float o[DM][4], m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
#pragma unroll
    for (uint32_t dm = 0; dm < DM; dm++) o[dm][0] = o[dm][1] = o[dm][2] = o[dm][3] = 0.0f;

    const uint32_t* pages = a.kv.page_table + size_t(v.slot) * a.kv.max_pages;
    const uint16_t* K = static_cast<const uint16_t*>(a.kv.k);
    const uint16_t* V = static_cast<const uint16_t*>(a.kv.v);
    const uint32_t wbuf = smem_u32(smem) + warp * STAGES * (KB + VB);
    auto issue = [&](uint32_t i) {  // this warp's tile i: 16 neighbouring rows of K and of V
        const uint32_t key0 = walk.at(begin + warp + i * WARPS) * TILE;
        const size_t r0 = ((size_t(pages[key0 >> PAGE_SHIFT]) * a.kv.n_kv + kvh) << PAGE_SHIFT) + (key0 & (PAGE - 1));
        const uint32_t dst = wbuf + (i % STAGES) * (KB + VB);
#pragma unroll
        for (uint32_t c = lane; c < TILE * KC; c += 32) {
            const uint32_t key = c / KC, piece = c % KC;
            cp_async16(dst + key * DK * 2 + ((piece ^ (key & 7)) << 4), K + (r0 + key) * DK + piece * 8);
        }
#pragma unroll
        for (uint32_t c = lane; c < TILE * VC; c += 32) {
            const uint32_t key = c / VC, piece = c % VC;
            cp_async16(dst + KB + key * DV * 2 + ((piece ^ (key & 7)) << 4), V + (r0 + key) * DV + piece * 8);
        }
    };
#pragma unroll
    for (uint32_t i = 0; i < STAGES; i++) {
        if (i < my) issue(i);
        cp_async_commit();
    }
    // ldmatrix lane roles: matrix lm = lane / 8, row lr = lane % 8. K as A (keys x dims): key 8 (lm & 1) + lr, piece
    // 2 ks + (lm >> 1). V^T as A (dims x keys, .trans): key 8 (lm >> 1) + lr, piece 2 dm + (lm & 1).
    const uint32_t lm = lane >> 3, lr = lane & 7;
    const uint32_t k_row = (8 * (lm & 1) + lr) * DK * 2, k_c = lm >> 1, v_row = (8 * (lm >> 1) + lr) * DV * 2, v_c = lm & 1;
    for (uint32_t i = 0; i < my; i++) {
        cp_async_wait<STAGES - 1>();
        __syncwarp();
        const uint32_t kbase = wbuf + (i % STAGES) * (KB + VB), vbase = kbase + KB, key0 = walk.at(begin + warp + i * WARPS) * TILE;
        float s[4] = {0.0f, 0.0f, 0.0f, 0.0f};  // [0, 1] key g, columns 2 tq, 2 tq + 1; [2, 3] key g + 8
#pragma unroll
        for (uint32_t ks = 0; ks < KS; ks++) {
            uint32_t ka[4];
            ldmatrix_x4(ka, kbase + k_row + (((2 * ks + k_c) ^ lr) << 4));
            mma16816(s, ka, q[ks][0], q[ks][1]);
        }
        if (a.softcap > 0) {
#pragma unroll
            for (int e = 0; e < 4; e++) s[e] = capped(s[e], cap, cap_inv);
        }
        if (a.slopes) {
            const bool tree = key0 + TILE > v.first;
#pragma unroll
            for (uint32_t r = 0; r < 2; r++) {
                const uint32_t key = key0 + g + 8 * r;
                const float back = tree && sees(v, key) ? distance(a, v, key) : float(int(v.pos) - int(key));
#pragma unroll
                for (uint32_t e = 0; e < 2; e++) s[2 * r + e] = fmaf(-slope[e], back, s[2 * r + e]);
            }
        }
        if (key0 < v.lo || key0 + TILE > v.first) {
            if (!sees(v, key0 + g)) s[0] = s[1] = -INFINITY;
            if (!sees(v, key0 + g + 8)) s[2] = s[3] = -INFINITY;
        }
        // The running maximum only has to keep 2^(s - m) in range: it moves when a score exceeds it by more than 8.
        bool over = false;
#pragma unroll
        for (int e = 0; e < 2; e++) over = over || fmaxf(s[e], s[e + 2]) > m_run[e] + 8.0f;
        if (__any_sync(0xffffffffu, over)) {
#pragma unroll
            for (int e = 0; e < 2; e++) {
                float mx = fmaxf(s[e], s[e + 2]);
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
                const float m_new = fmaxf(m_run[e], mx), corr = fast_exp2(m_run[e] - (m_new == -INFINITY ? 0.0f : m_new));
                m_run[e] = m_new;
                l_run[e] *= corr;
#pragma unroll
                for (uint32_t dm = 0; dm < DM; dm++) {
                    o[dm][e] *= corr;
                    o[dm][e + 2] *= corr;
                }
            }
        }
        const float m0 = m_run[0] == -INFINITY ? 0.0f : m_run[0], m1 = m_run[1] == -INFINITY ? 0.0f : m_run[1];
        const float p0a = fast_exp2(s[0] - m0), p0b = fast_exp2(s[1] - m1), p1a = fast_exp2(s[2] - m0), p1b = fast_exp2(s[3] - m1);
        l_run[0] += p0a + p1a;
        l_run[1] += p0b + p1b;
        const uint32_t pb0 = movmatrix_trans(pack_bf16(p0a, p0b)), pb1 = movmatrix_trans(pack_bf16(p1a, p1b));
#pragma unroll
        for (uint32_t dm = 0; dm < DM; dm++) {
            uint32_t va[4];
            ldmatrix_x4_trans(va, vbase + v_row + (((2 * dm + v_c) ^ lr) << 4));
            mma16816(o[dm], va, pb0, pb1);
        }
        __syncwarp();  // every lane is done with the stage before it is refilled
        if (i + STAGES < my) issue(i + STAGES);
        cp_async_commit();
    }
    cp_async_wait<0>();
#pragma unroll
    for (int e = 0; e < 2; e++) {
        l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 4);
        l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 8);
        l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 16);
    }
    // The warps' sums meet in shared memory (the rings are free now); warp w finishes columns w and w + 4.
    __syncthreads();
    constexpr uint32_t OS = DV + 4;
    float *ms = reinterpret_cast<float*>(smem), *ls = ms + WARPS * 8, *os = ls + WARPS * 8;
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const uint32_t col = 2 * tq + e;
        if (g == 0) {
            ms[warp * 8 + col] = m_run[e];
            ls[warp * 8 + col] = l_run[e];
        }
#pragma unroll
        for (uint32_t dm = 0; dm < DM; dm++) {
            os[(warp * 8 + col) * OS + 16 * dm + g] = o[dm][e];
            os[(warp * 8 + col) * OS + 16 * dm + g + 8] = o[dm][e + 2];
        }
    }
    __syncthreads();
    constexpr uint32_t PER = DV / 32;  // dims per lane: lane, lane + 32, ...
    float mm[2], ll[2], oo[2][PER];
#pragma unroll
    for (uint32_t c2 = 0; c2 < 2; c2++) {
        const uint32_t col = warp + 4 * c2;
        mm[c2] = fmaxf(fmaxf(ms[col], ms[8 + col]), fmaxf(ms[16 + col], ms[24 + col]));
        ll[c2] = 0.0f;
#pragma unroll
        for (uint32_t j = 0; j < PER; j++) oo[c2][j] = 0.0f;
#pragma unroll
        for (uint32_t k = 0; k < WARPS; k++) {
            const float mk = ms[k * 8 + col], wk = mk == -INFINITY ? 0.0f : fast_exp2(mk - mm[c2]);
            ll[c2] += ls[k * 8 + col] * wk;
#pragma unroll
            for (uint32_t j = 0; j < PER; j++) oo[c2][j] += os[(k * 8 + col) * OS + lane + 32 * j] * wk;
        }
    }
    if (gridDim.z > 1) {
        // The cluster meets in its first block's shared memory, [rank][column][m, l, o]: the first barrier says that every
        // block has read its own sums out of it, the second that every partial has arrived. All threads reach both.
        cluster_sync();
#pragma unroll
        for (uint32_t c2 = 0; c2 < 2; c2++) {
            const uint32_t dst = cluster_addr(smem_u32(smem) + (sp * 8 + warp + 4 * c2) * OS * 4, 0);
            if (lane == 0) {
                asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(mm[c2]) : "memory");
                asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst + 4), "f"(ll[c2]) : "memory");
            }
#pragma unroll
            for (uint32_t j = 0; j < PER; j++) asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst + (4 + lane + 32 * j) * 4), "f"(oo[c2][j]) : "memory");
        }
        cluster_sync();
        if (sp) return;
        const float* recv = reinterpret_cast<const float*>(smem);
#pragma unroll
        for (uint32_t c2 = 0; c2 < 2; c2++) {
            const uint32_t col = warp + 4 * c2;
            mm[c2] = -INFINITY;
            ll[c2] = 0.0f;
            for (uint32_t k = 0; k < gridDim.z; k++) mm[c2] = fmaxf(mm[c2], recv[(k * 8 + col) * OS]);
#pragma unroll
            for (uint32_t j = 0; j < PER; j++) oo[c2][j] = 0.0f;
            for (uint32_t k = 0; k < gridDim.z; k++) {
                const float* pk = recv + (k * 8 + col) * OS;
                const float wk = pk[0] == -INFINITY ? 0.0f : fast_exp2(pk[0] - mm[c2]);
                ll[c2] += pk[1] * wk;
#pragma unroll
                for (uint32_t j = 0; j < PER; j++) oo[c2][j] += pk[4 + lane + 32 * j] * wk;
            }
        }
    }
#pragma unroll
    for (uint32_t c2 = 0; c2 < 2; c2++) {
        const uint32_t col = warp + 4 * c2;
        if (col >= cols) continue;
#pragma unroll
        for (uint32_t j = 0; j < PER; j++) {
            const uint32_t c = lane + 32 * j;
            float y = oo[c2][j] / ll[c2];
            if (a.gate) y = gated(y, a.gate[size_t(t) * a.ldg + (h0 + col) * DV + c]);
            const size_t at = (size_t(t) * a.heads + h0 + col) * DV + c;
            if (a.out) a.out[at] = y;
            a.out_b[at] = f32_to_bf16(y);
        }
    }
}

constexpr uint32_t CK = PAGE, GROUPS = 2;
template <uint32_t DK, uint32_t DV>
constexpr uint32_t prefill_stages() { return DK + DV > 128 ? 2 : 3; }
template <uint32_t DK, uint32_t DV>
constexpr uint32_t prefill_smem() { return GROUPS * prefill_stages<DK, DV>() * CK * (DK + DV) * 2; }

// grid (chunk tiles, query heads), 256 threads: warp w of a group has rows 16 w .. 16 w + 15 of the tile. SLOPES: with a.slopes.
template <uint32_t DK, uint32_t DV, bool SLOPES>
__global__ void __launch_bounds__(GROUPS * WARPS * 32) chunk_prefill_kernel(const ChunkedAttnArgs a) {
    pdl_start();
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr uint32_t KB = CK * DK * 2, VB = CK * DV * 2, KS = DK / 16, ND = DV / 8, KC = DK / 8, VC = DV / 8, ST = prefill_stages<DK, DV>();
    __shared__ uint32_t lows[WARPS], ends[WARPS];
    static_assert(64 * (DV + 4) * 4 <= prefill_smem<DK, DV>() / GROUPS, "the second group's sums must fit in a ring");
    const uint32_t tile = blockIdx.x, h = blockIdx.y, kvh = h / (a.heads / a.kv.n_kv);
    const uint32_t grp = threadIdx.x / (WARPS * 32), tid = threadIdx.x % (WARPS * 32), warp = tid / 32, lane = tid % 32, g = lane >> 2, tq = lane & 3;
    const uint32_t t0 = a.ctiles[2 * tile], rows = a.ctiles[2 * tile + 1];
    const float cap = a.softcap * LOG2E, cap_inv = 2.0f / a.softcap;
    uint32_t tok[2], low = 0xffffffffu, end = 0;
    bool live[2];
    View v[2];
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const uint32_t row = warp * 16 + g + 8 * r;
        live[r] = row < rows;
        tok[r] = t0 + (live[r] ? row : 0);
        v[r] = view_of(a, tok[r]);
        if (live[r]) {
            low = min(low, v[r].lo);
            end = max(end, v[r].first + 32 - __clz(v[r].mask));
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        low = min(low, __shfl_xor_sync(0xffffffffu, low, o));
        end = max(end, __shfl_xor_sync(0xffffffffu, end, o));
    }
    if (lane == 0 && grp == 0) { lows[warp] = low; ends[warp] = end; }
    __syncthreads();
    const Tiles<CK> walk(min(min(lows[0], lows[1]), min(lows[2], lows[3])), a.keep);
    const uint32_t b0 = grp, b1 = walk.count(max(max(ends[0], ends[1]), max(ends[2], ends[3])));
    const float slope = SLOPES ? a.slopes[h] * LOG2E : 0.0f;

    const uint32_t* pages = a.kv.page_table + size_t(v[0].slot) * a.kv.max_pages;
    const uint16_t* K = static_cast<const uint16_t*>(a.kv.k);
    const uint16_t* V = static_cast<const uint16_t*>(a.kv.v);
    const uint32_t ring = smem_u32(smem) + grp * ST * (KB + VB);
    auto group_sync = [&] { asm volatile("bar.sync %0, %1;" ::"r"(1 + grp), "n"(WARPS * 32) : "memory"); };
    auto issue = [&](uint32_t b) {  // a page of keys
        const size_t r0 = (size_t(pages[walk.at(b)]) * a.kv.n_kv + kvh) << PAGE_SHIFT;
        const uint32_t dst = ring + (b - b0) / GROUPS % ST * (KB + VB);
#pragma unroll
        for (uint32_t c = tid; c < CK * KC; c += WARPS * 32) {
            const uint32_t key = c / KC, piece = c % KC;
            cp_async16(dst + key * DK * 2 + ((piece ^ (key & 7)) << 4), K + (r0 + key) * DK + piece * 8);
        }
#pragma unroll
        for (uint32_t c = tid; c < CK * VC; c += WARPS * 32) {
            const uint32_t key = c / VC, piece = c % VC;
            cp_async16(dst + KB + key * DV * 2 + ((piece ^ (key & 7)) << 4), V + (r0 + key) * DV + piece * 8);
        }
    };
#pragma unroll
    for (uint32_t i = 0; i < ST; i++) {
        if (b0 + i * GROUPS < b1) issue(b0 + i * GROUPS);
        cp_async_commit();
    }
    uint32_t qa[KS][4];
    {
        const uint32_t* q32 = reinterpret_cast<const uint32_t*>(a.q_b);
#pragma unroll
        for (uint32_t ks = 0; ks < KS; ks++) {
            const size_t r0 = (size_t(tok[0]) * a.heads + h) * (DK / 2) + 8 * ks + tq, r1 = (size_t(tok[1]) * a.heads + h) * (DK / 2) + 8 * ks + tq;
            qa[ks][0] = live[0] ? q32[r0] : 0u;
            qa[ks][1] = live[1] ? q32[r1] : 0u;
            qa[ks][2] = live[0] ? q32[r0 + 4] : 0u;
            qa[ks][3] = live[1] ? q32[r1 + 4] : 0u;
        }
    }
    const uint32_t lm = lane >> 3, lr = lane & 7;
    float o[ND][4], m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
#pragma unroll
    for (uint32_t j = 0; j < ND; j++) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.0f;
    const uint32_t lo_max = max(v[0].lo, v[1].lo), first_min = min(v[0].first, v[1].first);
    for (uint32_t b = b0; b < b1; b += GROUPS) {
        cp_async_wait<ST - 1>();
        group_sync();  // everybody's copies of the page are in
        const uint32_t kbase = ring + (b - b0) / GROUPS % ST * (KB + VB), vbase = kbase + KB, key0 = walk.at(b) * CK;
        if (key0 < ends[warp] && (key0 + CK > lows[warp] || key0 < a.keep)) {  // (a warp whose rows see nothing of the page skips the arithmetic, not the barriers)
            float s[8][4];
#pragma unroll
            for (uint32_t j = 0; j < 8; j++) {
                s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
                const uint32_t kaddr = kbase + (8 * j + lr) * DK * 2;
#pragma unroll
                for (uint32_t kp = 0; kp < KS / 2; kp++) {
                    uint32_t kb[4];
                    ldmatrix_x4(kb, kaddr + (((4 * kp + lm) ^ lr) << 4));
                    mma16816(s[j], qa[2 * kp], kb[0], kb[1]);
                    mma16816(s[j], qa[2 * kp + 1], kb[2], kb[3]);
                }
            }
            if (a.softcap > 0) {
#pragma unroll
                for (uint32_t j = 0; j < 8; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) s[j][e] = capped(s[j][e], cap, cap_inv);
            }
            if (SLOPES) {
                const bool tree = key0 + CK > first_min;
#pragma unroll
                for (uint32_t j = 0; j < 8; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const View& w = v[e >> 1];
                        const uint32_t key = key0 + 8 * j + 2 * tq + (e & 1);
                        const float back = tree && key >= w.first && live[e >> 1] && sees(w, key) ? distance(a, w, key) : float(int(w.pos) - int(key));
                        s[j][e] = fmaf(-slope, back, s[j][e]);
                    }
            }
            if (key0 < lo_max || key0 + CK > first_min || !live[0] || !live[1]) {
#pragma unroll
                for (uint32_t j = 0; j < 8; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++)
                        if (!live[e >> 1] || !sees(v[e >> 1], key0 + 8 * j + 2 * tq + (e & 1))) s[j][e] = -INFINITY;
            }
            float corr[2];
#pragma unroll
            for (int r = 0; r < 2; r++) {
                float mx = -INFINITY;
#pragma unroll
                for (uint32_t j = 0; j < 8; j++) mx = fmaxf(mx, fmaxf(s[j][2 * r], s[j][2 * r + 1]));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                const float m_new = fmaxf(m_run[r], mx), m_use = m_new == -INFINITY ? 0.0f : m_new;
                corr[r] = fast_exp2(m_run[r] - m_use);
                m_run[r] = m_new;
                float sum = 0.0f;
#pragma unroll
                for (uint32_t j = 0; j < 8; j++) {
                    s[j][2 * r] = fast_exp2(s[j][2 * r] - m_use);
                    s[j][2 * r + 1] = fast_exp2(s[j][2 * r + 1] - m_use);
                    sum += s[j][2 * r] + s[j][2 * r + 1];
                }
                l_run[r] = l_run[r] * corr[r] + sum;
            }
#pragma unroll
            for (uint32_t j = 0; j < ND; j++) {
                o[j][0] *= corr[0];
                o[j][1] *= corr[0];
                o[j][2] *= corr[1];
                o[j][3] *= corr[1];
            }
#pragma unroll
            for (uint32_t kk = 0; kk < 4; kk++) {
                uint32_t pa[4];
                pa[0] = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
                pa[1] = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
                pa[2] = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
                pa[3] = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
                const uint32_t vaddr = vbase + (16 * kk + 8 * (lm & 1) + lr) * DV * 2;
#pragma unroll
                for (uint32_t dp = 0; dp < DV / 16; dp++) {
                    uint32_t vb[4];
                    ldmatrix_x4_trans(vb, vaddr + (((2 * dp + (lm >> 1)) ^ lr) << 4));
                    mma16816(o[2 * dp], pa, vb[0], vb[1]);
                    mma16816(o[2 * dp + 1], pa, vb[2], vb[3]);
                }
            }
        }
        group_sync();  // every warp of the group is done with the stage
        if (b + ST * GROUPS < b1) issue(b + ST * GROUPS);
        cp_async_commit();
    }
    cp_async_wait<0>();
#pragma unroll
    for (int r = 0; r < 2; r++) {
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    }
    // The second group's (m, l, o) to the first through its own ring: a row's o, then m and l.
    constexpr uint32_t OS = DV + 4;
    float* sums = reinterpret_cast<float*>(smem + ST * (KB + VB));
    if (grp) {
#pragma unroll
        for (int r = 0; r < 2; r++) {
            float* row = sums + (warp * 16 + g + 8 * r) * OS;
#pragma unroll
            for (uint32_t j = 0; j < ND; j++) *reinterpret_cast<float2*>(row + 8 * j + 2 * tq) = make_float2(o[j][2 * r], o[j][2 * r + 1]);
            if (tq == 0) { row[DV] = m_run[r]; row[DV + 1] = l_run[r]; }
        }
    }
    __syncthreads();
    if (grp) return;
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const float* row = sums + (warp * 16 + g + 8 * r) * OS;
        const float m1 = row[DV], m = fmaxf(m_run[r], m1), w0 = m_run[r] == -INFINITY ? 0.0f : fast_exp2(m_run[r] - m), w1 = m1 == -INFINITY ? 0.0f : fast_exp2(m1 - m);
        const float l = l_run[r] * w0 + row[DV + 1] * w1;
#pragma unroll
        for (uint32_t j = 0; j < ND; j++) {
            const float2 other = *reinterpret_cast<const float2*>(row + 8 * j + 2 * tq);
            o[j][2 * r] = o[j][2 * r] * w0 + other.x * w1;
            o[j][2 * r + 1] = o[j][2 * r + 1] * w0 + other.y * w1;
        }
        if (!live[r]) continue;
        const float inv = l > 0.0f ? 1.0f / l : 0.0f;
        const size_t at = (size_t(tok[r]) * a.heads + h) * DV;
        const float* gate = a.gate ? a.gate + size_t(tok[r]) * a.ldg + h * DV : nullptr;
#pragma unroll
        for (uint32_t j = 0; j < ND; j++) {
            const uint32_t c = 8 * j + 2 * tq;
            float x = o[j][2 * r] * inv, y = o[j][2 * r + 1] * inv;
            if (gate) { x = gated(x, gate[c]); y = gated(y, gate[c + 1]); }
            if (a.out) { a.out[at + c] = x; a.out[at + c + 1] = y; }
            *reinterpret_cast<uint32_t*>(a.out_b + at + c) = pack_bf16(x, y);
        }
    }
}

template <uint32_t DK, uint32_t DV>
void launch(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t splits, cudaStream_t s) {
    static PerDevice configured;
    constexpr uint32_t dsm = decode_smem<DK, DV>(), psm = prefill_smem<DK, DV>();
    configured.once([] {
        VLT_CUDA(cudaFuncSetAttribute(chunk_decode_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(dsm)));
        VLT_CUDA(cudaFuncSetAttribute(chunk_decode_kernel<DK, DV>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
        for (auto f : {chunk_prefill_kernel<DK, DV, false>, chunk_prefill_kernel<DK, DV, true>}) VLT_CUDA(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, int(psm)));
    });
    if (n_ctiles) {
        launch_pdl(a.slopes ? chunk_prefill_kernel<DK, DV, true> : chunk_prefill_kernel<DK, DV, false>, dim3(n_ctiles, a.heads), GROUPS * WARPS * 32, psm, s, a);
        return;
    }
    const uint32_t groups = (a.heads / a.kv.n_kv + 7) / 8;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(n, a.kv.n_kv * groups, splits);
    cfg.blockDim = dim3(WARPS * 32);
    cfg.dynamicSmemBytes = dsm;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = splits;
    cfg.attrs = attr;
    cfg.numAttrs = splits > 1 ? 2 : 1;
    VLT_CUDA(cudaLaunchKernelEx(&cfg, chunk_decode_kernel<DK, DV>, a));
    launch_counter()++;
}

}  // namespace chunked

bool chunk_attn_fits(uint32_t dk, uint32_t dv, uint32_t page) { return (dk == 64 || dk == 128) && (dv == 64 || dv == 128) && page == chunked::PAGE; }

// n_ctiles: tiles of at most 64 rows, if the step holds a run longer than a verified one (then every row goes by tile);
// max_keys: the most keys a row may see; keys_per_block overrides the split.
void launch_attn_chunked(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t max_keys, uint32_t sm_count, uint32_t keys_per_block, cudaStream_t s) {
    if (a.sink) throw Error("internal: attention over chunks has no sinks");
    // A row's keys over at most 8 blocks, or 16 where 8 leave most SMs idle: the count that makes waves of blocks (three an SM) times a block's keys, plus a
    // fixed part of about 128 keys' worth, least.
    const uint32_t units = std::max(n * a.kv.n_kv * ((a.heads / a.kv.n_kv + 7) / 8), 1u), slots = 3 * sm_count;
    uint32_t splits = 1;
    uint64_t best = ~0ull;
    const uint32_t most = units * 16 <= sm_count ? chunked::MAX_SPLITS : 8;
    for (uint32_t c = 1; c <= most && (c == 1 || max_keys / c >= 64); c++) {
        const uint64_t cost = uint64_t((units * c + slots - 1) / slots) * ((max_keys + c - 1) / c + 128);
        if (cost < best) { best = cost; splits = c; }
    }
    if (keys_per_block) splits = std::max(1u, std::min(chunked::MAX_SPLITS, (max_keys + keys_per_block - 1) / keys_per_block));
    if (a.kv.dk == 64 && a.kv.dv == 64) chunked::launch<64, 64>(a, n, n_ctiles, splits, s);
    else if (a.kv.dk == 64) chunked::launch<64, 128>(a, n, n_ctiles, splits, s);
    else if (a.kv.dv == 64) chunked::launch<128, 64>(a, n, n_ctiles, splits, s);
    else chunked::launch<128, 128>(a, n, n_ctiles, splits, s);
}

}  // namespace vlt
