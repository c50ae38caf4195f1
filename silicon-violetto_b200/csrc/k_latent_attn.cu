// Latent attention over paged rows (c ; r) on the tensor cores (sizes it does not take and fp32 caches: k_mixer.cu's scalar kernel).
// All query heads read one row per position, whose first part is the value as well: what a row costs to fetch is shared by as
// many (token, head) rows as a block holds.
//
//   A block has 16, 32 or 64 (token, head) rows of one run -- decoding, a token's heads; a prompt's portion, the heads of several
//   neighbouring tokens -- and goes through its share of the run's pages 32 positions at a time, which asynchronous copies bring
//   into a ring. Eight warps split the scores by rows and positions (16 rows: also by the columns they sum over), meet in shared
//   memory for the softmax in fp32, and split the sums of c by rows and columns. A row's positions may be split over a cluster of
//   blocks, each of which finishes a span of the columns from what the others store into its shared memory.
//
// It takes q with scale * log2(e) folded in, rounded to bf16, and leaves the sums in bf16 for the per-head product after it.
#include <algorithm>

#include "paged_attn.cuh"

namespace vlt {

namespace latent {

using namespace paged;

constexpr uint32_t WARPS = 8, THREADS = WARPS * 32, KT = 32, EXTRA = 64, MAX_SPLITS = 16;  // EXTRA: room for the rotated part behind R columns

// R: columns of c a block is laid out for; ROWS: its (token, head) rows.
template <uint32_t R, uint32_t ROWS>
struct Shape {
    static constexpr uint32_t WIDTH = R + EXTRA, PITCH = WIDTH * 2 + 16, STAGE = KT * PITCH;           // a staged row; bytes that keep ldmatrix free of conflicts
    static constexpr uint32_t RG = ROWS / 16, KG = RG == 4 ? 2 : 4, KH = WARPS / (RG * KG);             // row groups, key groups, parts of the columns
    static constexpr uint32_t NT = KT / KG / 8;                                                         // scores: tiles of 8 keys of a warp
    static constexpr uint32_t CG = WARPS / RG, CW = R / CG < 16 ? 16 : R / CG;                          // sums: column groups, columns of a warp
    static constexpr uint32_t STAGES = ROWS == 16 ? 5 : ROWS == 32 ? 4 : 3;
    static constexpr uint32_t TPR = THREADS / ROWS, KPT = KT / TPR, SP = KT + 4, PP = KT + 8;           // softmax: threads of a row, keys of a thread; pitches
    static constexpr uint32_t O_Q = STAGES * STAGE, O_S = O_Q + ROWS * PITCH, O_P = O_S + KH * ROWS * SP * 4, O_STAT = O_P + ROWS * PP * 2;
    static constexpr uint32_t BYTES = O_STAT + ROWS * 12 + MAX_SPLITS * ROWS * 8;
    static_assert(ROWS * R * 4 <= O_STAT, "the cluster's sums must fit in front of the statistics");
    static_assert(BYTES <= 227 * 1024, "shared memory");
};

// grid (tiles, 1, key splits). Prompts (sub > 0): tile = (chunk tile, one of its `sub` spans of `toks` tokens, group of ROWS heads); else
// (token, group).
template <uint32_t R, uint32_t ROWS>
__global__ void __launch_bounds__(THREADS, 1) latent_kernel(const ChunkedAttnArgs a, uint32_t groups, uint32_t sub, uint32_t toks) {
    pdl_start();
    using S = Shape<R, ROWS>;
    extern __shared__ __align__(1024) uint8_t smem[];
    __shared__ uint32_t end_s;
    const uint32_t tid = threadIdx.x, warp = tid / 32, lane = tid % 32, g = lane >> 2, tq = lane & 3, lm = lane >> 3, lr = lane & 7;
    const uint32_t grp = blockIdx.x % groups, unit = blockIdx.x / groups, sp = blockIdx.z, splits = gridDim.z;
    uint32_t t0 = unit, n_tok = 1;
    if (sub) {
        const uint32_t tile = unit / sub, at = unit % sub * toks, rows = a.ctiles[2 * tile + 1];
        if (at >= rows) return;  // (all of a cluster's blocks together)
        t0 = a.ctiles[2 * tile] + at;
        n_tok = min(toks, rows - at);
    }
    const uint32_t hpt = min(a.heads, ROWS), dk = a.kv.dk, rank = a.kv.dv;
    auto row_at = [&](uint32_t r, uint32_t& tok, uint32_t& head) {  // whether row r of the tile exists
        tok = t0 + r / hpt;
        head = grp * ROWS + r % hpt;
        return r / hpt < n_tok && head < a.heads;
    };
    // The softmax's row of this thread.
    const uint32_t my_row = tid / S::TPR, my_key = tid % S::TPR * S::KPT;
    uint32_t my_tok, my_head;
    const bool live = row_at(my_row, my_tok, my_head);
    const View v = view_of(a, live ? my_tok : t0);
    if (tid == 0) end_s = 0;
    __syncthreads();
    if (live && tid % S::TPR == 0) atomicMax(&end_s, v.first + 32 - __clz(v.mask));
    // The query rows, zeros where there are none, and zeros behind the staged rows' ends (no copy writes there).
    const uint32_t pieces = dk / 8, whole = S::WIDTH / 8;
    for (uint32_t i = tid; i < ROWS * whole; i += THREADS) {
        const uint32_t r = i / whole, c = i % whole;
        uint32_t tok, head;
        uint4 x = make_uint4(0, 0, 0, 0);
        if (row_at(r, tok, head) && c < pieces) x = reinterpret_cast<const uint4*>(a.q_b + (size_t(tok) * a.heads + head) * dk)[c];
        *reinterpret_cast<uint4*>(smem + S::O_Q + r * S::PITCH + c * 16) = x;
    }
    for (uint32_t i = tid; i < S::STAGES * KT * (whole - pieces); i += THREADS)
        *reinterpret_cast<uint4*>(smem + i / (whole - pieces) * S::PITCH + (pieces + i % (whole - pieces)) * 16) = make_uint4(0, 0, 0, 0);
    __syncthreads();
    const uint32_t tiles = (end_s + KT - 1) / KT, share = (tiles + splits - 1) / splits, begin = min(sp * share, tiles), n = min(share, tiles - begin);

    const uint32_t* pages = a.kv.page_table + size_t(v.slot) * a.kv.max_pages;
    const uint16_t* K = static_cast<const uint16_t*>(a.kv.k);
    const uint32_t base = smem_u32(smem);
    auto issue = [&](uint32_t i) {
        const uint32_t key0 = (begin + i) * KT;
        const uint16_t* src = K + ((size_t(pages[key0 >> PAGE_SHIFT]) << PAGE_SHIFT) + (key0 & (PAGE - 1))) * dk;
        const uint32_t dst = base + i % S::STAGES * S::STAGE;
        uint32_t key = tid / pieces, c = tid % pieces;
        const uint32_t dkey = THREADS / pieces, dc = THREADS % pieces;
        while (key < KT) {
            cp_async16(dst + key * S::PITCH + c * 16, src + size_t(key) * dk + c * 8);
            key += dkey;
            c += dc;
            if (c >= pieces) { c -= pieces; key++; }
        }
    };
#pragma unroll
    for (uint32_t i = 0; i < S::STAGES - 1; i++) {
        if (i < n) issue(i);
        cp_async_commit();
    }
    float *scores = reinterpret_cast<float*>(smem + S::O_S), *corr_s = reinterpret_cast<float*>(smem + S::O_STAT), *m_s = corr_s + ROWS, *l_s = m_s + ROWS;
    uint16_t* probs = reinterpret_cast<uint16_t*>(smem + S::O_P);
    const uint32_t rg = warp % S::RG, kg = warp / S::RG % S::KG, kh = warp / (S::RG * S::KG), cg = warp / S::RG, col0 = cg * S::CW;
    const bool sums = col0 < R;
    float o[S::CW / 8][4], m_run = -INFINITY, l_run = 0.0f;
#pragma unroll
    for (uint32_t j = 0; j < S::CW / 8; j++) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.0f;
    const uint32_t q_addr = base + S::O_Q + (rg * 16 + lane % 16) * S::PITCH + lane / 16 * 16, p_addr = base + S::O_P + ((rg * 16 + lane % 16) * S::PP + lane / 16 * 8) * 2;
    const float cap = a.softcap * LOG2E, cap_inv = 2.0f / a.softcap;
    for (uint32_t i = 0; i < n; i++) {
        cp_async_wait<S::STAGES - 2>();
        __syncthreads();  // everybody's copies of the tile are in, and everybody is done with the tile before
        if (i + S::STAGES - 1 < n) issue(i + S::STAGES - 1);
        cp_async_commit();
        const uint32_t stage = base + i % S::STAGES * S::STAGE, key0 = (begin + i) * KT;
        {
            float s[S::NT][2][4];
#pragma unroll
            for (uint32_t j = 0; j < S::NT; j++)
#pragma unroll
                for (uint32_t e = 0; e < 4; e++) s[j][0][e] = s[j][1][e] = 0.0f;
            constexpr uint32_t PAIRS = S::WIDTH / 32 / S::KH;  // pairs of 16 columns
            const uint32_t k_addr = stage + (kg * S::NT * 8 + lr) * S::PITCH + lm * 16 + kh * PAIRS * 64, qa = q_addr + kh * PAIRS * 64;
#pragma unroll 6
            for (uint32_t kp = 0; kp < PAIRS; kp++) {
                uint32_t a0[4], a1[4];
                ldmatrix_x4(a0, qa + kp * 64);
                ldmatrix_x4(a1, qa + kp * 64 + 32);
#pragma unroll
                for (uint32_t j = 0; j < S::NT; j++) {
                    uint32_t kb[4];
                    ldmatrix_x4(kb, k_addr + j * 8 * S::PITCH + kp * 64);
                    mma16816(s[j][0], a0, kb[0], kb[1]);
                    mma16816(s[j][1], a1, kb[2], kb[3]);
                }
            }
            float* dst = scores + (kh * ROWS + rg * 16 + g) * S::SP + kg * S::NT * 8 + 2 * tq;
#pragma unroll
            for (uint32_t j = 0; j < S::NT; j++) {
                *reinterpret_cast<float2*>(dst + 8 * j) = make_float2(s[j][0][0] + s[j][1][0], s[j][0][1] + s[j][1][1]);
                *reinterpret_cast<float2*>(dst + 8 * S::SP + 8 * j) = make_float2(s[j][0][2] + s[j][1][2], s[j][0][3] + s[j][1][3]);
            }
        }
        __syncthreads();
        {
            float s[S::KPT], mx = -INFINITY;
#pragma unroll
            for (uint32_t e = 0; e < S::KPT; e++) {
                s[e] = scores[my_row * S::SP + my_key + e];
                if (S::KH == 2) s[e] += scores[(ROWS + my_row) * S::SP + my_key + e];
                if (a.softcap > 0) s[e] = capped(s[e], cap, cap_inv);
                const uint32_t key = key0 + my_key + e;
                if (!live || (key >= v.first && !sees(v, key))) s[e] = -INFINITY;
                mx = fmaxf(mx, s[e]);
            }
#pragma unroll
            for (uint32_t x = 1; x < S::TPR; x *= 2) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
            // The running maximum only has to keep 2^(s - m) in range: it moves when a score exceeds it by more than 8.
            float corr = 1.0f;
            if (mx > m_run + 8.0f) {
                corr = fast_exp2(m_run - mx);  // (0 from -infinity)
                m_run = mx;
            }
            const float m = m_run == -INFINITY ? 0.0f : m_run;
            float sum = 0.0f;
            uint32_t packed[S::KPT / 2];
#pragma unroll
            for (uint32_t e = 0; e < S::KPT; e += 2) {
                const float p0 = fast_exp2(s[e] - m), p1 = fast_exp2(s[e + 1] - m);
                sum += p0 + p1;
                packed[e / 2] = pack_bf16(p0, p1);
                *reinterpret_cast<uint32_t*>(probs + my_row * S::PP + my_key + e) = packed[e / 2];
            }
            l_run = l_run * corr + sum;
            if (tid % S::TPR == 0) corr_s[my_row] = corr;
        }
        __syncthreads();
        const float c0 = corr_s[rg * 16 + g], c1 = corr_s[rg * 16 + g + 8];
        if (__any_sync(0xffffffffu, c0 != 1.0f || c1 != 1.0f)) {
#pragma unroll
            for (uint32_t j = 0; j < S::CW / 8; j++) {
                o[j][0] *= c0;
                o[j][1] *= c0;
                o[j][2] *= c1;
                o[j][3] *= c1;
            }
        }
        if (sums) {
            uint32_t pa[KT / 16][4];
#pragma unroll
            for (uint32_t kk = 0; kk < KT / 16; kk++) ldmatrix_x4(pa[kk], p_addr + kk * 32);
            const uint32_t v_addr = stage + (8 * (lm & 1) + lr) * S::PITCH + (col0 + 8 * (lm >> 1)) * 2;
#pragma unroll
            for (uint32_t dp = 0; dp < S::CW / 16; dp++)
#pragma unroll
                for (uint32_t kk = 0; kk < KT / 16; kk++) {
                    uint32_t vb[4];
                    ldmatrix_x4_trans(vb, v_addr + kk * 16 * S::PITCH + dp * 32);
                    mma16816(o[2 * dp], pa[kk], vb[0], vb[1]);
                    mma16816(o[2 * dp + 1], pa[kk], vb[2], vb[3]);
                }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (uint32_t x = 1; x < S::TPR; x *= 2) l_run += __shfl_xor_sync(0xffffffffu, l_run, x);
    if (splits == 1) {
        if (tid % S::TPR == 0) l_s[my_row] = l_run;
        __syncthreads();
        if (!sums) return;
#pragma unroll
        for (uint32_t r = 0; r < 2; r++) {
            const uint32_t row = rg * 16 + g + 8 * r;
            uint32_t tok, head;
            if (!row_at(row, tok, head)) continue;
            const float inv = 1.0f / l_s[row];
            const size_t at = (size_t(tok) * a.heads + head) * rank;
#pragma unroll
            for (uint32_t j = 0; j < S::CW / 8; j++) {
                const uint32_t c = col0 + 8 * j + 2 * tq;
                if (c < rank) *reinterpret_cast<uint32_t*>(a.out_b + at + c) = pack_bf16(o[j][2 * r] * inv, o[j][2 * r + 1] * inv);
            }
        }
        return;
    }
    // The cluster: block b finishes columns b R / splits on. [source][row][column of the span] in front of the statistics, (m, l) per
    // (source, row) behind them. The first barrier: every block is done with its ring; the second: every partial has arrived.
    cluster_sync();
    const uint32_t span = R / splits, ml = S::O_STAT + ROWS * 12;
    if (tid % S::TPR == 0)
        for (uint32_t b = 0; b < splits; b++) {
            const uint32_t dst = cluster_addr(base + ml + (sp * ROWS + my_row) * 8, b);
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(m_run) : "memory");
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst + 4), "f"(l_run) : "memory");
        }
    if (sums) {
#pragma unroll
        for (uint32_t j = 0; j < S::CW / 8; j++) {
            const uint32_t c = col0 + 8 * j + 2 * tq, owner = c / span;
            const uint32_t dst = cluster_addr(base + ((sp * ROWS + rg * 16 + g) * span + c % span) * 4, owner);
#pragma unroll
            for (uint32_t r = 0; r < 2; r++) {
                asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst + r * 8 * span * 4), "f"(o[j][2 * r]) : "memory");
                asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst + r * 8 * span * 4 + 4), "f"(o[j][2 * r + 1]) : "memory");
            }
        }
    }
    cluster_sync();
    const float *recv = reinterpret_cast<const float*>(smem), *stat = reinterpret_cast<const float*>(smem + ml);
    for (uint32_t i = tid; i < ROWS * span / 2; i += THREADS) {
        const uint32_t row = i / (span / 2), x = i % (span / 2) * 2, c = sp * span + x;
        uint32_t tok, head;
        if (!row_at(row, tok, head) || c >= rank) continue;
        float m = -INFINITY, l = 0.0f, y0 = 0.0f, y1 = 0.0f;
        for (uint32_t k = 0; k < splits; k++) m = fmaxf(m, stat[(k * ROWS + row) * 2]);
        for (uint32_t k = 0; k < splits; k++) {
            const float mk = stat[(k * ROWS + row) * 2], w = mk == -INFINITY ? 0.0f : fast_exp2(mk - m);
            const float2 y = *reinterpret_cast<const float2*>(recv + (k * ROWS + row) * span + x);
            l += stat[(k * ROWS + row) * 2 + 1] * w;
            y0 += y.x * w;
            y1 += y.y * w;
        }
        *reinterpret_cast<uint32_t*>(a.out_b + (size_t(tok) * a.heads + head) * rank + c) = pack_bf16(y0 / l, y1 / l);
    }
}

template <uint32_t R, uint32_t ROWS>
void launch(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t max_keys, uint32_t sm_count, uint32_t keys_per_block, cudaStream_t s) {
    using S = Shape<R, ROWS>;
    static PerDevice configured;
    configured.once([] {
        VLT_CUDA(cudaFuncSetAttribute(latent_kernel<R, ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(S::BYTES)));
        VLT_CUDA(cudaFuncSetAttribute(latent_kernel<R, ROWS>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    });
    const uint32_t groups = (a.heads + ROWS - 1) / ROWS, toks = n_ctiles ? std::max(1u, ROWS / a.heads) : 1, sub = n_ctiles ? (64 + toks - 1) / toks : 0;
    // A tile's positions over 1, 2, 4 or 8 blocks, or 16 where 8 leave most SMs idle: the count that makes waves of blocks (one an SM where
    // the ring is large) times a block's positions, plus a fixed part, least.
    const uint32_t units = std::max(1u, (n + toks - 1) / toks * groups), most = units * 16 <= sm_count ? MAX_SPLITS : 8;
    uint32_t splits = 1;
    uint64_t best = ~0ull;
    for (uint32_t c = 1; c <= most && (c == 1 || max_keys / c >= 64); c *= 2) {
        const uint64_t cost = uint64_t((units * c + sm_count - 1) / sm_count) * ((max_keys + c - 1) / c + 128);
        if (cost < best) { best = cost; splits = c; }
    }
    if (keys_per_block)
        for (splits = 1; splits < MAX_SPLITS && splits * keys_per_block < max_keys;) splits *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((sub ? n_ctiles * sub : n) * groups, 1, splits);
    cfg.blockDim = dim3(THREADS);
    cfg.dynamicSmemBytes = S::BYTES;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = splits;
    cfg.attrs = attr;
    cfg.numAttrs = splits > 1 ? 2 : 1;
    VLT_CUDA(cudaLaunchKernelEx(&cfg, latent_kernel<R, ROWS>, a, groups, sub, toks));
    launch_counter()++;
}
template <uint32_t R>
void by_rows(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t max_keys, uint32_t sm_count, uint32_t keys_per_block, cudaStream_t s) {
    if (n_ctiles || a.heads > 32) launch<R, 64>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, s);
    else if (a.heads > 16) launch<R, 32>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, s);
    else launch<R, 16>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, s);
}
static uint32_t columns(uint32_t rank) { return rank <= 64 ? 64 : rank <= 128 ? 128 : rank <= 256 ? 256 : 512; }

}  // namespace latent

bool latent_attn_fits(uint32_t kv_rank, uint32_t rot_dim, uint32_t page) {
    return page == paged::PAGE && kv_rank <= 512 && kv_rank % 8 == 0 && rot_dim % 8 == 0 && kv_rank + rot_dim <= latent::columns(kv_rank) + latent::EXTRA;
}
void launch_attn_latent(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t max_keys, uint32_t sm_count, uint32_t keys_per_block, cudaStream_t s) {
    switch (latent::columns(a.kv.dv)) {
    case 64: latent::by_rows<64>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, s); break;
    case 128: latent::by_rows<128>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, s); break;
    case 256: latent::by_rows<256>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, s); break;
    default: latent::by_rows<512>(a, n, n_ctiles, max_keys, sm_count, keys_per_block, s);
    }
}

}  // namespace vlt
