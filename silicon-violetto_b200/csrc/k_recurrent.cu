// Linear recurrences over a state per head, and what stands around them in a layer: the state space's short convolution with silu
// and its step sizes, time mixing's mixes of neighbouring rows and its decays, and the gated norm of the outputs.
//
// The recurrence S = D S + k v^T runs token by token in fp32, the state in registers: a block has 16 value channels of one head of
// one run; 8, 16 or 32 lanes share two or four value channels and hold four key channels (or a few times four) of each, in pairs
// for the packed fp32 instructions: what a lane reads of q, k and decays serves several columns. Rows come in by asynchronous
// copies, a chunk of tokens ahead; the output's sums over the lanes are taken for eight tokens at a time, by exchanges that halve
// what a lane carries. A prompt's portion reads and writes the state once, like a decoded token. A row's result depends on nothing
// but the rows before it, however they are cut into steps. (Longer portions of the state space's go to k_ssd.cu.)
#include <algorithm>

#include "kernels.h"

namespace vlt {

namespace recurrent {

constexpr uint32_t COLS = 16;  // value channels of a block; PC: of a thread

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ void cp_async4(float* dst, const float* src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(uint32_t(__cvta_generic_to_shared(dst))), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(uint32_t(__cvta_generic_to_shared(dst))), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// A thread's way through a matrix of `width` columns, `threads` elements at a time: one division where it begins.
struct Walk {
    uint32_t r, c, dr, dc, width;
    __device__ __forceinline__ Walk(uint32_t start, uint32_t threads, uint32_t w) : r(start / w), c(start % w), dr(threads / w), dc(threads % w), width(w) {}
    __device__ __forceinline__ void next() {
        r += dr;
        c += dc;
        if (c >= width) { c -= width; r++; }
    }
};

// A chunk of tokens in shared memory: q and k rows, decays (per channel or two numbers), values, the bonus.
template <bool CHANNEL>
__host__ __device__ constexpr uint32_t stage_floats(uint32_t np, uint32_t tokens) { return tokens * ((CHANNEL ? 3 : 2) * np + COLS + 4); }
struct Stage {
    float *q, *k, *w, *v, *s;  // s: [token][4]: key factor, decay | bonus
};
template <bool CHANNEL>
__device__ __forceinline__ Stage stage_at(float* base, uint32_t np, uint32_t tokens) {
    Stage st;
    st.q = base;
    st.k = st.q + tokens * np;
    st.w = st.k + tokens * np;
    st.v = CHANNEL ? st.w + tokens * np : st.w;
    st.s = st.v + tokens * COLS;
    return st;
}

// The state as a thread holds it: key channels 4 lane + 4 L i .. + 3 of PC neighbouring value channels, in two pairs each.
template <uint32_t NV, uint32_t PC>
struct State {
    float2 a[NV][PC], b[NV][PC];
    __device__ __forceinline__ void clear() {
#pragma unroll
        for (uint32_t i = 0; i < NV; i++)
#pragma unroll
            for (uint32_t c = 0; c < PC; c++) a[i][c] = b[i][c] = make_float2(0.0f, 0.0f);
    }
};
template <uint32_t L, uint32_t NV, uint32_t PC>
__device__ __forceinline__ void load_state(State<NV, PC>& S, const float* p, uint32_t cols) {  // cols: of the PC, those that exist
#pragma unroll
    for (uint32_t i = 0; i < NV; i++)
#pragma unroll
        for (uint32_t c = 0; c < PC; c++) {
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (c < cols) x = *reinterpret_cast<const float4*>(p + (c * NV + i) * 4 * L);
            S.a[i][c] = make_float2(x.x, x.y);
            S.b[i][c] = make_float2(x.z, x.w);
        }
}
template <uint32_t L, uint32_t NV, uint32_t PC>
__device__ __forceinline__ void store_state(const State<NV, PC>& S, float* p, uint32_t cols) {
#pragma unroll
    for (uint32_t i = 0; i < NV; i++)
#pragma unroll
        for (uint32_t c = 0; c < PC; c++)
            if (c < cols) *reinterpret_cast<float4*>(p + (c * NV + i) * 4 * L) = make_float4(S.a[i][c].x, S.a[i][c].y, S.b[i][c].x, S.b[i][c].y);
}

// What a lane reads of a token.
template <uint32_t NV, uint32_t PC, bool CHANNEL>
struct Token {
    float4 q[NV], k[NV], w[CHANNEL ? NV : 1];
    float v[PC];
    float2 step;
};
template <uint32_t L, uint32_t NV, uint32_t PC, bool CHANNEL>
__device__ __forceinline__ void load_token(Token<NV, PC, CHANNEL>& t, const Stage& st, uint32_t j, uint32_t lane, uint32_t col) {
    constexpr uint32_t NP = 4 * L * NV;
#pragma unroll
    for (uint32_t i = 0; i < NV; i++) {
        const uint32_t at = j * NP + 4 * lane + 4 * L * i;
        t.q[i] = *reinterpret_cast<const float4*>(st.q + at);
        t.k[i] = *reinterpret_cast<const float4*>(st.k + at);
        if constexpr (CHANNEL) t.w[i] = *reinterpret_cast<const float4*>(st.w + at);
    }
    if constexpr (PC == 4) {
        load_f32<4>(t.v, st.v + j * COLS + col);
    } else {
        const float2 v2 = *reinterpret_cast<const float2*>(st.v + j * COLS + col);
        t.v[0] = v2.x;
        t.v[1] = v2.y;
    }
    if constexpr (!CHANNEL) t.step = *reinterpret_cast<const float2*>(st.s + 4 * j);
}

// One token: the state advances; part[c] is this lane's part of q . S (before the update with channel decays, after it without).
template <uint32_t NV, uint32_t PC, bool CHANNEL>
__device__ __forceinline__ void advance(State<NV, PC>& S, const Token<NV, PC, CHANNEL>& t, float* part) {
    float2 acc[PC];
#pragma unroll
    for (uint32_t c = 0; c < PC; c++) acc[c] = make_float2(0.0f, 0.0f);
#pragma unroll
    for (uint32_t i = 0; i < NV; i++) {
        const float2 qa = make_float2(t.q[i].x, t.q[i].y), qb = make_float2(t.q[i].z, t.q[i].w), ka = make_float2(t.k[i].x, t.k[i].y), kb = make_float2(t.k[i].z, t.k[i].w);
        float2 wa, wb;
        if constexpr (CHANNEL) {
            wa = make_float2(t.w[i].x, t.w[i].y);
            wb = make_float2(t.w[i].z, t.w[i].w);
        } else {
            wa = wb = make_float2(t.step.y, t.step.y);
        }
#pragma unroll
        for (uint32_t c = 0; c < PC; c++) {
            const float v = CHANNEL ? t.v[c] : t.v[c] * t.step.x;
            const float2 vv = make_float2(v, v);
            if (CHANNEL) {
                acc[c] = __ffma2_rn(qa, S.a[i][c], acc[c]);
                acc[c] = __ffma2_rn(qb, S.b[i][c], acc[c]);
            }
            S.a[i][c] = __ffma2_rn(wa, S.a[i][c], __fmul2_rn(ka, vv));
            S.b[i][c] = __ffma2_rn(wb, S.b[i][c], __fmul2_rn(kb, vv));
            if (!CHANNEL) {
                acc[c] = __ffma2_rn(qa, S.a[i][c], acc[c]);
                acc[c] = __ffma2_rn(qb, S.b[i][c], acc[c]);
            }
        }
    }
#pragma unroll
    for (uint32_t c = 0; c < PC; c++) part[c] = acc[c].x + acc[c].y;
}
template <uint32_t L, uint32_t NV, uint32_t PC, bool CHANNEL>
__device__ __forceinline__ void advance(State<NV, PC>& S, const Stage& st, uint32_t j, uint32_t lane, uint32_t col, float* part) {
    Token<NV, PC, CHANNEL> t;
    load_token<L, NV, PC, CHANNEL>(t, st, j, lane, col);
    advance<NV, PC, CHANNEL>(S, t, part);
}

// SUMS sums over L lanes: each exchange halves what a lane still carries, down to one; lane l ends with sums l SUMS / L .. in part[0]
// on (more lanes than sums: L / SUMS lanes with the same one).
template <uint32_t L, uint32_t SUMS>
__device__ __forceinline__ void spread_sums(float* part, uint32_t lane) {
    uint32_t left = SUMS;
#pragma unroll
    for (uint32_t o = L / 2; o > 0; o /= 2) {
        if (left == 1) {
            part[0] += __shfl_xor_sync(0xffffffffu, part[0], o);
            continue;
        }
        left /= 2;
        const bool up = lane & o;
#pragma unroll
        for (uint32_t u = 0; u < SUMS / 2; u++) {
            if (u >= left) break;
            const float keep = up ? part[u + left] : part[u], give = up ? part[u] : part[u + left];
            part[u] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
}

// grid (heads x slices of 16 value channels, runs), 16 L / PC threads: L lanes share PC (2 or 4) value channels. tc: tokens a chunk, a multiple of
// 8; two chunks in shared memory if a run is longer. GROUP: tokens whose sums are taken together (1: steps of short runs, whose
// kernel holds fewer registers and so has more of the states in flight).
template <uint32_t L, uint32_t NV, uint32_t PC, bool CHANNEL, uint32_t GROUP>
__global__ void __launch_bounds__(L * COLS / PC, GROUP == 1 ? 0 : 1) scan_kernel(const ScanArgs a, uint32_t tc, bool aligned) {
    pdl_start();
    extern __shared__ __align__(16) float sm[];
    constexpr uint32_t NP = 4 * L * NV, THREADS = L * COLS / PC, SUMS = GROUP * PC, PER = SUMS > L ? SUMS / L : 1;
    const RecurrentCache& c = a.c;
    const uint32_t slices = (c.P + COLS - 1) / COLS, head = blockIdx.x / slices, p0 = blockIdx.x % slices * COLS, tid = threadIdx.x, lane = tid % L, col = tid / L * PC;
    const RunIn run = a.runs[blockIdx.y];
    if (a.tensor_min && run.count >= a.tensor_min) return;
    const uint32_t t0 = run.first, count = run.count, cols = min(COLS, c.P - p0), mine = col < cols ? min(PC, cols - col) : 0;
    const bool verify = run.verify && count > 1, two = a.max_run > tc;
    const uint32_t stage_len = stage_floats<CHANNEL>(NP, tc);
    if (c.N != NP || cols != COLS) {  // what no copy writes stays zero
        for (uint32_t i = tid; i < stage_len * (two ? 2 : 1); i += THREADS) sm[i] = 0.0f;
        __syncthreads();
    }
    const float *Q = a.q + size_t(t0) * a.ldq + size_t(head / c.per) * c.N, *K = a.k + size_t(t0) * a.ldk + size_t(head / c.per) * c.N, *V = a.v + size_t(t0) * a.ldv + size_t(head) * c.P + p0;
    const float* D = a.decay + (size_t(t0) * c.heads + head) * (CHANNEL ? c.N : 2);  // (not read where the decays are fixed)
    const float fixed = !CHANNEL && c.fixed ? c.fixed[head] : 1.0f;
    const Walk key0(tid, THREADS, aligned ? c.N / 4 : c.N), value0(tid, THREADS, aligned ? cols / 4 : cols);
    auto rows = [&](Walk at, float* dst, uint32_t pitch, const float* src, size_t ld, uint32_t n) {
        if (aligned)
            for (; at.r < n; at.next()) cp_async16(dst + at.r * pitch + at.c * 4, src + at.r * ld + at.c * 4);
        else
            for (; at.r < n; at.next()) cp_async4(dst + at.r * pitch + at.c, src + at.r * ld + at.c);
    };
    auto fetch = [&](uint32_t i0) {
        const uint32_t n = min(tc, count - i0);
        const Stage st = stage_at<CHANNEL>(sm + (i0 / tc & 1) * stage_len, NP, tc);
        rows(key0, st.q, NP, Q + size_t(i0) * a.ldq, a.ldq, n);
        rows(key0, st.k, NP, K + size_t(i0) * a.ldk, a.ldk, n);
        rows(value0, st.v, COLS, V + size_t(i0) * a.ldv, a.ldv, n);
        if (CHANNEL) {
            rows(key0, st.w, NP, D + size_t(i0) * c.heads * c.N, size_t(c.heads) * c.N, n);
            for (uint32_t i = tid; i < n; i += THREADS) cp_async4(st.s + 4 * i, a.bonus + size_t(t0 + i0 + i) * c.heads + head);
        } else {
            if (!c.fixed)
                for (uint32_t i = tid; i < 2 * n; i += THREADS) cp_async4(st.s + 4 * (i / 2) + i % 2, D + size_t(i0 + i / 2) * c.heads * 2 + i % 2);
            else
                for (uint32_t i = tid; i < n; i += THREADS) *reinterpret_cast<float2*>(st.s + 4 * i) = make_float2(1.0f, fixed);
        }
    };
    float* home = c.state + ((size_t(run.slot) * c.heads + head) * c.P + p0 + (mine ? col : 0)) * NP + 4 * lane;
    State<NV, PC> S;
    load_state<L, NV, PC>(S, home, mine);
    fetch(0);
    cp_async_commit();
    const bool fresh = a.meta[2 * t0 + 1] == 0;  // a sequence begins: nothing of the slot's last one
    if (fresh) S.clear();
    const float skip = CHANNEL || !a.skip ? 0.0f : bf16_to_f32(a.skip[head]);
    const size_t ldy = size_t(c.heads) * c.P;
    float* Y = a.y + size_t(t0) * ldy + size_t(head) * c.P + p0 + col;
    if (verify) {
        // A verified run's rows, at most eight of one tile: each from the state before the run over the rows it descends from. The
        // state itself waits for the accepted path; what it will take is kept.
        cp_async_wait<0>();
        __syncthreads();
        const Stage st = stage_at<CHANNEL>(sm, NP, tc);
        const size_t kept = size_t(run.slot) * VERIFY_T;
        for (uint32_t i = 0; i < count; i++) {
            const size_t row = kept + i;
            for (uint32_t p = tid; p < cols; p += THREADS) c.keep_v[row * ldy + size_t(head) * c.P + p0 + p] = st.v[i * COLS + p];
            if (p0) continue;
            if (head % c.per == 0)
                for (uint32_t n = tid; n < c.N; n += THREADS) c.keep_k[(row * (c.heads / c.per) + head / c.per) * c.N + n] = st.k[i * NP + n];
            if (CHANNEL)
                for (uint32_t n = tid; n < c.N; n += THREADS) c.keep_d[(row * c.heads + head) * c.N + n] = st.w[i * NP + n];
            else if (tid < 2)
                c.keep_d[(row * c.heads + head) * 2 + tid] = st.s[4 * i + tid];
        }
        for (uint32_t i = 0; i < count; i++) {
            float part[PC];
            if (i) {
                if (fresh) S.clear();
                else load_state<L, NV, PC>(S, home, mine);
                for (uint32_t before = a.vis[t0 + i] & ((1u << i) - 1); before; before &= before - 1) advance<L, NV, PC, CHANNEL>(S, st, __ffs(before) - 1, lane, col, part);
            }
            advance<L, NV, PC, CHANNEL>(S, st, i, lane, col, part);
#pragma unroll
            for (uint32_t p = 0; p < PC; p++) {
#pragma unroll
                for (uint32_t o = L / 2; o > 0; o /= 2) part[p] += __shfl_xor_sync(0xffffffffu, part[p], o);
                if (lane == 0 && p < mine) Y[i * ldy + p] = part[p] + (CHANNEL ? st.s[4 * i] : skip) * st.v[i * COLS + col + p];
            }
        }
        return;
    }
    for (uint32_t i0 = 0; i0 < count; i0 += tc) {
        if (i0 + tc < count) fetch(i0 + tc);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const Stage st = stage_at<CHANNEL>(sm + (i0 / tc & 1) * stage_len, NP, tc);
        const uint32_t n = min(tc, count - i0);
        for (uint32_t j0 = 0; j0 < n; j0 += GROUP) {
            float part[GROUP * PC];
            if (j0 + GROUP <= n) {
                Token<NV, PC, CHANNEL> t[2];  // the next token's operands are on their way
                load_token<L, NV, PC, CHANNEL>(t[0], st, j0, lane, col);
#pragma unroll
                for (uint32_t u = 0; u < GROUP; u++) {
                    if (u + 1 < GROUP) load_token<L, NV, PC, CHANNEL>(t[(u + 1) & 1], st, j0 + u + 1, lane, col);
                    advance<NV, PC, CHANNEL>(S, t[u & 1], part + PC * u);
                }
            } else {
#pragma unroll
                for (uint32_t u = 0; u < GROUP; u++) {
                    if (j0 + u < n) {
                        advance<L, NV, PC, CHANNEL>(S, st, j0 + u, lane, col, part + PC * u);
                    } else {
#pragma unroll
                        for (uint32_t p = 0; p < PC; p++) part[PC * u + p] = 0.0f;
                    }
                }
            }
            spread_sums<L, SUMS>(part, lane);
            if (SUMS < L && lane % (L / SUMS > 0 ? L / SUMS : 1)) continue;  // (another lane has the same sum)
#pragma unroll
            for (uint32_t r = 0; r < PER; r++) {
                const uint32_t sum = SUMS < L ? lane * SUMS / L : lane * PER + r, j = j0 + sum / PC, p = sum % PC;
                if (j < n && p < mine) Y[(i0 + j) * ldy + p] = part[r] + (CHANNEL ? st.s[4 * j] : skip) * st.v[j * COLS + col + p];
            }
        }
        __syncthreads();  // the chunk's place is free
    }
    if (mine && !a.gen[run.slot].done) store_state<L, NV, PC>(S, home, mine);
}

// grid (heads, caches, runs).
__global__ void __launch_bounds__(256) recurrent_commit_kernel(const RunIn* __restrict__ runs, const uint32_t* __restrict__ path, const uint32_t* __restrict__ path_len,
                                                               const uint32_t* __restrict__ lens, const RecurrentCache* __restrict__ caches) {
    pdl_start();
    const uint32_t r = blockIdx.z, k = path_len[r], head = blockIdx.x;
    const RunIn run = runs[r];
    const RecurrentCache c = caches[blockIdx.y];
    if (!run.verify || run.count < 2 || k == 0 || head >= c.heads) return;
    const bool fresh = lens[run.slot] == k;
    float* S = c.state + (size_t(run.slot) * c.heads + head) * c.P * c.Np;
    for (uint32_t e = threadIdx.x; e < c.P * c.Np; e += 256) {
        const uint32_t p = e / c.Np, n = e % c.Np;
        if (n >= c.N) continue;
        float s = fresh ? 0.0f : S[e];
        for (uint32_t j = 0; j < k; j++) {
            const size_t row = size_t(run.slot) * VERIFY_T + path[r * FEED_W + j];
            const float key = c.keep_k[(row * (c.heads / c.per) + head / c.per) * c.N + n], v = c.keep_v[(row * c.heads + head) * c.P + p];
            const float* d = c.keep_d + (row * c.heads + head) * (c.channel_decay ? c.N : 2);  // (with fixed decays: 1 and the decay)
            s = c.channel_decay ? fmaf(d[n], s, key * v) : fmaf(d[1], s, key * (v * d[0]));
        }
        S[e] = s;
    }
}

// Small pseudo-random states for sequences whose context is not computed (benchmarks). grid (caches).
__global__ void __launch_bounds__(256) recurrent_fill_kernel(const RecurrentCache* __restrict__ caches, uint32_t slot, uint32_t seed) {
    const RecurrentCache c = caches[blockIdx.x];
    const size_t all = size_t(c.heads) * c.P * c.Np;
    for (size_t e = threadIdx.x; e < all; e += 256)
        c.state[slot * all + e] = e % c.Np < c.N ? (float(philox(make_uint4(uint32_t(e), blockIdx.x, slot, 0), seed, 0x57a7eu).x >> 8) * 0x1p-24f - 0.5f) * 0.5f : 0.0f;
}

// grid (tokens / TB, spans of 128 channels, and one more for the step sizes).
template <uint32_t TB>
__global__ void __launch_bounds__(128) conv_silu_kernel(const ConvArgs a, const StepSizeArgs st, uint32_t n, float* __restrict__ y, uint16_t* __restrict__ y_b) {
    pdl_start();
    __shared__ const float* from[TB][32];
    __shared__ float* into[TB];
    const uint32_t t0 = blockIdx.x * TB, tid = threadIdx.x, nt = min(TB, n - t0);
    if (blockIdx.y == gridDim.y - 1) {
        for (uint32_t i = tid; i < nt * st.heads; i += 128) {
            const uint32_t t = t0 + i / st.heads, h = i % st.heads;
            const float z = st.dt[size_t(t) * st.ld + h] + bf16_to_f32(st.bias[h]);
            const float dt = z > 20.0f ? z : log1pf(expf(z));  // (past 20 the two are the same number in fp32)
            reinterpret_cast<float2*>(st.out)[size_t(t) * st.heads + h] = make_float2(dt, expf(-expf(bf16_to_f32(st.a_log[h])) * dt));
        }
        return;
    }
    // (a block's last tokens past the step repeat its first: their rows exist, and are not stored)
    const uint32_t mine = tid / 32, back = tid % 32;
    if (mine < TB) {
        const uint32_t t = t0 + (mine < nt ? mine : 0);
        if (back < a.taps) from[mine][back] = row_before(a, t, back);
        if (back == 0 && a.write_ring) {
            const uint32_t row = a.tin[2 * t + 1], cpos = a.meta[2 * (t - row) + 1] + row;
            into[mine] = a.ring + (size_t(a.meta[2 * t]) * a.ring_len + cpos % a.ring_len) * a.conv_channels;
        }
    }
    __syncthreads();
    const uint32_t c = blockIdx.y * 128 + tid;
    if (c >= a.conv_channels) return;
    const uint16_t* w = a.w + size_t(c) * a.taps;
    float s[TB], last[TB];
#pragma unroll
    for (uint32_t i = 0; i < TB; i++) s[i] = a.bias ? bf16_to_f32(a.bias[c]) : 0.0f;
    for (uint32_t j = 0; j < a.taps; j++) {
        const float wj = bf16_to_f32(w[j]);
#pragma unroll
        for (uint32_t i = 0; i < TB; i++) {
            const float* p = from[i][a.taps - 1 - j];
            last[i] = p ? p[c] : 0.0f;
            s[i] = fmaf(wj, last[i], s[i]);
        }
    }
#pragma unroll
    for (uint32_t i = 0; i < TB; i++) {
        if (i >= nt) break;
        const float v = silu(s[i]);
        if (y) y[size_t(t0 + i) * a.conv_channels + c] = v;
        if (y_b) y_b[size_t(t0 + i) * a.conv_channels + c] = f32_to_bf16(v);
        if (a.write_ring) into[i][c] = last[i];
    }
}

// grid (tokens, spans of the row).
template <uint32_t V>
__global__ void __launch_bounds__(256) token_shift_kernel(const ShiftArgs a, uint32_t n) {
    pdl_start();
    const uint32_t t = blockIdx.x, tid = threadIdx.x, d = a.c.conv_channels;
    if (t == 0 && blockIdx.y == 0) {
        const uint32_t per = (n + a.tile - 1) / a.tile;
        for (uint32_t i = tid; i < 4 * per; i += 256) {
            const uint32_t g = i / per, p = i % per * a.tile;
            a.tiles[3 * i] = g;
            a.tiles[3 * i + 1] = g * n + p;  // (of the rows behind the first mix)
            a.tiles[3 * i + 2] = min(a.tile, n - p);
        }
        if (tid == 0) *a.n_tiles = 4 * per;
    }
    const uint32_t i = (blockIdx.y * 256 + tid) * V;
    if (i >= d) return;
    const float *h = row_before(a.c, t, 0), *before = row_before(a.c, t, 1);
    float x[V], dx[V];
    load_f32<V>(x, h + i);
#pragma unroll
    for (uint32_t j = 0; j < V; j++) dx[j] = 0.0f;
    if (before) load_f32<V>(dx, before + i);
#pragma unroll
    for (uint32_t j = 0; j < V; j++) dx[j] -= x[j];
#pragma unroll
    for (uint32_t m = 0; m < 5; m++) {
        float y[V];
        load_bf16<V>(y, a.mu[m] + i);
#pragma unroll
        for (uint32_t j = 0; j < V; j++) y[j] = fmaf(dx[j], y[j], x[j]);
        const size_t o = (size_t((m + 1) % 5) * n + t) * d + i;
        if (a.out_f32) store_f32<V>(a.out_f32 + o, y);
        if (a.out_bf16) store_bf16<V>(a.out_bf16 + o, y);
    }
    if (a.c.write_ring) {
        const uint32_t row = a.c.tin[2 * t + 1], cpos = a.c.meta[2 * (t - row) + 1] + row;
        store_f32<V>(a.c.ring + (size_t(a.c.meta[2 * t]) * a.c.ring_len + cpos % a.c.ring_len) * d + i, x);
    }
}

// grid (tokens / TT, heads): the head's rows of w2 and the tokens' hidden rows in shared memory, a channel and TT / 2 tokens a thread
// at a time.
template <uint32_t TT>
__global__ void __launch_bounds__(128) decay_kernel(const DecayArgs a, uint32_t n) {
    pdl_start();
    extern __shared__ __align__(16) float sm[];
    const uint32_t rp = (a.rank + 3) / 4 * 4, wp = (a.rank + 7) / 8 * 8 + 8;  // the rows' pitches, in floats and in halves
    const uint32_t t0 = blockIdx.x * TT, head = blockIdx.y, tid = threadIdx.x, nt = min(TT, n - t0), warp = tid / 32, lane = tid % 32, K = a.heads * a.dim;
    float* th = sm;                                               // [TT][rp]
    uint16_t* w = reinterpret_cast<uint16_t*>(sm + TT * rp);      // [dim][wp]
    const float* hid = a.hid + size_t(t0) * a.ldh;
    const uint16_t* w2 = a.w2 + size_t(head) * a.dim * a.rank;
    if (a.rank % 8 == 0 && a.ldh % 4 == 0) {
        for (Walk at(tid, 128, a.rank / 4); at.r < nt; at.next()) cp_async16(th + at.r * rp + 4 * at.c, hid + size_t(at.r) * a.ldh + 4 * at.c);
        for (Walk at(tid, 128, a.rank / 8); at.r < a.dim; at.next()) cp_async16(w + at.r * wp + 8 * at.c, w2 + at.r * a.rank + 8 * at.c);
    } else {
        for (Walk at(tid, 128, rp); at.r < nt; at.next()) th[at.r * rp + at.c] = at.c < a.rank ? hid[size_t(at.r) * a.ldh + at.c] : 0.0f;
        for (Walk at(tid, 128, rp); at.r < a.dim; at.next()) w[at.r * wp + at.c] = at.c < a.rank ? w2[at.r * a.rank + at.c] : uint16_t(0);
    }
    cp_async_commit();
#pragma unroll 4
    for (uint32_t i = warp; i < nt; i += 4) {
        float s = 0.0f;
        for (uint32_t c = lane; c < a.dim; c += 32) {
            const size_t at = size_t(t0 + i) * K + head * a.dim + c;
            s += a.r[at] * a.k[at] * bf16_to_f32(a.u[head * a.dim + c]);
        }
        s = warp_sum(s);
        if (lane == 0) a.bonus[size_t(t0 + i) * a.heads + head] = s;
    }
    cp_async_wait<0>();
    __syncthreads();
    for (uint32_t i = tid; i < TT * rp; i += 128) th[i] = i < nt * rp ? tanhf(th[i]) : 0.0f;
    __syncthreads();
    constexpr uint32_t PER = TT / 2;
    for (uint32_t i = tid; i < 2 * a.dim; i += 128) {
        const uint32_t c = i % a.dim, q0 = i / a.dim * PER;
        if (q0 >= nt) continue;
        float s[PER] = {};
        for (uint32_t j = 0; j < rp; j += 4) {
            float wj[4];
            load_bf16<4>(wj, w + c * wp + j);
#pragma unroll
            for (uint32_t u = 0; u < PER; u++) {
                const float4 h = *reinterpret_cast<const float4*>(th + (q0 + u) * rp + j);
                s[u] = fmaf(wj[3], h.w, fmaf(wj[2], h.z, fmaf(wj[1], h.y, fmaf(wj[0], h.x, s[u]))));
            }
        }
        const float w0 = bf16_to_f32(a.w0[head * a.dim + c]);
#pragma unroll
        for (uint32_t u = 0; u < PER; u++)
            if (q0 + u < nt) a.decay[size_t(t0 + q0 + u) * K + head * a.dim + c] = expf(-expf(s[u] + w0));
    }
}

// A block per token, which keeps the row in shared memory: with eight parts or more a warp takes one at a time, else all threads
// together.
template <uint32_t V>
__global__ void __launch_bounds__(1024) gated_norm_kernel(const GatedNormArgs a) {
    pdl_start();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[32];
    const uint32_t t = blockIdx.x, tid = threadIdx.x, width = a.width / a.groups;
    const bool alone = a.groups >= 8;
    const uint32_t lanes = alone ? 32 : blockDim.x, lane = tid % lanes, first = tid / lanes, step = blockDim.x / lanes;
    const float *y = a.y + size_t(t) * a.width, *gate = a.gate + size_t(t) * a.ldg;
    for (uint32_t g = first; g < a.groups; g += step) {
        const uint32_t c0 = g * width;
        float ss = 0.0f;
        for (uint32_t c = lane * V; c < width; c += lanes * V) {
            float v[V], z[V], w[V];
            load_f32<V>(v, y + c0 + c);
            load_f32<V>(z, gate + c0 + c);
            load_bf16<V>(w, a.w + c0 + c);
#pragma unroll
            for (uint32_t j = 0; j < V; j++) {
                const float s = a.sigmoid ? sigmoid_of(z[j]) : silu(z[j]), gated = v[j] * s;
                ss += a.gate_first ? gated * gated : v[j] * v[j];
                v[j] = gated * w[j];
            }
            store_f32<V>(row + c0 + c, v);
        }
        if (alone) {
            ss = warp_sum(ss);
        } else {
            __syncthreads();  // (`red` has been read for the part before this one)
            ss = block_sum(ss, red);
        }
        const float inv = 1.0f / sqrtf(ss / float(width) + a.eps);
        for (uint32_t c = lane * V; c < width; c += lanes * V) {  // (a thread reads back what it wrote)
            float v[V];
            load_f32<V>(v, row + c0 + c);
#pragma unroll
            for (uint32_t j = 0; j < V; j++) v[j] *= inv;
            const size_t o = size_t(t) * a.width + c0 + c;
            if (a.out_f32) store_f32<V>(a.out_f32 + o, v);
            if (a.out_bf16) store_bf16<V>(a.out_bf16 + o, v);
        }
    }
}

template <uint32_t L, uint32_t NV, uint32_t PC, bool CHANNEL, uint32_t GROUP>
void scan(const ScanArgs& a, cudaStream_t s) {
    static PerDevice configured;
    auto* kernel = scan_kernel<L, NV, PC, CHANNEL, GROUP>;
    configured.once([&] { VLT_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024)); });
    const uint32_t slices = (a.c.P + COLS - 1) / COLS;
    constexpr uint32_t NP = 4 * L * NV;
    uint32_t tc = 8;
    while (tc < 32 && tc < a.max_run && 2 * stage_floats<CHANNEL>(NP, 2 * tc) * 4 <= 72 * 1024) tc *= 2;
    if (a.max_run < tc) tc = a.max_run;
    const size_t smem = size_t(stage_floats<CHANNEL>(NP, tc)) * 4 * (a.max_run > tc ? 2 : 1);
    auto whole = [](const void* p, size_t ld) { return reinterpret_cast<uintptr_t>(p) % 16 == 0 && ld % 4 == 0; };
    const bool aligned = a.c.N % 4 == 0 && a.c.P % 4 == 0 && whole(a.q, a.ldq) && whole(a.k, a.ldk) && whole(a.v, a.ldv) && whole(a.decay, 0);
    launch_pdl(kernel, dim3(a.c.heads * slices, a.n_runs), L * COLS / PC, smem, s, a, tc, aligned);
}
// Per pitch: steps of short runs (bound by the states' traffic) with four columns a lane, longer ones (bound by instructions and
// their latencies) with two and twice the threads.
struct Kernel {
    uint32_t pitch;
    void (*short_plain)(const ScanArgs&, cudaStream_t);
    void (*short_channel)(const ScanArgs&, cudaStream_t);
    void (*plain)(const ScanArgs&, cudaStream_t);
    void (*channel)(const ScanArgs&, cudaStream_t);
};
static const Kernel kernels[] = {{32, scan<8, 1, 4, false, 1>, scan<8, 1, 4, true, 1>, scan<8, 1, 2, false, 8>, scan<8, 1, 2, true, 8>},
                                 {64, scan<16, 1, 4, false, 1>, scan<16, 1, 4, true, 1>, scan<16, 1, 2, false, 8>, scan<16, 1, 2, true, 8>},
                                 {128, scan<32, 1, 4, false, 1>, scan<32, 1, 4, true, 1>, scan<32, 1, 2, false, 8>, scan<32, 1, 2, true, 8>},
                                 {256, scan<32, 2, 4, false, 1>, scan<32, 2, 4, true, 1>, scan<32, 2, 2, false, 8>, scan<32, 2, 2, true, 8>},
                                 {384, scan<32, 3, 4, false, 1>, scan<32, 3, 4, true, 1>, scan<32, 3, 2, false, 8>, scan<32, 3, 2, true, 8>},
                                 {512, scan<32, 4, 4, false, 1>, scan<32, 4, 4, true, 1>, scan<32, 4, 2, false, 8>, scan<32, 4, 2, true, 8>}};

}  // namespace recurrent

void launch_scan(const ScanArgs& all, cudaStream_t s) {
    using namespace recurrent;
    ScanArgs a = all;
    if (!a.n_runs) return;
    if (a.q_b && a.max_run >= SSD_MIN_RUN) {
        a.tensor_min = SSD_MIN_RUN;
        launch_ssd(a, s);
        if (a.n_runs == 1) return;
        a.max_run = SSD_MIN_RUN - 1;  // at most, of the runs that are left
    }
    for (const Kernel& k : kernels)
        if (k.pitch == a.c.Np) {
            if (a.max_run <= VERIFY_T) (a.c.channel_decay ? k.short_channel : k.short_plain)(a, s);
            else (a.c.channel_decay ? k.channel : k.plain)(a, s);
            return;
        }
    throw Error("internal: a recurrence over " + std::to_string(a.c.N) + " key channels");
}
// The key channels a state is laid out for: those of the smallest kernel that takes N.
uint32_t recurrent_pitch(uint32_t N) {
    for (const recurrent::Kernel& k : recurrent::kernels)
        if (N <= k.pitch) return k.pitch;
    throw Error("internal: a recurrence over " + std::to_string(N) + " key channels");
}
void launch_recurrent_commit(const RunIn* runs, const uint32_t* path, const uint32_t* path_len, const uint32_t* lens, const RecurrentCache* caches, uint32_t n_runs,
                             uint32_t n_caches, uint32_t max_heads, cudaStream_t s) {
    if (n_runs && n_caches) launch_pdl(recurrent::recurrent_commit_kernel, dim3(max_heads, n_caches, n_runs), 256, 0, s, runs, path, path_len, lens, caches);
}
void launch_recurrent_fill(const RecurrentCache* caches, uint32_t n_caches, uint32_t slot, uint32_t seed, cudaStream_t s) {
    if (!n_caches) return;
    recurrent::recurrent_fill_kernel<<<n_caches, 256, 0, s>>>(caches, slot, seed);
    launch_counter()++;
}
void launch_conv_silu(const ConvArgs& a, const StepSizeArgs& st, uint32_t n, float* y, uint16_t* y_b, cudaStream_t s) {
    const uint32_t spans = (a.conv_channels + 127) / 128 + 1;
    if (n >= 64) launch_pdl(recurrent::conv_silu_kernel<4>, dim3((n + 3) / 4, spans), 128, 0, s, a, st, n, y, y_b);
    else launch_pdl(recurrent::conv_silu_kernel<1>, dim3(n, spans), 128, 0, s, a, st, n, y, y_b);
}
void launch_token_shift(const ShiftArgs& a, uint32_t n, cudaStream_t s) {
    const uint32_t d = a.c.conv_channels;
    if (d % 4 == 0) launch_pdl(recurrent::token_shift_kernel<4>, dim3(n, (d + 1023) / 1024), 256, 0, s, a, n);
    else launch_pdl(recurrent::token_shift_kernel<1>, dim3(n, (d + 255) / 256), 256, 0, s, a, n);
}
static size_t decay_smem(size_t tokens, size_t rank, size_t dim) { return tokens * ((rank + 3) / 4 * 4) * 4 + dim * ((rank + 7) / 8 * 8 + 8) * 2; }
bool decay_fits(uint32_t rank, uint32_t dim) { return decay_smem(32, rank, dim) <= 220 * 1024; }
void launch_decay(const DecayArgs& a, uint32_t n, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] {
        for (auto f : {recurrent::decay_kernel<8>, recurrent::decay_kernel<32>}) VLT_CUDA(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    });
    const uint32_t tt = n >= 64 ? 32 : 8;
    const size_t smem = decay_smem(tt, a.rank, a.dim);
    if (tt == 32) launch_pdl(recurrent::decay_kernel<32>, dim3((n + 31) / 32, a.heads), 128, smem, s, a, n);
    else launch_pdl(recurrent::decay_kernel<8>, dim3((n + 7) / 8, a.heads), 128, smem, s, a, n);
}
void launch_gated_norm(const GatedNormArgs& a, uint32_t n, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] {
        for (auto f : {recurrent::gated_norm_kernel<1>, recurrent::gated_norm_kernel<4>}) VLT_CUDA(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    });
    const bool four = a.width / a.groups % 4 == 0 && a.ldg % 4 == 0 && reinterpret_cast<uintptr_t>(a.gate) % 16 == 0;
    if (four) launch_pdl(recurrent::gated_norm_kernel<4>, n, row_threads(a.width, 4), size_t(a.width) * 4, s, a);
    else launch_pdl(recurrent::gated_norm_kernel<1>, n, row_threads(a.width, 1), size_t(a.width) * 4, s, a);
}

}  // namespace vlt
