// Linear recurrences over a state per head, and what stands around them in a layer: the state space's short convolution with silu
// and its step sizes, time mixing's mixes of neighbouring rows and its decays, and the gated norm of the outputs.
//
// The recurrence S = D S + k v^T runs token by token in fp32, the state in registers: a block has 16 value channels of one head of
// one run, eight lanes share a value channel and hold an eighth of its key channels each, in pairs for the packed fp32
// instructions. Rows come in by asynchronous copies, a chunk of tokens ahead; the output's sums over the eight lanes are taken
// for eight tokens at a time, so that a token costs one exchange between lanes. A prompt's portion reads and writes the state
// once, like a decoded token. The result of a row depends on nothing but the rows before it, however they are cut into steps.
#include <algorithm>

#include "kernels.h"

namespace vlt {

namespace recurrent {

constexpr uint32_t LANES = 8, COLS = 16, THREADS = LANES * COLS;

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ void cp_async4(float* dst, const float* src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(uint32_t(__cvta_generic_to_shared(dst))), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_async16(float* dst, const float* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(uint32_t(__cvta_generic_to_shared(dst))), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

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

// The state as a thread holds it: key channels 4 lane + 32 i .. + 3 of its value channel, in two pairs each.
template <uint32_t NV>
struct State {
    float2 a[NV], b[NV];
    __device__ __forceinline__ void clear() {
#pragma unroll
        for (uint32_t i = 0; i < NV; i++) a[i] = b[i] = make_float2(0.0f, 0.0f);
    }
    __device__ __forceinline__ void load(const float* p) {
#pragma unroll
        for (uint32_t i = 0; i < NV; i++) {
            const float4 x = *reinterpret_cast<const float4*>(p + 32 * i);
            a[i] = make_float2(x.x, x.y);
            b[i] = make_float2(x.z, x.w);
        }
    }
    __device__ __forceinline__ void store(float* p) const {
#pragma unroll
        for (uint32_t i = 0; i < NV; i++) *reinterpret_cast<float4*>(p + 32 * i) = make_float4(a[i].x, a[i].y, b[i].x, b[i].y);
    }
};

// One token: the state advances; the returned sum is this lane's part of q . S (before the update with channel decays, after it
// without).
template <uint32_t NV, bool CHANNEL>
__device__ __forceinline__ float advance(State<NV>& S, const Stage& st, uint32_t np, uint32_t j, uint32_t n0, uint32_t col) {
    const float factor = CHANNEL ? 1.0f : st.s[4 * j], v = st.v[j * COLS + col] * factor;
    const float2 vv = make_float2(v, v);
    float2 acc = make_float2(0.0f, 0.0f), d = acc;
    if (!CHANNEL) d = make_float2(st.s[4 * j + 1], st.s[4 * j + 1]);
    const float *q = st.q + j * np + n0, *k = st.k + j * np + n0, *w = st.w + j * np + n0;
#pragma unroll
    for (uint32_t i = 0; i < NV; i++) {
        const float4 q4 = *reinterpret_cast<const float4*>(q + 32 * i), k4 = *reinterpret_cast<const float4*>(k + 32 * i);
        const float2 kva = __fmul2_rn(make_float2(k4.x, k4.y), vv), kvb = __fmul2_rn(make_float2(k4.z, k4.w), vv);
        if (CHANNEL) {
            const float4 w4 = *reinterpret_cast<const float4*>(w + 32 * i);
            acc = __ffma2_rn(make_float2(q4.x, q4.y), S.a[i], acc);
            acc = __ffma2_rn(make_float2(q4.z, q4.w), S.b[i], acc);
            S.a[i] = __ffma2_rn(make_float2(w4.x, w4.y), S.a[i], kva);
            S.b[i] = __ffma2_rn(make_float2(w4.z, w4.w), S.b[i], kvb);
        } else {
            S.a[i] = __ffma2_rn(d, S.a[i], kva);
            S.b[i] = __ffma2_rn(d, S.b[i], kvb);
            acc = __ffma2_rn(make_float2(q4.x, q4.y), S.a[i], acc);
            acc = __ffma2_rn(make_float2(q4.z, q4.w), S.b[i], acc);
        }
    }
    return acc.x + acc.y;
}

// grid (heads x slices of 16 value channels, runs). tc: tokens a chunk, a multiple of 8; two chunks in shared memory if a run is longer.
template <uint32_t NV, bool CHANNEL>
__global__ void __launch_bounds__(THREADS) scan_kernel(const ScanArgs a, uint32_t tc, bool aligned) {
    pdl_start();
    extern __shared__ __align__(16) float sm[];
    constexpr uint32_t NP = 32 * NV;
    const RecurrentCache& c = a.c;
    const uint32_t slices = (c.P + COLS - 1) / COLS, head = blockIdx.x / slices, p0 = blockIdx.x % slices * COLS, tid = threadIdx.x, lane = tid % LANES, col = tid / LANES;
    const RunIn run = a.runs[blockIdx.y];
    const uint32_t t0 = run.first, count = run.count, cols = min(COLS, c.P - p0), n0 = 4 * lane;
    const bool verify = run.verify && count > 1, two = a.max_run > tc;
    const uint32_t stage_len = stage_floats<CHANNEL>(NP, tc);
    if (c.N != NP || cols != COLS) {  // what no copy writes stays zero
        for (uint32_t i = tid; i < stage_len * (two ? 2 : 1); i += THREADS) sm[i] = 0.0f;
        __syncthreads();
    }
    const float *Q = a.q + size_t(t0) * a.ldq + size_t(head / c.per) * c.N, *K = a.k + size_t(t0) * a.ldk + size_t(head / c.per) * c.N, *V = a.v + size_t(t0) * a.ldv + size_t(head) * c.P + p0;
    const float* D = CHANNEL ? a.decay + (size_t(t0) * c.heads + head) * c.N : a.decay + (size_t(t0) * c.heads + head) * 2;
    auto rows = [&](float* dst, uint32_t pitch, const float* src, size_t ld, uint32_t width, uint32_t n) {
        if (aligned) {
            const uint32_t w4 = width / 4;
            for (uint32_t i = tid; i < n * w4; i += THREADS) cp_async16(dst + i / w4 * pitch + i % w4 * 4, src + i / w4 * ld + i % w4 * 4);
        } else {
            for (uint32_t i = tid; i < n * width; i += THREADS) cp_async4(dst + i / width * pitch + i % width, src + i / width * ld + i % width);
        }
    };
    auto fetch = [&](uint32_t i0) {
        const uint32_t n = min(tc, count - i0);
        const Stage st = stage_at<CHANNEL>(sm + (i0 / tc & 1) * stage_len, NP, tc);
        rows(st.q, NP, Q + size_t(i0) * a.ldq, a.ldq, c.N, n);
        rows(st.k, NP, K + size_t(i0) * a.ldk, a.ldk, c.N, n);
        rows(st.v, COLS, V + size_t(i0) * a.ldv, a.ldv, cols, n);
        if (CHANNEL) {
            rows(st.w, NP, D + size_t(i0) * c.heads * c.N, size_t(c.heads) * c.N, c.N, n);
            for (uint32_t i = tid; i < n; i += THREADS) cp_async4(st.s + 4 * i, a.bonus + size_t(t0 + i0 + i) * c.heads + head);
        } else {
            for (uint32_t i = tid; i < 2 * n; i += THREADS) cp_async4(st.s + 4 * (i / 2) + i % 2, D + size_t(i0 + i / 2) * c.heads * 2 + i % 2);
        }
    };
    fetch(0);
    cp_async_commit();
    const bool mine = col < cols;
    float* home = c.state + ((size_t(run.slot) * c.heads + head) * c.P + p0 + (mine ? col : 0)) * NP + n0;
    const bool fresh = a.meta[2 * t0 + 1] == 0;  // a sequence begins: nothing of the slot's last one
    State<NV> S;
    if (fresh) S.clear();
    else S.load(home);
    const float skip = CHANNEL ? 0.0f : bf16_to_f32(a.skip[head]);
    float* Y = a.y + size_t(t0) * c.heads * c.P + size_t(head) * c.P + p0 + col;
    if (verify) {
        // A verified run's rows, at most eight of one tile: each from the state before the run over the rows it descends from. The
        // state itself waits for the accepted path; what it will take is kept.
        cp_async_wait<0>();
        __syncthreads();
        const Stage st = stage_at<CHANNEL>(sm, NP, tc);
        const size_t kept = size_t(run.slot) * VERIFY_T;
        for (uint32_t i = 0; i < count; i++) {
            const size_t row = kept + i;
            if (tid < cols) c.keep_v[row * c.heads * c.P + size_t(head) * c.P + p0 + tid] = st.v[i * COLS + tid];
            if (p0) continue;
            if (head % c.per == 0)
                for (uint32_t n = tid; n < c.N; n += THREADS) c.keep_k[(row * (c.heads / c.per) + head / c.per) * c.N + n] = st.k[i * NP + n];
            if (CHANNEL)
                for (uint32_t n = tid; n < c.N; n += THREADS) c.keep_d[(row * c.heads + head) * c.N + n] = st.w[i * NP + n];
            else if (tid < 2)
                c.keep_d[(row * c.heads + head) * 2 + tid] = st.s[4 * i + tid];
        }
        for (uint32_t i = 0; i < count; i++) {
            if (i) {
                if (fresh) S.clear();
                else S.load(home);
                for (uint32_t before = a.vis[t0 + i] & ((1u << i) - 1); before; before &= before - 1) advance<NV, CHANNEL>(S, st, NP, __ffs(before) - 1, n0, col);
            }
            float y = advance<NV, CHANNEL>(S, st, NP, i, n0, col);
#pragma unroll
            for (uint32_t o = LANES / 2; o > 0; o /= 2) y += __shfl_xor_sync(0xffffffffu, y, o);
            if (lane == 0 && mine) Y[size_t(i) * c.heads * c.P] = y + (CHANNEL ? st.s[4 * i] : skip) * st.v[i * COLS + col];
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
        for (uint32_t j0 = 0; j0 < n; j0 += LANES) {
            float part[LANES];
            if (j0 + LANES <= n) {
#pragma unroll
                for (uint32_t u = 0; u < LANES; u++) part[u] = advance<NV, CHANNEL>(S, st, NP, j0 + u, n0, col);
            } else {
#pragma unroll
                for (uint32_t u = 0; u < LANES; u++) part[u] = j0 + u < n ? advance<NV, CHANNEL>(S, st, NP, j0 + u, n0, col) : 0.0f;
            }
            // Eight sums over eight lanes: each exchange halves what a lane still carries; lane u ends with token u's.
#pragma unroll
            for (uint32_t o = LANES / 2; o > 0; o /= 2) {
                const bool up = lane & o;
#pragma unroll
                for (uint32_t u = 0; u < o; u++) {
                    const float keep = up ? part[u + o] : part[u], give = up ? part[u] : part[u + o];
                    part[u] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                }
            }
            const uint32_t j = j0 + lane;
            if (j < n && mine) Y[size_t(i0 + j) * c.heads * c.P] = part[0] + (CHANNEL ? st.s[4 * j] : skip) * st.v[j * COLS + col];
        }
        __syncthreads();  // the chunk's place is free
    }
    if (mine && !a.gen[run.slot].done) S.store(home);
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
            const float* d = c.keep_d + (row * c.heads + head) * (c.channel_decay ? c.N : 2);
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
__global__ void __launch_bounds__(128) conv_silu_kernel(const ConvArgs a, const StepSizeArgs st, uint32_t n, float* __restrict__ y) {
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
        y[size_t(t0 + i) * a.conv_channels + c] = silu(s[i]);
        if (a.write_ring) into[i][c] = last[i];
    }
}

// A block per token.
__global__ void __launch_bounds__(256) token_shift_kernel(const ShiftArgs a, uint32_t n) {
    pdl_start();
    const uint32_t t = blockIdx.x, tid = threadIdx.x, d = a.c.conv_channels;
    if (t == 0) {
        const uint32_t per = (n + a.tile - 1) / a.tile;
        for (uint32_t i = tid; i < 4 * per; i += 256) {
            const uint32_t g = i / per, p = i % per * a.tile;
            a.tiles[3 * i] = g;
            a.tiles[3 * i + 1] = g * n + p;  // (of the rows behind the first mix)
            a.tiles[3 * i + 2] = min(a.tile, n - p);
        }
        if (tid == 0) *a.n_tiles = 4 * per;
    }
    const float *h = row_before(a.c, t, 0), *before = row_before(a.c, t, 1);
    const uint32_t row = a.c.tin[2 * t + 1], cpos = a.c.meta[2 * (t - row) + 1] + row;
    float* ring = a.c.ring + (size_t(a.c.meta[2 * t]) * a.c.ring_len + cpos % a.c.ring_len) * d;
    for (uint32_t i = tid; i < d; i += 256) {
        const float x = h[i], dx = (before ? before[i] : 0.0f) - x;
#pragma unroll
        for (uint32_t m = 0; m < 5; m++) {
            const float y = fmaf(dx, bf16_to_f32(a.mu[m][i]), x);
            const size_t o = (size_t((m + 1) % 5) * n + t) * d + i;
            if (a.out_f32) a.out_f32[o] = y;
            if (a.out_bf16) a.out_bf16[o] = f32_to_bf16(y);
        }
        if (a.c.write_ring) ring[i] = x;
    }
}

// grid (tokens / 8, heads).
__global__ void __launch_bounds__(128) decay_kernel(const DecayArgs a, uint32_t n) {
    pdl_start();
    extern __shared__ float th[];  // [8][rank]
    const uint32_t t0 = blockIdx.x * 8, head = blockIdx.y, tid = threadIdx.x, nt = min(8u, n - t0), warp = tid / 32, lane = tid % 32, K = a.heads * a.dim;
    for (uint32_t i = tid; i < 8 * a.rank; i += 128) th[i] = i / a.rank < nt ? tanhf(a.hid[size_t(t0 + i / a.rank) * a.ldh + i % a.rank]) : 0.0f;
    for (uint32_t i = warp; i < nt; i += 4) {
        float s = 0.0f;
        for (uint32_t c = lane; c < a.dim; c += 32) {
            const size_t at = size_t(t0 + i) * K + head * a.dim + c;
            s += a.r[at] * a.k[at] * bf16_to_f32(a.u[head * a.dim + c]);
        }
        s = warp_sum(s);
        if (lane == 0) a.bonus[size_t(t0 + i) * a.heads + head] = s;
    }
    __syncthreads();
    for (uint32_t i = tid; i < 2 * a.dim; i += 128) {  // a channel, four tokens
        const uint32_t c = head * a.dim + i % a.dim, q0 = i / a.dim * 4;
        if (q0 >= nt) continue;
        const uint16_t* w = a.w2 + size_t(c) * a.rank;
        float s[4] = {};
        for (uint32_t j = 0; j < a.rank; j++) {
            const float wj = bf16_to_f32(w[j]);
#pragma unroll
            for (uint32_t u = 0; u < 4; u++) s[u] = fmaf(wj, th[(q0 + u) * a.rank + j], s[u]);
        }
        const float w0 = bf16_to_f32(a.w0[c]);
#pragma unroll
        for (uint32_t u = 0; u < 4; u++)
            if (q0 + u < nt) a.decay[size_t(t0 + q0 + u) * K + c] = expf(-expf(s[u] + w0));
    }
}

// A block per token: with eight parts or more a warp takes one at a time, else all threads together.
__global__ void __launch_bounds__(256) gated_norm_kernel(const GatedNormArgs a) {
    pdl_start();
    __shared__ float red[8];
    const uint32_t t = blockIdx.x, tid = threadIdx.x, width = a.width / a.groups;
    const bool alone = a.groups >= 8;
    const uint32_t lanes = alone ? 32 : 256, lane = tid % lanes, first = tid / lanes, step = 256 / lanes;
    const float *y = a.y + size_t(t) * a.width, *gate = a.gate + size_t(t) * a.ldg;
    for (uint32_t g = first; g < a.groups; g += step) {
        const uint32_t c0 = g * width;
        float ss = 0.0f;
        for (uint32_t c = lane; c < width; c += lanes) {
            const float v = a.gate_first ? y[c0 + c] * silu(gate[c0 + c]) : y[c0 + c];
            ss += v * v;
        }
        ss = warp_sum(ss);
        if (!alone) {
            __syncthreads();  // (the part before this one has been read)
            if (tid % 32 == 0) red[tid / 32] = ss;
            __syncthreads();
            ss = 0.0f;
            for (uint32_t i = 0; i < 8; i++) ss += red[i];
        }
        const float inv = 1.0f / sqrtf(ss / float(width) + a.eps);
        for (uint32_t c = lane; c < width; c += lanes) {
            const float z = silu(gate[c0 + c]), v = y[c0 + c] * inv * bf16_to_f32(a.w[c0 + c]) * z;
            if (a.out_f32) a.out_f32[size_t(t) * a.width + c0 + c] = v;
            if (a.out_bf16) a.out_bf16[size_t(t) * a.width + c0 + c] = f32_to_bf16(v);
        }
    }
}

template <uint32_t NV, bool CHANNEL>
void scan(const ScanArgs& a, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] { VLT_CUDA(cudaFuncSetAttribute(scan_kernel<NV, CHANNEL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024)); });
    const uint32_t slices = (a.c.P + COLS - 1) / COLS;
    uint32_t tc = 8;
    while (tc < 32 && tc < a.max_run && 2 * stage_floats<CHANNEL>(32 * NV, 2 * tc) * 4 <= 72 * 1024) tc *= 2;
    const size_t smem = size_t(stage_floats<CHANNEL>(32 * NV, tc)) * 4 * (a.max_run > tc ? 2 : 1);
    auto whole = [](const void* p, size_t ld) { return reinterpret_cast<uintptr_t>(p) % 16 == 0 && ld % 4 == 0; };
    const bool aligned = a.c.N % 4 == 0 && a.c.P % 4 == 0 && whole(a.q, a.ldq) && whole(a.k, a.ldk) && whole(a.v, a.ldv) && whole(a.decay, 0);
    launch_pdl(scan_kernel<NV, CHANNEL>, dim3(a.c.heads * slices, a.n_runs), THREADS, smem, s, a, tc, aligned);
}

}  // namespace recurrent

void launch_scan(const ScanArgs& a, cudaStream_t s) {
    using namespace recurrent;
    if (!a.n_runs) return;
    using Fn = void (*)(const ScanArgs&, cudaStream_t);
    static const struct { uint32_t nv; Fn plain, channel; } kernels[] = {{1, scan<1, false>, scan<1, true>}, {2, scan<2, false>, scan<2, true>},   {3, scan<3, false>, scan<3, true>},
                                                                         {4, scan<4, false>, scan<4, true>}, {6, scan<6, false>, scan<6, true>},   {8, scan<8, false>, scan<8, true>},
                                                                         {12, scan<12, false>, scan<12, true>}, {16, scan<16, false>, scan<16, true>}};
    for (const auto& k : kernels)
        if (32 * k.nv == a.c.Np) { (a.c.channel_decay ? k.channel : k.plain)(a, s); return; }
    throw Error("internal: a recurrence over " + std::to_string(a.c.N) + " key channels");
}
// The key channels a state is laid out for: those of the smallest kernel that takes N.
uint32_t recurrent_pitch(uint32_t N) {
    for (uint32_t nv : {1u, 2u, 3u, 4u, 6u, 8u, 12u, 16u})
        if (N <= 32 * nv) return 32 * nv;
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
void launch_conv_silu(const ConvArgs& a, const StepSizeArgs& st, uint32_t n, float* y, cudaStream_t s) {
    const uint32_t spans = (a.conv_channels + 127) / 128 + 1;
    if (n >= 64) launch_pdl(recurrent::conv_silu_kernel<4>, dim3((n + 3) / 4, spans), 128, 0, s, a, st, n, y);
    else launch_pdl(recurrent::conv_silu_kernel<1>, dim3(n, spans), 128, 0, s, a, st, n, y);
}
void launch_token_shift(const ShiftArgs& a, uint32_t n, cudaStream_t s) { launch_pdl(recurrent::token_shift_kernel, n, 256, 0, s, a, n); }
void launch_decay(const DecayArgs& a, uint32_t n, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] { VLT_CUDA(cudaFuncSetAttribute(recurrent::decay_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); });
    launch_pdl(recurrent::decay_kernel, dim3((n + 7) / 8, a.heads), 128, size_t(8) * a.rank * 4, s, a, n);
}
void launch_gated_norm(const GatedNormArgs& a, uint32_t n, cudaStream_t s) { launch_pdl(recurrent::gated_norm_kernel, n, 256, 0, s, a); }

}  // namespace vlt
