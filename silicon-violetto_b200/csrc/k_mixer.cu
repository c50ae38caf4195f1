// The attention mixer's work between its projections and its attention, as parameterised kernels: a short causal
// convolution over time on q, k and v, rotation of pairs, q, k and v heads of unit length, queries that grow with
// their position, values mixed with an earlier layer's (each of them optional), K and V into a paged cache whose heads may have
// different key and value sizes; the convolution's state -- the projected rows before the step -- in a ring per sequence
// slot; and a scalar form of the chunked or windowed attention for any head sizes and for fp32 caches.
#include <algorithm>

#include "kernels.h"
#include "paged_attn.cuh"

namespace vlt {

namespace mixer {

__device__ __forceinline__ void store_kv(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_kv(uint16_t* p, float v) { *p = f32_to_bf16(v); }
__device__ __forceinline__ float load_kv(const float* p) { return *p; }
__device__ __forceinline__ float load_kv(const uint16_t* p) { return bf16_to_f32(*p); }

// grid (tokens / TB, heads + 2 kv heads): one q, k or v head of TB tokens a block (a step of many tokens: the tokens' chains of
// dependent loads run side by side).
template <typename T, uint32_t TB>
__global__ void __launch_bounds__(128) conv_qkv_kernel(const ConvArgs a, uint32_t n) {
    pdl_start();
    extern __shared__ float y[];  // [TB][width]: the head after its convolution
    __shared__ const float* from[TB][32];
    __shared__ uint32_t pos_s[TB], cpos_s[TB], slot_s[TB];
    __shared__ size_t row_s[TB];  // where the head's key or value goes in the cache
    __shared__ float factor[TB];  // what multiplies the head
    const uint32_t t0 = blockIdx.x * TB, unit = blockIdx.y, tid = threadIdx.x, nt = min(TB, n - t0);
    const uint32_t kind = unit < a.heads ? 0u : unit < a.heads + a.kv.n_kv ? 1u : 2u;
    const uint32_t head = kind == 0 ? unit : kind == 1 ? unit - a.heads : unit - a.heads - a.kv.n_kv, width = kind == 2 ? a.kv.dv : a.kv.dk;
    const uint32_t c0 = kind == 2 ? (a.heads + a.kv.n_kv) * a.kv.dk + head * a.kv.dv : unit * a.kv.dk;
    // (a block's last tokens past the step repeat its first: their rows exist, and are not stored)
    const uint32_t mine = tid / 32, back = tid % 32;  // a warp per token works out where its rows lie
    if (mine < TB) {
        const uint32_t t = t0 + (mine < nt ? mine : 0);
        if (back < a.taps) from[mine][back] = row_before(a, t, back);  // (without a convolution: the row itself)
        if (back == 0) {
            const uint32_t row = a.tin[2 * t + 1];
            slot_s[mine] = a.meta[2 * t];
            pos_s[mine] = a.meta[2 * t + 1];
            cpos_s[mine] = a.meta[2 * (t - row) + 1] + row;
            row_s[mine] = kind ? page_row(a.kv, slot_s[mine], head, cpos_s[mine]) : 0;
            factor[mine] = kind == 0 && a.temp.every > 0 ? 1.0f + a.temp.coef * logf(float(floor(double(pos_s[mine] + 1) / a.temp.every)) + 1.0f) : 1.0f;
        }
    }
    __syncthreads();
    for (uint32_t c = tid; c < width; c += 128) {
        const uint16_t* w = a.w ? a.w + size_t(c0 + c) * a.taps : nullptr;
        float s[TB] = {}, last[TB] = {};
        for (uint32_t j0 = 0; j0 < a.taps; j0 += 4) {  // four taps' loads together
            float wj[4], u[4][TB];
#pragma unroll
            for (uint32_t k = 0; k < 4; k++) {
                const bool real = j0 + k < a.taps;
                wj[k] = !real ? 0.0f : w ? bf16_to_f32(w[j0 + k]) : 1.0f;
#pragma unroll
                for (uint32_t i = 0; i < TB; i++) {
                    const float* p = real ? from[i][a.taps - 1 - j0 - k] : nullptr;
                    u[k][i] = p ? p[c0 + c] : 0.0f;
                }
            }
#pragma unroll
            for (uint32_t k = 0; k < 4; k++)
#pragma unroll
                for (uint32_t i = 0; i < TB; i++) {
                    s[i] = fmaf(wj[k], u[k][i], s[i]);
                    if (j0 + k + 1 == a.taps) last[i] = u[k][i];
                }
        }
#pragma unroll
        for (uint32_t i = 0; i < TB; i++) {
            y[i * width + c] = s[i];
            if (a.write_ring && i < nt) a.ring[(size_t(slot_s[i]) * a.ring_len + cpos_s[i] % a.ring_len) * a.conv_channels + c0 + c] = last[i];
        }
    }
    __syncthreads();
    if (kind < 2 ? a.unit_qk : a.unit_v) {  // a warp per token
        if (mine < TB) {
            float ss = 0.0f;
            for (uint32_t c = back; c < width; c += 32) ss += y[mine * width + c] * y[mine * width + c];
            ss = warp_sum(ss);
            if (back == 0) factor[mine] *= 1.0f / sqrtf(ss / float(width) + a.unit_eps);
            const RowNorm& weight = kind == 0 ? a.q_norm : a.k_norm;
            if (kind < 2 && weight.w)
                for (uint32_t c = back; c < width; c += 32) y[mine * width + c] *= weight_of(weight, c);
        }
        __syncthreads();
    }
    const uint32_t half = a.rot_dims / 2;
    const float share = kind == 2 && a.mix.share && !a.mix.first ? bf16_to_f32(*a.mix.share) : 0.0f;
    for (uint32_t c = tid; c < width; c += 128) {
#pragma unroll
        for (uint32_t i = 0; i < TB; i++) {
            if (i >= nt) break;
            const float* yi = y + i * width;
            float v = yi[c];
            if (kind < 2) v = rotated(yi, c, a.rot_dims, a.neighbours, reinterpret_cast<const float2*>(a.rope) + size_t(pos_s[i]) * half);
            v *= factor[i];
            if (kind == 2 && a.mix.share) {
                float* first = a.v_first + (size_t(t0 + i) * a.kv.n_kv + head) * width + c;
                if (a.mix.first) *first = v;
                else v = (1.0f - share) * v + share * *first;
            }
            if (kind == 0) {
                const size_t o = (size_t(t0 + i) * a.heads + head) * width + c;
                if (a.q_f) a.q_f[o] = v;
                if (a.q_b) a.q_b[o] = f32_to_bf16(v * a.q_scale);
            } else {
                store_kv(static_cast<T*>(kind == 1 ? a.kv.k : a.kv.v) + row_s[i] * width + c, v);
            }
        }
    }
}

// The last rows of every run into its slot's ring, for steps whose runs are long enough to wrap it (a run's first rows must
// have read the ring before its last ones overwrite it). grid (runs, rows of the ring, spans of 1024 channels).
__global__ void __launch_bounds__(256) conv_state_kernel(const ConvArgs a, const RunIn* __restrict__ runs) {
    pdl_start();
    const RunIn ru = runs[blockIdx.x];
    if (blockIdx.y >= ru.count) return;
    const uint32_t row = ru.count - 1 - blockIdx.y, pos = a.meta[2 * ru.first + 1] + row;
    const float* src = a.u + size_t(ru.first + row) * a.ldu;
    float* dst = a.ring + (size_t(ru.slot) * a.ring_len + pos % a.ring_len) * a.conv_channels;
    const uint32_t end = min(a.conv_channels, (blockIdx.z + 1) * 1024);
#pragma unroll
    for (uint32_t u = 0; u < 4; u++) {
        const uint32_t c = blockIdx.z * 1024 + u * 256 + threadIdx.x;
        if (c < end) dst[c] = src[c];
    }
}

// Attention of one token and query head per block: the cached keys that are kept and those from the chunk's or window's first position
// (or the sequence's) up to the token's tile of 8, then the tile's rows its `vis` names that it sees; softmax in fp32 with a running
// maximum over blocks of 128 keys; a sink's share and the gate, if there are such, on the result.
template <typename T>
__global__ void __launch_bounds__(128) attn_any_kernel(const ChunkedAttnArgs a) {
    pdl_start();
    extern __shared__ float sm[];
    float *q = sm, *o = sm + a.kv.dk, *p = o + a.kv.dv;
    __shared__ uint32_t rows[128];  // (a key's row in the pool; pools of more than 2^32 rows do not exist)
    __shared__ float red[8];
    const uint32_t t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, g = h / (a.heads / a.kv.n_kv);
    const paged::View view = paged::view_of(a, t);
    const uint32_t kept = min(view.keep, min(view.lo, view.first)), n_old = kept + (view.first > view.lo ? view.first - view.lo : 0);  // keys in front of the tile
    const T* K = static_cast<const T*>(a.kv.k);
    const T* V = static_cast<const T*>(a.kv.v);
    const uint32_t ldv = a.kv.v == a.kv.k ? a.kv.dk : a.kv.dv;
    for (uint32_t c = tid; c < a.kv.dk; c += 128) q[c] = a.q_f[(size_t(t) * a.heads + h) * a.kv.dk + c];
    for (uint32_t c = tid; c < a.kv.dv; c += 128) o[c] = 0.0f;
    float m = -INFINITY, l = 0.0f;
    const float slope = a.slopes ? a.slopes[h] : 0.0f;
    __syncthreads();
    for (uint32_t i0 = 0; i0 < n_old + 8; i0 += 128) {
        const uint32_t i = i0 + tid;
        float s = -INFINITY;
        const uint32_t kp = i < kept ? i : i < n_old ? view.lo + i - kept : view.first + i - n_old;
        if (i < n_old + 8 && paged::sees(view, kp)) {
            const size_t r = page_row(a.kv, view.slot, g, kp);
            rows[tid] = uint32_t(r);
            const T* k = K + r * a.kv.dk;
            float d = 0.0f;
            for (uint32_t c = 0; c < a.kv.dk; c++) d = fmaf(q[c], load_kv(k + c), d);
            s = d * a.scale;
            if (a.softcap > 0) s = a.softcap * tanhf(s / a.softcap);
            if (a.slopes) s -= slope * paged::distance(a, view, kp);
        }
        float mx = warp_max(s);
        if (tid % 32 == 0) red[tid / 32] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float mn = fmaxf(m, mx), corr = m == -INFINITY ? 0.0f : expf(m - mn), w = s == -INFINITY ? 0.0f : expf(s - mn);
        p[tid] = w;
        const float sum = warp_sum(w);
        if (tid % 32 == 0) red[4 + tid / 32] = sum;
        __syncthreads();
        if (mx != -INFINITY) {
            l = l * corr + ((red[4] + red[5]) + (red[6] + red[7]));
            m = mn;
            const uint32_t n = min(128u, n_old + 8 - i0);
            for (uint32_t c = tid; c < a.kv.dv; c += 128) {
                float acc = o[c] * corr;
                for (uint32_t j = 0; j < n; j++)
                    if (p[j] != 0.0f) acc = fmaf(p[j], load_kv(V + size_t(rows[j]) * ldv + c), acc);
                o[c] = acc;
            }
        }
        __syncthreads();
    }
    if (a.sink) l += expf(bf16_to_f32(a.sink[h]) - m);
    for (uint32_t c = tid; c < a.kv.dv; c += 128) {
        const float gt = a.gate ? 1.0f / (1.0f + expf(-a.gate[size_t(t) * a.ldg + h * a.kv.dv + c])) : 1.0f, y = o[c] / l * gt;
        const size_t at = (size_t(t) * a.heads + h) * a.kv.dv + c;
        if (a.out) a.out[at] = y;
        if (a.out_b) a.out_b[at] = f32_to_bf16(y);
    }
}

// The accepted path's rows of a verified draft tree, from where they were computed to where they belong: K and V in every
// layer run's pages, and the convolution's ring rows. grid (runs, mixers' caches); a thread keeps to its own columns.
template <typename T>
__global__ void __launch_bounds__(256) mixer_compact_kernel(const RunIn* __restrict__ runs, const uint32_t* __restrict__ path, const uint32_t* __restrict__ path_len,
                                                            const uint32_t* __restrict__ lens, const MixerCache* __restrict__ caches) {
    pdl_start();
    const uint32_t r = blockIdx.x, k = path_len[r];
    if (k < 2) return;
    const MixerCache mc = caches[blockIdx.y];
    const uint32_t slot = runs[r].slot, p0 = lens[slot] - k;
    for (uint32_t j = 1; j < k; j++) {
        const uint32_t from = path[r * FEED_W + j];
        if (from == j) continue;
        for (uint32_t g = 0; g < mc.kv.n_kv; g++) {
            const size_t src = page_row(mc.kv, slot, g, p0 + from), dst = page_row(mc.kv, slot, g, p0 + j);
            for (uint32_t c = threadIdx.x; c < mc.kv.dk; c += 256) static_cast<T*>(mc.kv.k)[dst * mc.kv.dk + c] = static_cast<const T*>(mc.kv.k)[src * mc.kv.dk + c];
            if (mc.kv.v != mc.kv.k)
                for (uint32_t c = threadIdx.x; c < mc.kv.dv; c += 256) static_cast<T*>(mc.kv.v)[dst * mc.kv.dv + c] = static_cast<const T*>(mc.kv.v)[src * mc.kv.dv + c];
        }
        float* ring = mc.ring + size_t(slot) * mc.ring_len * mc.channels;
        for (uint32_t c = threadIdx.x; c < mc.channels; c += 256) ring[size_t((p0 + j) % mc.ring_len) * mc.channels + c] = ring[size_t((p0 + from) % mc.ring_len) * mc.channels + c];
    }
}

// Small pseudo-random keys and values for positions that are not computed (benchmarks). grid (positions, mixers' caches).
template <typename T>
__global__ void __launch_bounds__(256) mixer_fill_kernel(const MixerCache* __restrict__ caches, uint32_t slot, uint32_t from, uint32_t seed) {
    const MixerCache mc = caches[blockIdx.y];
    const uint32_t pos = from + blockIdx.x;
    for (uint32_t g = 0; g < mc.kv.n_kv; g++) {
        const size_t r = page_row(mc.kv, slot, g, pos);
        for (uint32_t c = threadIdx.x; c < mc.kv.dk + (mc.kv.v == mc.kv.k ? 0 : mc.kv.dv); c += 256) {
            const float v = (float(philox(make_uint4(pos, blockIdx.y * 131 + g, c, slot), seed, 0xf111u).x >> 8) * 0x1p-24f - 0.5f) * 0.5f;
            if (c < mc.kv.dk) store_kv(static_cast<T*>(mc.kv.k) + r * mc.kv.dk + c, v);
            else store_kv(static_cast<T*>(mc.kv.v) + r * mc.kv.dv + c - mc.kv.dk, v);
        }
    }
}

}  // namespace mixer

void launch_conv_qkv(const ConvArgs& a, uint32_t n, bool fp32, cudaStream_t s) {
    const uint32_t units = a.heads + 2 * a.kv.n_kv, tb = n >= 64 ? 4 : 1;
    const dim3 grid((n + tb - 1) / tb, units);
    const size_t smem = size_t(tb) * std::max(a.kv.dk, a.kv.dv) * 4;
    if (tb == 1 && fp32) launch_pdl(mixer::conv_qkv_kernel<float, 1>, grid, 128, smem, s, a, n);
    else if (tb == 1) launch_pdl(mixer::conv_qkv_kernel<uint16_t, 1>, grid, 128, smem, s, a, n);
    else if (fp32) launch_pdl(mixer::conv_qkv_kernel<float, 4>, grid, 128, smem, s, a, n);
    else launch_pdl(mixer::conv_qkv_kernel<uint16_t, 4>, grid, 128, smem, s, a, n);
}
void launch_conv_state(const ConvArgs& a, const RunIn* runs, uint32_t n_runs, cudaStream_t s) {
    if (n_runs) launch_pdl(mixer::conv_state_kernel, dim3(n_runs, a.ring_len, (a.conv_channels + 1023) / 1024), 256, 0, s, a, runs);
}
void launch_attn_any(const ChunkedAttnArgs& a, uint32_t n, bool fp32, cudaStream_t s) {
    const size_t smem = (a.kv.dk + a.kv.dv + 128) * 4;  // (past 48 KB for rows of some 12 000 entries)
    if (fp32) launch_pdl(mixer::attn_any_kernel<float>, dim3(n, a.heads), 128, smem, s, a);
    else launch_pdl(mixer::attn_any_kernel<uint16_t>, dim3(n, a.heads), 128, smem, s, a);
}
void launch_mixer_compact(const RunIn* runs, const uint32_t* path, const uint32_t* path_len, const uint32_t* lens, const MixerCache* caches, uint32_t n_runs, uint32_t n_caches,
                          bool fp32, cudaStream_t s) {
    if (!n_runs) return;
    if (fp32) launch_pdl(mixer::mixer_compact_kernel<float>, dim3(n_runs, n_caches), 256, 0, s, runs, path, path_len, lens, caches);
    else launch_pdl(mixer::mixer_compact_kernel<uint16_t>, dim3(n_runs, n_caches), 256, 0, s, runs, path, path_len, lens, caches);
}
void launch_mixer_fill(const MixerCache* caches, uint32_t n_caches, uint32_t slot, uint32_t from, uint32_t to, uint32_t seed, bool fp32, cudaStream_t s) {
    if (to <= from) return;
    const dim3 grid(to - from, n_caches);
    if (fp32) mixer::mixer_fill_kernel<float><<<grid, 256, 0, s>>>(caches, slot, from, seed);
    else mixer::mixer_fill_kernel<uint16_t><<<grid, 256, 0, s>>>(caches, slot, from, seed);
    launch_counter()++;
}

}  // namespace vlt
