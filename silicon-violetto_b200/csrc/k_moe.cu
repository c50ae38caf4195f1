// A mixture of experts: the router (fp32 scores over the experts and the identity experts, by softmax or sigmoid; a correction that
// moves the choice but not the weights), the tokens sorted by expert, and the (weighted) sum of what the experts left. The experts' own
// matrices are grouped linear layers (k_linear.cu, k_grouped.cu).
#include <algorithm>

#include "kernels.h"

namespace vlt {

namespace moe {

// One block per TOK tokens: the RMS norm of their rows (kept for the experts; without a weight, the rows as they are), the scores'
// logits with a warp per output, the scores and the choice with a warp per token. Ties go to the lower index.
template <uint32_t TOK, uint32_t ROUTER_THREADS>
__global__ void __launch_bounds__(ROUTER_THREADS) router_kernel(const RouterArgs a) {
    pdl_start();
    extern __shared__ __align__(16) float sm[];
    constexpr uint32_t NW = ROUTER_THREADS / 32;
    const uint32_t t0 = blockIdx.x * TOK, tid = threadIdx.x, warp = tid / 32, lane = tid % 32, nt = min(TOK, a.n - t0);
    float *x = sm, *z = sm + TOK * a.d;  // the normed rows, the scores
    __shared__ float red[TOK][NW];
#pragma unroll
    for (uint32_t j = 0; j < TOK; j++) {
        float ss = 0.0f;
        if (j < nt)
            for (uint32_t i = tid; i < a.d; i += ROUTER_THREADS) {
                const float v = a.x[size_t(t0 + j) * a.d + i];
                x[j * a.d + i] = v;
                ss += v * v;
            }
        else
            for (uint32_t i = tid; i < a.d; i += ROUTER_THREADS) x[j * a.d + i] = 0.0f;
        ss = warp_sum(ss);
        if (lane == 0) red[j][warp] = ss;
    }
    __syncthreads();
#pragma unroll
    for (uint32_t j = 0; j < TOK; j++) {
        if (j >= nt) break;
        float tot = 0.0f;
        for (uint32_t w = 0; w < NW; w++) tot += red[j][w];
        if (!a.norm.w) break;
        const float inv = 1.0f / sqrtf(tot / float(a.d) + a.eps);
        for (uint32_t i = tid; i < a.d; i += ROUTER_THREADS) {
            const float v = x[j * a.d + i] * inv * weight_of(a.norm, i);
            x[j * a.d + i] = v;
            const size_t o = size_t(t0 + j) * a.d + i;
            if (a.xn) a.xn[o] = v;
            if (a.xn_b) a.xn_b[o] = f32_to_bf16(v);
        }
    }
    __syncthreads();
    const uint32_t all = a.experts + a.identity;
    // A warp takes EX outputs at a time over all the block's tokens, four neighbouring columns a lane and round: one read of x
    // serves EX outputs, one of the weights TOK tokens, and the loads of U rounds go out together.
    constexpr uint32_t EX = TOK == 1 ? 1 : 4, U = TOK == 1 ? 16 : 2;
    for (uint32_t e0 = warp * EX; e0 < all; e0 += NW * EX) {
        float s[EX][TOK] = {};
        uint32_t done = 0;
        if (a.d % 4 == 0) {
            const uint32_t groups = a.d / 4;
            for (uint32_t g0 = lane; g0 < groups; g0 += 32 * U) {
                uint2 v[U][EX];
#pragma unroll
                for (uint32_t u = 0; u < U; u++)
#pragma unroll
                    for (uint32_t k = 0; k < EX; k++)
                        v[u][k] = g0 + 32 * u < groups && e0 + k < all ? __ldg(reinterpret_cast<const uint2*>(a.router + size_t(e0 + k) * a.d) + g0 + 32 * u) : make_uint2(0, 0);
#pragma unroll
                for (uint32_t u = 0; u < U; u++) {
                    if (g0 + 32 * u >= groups) break;
#pragma unroll
                    for (uint32_t j = 0; j < TOK; j++) {
                        const float4 xv = *reinterpret_cast<const float4*>(x + j * a.d + (g0 + 32 * u) * 4);
#pragma unroll
                        for (uint32_t k = 0; k < EX; k++)
                            s[k][j] = fmaf(bf16lo(v[u][k].x), xv.x, fmaf(bf16hi(v[u][k].x), xv.y, fmaf(bf16lo(v[u][k].y), xv.z, fmaf(bf16hi(v[u][k].y), xv.w, s[k][j]))));
                    }
                }
            }
            done = a.d;
        }
        for (uint32_t i = done + lane; i < a.d; i += 32)
#pragma unroll
            for (uint32_t k = 0; k < EX; k++) {
                const float wv = e0 + k < all ? bf16_to_f32(a.router[size_t(e0 + k) * a.d + i]) : 0.0f;
#pragma unroll
                for (uint32_t j = 0; j < TOK; j++) s[k][j] = fmaf(wv, x[j * a.d + i], s[k][j]);
            }
#pragma unroll
        for (uint32_t k = 0; k < EX; k++)
#pragma unroll
            for (uint32_t j = 0; j < TOK; j++) {
                const float sum = warp_sum(s[k][j]);
                if (lane == 0 && e0 + k < all) z[j * all + e0 + k] = sum;
            }
    }
    __syncthreads();
    if (warp >= nt) return;
    for (uint32_t j = warp; j < nt; j += NW) {
        float* zt = z + j * all;
        const uint32_t t = t0 + j;
        if (a.sigmoid) {
            for (uint32_t e = lane; e < all; e += 32) zt[e] = sigmoid_of(zt[e]);
        } else {
            float m = -INFINITY, sum = 0.0f;
            for (uint32_t e = lane; e < all; e += 32) m = fmaxf(m, zt[e]);
            m = warp_max(m);
            for (uint32_t e = lane; e < all; e += 32) {
                const float p = expf(zt[e] - m);
                zt[e] = p;
                sum += p;
            }
            sum = warp_sum(sum);
            for (uint32_t e = lane; e < all; e += 32) zt[e] = zt[e] / sum;
        }
        __syncwarp();
        // The choice: the largest score + correction, `top` times, ties to the lower index. Kept as integers that order as
        // the numbers do (0: chosen already), so that a warp's maximum is one instruction.
        uint32_t* ct = reinterpret_cast<uint32_t*>(z + TOK * all) + j * all;
        for (uint32_t e = lane; e < all; e += 32) {
            const uint32_t u = __float_as_uint(a.correction ? zt[e] + bf16_to_f32(a.correction[e]) : zt[e]);
            ct[e] = max(u & 0x80000000u ? ~u : u | 0x80000000u, 1u);
        }
        __syncwarp();
        float total = 0.0f, kept = 0.0f;  // lane k keeps choice k's score (past 32 they wait in memory)
        for (uint32_t k = 0; k < a.top; k++) {
            uint32_t bv = 0, bi = all;
            for (uint32_t e = lane; e < all; e += 32)
                if (ct[e] > bv) { bv = ct[e]; bi = e; }
            const uint32_t best = __reduce_max_sync(0xffffffffu, bv);
            bi = __reduce_min_sync(0xffffffffu, bv == best ? bi : all);
            if (bi >= all) bi = 0;  // (never: there are at least `top` outputs)
            const float s = zt[bi];
            total += s;
            __syncwarp();
            if (lane == 0) {
                ct[bi] = 0;
                a.ids[size_t(t) * a.top + k] = bi;
                if (k >= 32) a.weights[size_t(t) * a.top + k] = s;
            }
            if (lane == k) kept = s;
            __syncwarp();
        }
        const float inv = a.renormalized ? 1.0f / (total + 1e-20f) : 1.0f;
        if (lane < a.top) a.weights[size_t(t) * a.top + lane] = kept * inv;
        for (uint32_t k = 32 + lane; k < a.top; k += 32) a.weights[size_t(t) * a.top + k] *= inv;
    }
}

// The (token, choice) pairs in expert order, by one block: counts, their prefix sums, the pairs' places, and the table of
// (expert, first row, rows <= tile) tiles the grouped linear layers run over. Which of an expert's rows a token gets is left
// to the atomics; nothing depends on it.
__global__ void __launch_bounds__(1024) sort_kernel(const SortArgs a) {
    pdl_start();
    extern __shared__ uint32_t sh[];
    uint32_t *cnt = sh, *cur = sh + a.experts, *tile0 = cur + a.experts;
    __shared__ uint32_t n_tiles;
    const uint32_t tid = threadIdx.x, pairs = a.n * a.top;
    for (uint32_t e = tid; e < a.experts; e += 1024) cnt[e] = 0;
    __syncthreads();
    for (uint32_t i = tid; i < pairs; i += 1024) {
        const uint32_t e = a.ids[i];
        if (e < a.experts) atomicAdd(cnt + e, 1u);
    }
    __syncthreads();
    if (tid < 32) {
        uint32_t rows = 0, tiles = 0;
        for (uint32_t e0 = 0; e0 < a.experts; e0 += 32) {
            const uint32_t e = e0 + tid, c = e < a.experts ? cnt[e] : 0, k = (c + a.tile - 1) / a.tile;
            uint32_t sc = c, sk = k;
#pragma unroll
            for (uint32_t o = 1; o < 32; o *= 2) {
                const uint32_t pc = __shfl_up_sync(0xffffffffu, sc, o), pk = __shfl_up_sync(0xffffffffu, sk, o);
                if (tid >= o) { sc += pc; sk += pk; }
            }
            if (e < a.experts) { cur[e] = rows + sc - c; tile0[e] = tiles + sk - k; }
            rows += __shfl_sync(0xffffffffu, sc, 31);
            tiles += __shfl_sync(0xffffffffu, sk, 31);
        }
        if (tid == 0) { n_tiles = tiles; *a.n_tiles = tiles; }
    }
    __syncthreads();
    for (uint32_t e = tid; e < a.experts; e += 1024)
        for (uint32_t k = 0, at = tile0[e]; k < cnt[e]; k += a.tile, at++) {
            a.tiles[3 * at] = e;
            a.tiles[3 * at + 1] = cur[e] + k;
            a.tiles[3 * at + 2] = min(a.tile, cnt[e] - k);
        }
    __syncthreads();
    for (uint32_t i = tid; i < pairs; i += 1024) {
        const uint32_t e = a.ids[i];
        if (e < a.experts) {
            const uint32_t p = atomicAdd(cur + e, 1u);
            a.src[p] = i / a.top;
            a.place[i] = p;
            if (a.row_weight) a.row_weight[p] = a.weights[i];
        }
    }
}

// out[t] = x[t] + sum_k weight_k (expert k's row, or the token's own normed row for an identity expert) + the shared
// expert's row, in the order of the choice; and, if asked, the next layer's RMS norm of it. With `post`, what is added to x[t] is
// the sum's RMS norm. A block per token; V: the columns a thread takes at a time.
template <typename V>
__device__ __forceinline__ void fma_v(V& y, float w, const V& v);
template <>
__device__ __forceinline__ void fma_v<float>(float& y, float w, const float& v) { y = fmaf(w, v, y); }
template <>
__device__ __forceinline__ void fma_v<float4>(float4& y, float w, const float4& v) {
    y.x = fmaf(w, v.x, y.x);
    y.y = fmaf(w, v.y, y.y);
    y.z = fmaf(w, v.z, y.z);
    y.w = fmaf(w, v.w, y.w);
}
__device__ __forceinline__ float square(float y) { return y * y; }
__device__ __forceinline__ float square(const float4& y) { return (y.x * y.x + y.y * y.y) + (y.z * y.z + y.w * y.w); }

template <typename V>
__global__ void __launch_bounds__(256) combine_kernel(const CombineArgs a) {
    pdl_start();
    extern __shared__ __align__(16) float row[];  // the new row, then the choices' weights and rows
    constexpr uint32_t W = sizeof(V) / 4;
    __shared__ float red[8];
    const uint32_t t = blockIdx.x, tid = threadIdx.x, dv = a.d / W;
    float* wt = row + (a.d + 3) / 4 * 4;
    const float** src = reinterpret_cast<const float**>(wt + (a.top + 1) / 2 * 2);
    for (uint32_t k = tid; k < a.top; k += 256) {
        const size_t i = size_t(t) * a.top + k;
        wt[k] = a.weights ? a.weights[i] : 1.0f;
        src[k] = a.ids[i] < a.experts ? a.y + size_t(a.place[i]) * a.d : a.xn + size_t(t) * a.d;
    }
    __syncthreads();
    const V one{};
    float ss = 0.0f;
    for (uint32_t i = tid; i < dv; i += 256) {
        V y = one, x = one, sh = one;
        if (!a.post.w) x = reinterpret_cast<const V*>(a.x + size_t(t) * a.d)[i];
        if (a.shared) sh = reinterpret_cast<const V*>(a.shared + size_t(t) * a.d)[i];
        for (uint32_t k0 = 0; k0 < a.top; k0 += 8) {
            V v[8];
#pragma unroll
            for (uint32_t u = 0; u < 8; u++) v[u] = k0 + u < a.top ? reinterpret_cast<const V*>(src[k0 + u])[i] : one;
#pragma unroll
            for (uint32_t u = 0; u < 8; u++)
                if (k0 + u < a.top) fma_v(y, wt[k0 + u], v[u]);
        }
        fma_v(y, 1.0f, sh);
        fma_v(y, 1.0f, x);
        if (!a.post.w) reinterpret_cast<V*>(a.out + size_t(t) * a.d)[i] = y;
        reinterpret_cast<V*>(row)[i] = y;
        ss += square(y);
    }
    if (!a.norm.w && !a.post.w) return;
    ss = warp_sum(ss);
    if (tid % 32 == 0) red[tid / 32] = ss;
    __syncthreads();
    float tot = 0.0f;
    for (uint32_t w = 0; w < 8; w++) tot += red[w];
    const float inv = 1.0f / sqrtf(tot / float(a.d) + a.eps);
    if (a.post.w) {
        for (uint32_t i = tid * W; i < a.d; i += 256 * W) {
            const size_t o = size_t(t) * a.d + i;
            float x[W], y[W], w[W];
            load_f32<W>(x, a.x + o);
            load_f32<W>(y, row + i);
            weights_of<W>(w, a.post, i);
#pragma unroll
            for (uint32_t j = 0; j < W; j++) x[j] += y[j] * inv * w[j];
            store_f32<W>(a.out + o, x);
            if (a.next_b) store_bf16<W>(a.next_b + o, x);
        }
        return;
    }
    for (uint32_t i = tid; i < a.d; i += 256) {
        const size_t o = size_t(t) * a.d + i;
        const float v = row[i] * inv * weight_of(a.norm, i);
        if (a.next) a.next[o] = v;
        if (a.next_b) a.next_b[o] = f32_to_bf16(v);
    }
}

}  // namespace moe

void launch_router(const RouterArgs& a, cudaStream_t s) {
    const uint32_t all = a.experts + a.identity;
    static PerDevice configured;
    configured.once([] {
        VLT_CUDA(cudaFuncSetAttribute(moe::router_kernel<1, 1024>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        VLT_CUDA(cudaFuncSetAttribute(moe::router_kernel<1, 512>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        VLT_CUDA(cudaFuncSetAttribute(moe::router_kernel<4, 512>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    });
    // Many tokens share a read of the router's matrix, four a block; few spread over the SMs one by one.
    const size_t one = (size_t(a.d) + 2 * all) * 4;  // the normed row, the scores, what the choice goes by
    if (a.n >= 256 && one <= 25 * 1024) launch_pdl(moe::router_kernel<4, 512>, (a.n + 3) / 4, 512, 4 * one, s, a);
    else if (a.n > 148) launch_pdl(moe::router_kernel<1, 512>, a.n, 512, one, s, a);
    else launch_pdl(moe::router_kernel<1, 1024>, a.n, 1024, one, s, a);
}
void launch_expert_sort(const SortArgs& a, cudaStream_t s) { launch_pdl(moe::sort_kernel, 1, 1024, size_t(a.experts) * 12, s, a); }
void launch_combine(const CombineArgs& a, uint32_t n, cudaStream_t s) {
    const size_t smem = (size_t(a.d) + 3) / 4 * 16 + (size_t(a.top) + 1) / 2 * 8 + size_t(a.top) * 8;
    static PerDevice configured;
    configured.once([] {
        VLT_CUDA(cudaFuncSetAttribute(moe::combine_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        VLT_CUDA(cudaFuncSetAttribute(moe::combine_kernel<float4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    });
    if (a.d % 4 == 0) launch_pdl(moe::combine_kernel<float4>, n, 256, smem, s, a);
    else launch_pdl(moe::combine_kernel<float>, n, 256, smem, s, a);
}

}  // namespace vlt
