// Latent attention's rows between its projections: the normed query row and the cached (c ; r) from the first one, and the queries
// as the per-head products and the attention take them from the second.
#include <algorithm>

#include "kernels.h"

namespace vlt {

namespace latent {

__device__ __forceinline__ void store(float* p, float v) { *p = v; }
__device__ __forceinline__ void store(uint16_t* p, float v) { *p = f32_to_bf16(v); }

// Token t's query row, or its (c ; r). T: the cache's element.
template <typename T>
__device__ __forceinline__ void normed_row(const LatentRowsArgs& a, uint32_t t, bool key, float* red) {
    const uint32_t tid = threadIdx.x, width = key ? a.kv_rank : a.q_rank;
    const float* u = a.u + size_t(t) * a.ldu + (key ? a.key_at : 0);
    const RowNorm& norm = key ? a.kv_norm : a.q_norm;
    float ss = 0.0f;
    for (uint32_t i = tid; i < width; i += 256) ss += u[i] * u[i];
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / float(width) + a.eps);
    if (!key) {
        for (uint32_t i = tid; i < width; i += 256) {
            const float v = u[i] * inv * weight_of(norm, i);
            if (a.q_f) a.q_f[size_t(t) * width + i] = v;
            if (a.q_b) a.q_b[size_t(t) * width + i] = f32_to_bf16(v);
        }
        return;
    }
    const uint32_t pos = a.meta[2 * t + 1], row = a.tin[2 * t + 1], cpos = a.meta[2 * (t - row) + 1] + row;
    T* dst = static_cast<T*>(a.kv.k) + page_row(a.kv, a.meta[2 * t], 0, cpos) * a.kv.dk;
    for (uint32_t i = tid; i < width; i += 256) store(dst + i, u[i] * inv * weight_of(norm, i));
    const float2* cs = reinterpret_cast<const float2*>(a.rope) + size_t(pos) * (a.rot_dim / 2);
    for (uint32_t i = tid; i < a.rot_dim; i += 256) store(dst + width + i, rotated(u + width, i, a.rot_dim, a.neighbours, cs));
}

// Token t's queries, a span of 1024 of their entries.
__device__ __forceinline__ void query_span(const LatentQueryArgs& a, uint32_t t, uint32_t span) {
    const uint32_t tid = threadIdx.x, head_w = a.dim + a.rot_dim, all = a.heads * head_w;
    if (t == 0 && span == 0) {
        const uint32_t per = (a.n + a.tile - 1) / a.tile;
        for (uint32_t i = tid; i < a.heads * per; i += 256) {
            const uint32_t h = i / per, p = i % per * a.tile;
            a.tiles[3 * i] = h;
            a.tiles[3 * i + 1] = h * a.n + p;
            a.tiles[3 * i + 2] = min(a.tile, a.n - p);
        }
        if (tid == 0) *a.n_tiles = a.heads * per;
    }
    const float* u = a.u + size_t(t) * a.ldu;
    const float2* cs = reinterpret_cast<const float2*>(a.rope) + size_t(a.meta[2 * t + 1]) * (a.rot_dim / 2);
    const uint32_t end = min(all, (span + 1) * 1024);
    for (uint32_t i = span * 1024 + tid; i < end; i += 256) {
        const uint32_t h = i / head_w, c = i % head_w;
        if (c < a.dim) {
            const size_t o = (size_t(t) * a.heads + h) * a.dim + c;
            const float v = u[i] * a.factor;
            if (a.part_f) a.part_f[o] = v;
            if (a.part_b) a.part_b[o] = f32_to_bf16(v);
        } else {
            const size_t o = (size_t(t) * a.heads + h) * (a.kv_rank + a.rot_dim) + a.kv_rank + c - a.dim;
            const float v = rotated(u + h * head_w + a.dim, c - a.dim, a.rot_dim, a.neighbours, cs) * a.factor;
            if (a.q_f) a.q_f[o] = v;
            if (a.q_b) a.q_b[o] = f32_to_bf16(v);
        }
    }
}

// grid (tokens, 1 or 2): the query row; (c ; r) if it is this layer's own.
template <typename T>
__global__ void __launch_bounds__(256) rows_kernel(const LatentRowsArgs a) {
    pdl_start();
    __shared__ float red[32];
    normed_row<T>(a, blockIdx.x, blockIdx.y == 1, red);
}

// grid (tokens, spans).
__global__ void __launch_bounds__(256) query_kernel(const LatentQueryArgs a) {
    pdl_start();
    query_span(a, blockIdx.x, blockIdx.y);
}

// grid (tokens, 1 + spans).
template <typename T>
__global__ void __launch_bounds__(256) split_kernel(const LatentRowsArgs r, const LatentQueryArgs q) {
    pdl_start();
    __shared__ float red[32];
    if (blockIdx.y == 0) normed_row<T>(r, blockIdx.x, true, red);
    else query_span(q, blockIdx.x, blockIdx.y - 1);
}

}  // namespace latent

void launch_latent_rows(const LatentRowsArgs& a, uint32_t n, bool fp32, cudaStream_t s) {
    const dim3 grid(n, a.own ? 2 : 1);
    if (fp32) launch_pdl(latent::rows_kernel<float>, grid, 256, 0, s, a);
    else launch_pdl(latent::rows_kernel<uint16_t>, grid, 256, 0, s, a);
}
void launch_latent_query(const LatentQueryArgs& a, cudaStream_t s) {
    launch_pdl(latent::query_kernel, dim3(a.n, (a.heads * (a.dim + a.rot_dim) + 1023) / 1024), 256, 0, s, a);
}
void launch_latent_split(const LatentRowsArgs& r, const LatentQueryArgs& q, bool fp32, cudaStream_t s) {
    const dim3 grid(q.n, 1 + (q.heads * (q.dim + q.rot_dim) + 1023) / 1024);
    if (fp32) launch_pdl(latent::split_kernel<float>, grid, 256, 0, s, r, q);
    else launch_pdl(latent::split_kernel<uint16_t>, grid, 256, 0, s, r, q);
}

}  // namespace vlt
