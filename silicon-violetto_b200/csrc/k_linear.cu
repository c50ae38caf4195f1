// Linear layers on the CUDA cores, for what the tensor-core kernels do not take: activations in fp32 throughout (true fp32
// products and sums: bf16 weights are exact in fp32), and matrices whose sizes fit neither the streamed kernel nor the GEMM.
// Also the row passes around a projection: norms in front of it or of what it leaves, two streams side by side, two mixers'
// outputs onto the stream, the average over the layers' results, and a side input's gate.
#include <algorithm>

#include "kernels.h"

namespace vlt {

namespace linear {

constexpr uint32_t BM = 64, BN = 64, BK = 16;  // weight rows x tokens x k of a block's tile

__device__ __forceinline__ float load_x(const float* p) { return *p; }
__device__ __forceinline__ float load_x(const uint16_t* p) { return bf16_to_f32(*p); }

// Y[p][r] = epilogue(W_g[r] . X[src(p)]) for the rows r of a 64-row tile and the tokens p of a tile of at most 64. One
// group: the tiles are the tokens in order; several (experts): a table of (group, first row, rows) tiles built on the device.
template <typename T>
__global__ void __launch_bounds__(256) linear_kernel(const LinearArgs a) {
    pdl_start();
    __shared__ float ws[BK][BM + 4], xs[BK][BN + 4];
    uint32_t group = 0, p0 = blockIdx.y * BN, count;
    if (a.tiles) {
        if (blockIdx.y >= *a.n_tiles) return;
        group = a.tiles[3 * blockIdx.y];
        p0 = a.tiles[3 * blockIdx.y + 1];
        count = a.tiles[3 * blockIdx.y + 2];
    } else {
        count = min(BN, a.n - p0);
    }
    const uint32_t r0 = blockIdx.x * BM, tid = threadIdx.x;
    const uint16_t* W = a.W + size_t(group) * a.m * a.k;
    const T* X = static_cast<const T*>(a.X);
    const uint32_t tr = tid % 16, tt = tid / 16;  // rows tr + 16 i, tokens tt + 16 j of the tile
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < a.k; k0 += BK) {
        for (uint32_t i = tid; i < BM * BK; i += 256) {
            const uint32_t kk = i % BK, r = i / BK;
            ws[kk][r] = r0 + r < a.m && k0 + kk < a.k ? bf16_to_f32(W[size_t(r0 + r) * a.k + k0 + kk]) : 0.0f;
            const uint32_t p = p0 + r;
            const size_t from = a.src ? a.src[p] : a.by_head ? size_t(p - group * a.by_head) * a.heads + group : p;
            xs[kk][r] = r < count && k0 + kk < a.k ? load_x(X + from * a.k + k0 + kk) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (uint32_t kk = 0; kk < BK; kk++) {
            float w[4], x[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { w[i] = ws[kk][tr + 16 * i]; x[i] = xs[kk][tt + 16 * i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(w[i], x[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 4; j++) {
        const uint32_t p = tt + 16 * j;
        const float scale = a.row_scale && p < count ? a.row_scale[p0 + p] : 1.0f;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const uint32_t r = r0 + tr + 16 * i;
            float y = acc[i][j] * scale;
            if (a.bias && r < a.m) y += bf16_to_f32(a.bias[r]);
            const bool pairs = epi_pairs(a.epi);  // (a pair's rows are neighbouring lanes')
            const float u = pairs ? __shfl_xor_sync(0xffffffffu, y, 1) : 0.0f;
            if (p >= count || r >= a.m || (pairs && r % 2)) continue;
            size_t o = pairs ? size_t(p0 + p) * (a.m / 2) + r / 2 : size_t(p0 + p) * a.m + r;
            if (a.by_head) {
                const size_t t = p0 + p - group * a.by_head;
                if (a.gate) y *= sigmoid_of(a.gate[t * a.ldg + (a.gate_w == 1 ? group : size_t(group) * a.m + r)]);
                o = (t * a.heads + group) * a.ldy + r;
            }
            if (a.epi == EPI_RESID) y += a.base[o];
            else if (a.epi == EPI_RELU2) y = y > 0.0f ? y * y : 0.0f;
            else if (a.epi == EPI_SILU) y = r < a.act_rows ? y * sigmoid_of(y) : y;
            else if (a.epi == EPI_GLU) y = y * sigmoid_of(y) * u;
            else if (a.epi == EPI_GLU_CLAMP) y = clamped_glu(y, u, a.limit);
            if (a.Y) a.Y[o] = y;
            if (a.Yb) a.Yb[o] = f32_to_bf16(y);
        }
    }
}

// What a norm makes of the row a block keeps in shared memory, each thread its own entries; ss: their squares' sum if it is not centered.
template <uint32_t V>
__device__ __forceinline__ void norm_row(float* row, uint32_t width, const RowNorm& norm, float ss, float eps, float scale, float* red, float* out, uint16_t* out_b) {
    const uint32_t tid = threadIdx.x * V, step = blockDim.x * V;
    float mean = 0.0f;
    if (norm.centered) {  // (the squares in a pass of their own: of what is left of the row)
        float sum = 0.0f;
        for (uint32_t i = tid; i < width; i += step)
#pragma unroll
            for (uint32_t j = 0; j < V; j++) sum += row[i + j];
        mean = block_sum(sum, red) / float(width);
        red += 32;
        ss = 0.0f;
        for (uint32_t i = tid; i < width; i += step)
#pragma unroll
            for (uint32_t j = 0; j < V; j++) ss += (row[i + j] - mean) * (row[i + j] - mean);
    }
    const float inv = scale / sqrtf(block_sum(ss, red) / float(width) + eps);
    for (uint32_t i = tid; i < width; i += step) {
        float x[V], w[V];
        load_f32<V>(x, row + i);
        weights_of<V>(w, norm, i);
        if (norm.centered)
#pragma unroll
            for (uint32_t j = 0; j < V; j++) x[j] -= mean;
#pragma unroll
        for (uint32_t j = 0; j < V; j++) x[j] *= inv * w[j];
        if (norm.b) {
            load_bf16<V>(w, norm.b + i);
#pragma unroll
            for (uint32_t j = 0; j < V; j++) x[j] += scale * w[j];
        }
        if (out) store_f32<V>(out + i, x);
        if (out_b) store_bf16<V>(out_b + i, x);
    }
}

// See NormArgs. A block per row.
template <uint32_t V>
__global__ void __launch_bounds__(1024) norm_rows_kernel(const NormArgs a) {
    pdl_start();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[64];
    const uint32_t r = blockIdx.x, tid = threadIdx.x * V, step = blockDim.x * V;
    const size_t from = size_t(a.rows ? a.rows[r] : r) * a.k;
    float ss = 0.0f;
    for (uint32_t i = tid; i < a.k; i += step) {
        float x[V];
        load_f32<V>(x, a.in + from + i);
        if (a.add) {
            float y[V];
            load_f32<V>(y, a.add + from + i);
#pragma unroll
            for (uint32_t j = 0; j < V; j++) x[j] += y[j];
            store_f32<V>(a.sum + from + i, x);
        }
        store_f32<V>(row + i, x);
#pragma unroll
        for (uint32_t j = 0; j < V; j++) ss += x[j] * x[j];
    }
    const size_t to = size_t(r) * a.k;
    norm_row<V>(row, a.k, a.norm, ss, a.eps, a.scale, red, a.out_f32 ? a.out_f32 + to : nullptr, a.out_bf16 ? a.out_bf16 + to : nullptr);
}

// See DepthArgs. A block per row.
template <uint32_t V>
__global__ void __launch_bounds__(1024) depth_average_kernel(const DepthArgs a) {
    pdl_start();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[64];
    const uint32_t tid = threadIdx.x * V, step = blockDim.x * V;
    const size_t from = size_t(blockIdx.x) * a.d;
    constexpr uint32_t AT_ONCE = 4;  // results whose loads go out together
    float ss = 0.0f;
    for (uint32_t i = tid; i < a.d; i += step) {
        float sum[V] = {};
        for (uint32_t j0 = 0; j0 < a.count; j0 += AT_ONCE) {
            float x[AT_ONCE][V], share[AT_ONCE];
#pragma unroll
            for (uint32_t k = 0; k < AT_ONCE; k++) {
                const uint32_t j = min(j0 + k, a.count - 1);
                share[k] = j0 + k < a.count ? bf16_to_f32(a.share[j]) : 0.0f;
                load_f32<V>(x[k], a.x + j * a.stride + from + i);
            }
#pragma unroll
            for (uint32_t k = 0; k < AT_ONCE; k++)
                if (j0 + k < a.count)
#pragma unroll
                    for (uint32_t v = 0; v < V; v++) sum[v] = fmaf(share[k], x[k][v], sum[v]);
        }
        store_f32<V>(a.out + from + i, sum);
        store_f32<V>(row + i, sum);
#pragma unroll
        for (uint32_t v = 0; v < V; v++) ss += sum[v] * sum[v];
    }
    if (a.norm.w) norm_row<V>(row, a.d, a.norm, ss, a.eps, 1.0f, red, a.next ? a.next + from : nullptr, a.next_b ? a.next_b + from : nullptr);
}

// See MergeArgs. A block per row.
template <uint32_t V>
__global__ void __launch_bounds__(1024) merge_rows_kernel(const MergeArgs a) {
    pdl_start();
    extern __shared__ __align__(16) float rows[];  // the two outputs; the first then holds the sum
    __shared__ float red[3][32];
    float *ra = rows, *rb = rows + a.d;
    const uint32_t tid = threadIdx.x * V, step = blockDim.x * V;
    const size_t from = size_t(blockIdx.x) * a.d;
    float sa = 0.0f, sb = 0.0f;
    for (uint32_t i = tid; i < a.d; i += step) {
        float p[V], q[V];
        load_f32<V>(p, a.a + from + i);
        load_f32<V>(q, a.b + from + i);
        store_f32<V>(ra + i, p);
        store_f32<V>(rb + i, q);
#pragma unroll
        for (uint32_t j = 0; j < V; j++) { sa += p[j] * p[j]; sb += q[j] * q[j]; }
    }
    const float ia = 0.5f / sqrtf(block_sum(sa, red[0]) / float(a.d) + a.eps), ib = 0.5f / sqrtf(block_sum(sb, red[1]) / float(a.d) + a.eps);
    float ss = 0.0f;
    for (uint32_t i = tid; i < a.d; i += step) {
        float p[V], q[V], x[V], wa[V], wb[V];
        load_f32<V>(p, ra + i);
        load_f32<V>(q, rb + i);
        load_f32<V>(x, a.x + from + i);
        weights_of<V>(wa, a.norm_a, i);
        weights_of<V>(wb, a.norm_b, i);
#pragma unroll
        for (uint32_t j = 0; j < V; j++) {
            x[j] += p[j] * ia * wa[j] + q[j] * ib * wb[j];
            ss += x[j] * x[j];
        }
        store_f32<V>(a.out + from + i, x);
        store_f32<V>(ra + i, x);
    }
    if (!a.norm.w) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, red[2]) / float(a.d) + a.eps);
    for (uint32_t i = tid; i < a.d; i += step) {
        float x[V], w[V];
        load_f32<V>(x, ra + i);
        weights_of<V>(w, a.norm, i);
#pragma unroll
        for (uint32_t j = 0; j < V; j++) x[j] *= inv * w[j];
        if (a.next) store_f32<V>(a.next + from + i, x);
        if (a.next_b) store_bf16<V>(a.next_b + from + i, x);
    }
}

// See AddNormArgs. A block per row.
template <uint32_t V>
__global__ void __launch_bounds__(1024) add_norm_kernel(const AddNormArgs a) {
    pdl_start();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[32];
    const uint32_t tid = threadIdx.x * V, step = blockDim.x * V;
    const size_t from = size_t(blockIdx.x) * a.d;
    float ss = 0.0f;
    for (uint32_t i = tid; i < a.d; i += step) {
        float y[V];
        load_f32<V>(y, a.y + from + i);
        store_f32<V>(row + i, y);
#pragma unroll
        for (uint32_t j = 0; j < V; j++) ss += y[j] * y[j];
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / float(a.d) + a.eps);
    for (uint32_t i = tid; i < a.d; i += step) {
        float x[V], y[V], w[V];
        load_f32<V>(x, a.x + from + i);
        load_f32<V>(y, row + i);
        weights_of<V>(w, a.norm, i);
#pragma unroll
        for (uint32_t j = 0; j < V; j++) x[j] += y[j] * inv * w[j];
        store_f32<V>(a.out + from + i, x);
        if (a.out_b) store_bf16<V>(a.out_b + from + i, x);
    }
}

// See SideGateArgs. grid (tokens, spans of 256 columns).
__global__ void __launch_bounds__(256) side_gate_kernel(const SideGateArgs a) {
    pdl_start();
    const uint32_t t = blockIdx.x, i = blockIdx.y * 256 + threadIdx.x;
    if (i >= a.side.wide) return;
    const float y = side_of(a.side, t, i, i < a.side.dim ? a.x[size_t(t) * a.ldx + i] : 0.0f);
    const size_t o = size_t(t) * a.side.wide + i;
    if (a.out_f32) a.out_f32[o] = y;
    if (a.out_bf16) a.out_bf16[o] = f32_to_bf16(y);
}

// out[r] = (a[r] ; b[r]).
__global__ void __launch_bounds__(256) concat_rows_kernel(const float* __restrict__ a, const float* __restrict__ b, uint32_t d, float* out_f32, uint16_t* out_bf16) {
    pdl_start();
    const size_t r = blockIdx.x;
    for (uint32_t i = threadIdx.x; i < 2 * d; i += 256) {
        const float v = i < d ? a[r * d + i] : b[r * d + i - d];
        if (out_f32) out_f32[r * 2 * d + i] = v;
        if (out_bf16) out_bf16[r * 2 * d + i] = f32_to_bf16(v);
    }
}

}  // namespace linear

void launch_linear(const LinearArgs& a, bool x_bf16, cudaStream_t s) {
    const uint32_t tiles = a.tiles ? a.max_tiles : (a.n + linear::BN - 1) / linear::BN;
    if (!tiles) return;
    const dim3 grid((a.m + linear::BM - 1) / linear::BM, tiles);
    if (x_bf16) launch_pdl(linear::linear_kernel<uint16_t>, grid, 256, 0, s, a);
    else launch_pdl(linear::linear_kernel<float>, grid, 256, 0, s, a);
}
void launch_norm_rows(const NormArgs& a, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] {
        for (auto f : {linear::norm_rows_kernel<1>, linear::norm_rows_kernel<4>}) VLT_CUDA(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    });
    if (!a.n) return;
    if (a.k % 4 == 0) launch_pdl(linear::norm_rows_kernel<4>, a.n, row_threads(a.k, 4), size_t(a.k) * 4, s, a);
    else launch_pdl(linear::norm_rows_kernel<1>, a.n, row_threads(a.k, 1), size_t(a.k) * 4, s, a);
}
void launch_merge_rows(const MergeArgs& a, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] {
        for (auto f : {linear::merge_rows_kernel<1>, linear::merge_rows_kernel<4>}) VLT_CUDA(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    });
    if (!a.n) return;
    if (a.d % 4 == 0) launch_pdl(linear::merge_rows_kernel<4>, a.n, row_threads(a.d, 4), size_t(a.d) * 8, s, a);
    else launch_pdl(linear::merge_rows_kernel<1>, a.n, row_threads(a.d, 1), size_t(a.d) * 8, s, a);
}
void launch_add_norm(const AddNormArgs& a, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] {
        for (auto f : {linear::add_norm_kernel<1>, linear::add_norm_kernel<4>}) VLT_CUDA(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    });
    if (!a.n) return;
    if (a.d % 4 == 0) launch_pdl(linear::add_norm_kernel<4>, a.n, row_threads(a.d, 4), size_t(a.d) * 4, s, a);
    else launch_pdl(linear::add_norm_kernel<1>, a.n, row_threads(a.d, 1), size_t(a.d) * 4, s, a);
}
void launch_depth_average(const DepthArgs& a, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] {
        for (auto f : {linear::depth_average_kernel<1>, linear::depth_average_kernel<4>}) VLT_CUDA(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    });
    if (!a.n) return;
    if (a.d % 4 == 0) launch_pdl(linear::depth_average_kernel<4>, a.n, row_threads(a.d, 4), size_t(a.d) * 4, s, a);
    else launch_pdl(linear::depth_average_kernel<1>, a.n, row_threads(a.d, 1), size_t(a.d) * 4, s, a);
}
void launch_side_gate(const SideGateArgs& a, cudaStream_t s) {
    if (a.n) launch_pdl(linear::side_gate_kernel, dim3(a.n, (a.side.wide + 255) / 256), 256, 0, s, a);
}
void launch_concat_rows(const float* a, const float* b, uint32_t n, uint32_t d, float* out_f32, uint16_t* out_bf16, cudaStream_t s) {
    if (n) launch_pdl(linear::concat_rows_kernel, n, 256, 0, s, a, b, d, out_f32, out_bf16);
}

}  // namespace vlt
