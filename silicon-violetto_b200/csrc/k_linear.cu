// Linear layers on the CUDA cores, for what the tensor-core kernels do not take: activations in fp32 throughout (true fp32
// products and sums: bf16 weights are exact in fp32), and matrices whose sizes fit neither the streamed kernel nor the GEMM.
// Also the row passes in front of a projection: RMS norms, two streams side by side, and two mixers' outputs onto the stream.
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
            xs[kk][r] = r < count && k0 + kk < a.k ? load_x(X + size_t(a.src ? a.src[p] : p) * a.k + k0 + kk) : 0.0f;
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
        if (p >= count) continue;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const uint32_t r = r0 + tr + 16 * i;
            if (r >= a.m) continue;
            const size_t o = size_t(p0 + p) * a.m + r;
            float y = acc[i][j];
            if (a.epi == EPI_RESID) y += a.base[o];
            else if (a.epi == EPI_RELU2) y = y > 0.0f ? y * y : 0.0f;
            if (a.Y) a.Y[o] = y;
            if (a.Yb) a.Yb[o] = f32_to_bf16(y);
        }
    }
}

__device__ __forceinline__ float block_sum(float v, float* red) {  // 256 threads; `red` of 8, free to use again after the next barrier
    v = warp_sum(v);
    if (threadIdx.x % 32 == 0) red[threadIdx.x / 32] = v;
    __syncthreads();
    float tot = 0.0f;
    for (uint32_t i = 0; i < 8; i++) tot += red[i];
    return tot;
}
// See NormArgs. A block per row, which it keeps in shared memory.
__global__ void __launch_bounds__(256) norm_rows_kernel(const NormArgs a) {
    pdl_start();
    extern __shared__ float row[];
    __shared__ float red[8];
    const uint32_t r = blockIdx.x, tid = threadIdx.x;
    const size_t from = size_t(a.rows ? a.rows[r] : r) * a.k;
    float ss = 0.0f;
    for (uint32_t i = tid; i < a.k; i += 256) {
        float x = a.in[from + i];
        if (a.add) {
            x += a.add[from + i];
            a.sum[from + i] = x;
        }
        row[i] = x;
        ss += x * x;
    }
    const float inv = a.scale / sqrtf(block_sum(ss, red) / float(a.k) + a.eps);
    for (uint32_t i = tid; i < a.k; i += 256) {
        const float v = row[i] * inv * weight_of(a.norm, i);
        if (a.out_f32) a.out_f32[size_t(r) * a.k + i] = v;
        if (a.out_bf16) a.out_bf16[size_t(r) * a.k + i] = f32_to_bf16(v);
    }
}

// See MergeArgs. A block per row.
__global__ void __launch_bounds__(256) merge_rows_kernel(const MergeArgs a) {
    pdl_start();
    extern __shared__ float row[];
    __shared__ float red[3][8];
    const uint32_t tid = threadIdx.x;
    const size_t from = size_t(blockIdx.x) * a.d;
    float sa = 0.0f, sb = 0.0f;
    for (uint32_t i = tid; i < a.d; i += 256) {
        const float p = a.a[from + i], q = a.b[from + i];
        sa += p * p;
        sb += q * q;
    }
    const float ia = 0.5f / sqrtf(block_sum(sa, red[0]) / float(a.d) + a.eps), ib = 0.5f / sqrtf(block_sum(sb, red[1]) / float(a.d) + a.eps);
    float ss = 0.0f;
    for (uint32_t i = tid; i < a.d; i += 256) {
        const float y = a.x[from + i] + (a.a[from + i] * ia * weight_of(a.norm_a, i) + a.b[from + i] * ib * weight_of(a.norm_b, i));
        a.out[from + i] = y;
        row[i] = y;
        ss += y * y;
    }
    if (!a.norm.w) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, red[2]) / float(a.d) + a.eps);
    for (uint32_t i = tid; i < a.d; i += 256) {
        const float v = row[i] * inv * weight_of(a.norm, i);
        if (a.next) a.next[from + i] = v;
        if (a.next_b) a.next_b[from + i] = f32_to_bf16(v);
    }
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
    configured.once([] { VLT_CUDA(cudaFuncSetAttribute(linear::norm_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); });
    if (a.n) launch_pdl(linear::norm_rows_kernel, a.n, 256, size_t(a.k) * 4, s, a);
}
void launch_merge_rows(const MergeArgs& a, cudaStream_t s) {
    static PerDevice configured;
    configured.once([] { VLT_CUDA(cudaFuncSetAttribute(linear::merge_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); });
    if (a.n) launch_pdl(linear::merge_rows_kernel, a.n, 256, size_t(a.d) * 4, s, a);
}
void launch_concat_rows(const float* a, const float* b, uint32_t n, uint32_t d, float* out_f32, uint16_t* out_bf16, cudaStream_t s) {
    if (n) launch_pdl(linear::concat_rows_kernel, n, 256, 0, s, a, b, d, out_f32, out_bf16);
}

}  // namespace vlt
