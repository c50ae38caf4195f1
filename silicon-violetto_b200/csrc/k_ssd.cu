// Recurrences with a number per head and token as their decay, over a prompt's portion on the tensor cores: S_t = d_t S_(t-1) + e_t k_t v_t^T
// (the state space's; with e = 1 and a fixed d, linear attention's), 64 tokens at a time. With c_t the sum of the logarithms of d up to t within a chunk,
//
//   y_t = sum_(s <= t) (q_t . k_s) 2^(c_t - c_s) e_s v_s + 2^(c_t) q_t S,      S <- 2^(c_end) S + sum_s k_s (2^(c_end - c_s) e_s v_s)^T.
//
// A block has 32 (or 16, where there are few blocks) value channels of one head of one run and goes through the run's chunks in order: four warps, q, k and v rows in
// bf16 (a convolution's outputs), the state in the fp32 accumulators of the last product. What is computed in 32-bit and enters a
// product -- the weights of the first sum, the state as it is read, the scaled values -- does so as two bf16 parts, whose sum
// has 16 bits. No exponent is positive: every term weighs at most its step size.
#include <algorithm>

#include "kernels.h"
#include "mma.cuh"

namespace vlt {

namespace ssd {

constexpr uint32_t T = 64, THREADS = 128;  // tokens of a chunk

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
// v0 and v1 as bf16 pairs: the rounded values and what the rounding left.
__device__ __forceinline__ void split(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(v0, v1);
    lo = pack_bf16(v0 - bf16lo(hi), v1 - bf16hi(hi));
}

// PS: value channels of a block.
template <uint32_t N, uint32_t PS>
struct Shared {
    static constexpr uint32_t NP = N + 8, PP = PS + 8;  // pitches that keep ldmatrix free of conflicts
    uint16_t q[2][T * NP], k[2][T * NP], v[2][T * PP];
    uint16_t vh[T * PP], vl[T * PP], sh[N * PP], sl[N * PP];  // the scaled values and the state in two parts
    float cum[T], step[T], weight[T];
};

// grid (heads x spans of PS value channels, runs).
template <uint32_t N, uint32_t PS>
__global__ void __launch_bounds__(THREADS) ssd_kernel(const ScanArgs a) {
    pdl_start();
    extern __shared__ __align__(16) uint8_t raw[];
    using Sh = Shared<N, PS>;
    Sh& sm = *reinterpret_cast<Sh*>(raw);
    constexpr uint32_t NP = Sh::NP, PP = Sh::PP, MT = N / 64, KS = N / 16, PT = PS / 8;
    const RunIn run = a.runs[blockIdx.y];
    if (run.count < a.tensor_min) return;
    const RecurrentCache& c = a.c;
    const uint32_t spans = c.P / PS, head = blockIdx.x / spans, p0 = blockIdx.x % spans * PS, tid = threadIdx.x, warp = tid / 32, lane = tid % 32, g = lane >> 2, tq = lane & 3;
    const uint32_t t0 = run.first, count = run.count, chunks = (count + T - 1) / T;
    const uint16_t *Q = a.q_b + size_t(t0) * a.ldq + head / c.per * N, *K = a.k_b + size_t(t0) * a.ldk + head / c.per * N, *V = a.v_b + size_t(t0) * a.ldv + head * c.P + p0;
    if (count % T) {  // (rows past the last token: finite, and weighed by zero)
        for (uint32_t i = tid; i < sizeof(Sh) / 16; i += THREADS) reinterpret_cast<uint4*>(raw)[i] = make_uint4(0, 0, 0, 0);
        __syncthreads();
    }
    auto fetch = [&](uint32_t ch) {
        const uint32_t b = ch & 1, n = min(T, count - ch * T), i0 = ch * T;
        for (uint32_t i = tid; i < n * (N / 8); i += THREADS) {
            const uint32_t r = i / (N / 8), x = i % (N / 8) * 8;
            cp_async16(smem_u32(sm.q[b] + r * NP + x), Q + size_t(i0 + r) * a.ldq + x);
            cp_async16(smem_u32(sm.k[b] + r * NP + x), K + size_t(i0 + r) * a.ldk + x);
        }
        for (uint32_t i = tid; i < n * (PS / 8); i += THREADS) {
            const uint32_t r = i / (PS / 8), x = i % (PS / 8) * 8;
            cp_async16(smem_u32(sm.v[b] + r * PP + x), V + size_t(i0 + r) * a.ldv + x);
        }
    };
    fetch(0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const bool fresh = a.meta[2 * t0 + 1] == 0;
    const float rate = c.fixed ? log2f(c.fixed[head]) : -expf(bf16_to_f32(a.a_log[head])) * LOG2E, skip = a.skip ? bf16_to_f32(a.skip[head]) : 0.0f;
    // The state: rows (key channels) n0 + 16 m + g and + 8, columns (value channels) 8 j + 2 tq and + 1.
    const uint32_t n0 = warp * 16 * MT;
    float* home = c.state + ((size_t(run.slot) * c.heads + head) * c.P + p0) * c.Np;
    float S[MT][PT][4];
#pragma unroll
    for (uint32_t m = 0; m < MT; m++)
#pragma unroll
        for (uint32_t j = 0; j < PT; j++)
#pragma unroll
            for (uint32_t e = 0; e < 4; e++) S[m][j][e] = fresh ? 0.0f : home[(8 * j + 2 * tq + (e & 1)) * c.Np + n0 + 16 * m + g + 8 * (e >> 1)];
    auto publish = [&] {  // the state as the next chunk reads it
#pragma unroll
        for (uint32_t m = 0; m < MT; m++)
#pragma unroll
            for (uint32_t j = 0; j < PT; j++)
#pragma unroll
                for (uint32_t r = 0; r < 2; r++) {
                    uint32_t hi, lo;
                    split(S[m][j][2 * r], S[m][j][2 * r + 1], hi, lo);
                    const uint32_t at = (n0 + 16 * m + g + 8 * r) * PP + 8 * j + 2 * tq;
                    *reinterpret_cast<uint32_t*>(sm.sh + at) = hi;
                    *reinterpret_cast<uint32_t*>(sm.sl + at) = lo;
                }
    };
    publish();
    // ldmatrix roles: rows of an A operand or of a transposed B operand; of a B operand that lies with its k contiguous; of a
    // transposed A operand.
    const uint32_t a_row = lane % 16, a_col = lane / 16 * 8, b_row = lane % 8 + lane / 16 * 8, b_col = (lane / 8 & 1) * 8, ta_row = lane % 8 + (lane / 16) * 8, ta_col = (lane / 8 & 1) * 8;
    const size_t ldy = size_t(c.heads) * c.P;
    float ahead[2];  // the first warp's step sizes of the chunk to come
    auto steps = [&](uint32_t ch) {
#pragma unroll
        for (uint32_t u = 0; u < 2; u++) {
            const uint32_t i = ch * T + 2 * lane + u;
            ahead[u] = i >= count ? 0.0f : c.fixed ? 1.0f : a.decay[(size_t(t0 + i) * c.heads + head) * 2];
        }
    };
    if (warp == 0) steps(0);
    for (uint32_t ch = 0; ch < chunks; ch++) {
        const uint32_t b = ch & 1, i0 = ch * T, n = min(T, count - i0);
        if (warp == 0) {  // the step sizes, and c as a running sum over the lanes' pairs of tokens
            const float e[2] = {ahead[0], ahead[1]}, l[2] = {rate * e[0], rate * e[1]};
            float sum = l[0] + l[1];
#pragma unroll
            for (uint32_t o = 1; o < 32; o *= 2) {
                const float up = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += up;
            }
            const float end = __shfl_sync(0xffffffffu, sum, 31), first = sum - l[1];
            sm.cum[2 * lane] = first;
            sm.cum[2 * lane + 1] = sum;
            sm.step[2 * lane] = e[0];
            sm.step[2 * lane + 1] = e[1];
            sm.weight[2 * lane] = exp2f(end - first) * e[0];
            sm.weight[2 * lane + 1] = exp2f(end - sum) * e[1];
            if (ch + 1 < chunks) steps(ch + 1);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the chunk's rows and step sizes, and the state's parts, are there; the other buffer is free
        if (ch + 1 < chunks) fetch(ch + 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        for (uint32_t i = tid; i < T * PS / 2; i += THREADS) {
            const uint32_t s = i / (PS / 2), at = s * PP + i % (PS / 2) * 2, pair = *reinterpret_cast<const uint32_t*>(sm.v[b] + at);
            const float w = sm.weight[s];
            uint32_t hi, lo;
            split(bf16lo(pair) * w, bf16hi(pair) * w, hi, lo);
            *reinterpret_cast<uint32_t*>(sm.vh + at) = hi;
            *reinterpret_cast<uint32_t*>(sm.vl + at) = lo;
        }
        // This warp's 16 tokens: q . k against the tokens up to them, and q . S.
        const uint32_t row0 = warp * 16;
        float G[T / 8][4], R[PT][4], Y[PT][4];
#pragma unroll
        for (uint32_t j = 0; j < T / 8; j++) G[j][0] = G[j][1] = G[j][2] = G[j][3] = 0.0f;
#pragma unroll
        for (uint32_t j = 0; j < PT; j++)
#pragma unroll
            for (uint32_t e = 0; e < 4; e++) R[j][e] = Y[j][e] = 0.0f;
#pragma unroll
        for (uint32_t ks = 0; ks < KS; ks++) {
            uint32_t qa[4];
            ldmatrix_x4(qa, smem_u32(sm.q[b] + (row0 + a_row) * NP + 16 * ks + a_col));
#pragma unroll
            for (uint32_t j = 0; j < T / 16; j++) {
                if (j > warp) break;
                uint32_t kb[4];
                ldmatrix_x4(kb, smem_u32(sm.k[b] + (16 * j + b_row) * NP + 16 * ks + b_col));
                mma16816(G[2 * j], qa, kb[0], kb[1]);
                mma16816(G[2 * j + 1], qa, kb[2], kb[3]);
            }
#pragma unroll
            for (uint32_t j = 0; j < PT / 2; j++) {
                uint32_t hb[4], lb[4];
                ldmatrix_x4_trans(hb, smem_u32(sm.sh + (16 * ks + a_row) * PP + 16 * j + a_col));
                ldmatrix_x4_trans(lb, smem_u32(sm.sl + (16 * ks + a_row) * PP + 16 * j + a_col));
                mma16816(R[2 * j], qa, hb[0], hb[1]);
                mma16816(R[2 * j + 1], qa, hb[2], hb[3]);
                mma16816(R[2 * j], qa, lb[0], lb[1]);
                mma16816(R[2 * j + 1], qa, lb[2], lb[3]);
            }
        }
        const float c0 = sm.cum[row0 + g], c1 = sm.cum[row0 + g + 8];
#pragma unroll
        for (uint32_t kk = 0; kk < T / 16; kk++) {
            if (kk > warp) break;
            uint32_t mh[4], ml[4];
#pragma unroll
            for (uint32_t h = 0; h < 2; h++) {
                const uint32_t s = 16 * kk + 8 * h + 2 * tq;
                const float2 cs = *reinterpret_cast<const float2*>(sm.cum + s), es = *reinterpret_cast<const float2*>(sm.step + s);
                float* v = G[2 * kk + h];
                v[0] = s <= row0 + g ? v[0] * fast_exp2(c0 - cs.x) * es.x : 0.0f;
                v[1] = s + 1 <= row0 + g ? v[1] * fast_exp2(c0 - cs.y) * es.y : 0.0f;
                v[2] = s <= row0 + g + 8 ? v[2] * fast_exp2(c1 - cs.x) * es.x : 0.0f;
                v[3] = s + 1 <= row0 + g + 8 ? v[3] * fast_exp2(c1 - cs.y) * es.y : 0.0f;
                split(v[0], v[1], mh[2 * h], ml[2 * h]);
                split(v[2], v[3], mh[2 * h + 1], ml[2 * h + 1]);
            }
#pragma unroll
            for (uint32_t j = 0; j < PT / 2; j++) {
                uint32_t vb[4];
                ldmatrix_x4_trans(vb, smem_u32(sm.v[b] + (16 * kk + a_row) * PP + 16 * j + a_col));
                mma16816(Y[2 * j], mh, vb[0], vb[1]);
                mma16816(Y[2 * j + 1], mh, vb[2], vb[3]);
                mma16816(Y[2 * j], ml, vb[0], vb[1]);
                mma16816(Y[2 * j + 1], ml, vb[2], vb[3]);
            }
        }
        const float d0 = fast_exp2(c0), d1 = fast_exp2(c1);
#pragma unroll
        for (uint32_t j = 0; j < PT; j++)
#pragma unroll
            for (uint32_t r = 0; r < 2; r++) {
                const uint32_t t = row0 + g + 8 * r;
                if (t >= n) continue;
                const uint32_t x = *reinterpret_cast<const uint32_t*>(sm.v[b] + t * PP + 8 * j + 2 * tq);
                const float d = r ? d1 : d0;
                *reinterpret_cast<float2*>(a.y + size_t(t0 + i0 + t) * ldy + head * c.P + p0 + 8 * j + 2 * tq) =
                    make_float2(Y[j][2 * r] + d * R[j][2 * r] + skip * bf16lo(x), Y[j][2 * r + 1] + d * R[j][2 * r + 1] + skip * bf16hi(x));
            }
        __syncthreads();  // the scaled values are there; everybody has read the state
        const float keep = exp2f(sm.cum[T - 1]);
#pragma unroll
        for (uint32_t m = 0; m < MT; m++)
#pragma unroll
            for (uint32_t j = 0; j < PT; j++)
#pragma unroll
                for (uint32_t e = 0; e < 4; e++) S[m][j][e] *= keep;
#pragma unroll
        for (uint32_t kk = 0; kk < T / 16; kk++) {
            uint32_t hb[PT / 2][4], lb[PT / 2][4];
#pragma unroll
            for (uint32_t j = 0; j < PT / 2; j++) {
                ldmatrix_x4_trans(hb[j], smem_u32(sm.vh + (16 * kk + a_row) * PP + 16 * j + a_col));
                ldmatrix_x4_trans(lb[j], smem_u32(sm.vl + (16 * kk + a_row) * PP + 16 * j + a_col));
            }
#pragma unroll
            for (uint32_t m = 0; m < MT; m++) {
                uint32_t ka[4];
                ldmatrix_x4_trans(ka, smem_u32(sm.k[b] + (16 * kk + ta_row) * NP + n0 + 16 * m + ta_col));
#pragma unroll
                for (uint32_t j = 0; j < PT / 2; j++) {
                    mma16816(S[m][2 * j], ka, hb[j][0], hb[j][1]);
                    mma16816(S[m][2 * j + 1], ka, hb[j][2], hb[j][3]);
                    mma16816(S[m][2 * j], ka, lb[j][0], lb[j][1]);
                    mma16816(S[m][2 * j + 1], ka, lb[j][2], lb[j][3]);
                }
            }
        }
        publish();
        __syncthreads();  // nobody reads this chunk's sums and buffer any more
    }
    if (a.gen[run.slot].done) return;
#pragma unroll
    for (uint32_t m = 0; m < MT; m++)
#pragma unroll
        for (uint32_t j = 0; j < PT; j++)
#pragma unroll
            for (uint32_t e = 0; e < 4; e++) home[(8 * j + 2 * tq + (e & 1)) * c.Np + n0 + 16 * m + g + 8 * (e >> 1)] = S[m][j][e];
}

template <uint32_t N, uint32_t PS>
void launch(const ScanArgs& a, cudaStream_t s) {
    using Sh = Shared<N, PS>;
    static PerDevice configured;
    configured.once([] { VLT_CUDA(cudaFuncSetAttribute(ssd_kernel<N, PS>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(sizeof(Sh)))); });
    static_assert(sizeof(Sh) % 16 == 0, "cleared by 16 bytes");
    launch_pdl(ssd_kernel<N, PS>, dim3(a.c.heads * (a.c.P / PS), a.n_runs), THREADS, sizeof(Sh), s, a);
}

}  // namespace ssd

bool ssd_fits(uint32_t N, uint32_t P) { return (N == 64 || N == 128) && P % 32 == 0; }
void launch_ssd(const ScanArgs& a, cudaStream_t s) {
    const bool few = a.c.heads * (a.c.P / 32) * a.n_runs <= 74;  // (half the SMs)
    if (a.c.N == 64) few ? ssd::launch<64, 16>(a, s) : ssd::launch<64, 32>(a, s);
    else few ? ssd::launch<128, 16>(a, s) : ssd::launch<128, 32>(a, s);
}

}  // namespace vlt
