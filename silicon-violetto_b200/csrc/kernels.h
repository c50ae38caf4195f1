// Launchers of the CUDA kernels (all asynchronous on the given stream).
#pragma once
#include <cuda_runtime.h>

#include "common.h"
#include "device.cuh"
#include "layered.h"
#include "weights.h"

namespace vlt {

// Epilogues of a matmul, engine/src/engine/kernels.rs:3-9 and kernels.metal:154-209.
enum : uint32_t { EPI_NORM = 1, EPI_RESID = 2, EPI_SWIGLU = 3, EPI_HEAD = 4, EPI_RAW = 5, EPI_QKV = 6, EPI_HEAD_CAP = 7, EPI_RELU2 = 8,  // 7: 23 sigmoid((acc + 5) / 7.5), kernels.metal:196-199; 8: max(acc, 0)^2
                EPI_SILU = 9,        // silu(acc) for rows below vocab_real, the others as they are
                EPI_GLU = 10,        // rows in pairs (g, u): silu(g) u, half as many outputs; EPI_SWIGLU's without a norm
                EPI_SIDE = 12,       // gelu(acc) times an entry of the token's row in a table (MatArgs::side)
                EPI_GLU_CLAMP = 11   // EPI_GLU's pairs: g sigmoid(1.702 g) (u + 1), g cut off above a limit, u outside of +- the limit
};
// Rows 2 i and 2 i + 1 make output i.
__host__ __device__ constexpr bool epi_pairs(uint32_t epi) { return epi == EPI_SWIGLU || epi == EPI_GLU || epi == EPI_GLU_CLAMP; }

// What the tensor-core GEMM's EPI_QKV epilogue needs to finish the qkv projection the way `qkv_post` does
// (kernels.metal:749-801): RoPE on q and k, q scaled and rounded to bf16 for the attention, k and v rounded
// into the paged cache at each token's position.
struct QkvEpilogue {
    const uint32_t* meta;        // (slot, position) per token
    const uint32_t* tin;         // (slot, row in its run) per token
    const uint32_t* cpos;        // optional: cache position per token (NO_TOK: no write); NULL: its run's first position + its row
    const float* rope;           // [position][head_dim / 2] (cos, sin)
    const uint32_t* page_table;
    KvArgs kv;
    uint32_t layer, n_heads;
    float scale_log2;
    uint16_t* q_b;               // [token][head][head_dim] bf16
    uint16_t* k_cache;
    uint16_t* v_cache;
};

__device__ __forceinline__ float weight_of(const RowNorm& n, uint32_t i) { return (n.around_zero ? 1.0f : 0.0f) + bf16_to_f32(n.w[i]); }

__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }
// FAST: by the hardware's exponential and quotient, whose errors are far below a rounding to bf16.
template <bool FAST = false>
__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * (FAST ? __fdividef(1.0f, 1.0f + __expf(-1.702f * g)) : sigmoid_of(1.702f * g)) * (u + 1.0f);
}
template <uint32_t V>
__device__ __forceinline__ void weights_of(float (&x)[V], const RowNorm& n, uint32_t i) {
    load_bf16<V>(x, n.w + i);
    if (n.around_zero)
#pragma unroll
        for (uint32_t j = 0; j < V; j++) x[j] += 1.0f;
}

// A row's gate (launch_side_gate, EPI_SIDE): entry i < dim is gelu(z_i) times entry first + i of the token's row in a bf16 table; zeros
// from there to `wide`.
struct SideTable {
    const uint16_t* table;   // [vocab][ld]
    const uint32_t* tokens;
    uint32_t ld, first, dim, wide;
};
__device__ __forceinline__ float side_of(const SideTable& s, uint32_t t, uint32_t i, float z) {
    if (i >= s.dim) return 0.0f;
    const float g = z * sigmoid_of(1.5957691216057308f * (z + 0.044715f * z * z * z));  // (1 + tanh u) / 2 is sigmoid(2 u), u = sqrt(2 / pi) (z + ...)
    return g * bf16_to_f32(s.table[size_t(s.tokens[t]) * s.ld + s.first + i]);
}

// Y[t][row] = epilogue(W[row] . bf16(X[t])). X fp32 [n][k]; Y fp32 (SWIGLU: [n][m/2]).
struct MatArgs {
    const uint8_t* W;
    const uint16_t* scales;  // int8: bf16 [m][k / group]
    const float* X;          // [n][k]
    const uint16_t* Xb;      // bf16 copy of X [n_pad][k]: the tensor-core GEMM's input; the streamed matmul takes it instead of X if given (needs no 1/rms then)
    float* Y;
    const float* base;  // EPI_RESID: y = base + acc (may alias Y)
    float* inv_out;     // EPI_NORM / EPI_SWIGLU / EPI_HEAD: 1 / rms(X[t]) is computed here ...
    const float* inv_in;  // ... or, if not null, read from here (tensor-core GEMM)
    uint16_t* Yb;       // optional bf16 copy of Y (feeds the next tensor-core GEMM)
    uint32_t n, k, m, group;  // group: 0 for bf16 weights
    uint32_t epi, vocab_real;  // vocab_real: a head's rows from there on are padding; EPI_SILU: rows from there on stay as they are
    float eps;
    const uint16_t* bias;  // optional, bf16 [m] (bf16 weights): onto the sums in front of everything else
    float limit;           // EPI_GLU_CLAMP
    // kernels.metal:164-165,188-193: the matrix scale (qkv_scale, o_scale) and EPI_RESID's y = ra base + rb (scale acc). 1 for a
    // plain decoder.
    float scale = 1.0f, ra = 1.0f, rb = 1.0f;
    bool int8;
    QkvEpilogue q;   // EPI_QKV only
    SideTable side;  // EPI_SIDE only, whose outputs are `side.wide` to a token
    uint32_t t0;    // EPI_QKV in the streamed matmul: the step's token that this launch's token 0 is
    uint32_t* err_flag;  // streamed matmul: device word set if a bounded wait ran out (optional)
    // The residual stream's sum of squares per token, kept by the tensor-core GEMMs themselves so that no row pass is
    // needed between them: an EPI_RESID GEMM with ssq_out writes, per 128-row tile of its output, sum(y^2) over the
    // tile's rows ([tile][ssq_stride]); a GEMM with ssq_in (and no inv_in) takes 1/rms = rsqrt(sum over ssq_tiles / k + eps).
    float* ssq_out;
    const float* ssq_in;
    uint32_t ssq_tiles, ssq_stride;
};

void launch_embed(const uint16_t* table, uint32_t* tokens, float* out, const uint32_t* tin, uint32_t* meta, const uint32_t* lens,
                  const uint32_t* feed, const uint32_t* tree, uint32_t* vis, uint32_t n, uint32_t d, uint32_t vocab, cudaStream_t s,
                  const uint16_t* positions = nullptr, uint32_t n_positions = 0,  // positions: [n_positions][d], a vector per position to add
                  uint16_t* out_b = nullptr,                                      // out in bf16
                  float scale = 1.0f);                                            // of the table's rows
void launch_qkv_post(const float* qkv, const uint32_t* meta, const uint32_t* tin, const float* rope, uint16_t* k_cache, uint16_t* v_cache,
                     const uint32_t* page_table, KvArgs kv, uint32_t layer, uint32_t n, uint32_t n_heads, float scale_log2, uint16_t* q_b, const uint32_t* cpos, cudaStream_t s);
// q | k | v rows as the attention sees them before rounding (RoPE on q and k, kernels.metal:727-736), for step_capture.
void launch_qkv_capture(const float* qkv, const uint32_t* meta, const float* rope, uint32_t n, uint32_t n_heads, KvArgs kv, float* out, cudaStream_t s);
void launch_attn_plain(const float* qkv, const uint32_t* meta, const uint32_t* tiles, const uint32_t* vis, const float* rope, const uint16_t* k_cache,
                       const uint16_t* v_cache, const uint32_t* page_table, KvArgs kv, uint32_t layer, uint32_t n_tiles, uint32_t n_heads,
                       float scale_log2, float* out, cudaStream_t s);
// Tensor-core decode attention over paged KV, split over keys; then the merge of the splits.
// The TMA descriptors of the K and V pools (opaque 128-byte CUtensorMap objects).
struct alignas(64) AttnMaps {
    alignas(64) uint8_t k[128];
    alignas(64) uint8_t v[128];
};
void attn_maps_init(AttnMaps* m, const uint16_t* k_cache, const uint16_t* v_cache, uint64_t total_rows);
void make_tensor_map_2d(void* out_map, const void* base, uint64_t inner, uint64_t rows, uint32_t box_inner, uint32_t box_rows, uint32_t elem_bytes,
                        bool swizzle128, bool swizzle64 = false);
struct AttnArgs {
    const AttnMaps* maps;  // host pointer
    uint32_t* err_flag;    // device word set if a bounded wait ran out
    const uint16_t* q_b;  // [token][head][64] bf16: q after RoPE, scale * log2(e) folded in (qkv_post writes it)
    const uint32_t* meta;
    const uint32_t* tiles;
    const uint32_t* vis;
    const uint16_t* k_cache;
    const uint16_t* v_cache;
    const uint32_t* page_table;
    KvArgs kv;
    uint32_t layer, n_tiles, n_heads;
    float scale_log2;
    uint32_t keys_per_split, max_splits;
    uint32_t max_rows;  // the longest tile's rows in this launch (0: unknown, VERIFY_T)
    uint32_t window;    // 0: every key; else a tile sees its last `window` keys, extended down to a page boundary
    float* part;  // [token][head][max_splits][PART]
    float* out;   // [n][n_heads * hd]
    uint16_t* out_b;  // optional bf16 copy
    uint32_t n;
};
constexpr uint32_t ATTN_PART = 68;  // floats per partial: m, l, 2 pad, o[64]
void launch_attn_mma(const AttnArgs& a, cudaStream_t s);
void launch_attn_combine(const AttnArgs& a, cudaStream_t s);

// Chunk (prefill) attention, k_prefill.cu: blocks of 64 rows of one run x one query head over all the keys the rows see,
// no key split; writes the normalised rows (fp32 and, optionally, bf16).
struct ChunkAttnArgs {
    const AttnMaps* maps;  // host pointer
    uint32_t* err_flag;
    const uint16_t* q_b;  // [token][head][64] bf16, rotated and scaled
    const uint32_t* meta;
    const uint32_t* tin;
    const uint32_t* ctiles;  // (first token, rows <= 64) per chunk tile, never across runs
    const uint32_t* vis;
    const uint32_t* page_table;
    KvArgs kv;
    uint32_t layer, n_ctiles, n_heads;
    float* out;
    uint16_t* out_b;
};
void launch_attn_chunk(const ChunkAttnArgs& a, cudaStream_t s);

// The chain drafter's own kernels (k_draft.cu): inputs of the catch-up pass and of a draft pass, the
// carried tap, and the argmax pick into feed / tree.
void launch_draft_catchup_in(const uint32_t* tokens, const uint32_t* tin, const uint32_t* meta, const uint32_t* on_path, const float* taps, const float* carry,
                             const uint16_t* embed, uint32_t n, uint32_t d, float* x, uint16_t* xb, uint32_t* cpos, cudaStream_t s);
void launch_draft_pass_in(const RunIn* runs, const uint32_t* lens, const uint32_t* feed, const uint32_t* path, const uint32_t* path_len, const uint32_t* on_path,
                          const uint32_t* emitted, const float* taps, const float* dfeat, const uint16_t* embed, uint32_t n_runs, uint32_t d, uint32_t vocab,
                          uint32_t i, uint32_t max_seq_len, float* x, uint16_t* xb, uint32_t* dmeta, uint32_t* dtin, uint32_t* dvis, uint32_t* dcpos, uint32_t* live,
                          cudaStream_t s);
void launch_draft_carry(const RunIn* runs, const uint32_t* path, const uint32_t* path_len, const uint32_t* on_path, const float* taps, uint32_t n_runs,
                        uint32_t d, float* carry, cudaStream_t s);
void launch_draft_pick(const float* logits, uint32_t v, const uint32_t* vocab_ids, const RunIn* runs, const uint32_t* live, uint32_t n_runs, uint32_t i,
                       uint32_t* feed, uint32_t* tree, cudaStream_t s);

// The reference drafter's candidate kernels (kernels.metal:1846-1934): the best `ncand` (<= 4) entries of each row of draft
// logits with their probabilities, then a draft tree per block of rows grown by path probability.
void launch_draft_top(const float* logits, uint32_t n_rows, uint32_t nv, const uint32_t* vocab_ids, const uint32_t* tin, float inv_t, uint32_t ncand, uint32_t* cand,
                      float* cand_q, cudaStream_t s);  // tin (optional): (slot, row) per row; rows numbered 0 are skipped
void launch_draft_tree(const uint32_t* blocks, const uint32_t* slots, uint32_t n_blocks, const uint32_t* cand, const float* cand_q, uint32_t ncand, uint32_t* feed,
                       uint32_t* tree, cudaStream_t s);

// The reference's block drafter (k_block.cu): its shapes and state sizes, and its own kernels.
struct BlockDrafterDims {
    uint32_t hidden, n_q, n_kv, n_layers;  // heads are 128 wide
    uint32_t ring, max_seqs, window, ctx_ring_len;
    float eps, scale;
};
constexpr uint32_t BLOCK_CONV_KC = 192;  // a convolution's correction rows (2 * hidden / 16, padded; tools/spec/export.py:14)
void launch_block_context(const float* kvp, const float* ctx, const float* ctx_inv, const uint32_t* meta, const uint32_t* on_path, const float* rope,
                          const BlockDrafterDims& b, uint32_t n, uint16_t* k_ring, uint16_t* v_ring, float* ctx_ring, cudaStream_t s);
void launch_block_embed(const uint16_t* table, const uint32_t* tin, const uint32_t* lens, const uint32_t* feed, const float* mask_emb, const float* ctx_ring,
                        const BlockDrafterDims& b, uint32_t vocab, uint32_t rows, float* x, float* last, uint32_t* meta, cudaStream_t s);
void launch_block_conv(const float* x, const float* corr, uint32_t corr_stride, const float* base, const uint32_t* tin, const float* resid, uint32_t hidden,
                       uint32_t rows, float* out, cudaStream_t s);
void launch_block_qkv_post(float* qkv, const uint32_t* meta, const float* rope, const BlockDrafterDims& b, uint32_t layer, uint32_t rows, uint16_t* k_ring,
                           uint16_t* v_ring, cudaStream_t s);
void launch_block_attn(const float* qkv, const uint32_t* meta, const uint32_t* tin, const uint32_t* rows_of, const uint16_t* k_ring, const uint16_t* v_ring,
                       const BlockDrafterDims& b, uint32_t layer, uint32_t rows, float* out, cudaStream_t s);

// The reference's own architecture (k_limite.cu). A layer's cache: a ring per (local layer, slot) or the paged pool of the
// global layers (kernels.metal:692-715); heads are 128 wide.
struct LimiteKv {
    uint32_t is_global, layer;  // layer: its index among the local or among the global layers
    uint32_t n_kv, ring, max_seqs;
    uint32_t n_pages, max_pages, page_shift;
    const uint32_t* page_table;
};
void launch_limite_mudd(const float* cur, const float* tap0, const float* tap1, const float* dense1, const float* mix, uint32_t hidden, float eps, uint32_t n,
                        float* out_attn, float* out_base, cudaStream_t s);
void launch_limite_qkv_post(float* qkv, const float* x, const float* inv_rms, const uint32_t* meta, const uint32_t* tin, const uint32_t* tokens, const uint16_t* ve_table,
                            const float* ve_gate, const float* attn_gate, const float* rope, const LimiteKv& kv, uint32_t hidden, uint32_t n_q, float eps, uint32_t vocab,
                            uint32_t n, uint16_t* k_cache, uint16_t* v_cache, float* vdir, float* gates, const float* ssq, uint32_t ssq_tiles, uint32_t ssq_stride,
                            cudaStream_t s);
constexpr uint32_t LIMITE_MAX_SPLITS = 128, LIMITE_PART = 132;  // key splits a row's attention may take; floats per partial
void launch_limite_attn_mma(const float* qkv, const uint32_t* meta, const uint32_t* tin, const uint32_t* vis, const uint16_t* k_cache, const uint16_t* v_cache,
                            const LimiteKv& kv, uint32_t n_q, uint32_t window, float scale, uint32_t n, uint32_t keys_per_split, uint32_t splits, float* part,
                            cudaStream_t s);
void launch_limite_attn_cluster(const float* qkv, const uint32_t* meta, const uint32_t* tin, const uint32_t* vis, const uint16_t* k_cache, const uint16_t* v_cache,
                                const LimiteKv& kv, uint32_t n_q, uint32_t window, float scale, const float* vdir, const float* gates, const float* xsa, uint32_t n,
                                uint32_t keys_per_split, uint32_t splits, float* out, uint16_t* out_b, cudaStream_t s);
void launch_limite_attn_rows(const float* qkv, const uint32_t* meta, const uint32_t* tin, const uint32_t* vis, const uint32_t* tiles, const uint16_t* k_cache,
                             const uint16_t* v_cache, const LimiteKv& kv, uint32_t n_q, uint32_t window, float scale, uint32_t n_tiles, uint32_t keys_per_split,
                             uint32_t splits, float* part, cudaStream_t s);
void launch_limite_attn(const float* qkv, const uint32_t* meta, const uint32_t* tin, const uint32_t* vis, const uint32_t* tiles, uint32_t n_tiles, const uint16_t* k_cache, const uint16_t* v_cache,
                        const LimiteKv& kv, uint32_t n_q, uint32_t window, float scale, const float* vdir, const float* gates, const float* xsa, uint32_t n,
                        uint32_t max_keys, float* part, float* out, uint16_t* out_b, uint32_t keys_per_block, cudaStream_t s);  // out_b: optional bf16 copy (heads per kv head 1, 2 or 5)
void launch_limite_compact(const RunIn* runs, const uint32_t* path, const uint32_t* path_len, const uint32_t* lens, uint16_t* k_local, uint16_t* v_local,
                           uint16_t* k_global, uint16_t* v_global, const LimiteKv& local, const LimiteKv& global, uint32_t n_local, uint32_t n_global, uint32_t n_runs,
                           cudaStream_t s);

// The tcgen05 GEMM for 16..256 tokens: needs Xb (bf16 X, rows padded to 16), inv_in for the
// normed epilogues, m a multiple of 128, one int8 scale per row.
bool gemm_supported(const MatArgs& a);
void launch_gemm(const MatArgs& a, uint32_t sm_count, uint32_t* err_flag, cudaStream_t s, bool allow_paired = true);
void launch_matmul_stream(const MatArgs& a, uint32_t sm_count, cudaStream_t s);  // n <= 8, tensor cores fed from registers
bool matmul_stream_fits(const MatArgs& a);                                      // else launch_matmul_stream falls back to the scalar kernel
void launch_matmul_rows(const MatArgs& a, cudaStream_t s);                      // any n, scalar (cross-check, odd scale groups)
// out[r] = in[rows ? rows[r] : r] as fp32 (and bf16); inv[r] = 1 / rms (kernels.metal:117-148).
void launch_prep_rows(const float* in, const uint32_t* rows, uint32_t n, uint32_t k, float eps, float* out_f32, uint16_t* out_bf16, float* inv,
                      bool normalize, bool round_out, cudaStream_t s);

// Linear layers of any shape on the CUDA cores (k_linear.cu): bf16 weights, activations in fp32 or bf16, fp32 products and
// sums. With `tiles`, a grouped layer: tile j multiplies rows p0 .. p0 + count - 1 by group g's matrix W + g m k.
struct LinearArgs {
    const uint16_t* W;
    const void* X;           // [rows][k] fp32 or bf16
    const uint32_t* src;     // optional: the row of X that row p multiplies
    const float* base;       // EPI_RESID
    float* Y;                // optional, as is
    uint16_t* Yb;            // its bf16 copy
    uint32_t n, m, k, epi;   // EPI_RAW, EPI_RESID, EPI_RELU2, EPI_SILU, EPI_GLU or EPI_GLU_CLAMP
    uint32_t act_rows;       // EPI_SILU
    float limit;             // EPI_GLU_CLAMP
    const uint16_t* bias;    // optional, without tiles: [m], onto the sums
    const float* row_scale;  // optional, with tiles: what row p's products are multiplied by, before the epilogue
    // A matrix per head against that head's part of every token (by_head tokens; 0: not so): group g's rows are p = g by_head + t,
    // read at row t heads + g of X and written at row t heads + g of Y, `ldy` apart. gate (optional): [by_head][ldg], the output is
    // multiplied by the sigmoid of row t's column g m + r, or (gate_w 1) g.
    uint32_t by_head, heads, ldy, ldg, gate_w;
    const float* gate;
    const uint32_t* tiles;   // [.][3]: (group, first row, rows)
    const uint32_t* n_tiles;
    uint32_t max_tiles;      // at most so many tiles (the grid)
};
void launch_linear(const LinearArgs& a, bool x_bf16, cudaStream_t s);
bool grouped_fits(uint32_t m, uint32_t k);  // the tensor-core form (k_grouped.cu): bf16 activations, EPI_RAW, EPI_RELU2 or EPI_GLU_CLAMP
void launch_grouped(const LinearArgs& a, uint32_t n_groups, uint32_t tile, uint32_t* err_flag, cudaStream_t s);
// out[r] = x / sqrt(mean x^2 + eps) times the weight times `scale`, x being row rows[r] (or r) of `in`, plus that of `add`, the
// sum then left in `sum`. (A centered norm: of x less its mean, plus its b times `scale`.)
struct NormArgs {
    const float* in;
    const uint32_t* rows;    // optional
    const float* add;        // optional
    float* sum;              // with add
    uint32_t n, k;
    float eps;
    RowNorm norm;
    float scale;
    float* out_f32;          // optional
    uint16_t* out_bf16;      // optional
};
void launch_norm_rows(const NormArgs& a, cudaStream_t s);
// x[r] += the mean of two rows, each divided by its root mean square and times its weight; norm.w (optional): the normed rows of
// the sum as well.
struct MergeArgs {
    const float *x, *a, *b;
    RowNorm norm_a, norm_b, norm;
    float* out;              // may be x
    float* next;             // optional
    uint16_t* next_b;        // optional
    uint32_t n, d;
    float eps;
};
void launch_merge_rows(const MergeArgs& a, cudaStream_t s);
// out[r] = x[r] + y[r] / sqrt(mean y^2 + eps) times the weight, and its bf16 copy.
struct AddNormArgs {
    const float *x, *y;
    RowNorm norm;
    float* out;              // may be x
    uint16_t* out_b;         // optional
    uint32_t n, d;
    float eps;
};
void launch_add_norm(const AddNormArgs& a, cudaStream_t s);
// out[r] = the sum over j < count of share[j] X_j[r], X_j at x + j stride; norm.w (optional): its normed rows as well.
struct DepthArgs {
    const float* x;
    size_t stride;
    const uint16_t* share;
    float* out;              // none of the X_j
    RowNorm norm;
    float* next;             // optional
    uint16_t* next_b;        // optional
    uint32_t count, n, d;
    float eps;
};
void launch_depth_average(const DepthArgs& a, cudaStream_t s);
struct SideGateArgs {
    const float* x;          // [n][ldx]
    SideTable side;
    float* out_f32;          // optional, [n][wide]
    uint16_t* out_bf16;      // optional
    uint32_t n, ldx;
};
void launch_side_gate(const SideGateArgs& a, cudaStream_t s);
void launch_concat_rows(const float* a, const float* b, uint32_t n, uint32_t d, float* out_f32, uint16_t* out_bf16, cudaStream_t s);

// One layer run's pages: [page][kv head][position in page][dk or dv] for K and for V, bf16 or fp32. v == k: a value is its key's
// first dv entries, and there is no V pool.
struct PagedKv {
    void *k, *v;
    const uint32_t* page_table;
    uint32_t max_pages, page_shift, n_kv, dk, dv;
    uint32_t n_pages;  // of the pool
};
__device__ __forceinline__ size_t page_row(const PagedKv& kv, uint32_t slot, uint32_t g, uint32_t pos) {
    const uint32_t page = kv.page_table[size_t(slot) * kv.max_pages + (pos >> kv.page_shift)], psize = 1u << kv.page_shift;
    return (size_t(page) * kv.n_kv + g) * psize + (pos & (psize - 1));
}
// Entry c of a vector whose first `dims` entries turn (see Rotation); cs: the position's (cos, sin) per pair.
__device__ __forceinline__ float rotated(const float* y, uint32_t c, uint32_t dims, bool neighbours, const float2* cs) {
    const uint32_t half = dims / 2;
    if (c >= dims) return y[c];
    const float2 t = cs[neighbours ? c / 2 : c < half ? c : c - half];
    const bool first = neighbours ? c % 2 == 0 : c < half;
    const float other = y[neighbours ? c ^ 1u : first ? c + half : c - half];
    return first ? y[c] * t.x - other * t.y : y[c] * t.x + other * t.y;
}
// A mixer's cache as the path compaction and the benchmark's fill see it (kv.n_kv 0: no pages; channels 0: no ring).
struct MixerCache {
    PagedKv kv;
    float* ring;
    uint32_t ring_len, channels;
    uint32_t recurrent;  // a recurrence's index among the model's (see RecurrentCache)
    const float* per_head;  // the mixer's fixed decays or slopes
};
// The work between an attention mixer's projections and its attention (k_mixer.cu).
struct ConvArgs {
    const float* u;                       // projected rows, q | k | v | ... [n][ldu]
    const uint16_t* w;                    // [channels][taps]; NULL: no convolution (taps is 1, and there is no ring)
    const uint16_t* bias;                 // [channels] (launch_conv_silu), optional
    float* ring;                          // [slot][ring_len][channels]: the projected rows of the positions before the step
    const uint32_t *meta, *tin, *vis;
    const float* rope;                    // [position][rot_dims / 2] (cos, sin)
    PagedKv kv;
    float* q_f;                           // optional: [n][heads][dk]
    uint16_t* q_b;                        // optional: the same times q_scale, bf16
    float q_scale;
    uint32_t ldu, taps, ring_len, conv_channels, heads, rot_dims;
    bool write_ring;                      // false: launch_conv_state does it afterwards
    float unit_eps;                       // with unit_qk: q's and k's heads over sqrt(mean square + unit_eps), times a weight (optional)
    bool unit_qk, unit_v, neighbours;     // unit_v: v's heads likewise, without a weight; neighbours: see Rotation
    ValueMix mix;                         // (behind unit_v; without a convolution)
    float* v_first;                       // [n][kv heads dv]: the values mixed in, which the first layer leaves there
    RowNorm q_norm, k_norm;
    QueryTemperature temp;
};
// Where the row `back` positions before token t lies: among the rows of its own tile of 8 that it descends from (its `vis` mask
// names them: a chain's all, a draft tree's its ancestors), then among the run's earlier rows, then in the slot's ring of rows
// that earlier steps left; none before the sequence's start.
__device__ __forceinline__ const float* row_before(const ConvArgs& a, uint32_t t, uint32_t back) {
    const uint32_t row = a.tin[2 * t + 1], i = row % 8;
    if (back == 0) return a.u + size_t(t) * a.ldu;
    uint32_t anc = a.vis[t] & ((1u << i) - 1);
    const uint32_t n = __popc(anc);
    if (back <= n) {
        uint32_t bit = 0;
        for (uint32_t k = 0; k < back; k++) {
            bit = 31 - __clz(anc);
            anc &= ~(1u << bit);
        }
        return a.u + size_t(t - i + bit) * a.ldu;
    }
    const uint32_t over = back - n;  // positions before the tile
    if (over <= row - i) return a.u + size_t(t - i - over) * a.ldu;
    const uint32_t before = over - (row - i), start = a.meta[2 * (t - row) + 1];  // positions before the run
    if (before > start) return nullptr;
    return a.ring + (size_t(a.tin[2 * t]) * a.ring_len + (start - before) % a.ring_len) * a.conv_channels;
}
void launch_conv_qkv(const ConvArgs& a, uint32_t n, bool fp32, cudaStream_t s);
void launch_conv_state(const ConvArgs& a, const RunIn* runs, uint32_t n_runs, cudaStream_t s);
struct ChunkedAttnArgs {
    const float* q_f;                     // the scalar kernel's q
    const uint16_t* q_b;                  // the tensor-core kernels' q, scale * log2(e) folded in
    const uint32_t *meta, *tin, *vis;
    const uint32_t* ctiles;               // the prefill kernel's (first token, rows <= 64) tiles
    PagedKv kv;
    const float* gate;                    // optional [n][ldg]: the output is multiplied by sigmoid(gate)
    uint32_t ldg, heads, chunk, window;   // what a position sees (see Attention); both 0: every position before
    uint32_t keep;                        // with a window: it sees the first `keep` positions as well
    float scale, softcap;                 // softcap: see Attention
    const float* slopes;                  // optional [heads]: see Attention (not launch_attn_latent)
    const uint16_t* sink;                 // optional [heads], bf16: see LatentAttention (not launch_attn_chunked)
    float* out;                           // optional [n][heads][dv]
    uint16_t* out_b;                      // optional
};
bool chunk_attn_fits(uint32_t dk, uint32_t dv, uint32_t page);  // k_chunk_attn.cu's kernels, bf16 caches; else launch_attn_any
void launch_attn_chunked(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t max_keys, uint32_t sm_count, uint32_t keys_per_block, cudaStream_t s);
void launch_attn_any(const ChunkedAttnArgs& a, uint32_t n, bool fp32, cudaStream_t s);
// What stands between a latent attention's projections (k_latent.cu). From the rows q | c | r of the first one, c at column key_at:
// n(q) for the query projection (with q_rank), and n(c) and r rotated into the cache (kv.dk entries a row).
struct LatentRowsArgs {
    const float* u;                       // [n][ldu]
    RowNorm q_norm, kv_norm;
    const float* rope;
    const uint32_t *meta, *tin;
    PagedKv kv;
    float* q_f;                           // optional: [n][q_rank]
    uint16_t* q_b;                        // optional
    uint32_t ldu, q_rank, key_at, kv_rank, rot_dim;
    bool own, neighbours;                 // own: (c ; r) is this layer's to write
    float eps;
};
void launch_latent_rows(const LatentRowsArgs& a, uint32_t n, bool fp32, cudaStream_t s);
// From the query projection's rows, per head dim | rot_dim: the first parts gathered [n][heads][dim], the rotated ones into their
// place behind kv_rank entries of q [n][heads][kv_rank + rot_dim], all times `factor`; and the per-head products' table of tiles.
struct LatentQueryArgs {
    const float* u;                       // [n][ldu]
    const float* rope;
    const uint32_t* meta;
    float *part_f, *q_f;                  // fp32 ...
    uint16_t *part_b, *q_b;               // ... or bf16, each pair optional
    uint32_t *tiles, *n_tiles;
    uint32_t n, ldu, heads, dim, rot_dim, kv_rank, tile;
    bool neighbours;
    float factor;
};
void launch_latent_query(const LatentQueryArgs& a, cudaStream_t s);
// Both in one launch, where the queries come with (c ; r) from the first projection.
void launch_latent_split(const LatentRowsArgs& r, const LatentQueryArgs& q, bool fp32, cudaStream_t s);
bool latent_attn_fits(uint32_t kv_rank, uint32_t rot_dim, uint32_t page);  // k_latent_attn.cu's kernels, bf16 caches; else launch_attn_any
void launch_attn_latent(const ChunkedAttnArgs& a, uint32_t n, uint32_t n_ctiles, uint32_t max_keys, uint32_t sm_count, uint32_t keys_per_block, uint32_t* err_flag, cudaStream_t s);
void launch_mixer_compact(const RunIn* runs, const uint32_t* path, const uint32_t* path_len, const uint32_t* lens, const MixerCache* caches, uint32_t n_runs, uint32_t n_caches,
                          bool fp32, cudaStream_t s);
void launch_mixer_fill(const MixerCache* caches, uint32_t n_caches, uint32_t slot, uint32_t from, uint32_t to, uint32_t seed, bool fp32, cudaStream_t s);

// Linear recurrences (k_recurrent.cu): per head S_t = D_t S_(t-1) + k_t v_t^T over a state of [N key channels][P value channels]
// in fp32, D_t a number per head (the state space) or one per key channel (time mixing). The state lies as [slot][head][P][Np],
// Np being N rounded up to a multiple of 32 (recurrent_pitch) with zeros behind.
struct RecurrentCache {
    float* state;
    const float* fixed;  // optional, without channel decays: [heads], every token's decay (its key's factor is 1)
    // The rows of a verified run, kept until it is known which of them stand: keys [slot][8][heads / per][N], decays
    // [slot][8][heads][N] or (key scale, decay) [slot][8][heads][2], values [slot][8][heads][P].
    float *keep_k, *keep_d, *keep_v;
    uint32_t heads, per, N, Np, P;  // per: heads that share a key row
    bool channel_decay;
};
struct ScanArgs {
    const float *q, *k, *v;  // row t's of head h at q + t ldq + (h / per) N, k likewise, v + t ldv + h P
    uint32_t ldq, ldk, ldv;
    const float* decay;      // per channel: [n][heads][N]; else [n][heads][2] (the key's factor, the decay), unless c.fixed has them
    const float* bonus;      // per channel: [n][heads], what of v is added to the output, which is read before the update; ...
    const uint16_t* skip;    // ... else per head bf16 (optional), the output being read after it
    RecurrentCache c;
    const RunIn* runs;
    const GenState* gen;     // a sequence that has ended keeps its state
    const uint32_t *meta, *vis;
    uint32_t n_runs, max_run;
    float* y;                // [n][heads P]
    // Optional, without channel decays, of shapes that ssd_fits takes: the rows in bf16, as q, k and v are laid out. Runs of
    // SSD_MIN_RUN tokens or more then go to the tensor cores (k_ssd.cu), and only shorter ones read q, k and v.
    const uint16_t *q_b, *k_b, *v_b, *a_log;
    uint32_t tensor_min;     // (launch_scan's: runs from here on are the tensor cores')
};
constexpr uint32_t SSD_MIN_RUN = 32;
bool ssd_fits(uint32_t N, uint32_t P);
void launch_ssd(const ScanArgs& a, cudaStream_t s);
uint32_t recurrent_pitch(uint32_t N);  // Np
void launch_scan(const ScanArgs& a, cudaStream_t s);
// After acceptance: the states of the verified runs advance over the accepted path's rows.
void launch_recurrent_commit(const RunIn* runs, const uint32_t* path, const uint32_t* path_len, const uint32_t* lens, const RecurrentCache* caches, uint32_t n_runs,
                             uint32_t n_caches, uint32_t max_heads, cudaStream_t s);
void launch_recurrent_fill(const RecurrentCache* caches, uint32_t n_caches, uint32_t slot, uint32_t seed, cudaStream_t s);
// y[t][c] = silu(bias + convolution) for a.conv_channels channels, fp32 and / or bf16, and per head softplus(dt + dt_bias) and exp(-exp(a_log) of that).
struct StepSizeArgs {
    const float* dt;         // [n][ld]
    uint32_t ld, heads;
    const uint16_t *bias, *a_log;
    float* out;              // [n][heads][2]
};
void launch_conv_silu(const ConvArgs& a, const StepSizeArgs& st, uint32_t n, float* y, uint16_t* y_b, cudaStream_t s);
// Row t's mixes with the row before it, h + (h' - h) mu, five of them: [mix][n][channels], fp32 and / or bf16, the last mu's
// first. tiles: the grouped projection's table over the four behind it (group, first row, rows), `tile` rows at most.
struct ShiftArgs {
    ConvArgs c;              // u: the normed rows; the ring
    const uint16_t* mu[5];
    float* out_f32;
    uint16_t* out_bf16;
    uint32_t *tiles, *n_tiles;
    uint32_t tile;
};
void launch_token_shift(const ShiftArgs& a, uint32_t n, cudaStream_t s);
// exp(-exp(w0 + w2 tanh(hid))) per key channel, and per head the sum of r k u over its channels.
struct DecayArgs {
    const float* hid;        // [n][ldh]: w1's product
    const float *r, *k;      // [n][heads dim]
    const uint16_t *w2, *w0, *u;
    uint32_t ldh, rank, heads, dim;
    float *decay, *bonus;    // [n][heads][dim], [n][heads]
};
void launch_decay(const DecayArgs& a, uint32_t n, cudaStream_t s);
// Rows of `groups` equal parts, each over its own root mean square, times w; silu(gate), or sigmoid(gate), goes on before the norm
// or at the end.
struct GatedNormArgs {
    const float *y, *gate;   // [n][width], [n][ldg]
    const uint16_t* w;
    uint32_t width, ldg, groups;
    bool gate_first, sigmoid;
    float eps;
    float* out_f32;          // optional
    uint16_t* out_bf16;      // optional
};
void launch_gated_norm(const GatedNormArgs& a, uint32_t n, cudaStream_t s);

// A mixture of experts (k_moe.cu).
struct RouterArgs {
    const float* x;                       // the stream [n][d]
    RowNorm norm;                         // optional
    const uint16_t *router, *correction;  // correction: optional
    bool sigmoid, renormalized;           // see ExpertLayer
    float* xn;                            // optional: its normed rows
    uint16_t* xn_b;                       // optional, bf16
    uint32_t* ids;                        // [n][top]; experts and beyond: an identity expert
    float* weights;                       // [n][top]
    uint32_t n, d, experts, identity, top;
    float eps;
};
void launch_router(const RouterArgs& a, cudaStream_t s);
struct SortArgs {
    const uint32_t* ids;
    uint32_t *src, *place;                // row -> token, (token, choice) -> row
    const float* weights;                 // with row_weight: [n][top], sorted into it
    float* row_weight;                    // optional
    uint32_t *tiles, *n_tiles;
    uint32_t n, top, experts, tile;
};
void launch_expert_sort(const SortArgs& a, cudaStream_t s);
struct CombineArgs {
    const float *x, *y, *xn, *shared;     // the stream, the experts' rows, the normed stream, the shared expert's rows (optional)
    const uint32_t *ids, *place;
    const float* weights;                 // optional (1)
    float* out;                           // may be x
    RowNorm post;                         // optional: of the sum, before it goes onto x; next_b is then the new row itself
    RowNorm norm;                         // optional: the next layer's norm, into next / next_b
    float* next;
    uint16_t* next_b;
    uint32_t d, experts, top;
    float eps;
};
void launch_combine(const CombineArgs& a, uint32_t n, cudaStream_t s);

// row_skip (optional): rows marked 1 are left untouched (another rule decides them).
void launch_sample(const float* logits, const SampleRow* rows, uint32_t* out, const uint32_t* meta, uint32_t n_rows, uint32_t vocab, cudaStream_t s,
                   const uint32_t* row_skip = nullptr);
// spec_e (optional): a run with spec_e[run] != 0 has that many candidates already settled in out[head0 ..], its path rows 0 .. spec_e - 1.
void launch_accept(const RunIn* runs, const uint32_t* tokens, uint32_t* out, uint32_t* lens, uint32_t* feed, GenState* gen, uint32_t* emitted,
                   uint32_t n_runs, const uint32_t* tree, uint32_t* path, uint32_t* path_len, uint32_t* on_path, cudaStream_t s, const uint32_t* spec_e = nullptr);
void launch_kv_compact(const RunIn* runs, const uint32_t* path, const uint32_t* path_len, const uint32_t* lens, uint16_t* k_cache, uint16_t* v_cache,
                       const uint32_t* page_table, KvArgs kv, uint32_t n_runs, uint32_t n_layers, cudaStream_t s);
void launch_replay_draft(const RunIn* runs, const uint32_t* lens, uint32_t* feed, const uint32_t* trace, const uint32_t* trace_len, ReplayArgs ra,
                         uint32_t n_runs, uint32_t* tree, cudaStream_t s);
// A row of logits' statistics for the rejection-sampling rule: maximum, argmax (ties to the lowest id), and the sum
// of 2^((x - max) log2(e) / T) in the sampler's order.
struct SpecRowStats {
    float max;
    uint32_t argmax;
    float z;
    uint32_t pad;
};
// The rule inside the engine's step (k_spec.cu), device pointers throughout.
struct SpecStepArgs {
    const RunIn* runs;
    uint32_t n_runs, n_head, max_head_rows;
    const SampleRow* samples;  // per head row
    const uint32_t* tokens;    // the step's tokens, resolved
    const uint32_t* meta;      // (slot, position) per token
    const uint32_t* tree;      // [slot][FEED_W]
    const float* logits;       // [head row][vocab]
    uint32_t vocab;
    const float* q_keep;       // [slot][VERIFY_T - 1][v]: the rows the slot's drafts were drawn from
    uint32_t v;
    uint32_t* q_rows;          // [slot]: how many of them are current
    const uint32_t* index_of;  // [vocab]: a target id's index in the draft vocabulary, or NO_TOK
    SpecRowStats* stats;       // [max_head_rows + max_seqs (VERIFY_T - 1)]
    uint32_t* row_skip;        // [head row]: 1 if the sampler is to leave the row to this rule
    uint32_t* spec_e;          // [run]: the candidates this rule settled (0: the run is not its)
    uint32_t* out;             // out_ids
};
void launch_spec_step_stats(const SpecStepArgs& a, cudaStream_t s);
void launch_spec_step_decide(const SpecStepArgs& a, cudaStream_t s);
// The chain drafter's pick of pass i: argmax, or (rule 1, a sampling sequence) a draw from softmax(q / T) with the row kept.
void launch_draft_draw(const float* logits, uint32_t v, const uint32_t* vocab_ids, const RunIn* runs, const SampleRow* samples, const uint32_t* live,
                       const uint32_t* lens, uint32_t n_runs, uint32_t i, uint32_t rule, uint32_t* feed, uint32_t* tree, float* q_keep, uint32_t* q_rows,
                       cudaStream_t s);
// Rejection-sampling acceptance over bf16 draft and target logits on the device (k_spec.cu).
void launch_spec_accept(const uint16_t* p, const uint16_t* q, const uint32_t* drafts, uint32_t streams, uint32_t k, uint32_t vocab, float temperature,
                        const uint64_t* seeds, const uint32_t* pos0, void* stats, uint32_t* accepted, uint32_t* token, uint32_t* rollback, cudaStream_t s);
// The same with its scratch in static device arrays: allocates nothing; device pointers throughout.
// Returns NULL or an error message (a literal).
uint32_t spec_accept_static_max_rows();
const char* launch_spec_accept_static(const uint16_t* p, const uint16_t* q, const uint32_t* drafts, uint32_t streams, uint32_t k, uint32_t vocab,
                                      float temperature, const uint64_t* seeds, const uint32_t* pos0, uint32_t* accepted, uint32_t* token,
                                      uint32_t* rollback, cudaStream_t s);
// A kernel whose (bounded) wait runs out on purpose and sets the error word to `code`: for testing how that is reported.
void launch_stalled_wait(uint32_t* err_flag, uint32_t polls, uint32_t code, cudaStream_t s);
void launch_kv_fill(uint16_t* k_cache, uint16_t* v_cache, const uint32_t* page_table, KvArgs kv, uint32_t n_layers, uint32_t slot, uint32_t from,
                    uint32_t to, uint32_t seed, cudaStream_t s);

}  // namespace vlt
