// Model folders: decoders whose config.json lists their layers one by one. This file has the mechanisms a layer can hold, each a
// parameter struct of its own, the list of layer runs, and what the readers of the designs (lonasun.h, leduvik.h, pasovik.h, sopetar.h) share: the
// tensors' places and the loop over a span of layers. A design's reader fills it; engine_layered.cu runs it.
#pragma once
#include <memory>

#include "weights.h"

namespace vlt {

bool decay_fits(uint32_t rank, uint32_t dim);  // of a TimeMix (k_recurrent.cu)

// Of rows: x / sqrt(mean x^2 + eps), times the weight (as stored, or stored around zero: 1 + w). centered: of x less its mean
// (in front of layers and the head only).
struct RowNorm {
    const uint16_t *w = nullptr, *b = nullptr;  // b: what is added at the end (optional, with centered)
    bool around_zero = false, centered = false;
};
// y_t = b[c] + sum_j w[c][j] u_(t - taps + 1 + j) per channel.
struct ShortConv {
    const uint16_t *w = nullptr, *b = nullptr;  // [channels][taps] bf16, no weights: none; [channels], optional
    uint32_t channels = 0, taps = 1;
};
// Pairs of a head's first `dims` dimensions -- i and i + dims / 2, or the neighbours 2 i and 2 i + 1 -- turn by
// position * base^(-2 i / dims) / factor.
struct Rotation {
    uint32_t dims = 0;
    double base = 1, factor = 1;
    bool neighbours = false;
    uint32_t table = 0;  // index among the model's rotations
};
// Queries are multiplied by 1 + coef ln(floor((position + 1) / every) + 1). every 0: not at all.
struct QueryTemperature {
    float coef = 0;
    double every = 0;
};
// Values v of a layer become (1 - share) v + share v', v' being the same token's in the first layer that takes part.
struct ValueMix {
    const uint16_t* share = nullptr;  // one number; none: the layer takes no part
    bool first = false;
};
// Attention over pages of keys. What a position sees of the positions up to its own: those of its own block of `chunk`, or the
// last `window` and the sequence's first `keep`, or (both 0) all.
struct Attention {
    uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, chunk = 0, window = 0, keep = 0;
    float scale = 1;
    float softcap = 0;       // scores become softcap tanh(score / softcap); 0: they stay
    std::vector<float> slopes;  // per head (or none): what a score loses per position between the query and its key, behind the cap
    bool unit_qk = false;    // q's and k's heads are divided by their root mean square, ...
    RowNorm q_norm, k_norm;  // ... and multiplied by a weight of one head's size (optional)
    bool unit_v = false;     // v's heads are divided by their root mean square
    ValueMix mix;            // behind that
    bool gated = false;      // the output times sigmoid(gate)
    Rotation rot;
    QueryTemperature temp;
    ShortConv conv;  // over q | k | v
    Matrix proj, o;  // proj: the rows of q, k, v and, if gated, the gate stacked
    uint32_t v_w() const { return kv_heads * vdim; }
    uint32_t qkv_w() const { return (heads + kv_heads) * dim + kv_heads * vdim; }
    uint32_t out_w() const { return heads * vdim; }
};
// A selective state space: S = exp(-exp(A_h) dt) S + dt B x^T, y = S^T C + D_h x per head; x, B and C out of a short convolution
// and silu, dt = softplus(dt + dt_bias); y silu(z) normed in equal parts.
struct StateSpace {
    uint32_t heads = 0, vdim = 0, state = 0, groups = 1, norm_groups = 1;
    ShortConv conv;  // over x | B | C
    Matrix in, o;    // in: z | x | B | C | dt
    const uint16_t *dt_bias = nullptr, *a_log = nullptr, *skip = nullptr, *norm = nullptr;
    uint32_t inner() const { return heads * vdim; }
    uint32_t channels() const { return inner() + 2 * groups * state; }
};
// A linear recurrence with a decay per key channel: o = r^T (S + diag(u) k v^T), S = diag(w) S + k v^T per head, the inputs each
// read from their own mix of a row and the row before it; o per head to unit rms, normed, times silu(gate).
struct TimeMix {
    uint32_t heads = 0, dim = 0, rank = 0;
    const uint16_t* mu[5] = {};  // r, k, v, g, w: [d]
    Matrix rkvg;                 // four matrices [heads dim][d] stacked
    Matrix w1, o;                // w1 [rank][d]
    const uint16_t *w2 = nullptr, *w0 = nullptr, *bonus = nullptr, *norm = nullptr;  // w2 [heads dim][rank], bonus [heads][dim]
    uint32_t inner() const { return heads * dim; }
};
// Attention whose keys and values are linear in a short normed row c of every position: per head, the key is (W_uk c ; r) with a
// rotated part r that all heads share, the value W_uv c. Only (c ; r) is kept. W_uk goes onto the queries and W_uv onto the sums of
// c: the heads are query heads of one kv head whose key is (c ; r) and whose value is c. Queries come from a normed row of their own,
// or (q_rank 0) straight from the layer's.
struct LatentAttention {
    static constexpr uint32_t OWN = 0xffffffffu;
    uint32_t heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0, q_rank = 0;
    uint32_t window = 0;      // a position sees the last `window` up to its own; 0: all
    float scale = 1;
    Rotation rot;             // of the rotated parts
    uint32_t kv_from = OWN;   // the layer whose (c ; r) this one reads
    const uint16_t* sink = nullptr;  // per head (optional): a logit that takes its share of the softmax and has no value
    bool gate_by_head = false;       // the gate has a row per head, not per output
    Matrix in;                // W_dq (or W_q) | W_dkv (unless kv_from) | W_g stacked
    Matrix uq, uk_t, uv, o;   // uk_t, uv: per head [kv_rank][dim] and [vdim][kv_rank], stacked
    RowNorm q_norm, kv_norm;
    uint32_t key_w() const { return kv_rank + rot_dim; }
    uint32_t query_w() const { return heads * (dim + rot_dim); }
    uint32_t first_w() const { return q_rank ? q_rank : query_w(); }  // rows of `in` in front of W_dkv
    uint32_t gate_w() const { return gate_by_head ? heads : out_w(); }
    uint32_t out_w() const { return heads * vdim; }
    uint32_t kv_w() const { return kv_from == OWN ? key_w() : 0; }  // rows of W_dkv in `in`
};
// Linear attention with a fixed decay per head: S = d_h S + k v^T, o = S^T q; q, k and v through silu; o normed as one row, times
// sigmoid(gate).
struct LinearAttention {
    uint32_t heads = 0, dim = 0, vdim = 0;
    std::vector<float> decay;
    Matrix proj, o;  // proj: q | k | v | gate
    RowNorm norm;
    uint32_t qkv_w() const { return heads * (2 * dim + vdim); }
    uint32_t out_w() const { return heads * vdim; }
};
enum class MixerKind { Attention, StateSpace, TimeMix, Latent, Linear };
struct Mixer {
    MixerKind kind = MixerKind::Attention;
    Attention attn;
    StateSpace ssm;
    TimeMix tmix;
    LatentAttention latent;
    LinearAttention linear;
    RowNorm out;  // on the output, in layers of several mixers
};
// A feed-forward's hidden rows: relu(W_up h)^2; silu(g) u with (g, u) = (W_gate, W_up) h; or g sigmoid(1.702 g) (u + 1) with g cut
// off above `limit` and u outside of +- limit.
enum class Hidden { Relu2, SiluGlu, ClampedGlu };
inline uint32_t hidden_rows(Hidden h, uint32_t ff) { return h == Hidden::Relu2 ? ff : 2 * ff; }  // of `up`: with a gate, its rows and W_up's in turn
// `top` of `experts` + `identity` per token, scores by softmax or sigmoid, the chosen ones' summing to 1 or as they are; a shared
// expert (ff 0: none).
struct ExpertLayer {
    uint32_t experts = 0, identity = 0, top = 0, ff = 0, shared_ff = 0;
    Hidden hidden = Hidden::Relu2;
    float limit = 0;
    bool sigmoid = false, renormalized = true;
    bool scales_input = false;                                // a score multiplies its expert's input, not its output
    const uint16_t *router = nullptr, *correction = nullptr;  // [experts + identity][d], [experts + identity] (optional)
    Matrix up, down;                                          // all experts': [experts * rows][d], [experts * d][ff]
    Matrix shared_up, shared_down;
};
struct DenseLayer {
    Hidden hidden = Hidden::Relu2;
    float limit = 0;
    Matrix up, down;
};
// n(W_proj (gelu(W_gate x) * e)) onto the stream, e a span of the token's row in the model's side table; gelu by tanh.
struct SideInput {
    uint32_t dim = 0, first = 0;  // the span; dim 0: none
    Matrix gate, proj;            // gate's rows and proj's columns padded with zeros
    RowNorm norm;
};
enum class MlpKind { None, Experts, Dense };
struct FolderLayer {
    RowNorm norm1, norm2;
    std::vector<Mixer> mix;  // several: side by side on the same rows, each output normed, the mean added
    MlpKind mlp = MlpKind::None;
    ExpertLayer experts;
    DenseLayer dense;
    bool post_norm = false;  // norm1 and norm2 go onto what the mixer and the feed-forward leave; both read the stream itself
    SideInput side;          // (layers with post_norm)
    bool parallel = false;   // the feed-forward reads norm1's rows, beside the mixer (dense ones; one mixer)
    // X_0 being the embedding and X_(i + 1) what layer run i leaves: what goes on from this run is the sum over j <= i + 1 of depth[j] X_j
    // (optional; all layers or none).
    const uint16_t* depth = nullptr;
};
// A layer run: with a loop a layer runs several times, each with a cache of its own.
struct LayerRun {
    uint32_t layer;
    bool loop_in;    // (stream ; embedding) goes through loop_in first
    bool add_embed;  // the embedding is added to the stream first
};

inline Json read_json(const std::string& path) {
    FILE* f = std::fopen(path.c_str(), "rb");
    if (!f) throw Error(path + ": cannot open");
    std::string text;
    char buf[65536];
    for (size_t n; (n = std::fread(buf, 1, sizeof buf, f)) > 0;) text.append(buf, n);
    std::fclose(f);
    return Json::parse(text.data(), text.size(), path);
}

struct LayeredModel {
    static constexpr uint32_t PAGE = 64;       // positions per cache page
    static constexpr uint32_t MAX_TAPS = 32;   // of a short convolution
    static constexpr uint32_t MAX_STATE = 512; // key channels of a recurrence
    SafeTensors w;
    std::string where;  // for messages
    std::vector<FolderLayer> layers;
    std::vector<LayerRun> runs;
    std::vector<Rotation> rotations;  // the distinct ones
    Matrix loop_in, head;
    const uint16_t *embed = nullptr, *positions = nullptr;  // positions: a learned vector per position (optional)
    uint32_t n_positions = 0;                               // rows of it; sequences are no longer than that
    const uint16_t* side = nullptr;                         // the layers' side inputs: a row of side_w per token id (optional)
    uint32_t side_w = 0;
    RowNorm final_norm;
    float logit_scale = 1, embed_scale = 1;

    // A design's reader: its own part of config.json and the tensors it names.
    using Reader = void (*)(LayeredModel&, const Json&, ModelDesc&);
    static std::unique_ptr<LayeredModel> load(Reader read, const Json& cfg, const std::string& dir, bool host_only, ModelDesc& md) {
        auto m = std::make_unique<LayeredModel>();
        m->where = dir;
        m->w.open(dir + "/model.safetensors");
        md.d = cfg.at("width").count("width");
        md.vocab = md.vocab_real = cfg.at("vocab").count("vocab");
        md.eps = float(cfg.at("norm").at("eps").number("norm.eps"));
        md.page = PAGE;
        m->layers.resize(cfg.at("layers").items.size());  // (their addresses are kept in `fixups` from here on)
        if (m->layers.empty() || md.d == 0 || md.vocab == 0) throw Error(dir + ": a model needs layers, a width and a vocabulary");
        read(*m, cfg, md);
        m->describe(md);
        m->w.to_device(host_only);
        const uint8_t* base = m->w.buffer.as<uint8_t>();
        for (auto& fix : m->fixups) *fix.first = base + fix.second;  // the tensors' addresses, now that they have one
        m->fixups.clear();
        m->w.unmap();
        return m;
    }

    void point(const uint16_t*& p, size_t offset) { fixups.emplace_back(reinterpret_cast<const uint8_t**>(&p), offset); }
    void point(const uint16_t*& p, const std::string& name, const std::vector<uint32_t>& shape) { point(p, w.place(name, shape)); }
    void matrix(Matrix& m, uint32_t rows, uint32_t k, size_t offset) {
        m.m = rows;
        m.k = k;
        fixups.emplace_back(&m.w, offset);
    }
    void matrix(Matrix& m, const std::string& name, uint32_t rows, uint32_t k) { matrix(m, rows, k, w.place(name, {rows, k})); }
    // Rows of zeros after the stack placed last, up to whole tiles of the tensor-core GEMM (where its k fits it): for projections
    // whose consumers read a part of each output row.
    void padded(Matrix& m, uint32_t rows, uint32_t k, size_t offset) {
        const uint32_t whole = k % 64 == 0 ? (rows + 127) / 128 * 128 : rows;
        w.zeros(size_t(whole - rows) * k * 2);
        matrix(m, whole, k, offset);
    }
    // The bias of a matrix whose last rows may be padding: it is the tensor, or the stack, placed last.
    void bias(Matrix& m, uint32_t rows, size_t offset) {
        w.zeros(size_t(m.m - rows) * 2);
        point(m.bias, offset);
    }
    // q, k, v and, if gated, g of an attention, and its output matrix; biased: q, k and v have biases.
    void attention_matrices(Attention& a, const std::string& pre, uint32_t d, bool biased = false) {
        if (a.kv_heads == 0 || a.heads == 0 || a.heads % a.kv_heads || a.dim == 0 || a.vdim == 0) throw Error(pre + ": the heads do not fit the kv heads");
        const uint32_t qw = a.heads * a.dim, kw = a.kv_heads * a.dim, vw = a.kv_heads * a.vdim;
        const size_t at = w.place(pre + "q", {qw, d});
        w.place(pre + "k", {kw, d}, false);
        w.place(pre + "v", {vw, d}, false);
        if (a.gated) w.place(pre + "g", {a.out_w(), d}, false);
        padded(a.proj, qw + kw + vw + (a.gated ? a.out_w() : 0), d, at);
        matrix(a.o, pre + "o", d, a.out_w());
        if (!biased) return;
        const size_t b = w.place(pre + "q.b", {qw});
        w.place(pre + "k.b", {kw}, false);
        w.place(pre + "v.b", {vw}, false);
        bias(a.proj, qw + kw + vw, b);
    }
    // Neighbouring pairs of the first rot.dims of `width` dimensions.
    void neighbours(Rotation& rot, const Json& r, const std::string& pre, uint32_t width) {
        rot.dims = r.at("dims").count("rot.dims");
        rot.base = r.at("base").number("rot.base");
        if (!r["scaling"].is_null()) rot.factor = r["scaling"].at("factor").number("rot.scaling.factor");
        rot.neighbours = true;
        if (rot.dims % 2 || rot.dims > width) throw Error(pre + ": rot.dims does not fit the heads");
        if (!(rot.base > 0) || !(rot.factor > 0)) throw Error(pre + ": rot.base and rot.scaling.factor must be positive");
        share(rot);
    }
    // The sizes of a latent attention (q_rank: if its queries have one) and its rotation.
    void sizes(LatentAttention& a, const Json& m, const std::string& pre) {
        a.heads = m.at("heads").count("heads");
        a.dim = m.at("dim").count("dim");
        a.rot_dim = m.at("rot_dim").count("rot_dim");
        a.vdim = m.at("vdim").count("vdim");
        a.kv_rank = m.at("kv_rank").count("kv_rank");
        a.scale = float(m.at("scale").number("scale"));
        if (a.heads == 0 || a.dim == 0 || a.vdim == 0 || a.kv_rank == 0) throw Error(pre + ": a size of 0");
        neighbours(a.rot, m.at("rot"), pre, a.rot_dim);
        if (a.rot.dims != a.rot_dim) throw Error(pre + ": rot.dims is not rot_dim");
    }
    // What its heads make of the latents, and its output matrix.
    void latent_matrices(LatentAttention& a, const std::string& pre, uint32_t d) {
        matrix(a.uk_t, a.heads * a.kv_rank, a.dim, w.place_transposed(pre + "uk", a.heads, a.dim, a.kv_rank));
        matrix(a.uv, pre + "uv", a.heads * a.vdim, a.kv_rank);
        matrix(a.o, pre + "o", d, a.out_w());
    }
    static void sizes(Attention& a, const Json& m) {
        a.heads = m.at("heads").count("heads");
        a.kv_heads = m.at("kv_heads").count("kv_heads");
        a.dim = m.at("dim").count("dim");
        a.vdim = m.at("vdim").count("vdim");
        a.scale = float(m.at("scale").number("scale"));
    }
    // The rotation's table is the model's: one for all layers that turn alike.
    void share(Rotation& rot) {
        rot.table = uint32_t(std::find_if(rotations.begin(), rotations.end(), [&](const Rotation& r) { return r.dims == rot.dims && r.base == rot.base && r.factor == rot.factor; }) - rotations.begin());
        if (rot.table == rotations.size()) rotations.push_back(rot);
    }
    void check_taps(const ShortConv& c, const std::string& pre) const {
        if (c.taps == 0 || c.taps > MAX_TAPS) throw Error(pre + ": a convolution takes 1 to " + std::to_string(MAX_TAPS) + " taps");
    }
    // The layers' order: a span of them several times in a row. begins(pass): what a pass's first run does with the embedding.
    template <typename F>
    void order(const Json& loop, F&& begins) {
        const uint32_t n = uint32_t(layers.size());
        uint32_t start = 0, stop = 0, times = 0;
        if (!loop.is_null()) {
            start = loop.at("start").count("loop.start");
            stop = loop.at("stop").count("loop.stop");
            times = loop.at("times").count("loop.times");
            if (start >= stop || stop > n || times == 0) throw Error(where + ": the loop does not fit the layers");
        }
        for (uint32_t i = 0; i < start; i++) runs.push_back({i, false, false});
        for (uint32_t t = 0; t < times; t++)
            for (uint32_t i = start; i < stop; i++) {
                LayerRun r{i, false, false};
                if (i == start) begins(r, t);
                runs.push_back(r);
            }
        for (uint32_t i = stop; i < n; i++) runs.push_back({i, false, false});
    }

  private:
    std::vector<std::pair<const uint8_t**, size_t>> fixups;
    // What the step's shared machinery asks about: the widest layer.
    void describe(ModelDesc& md) const {
        md.n_layers = uint32_t(runs.size());
        for (const FolderLayer& l : layers) {
            for (const Mixer& x : l.mix) {
                if (x.kind == MixerKind::Latent) {
                    md.n_heads = std::max(md.n_heads, x.latent.heads);
                    md.n_kv = std::max(md.n_kv, 1u);
                    md.hd = std::max(md.hd, x.latent.dim + x.latent.rot_dim);
                    if (md.attn_scale == 0) md.attn_scale = x.latent.scale;
                }
                if (x.kind != MixerKind::Attention) continue;
                md.n_heads = std::max(md.n_heads, x.attn.heads);
                md.n_kv = std::max(md.n_kv, x.attn.kv_heads);
                md.hd = std::max(md.hd, x.attn.dim);
                if (md.attn_scale == 0) md.attn_scale = x.attn.scale;
            }
            md.ffn = std::max(md.ffn, std::max(l.experts.ff, l.dense.down.k));
        }
    }
};

}  // namespace vlt
