// The Lonasun design: a decoder whose config.json lists its layers one by one -- each an attention mixer with sizes of its
// own (short convolutions behind q, k and v, rotation of the heads' first dimensions, positions grouped into chunks, an
// output gate) and optionally a mixture of experts with identity experts and a shared one -- and a span of layers that
// runs several times in a row, each pass beginning with a projection of (stream ; embedding) and keeping its own cache.
// The mechanisms are parameter structs of their own, which other designs' layers can hold as well.
#pragma once
#include <memory>

#include "weights.h"

namespace vlt {

// y_t = sum_j w[c][j] u_(t - taps + 1 + j) per channel.
struct ShortConv {
    const uint16_t* w = nullptr;  // [channels][taps] bf16
    uint32_t channels = 0, taps = 1;
};
// Dimensions i and i + dims / 2 of a head's first `dims` turn by position * base^(-2 i / dims).
struct Rotation {
    uint32_t dims = 0;
    double base = 1;
    uint32_t table = 0;  // index among the model's rotations
};
// Attention over pages of keys; chunk: a position sees the keys of its own block of `chunk` positions (0: all before it).
struct GatedAttention {
    uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, chunk = 0;
    float scale = 1;
    Rotation rot;
    ShortConv conv;  // over q | k | v
    Matrix qkvg, o;  // qkvg: the rows of q, k, v and the gate stacked
    uint32_t qkv_w() const { return (heads + kv_heads) * dim + kv_heads * vdim; }
    uint32_t out_w() const { return heads * vdim; }
};
// relu(W_up h)^2 through W_down, `top` of `experts` + `identity` per token, softmax scores, a shared expert (ff 0: none).
struct ExpertLayer {
    uint32_t experts = 0, identity = 0, top = 0, ff = 0, shared_ff = 0;
    const uint16_t *router = nullptr, *correction = nullptr;  // [experts + identity][d], [experts + identity]
    Matrix up, down;                                          // all experts': [experts * ff][d], [experts * d][ff]
    Matrix shared_up, shared_down;
};
struct LonasunLayer {
    const uint16_t *norm1 = nullptr, *norm2 = nullptr;  // stored around zero
    GatedAttention mix;
    bool has_mlp = false;
    ExpertLayer mlp;
};
// A layer run: with a loop a layer runs several times, each with a cache of its own.
struct LayerRun {
    uint32_t layer;
    bool loop_in;  // (stream ; embedding) goes through loop.in first
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

struct LonasunModel {
    static constexpr uint32_t PAGE = 64;      // positions per cache page
    static constexpr uint32_t MAX_TAPS = 32;  // of a short convolution
    SafeTensors w;
    std::vector<LonasunLayer> layers;
    std::vector<LayerRun> runs;
    std::vector<Rotation> rotations;  // the distinct ones
    Matrix loop_in, head;
    const uint16_t *embed = nullptr, *final_norm = nullptr;

    static std::unique_ptr<LonasunModel> load(const Json& cfg, const std::string& dir, bool host_only, ModelDesc& md) {
        auto m = std::make_unique<LonasunModel>();
        m->read(cfg, dir, md);
        m->w.to_device(host_only);
        const uint8_t* base = m->w.buffer.as<uint8_t>();
        for (auto& fix : m->fixups) *fix.first = base + fix.second;  // the tensors' addresses, now that they have one
        m->fixups.clear();
        m->w.unmap();
        return m;
    }

  private:
    std::vector<std::pair<const uint8_t**, size_t>> fixups;
    void point(const uint16_t*& p, size_t offset) { fixups.emplace_back(reinterpret_cast<const uint8_t**>(&p), offset); }
    void matrix(Matrix& m, uint32_t rows, uint32_t k, size_t offset) {
        m.m = rows;
        m.k = k;
        fixups.emplace_back(&m.w, offset);
    }
    void matrix(Matrix& m, const std::string& name, uint32_t rows, uint32_t k) { matrix(m, rows, k, w.place(name, {rows, k})); }

    void read(const Json& cfg, const std::string& dir, ModelDesc& md) {
        w.open(dir + "/model.safetensors");
        md.d = cfg.at("width").count("width");
        md.vocab = md.vocab_real = cfg.at("vocab").count("vocab");
        md.eps = float(cfg.at("norm").at("eps").number("norm.eps"));
        md.page = PAGE;
        const std::vector<Json>& list = cfg.at("layers").items;
        if (list.empty() || md.d == 0 || md.vocab == 0) throw Error(dir + ": a model needs layers, a width and a vocabulary");
        layers.resize(list.size());  // (their addresses are kept in `fixups` from here on)
        point(embed, w.place("embed", {md.vocab, md.d}));
        for (uint32_t i = 0; i < list.size(); i++) read_layer(list[i], "l" + std::to_string(i) + ".", layers[i], md.d);
        point(final_norm, w.place("final.norm", {md.d}));
        matrix(head, "head", md.vocab, md.d);
        const uint32_t n = uint32_t(layers.size());
        const Json& loop = cfg["loop"];
        uint32_t start = 0, stop = 0, times = 0;
        if (!loop.is_null()) {
            start = loop.at("start").count("loop.start");
            stop = loop.at("stop").count("loop.stop");
            times = loop.at("times").count("loop.times");
            if (start >= stop || stop > n || times == 0) throw Error(dir + ": the loop does not fit the layers");
            matrix(loop_in, "loop.in", md.d, 2 * md.d);
        }
        for (uint32_t i = 0; i < start; i++) runs.push_back({i, false});
        for (uint32_t t = 0; t < times; t++)
            for (uint32_t i = start; i < stop; i++) runs.push_back({i, i == start});
        for (uint32_t i = stop; i < n; i++) runs.push_back({i, false});
        // What the step's shared machinery asks about: the widest layer.
        md.n_layers = uint32_t(runs.size());
        for (const LonasunLayer& l : layers) {
            md.n_heads = std::max(md.n_heads, l.mix.heads);
            md.n_kv = std::max(md.n_kv, l.mix.kv_heads);
            md.hd = std::max(md.hd, l.mix.dim);
            md.ffn = std::max(md.ffn, l.mlp.ff);
        }
        md.attn_scale = layers[0].mix.scale;
    }

    void read_layer(const Json& c, const std::string& pre, LonasunLayer& l, uint32_t d) {
        const std::string& type = c.at("type").text("type");
        if (type != "attention") throw Error(pre + ": no mixer named " + type);
        point(l.norm1, w.place(pre + "norm1", {d}));
        const Json& m = c.at("mixer");
        GatedAttention& a = l.mix;
        a.heads = m.at("heads").count("heads");
        a.kv_heads = m.at("kv_heads").count("kv_heads");
        a.dim = m.at("dim").count("dim");
        a.vdim = m.at("vdim").count("vdim");
        a.scale = float(m.at("scale").number("scale"));
        if (!m["mask"].is_null()) a.chunk = m["mask"].at("size").count("mask.size");
        a.conv.taps = m.at("conv").count("conv");
        a.rot.dims = m.at("rot").at("dims").count("rot.dims");
        a.rot.base = m.at("rot").at("base").number("rot.base");
        if (a.kv_heads == 0 || a.heads % a.kv_heads || a.dim == 0 || a.vdim == 0) throw Error(pre + ": the heads do not fit the kv heads");
        if (a.rot.dims % 2 || a.rot.dims > a.dim) throw Error(pre + ": rot.dims does not fit the heads");
        if (a.conv.taps == 0 || a.conv.taps > MAX_TAPS) throw Error(pre + ": a convolution takes 1 to " + std::to_string(MAX_TAPS) + " taps");
        a.rot.table = uint32_t(std::find_if(rotations.begin(), rotations.end(), [&](const Rotation& r) { return r.dims == a.rot.dims && r.base == a.rot.base; }) - rotations.begin());
        if (a.rot.table == rotations.size()) rotations.push_back(a.rot);
        const std::string mx = pre + "mix.";
        const uint32_t qw = a.heads * a.dim, kw = a.kv_heads * a.dim, vw = a.kv_heads * a.vdim, gw = a.out_w();
        const size_t proj = w.place(mx + "q", {qw, d});
        w.place(mx + "k", {kw, d}, false);
        w.place(mx + "v", {vw, d}, false);
        w.place(mx + "g", {gw, d}, false);
        matrix(a.qkvg, qw + kw + vw + gw, d, proj);
        a.conv.channels = qw + kw + vw;
        point(a.conv.w, w.place(mx + "q.conv", {qw, a.conv.taps}));
        w.place(mx + "k.conv", {kw, a.conv.taps}, false);
        w.place(mx + "v.conv", {vw, a.conv.taps}, false);
        matrix(a.o, mx + "o", d, gw);
        const Json& f = c["mlp"];
        if (f.is_null()) return;
        const std::string& kind = f.at("kind").text("mlp.kind");
        if (kind != "moe") throw Error(pre + ": no feed-forward named " + kind);
        l.has_mlp = true;
        point(l.norm2, w.place(pre + "norm2", {d}));
        ExpertLayer& e = l.mlp;
        const std::string ml = pre + "mlp.";
        e.experts = f.at("router").at("experts").count("router.experts");
        e.top = f.at("router").at("top").count("router.top");
        if (!f.at("router")["identity"].is_null()) e.identity = f.at("router")["identity"].count("router.identity");
        e.ff = f.at("expert").at("ff").count("expert.ff");
        if (!f["shared"].is_null()) e.shared_ff = f["shared"].at("ff").count("shared.ff");
        const uint32_t all = e.experts + e.identity;
        if (e.experts == 0 || e.ff == 0 || e.top == 0 || e.top > all) throw Error(pre + ": the router does not fit its experts");
        point(e.router, w.place(ml + "router", {all, d}));
        point(e.correction, w.place(ml + "correction", {all}));
        size_t up = 0, down = 0;
        for (uint32_t i = 0; i < e.experts; i++) {
            const size_t at = w.place(ml + "e" + std::to_string(i) + ".up", {e.ff, d}, i == 0);
            if (i == 0) up = at;
        }
        for (uint32_t i = 0; i < e.experts; i++) {
            const size_t at = w.place(ml + "e" + std::to_string(i) + ".down", {d, e.ff}, i == 0);
            if (i == 0) down = at;
        }
        matrix(e.up, e.experts * e.ff, d, up);
        matrix(e.down, e.experts * d, e.ff, down);
        if (e.shared_ff) {
            matrix(e.shared_up, ml + "shared.up", e.shared_ff, d);
            matrix(e.shared_down, ml + "shared.down", d, e.shared_ff);
        }
    }
};

}  // namespace vlt
