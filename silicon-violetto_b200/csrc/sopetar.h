// The Sopetar design's reader: layers of two kinds -- latent attention over a window, with queries straight from the layer's rows, a
// sink and a gate per head; attention over a window and the sequence's first positions, with unit heads, soft-capped scores that
// distance lowers, and values mixed with an earlier layer's -- each beside a clamped gated feed-forward with biases, or alone, behind
// one layer norm; and an average over all the layers' results so far behind every layer.
#pragma once
#include "layered.h"

namespace vlt {

namespace sopetar {

inline void layer_norm(LayeredModel& model, RowNorm& n, const std::string& name, uint32_t d) {
    n.centered = true;
    model.point(n.w, name, {d});
    model.point(n.b, name + ".b", {d});
}

inline uint32_t window(const Json& mask, const std::string& pre) {
    const uint32_t size = mask.at("size").count("mask.size");
    if (size == 0) throw Error(pre + ": mask.size must be positive");
    return size;
}

inline void attention(LayeredModel& model, const Json& m, const std::string& pre, Attention& a, const Attention*& first, uint32_t d) {
    LayeredModel::sizes(a, m);
    a.unit_qk = a.unit_v = true;
    a.softcap = float(m.at("softcap").number("softcap"));
    if (!(a.softcap > 0)) throw Error(pre + ": softcap must be positive");
    a.window = window(m.at("mask"), pre);
    if (!m.at("mask")["keep_first"].is_null()) a.keep = m.at("mask")["keep_first"].count("mask.keep_first");
    model.attention_matrices(a, pre, d, true);
    for (uint32_t h = 0; h < a.heads; h++) a.slopes.push_back(float(std::exp2(-8.0 * (h + 1) / a.heads)));
    if (!m["v_mix"].flag("v_mix")) return;
    a.mix.first = first == nullptr;
    if (first && (first->kv_heads != a.kv_heads || first->vdim != a.vdim)) throw Error(pre + ": its values do not fit those of the first layer that mixes them");
    if (!first) first = &a;
    model.point(a.mix.share, pre + "vmix", {});
}

inline void latent_attention(LayeredModel& model, const Json& m, const std::string& pre, LatentAttention& a, uint32_t d) {
    SafeTensors& w = model.w;
    model.sizes(a, m, pre);
    a.window = window(m.at("mask"), pre);
    a.gate_by_head = true;
    const size_t at = w.place(pre + "q", {a.query_w(), d});
    w.place(pre + "dkv", {a.kv_w(), d}, false);
    w.place(pre + "g", {a.heads, d}, false);
    model.padded(a.in, a.query_w() + a.kv_w() + a.heads, d, at);
    model.point(a.kv_norm.w, pre + "dkv.norm", {a.kv_rank});
    model.point(a.sink, pre + "sink", {a.heads});
    model.latent_matrices(a, pre, d);
}

inline void dense(LayeredModel& model, const Json& f, const std::string& pre, DenseLayer& l, uint32_t d) {
    SafeTensors& w = model.w;
    const uint32_t ff = f.at("ff").count("mlp.ff");
    if (ff == 0) throw Error(pre + ": a feed-forward of width 0");
    l.hidden = Hidden::ClampedGlu;
    l.limit = float(f.at("limit").number("mlp.limit"));
    model.matrix(l.up, 2 * ff, d, w.place_pairs(pre + "gate", pre + "up", {ff, d}));
    model.bias(l.up, 2 * ff, w.place_pairs(pre + "gate.b", pre + "up.b", {ff}));
    model.matrix(l.down, pre + "down", d, ff);
    model.bias(l.down, d, w.place(pre + "down.b", {d}));
}

inline void read(LayeredModel& m, const Json& cfg, ModelDesc& md) {
    const std::vector<Json>& list = cfg.at("layers").items;
    m.point(m.embed, "embed", {md.vocab, md.d});
    m.embed_scale = float(cfg.at("embedding").at("scale").number("embedding.scale"));
    const Attention* first = nullptr;  // the first layer whose values the others mix in
    for (uint32_t i = 0; i < list.size(); i++) {
        const Json& c = list[i];
        FolderLayer& l = m.layers[i];
        const std::string &type = c.at("type").text("type"), pre = "l" + std::to_string(i) + ".";
        l.parallel = true;
        layer_norm(m, l.norm1, pre + "norm1", md.d);
        l.mix.resize(1);
        if (type == "attention") {
            attention(m, c.at("mixer"), pre + "mix.", l.mix[0].attn, first, md.d);
        } else if (type == "latent_attention") {
            l.mix[0].kind = MixerKind::Latent;
            latent_attention(m, c.at("mixer"), pre + "mix.", l.mix[0].latent, md.d);
        } else {
            throw Error(pre + ": no mixer named " + type);
        }
        const Json& f = c["mlp"];
        if (!f.is_null()) {
            const std::string& kind = f.at("kind").text("mlp.kind");
            if (kind != "dense") throw Error(pre + ": no feed-forward named " + kind);
            l.mlp = MlpKind::Dense;
            dense(m, f, pre + "mlp.", l.dense, md.d);
        }
        m.point(l.depth, pre + "dwa", {i + 2});
    }
    layer_norm(m, m.final_norm, "final.norm", md.d);
    m.matrix(m.head, "head", md.vocab, md.d);
    m.order(Json{}, [](LayerRun&, uint32_t) {});
}

}  // namespace sopetar

}  // namespace vlt
