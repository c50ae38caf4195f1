// The Pasovik design's reader: layers of three kinds -- attention over all positions with normed q and k heads, rotated neighbours
// and soft-capped scores; latent attention with an output gate, some of whose layers read an earlier one's latents; linear
// attention with a fixed decay per head -- each followed by a gated feed-forward, by a mixture of gated experts whose scores go
// onto their inputs, or by neither; norms on what the mixer and the feed-forward leave; and in every layer an input of the
// token's own.
#pragma once
#include "layered.h"

namespace vlt {

namespace pasovik {

inline void attention(LayeredModel& model, const Json& m, const std::string& pre, Attention& a, uint32_t d) {
    LayeredModel::sizes(a, m);
    a.unit_qk = true;
    if (!m["softcap"].is_null()) {
        a.softcap = float(m["softcap"].number("softcap"));
        if (!(a.softcap > 0)) throw Error(pre + ": softcap must be positive");
    }
    model.neighbours(a.rot, m.at("rot"), pre, a.dim);
    model.attention_matrices(a, pre, d);
    model.point(a.q_norm.w, pre + "q.norm", {a.dim});
    model.point(a.k_norm.w, pre + "k.norm", {a.dim});
}

inline void latent_attention(LayeredModel& model, const Json& m, const std::string& pre, uint32_t index, LatentAttention& a, uint32_t d) {
    SafeTensors& w = model.w;
    model.sizes(a, m, pre);
    a.q_rank = m.at("q_rank").count("q_rank");
    if (a.q_rank == 0) throw Error(pre + ": a size of 0");
    if (!m["kv_from"].is_null()) {
        a.kv_from = m["kv_from"].count("kv_from");
        const std::vector<Mixer>* from = a.kv_from < index ? &model.layers[a.kv_from].mix : nullptr;
        if (!from || (*from)[0].kind != MixerKind::Latent) throw Error(pre + ": kv_from " + std::to_string(a.kv_from) + " is no latent layer before this one");
        const LatentAttention& b = (*from)[0].latent;
        if (b.kv_from != LatentAttention::OWN) throw Error(pre + ": kv_from " + std::to_string(a.kv_from) + " has no latents of its own");
        if (b.kv_rank != a.kv_rank || b.rot_dim != a.rot_dim || b.rot.table != a.rot.table) throw Error(pre + ": the latents of layer " + std::to_string(a.kv_from) + " do not fit");
    }
    const size_t at = w.place(pre + "dq", {a.q_rank, d});
    if (a.kv_w()) w.place(pre + "dkv", {a.kv_w(), d}, false);
    w.place(pre + "g", {a.out_w(), d}, false);
    model.padded(a.in, a.q_rank + a.kv_w() + a.out_w(), d, at);
    model.point(a.q_norm.w, pre + "dq.norm", {a.q_rank});
    if (a.kv_w()) model.point(a.kv_norm.w, pre + "dkv.norm", {a.kv_rank});
    model.padded(a.uq, a.query_w(), a.q_rank, w.place(pre + "uq", {a.query_w(), a.q_rank}));
    model.latent_matrices(a, pre, d);
}

inline void lightning(LayeredModel& model, const Json& m, const std::string& pre, LinearAttention& a, uint32_t d) {
    SafeTensors& w = model.w;
    a.heads = m.at("heads").count("heads");
    a.dim = m.at("dim").count("dim");
    a.vdim = m.at("vdim").count("vdim");
    if (a.heads == 0 || a.vdim == 0 || a.dim == 0 || a.dim > LayeredModel::MAX_STATE) throw Error(pre + ": heads of 1 to " + std::to_string(LayeredModel::MAX_STATE) + " channels");
    for (const Json& x : m.at("decay").items) a.decay.push_back(float(x.number("decay")));
    if (a.decay.size() != a.heads) throw Error(pre + ": " + std::to_string(a.decay.size()) + " decays for " + std::to_string(a.heads) + " heads");
    const size_t at = w.place(pre + "q", {a.heads * a.dim, d});
    w.place(pre + "k", {a.heads * a.dim, d}, false);
    w.place(pre + "v", {a.out_w(), d}, false);
    w.place(pre + "g", {a.out_w(), d}, false);
    model.padded(a.proj, a.qkv_w() + a.out_w(), d, at);
    model.point(a.norm.w, pre + "norm", {a.out_w()});
    model.matrix(a.o, pre + "o", d, a.out_w());
}

inline void dense(LayeredModel& model, const Json& f, const std::string& pre, DenseLayer& l, uint32_t d) {
    const uint32_t ff = f.at("ff").count("mlp.ff");
    if (ff == 0) throw Error(pre + ": a feed-forward of width 0");
    l.hidden = Hidden::SiluGlu;
    model.matrix(l.up, 2 * ff, d, model.w.place_pairs(pre + "gate", pre + "up", {ff, d}));
    model.matrix(l.down, pre + "down", d, ff);
}

inline void experts(LayeredModel& model, const Json& f, const std::string& pre, ExpertLayer& e, uint32_t d) {
    SafeTensors& w = model.w;
    e.experts = f.at("router").at("experts").count("router.experts");
    e.top = f.at("router").at("top").count("router.top");
    e.ff = f.at("expert").at("ff").count("expert.ff");
    e.limit = float(f.at("expert").at("limit").number("expert.limit"));
    e.hidden = Hidden::ClampedGlu;
    e.sigmoid = e.scales_input = true;
    e.renormalized = false;
    if (e.experts == 0 || e.ff == 0 || e.top == 0 || e.top > e.experts) throw Error(pre + ": the router does not fit its experts");
    model.point(e.router, pre + "router", {e.experts, d});
    size_t up = 0, down = 0;
    for (uint32_t i = 0; i < e.experts; i++) {
        const std::string ei = pre + "e" + std::to_string(i);
        const size_t at = w.place_pairs(ei + ".gate", ei + ".up", {e.ff, d}, i == 0);
        if (i == 0) up = at;
    }
    for (uint32_t i = 0; i < e.experts; i++) {
        const size_t at = w.place(pre + "e" + std::to_string(i) + ".down", {d, e.ff}, i == 0);
        if (i == 0) down = at;
    }
    model.matrix(e.up, e.experts * 2 * e.ff, d, up);
    model.matrix(e.down, e.experts * d, e.ff, down);
}

inline void read_layer(LayeredModel& model, const Json& c, uint32_t index, FolderLayer& l, uint32_t d) {
    const std::string &type = c.at("type").text("type"), pre = "l" + std::to_string(index) + ".", mx = pre + "mix.";
    const Json& m = c.at("mixer");
    l.post_norm = true;
    model.point(l.norm1.w, pre + "norm1", {d});
    l.mix.resize(1);
    if (type == "attention") {
        attention(model, m, mx, l.mix[0].attn, d);
    } else if (type == "latent_attention") {
        l.mix[0].kind = MixerKind::Latent;
        latent_attention(model, m, mx, index, l.mix[0].latent, d);
    } else if (type == "lightning") {
        l.mix[0].kind = MixerKind::Linear;
        lightning(model, m, mx, l.mix[0].linear, d);
    } else {
        throw Error(pre + ": no mixer named " + type);
    }
    const Json& f = c["mlp"];
    if (!f.is_null()) {
        const std::string& kind = f.at("kind").text("mlp.kind");
        l.mlp = kind == "dense" ? MlpKind::Dense : MlpKind::Experts;
        if (kind == "dense") dense(model, f, pre + "mlp.", l.dense, d);
        else if (kind == "moe") experts(model, f, pre + "mlp.", l.experts, d);
        else throw Error(pre + ": no feed-forward named " + kind);
        model.point(l.norm2.w, pre + "norm2", {d});
    }
    if (!model.side_w) return;
    SideInput& s = l.side;
    s.dim = model.side_w / uint32_t(model.layers.size());
    s.first = index * s.dim;
    const uint32_t wide = (s.dim + 63) / 64 * 64;
    model.padded(s.gate, s.dim, d, model.w.place(pre + "side.gate", {s.dim, d}));
    model.matrix(s.proj, d, wide, model.w.place_wide(pre + "side.proj", d, s.dim, wide));
    model.point(s.norm.w, pre + "side.norm", {d});
}

inline void read(LayeredModel& m, const Json& cfg, ModelDesc& md) {
    const std::vector<Json>& list = cfg.at("layers").items;
    m.point(m.embed, "embed", {md.vocab, md.d});
    if (!cfg["token_side"].is_null()) {
        m.side_w = cfg["token_side"].at("dim").count("token_side.dim") * uint32_t(list.size());
        if (m.side_w == 0) throw Error(m.where + ": token_side.dim must be positive");
        m.point(m.side, "side.embed", {md.vocab, m.side_w});
    }
    for (uint32_t i = 0; i < list.size(); i++) read_layer(m, list[i], i, m.layers[i], md.d);
    m.point(m.final_norm.w, "final.norm", {md.d});
    m.matrix(m.head, "head", md.vocab, md.d);
    m.order(Json{}, [](LayerRun&, uint32_t) {});
}

}  // namespace pasovik

}  // namespace vlt
