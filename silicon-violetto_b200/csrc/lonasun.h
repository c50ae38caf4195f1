// The Lonasun design's reader: each layer an attention mixer with sizes of its own (short convolutions behind q, k and v, rotation
// of the heads' first dimensions, positions grouped into chunks, an output gate) and optionally a mixture of experts with
// identity experts and a shared one; a span of layers runs several times in a row, each pass beginning with a projection of
// (stream ; embedding).
#pragma once
#include "layered.h"

namespace vlt {

namespace lonasun {

inline void read_layer(LayeredModel& model, const Json& c, const std::string& pre, FolderLayer& l, uint32_t d) {
    SafeTensors& w = model.w;
    const std::string& type = c.at("type").text("type");
    if (type != "attention") throw Error(pre + ": no mixer named " + type);
    l.norm1.around_zero = l.norm2.around_zero = true;
    model.point(l.norm1.w, pre + "norm1", {d});
    const Json& m = c.at("mixer");
    l.mix.resize(1);
    Attention& a = l.mix[0].attn;
    LayeredModel::sizes(a, m);
    a.gated = true;
    if (!m["mask"].is_null()) a.chunk = m["mask"].at("size").count("mask.size");
    a.conv.taps = m.at("conv").count("conv");
    a.rot.dims = m.at("rot").at("dims").count("rot.dims");
    a.rot.base = m.at("rot").at("base").number("rot.base");
    if (a.rot.dims % 2 || a.rot.dims > a.dim) throw Error(pre + ": rot.dims does not fit the heads");
    model.check_taps(a.conv, pre);
    model.share(a.rot);
    const std::string mx = pre + "mix.";
    model.attention_matrices(a, mx, d);
    const uint32_t qw = a.heads * a.dim, kw = a.kv_heads * a.dim, vw = a.kv_heads * a.vdim;
    a.conv.channels = qw + kw + vw;
    model.point(a.conv.w, mx + "q.conv", {qw, a.conv.taps});
    w.place(mx + "k.conv", {kw, a.conv.taps}, false);
    w.place(mx + "v.conv", {vw, a.conv.taps}, false);
    const Json& f = c["mlp"];
    if (f.is_null()) return;
    const std::string& kind = f.at("kind").text("mlp.kind");
    if (kind != "moe") throw Error(pre + ": no feed-forward named " + kind);
    l.mlp = MlpKind::Experts;
    model.point(l.norm2.w, pre + "norm2", {d});
    ExpertLayer& e = l.experts;
    const std::string ml = pre + "mlp.";
    e.experts = f.at("router").at("experts").count("router.experts");
    e.top = f.at("router").at("top").count("router.top");
    if (!f.at("router")["identity"].is_null()) e.identity = f.at("router")["identity"].count("router.identity");
    e.ff = f.at("expert").at("ff").count("expert.ff");
    if (!f["shared"].is_null()) e.shared_ff = f["shared"].at("ff").count("shared.ff");
    const uint32_t all = e.experts + e.identity;
    if (e.experts == 0 || e.ff == 0 || e.top == 0 || e.top > all) throw Error(pre + ": the router does not fit its experts");
    model.point(e.router, ml + "router", {all, d});
    model.point(e.correction, ml + "correction", {all});
    size_t up = 0, down = 0;
    for (uint32_t i = 0; i < e.experts; i++) {
        const size_t at = w.place(ml + "e" + std::to_string(i) + ".up", {e.ff, d}, i == 0);
        if (i == 0) up = at;
    }
    for (uint32_t i = 0; i < e.experts; i++) {
        const size_t at = w.place(ml + "e" + std::to_string(i) + ".down", {d, e.ff}, i == 0);
        if (i == 0) down = at;
    }
    model.matrix(e.up, e.experts * e.ff, d, up);
    model.matrix(e.down, e.experts * d, e.ff, down);
    if (e.shared_ff) {
        model.matrix(e.shared_up, ml + "shared.up", e.shared_ff, d);
        model.matrix(e.shared_down, ml + "shared.down", d, e.shared_ff);
    }
}

inline void read(LayeredModel& m, const Json& cfg, ModelDesc& md) {
    const std::vector<Json>& list = cfg.at("layers").items;
    m.point(m.embed, "embed", {md.vocab, md.d});
    for (uint32_t i = 0; i < list.size(); i++) read_layer(m, list[i], "l" + std::to_string(i) + ".", m.layers[i], md.d);
    m.final_norm.around_zero = true;
    m.point(m.final_norm.w, "final.norm", {md.d});
    m.matrix(m.head, "head", md.vocab, md.d);
    m.order(cfg["loop"], [](LayerRun& r, uint32_t) { r.loop_in = true; });
    if (!cfg["loop"].is_null()) m.matrix(m.loop_in, "loop.in", md.d, 2 * md.d);
}

}  // namespace lonasun

}  // namespace vlt
