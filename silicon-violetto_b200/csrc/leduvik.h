// The Leduvik design's reader: layers of three kinds -- attention over a sliding window with q and k heads of unit length and no
// positions in its scores, a selective state space, and, side by side on the same rows, attention over all positions with
// longer queries the further on they are and a time-mixing recurrence -- each optionally followed by a dense feed-forward; a
// learned vector per position; a span of layers that runs several times in a row, the embedding added before each pass but
// the first; scaled logits.
#pragma once
#include "layered.h"

namespace vlt {

namespace leduvik {

inline void window_attention(LayeredModel& model, const Json& m, const std::string& pre, Attention& a, uint32_t d) {
    LayeredModel::sizes(a, m);
    a.unit_qk = true;
    if (!m["mask"].is_null()) {
        a.window = m["mask"].at("size").count("mask.size");
        if (a.window == 0) throw Error(pre + ": a window of 0 positions");
    }
    model.attention_matrices(a, pre, d);
}

inline void tempered_attention(LayeredModel& model, const Json& m, const std::string& pre, Attention& a, uint32_t d) {
    LayeredModel::sizes(a, m);
    if (!m["q_temp"].is_null()) {
        a.temp.coef = float(m["q_temp"].at("coef").number("q_temp.coef"));
        a.temp.every = m["q_temp"].at("every").number("q_temp.every");
        if (!(a.temp.every > 0)) throw Error(pre + ": q_temp.every must be positive");
    }
    model.attention_matrices(a, pre, d);
}

inline void state_space(LayeredModel& model, const Json& m, const std::string& pre, StateSpace& s, uint32_t d) {
    s.heads = m.at("heads").count("heads");
    s.vdim = m.at("vdim").count("vdim");
    s.state = m.at("state").count("state");
    s.groups = m.at("groups").count("groups");
    s.norm_groups = m.at("norm_groups").count("norm_groups");
    s.conv.taps = m.at("conv").count("conv");
    if (s.heads == 0 || s.vdim == 0 || s.state == 0 || s.groups == 0 || s.heads % s.groups) throw Error(pre + ": the heads do not fit the groups");
    if (s.state > LayeredModel::MAX_STATE) throw Error(pre + ": a state of at most " + std::to_string(LayeredModel::MAX_STATE) + " channels");
    if (s.norm_groups == 0 || s.inner() % s.norm_groups) throw Error(pre + ": the norm's groups do not fit the heads");
    model.check_taps(s.conv, pre);
    const uint32_t rows = s.inner() + s.channels() + s.heads;
    model.padded(s.in, rows, d, model.w.place(pre + "in", {rows, d}));
    s.conv.channels = s.channels();
    model.point(s.conv.w, pre + "conv", {s.channels(), s.conv.taps});
    model.point(s.conv.b, pre + "conv.b", {s.channels()});
    model.point(s.dt_bias, pre + "dt_bias", {s.heads});
    model.point(s.a_log, pre + "A_log", {s.heads});
    model.point(s.skip, pre + "D", {s.heads});
    model.point(s.norm, pre + "norm", {s.inner()});
    model.matrix(s.o, pre + "o", d, s.inner());
}

inline void time_mix(LayeredModel& model, const Json& m, const std::string& pre, TimeMix& t, uint32_t d) {
    SafeTensors& w = model.w;
    t.heads = m.at("heads").count("heads");
    t.dim = m.at("dim").count("dim");
    if (t.heads == 0 || t.dim == 0 || t.dim > LayeredModel::MAX_STATE) throw Error(pre + ": heads of 1 to " + std::to_string(LayeredModel::MAX_STATE) + " channels");
    const uint32_t K = t.inner();
    const char* mixes[5] = {"mu.r", "mu.k", "mu.v", "mu.g", "mu.w"};
    for (int i = 0; i < 5; i++) model.point(t.mu[i], pre + mixes[i], {d});
    const size_t at = w.place(pre + "r", {K, d});
    for (const char* c : {"k", "v", "g"}) w.place(pre + c, {K, d}, false);
    model.matrix(t.rkvg, K, d, at);
    t.rank = w.rows(pre + "w1");  // (no key of config.json has it)
    if (!decay_fits(t.rank, t.dim)) throw Error(pre + ": decays of rank " + std::to_string(t.rank) + " over heads of " + std::to_string(t.dim) + " do not fit shared memory");
    model.padded(t.w1, t.rank, d, w.place(pre + "w1", {t.rank, d}));
    model.point(t.w2, pre + "w2", {K, t.rank});
    model.point(t.w0, pre + "w0", {K});
    model.point(t.bonus, pre + "u", {t.heads, t.dim});
    model.point(t.norm, pre + "norm", {K});
    model.matrix(t.o, pre + "o", d, K);
}

inline void read_layer(LayeredModel& model, const Json& c, const std::string& pre, FolderLayer& l, uint32_t d) {
    const std::string &type = c.at("type").text("type"), mx = pre + "mix.";
    const Json& m = c.at("mixer");
    model.point(l.norm1.w, pre + "norm1", {d});
    l.mix.resize(type == "parallel" ? 2 : 1);
    if (type == "attention") {
        window_attention(model, m, mx, l.mix[0].attn, d);
    } else if (type == "mamba2") {
        l.mix[0].kind = MixerKind::StateSpace;
        state_space(model, m, mx, l.mix[0].ssm, d);
    } else if (type == "parallel") {
        tempered_attention(model, m.at("left"), mx + "left.", l.mix[0].attn, d);
        model.point(l.mix[0].out.w, mx + "left.out", {d});
        l.mix[1].kind = MixerKind::TimeMix;
        time_mix(model, m.at("right"), mx + "right.", l.mix[1].tmix, d);
        model.point(l.mix[1].out.w, mx + "right.out", {d});
    } else {
        throw Error(pre + ": no mixer named " + type);
    }
    const Json& f = c["mlp"];
    if (f.is_null()) return;
    const std::string& kind = f.at("kind").text("mlp.kind");
    if (kind != "dense") throw Error(pre + ": no feed-forward named " + kind);
    l.mlp = MlpKind::Dense;
    model.point(l.norm2.w, pre + "norm2", {d});
    const uint32_t ff = f.at("ff").count("mlp.ff");
    if (ff == 0) throw Error(pre + ": a feed-forward of width 0");
    model.matrix(l.dense.up, pre + "mlp.up", ff, d);
    model.matrix(l.dense.down, pre + "mlp.down", d, ff);
}

inline void read(LayeredModel& m, const Json& cfg, ModelDesc& md) {
    const std::vector<Json>& list = cfg.at("layers").items;
    m.point(m.embed, "embed", {md.vocab, md.d});
    m.n_positions = cfg.at("max_positions").count("max_positions");
    if (m.n_positions == 0) throw Error(m.where + ": max_positions must be positive");
    m.point(m.positions, "pos", {m.n_positions, md.d});
    for (uint32_t i = 0; i < list.size(); i++) read_layer(m, list[i], "l" + std::to_string(i) + ".", m.layers[i], md.d);
    m.point(m.final_norm.w, "final.norm", {md.d});
    m.matrix(m.head, "head", md.vocab, md.d);
    m.logit_scale = float(cfg.at("logit_scale").number("logit_scale"));
    m.order(cfg["loop"], [](LayerRun& r, uint32_t pass) { r.add_embed = pass > 0; });
}

}  // namespace leduvik

}  // namespace vlt
