// The step of a Lonasun model: its layer runs in order over the engine's planner, page table, sampler and acceptance.
#include <algorithm>
#include <cmath>

#include "engine.h"

namespace vlt {

void Engine::init_lonasun() {
    const LonasunModel& m = *model.lonasun;
    const ModelDesc& md = model.md;
    lz = std::make_unique<LonasunState>();
    LonasunState& z = *lz;
    const bool f32 = cfg.fp32;
    const size_t n = cfg.max_step_tokens, n16 = (n + 15) / 16 * 16, d = md.d;
    size_t proj = 0, q = 0, out = 0, pairs = 0, hid = 0, sff = 0, tiles = 0, top = 0, rows = 0;
    for (const LonasunLayer& l : m.layers) {
        proj = std::max<size_t>(proj, l.mix.qkvg.m);
        q = std::max<size_t>(q, l.mix.heads * l.mix.dim);
        out = std::max<size_t>(out, l.mix.out_w());
        if (!l.has_mlp) continue;
        const ExpertLayer& e = l.mlp;
        const size_t p = n * e.top;
        top = std::max<size_t>(top, e.top);
        pairs = std::max(pairs, p);
        hid = std::max(hid, p * e.ff);
        rows = std::max(rows, p * d);
        sff = std::max<size_t>(sff, e.shared_ff);
        tiles = std::max(tiles, p / EXPERT_TILE_MIN + std::min<size_t>(e.experts, p) + 1);
    }
    auto f = [](Buffer& b, size_t floats) { b.alloc(floats * 4, false); };
    auto h = [&](Buffer& b, size_t halves) { if (!f32) b.alloc(halves * 2, false); };  // the 16-bit copies
    auto w = [&](Buffer& b, size_t floats) { if (f32) b.alloc(floats * 4, false); };   // their 32-bit counterparts
    f(z.x0, n * d);
    w(z.xn_f, n * d);
    h(z.xn_b, n16 * d);
    if (m.loop_in.m) {
        w(z.cat_f, n * 2 * d);
        h(z.cat_b, n16 * 2 * d);
    }
    f(z.proj, n * proj);
    f(z.q_f, n * q);
    h(z.q_b, n16 * q);
    f(z.attn_f, n * out);
    h(z.attn_b, n16 * out);
    f(z.moe_x, n * d);
    h(z.moe_xb, n16 * d);
    f(z.ids, n * top);
    f(z.weights, n * top);
    f(z.src, pairs);
    f(z.place, pairs);
    f(z.tiles, 3 * tiles);
    f(z.n_tiles, 1);
    w(z.hid_f, hid);
    h(z.hid_b, hid + 256);
    f(z.rows, rows);
    w(z.sh_f, n * sff);
    h(z.sh_b, n16 * sff);
    f(z.shared, n * d);
    // Angles in double, the table in fp32: positions up to the longest sequence and a verified tree past it.
    for (const Rotation& r : m.rotations) {
        const uint32_t npos = cfg.max_seq_len + FEED_W, half = r.dims / 2;
        std::vector<float> tab(size_t(npos) * half * 2);
        for (uint32_t i = 0; i < half; i++) {
            const double freq = std::pow(r.base, -2.0 * i / r.dims);
            for (uint32_t p = 0; p < npos; p++) {
                tab[(size_t(p) * half + i) * 2] = float(std::cos(p * freq));
                tab[(size_t(p) * half + i) * 2 + 1] = float(std::sin(p * freq));
            }
        }
        z.rope.emplace_back();
        z.rope.back().alloc(std::max<size_t>(tab.size() * 4, 16), false);
        z.rope.back().write_vec(0, tab);
    }
    // A ring per (layer run, slot): the rows a convolution reaches back over, and room for a verified run past them.
    size_t ring = 0;
    std::vector<size_t> ring_off;
    for (const LayerRun& r : m.runs) {
        const GatedAttention& a = m.layers[r.layer].mix;
        ring_off.push_back(ring);
        ring += size_t(cfg.max_seqs) * (a.conv.taps - 1 + VERIFY_T) * a.conv.channels;
    }
    f(z.rings, ring);
    uint32_t shift = 0;
    while ((1u << shift) < md.page) shift++;
    const size_t es = f32 ? 4 : 2;
    for (uint32_t i = 0; i < m.runs.size(); i++) {
        const GatedAttention& a = m.layers[m.runs[i].layer].mix;
        MixerCache c{};
        c.kv = PagedKv{kv.k.as<uint8_t>() + kv.k_off[i] * es, kv.v.as<uint8_t>() + kv.v_off[i] * es, kv.page_table.as<uint32_t>(), kv.max_pages, shift, a.kv_heads, a.dim, a.vdim};
        c.ring = z.rings.as<float>() + ring_off[i];
        c.ring_len = a.conv.taps - 1 + VERIFY_T;
        c.channels = a.conv.channels;
        z.run.push_back(c);
    }
    z.caches.alloc(z.run.size() * sizeof(MixerCache), false);
    z.caches.write_vec(0, z.run);
}

void Engine::project(const Matrix& w, uint32_t n, const float* xf, const uint16_t* xb, float* y, uint16_t* yb, uint32_t epi, const float* base) {
    if (!cfg.fp32 && gemm_fits(w, n)) {
        matmul_gemm(w, n, xb, y, yb, epi, base, nullptr);
    } else if (!cfg.fp32 && stream_fits(w, n)) {
        matmul(w, n, nullptr, y, epi, base, nullptr, 0, nullptr, xb, yb);
    } else {
        LinearArgs a{};
        a.W = reinterpret_cast<const uint16_t*>(w.w);
        a.X = cfg.fp32 ? static_cast<const void*>(xf) : xb;
        a.base = base;
        a.Y = y;
        a.Yb = yb;
        a.n = n;
        a.m = w.m;
        a.k = w.k;
        a.epi = epi;
        launch_linear(a, !cfg.fp32, stream);
    }
}

void Engine::encode_forward_lonasun(uint32_t set, const Plan& p, const std::function<void(const LayerCapture&)>* capture) {
    const LonasunModel& m = *model.lonasun;
    const ModelDesc& md = model.md;
    begin_step(set, p);  // upload; the embedding into x0
    LonasunState& z = *lz;
    StepSet& st = sets[set];
    const bool f32 = cfg.fp32;
    const uint32_t n = p.n, d = md.d;
    float* h = s.h.as<float>();
    const float* cur = z.x0.as<float>();  // the stream; h from the first layer on
    // A step whose runs all fit a verified run leaves the convolutions' state as it goes (see MixerCache).
    const bool short_runs = p.max_run <= VERIFY_T;
    bool normed = false;  // the layer before has left norm1's rows
    auto host = [&](const float* dev, size_t count) {
        std::vector<float> v(count);
        VLT_CUDA(cudaMemcpyAsync(v.data(), dev, count * 4, cudaMemcpyDeviceToHost, stream));
        VLT_CUDA(cudaStreamSynchronize(stream));
        return v;
    };
    for (uint32_t ri = 0; ri < m.runs.size(); ri++) {
        const LonasunLayer& l = m.layers[m.runs[ri].layer];
        const GatedAttention& a = l.mix;
        const MixerCache& mc = z.run[ri];
        int sp;
        if (m.runs[ri].loop_in) {
            sp = span_begin(G_SMALL);
            launch_concat_rows(cur, z.x0.as<float>(), n, d, z.cat_f.as<float>(), z.cat_b.as<uint16_t>(), stream);
            span_end(sp);
            sp = span_begin(G_MATMUL);
            project(m.loop_in, n, z.cat_f.as<float>(), z.cat_b.as<uint16_t>(), h, nullptr, EPI_RAW);
            span_end(sp);
            cur = h;
        }
        std::vector<float> resid_in, sdpa;
        if (capture) resid_in = host(cur, size_t(n) * d);
        if (!normed) {
            sp = span_begin(G_SMALL);
            launch_norm_rows(cur, nullptr, n, d, md.eps, l.norm1, z.xn_f.as<float>(), z.xn_b.as<uint16_t>(), stream);
            span_end(sp);
        }
        sp = span_begin(G_MATMUL);
        project(a.qkvg, n, z.xn_f.as<float>(), z.xn_b.as<uint16_t>(), z.proj.as<float>(), nullptr, EPI_RAW);
        span_end(sp);
        ConvArgs c{};
        c.u = z.proj.as<float>();
        c.w = a.conv.w;
        c.ring = mc.ring;
        c.meta = s.meta.as<uint32_t>();
        c.tin = st.in<uint32_t>(st.o_tin);
        c.vis = st.in<uint32_t>(st.o_vis);
        c.rope = z.rope[a.rot.table].as<float>();
        c.kv = mc.kv;
        c.ldu = a.qkvg.m;
        c.taps = a.conv.taps;
        c.ring_len = mc.ring_len;
        c.conv_channels = mc.channels;
        c.heads = a.heads;
        c.rot_dims = a.rot.dims;
        c.write_ring = short_runs;
        const bool fast_attn = !f32 && !tuning.plain_attention && chunk_attn_fits(a.dim, a.vdim, md.page);
        if (fast_attn) c.q_b = z.q_b.as<uint16_t>();
        else c.q_f = z.q_f.as<float>();
        c.q_scale = a.scale * LOG2E;
        sp = span_begin(G_SMALL);
        launch_conv_qkv(c, n, f32, stream);
        if (!short_runs) launch_conv_state(c, st.in<RunIn>(st.o_runs), p.n_runs, stream);
        span_end(sp);
        ChunkedAttnArgs at{};
        at.q_f = z.q_f.as<float>();
        at.q_b = z.q_b.as<uint16_t>();
        at.ctiles = st.in<uint32_t>(st.o_ctiles);
        at.meta = c.meta;
        at.tin = c.tin;
        at.vis = c.vis;
        at.kv = mc.kv;
        at.gate = z.proj.as<float>() + a.qkv_w();
        at.ldg = a.qkvg.m;
        at.heads = a.heads;
        at.chunk = a.chunk;
        at.scale = a.scale;
        at.out = f32 || capture ? z.attn_f.as<float>() : nullptr;
        at.out_b = z.attn_b.as<uint16_t>();
        sp = span_begin(G_ATTN);
        if (fast_attn) launch_attn_chunked(at, n, p.chunked ? p.ctiles : 0, a.chunk ? std::min(p.max_keys, a.chunk) : p.max_keys, sm_count, tuning.attn_keys_per_cta, stream);
        else launch_attn_any(at, n, f32, stream);
        span_end(sp);
        if (capture) sdpa = host(z.attn_f.as<float>(), size_t(n) * a.out_w());
        sp = span_begin(G_MATMUL);
        project(a.o, n, z.attn_f.as<float>(), z.attn_b.as<uint16_t>(), h, nullptr, EPI_RESID, cur);
        span_end(sp);
        cur = h;
        normed = false;
        if (l.has_mlp) {
            const bool next_norm = ri + 1 < m.runs.size() && !m.runs[ri + 1].loop_in;
            encode_experts(l, n, next_norm ? m.layers[m.runs[ri + 1].layer].norm1 : nullptr);
            normed = next_norm;
        }
        if (capture) {
            const std::vector<float> resid_out = host(h, size_t(n) * d);
            LayerCapture lc{ri, n, resid_in.data(), nullptr, nullptr, sdpa.data(), nullptr, nullptr, nullptr};
            lc.resid_out = resid_out.data();
            lc.attn_width = a.out_w();
            (*capture)(lc);
        }
        // (kernels.metal:133-148 `tap_rows`, as the other architectures' taps)
        auto tap = std::find(tap_layers.begin(), tap_layers.end(), ri);
        if (tap != tap_layers.end()) launch_prep_rows(h, nullptr, n, d, md.eps, tap_bufs[tap - tap_layers.begin()].as<float>(), nullptr, nullptr, true, true, stream);
    }
    // The tail: the final norm of the hidden and head rows, the head, sampling, accept, compaction.
    const int sp = span_begin(G_TAIL);
    launch_norm_rows(h, st.in<uint32_t>(st.o_hidden_rows), p.n_hidden, d, md.eps, m.final_norm, s.hfin_all.as<float>(), nullptr, stream);
    if (p.n_head) {
        launch_norm_rows(h, st.in<uint32_t>(st.o_head_rows), p.n_head, d, md.eps, m.final_norm, s.hfin_head.as<float>(), f32 ? nullptr : s.hfin_b.as<uint16_t>(), stream);
        project(model.head, p.n_head, s.hfin_head.as<float>(), s.hfin_b.as<uint16_t>(), s.logits.as<float>(), nullptr, EPI_RAW);
        if (!forced_logits.empty()) {
            if (forced_logits.size() != size_t(p.n_head) * md.vocab) throw Error("forced logits: wrong size");
            VLT_CUDA(cudaMemcpyAsync(s.logits.dev, forced_logits.data(), forced_logits.size() * 4, cudaMemcpyHostToDevice, stream));
        }
        launch_sample(s.logits.as<float>(), st.in<SampleRow>(st.o_sample_rows), st.out<uint32_t>(st.o_out_ids), s.meta.as<uint32_t>(), p.n_head, md.vocab, stream, nullptr);
    }
    launch_accept(st.in<RunIn>(st.o_runs), st.in<uint32_t>(st.o_tokens), st.out<uint32_t>(st.o_out_ids), s.lens.as<uint32_t>(), s.feed.as<uint32_t>(), s.gen.as<GenState>(),
                  st.out<uint32_t>(st.o_emitted), p.n_runs, s.tree.as<uint32_t>(), s.path.as<uint32_t>(), s.path_len.as<uint32_t>(), s.on_path.as<uint32_t>(), stream, nullptr);
    if (p.branches)
        launch_mixer_compact(st.in<RunIn>(st.o_runs), s.path.as<uint32_t>(), s.path_len.as<uint32_t>(), s.lens.as<uint32_t>(), z.caches.as<MixerCache>(), p.n_runs,
                             md.n_layers, f32, stream);
    span_end(sp);
}

// h += the experts' weighted rows + the shared expert's, on norm2's rows of h; norm: the norm the next layer run begins
// with, whose rows are then left as well.
void Engine::encode_experts(const LonasunLayer& l, uint32_t n, const uint16_t* norm) {
    LonasunState& z = *lz;
    const ExpertLayer& e = l.mlp;
    const bool f32 = cfg.fp32;
    const uint32_t d = model.md.d, pairs = n * e.top;
    float* h = s.h.as<float>();
    RouterArgs r{};
    r.x = h;
    r.norm = l.norm2;
    r.router = e.router;
    r.correction = e.correction;
    r.xn = f32 || e.identity ? z.moe_x.as<float>() : nullptr;
    r.xn_b = z.moe_xb.as<uint16_t>();
    r.ids = z.ids.as<uint32_t>();
    r.weights = z.weights.as<float>();
    r.n = n;
    r.d = d;
    r.experts = e.experts;
    r.identity = e.identity;
    r.top = e.top;
    r.eps = model.md.eps;
    SortArgs so{};
    so.ids = r.ids;
    so.src = z.src.as<uint32_t>();
    so.place = z.place.as<uint32_t>();
    so.tiles = z.tiles.as<uint32_t>();
    so.n_tiles = z.n_tiles.as<uint32_t>();
    so.n = n;
    so.top = e.top;
    so.experts = e.experts;
    // The experts' matrices on the tensor cores where their sizes fit: tiles as long as an expert's rows on average, so that
    // its weights are read once. On the CUDA cores a tile has 64.
    const bool fast = !f32 && grouped_fits(e.ff, d) && grouped_fits(d, e.ff);
    so.tile = 64;
    if (fast)
        for (so.tile = EXPERT_TILE_MIN; so.tile < 128 && so.tile < 2 * pairs / (e.experts + e.identity);) so.tile *= 2;
    int sp = span_begin(G_SMALL);
    launch_router(r, stream);
    launch_expert_sort(so, stream);
    span_end(sp);
    sp = span_begin(G_MATMUL);
    LinearArgs up{};
    up.W = reinterpret_cast<const uint16_t*>(e.up.w);
    up.X = f32 ? static_cast<const void*>(z.moe_x.as<float>()) : z.moe_xb.as<uint16_t>();
    up.src = so.src;
    up.Y = z.hid_f.as<float>();
    up.Yb = z.hid_b.as<uint16_t>();
    up.m = e.ff;
    up.k = d;
    up.epi = EPI_RELU2;
    up.tiles = so.tiles;
    up.n_tiles = so.n_tiles;
    up.max_tiles = pairs / so.tile + std::min(e.experts, pairs);
    if (fast) launch_grouped(up, e.experts, so.tile, s.err_flag.as<uint32_t>(), stream);
    else launch_linear(up, !f32, stream);
    LinearArgs down = up;
    down.W = reinterpret_cast<const uint16_t*>(e.down.w);
    down.X = f32 ? static_cast<const void*>(z.hid_f.as<float>()) : z.hid_b.as<uint16_t>();
    down.src = nullptr;
    down.Y = z.rows.as<float>();
    down.Yb = nullptr;
    down.m = d;
    down.k = e.ff;
    down.epi = EPI_RAW;
    if (fast) launch_grouped(down, e.experts, so.tile, s.err_flag.as<uint32_t>(), stream);
    else launch_linear(down, !f32, stream);
    if (e.shared_ff) {
        project(e.shared_up, n, z.moe_x.as<float>(), z.moe_xb.as<uint16_t>(), z.sh_f.as<float>(), z.sh_b.as<uint16_t>(), EPI_RELU2);
        project(e.shared_down, n, z.sh_f.as<float>(), z.sh_b.as<uint16_t>(), z.shared.as<float>(), nullptr, EPI_RAW);
    }
    span_end(sp);
    CombineArgs c{};
    c.x = h;
    c.y = z.rows.as<float>();
    c.xn = z.moe_x.as<float>();
    c.shared = e.shared_ff ? z.shared.as<float>() : nullptr;
    c.ids = r.ids;
    c.place = so.place;
    c.weights = r.weights;
    c.out = h;
    c.norm = norm;
    c.next = z.xn_f.as<float>();
    c.next_b = z.xn_b.as<uint16_t>();
    c.d = d;
    c.experts = e.experts;
    c.top = e.top;
    c.eps = model.md.eps;
    sp = span_begin(G_SMALL);
    launch_combine(c, n, stream);
    span_end(sp);
}

}  // namespace vlt
