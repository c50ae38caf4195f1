// The step of a model folder: its layer runs in order over the engine's planner, page table, sampler and acceptance.
#include <algorithm>
#include <cmath>

#include "engine.h"

namespace vlt {

void Engine::init_layered() {
    const LayeredModel& m = *model.layered;
    const ModelDesc& md = model.md;
    lay = std::make_unique<LayeredState>();
    LayeredState& z = *lay;
    const bool f32 = cfg.fp32;
    const size_t n = cfg.max_step_tokens, n16 = (n + 15) / 16 * 16, d = md.d;
    size_t proj = 0, q = 0, out = 0, pairs = 0, hid = 0, sff = 0, tiles = 0, top = 0, rows = 0, ff = 0, branch = 0, channels = 0, y = 0, inner = 0, heads = 0, low = 0;
    size_t halves = 0, lat = 0, uq = 0, part = 0, mid = 0, side = 0, side_wide = 0, v_first = 0;
    bool shift = false, depth = false;
    for (const FolderLayer& l : m.layers) {
        if (l.mix.size() > 1) branch = 2 * d;
        else if (l.post_norm) branch = std::max(branch, d);
        depth = depth || l.depth;
        side = std::max<size_t>(side, l.side.gate.m);
        side_wide = std::max<size_t>(side_wide, l.side.proj.k);
        for (const Mixer& x : l.mix) {
            if (x.kind == MixerKind::Attention) {
                proj = std::max<size_t>(proj, x.attn.proj.m);
                q = std::max<size_t>(q, x.attn.heads * x.attn.dim);
                out = std::max<size_t>(out, x.attn.out_w());
                if (x.attn.mix.share) v_first = std::max<size_t>(v_first, x.attn.v_w());
            } else if (x.kind == MixerKind::StateSpace) {
                proj = std::max<size_t>(proj, x.ssm.in.m);
                channels = std::max<size_t>(channels, x.ssm.channels());
                y = std::max<size_t>(y, x.ssm.inner());
                out = std::max<size_t>(out, x.ssm.inner());
                heads = std::max<size_t>(heads, 2 * x.ssm.heads);
            } else if (x.kind == MixerKind::Latent) {
                const LatentAttention& a = x.latent;
                proj = std::max<size_t>(proj, a.in.m);
                q = std::max<size_t>(q, a.heads * a.key_w());
                out = std::max<size_t>(out, a.out_w());
                lat = std::max<size_t>(lat, a.q_rank);
                uq = std::max<size_t>(uq, a.uq.m);
                part = std::max<size_t>(part, a.heads * a.dim);
                mid = std::max<size_t>(mid, a.heads * a.kv_rank);
                tiles = std::max<size_t>(tiles, a.heads * (n / SHIFT_TILE_MIN + 1));
            } else if (x.kind == MixerKind::Linear) {
                proj = std::max<size_t>(proj, x.linear.proj.m);
                halves = std::max<size_t>(halves, x.linear.proj.m);
                y = std::max<size_t>(y, x.linear.out_w());
                out = std::max<size_t>(out, x.linear.out_w());
            } else {
                shift = true;
                proj = std::max<size_t>(proj, 4 * x.tmix.inner());
                inner = std::max<size_t>(inner, x.tmix.inner());
                y = std::max<size_t>(y, x.tmix.inner());
                out = std::max<size_t>(out, x.tmix.inner());
                heads = std::max<size_t>(heads, x.tmix.heads);
                low = std::max<size_t>(low, x.tmix.w1.m);
                tiles = std::max<size_t>(tiles, 4 * (n / SHIFT_TILE_MIN + 1));
            }
        }
        if (l.mlp == MlpKind::Dense) ff = std::max<size_t>(ff, l.dense.down.k);
        if (l.mlp != MlpKind::Experts) continue;
        const ExpertLayer& e = l.experts;
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
    f(z.x0, (depth ? m.runs.size() + 1 : 1) * n * d);
    f(z.v_first, n * v_first);
    if (shift) f(z.xn_f, n * d);  // (rows are mixed in 32-bit)
    else w(z.xn_f, n * d);
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
    if (pairs) {
        f(z.moe_x, n * d);
        h(z.moe_xb, n16 * d);
        f(z.ids, n * top);
        f(z.weights, n * top);
        f(z.src, pairs);
        f(z.place, pairs);
        w(z.hid_f, hid);
        h(z.hid_b, hid + 256);
        f(z.rows, rows);
        w(z.sh_f, n * sff);
        h(z.sh_b, n16 * sff);
        f(z.shared, n * d);
        f(z.row_weight, pairs);
    }
    w(z.lat_f, n * lat);
    h(z.lat_b, n16 * lat);
    f(z.uq, n * uq);
    w(z.part_f, n * part);
    h(z.part_b, n16 * part);
    w(z.mid_f, n * mid);
    h(z.mid_b, n16 * mid);
    f(z.side, n * side);
    w(z.side_f, n * side_wide);
    h(z.side_b, n16 * side_wide);
    f(z.tiles, 3 * tiles);
    f(z.n_tiles, 1);
    w(z.ff_f, n * ff);
    h(z.ff_b, n16 * ff);
    f(z.branch, n * branch);
    f(z.conv, n * channels);
    h(z.conv_b, n * std::max(channels, halves));
    f(z.steps, n * heads);
    f(z.y, n * y);
    if (shift) {
        w(z.mix_f, 5 * n * d);
        h(z.mix_b, 5 * n * d + 16 * d);
        f(z.low, n * low);
        f(z.decay, n * inner);
    }
    // Angles in double, the table in fp32: positions up to the longest sequence and a verified tree past it.
    for (const Rotation& r : m.rotations) {
        const uint32_t npos = cfg.max_seq_len + FEED_W, half = r.dims / 2;
        std::vector<float> tab(size_t(npos) * half * 2);
        for (uint32_t i = 0; i < half; i++) {
            const double freq = std::pow(r.base, -2.0 * i / r.dims) / r.factor;
            for (uint32_t p = 0; p < npos; p++) {
                tab[(size_t(p) * half + i) * 2] = float(std::cos(p * freq));
                tab[(size_t(p) * half + i) * 2 + 1] = float(std::sin(p * freq));
            }
        }
        z.rope.emplace_back();
        z.rope.back().alloc(std::max<size_t>(tab.size() * 4, 16), false);
        z.rope.back().write_vec(0, tab);
    }
    // Per (layer run, mixer): its pages; a ring per slot of the rows a convolution or shift reaches back over, and room for a
    // verified run past them; a recurrence's state per slot and what a verified run leaves for it.
    uint32_t page_shift = 0;
    std::vector<bool> shared;  // per cache: its pages are another's, which are compacted and filled there
    while ((1u << page_shift) < md.page) page_shift++;
    const size_t es = f32 ? 4 : 2;
    std::vector<float> per_head;  // the layers' fixed decays and slopes, one after the other
    std::vector<size_t> from;     // where a layer's begin
    for (const FolderLayer& l : m.layers) {
        from.push_back(per_head.size());
        for (const Mixer& x : l.mix)
            for (const std::vector<float>* v : {&x.linear.decay, &x.attn.slopes}) per_head.insert(per_head.end(), v->begin(), v->end());
    }
    f(z.per_head, std::max<size_t>(per_head.size(), 1));
    if (!per_head.empty()) z.per_head.write_vec(0, per_head);
    size_t ring = 0, state = 0;
    for (int pass = 0; pass < 2; pass++) {  // sizes, then addresses
        float *rings = z.rings.as<float>(), *states = z.states.as<float>();
        ring = state = 0;
        uint32_t i = 0;
        auto take = [&](size_t floats) {
            float* p = states + state;
            state += (floats + 31) / 32 * 32;
            return p;
        };
        z.run.clear();
        z.first.clear();
        z.recurrent.clear();
        std::vector<uint32_t> last(m.layers.size());  // a layer's first cache in its latest run so far
        shared.clear();
        for (const LayerRun& r : m.runs) {
            z.first.push_back(i);
            last[r.layer] = i;
            const float* mine = z.per_head.as<float>() + from[r.layer];
            for (const Mixer& x : m.layers[r.layer].mix) {
                MixerCache c{};
                c.per_head = mine;
                mine += x.linear.decay.size() + x.attn.slopes.size();
                shared.push_back(x.kind == MixerKind::Latent && x.latent.kv_from != LatentAttention::OWN);
                if (x.kind == MixerKind::Attention) {
                    const Attention& a = x.attn;
                    c.kv = PagedKv{kv.k.as<uint8_t>() + kv.k_off[i] * es, kv.v.as<uint8_t>() + kv.v_off[i] * es, kv.page_table.as<uint32_t>(), kv.max_pages, page_shift, a.kv_heads, a.dim, a.vdim, kv.n_pages};
                    if (a.conv.w) { c.channels = a.conv.channels; c.ring_len = a.conv.taps - 1 + VERIFY_T; }
                } else if (x.kind == MixerKind::Latent) {
                    const LatentAttention& a = x.latent;
                    void* keys = kv.k.as<uint8_t>() + kv.k_off[i] * es;
                    c.kv = PagedKv{keys, keys, kv.page_table.as<uint32_t>(), kv.max_pages, page_shift, 1, a.key_w(), a.kv_rank, kv.n_pages};
                    if (shared.back()) c.kv = z.run[last[a.kv_from]].kv;
                } else {
                    const bool tm = x.kind == MixerKind::TimeMix, lin = x.kind == MixerKind::Linear;
                    if (!lin) {
                        c.channels = tm ? md.d : x.ssm.channels();
                        c.ring_len = (tm ? 2 : x.ssm.conv.taps) - 1 + VERIFY_T;
                    }
                    RecurrentCache rc{};
                    rc.heads = lin ? x.linear.heads : tm ? x.tmix.heads : x.ssm.heads;
                    rc.per = tm || lin ? 1 : x.ssm.heads / x.ssm.groups;
                    rc.N = lin ? x.linear.dim : tm ? x.tmix.dim : x.ssm.state;
                    rc.Np = recurrent_pitch(rc.N);
                    rc.P = lin ? x.linear.vdim : tm ? x.tmix.dim : x.ssm.vdim;
                    rc.channel_decay = tm;
                    if (lin) rc.fixed = c.per_head;
                    const size_t kept = size_t(cfg.max_seqs) * VERIFY_T;
                    rc.state = take(size_t(cfg.max_seqs) * rc.heads * rc.P * rc.Np);
                    rc.keep_k = take(kept * (rc.heads / rc.per) * rc.N);
                    rc.keep_d = take(kept * rc.heads * (tm ? rc.N : 2));
                    rc.keep_v = take(kept * rc.heads * rc.P);
                    c.recurrent = uint32_t(z.recurrent.size());
                    z.recurrent.push_back(rc);
                    z.max_heads = std::max(z.max_heads, rc.heads);
                }
                c.ring = rings + ring;
                ring += size_t(cfg.max_seqs) * c.ring_len * c.channels;
                z.run.push_back(c);
                i++;
            }
        }
        if (pass == 0) {
            f(z.rings, ring);
            f(z.states, state);
        }
    }
    z.caches.alloc(z.run.size() * sizeof(MixerCache), false);
    std::vector<MixerCache> listed = z.run;
    for (size_t j = 0; j < listed.size(); j++)
        if (shared[j]) listed[j].kv.n_kv = 0;
    z.caches.write_vec(0, listed);
    if (z.recurrent.empty()) return;
    z.recurrent_dev.alloc(z.recurrent.size() * sizeof(RecurrentCache), false);
    z.recurrent_dev.write_vec(0, z.recurrent);
}

void Engine::project(const Matrix& w, uint32_t n, const float* xf, const uint16_t* xb, float* y, uint16_t* yb, uint32_t epi, const float* base, uint32_t act_rows, const SideTable* side, float limit) {
    const bool gemm = !cfg.fp32 && w.m % 128 == 0 && w.k % 64 == 0, stream_takes = !cfg.fp32 && stream_fits(w, n);
    if (gemm && (gemm_fits(w, n) || !stream_takes)) {  // (few rows that are too long for the streamed kernel's shared memory, too)
        matmul_gemm(w, n, xb, y, yb, epi, base, nullptr, act_rows, nullptr, nullptr, nullptr, 1.0f, 1.0f, 1.0f, side, limit);
    } else if (stream_takes) {
        matmul(w, n, nullptr, y, epi, base, nullptr, act_rows, nullptr, xb, yb, 1.0f, 1.0f, 1.0f, side, limit);
    } else {
        LinearArgs a{};
        a.W = reinterpret_cast<const uint16_t*>(w.w);
        a.X = cfg.fp32 ? static_cast<const void*>(xf) : xb;
        a.base = base;
        a.Y = y;
        a.Yb = cfg.fp32 ? nullptr : yb;
        a.n = n;
        a.m = w.m;
        a.k = w.k;
        a.epi = epi;
        a.act_rows = act_rows;
        a.bias = w.bias;
        a.limit = limit;
        launch_linear(a, !cfg.fp32, stream);
    }
}

// A mixer's output: onto the stream (from `cur`, the residual added) or, as one of several, into a place of its own.
void Engine::mixer_out(const Matrix& o, uint32_t n, const float* cur, float* alone) {
    LayeredState& z = *lay;
    const int sp = span_begin(G_MATMUL);
    project(o, n, z.attn_f.as<float>(), z.attn_b.as<uint16_t>(), alone ? alone : z.result, nullptr, alone ? EPI_RAW : EPI_RESID, alone ? nullptr : cur);
    span_end(sp);
}

// What a convolution or shift over rows u needs to find the rows before them, and to leave its own.
ConvArgs Engine::conv_args(StepSet& st, const Plan& p, const MixerCache& mc, const float* u, uint32_t ldu, uint32_t taps) {
    ConvArgs c{};
    c.u = u;
    c.ldu = ldu;
    c.taps = taps;
    c.ring = mc.ring;
    c.ring_len = mc.ring_len;
    c.conv_channels = mc.channels;
    c.write_ring = mc.channels && p.max_run <= VERIFY_T;  // a step whose runs all fit a verified run leaves the rows as it goes
    c.meta = s.meta.as<uint32_t>();
    c.tin = st.in<uint32_t>(st.o_tin);
    c.vis = st.in<uint32_t>(st.o_vis);
    return c;
}

void Engine::encode_attention(StepSet& st, const Plan& p, const Attention& a, const MixerCache& mc, const float* cur, float* alone, bool capture) {
    LayeredState& z = *lay;
    const uint32_t n = p.n;
    const bool f32 = cfg.fp32;
    int sp = span_begin(G_MATMUL);
    project(a.proj, n, z.in_f, z.xn_b.as<uint16_t>(), z.proj.as<float>(), nullptr, EPI_RAW);
    span_end(sp);
    ConvArgs c = conv_args(st, p, mc, z.proj.as<float>(), a.proj.m, a.conv.w ? a.conv.taps : 1);
    c.w = a.conv.w;
    c.rope = a.rot.dims ? z.rope[a.rot.table].as<float>() : nullptr;
    c.kv = mc.kv;
    c.heads = a.heads;
    c.rot_dims = a.rot.dims;
    c.unit_qk = a.unit_qk;
    c.unit_v = a.unit_v;
    c.mix = a.mix;
    c.v_first = z.v_first.as<float>();
    c.neighbours = a.rot.neighbours;
    c.q_norm = a.q_norm;
    c.k_norm = a.k_norm;
    c.unit_eps = model.md.eps;
    c.temp = a.temp;
    const bool fast_attn = !f32 && !tuning.plain_attention && chunk_attn_fits(a.dim, a.vdim, model.md.page);
    if (fast_attn) c.q_b = z.q_b.as<uint16_t>();
    else c.q_f = z.q_f.as<float>();
    c.q_scale = a.scale * LOG2E;
    sp = span_begin(G_SMALL);
    launch_conv_qkv(c, n, f32, stream);
    if (mc.channels && !c.write_ring) launch_conv_state(c, st.in<RunIn>(st.o_runs), p.n_runs, stream);
    span_end(sp);
    ChunkedAttnArgs at{};
    at.q_f = z.q_f.as<float>();
    at.q_b = z.q_b.as<uint16_t>();
    at.ctiles = st.in<uint32_t>(st.o_ctiles);
    at.meta = c.meta;
    at.tin = c.tin;
    at.vis = c.vis;
    at.kv = mc.kv;
    at.gate = a.gated ? z.proj.as<float>() + a.qkv_w() : nullptr;
    at.ldg = a.proj.m;
    at.heads = a.heads;
    at.chunk = a.chunk;
    at.window = a.window;
    at.keep = a.keep;
    at.scale = a.scale;
    at.softcap = a.softcap;
    at.slopes = a.slopes.empty() ? nullptr : mc.per_head;
    at.out = f32 || capture ? z.attn_f.as<float>() : nullptr;
    at.out_b = z.attn_b.as<uint16_t>();
    uint32_t most = p.max_keys;  // keys a row may see
    for (uint32_t bound : {a.chunk, a.window})
        if (bound) most = std::min(most, bound + a.keep);
    sp = span_begin(G_ATTN);
    if (fast_attn) launch_attn_chunked(at, n, p.chunked ? p.ctiles : 0, most, sm_count, tuning.attn_keys_per_cta, stream);
    else launch_attn_any(at, n, f32, stream);
    span_end(sp);
    mixer_out(a.o, n, cur, alone);
}

// The recurrence itself and the norm and gate of its outputs, from the rows that the mixer has prepared.
void Engine::encode_recurrence(StepSet& st, const Plan& p, ScanArgs& a, GatedNormArgs& g) {
    LayeredState& z = *lay;
    a.runs = st.in<RunIn>(st.o_runs);
    a.gen = s.gen.as<GenState>();
    a.meta = s.meta.as<uint32_t>();
    a.vis = st.in<uint32_t>(st.o_vis);
    a.n_runs = p.n_runs;
    a.max_run = p.max_run;
    a.y = z.y.as<float>();
    g.y = a.y;
    g.width = a.c.heads * a.c.P;
    g.eps = model.md.eps;
    g.out_f32 = cfg.fp32 ? z.attn_f.as<float>() : nullptr;
    g.out_bf16 = z.attn_b.as<uint16_t>();
    int sp = span_begin(G_RECURRENCE);
    launch_scan(a, stream);
    span_end(sp);
    sp = span_begin(G_SMALL);
    launch_gated_norm(g, p.n, stream);
    span_end(sp);
}

void Engine::encode_state_space(StepSet& st, const Plan& p, const StateSpace& x, const MixerCache& mc, const float* cur, float* alone) {
    LayeredState& z = *lay;
    const uint32_t n = p.n, inner = x.inner(), ld = x.in.m;
    float* proj = z.proj.as<float>();
    int sp = span_begin(G_MATMUL);
    project(x.in, n, z.in_f, z.xn_b.as<uint16_t>(), proj, nullptr, EPI_RAW);
    span_end(sp);
    ConvArgs c = conv_args(st, p, mc, proj + inner, ld, x.conv.taps);
    c.w = x.conv.w;
    c.bias = x.conv.b;
    sp = span_begin(G_SMALL);
    // Long runs on the tensor cores take the convolution's outputs in bf16; the others' recurrence takes them as they are.
    const bool tensor = !cfg.fp32 && !tuning.plain_attention && ssd_fits(x.state, x.vdim) && p.max_run >= SSD_MIN_RUN;
    launch_conv_silu(c, StepSizeArgs{proj + inner + x.channels(), ld, x.heads, x.dt_bias, x.a_log, z.steps.as<float>()}, n, tensor && p.n_runs == 1 ? nullptr : z.conv.as<float>(),
                     tensor ? z.conv_b.as<uint16_t>() : nullptr, stream);
    if (!c.write_ring) launch_conv_state(c, st.in<RunIn>(st.o_runs), p.n_runs, stream);
    span_end(sp);
    ScanArgs a{};
    a.c = z.recurrent[mc.recurrent];
    a.v = z.conv.as<float>();
    a.k = a.v + inner;
    a.q = a.k + x.groups * x.state;
    a.ldq = a.ldk = a.ldv = x.channels();
    a.decay = z.steps.as<float>();
    a.skip = x.skip;
    if (tensor) {
        a.v_b = z.conv_b.as<uint16_t>();
        a.k_b = a.v_b + inner;
        a.q_b = a.k_b + x.groups * x.state;
        a.a_log = x.a_log;
    }
    GatedNormArgs g{};
    g.gate = proj;
    g.ldg = ld;
    g.w = x.norm;
    g.groups = x.norm_groups;
    g.gate_first = true;
    encode_recurrence(st, p, a, g);
    mixer_out(x.o, n, cur, alone);
}

void Engine::encode_time_mix(StepSet& st, const Plan& p, const TimeMix& x, const MixerCache& mc, const float* cur, float* alone) {
    LayeredState& z = *lay;
    const uint32_t n = p.n, d = model.md.d, K = x.inner();
    const bool f32 = cfg.fp32;
    // r, k, v and g are one grouped product over the four mixes they read.
    const bool fast = !f32 && grouped_fits(K, d);
    ShiftArgs sh{};
    sh.c = conv_args(st, p, mc, z.in_f, d, 2);
    for (int i = 0; i < 5; i++) sh.mu[i] = x.mu[i];
    sh.out_f32 = z.mix_f.as<float>();
    sh.out_bf16 = z.mix_b.as<uint16_t>();
    sh.tiles = z.tiles.as<uint32_t>();
    sh.n_tiles = z.n_tiles.as<uint32_t>();
    sh.tile = 64;
    if (fast)
        for (sh.tile = SHIFT_TILE_MIN; sh.tile < 128 && sh.tile < n;) sh.tile *= 2;
    int sp = span_begin(G_SMALL);
    launch_token_shift(sh, n, stream);
    if (!sh.c.write_ring) launch_conv_state(sh.c, st.in<RunIn>(st.o_runs), p.n_runs, stream);
    span_end(sp);
    sp = span_begin(G_MATMUL);
    LinearArgs l{};
    l.W = reinterpret_cast<const uint16_t*>(x.rkvg.w);
    const size_t one = size_t(n) * d;  // (the decay's mix lies first, at an address that does not depend on n)
    l.X = f32 ? static_cast<const void*>(sh.out_f32 + one) : sh.out_bf16 + one;
    l.Y = z.proj.as<float>();
    l.m = K;
    l.k = d;
    l.epi = EPI_RAW;
    l.tiles = sh.tiles;
    l.n_tiles = sh.n_tiles;
    l.max_tiles = 4 * ((n + sh.tile - 1) / sh.tile);
    if (fast) launch_grouped(l, 4, sh.tile, s.err_flag.as<uint32_t>(), stream);
    else launch_linear(l, !f32, stream);
    project(x.w1, n, sh.out_f32, sh.out_bf16, z.low.as<float>(), nullptr, EPI_RAW);
    span_end(sp);
    const size_t rows = size_t(n) * K;
    DecayArgs dc{};
    dc.hid = z.low.as<float>();
    dc.ldh = x.w1.m;
    dc.r = l.Y;
    dc.k = l.Y + rows;
    dc.w2 = x.w2;
    dc.w0 = x.w0;
    dc.u = x.bonus;
    dc.rank = x.rank;
    dc.heads = x.heads;
    dc.dim = x.dim;
    dc.decay = z.decay.as<float>();
    dc.bonus = z.steps.as<float>();
    sp = span_begin(G_SMALL);
    launch_decay(dc, n, stream);
    span_end(sp);
    ScanArgs a{};
    a.c = z.recurrent[mc.recurrent];
    a.q = dc.r;
    a.k = dc.k;
    a.v = l.Y + 2 * rows;
    a.ldq = a.ldk = a.ldv = K;
    a.decay = dc.decay;
    a.bonus = dc.bonus;
    GatedNormArgs g{};
    g.gate = l.Y + 3 * rows;
    g.ldg = K;
    g.w = x.norm;
    g.groups = x.heads;
    encode_recurrence(st, p, a, g);
    mixer_out(x.o, n, cur, alone);
}

// Latent attention: the per-head matrices on the queries' side and on the sums' side, so that all heads read the rows the cache holds.
void Engine::encode_latent(StepSet& st, const Plan& p, const LatentAttention& x, const MixerCache& mc, const float* cur, float* alone, bool capture) {
    LayeredState& z = *lay;
    const uint32_t n = p.n;
    const bool f32 = cfg.fp32, direct = x.q_rank == 0;  // direct: the queries are in the first projection
    float* proj = z.proj.as<float>();
    int sp = span_begin(G_MATMUL);
    project(x.in, n, z.in_f, z.xn_b.as<uint16_t>(), proj, nullptr, EPI_RAW);
    span_end(sp);
    LatentRowsArgs r{};
    r.u = proj;
    r.ldu = x.in.m;
    r.q_norm = x.q_norm;
    r.kv_norm = x.kv_norm;
    r.rope = z.rope[x.rot.table].as<float>();
    r.meta = s.meta.as<uint32_t>();
    r.tin = st.in<uint32_t>(st.o_tin);
    r.kv = mc.kv;
    r.q_f = f32 ? z.lat_f.as<float>() : nullptr;
    r.q_b = f32 ? nullptr : z.lat_b.as<uint16_t>();
    r.q_rank = x.q_rank;
    r.key_at = x.first_w();
    r.kv_rank = x.kv_rank;
    r.rot_dim = x.rot_dim;
    r.own = x.kv_from == LatentAttention::OWN;
    r.neighbours = x.rot.neighbours;
    r.eps = model.md.eps;
    if (!direct) {
        sp = span_begin(G_SMALL);
        launch_latent_rows(r, n, f32, stream);
        span_end(sp);
        sp = span_begin(G_MATMUL);
        project(x.uq, n, z.lat_f.as<float>(), z.lat_b.as<uint16_t>(), z.uq.as<float>(), nullptr, EPI_RAW);
        span_end(sp);
    }
    const bool fast_attn = !f32 && !tuning.plain_attention && latent_attn_fits(x.kv_rank, x.rot_dim, model.md.page);
    const bool fast_q = !f32 && grouped_fits(x.kv_rank, x.dim), fast_v = !f32 && grouped_fits(x.vdim, x.kv_rank);
    LatentQueryArgs q{};
    q.u = direct ? proj : z.uq.as<float>();
    q.ldu = direct ? x.in.m : x.uq.m;
    q.rope = r.rope;
    q.meta = r.meta;
    q.part_f = f32 ? z.part_f.as<float>() : nullptr;
    q.part_b = f32 ? nullptr : z.part_b.as<uint16_t>();
    q.q_f = fast_attn ? nullptr : z.q_f.as<float>();
    q.q_b = fast_attn ? z.q_b.as<uint16_t>() : nullptr;
    q.tiles = z.tiles.as<uint32_t>();
    q.n_tiles = z.n_tiles.as<uint32_t>();
    q.n = n;
    q.heads = x.heads;
    q.dim = x.dim;
    q.rot_dim = x.rot_dim;
    q.kv_rank = x.kv_rank;
    q.tile = 64;
    if (fast_q && fast_v)
        for (q.tile = SHIFT_TILE_MIN; q.tile < 128 && q.tile < n;) q.tile *= 2;
    else if (fast_q || fast_v)
        for (q.tile = SHIFT_TILE_MIN; q.tile < 64 && q.tile < n;) q.tile *= 2;  // (a tile of the CUDA cores has 64 rows at most)
    q.neighbours = x.rot.neighbours;
    q.factor = fast_attn ? x.scale * LOG2E : 1.0f;
    sp = span_begin(G_SMALL);
    if (direct) launch_latent_split(r, q, f32, stream);
    else launch_latent_query(q, stream);
    span_end(sp);
    LinearArgs l{};  // W_uk^T on a head's query: in front of the rotated part
    l.W = reinterpret_cast<const uint16_t*>(x.uk_t.w);
    l.X = f32 ? static_cast<const void*>(q.part_f) : q.part_b;
    l.Y = q.q_f;
    l.Yb = q.q_b;
    l.m = x.kv_rank;
    l.k = x.dim;
    l.epi = EPI_RAW;
    l.tiles = q.tiles;
    l.n_tiles = q.n_tiles;
    l.max_tiles = x.heads * ((n + q.tile - 1) / q.tile);
    l.by_head = n;
    l.heads = x.heads;
    l.ldy = x.key_w();
    sp = span_begin(G_MATMUL);
    if (fast_q) launch_grouped(l, x.heads, q.tile, s.err_flag.as<uint32_t>(), stream);
    else launch_linear(l, !f32, stream);
    span_end(sp);
    ChunkedAttnArgs at{};
    at.q_f = q.q_f;
    at.q_b = q.q_b;
    at.ctiles = st.in<uint32_t>(st.o_ctiles);
    at.meta = r.meta;
    at.tin = r.tin;
    at.vis = st.in<uint32_t>(st.o_vis);
    at.kv = mc.kv;
    at.heads = x.heads;
    at.window = x.window;
    at.sink = x.sink;
    at.scale = x.scale;
    at.out = f32 ? z.mid_f.as<float>() : nullptr;
    at.out_b = f32 ? nullptr : z.mid_b.as<uint16_t>();
    sp = span_begin(G_ATTN);
    const uint32_t most = x.window ? std::min(p.max_keys, x.window) : p.max_keys;  // keys a row may see
    if (fast_attn) launch_attn_latent(at, n, p.chunked ? p.ctiles : 0, most, sm_count, tuning.attn_keys_per_cta, s.err_flag.as<uint32_t>(), stream);
    else launch_attn_any(at, n, f32, stream);
    span_end(sp);
    l.W = reinterpret_cast<const uint16_t*>(x.uv.w);  // W_uv on a head's sum of c, and the gate
    l.X = f32 ? static_cast<const void*>(at.out) : at.out_b;
    l.Y = f32 || capture ? z.attn_f.as<float>() : nullptr;
    l.Yb = f32 ? nullptr : z.attn_b.as<uint16_t>();
    l.m = x.vdim;
    l.k = x.kv_rank;
    l.ldy = x.vdim;
    l.gate = proj + x.first_w() + x.kv_w();
    l.ldg = x.in.m;
    l.gate_w = x.gate_by_head ? 1 : x.vdim;
    sp = span_begin(G_MATMUL);
    if (fast_v) launch_grouped(l, x.heads, q.tile, s.err_flag.as<uint32_t>(), stream);
    else launch_linear(l, !f32, stream);
    span_end(sp);
    mixer_out(x.o, n, cur, alone);
}

void Engine::encode_linear(StepSet& st, const Plan& p, const LinearAttention& x, const MixerCache& mc, float* alone) {
    LayeredState& z = *lay;
    const uint32_t n = p.n, ld = x.proj.m;
    float* proj = z.proj.as<float>();
    // Long runs on the tensor cores take q, k and v in bf16; the others' recurrence takes them as they are.
    bool tensor = !cfg.fp32 && !tuning.plain_attention && ssd_fits(x.dim, x.vdim) && p.max_run >= SSD_MIN_RUN;
    for (float d : x.decay) tensor = tensor && d > 0 && d <= 1;  // (products of decays by sums of logarithms that are not positive)
    int sp = span_begin(G_MATMUL);
    project(x.proj, n, z.in_f, z.xn_b.as<uint16_t>(), proj, tensor ? z.conv_b.as<uint16_t>() : nullptr, EPI_SILU, nullptr, x.qkv_w());
    span_end(sp);
    ScanArgs a{};
    a.c = z.recurrent[mc.recurrent];
    a.q = proj;
    a.k = a.q + x.heads * x.dim;
    a.v = a.k + x.heads * x.dim;
    a.ldq = a.ldk = a.ldv = ld;
    if (tensor) {
        a.q_b = z.conv_b.as<uint16_t>();
        a.k_b = a.q_b + x.heads * x.dim;
        a.v_b = a.k_b + x.heads * x.dim;
    }
    GatedNormArgs g{};
    g.gate = proj + x.qkv_w();
    g.ldg = ld;
    g.w = x.norm.w;
    g.groups = 1;
    g.sigmoid = true;
    encode_recurrence(st, p, a, g);
    mixer_out(x.o, n, nullptr, alone);
}

// The stream h = x + the norm of what the sublayer has left in `branch`, and its bf16 rows for the next one.
void Engine::add_norm(const float* x, const RowNorm& norm, uint32_t n) {
    LayeredState& z = *lay;
    AddNormArgs a{};
    a.x = x;
    a.y = z.branch.as<float>();
    a.norm = norm;
    a.out = s.h.as<float>();
    a.out_b = cfg.fp32 ? nullptr : z.xn_b.as<uint16_t>();
    a.n = n;
    a.d = model.md.d;
    a.eps = model.md.eps;
    const int sp = span_begin(G_SMALL);
    launch_add_norm(a, stream);
    span_end(sp);
}

void Engine::encode_side(StepSet& st, const SideInput& x, uint32_t n) {
    LayeredState& z = *lay;
    SideGateArgs g{};
    g.side = SideTable{model.layered->side, st.in<uint32_t>(st.o_tokens), model.layered->side_w, x.first, x.dim, x.proj.k};
    g.out_f32 = cfg.fp32 ? z.side_f.as<float>() : nullptr;
    g.out_bf16 = cfg.fp32 ? nullptr : z.side_b.as<uint16_t>();
    const bool fused = !cfg.fp32 && x.gate.m >= x.proj.k && ((x.gate.m % 128 == 0 && x.gate.k % 64 == 0) || stream_fits(x.gate, n));  // (the kernels that have the gate as an epilogue)
    int sp = span_begin(G_MATMUL);
    if (fused) project(x.gate, n, nullptr, z.xn_b.as<uint16_t>(), nullptr, g.out_bf16, EPI_SIDE, nullptr, 0, &g.side);
    else project(x.gate, n, z.in_f, z.xn_b.as<uint16_t>(), z.side.as<float>(), nullptr, EPI_RAW);
    span_end(sp);
    if (!fused) {
        g.x = z.side.as<float>();
        g.ldx = x.gate.m;
        g.n = n;
        sp = span_begin(G_SMALL);
        launch_side_gate(g, stream);
        span_end(sp);
    }
    sp = span_begin(G_MATMUL);
    project(x.proj, n, g.out_f32, g.out_bf16, z.branch.as<float>(), nullptr, EPI_RAW);
    span_end(sp);
    add_norm(s.h.as<float>(), x.norm, n);
}

void Engine::encode_forward_layered(uint32_t set, const Plan& p, const std::function<void(const LayerCapture&)>* capture) {
    const LayeredModel& m = *model.layered;
    const ModelDesc& md = model.md;
    begin_step(set, p);  // upload; the embedding into x0
    LayeredState& z = *lay;
    StepSet& st = sets[set];
    const bool f32 = cfg.fp32;
    const uint32_t n = p.n, d = md.d;
    float* h = s.h.as<float>();
    const float* cur = z.x0.as<float>();  // the stream; h from the first layer on
    const size_t apart = size_t(cfg.max_step_tokens) * d;  // from one of the results an average takes to the next
    bool normed = false;  // the layer before has left norm1's rows
    auto host = [&](const float* dev, size_t count) {
        std::vector<float> v(count);
        VLT_CUDA(cudaMemcpyAsync(v.data(), dev, count * 4, cudaMemcpyDeviceToHost, stream));
        VLT_CUDA(cudaStreamSynchronize(stream));
        return v;
    };
    NormArgs na{};
    na.n = n;
    na.k = d;
    na.eps = md.eps;
    na.scale = 1.0f;
    na.out_f32 = z.xn_f.as<float>();
    na.out_bf16 = z.xn_b.as<uint16_t>();
    for (uint32_t ri = 0; ri < m.runs.size(); ri++) {
        const FolderLayer& l = m.layers[m.runs[ri].layer];
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
        uint32_t attn_width = 0;
        z.in_f = l.post_norm ? cur : z.xn_f.as<float>();
        z.result = l.depth ? z.x0.as<float>() + (ri + 1) * apart : h;
        if (!normed && !l.post_norm) {
            na.in = cur;
            na.add = m.runs[ri].add_embed ? z.x0.as<float>() : nullptr;
            na.sum = h;
            na.norm = l.norm1;
            sp = span_begin(G_SMALL);
            launch_norm_rows(na, stream);
            span_end(sp);
            if (na.add) cur = h;
            na.add = nullptr;
        }
        if (capture) resid_in = host(cur, size_t(n) * d);
        const bool several = l.mix.size() > 1, own = several || l.post_norm;  // own: a mixer's output goes to a place of its own
        for (uint32_t b = 0; b < l.mix.size(); b++) {
            const Mixer& x = l.mix[b];
            const MixerCache& mc = z.run[z.first[ri] + b];
            float* alone = own ? z.branch.as<float>() + size_t(b) * n * d : nullptr;
            switch (x.kind) {
            case MixerKind::Attention: encode_attention(st, p, x.attn, mc, cur, alone, capture != nullptr); break;
            case MixerKind::StateSpace: encode_state_space(st, p, x.ssm, mc, cur, alone); break;
            case MixerKind::TimeMix: encode_time_mix(st, p, x.tmix, mc, cur, alone); break;
            case MixerKind::Latent: encode_latent(st, p, x.latent, mc, cur, alone, capture != nullptr); break;
            case MixerKind::Linear: encode_linear(st, p, x.linear, mc, alone); break;
            }
            if (capture && (x.kind == MixerKind::Attention || x.kind == MixerKind::Latent)) {
                attn_width = x.kind == MixerKind::Latent ? x.latent.out_w() : x.attn.out_w();
                sdpa = host(z.attn_f.as<float>(), size_t(n) * attn_width);
            }
        }
        if (several) {
            MergeArgs mg{};
            mg.x = cur;
            mg.a = z.branch.as<float>();
            mg.b = mg.a + size_t(n) * d;
            mg.norm_a = l.mix[0].out;
            mg.norm_b = l.mix[1].out;
            if (l.mlp == MlpKind::Dense) mg.norm = l.norm2;
            mg.out = h;
            mg.next = na.out_f32;
            mg.next_b = na.out_bf16;
            mg.n = n;
            mg.d = d;
            mg.eps = md.eps;
            sp = span_begin(G_SMALL);
            launch_merge_rows(mg, stream);
            span_end(sp);
        }
        if (l.post_norm) add_norm(cur, l.norm1, n);
        float* res = z.result;
        cur = h;
        normed = false;
        if (l.post_norm) z.in_f = h;
        if (l.mlp == MlpKind::Experts) {
            const bool next_norm = !l.post_norm && ri + 1 < m.runs.size() && !m.runs[ri + 1].loop_in && !m.runs[ri + 1].add_embed;
            encode_experts(l, n, next_norm ? m.layers[m.runs[ri + 1].layer].norm1 : RowNorm{});
            normed = next_norm;
        } else if (l.mlp == MlpKind::Dense) {
            if (!several && !l.post_norm && !l.parallel) {
                na.in = res;
                na.norm = l.norm2;
                sp = span_begin(G_SMALL);
                launch_norm_rows(na, stream);
                span_end(sp);
            }
            sp = span_begin(G_MATMUL);
            project(l.dense.up, n, z.in_f, z.xn_b.as<uint16_t>(), f32 ? z.ff_f.as<float>() : nullptr, z.ff_b.as<uint16_t>(),
                    l.dense.hidden == Hidden::SiluGlu ? EPI_GLU : l.dense.hidden == Hidden::ClampedGlu ? EPI_GLU_CLAMP : EPI_RELU2, nullptr, 0, nullptr, l.dense.limit);
            project(l.dense.down, n, z.ff_f.as<float>(), z.ff_b.as<uint16_t>(), l.post_norm ? z.branch.as<float>() : res, nullptr, l.post_norm ? EPI_RAW : EPI_RESID,
                    l.post_norm ? nullptr : res);
            span_end(sp);
            if (l.post_norm) add_norm(h, l.norm2, n);
        }
        if (l.side.dim) encode_side(st, l.side, n);
        if (l.depth) {
            DepthArgs a{};
            a.x = z.x0.as<float>();
            a.stride = apart;
            a.share = l.depth;
            a.count = ri + 2;
            a.out = h;
            normed = ri + 1 < m.runs.size();
            if (normed) a.norm = m.layers[m.runs[ri + 1].layer].norm1;
            a.next = f32 ? na.out_f32 : nullptr;
            a.next_b = f32 ? nullptr : na.out_bf16;
            a.n = n;
            a.d = d;
            a.eps = md.eps;
            sp = span_begin(G_SMALL);
            launch_depth_average(a, stream);
            span_end(sp);
        }
        if (capture) {
            const std::vector<float> resid_out = host(h, size_t(n) * d);
            LayerCapture lc{ri, n, resid_in.data(), nullptr, nullptr, attn_width ? sdpa.data() : nullptr, nullptr, nullptr, nullptr};
            lc.resid_out = resid_out.data();
            lc.attn_width = attn_width;
            (*capture)(lc);
        }
        // (kernels.metal:133-148 `tap_rows`, as the other architectures' taps)
        auto tap = std::find(tap_layers.begin(), tap_layers.end(), ri);
        if (tap != tap_layers.end()) launch_prep_rows(h, nullptr, n, d, md.eps, tap_bufs[tap - tap_layers.begin()].as<float>(), nullptr, nullptr, true, true, stream);
    }
    // The tail: the final norm of the hidden and head rows, the head, sampling, accept, compaction.
    const int sp = span_begin(G_TAIL);
    na.in = h;
    na.norm = m.final_norm;
    na.rows = st.in<uint32_t>(st.o_hidden_rows);
    na.n = p.n_hidden;
    na.out_f32 = s.hfin_all.as<float>();
    na.out_bf16 = nullptr;
    launch_norm_rows(na, stream);
    if (p.n_head) {
        na.rows = st.in<uint32_t>(st.o_head_rows);
        na.n = p.n_head;
        na.scale = m.logit_scale;  // (the head is linear)
        na.out_f32 = s.hfin_head.as<float>();
        na.out_bf16 = f32 ? nullptr : s.hfin_b.as<uint16_t>();
        launch_norm_rows(na, stream);
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
                             uint32_t(z.run.size()), f32, stream);
    if (p.verified)
        launch_recurrent_commit(st.in<RunIn>(st.o_runs), s.path.as<uint32_t>(), s.path_len.as<uint32_t>(), s.lens.as<uint32_t>(), z.recurrent_dev.as<RecurrentCache>(), p.n_runs,
                                uint32_t(z.recurrent.size()), z.max_heads, stream);
    span_end(sp);
}

// h += the experts' weighted rows + the shared expert's, on norm2's rows of h; norm: the norm the next layer run begins
// with, whose rows are then left as well.
void Engine::encode_experts(const FolderLayer& l, uint32_t n, RowNorm norm) {
    LayeredState& z = *lay;
    const ExpertLayer& e = l.experts;
    const bool f32 = cfg.fp32;
    const uint32_t d = model.md.d, pairs = n * e.top;
    float* h = s.h.as<float>();
    RouterArgs r{};
    r.x = h;
    if (!l.post_norm) r.norm = l.norm2;
    r.router = e.router;
    r.sigmoid = e.sigmoid;
    r.renormalized = e.renormalized;
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
    so.weights = r.weights;
    so.row_weight = e.scales_input ? z.row_weight.as<float>() : nullptr;
    so.n = n;
    so.top = e.top;
    so.experts = e.experts;
    // The experts' matrices on the tensor cores where their sizes fit: tiles as long as an expert's rows on average, so that
    // its weights are read once. On the CUDA cores a tile has 64.
    const uint32_t hidden = hidden_rows(e.hidden, e.ff);
    const bool fast = !f32 && grouped_fits(hidden, d) && grouped_fits(d, e.ff);
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
    const float* in_f = l.post_norm ? z.in_f : z.moe_x.as<float>();  // what the experts read: the stream, or its normed rows
    const uint16_t* in_b = l.post_norm ? z.xn_b.as<uint16_t>() : z.moe_xb.as<uint16_t>();
    up.X = f32 ? static_cast<const void*>(in_f) : in_b;
    up.src = so.src;
    up.Y = z.hid_f.as<float>();
    up.Yb = z.hid_b.as<uint16_t>();
    up.m = hidden;
    up.k = d;
    up.epi = e.hidden == Hidden::ClampedGlu ? EPI_GLU_CLAMP : e.hidden == Hidden::SiluGlu ? EPI_GLU : EPI_RELU2;
    up.limit = e.limit;
    up.row_scale = so.row_weight;  // (the first products are linear: onto them instead of onto the rows)
    up.tiles = so.tiles;
    up.n_tiles = so.n_tiles;
    up.max_tiles = pairs / so.tile + std::min(e.experts, pairs);
    if (fast) launch_grouped(up, e.experts, so.tile, s.err_flag.as<uint32_t>(), stream);
    else launch_linear(up, !f32, stream);
    LinearArgs down = up;
    down.W = reinterpret_cast<const uint16_t*>(e.down.w);
    down.X = f32 ? static_cast<const void*>(z.hid_f.as<float>()) : z.hid_b.as<uint16_t>();
    down.src = nullptr;
    down.row_scale = nullptr;
    down.Y = z.rows.as<float>();
    down.Yb = nullptr;
    down.m = d;
    down.k = e.ff;
    down.epi = EPI_RAW;
    if (fast) launch_grouped(down, e.experts, so.tile, s.err_flag.as<uint32_t>(), stream);
    else launch_linear(down, !f32, stream);
    if (e.shared_ff) {
        project(e.shared_up, n, in_f, in_b, z.sh_f.as<float>(), z.sh_b.as<uint16_t>(), EPI_RELU2);
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
    c.weights = e.scales_input ? nullptr : r.weights;
    if (l.post_norm) c.post = l.norm2;
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
