// Layers of mixer-built decoders whose mixer and feed-forward read one normed row side by side (latent attention, minGRU), and
// the entry of a loop's pass.  A layer is: residual update + norm + token shift, one matmul for everything that reads the row
// (the mixer's projections read the shifted row, the feed-forward the plain one), the mixer, and one matmul over the mixer's
// and the feed-forward's columns together, whose result is the sum of both branches.  See mixer_lm.h.
#include "mixer_lm.h"
#include <algorithm>
#include <climits>
#include <cstring>

namespace mk {

namespace {

// Lanes with at least this many tokens in a tick have their keys and values expanded from the cached vectors; fewer tokens take
// their queries to the latent space instead.
constexpr int kWideFrom = 33;

int log2_of(int n) {
    int s = 0;
    while ((1 << s) < n) ++s;
    return s;
}

}  // namespace

// ---------------------------------------------------------------------------- load

void MixerLm::load_side_by_side(const SafetensorsFile& f, int l) {
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    Layer& w = lw_[(size_t)l];
    const int C = ms_.width;
    const std::string p = "l" + std::to_string(l) + ".", m = p + "mix.";
    upload_norm(f, p + "norm1", w.norm1);
    // inputs of the stacked projections: the shifted row, then the row itself (a shift of zero)
    std::vector<float> mu = f.values(p + "shift", {C});
    if (s.ff > 0) mu.resize(2 * (size_t)C, 0.f);
    upload_f32(mu, w.mu);

    std::vector<Part> parts;
    int at = 0;
    auto part = [&](const std::string& name, int rows) {
        const int here = at;
        parts.push_back({name, rows, here});
        at = pad_to(at + rows, 4);
        return here;
    };
    int mix = 0;  // columns the mixer hands to its output projection
    if (s.kind == MixerKind::Latent) {
        at = latent_qkv(m, s.latent, w, parts, at);
        mix = s.latent.heads * s.latent.vdim;
        load_latent(f, l);
    } else {
        w.c_q = part(m + "z", s.gru.width);
        w.c_v = part(m + "x", s.gru.width);
        w.c_g = part(m + "g", s.gru.width);
        upload_f32(f.values(m + "z.b", {s.gru.width}), w.z_b);
        upload_f32(f.values(m + "x.b", {s.gru.width}), w.x_b);
        mix = s.gru.width;
    }
    std::vector<Part> out = {{m + "o", C, 0, 1, 0, mix}};
    w.mix_cols = pad_to(mix, 64);
    if (s.ff > 0) {
        const int first = pad_to(at, 128);
        w.c_ff = first;
        parts.push_back({p + "mlp.up", s.ff, first});
        upload_dense(f, parts, first + pad_to(s.ff, 128), C, w.in, {first, pad_to(s.ff, 128)});
        out.push_back({p + "mlp.down", C, 0, 1, w.mix_cols, s.ff});
        upload_f32(f.values(p + "mlp.up.b", {s.ff}), w.up_b);
        upload_f32(f.values(p + "mlp.down.b", {C}), w.down_b);
        upload_f32(f.values(p + "mlp.act", {4}), w.poly);
    } else {
        upload_dense(f, parts, at, C, w.in);
    }
    upload_dense(f, out, C, w.mix_cols + s.ff, w.out);
}

// The projections of a latent-attention layer's input, from row `at` of the stacked matrix on; returns where they end.
int MixerLm::latent_qkv(const std::string& mix, const LatentSpec& s, Layer& w, std::vector<Part>& parts, int at) const {
    auto part = [&](const char* name, int rows) {
        const int here = at;
        parts.push_back({mix + name, rows, here});
        at = pad_to(at + rows, 4);
        return here;
    };
    w.c_q = part("dq", s.q_rank);
    w.c_kv = part("dkv", s.kv_rank + s.rot_dim);
    w.c_rot = w.c_kv + s.kv_rank;
    parts.back().turn_from = parts.back().turn_to = s.kv_rank;
    parts.back().turn_dims = s.rot.dims;
    if (s.gate != OutputGate::None) w.c_g = part("g", s.gate == OutputGate::Value ? s.heads * s.vdim : s.heads);
    return at;
}

int MixerLm::latent_geometry(int ctas, bool tc, bool wide, int window) {
    for (size_t i = 0; i < latent_geo_.size(); ++i)
        if (latent_geo_[i].ctas == ctas && latent_geo_[i].tc == tc && latent_geo_[i].wide == wide && latent_geo_[i].window == window) return (int)i;
    LatentGeometry g;
    g.ctas = ctas;
    g.tc = tc;
    g.wide = wide;
    g.window = window;
    if (wide) {
        for (g.lanes = 0; g.lanes < (int)wide_.size() && wide_[(size_t)g.lanes].window != window;) ++g.lanes;
        if (g.lanes == (int)wide_.size()) {
            wide_.emplace_back();
            wide_.back().window = window;
        }
    }
    latent_geo_.push_back(std::move(g));
    return (int)latent_geo_.size() - 1;
}

void MixerLm::load_latent(const SafetensorsFile& f, int l) {
    const LatentSpec& a = ms_.layers[(size_t)l].latent;
    Layer& w = lw_[(size_t)l];
    const std::string m = "l" + std::to_string(l) + ".mix.";
    const int H = a.heads;
    upload_f32(f.values(m + "dq.norm", {a.q_rank}), w.q_norm);
    upload_f32(f.values(m + "dkv.norm", {a.kv_rank}), w.k_norm);

    LatentColumns cols = !f32_ && cfg_.kv_f16 ? latent_tc_columns(a.kv_rank, a.rot_dim, cfg_.block_tokens) : LatentColumns{};
    const bool tc = cols.row > 0;
    if (!tc) cols = latent_general_columns(a.kv_rank, a.rot_dim);
    w.row_width = cols.row;
    w.value_width = cols.values;
    w.rot0 = cols.rot0;
    if (w.row_width > kLatentMaxRank) throw std::runtime_error("key/value latents above " + std::to_string(kLatentMaxRank) + " values are not supported");
    // a query head: its unrotated dimensions, then the rotated ones
    w.q_rot0 = a.rot_dim > 0 ? pad_to(a.dim, 8) : a.dim;
    const int q_dim = w.q_rot0 + a.rot_dim;
    w.q_width = f32_ ? 0 : attention_tc_prefill_width(H, H, q_dim, a.vdim, cfg_.block_tokens);
    const bool wide = w.q_width > 0;
    if (!wide) w.q_width = pad_to(q_dim, 64);
    w.geometry = latent_geometry(tc ? latent_tc_groups(H) : 1, tc, wide, a.window);
    if (a.rot_dim > 0) w.rope = rope_table(a.rot);
    if (a.sink) upload_f32(f.values(m + "sink", {H}), w.sink);
    if (wide && iota_.size() == 0) {
        std::vector<uint32_t> n((size_t)(pool_->max_blocks() + cfg_.max_batch_lanes));
        for (size_t i = 0; i < n.size(); ++i) n[i] = (uint32_t)i;
        iota_.upload(n.data(), n.size() * 4, stream_);
        MK_CUDA(cudaStreamSynchronize(stream_));
    }

    upload_dense(f, {{m + "uq", H * (a.dim + a.rot_dim), 0, 1, 0, 0, a.dim + a.rot_dim, w.q_width, a.dim, w.q_rot0, a.rot.dims}}, (int64_t)H * w.q_width, a.q_rank, w.uq);
    const int64_t uk_bytes = (int64_t)H * a.dim * a.kv_rank * esz_, uv_bytes = (int64_t)H * a.vdim * a.kv_rank * esz_;
    {
        // queries to the latent space: W_uk transposed, head by head; rotated parts pass as they are
        const int rows = pad_to(w.row_width, 128);
        const std::vector<float> v = f.values(m + "uk", {(int64_t)H * a.dim, a.kv_rank});
        std::vector<float> t((size_t)H * rows * w.q_width, 0.f);
#pragma omp parallel for
        for (int h = 0; h < H; ++h)
            for (int d = 0; d < a.dim; ++d)
                for (int j = 0; j < a.kv_rank; ++j) t[((size_t)h * rows + j) * w.q_width + d] = v[((size_t)h * a.dim + d) * a.kv_rank + j];
        for (int h = 0; h < H; ++h)
            for (int i = 0; i < a.rot_dim; ++i) t[((size_t)h * rows + w.rot0 + i) * w.q_width + w.q_rot0 + i] = 1.f;
        upload_matrix(t, (int64_t)H * rows, w.q_width, uk_bytes, w.uk, {}, H);
    }
    const Part values = {m + "uv", H * a.vdim, 0, 1, 0, a.kv_rank, a.vdim, pad_to(a.vdim, 128)};
    {
        const int64_t rows = (int64_t)H * values.pitch;
        std::vector<float> t((size_t)(rows * w.value_width), 0.f);
        place(f, values, a.kv_rank, w.value_width, t);
        upload_matrix(t, rows, w.value_width, uv_bytes, w.uv, {}, H);
    }
    if (wide) {
        const int64_t rows = (int64_t)2 * H * w.q_width;
        std::vector<float> t((size_t)(rows * w.row_width), 0.f);
        place(f, {m + "uk", H * a.dim, 0, 1, 0, a.kv_rank, a.dim, w.q_width}, a.kv_rank, w.row_width, t);
        for (int h = 0; h < H; ++h)  // the shared key part is every head's
            for (int i = 0; i < a.rot_dim; ++i) t[((size_t)h * w.q_width + w.q_rot0 + i) * w.row_width + w.rot0 + i] = 1.f;
        place(f, {m + "uv", H * a.vdim, H * w.q_width, 1, 0, a.kv_rank, a.vdim, w.q_width}, a.kv_rank, w.row_width, t);
        upload_matrix(t, rows, w.row_width, uk_bytes + uv_bytes, w.ukv, {}, 0, 0.0);
    }
}

// ---------------------------------------------------------------------------- a tick's work lists

void MixerLm::plan_latent(Tick& t, const std::vector<int32_t>& start, const std::vector<int32_t>& n_tokens, const std::vector<int32_t>& n_blocks, KvReservation& r) {
    for (LatentGeometry& g : latent_geo_) {
        plan_latent_attention(start.data(), n_tokens.data(), n_blocks.data(), t.B, g.ctas, g.wide ? kWideFrom : INT_MAX, g.tc, g.plan, g.window);
        g.off_entries = stage_bytes(t, g.plan.entries.data(), g.plan.entries.size() * 4);
        g.off_rows = stage_bytes(t, g.plan.rows.data(), g.plan.rows.size() * 4);
    }
    const int bt = cfg_.block_tokens, tile = attention_tc_tile_rows(1, 1);
    for (WideLanes& w : wide_) {
        const int window = w.window;
        w = WideLanes{};
        w.window = window;
        int packed = 0;
        for (int i = 0; i < t.B; packed += n_tokens[(size_t)i], ++i) {
            const int s0 = start[(size_t)i], n = n_tokens[(size_t)i], used = (s0 + n + bt - 1) / bt;
            const int first_key = attention_first_key(s0, window, 0), first = first_key / bt;
            w.hdr.push_back(LaneHeader{s0, n, (int32_t)w.blocks.size() - first, used});
            if (n < kWideFrom) continue;
            const std::vector<KvBlockId>& blocks = r.lane_blocks((size_t)i);
            for (int b = first; b < used; ++b) w.blocks.push_back((int32_t)blocks[(size_t)b].slot);
            for (int k = 0; k < n; ++k) {
                w.rows.push_back(packed + k);
                w.pairs += s0 + k + 1 - attention_first_key(s0 + k, window, 0);
            }
            for (int r0 = (n - 1) / tile * tile; r0 >= 0; r0 -= tile) {  // the longest walks first
                w.tiles.push_back(i);
                w.tiles.push_back(r0);
            }
            w.keys += s0 + n - first_key;
        }
        if (w.rows.empty()) continue;
        w.off_hdr = stage_bytes(t, w.hdr.data(), w.hdr.size() * sizeof(LaneHeader));
        w.off_tiles = stage_bytes(t, w.tiles.data(), w.tiles.size() * 4);
        w.off_rows = stage_bytes(t, w.rows.data(), w.rows.size() * 4);
        w.off_blocks = stage_bytes(t, w.blocks.data(), w.blocks.size() * 4);
    }
}

// ---------------------------------------------------------------------------- forward

void MixerLm::begin_pass(const Tick& t, int pass, Pending& pend) {
    const int C = ms_.width;
    const RowImage both = image(img_loop_, loop_in_.ld);
    RowUpdateArgs u;
    u.rows = t.T;
    apply_pending(u, pend, false);
    u.raw = both.part(0, loop_in_.ld / 2);
    prof_begin(KC_ROW_UPDATE, (double)t.T * C * (8.0 + 4.0 * u.n_add + esz_), 0);
    launch_row_update(u, stream_);
    prof_end();
    ++launches_;
    pend.n = 1;
    pend.y[0] = matmul(loop_in_, both, t.T, y_b_, 2);
    pend.bias = loop_step_.as<float>() + (size_t)pass * C;
    pend.replace = true;
}

void MixerLm::run_side_by_side(const Tick& t, int run, Pending& pend, const std::vector<LmLane>& lanes) {
    const int l = runs_[(size_t)run].layer;
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    Layer& w = lw_[(size_t)l];
    RunState& st = rs_[(size_t)run];
    const int T = t.T, C = ms_.width;
    RowUpdateArgs u;
    u.rows = T;
    apply_pending(u, pend, true);
    set_norm(u, w.norm1);
    u.n_mix = s.ff > 0 ? 2 : 1;
    u.mu = w.mu.as<float>();
    u.mixes = image(mixes_, w.in.ld);
    u.lanes = state_lanes_;
    u.token_lane = t.bd.token_lane;
    u.kept = st.kept.as<float>();
    prof_begin(KC_ROW_UPDATE, (double)T * C * (8.0 + 4.0 * u.n_add + (double)u.n_mix * esz_), 0);
    launch_row_update(u, stream_);
    prof_end();
    ++launches_;
    const Shares y = matmul(w.in, u.mixes, T, y_in_, 0);

    const RowImage both = image(img_cat_, w.out.ld);
    LatentPrepArgs p;
    p.y = y;
    p.rows = T;
    p.eps = ms_.eps;
    if (s.kind == MixerKind::Latent) {
        latent_prep_args(t, run, y, p);
    }
    if (s.ff > 0) {
        p.ff_col = w.c_ff;
        p.ff = s.ff;
        p.ff_bias = w.up_b.as<float>();
        p.poly = w.poly.as<float>();
        p.ff_image = both.part(w.mix_cols, w.out.ld - w.mix_cols);
    }
    if (p.q_rank > 0 || p.ff > 0) {
        prof_begin(KC_LATENT_PREP, (double)T * (p.q_rank + p.kv_rank + p.ff) * (4.0 + esz_), 0);
        launch_latent_prep(p, stream_);
        prof_end();
        ++launches_;
    }

    const RowImage mixed = both.part(0, w.mix_cols);
    if (s.kind == MixerKind::Latent) {
        run_latent(t, run, y, mixed, lanes);
    } else {
        MinGruArgs a;
        a.lanes = state_lanes_;
        a.width = s.gru.width;
        a.y = y;
        a.z_col = w.c_q;
        a.x_col = w.c_v;
        a.g_col = w.c_g;
        a.z_bias = w.z_b.as<float>();
        a.x_bias = w.x_b.as<float>();
        a.state = st.state.as<float>();
        a.image = mixed;
        a.longest = longest_;
        prof_begin(KC_MINGRU, (double)T * a.width * (12.0 + esz_) + 8.0 * t.B * a.width, 0);
        launch_mingru_scan(a, stream_);
        prof_end();
        ++launches_;
    }
    pend.n = 1;
    pend.y[0] = matmul(w.out, both, T, y_a_, 1);
    pend.bias = s.ff > 0 ? w.down_b.as<float>() : nullptr;
}

// Both latents' norms and the page write of a latent-attention layer.
void MixerLm::latent_prep_args(const Tick& t, int run, const Shares& y, LatentPrepArgs& p) {
    const int l = runs_[(size_t)run].layer;
    const LatentSpec& s = ms_.layers[(size_t)l].latent;
    Layer& w = lw_[(size_t)l];
    p.y = y;
    p.rows = t.T;
    p.eps = ms_.eps;
    p.q_col = w.c_q;
    p.q_rank = s.q_rank;
    p.q_norm = w.q_norm.as<float>();
    p.q_image = image(img_q_, w.uq.ld);
    p.kv_col = w.c_kv;
    p.kv_rank = s.kv_rank;
    p.kv_width = w.row_width;
    p.kv_norm = w.k_norm.as<float>();
    p.slots = t.bd.slots;
    p.pool = rs_[(size_t)run].k_pool.ptr();
    p.pool_f16 = cfg_.kv_f16 ? 1 : 0;
    if (s.rot_dim > 0) {
        p.rot_col = w.c_rot;
        p.rot0 = w.rot0;
        p.rot_width = s.rot_dim;
        p.rot_dims = s.rot.dims;
        p.cos_t = rope_[(size_t)w.rope]->cos_t.as<float>();
        p.sin_t = rope_[(size_t)w.rope]->sin_t.as<float>();
        p.positions = t.bd.positions;
    }
}

void MixerLm::run_latent(const Tick& t, int run, const Shares& y, const RowImage& out, const std::vector<LmLane>& lanes) {
    const int l = runs_[(size_t)run].layer, T = t.T;
    const LatentSpec& s = ms_.layers[(size_t)l].latent;
    Layer& w = lw_[(size_t)l];
    const LatentGeometry& g = latent_geo_[(size_t)w.geometry];
    const int H = s.heads, R = w.row_width, V = w.value_width, D = w.q_width, n = g.plan.n_rows();
    const int image_type = f32_ ? MatmulScatter::F32 : MatmulScatter::BF16;
    const RowImage q_latent = image(img_q_, w.uq.ld), per_head = image(img_uq_, D), latent_out = image(img_lat_, V);
    const int32_t* rows = n == T ? nullptr : reinterpret_cast<const int32_t*>(t.dp + g.off_rows);
    MatmulScatter to;
    if (n == T) {
        // every token of the tick stays in the latent space: the queries leave the matmul as the next one's per-head inputs
        to.out = img_uq_.ptr();
        to.type = image_type;
        to.part_rows = to.part_valid = D;
        to.ld_part = (int64_t)T * D;
        to.ld_row = D;
        matmul_scatter(w.uq, q_latent, T, to);
    } else {
        to.out = q_rot_.ptr();
        to.part_rows = to.part_valid = H * D;
        to.ld_row = (int64_t)H * D;
        matmul_scatter(w.uq, q_latent, T, to);
        if (n > 0) {
            prof_begin(KC_LATENT_ROWS, (double)n * H * D * 6.0, 0);
            launch_split_rows(q_rot_.as<float>(), H * D, rows, n, H, D, img_uq_.as<__nv_bfloat16>(), stream_);
            prof_end();
            ++launches_;
        }
    }
    if (n > 0) {
        to = MatmulScatter{};
        to.out = q_lat_.ptr();
        to.type = g.tc ? MatmulScatter::F16 : MatmulScatter::F32;
        to.part_rows = pad_to(R, 128);
        to.part_valid = R;
        to.ld_part = R;
        to.ld_row = (int64_t)H * R;
        matmul_scatter(w.uk, per_head, n, to);
        LatentAttnArgs a;
        if (g.tc) a.q_h = q_lat_.as<__half>();
        else a.q_f = q_lat_.as<float>();
        a.pool = rs_[(size_t)run].k_pool.ptr();
        a.pool_f16 = cfg_.kv_f16 ? 1 : 0;
        a.status = status_.as<int32_t>();
        a.tables = t.bd.tables;
        a.entries = reinterpret_cast<const int32_t*>(t.dp + g.off_entries);
        a.n_entries = g.plan.n_entries();
        a.n_rows = n;
        a.heads = H;
        a.rank = R;
        a.values = V;
        a.block_tokens = cfg_.block_tokens;
        a.scale = s.scale;
        a.window = s.window;
        a.sink = s.sink ? w.sink.as<float>() : nullptr;
        if (s.rot.dims > 0) {
            a.rot0 = w.rot0;
            a.rot_dims = s.rot.dims;
            a.cos_t = rope_[(size_t)w.rope]->cos_t.as<float>();
            a.sin_t = rope_[(size_t)w.rope]->sin_t.as<float>();
        }
        if (s.gate == OutputGate::Head) {
            a.gate = y;
            a.gate_col = w.c_g;
        }
        a.out = latent_out;
        a.part_o = lat_part_o_.as<float>();
        a.part_ml = lat_part_ml_.as<float>();
        a.counters = lat_counters_.as<int32_t>();
        double keys = 0, pairs = 0;
        for (const LmLane& ln : lanes) {
            if (g.wide && ln.n_tokens >= kWideFrom) continue;
            keys += (double)ln.start_pos + ln.n_tokens - attention_first_key(ln.start_pos, s.window, 0);
            for (int k = 0; k < ln.n_tokens; ++k) pairs += ln.start_pos + k + 1 - attention_first_key(ln.start_pos + k, s.window, 0);
        }
        prof_begin(KC_LATENT_ATTN, keys * (s.kv_rank + s.rot_dim) * (cfg_.kv_f16 ? 2.0 : 4.0) + (double)n * H * (2.0 * s.kv_rank + s.rot_dim) * (g.tc ? 2.0 : 0.5 * (4.0 + esz_)),
                   pairs * H * (4.0 * s.kv_rank + 2.0 * s.rot_dim));
        launch_latent_attention(a, stream_);
        prof_end();
        ++launches_;
        to = MatmulScatter{};
        to.out = f32_ ? (void*)out.f : (void*)out.h;
        to.type = image_type;
        to.part_rows = pad_to(s.vdim, 128);
        to.part_valid = s.vdim;
        to.ld_part = s.vdim;
        to.ld_row = out.ld;
        to.row_map = rows;
        if (s.gate == OutputGate::Value) {
            to.gate = y.p + w.c_g;
            to.gate_n = y.n;
            to.gate_ld = y.ld;
            to.gate_stride = y.stride;
        }
        matmul_scatter(w.uv, latent_out, n, to);
    }
    if (n < T) run_latent_wide(t, run, y, out);
}

void MixerLm::run_latent_wide(const Tick& t, int run, const Shares& y, const RowImage& out) {
    const int l = runs_[(size_t)run].layer;
    const LatentSpec& s = ms_.layers[(size_t)l].latent;
    Layer& w = lw_[(size_t)l];
    const int H = s.heads, R = w.row_width, D = w.q_width, bt = cfg_.block_tokens;
    const WideLanes& lanes = wide_[(size_t)latent_geo_[(size_t)w.geometry].lanes];
    const int blocks = (int)lanes.blocks.size(), keys = blocks * bt;
    wide_in_.ensure((size_t)keys * R * 2);
    wide_kv_.ensure((size_t)keys * 2 * H * D * 2);
    prof_begin(KC_LATENT_ROWS, (double)keys * R * (cfg_.kv_f16 ? 4.0 : 6.0), 0);
    launch_latent_gather(rs_[(size_t)run].k_pool.ptr(), cfg_.kv_f16 ? 1 : 0, reinterpret_cast<const int32_t*>(t.dp + lanes.off_blocks), blocks, bt, R,
                         wide_in_.as<__nv_bfloat16>(), stream_);
    prof_end();
    // pages [block][keys of every head, values of every head][bt][D]
    MatmulScatter to;
    to.out = wide_kv_.ptr();
    to.type = MatmulScatter::F16;
    to.part_rows = to.part_valid = D;
    to.ld_part = (int64_t)bt * D;
    to.ld_row = D;
    to.block_shift = log2_of(bt);
    to.ld_block = (int64_t)2 * H * bt * D;
    matmul_scatter(w.ukv, image(wide_in_, R), keys, to);
    AttnTcArgs a;
    a.q = q_rot_.as<float>();
    a.out = attn_.as<float>();
    a.k_pool = wide_kv_.ptr();
    a.v_pool = wide_kv_.as<__half>() + (size_t)H * bt * D;
    a.hdr = reinterpret_cast<const LaneHeader*>(t.dp + lanes.off_hdr);
    a.tables = iota_.as<uint32_t>();
    a.cu_seqlens = t.bd.cu_seqlens;
    a.tiles = reinterpret_cast<const int32_t*>(t.dp + lanes.off_tiles);
    a.n_tiles = (int)lanes.tiles.size() / 2;
    a.q_heads = a.kv_heads = H;
    a.d = D;
    a.block_tokens = bt;
    a.layers = 2;
    a.scale = s.scale;
    a.exact_weights = 1;
    a.window = s.window;
    a.sink = s.sink ? w.sink.as<float>() : nullptr;
    a.dv = s.vdim;
    if (s.rot.dims > 0) {
        a.rot_from = w.q_rot0;
        a.rot_dims = s.rot.dims;
        a.cos_t = rope_[(size_t)w.rope]->cos_t.as<float>();
        a.sin_t = rope_[(size_t)w.rope]->sin_t.as<float>();
    }
    prof_begin(KC_ATTN, lanes.keys * 2.0 * H * D * 2.0 + 8.0 * (double)lanes.rows.size() * H * D, 2.0 * lanes.pairs * H * (s.dim + s.rot_dim + s.vdim));
    launches_ += launch_paged_attention_tc(a, stream_);
    prof_end();
    prof_begin(KC_GATES, (double)lanes.rows.size() * H * s.vdim * (4.0 + (s.gate == OutputGate::Value ? 4.0 : 0.0) + esz_), 0);
    launch_head_gate(attn_.as<float>(), (int)lanes.rows.size(), H, D, s.vdim, y, w.c_g, out, stream_,
                     reinterpret_cast<const int32_t*>(t.dp + lanes.off_rows), s.gate);
    prof_end();
    launches_ += 2;
}

}  // namespace mk
