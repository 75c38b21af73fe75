// Layers of mixer-built decoders whose mixer reads its normed input plus a short causal convolution of it: windowed attention with
// shared keys and values beside the delta rule with channel gates, and windowed latent attention with a rotated part.  Both branches
// of the former share one output matmul over their columns, to which each comes times its constant.  See mixer_lm.h.
#include "mixer_lm.h"
#include <algorithm>

namespace mk {

namespace {

// Lanes with at least this many tokens in a tick run the delta rule in chunks of rows.
constexpr int kChunkFrom = 48;

}  // namespace

// ---------------------------------------------------------------------------- load

void MixerLm::load_conv_input(const SafetensorsFile& f, int l) {
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    Layer& w = lw_[(size_t)l];
    const int C = ms_.width, taps = ms_.conv_taps;
    const std::string p = "l" + std::to_string(l) + ".", m = p + "mix.";
    upload_norm(f, p + "norm1", w.norm1);
    const std::vector<float> conv = f.values(p + "canon1", {C, taps});
    std::vector<float> by_tap(conv.size());
    for (int c = 0; c < C; ++c)
        for (int j = 0; j < taps; ++j) by_tap[(size_t)j * C + c] = conv[(size_t)c * taps + j];
    upload_f32(by_tap, w.input_conv);

    std::vector<Part> parts;
    int at = 0;
    if (s.kind == MixerKind::Latent) {
        at = latent_qkv(m, s.latent, w, parts, at);
        load_latent(f, l);
        upload_dense(f, parts, at, C, w.in);
        w.mix_cols = s.latent.heads * s.latent.vdim;
        upload_dense(f, {{m + "o", C, 0}}, C, w.mix_cols, w.out);
    } else {
        const AttentionSpec& a = s.attn;
        const ChannelDeltaSpec& d = s.channel_delta;
        const std::string L = m + "left.", R = m + "right.";
        const int qw = a.heads * a.dim, kw = a.kv_heads * a.dim, n = d.heads * d.dim;
        auto part = [&](const std::string& name, int rows) {
            const int here = at;
            parts.push_back({name, rows, here});
            at = pad_to(at + rows, 4);
            return here;
        };
        w.c_q = part(L + "q", qw);
        w.c_k = part(L + "k", kw);
        w.d_q = part(R + "r", n);
        w.d_k = part(R + "k", n);
        w.d_v = part(R + "v", n);
        w.d_a = part(R + "a", n);
        w.d_g = part(R + "g", n);
        w.c_low = part(R + "w1", d.rank);
        upload_dense(f, parts, at, C, w.in);
        upload_f32(f.values(L + "q.b", {qw}), w.q_b);
        upload_f32(f.values(L + "k.b", {kw}), w.k_b);
        w.geometry = geometry_of(a);
        w.row_width = geo_[(size_t)w.geometry].row_width;
        w.rope = rope_table(a.rot);
        linear_state_key_pad(d.dim);  // refuses head dimensions the recurrence does not take
        upload_low_rank(f, R, n, d.rank, w);
        if (!f32_) {
            const std::vector<uint16_t> w2 = f.bf16_values(R + "w2", {n, d.rank});
            std::vector<uint16_t> t(w2.size());
            for (int c = 0; c < n; ++c)
                for (int j = 0; j < d.rank; ++j) t[(size_t)j * n + c] = w2[(size_t)c * d.rank + j];
            w.w2h.upload(t.data(), t.size() * 2, stream_);
            MK_CUDA(cudaStreamSynchronize(stream_));
        }
        upload_f32(f.values(R + "a.b", {n}), w.a_b);
        upload_f32(f.values(R + "norm", {n}), w.head_norm);
        w.mix_cols = pad_to(a.heads * a.vdim, 64);
        upload_dense(f, {{L + "o", C, 0, 1, 0, a.heads * a.vdim}, {R + "o", C, 0, 1, w.mix_cols, n}}, C, w.mix_cols + n, w.out);
    }
    if (s.ff > 0) {
        upload_norm(f, p + "norm2", w.norm2);
        upload_dense(f, {{p + "mlp.gate", s.ff, 0, 2}, {p + "mlp.up", s.ff, 1, 2}}, 2 * (int64_t)s.ff, C, w.gate_up);
        upload_dense(f, {{p + "mlp.down", C, 0}}, C, s.ff, w.down);
    }
}

// ---------------------------------------------------------------------------- forward

void MixerLm::run_conv_input(const Tick& t, int run, Pending& pend, const std::vector<LmLane>& lanes) {
    const int l = runs_[(size_t)run].layer;
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    Layer& w = lw_[(size_t)l];
    RunState& st = rs_[(size_t)run];
    const int T = t.T, C = ms_.width;
    RowUpdateArgs u;
    u.rows = T;
    apply_pending(u, pend, true);
    set_norm(u, w.norm1);
    u.normed = image(img_h_, w.in.ld);
    u.taps = ms_.conv_taps;
    u.conv = w.input_conv.as<float>();
    u.lanes = state_lanes_;
    u.token_lane = t.bd.token_lane;
    u.kept = st.kept.as<float>();
    prof_begin(KC_ROW_UPDATE, (double)T * C * (8.0 + 4.0 * u.n_add + esz_), 0);
    launch_row_update(u, stream_);
    prof_end();
    ++launches_;
    const Shares y = matmul(w.in, u.normed, T, y_in_, 0);
    const RowImage both = image(img_cat_, w.out.ld);
    if (s.kind == MixerKind::Latent) {
        LatentPrepArgs p;
        latent_prep_args(t, run, y, p);
        prof_begin(KC_LATENT_PREP, (double)T * (p.q_rank + p.kv_rank + p.rot_width) * (4.0 + esz_), 0);
        launch_latent_prep(p, stream_);
        prof_end();
        ++launches_;
        run_latent(t, run, y, both, lanes);
    } else {
        attend(t, run, s.attn, y, lanes);
        prof_begin(KC_GATES, (double)T * s.attn.heads * s.attn.vdim * (4.0 + esz_), 0);
        launch_head_gate(attn_.as<float>(), T, s.attn.heads, w.row_width, s.attn.vdim, Shares{}, 0, both.part(0, w.mix_cols), stream_, nullptr, s.attn.gate, s.left_scale);
        prof_end();
        ++launches_;
        run_channel_delta(t, run, y, both.part(w.mix_cols, w.out.ld - w.mix_cols));
    }
    pend.n = 1;
    pend.y[0] = matmul(w.out, both, T, y_a_, 1);
}

void MixerLm::run_channel_delta(const Tick& t, int run, const Shares& y, const RowImage& out) {
    const int l = runs_[(size_t)run].layer, T = t.T;
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    const ChannelDeltaSpec& d = s.channel_delta;
    Layer& w = lw_[(size_t)l];
    const double n = (double)d.heads * d.dim;
    ChannelDeltaArgs a;
    a.common.state = rs_[(size_t)run].state.as<float>();
    a.common.heads = d.heads;
    a.common.dim = a.common.vdim = d.dim;
    a.common.out = raw_.as<float>();
    a.common.gate_sigmoid = 1;
    a.common.out_scale = s.right_scale;
    a.common.norm_w = w.head_norm.as<float>();
    a.common.norm_per_head = 1;
    a.common.eps = ms_.eps;
    a.common.gate = y;
    a.common.gate_col = w.d_g;
    a.y = y;
    a.r_col = w.d_q;
    a.k_col = w.d_k;
    a.v_col = w.d_v;
    a.a_col = w.d_a;
    a.low_col = w.c_low;
    a.rank = d.rank;
    a.w2t = w.w2t.as<float>();
    a.w2h = w.w2h.as<__nv_bfloat16>();
    a.w0 = w.w0.as<float>();
    a.a_bias = w.a_b.as<float>();
    // Sets of lanes whose form this head size does not have go row by row.
    const bool step = channel_delta_can_step(d.dim, d.rank), chunk = !f32_ && channel_delta_can_chunk(d.dim);
    std::vector<const LaneSet*> by_row;
    if (delta_rows_.rows > 0) by_row.push_back(&delta_rows_);
    if (delta_one_.rows > 0 && !step) by_row.push_back(&delta_one_);
    if (delta_chunks_.rows > 0 && !chunk) by_row.push_back(&delta_chunks_);
    const bool chunks_run = chunk && delta_chunks_.rows > 0;
    auto state_io = [&](const LaneSet& l) { return 8.0 * l.lanes.lanes * n * d.dim; };
    bool unfinished = chunks_run;
    for (const LaneSet* l : by_row) unfinished |= l->longest > kShortLane || !linear_state_can_finish(d.dim, d.dim);
    for (const LaneSet* l : by_row) {
        ChannelGatesArgs g;
        g.y = y;
        g.k_col = w.d_k;
        g.a_col = w.d_a;
        g.low_col = w.c_low;
        g.lanes = a.common.lanes = l->lanes;
        g.longest = l->longest;
        g.heads = d.heads;
        g.dim = d.dim;
        g.rank = d.rank;
        g.w2t = a.w2t;
        g.w0 = a.w0;
        g.a_bias = a.a_bias;
        a.decay = g.decay = decay_.as<float>();
        a.removal = g.removal = removal_.as<float>();
        prof_begin(KC_CHANNEL_GATES, l->rows * (4.0 * n + d.rank) * 4.0 + n * d.rank * 4.0, 2.0 * l->rows * n * d.rank);
        launch_channel_gates(g, stream_);
        prof_end();
        a.common.image = unfinished ? RowImage{} : out;
        prof_begin(KC_DELTA_SCAN, 4.0 * l->rows * 6.0 * n + state_io(*l), 10.0 * l->rows * n * d.dim);
        launch_channel_delta_scan(a, stream_);
        prof_end();
        launches_ += 2;
    }
    if (chunks_run) {
        a.common.lanes = delta_chunks_.lanes;
        a.common.image = RowImage{};
        prof_begin(KC_DELTA_SCAN, 4.0 * delta_chunks_.rows * (5.0 * n + d.rank) + n * d.rank * 2.0 + state_io(delta_chunks_), delta_chunks_.rows * n * (10.0 * d.dim + 2.0 * d.rank));
        launch_channel_delta_chunks(a, delta_chunks_.longest, delta_scratch_.ptr(), stream_);
        prof_end();
        launches_ += 2;
    }
    if (unfinished) {  // all rows of the tick; the one-token lanes' are written over
        a.common.image = out;
        prof_begin(KC_GATES, T * n * (8.0 + esz_), 0);
        launch_head_norm_gate(a.common, T, stream_);
        prof_end();
        ++launches_;
    }
    if (delta_one_.rows > 0 && step) {
        a.common.lanes = delta_one_.lanes;
        a.common.image = out;
        prof_begin(KC_DELTA_SCAN, delta_one_.rows * n * (20.0 + esz_) + n * d.rank * (f32_ ? 4.0 : 2.0) + state_io(delta_one_), delta_one_.rows * n * (10.0 * d.dim + 2.0 * d.rank));
        launch_channel_delta_step(a, stream_);
        prof_end();
        ++launches_;
    }
}

// One-token lanes, lanes of a few tokens and prompts take different forms of the delta rule with channel gates.
void MixerLm::split_delta_lanes(Tick& t, const std::vector<StateLane>& lanes) {
    LaneSet* sets[] = {&delta_one_, &delta_rows_, &delta_chunks_};
    std::vector<StateLane> of[3];
    for (const StateLane& l : lanes) of[l.n <= 1 ? 0 : (l.n < kChunkFrom ? 1 : 2)].push_back(l);
    for (int i = 0; i < 3; ++i) {
        LaneSet& s = *sets[i];
        s = LaneSet{};
        s.lanes.lanes = (int)of[i].size();
        for (const StateLane& l : of[i]) {
            s.longest = std::max(s.longest, (int)l.n);
            s.rows += l.n;
        }
        s.off = stage_bytes(t, of[i].data(), of[i].size() * sizeof(StateLane));
    }
}

}  // namespace mk
