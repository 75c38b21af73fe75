// Layers of mixer-built decoders whose norms sit on what the sublayers give (mLSTM, attention, mixture of experts).  Mixer and
// feed-forward read the residual stream itself; norm, factor and bias of what they give are part of the next residual update.
// See mixer_lm.h.
#include "mixer_lm.h"

namespace mk {

// ---------------------------------------------------------------------------- load

void MixerLm::load_output_norm(const SafetensorsFile& f, int l) {
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    Layer& w = lw_[(size_t)l];
    const int C = ms_.width;
    const std::string p = "l" + std::to_string(l) + ".", m = p + "mix.";
    upload_norm(f, p + "norm1", w.norm1);
    std::vector<Part> parts;
    int at = 0;
    auto part = [&](const char* name, int rows) {
        const int here = at;
        parts.push_back({m + name, rows, here});
        at = pad_to(at + rows, 4);
        return here;
    };
    if (s.kind == MixerKind::Mlstm) {
        const MlstmSpec& x = s.mlstm;
        const int kw = x.heads * x.dim, vw = x.heads * x.vdim;
        w.c_q = part("q", kw);
        w.c_k = part("k", kw);
        w.c_v = part("v", vw);
        w.c_g = part("g", vw);
        w.c_i = part("i", x.heads);
        w.c_f = part("f", x.heads);
        upload_f32(f.values(m + "i.b", {x.heads}), w.i_b);
        upload_f32(f.values(m + "f.b", {x.heads}), w.f_b);
        upload_f32(f.values(m + "norm", {vw}), w.head_norm);
        linear_state_key_pad(x.dim);  // refuses head dimensions the recurrence does not take
        upload_dense(f, parts, at, C, w.in);
        upload_dense(f, {{m + "o", C, 0}}, C, vw, w.out);
    } else {
        const AttentionSpec& a = s.attn;
        const int qw = a.heads * a.dim, kw = a.kv_heads * a.dim, vw = a.kv_heads * a.vdim, ow = a.heads * a.vdim;
        w.c_q = part("q", qw);
        w.c_k = part("k", kw);
        w.c_v = part("v", vw);
        if (a.gate != OutputGate::None) w.c_g = part("g", a.gate == OutputGate::Value ? ow : a.heads);
        if (a.biases) {
            upload_f32(f.values(m + "q.b", {qw}), w.q_b);
            upload_f32(f.values(m + "k.b", {kw}), w.k_b);
            upload_f32(f.values(m + "v.b", {vw}), w.v_b);
            upload_f32(f.values(m + "o.b", {C}), w.o_b);
        }
        upload_f32(f.values(m + "q.norm", {a.qk_norm == QkNorm::Whole ? qw : a.dim}), w.q_norm);
        upload_f32(f.values(m + "k.norm", {a.qk_norm == QkNorm::Whole ? kw : a.dim}), w.k_norm);
        if (a.sink) upload_f32(f.values(m + "sink", {a.heads}), w.sink);
        w.geometry = geometry_of(a);
        w.row_width = geo_[(size_t)w.geometry].row_width;
        w.rope = rope_table(a.rot);
        upload_dense(f, parts, at, C, w.in);
        upload_dense(f, {{m + "o", C, 0}}, C, ow, w.out);
    }
    if (s.ff > 0) load_moe(f, l);
}

void MixerLm::load_moe(const SafetensorsFile& f, int l) {
    const MoeSpec& s = ms_.layers[(size_t)l].moe;
    Layer& w = lw_[(size_t)l];
    const int C = ms_.width;
    const std::string p = "l" + std::to_string(l) + ".", m = p + "mlp.";
    upload_norm(f, p + "norm2", w.norm2);
    std::vector<Part> router = {{m + "router", s.experts, 0}};
    if (s.shared_ff > 0) router.push_back({m + "shared.sg", 1, s.experts});
    upload_dense(f, router, pad_to(s.experts + 1, 4), C, w.router);
    // whole row tiles per expert, gate and up rows interleaved
    const int gu = pad_to(2 * s.ff, 128), down = pad_to(C, 128);
    std::vector<Part> gate_up, downs;
    for (int e = 0; e < s.experts; ++e) {
        const std::string x = m + "e" + std::to_string(e);
        gate_up.push_back({x + ".gate", s.ff, e * gu, 2});
        gate_up.push_back({x + ".up", s.ff, e * gu + 1, 2});
        downs.push_back({x + ".down", C, e * down});
    }
    const double share = (double)s.top / s.experts;
    upload_dense(f, gate_up, (int64_t)s.experts * gu, C, w.experts_gu, {}, share);
    upload_dense(f, downs, (int64_t)s.experts * down, s.ff, w.experts_down, {}, share);
    if (s.shared_ff > 0) {
        upload_dense(f, {{m + "shared.gate", s.shared_ff, 0, 2}, {m + "shared.up", s.shared_ff, 1, 2}}, 2 * (int64_t)s.shared_ff, C, w.gate_up);
        upload_dense(f, {{m + "shared.down", C, 0}}, C, s.shared_ff, w.down);
    }
}

// ---------------------------------------------------------------------------- forward

void MixerLm::run_output_norm(const Tick& t, int run, Pending& pend, const std::vector<LmLane>& lanes) {
    const int l = runs_[(size_t)run].layer;
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    Layer& w = lw_[(size_t)l];
    const int T = t.T, C = ms_.width;
    RowUpdateArgs u;
    u.rows = T;
    prof_begin(KC_ROW_UPDATE, (double)T * C * (8.0 + 4.0 * (pend.n + pend.routed_k) + esz_), 0);
    apply_pending(u, pend, false);
    u.raw = image(img_h_, w.in.ld);
    launch_row_update(u, stream_);
    prof_end();
    ++launches_;
    const Shares y = matmul(w.in, u.raw, T, y_in_, 0);
    RowImage mixed;
    if (s.kind == MixerKind::Mlstm) {
        mixed = image(img_b_, w.out.ld);
        run_mlstm(t, run, y, mixed);
    } else {
        mixed = image(img_a_, w.out.ld);
        attend(t, run, s.attn, y, lanes);
        const double gate = s.attn.gate == OutputGate::Value ? 4.0 : 0.0;
        prof_begin(KC_GATES, (double)T * s.attn.heads * s.attn.vdim * (4.0 + gate + esz_), 0);
        launch_head_gate(attn_.as<float>(), T, s.attn.heads, w.row_width, s.attn.vdim, y, w.c_g, mixed, stream_, nullptr, s.attn.gate);
        prof_end();
        ++launches_;
        if (s.attn.biases) pend.bias = w.o_b.as<float>();
    }
    pend.n = 1;
    pend.y[0] = matmul(w.out, mixed, T, y_a_, 1);
    pend.w[0] = w.norm1.w.as<float>();
    pend.coef = ms_.residual_mult;
    if (s.ff > 0) run_moe(t, l, pend);
}

void MixerLm::run_mlstm(const Tick& t, int run, const Shares& y, const RowImage& out) {
    const int l = runs_[(size_t)run].layer, T = t.T;
    const MlstmSpec& s = ms_.layers[(size_t)l].mlstm;
    Layer& w = lw_[(size_t)l];
    RunState& st = rs_[(size_t)run];
    MlstmScanArgs a;
    a.common.lanes = state_lanes_;
    a.common.state = st.state.as<float>();
    a.common.heads = s.heads;
    a.common.dim = s.dim;
    a.common.vdim = s.vdim;
    a.common.out = raw_.as<float>();
    a.common.normalised = 1;
    a.common.gate_sigmoid = 1;
    a.common.norm_w = w.head_norm.as<float>();
    a.common.norm_per_head = 1;
    a.common.eps = ms_.eps;
    a.common.gate = y;
    a.common.gate_col = w.c_g;
    a.y = y;
    a.q_col = w.c_q;
    a.k_col = w.c_k;
    a.v_col = w.c_v;
    a.i_col = w.c_i;
    a.f_col = w.c_f;
    a.i_bias = w.i_b.as<float>();
    a.f_bias = w.f_b.as<float>();
    a.cap = s.gate_cap;
    a.running_max = st.running_max.as<float>();
    const bool finish = short_lanes_ && linear_state_can_finish(s.dim, s.vdim);
    if (finish) a.common.image = out;
    const double vw = (double)s.heads * s.vdim, kw = (double)s.heads * s.dim;
    prof_begin(KC_MLSTM_SCAN, 4.0 * T * (2.0 * kw + vw) + T * vw * (finish ? 4.0 + esz_ : 4.0) + 8.0 * t.B * (vw + s.heads) * s.dim, 6.0 * T * vw * s.dim);
    launch_mlstm_scan(a, stream_);
    prof_end();
    ++launches_;
    if (!finish) {
        a.common.image = out;
        prof_begin(KC_GATES, T * vw * (8.0 + esz_), 0);
        launch_head_norm_gate(a.common, T, stream_);
        prof_end();
        ++launches_;
    }
}

void MixerLm::run_moe(const Tick& t, int layer, Pending& pend) {
    const MoeSpec& s = ms_.layers[(size_t)layer].moe;
    Layer& w = lw_[(size_t)layer];
    const int T = t.T, C = ms_.width, P = T * s.top;
    RowUpdateArgs u;
    u.rows = T;
    prof_begin(KC_ROW_UPDATE, (double)T * C * (8.0 + 4.0 * pend.n + esz_), 0);
    apply_pending(u, pend, false);
    u.raw = image(img_h_, w.router.ld);
    launch_row_update(u, stream_);
    prof_end();
    ++launches_;
    const Shares z = matmul(w.router, u.raw, T, y_in_, 0);
    MoeRows rows = moe_;
    if (s.shared_ff == 0) rows.shared_gate = nullptr;
    prof_begin(KC_MOE_ROWS, (double)T * s.experts * 4.0 + 2.0 * P * C * (double)esz_, 0);
    launches_ += launch_moe_rows(z, T, s.experts, s.top, rows, status_.as<int32_t>(), stream_);
    launch_moe_gather(f32_ ? (const void*)u.raw.f : (const void*)u.raw.h, T, s.top, (int64_t)w.router.ld * esz_, rows, img_rows_.ptr(), stream_);
    prof_end();
    ++launches_;

    // experts: a token's weight multiplies what goes in, so the gate and up sums of a grouped row
    const RowImage in = image(img_rows_, w.experts_gu.ld), act = image(img_expert_ff_, w.experts_down.ld);
    GatedAct ga;
    ga.kind = GatedAct::Clamped;
    ga.limit = s.limit;
    ga.pre = rows.weight_of_pos;
    const int gu_rows = pad_to(2 * s.ff, 128), down_rows = pad_to(C, 128);
    const double met = std::min<double>(s.experts, P);  // experts with rows, at most
    const double gu_bytes = (double)w.experts_gu.bytes / s.experts * met, down_bytes = (double)w.experts_down.bytes / s.experts * met;
    if (f32_) {
        prof_begin(KC_MOE_GEMM, gu_bytes + down_bytes + 4.0 * P * (2.0 * C + 5.0 * s.ff), 6.0 * P * (double)C * s.ff);
        launch_f32_matmul_experts(w.experts_gu.f32.as<float>(), s.experts, rows.offsets, gu_rows, gu_rows, w.experts_gu.ld, in.f, P, y_gu_.as<float>(), gu_rows, stream_);
        Shares gu;
        gu.p = y_gu_.as<float>();
        gu.ld = gu_rows;
        launch_gated_act(gu, P, s.ff, act, stream_, ga);
        launch_f32_matmul_experts(w.experts_down.f32.as<float>(), s.experts, rows.offsets, C, down_rows, w.experts_down.ld, act.f, P, routed_.as<float>(), C, stream_);
        prof_end();
        launches_ += 3;
    } else {
        HgemmScratch ws;
        ws.status = status_.as<int32_t>();
        ExpertRows er;
        er.experts = s.experts;
        er.offsets = rows.offsets;
        er.rows = er.rows_padded = gu_rows;
        prof_begin(KC_MOE_GEMM, gu_bytes + 2.0 * P * (C + s.ff), 4.0 * P * (double)C * s.ff);
        launch_hgemm_tc_experts(w.experts_gu.half, er, reinterpret_cast<const __half*>(in.h), P, nullptr, 0, &ga, reinterpret_cast<__half*>(act.h), act.ld, ws, stream_);
        prof_end();
        er.rows = C;
        er.rows_padded = down_rows;
        prof_begin(KC_MOE_GEMM, down_bytes + P * (2.0 * s.ff + 4.0 * C), 2.0 * P * (double)C * s.ff);
        launch_hgemm_tc_experts(w.experts_down.half, er, reinterpret_cast<const __half*>(act.h), P, routed_.as<float>(), C, nullptr, nullptr, 0, ws, stream_);
        prof_end();
        launches_ += 2;
    }
    pend.n = 1;
    pend.routed_at = rows.pos_of_pair;
    pend.routed_k = s.top;
    pend.w[0] = w.norm2.w.as<float>();
    pend.coef = ms_.residual_mult;
    if (s.shared_ff == 0) return;

    // the expert every token runs, times its gate
    const RowImage img = image(img_ff_, w.down.ld);
    ga.limit = s.shared_limit;
    ga.pre = nullptr;
    ga.post = rows.shared_gate;
    if (f32_) {
        const Shares gu = matmul(w.gate_up, u.raw, T, y_gu_, 0);
        prof_begin(KC_GATES, 12.0 * T * s.shared_ff, 0);
        launch_gated_act(gu, T, s.shared_ff, img, stream_, ga);
        prof_end();
    } else {
        prof_begin(T <= 64 ? KC_GEMM_NARROW : KC_GEMM, (double)w.gate_up.bytes + 2.0 * T * (C + s.shared_ff), 4.0 * T * (double)s.shared_ff * C);
        HgemmScratch ws;
        ws.status = status_.as<int32_t>();
        launch_hgemm_tc_gated(w.gate_up.half, reinterpret_cast<const __half*>(u.raw.h), T, ga, reinterpret_cast<__half*>(img.h), img.ld, ws, stream_);
        prof_end();
    }
    ++launches_;
    pend.y[0] = matmul(w.down, img, T, y_b_, 2);
}

}  // namespace mk
