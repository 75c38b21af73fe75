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
        at = pad_to(at + rows, 8);
        return here;
    };
    if (s.kind == MixerKind::Mlstm) {
        const MlstmSpec& x = s.mlstm;
        const int kw = x.heads * x.dim, vw = x.heads * x.vdim;
        w.c_q = part("q", kw);
        w.c_k = part("k", kw);
        w.c_v = part("v", vw);
        at = pad_to(at, 128);  // what stays in f32 on prompts begins here
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
        }
        if (a.out_bias) upload_f32(f.values(m + "o.b", {C}), w.o_b);
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
        upload_dense(f, {{m + "shared.gate", s.shared_ff, 0, 2}, {m + "shared.up", s.shared_ff, 1, 2}}, pad_to(2 * s.shared_ff, 128), C, w.gate_up);
        upload_dense(f, {{m + "shared.down", C, 0}}, down, s.shared_ff, w.down);
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
    RowImage mixed;
    if (s.kind == MixerKind::Mlstm) {
        mixed = image(img_b_, w.out.ld);
        run_mlstm(t, run, u.raw, mixed);
    } else {
        const Shares y = matmul(w.in, u.raw, T, y_in_, 0);
        mixed = image(img_a_, w.out.ld);
        attend(t, run, s.attn, y, lanes);
        const double gate = s.attn.gate == OutputGate::Value ? 4.0 : 0.0;
        prof_begin(KC_GATES, (double)T * s.attn.heads * s.attn.vdim * (4.0 + gate + esz_), 0);
        launch_head_gate(attn_.as<float>(), T, s.attn.heads, w.row_width, s.attn.vdim, y, w.c_g, mixed, stream_, nullptr, s.attn.gate);
        prof_end();
        ++launches_;
        if (s.attn.out_bias) pend.bias = w.o_b.as<float>();
    }
    pend.n = 1;
    pend.y[0] = matmul(w.out, mixed, T, y_a_, 1);
    pend.w[0] = w.norm1.w.as<float>();
    pend.coef = ms_.residual_mult;
    if (s.ff > 0) run_moe(t, l, pend);
}

void MixerLm::run_mlstm(const Tick& t, int run, const RowImage& in, const RowImage& out) {
    const int l = runs_[(size_t)run].layer, T = t.T;
    const MlstmSpec& s = ms_.layers[(size_t)l].mlstm;
    Layer& w = lw_[(size_t)l];
    RunState& st = rs_[(size_t)run];
    MlstmScanArgs a;
    const bool chunked = !f32_ && longest_ > 1;
    Shares y;
    int from = 0;  // the first projection column that `y` holds
    if (chunked) {
        // queries, keys and values leave the matmul as bfloat16, the gates as f32
        from = w.c_g;
        MatmulScatter to;
        to.out = img_qkv_.ptr();
        to.type = MatmulScatter::BF16;
        to.part_rows = to.part_valid = from;
        to.ld_row = from;
        to.rest = y_in_.as<float>();
        to.rest_from = from;
        to.ld_rest = w.in.rows - from;
        matmul_scatter(w.in, in, T, to);
        y.p = y_in_.as<float>();
        y.ld = (int)to.ld_rest;
        a.yh = img_qkv_.as<__nv_bfloat16>();
        a.ldh = from;
    } else {
        y = matmul(w.in, in, T, y_in_, 0);
    }
    a.common.lanes = state_lanes_;
    a.common.state = st.state.as<float>();
    a.common.heads = s.heads;
    a.common.dim = s.dim;
    a.common.vdim = s.vdim;
    a.common.out = raw_.as<float>();
    a.common.gate_sigmoid = 1;
    a.common.norm_w = w.head_norm.as<float>();
    a.common.norm_per_head = 1;
    a.common.eps = ms_.eps;
    a.common.gate = y;
    a.common.gate_col = w.c_g - from;
    a.y = y;
    a.q_col = w.c_q;
    a.k_col = w.c_k;
    a.v_col = w.c_v;
    a.i_col = w.c_i - from;
    a.f_col = w.c_f - from;
    a.i_bias = w.i_b.as<float>();
    a.f_bias = w.f_b.as<float>();
    a.cap = s.gate_cap;
    a.running_max = st.running_max.as<float>();
    a.common.image = out;
    a.counters = mlstm_counters_.as<int32_t>();
    a.rows = T;
    a.longest = longest_;
    a.rounded = f32_ ? 0 : 1;
    const double vw = (double)s.heads * s.vdim, kw = (double)s.heads * s.dim;
    prof_begin(KC_MLSTM_SCAN, (chunked ? 2.0 : 4.0) * T * (2.0 * kw + vw) + 4.0 * T * vw + T * vw * esz_ + 8.0 * t.B * (vw + s.heads) * s.dim, 6.0 * T * vw * s.dim);
    launches_ += launch_mlstm_scan(a, stream_);
    prof_end();
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
    const bool shared = s.shared_ff > 0;
    MoeRows rows = moe_;
    if (!shared) rows.shared_gate = nullptr;
    const int half = moe_half_;
    moe_half_ ^= 1;
    if (moe_router_is_narrow(T, s.experts, w.router.ld)) {
        prof_begin(KC_MOE_ROUTE, (double)w.router.bytes + (double)T * C * esz_, 2.0 * T * (double)C * (s.experts + 1));
        launch_moe_router(u.raw, f32_ ? w.router.f32.ptr() : w.router.half.values.ptr(), T, s.experts, s.top, rows, half, status_.as<int32_t>(), stream_);
        prof_end();
    } else {
        const Shares z = matmul(w.router, u.raw, T, y_in_, 0);
        prof_begin(KC_MOE_ROUTE, (double)T * (s.experts + 1) * 4.0, 0);
        launch_moe_route(z, T, s.experts, s.top, rows, half, status_.as<int32_t>(), stream_);
        prof_end();
    }
    prof_begin(KC_MOE_GATHER, (double)(T + P) * C * esz_, 0);
    launch_moe_gather(f32_ ? (const void*)u.raw.f : (const void*)u.raw.h, T, s.experts, s.top, (int64_t)w.router.ld * esz_, rows, half, img_rows_.ptr(), stream_);
    prof_end();
    launches_ += 2;

    // A token's weight multiplies what goes into an expert, so the gate and up sums of a grouped row; the shared expert's gate
    // multiplies what comes out, so the input of its last matrix.
    const RowImage in = image(img_rows_, w.experts_gu.ld), act = image(img_expert_ff_, w.experts_down.ld), every = image(img_ff_, shared ? w.down.ld : 64);
    float* routed = routed_.as<float>();
    float* of_every = routed + (size_t)P * C;
    GatedAct ga, gs;
    ga.kind = gs.kind = GatedAct::Clamped;
    ga.limit = s.limit;
    ga.pre = rows.weight_of_pos;
    gs.limit = s.shared_limit;
    gs.post = rows.shared_gate;
    const int gu_rows = pad_to(2 * s.ff, 128), shared_rows = pad_to(2 * s.shared_ff, 128), down_rows = pad_to(C, 128);
    const double met = std::min<double>(s.experts, P);  // experts with rows, at most
    const double gu_bytes = (double)w.experts_gu.bytes / s.experts * met + w.gate_up.bytes, down_bytes = (double)w.experts_down.bytes / s.experts * met + w.down.bytes;
    const double ff_rows = (double)P * s.ff + (double)T * s.shared_ff;
    const double gu_io = (double)esz_ * ((P + (shared ? T : 0.0)) * C + ff_rows), down_io = esz_ * ff_rows + 4.0 * (P + (shared ? T : 0.0)) * C;
    if (f32_) {
        prof_begin(KC_MOE_GEMM, gu_bytes + down_bytes + gu_io + down_io, 6.0 * C * ff_rows);
        Shares gu;
        gu.p = y_gu_.as<float>();
        gu.ld = gu_rows;
        launch_f32_matmul_experts(w.experts_gu.f32.as<float>(), s.experts, rows.offsets, gu_rows, gu_rows, w.experts_gu.ld, in.f, P, y_gu_.as<float>(), gu_rows, stream_);
        launch_gated_act(gu, P, s.ff, act, stream_, ga);
        launch_f32_matmul_experts(w.experts_down.f32.as<float>(), s.experts, rows.offsets, C, down_rows, w.experts_down.ld, act.f, P, routed, C, stream_);
        launches_ += 3;
        if (shared) {
            gu.ld = shared_rows;
            launch_f32_matmul(w.gate_up.f32.as<float>(), shared_rows, w.gate_up.ld, u.raw.f, T, y_gu_.as<float>(), shared_rows, 1, nullptr, stream_);
            launch_gated_act(gu, T, s.shared_ff, every, stream_, gs);
            launch_f32_matmul(w.down.f32.as<float>(), C, w.down.ld, every.f, T, of_every, C, 1, nullptr, stream_);
            launches_ += 3;
        }
        prof_end();
    } else {
        HgemmScratch ws;
        ws.status = status_.as<int32_t>();
        ExpertRows er, es;  // the experts; beside them the one every token runs
        er.W = &w.experts_gu.half;
        er.experts = s.experts;
        er.rows = er.rows_padded = gu_rows;
        er.offsets = rows.offsets;
        er.xh = reinterpret_cast<const __half*>(in.h);
        er.T = P;
        er.act = &ga;
        er.yh = reinterpret_cast<__half*>(act.h);
        er.ldyh = act.ld;
        es.W = &w.gate_up.half;
        es.experts = 1;
        es.rows = es.rows_padded = shared_rows;
        es.xh = reinterpret_cast<const __half*>(u.raw.h);
        es.T = T;
        es.act = &gs;
        es.yh = reinterpret_cast<__half*>(every.h);
        es.ldyh = every.ld;
        prof_begin(KC_MOE_GEMM, gu_bytes + gu_io, 4.0 * C * ff_rows);
        launch_hgemm_tc_experts(er, shared ? &es : nullptr, ws, stream_);
        prof_end();
        er.W = &w.experts_down.half;
        er.xh = er.yh;
        er.y = routed;
        es.W = &w.down.half;
        es.xh = es.yh;
        es.y = of_every;
        for (ExpertRows* e : {&er, &es}) {
            e->rows = C;
            e->rows_padded = down_rows;
            e->ldy = C;
            e->act = nullptr;
            e->yh = nullptr;
        }
        prof_begin(KC_MOE_GEMM, down_bytes + down_io, 2.0 * C * ff_rows);
        launch_hgemm_tc_experts(er, shared ? &es : nullptr, ws, stream_);
        prof_end();
        launches_ += 2;
    }
    pend.n = 1;
    if (shared) {
        pend.y[0].p = of_every;
        pend.y[0].ld = C;
    }
    pend.routed_at = rows.pos_of_pair;
    pend.routed_k = s.top;
    pend.w[0] = w.norm2.w.as<float>();
    pend.coef = ms_.residual_mult;
}

}  // namespace mk
