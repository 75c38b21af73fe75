// See mixer_lm.h.
#include "mixer_lm.h"
#include "model_registry.h"
#include "qstream_tc.h"
#include <algorithm>
#include <cmath>
#include <cstring>
#include <sys/stat.h>

namespace mk {

namespace {

const std::vector<const char*> class_names = {"hgemm_tc", "hgemm_tc_splitk", "f32_matmul", "wkv_scan", "delta_scan", "paged_attention", "rope_kv_scatter",
                                              "row_update", "delta_prep", "wkv_decay", "latent_attention", "mingru_scan", "latent_prep", "latent_rows",
                                              "mlstm_scan", "moe_gemm", "moe_route", "moe_gather", "gates", "channel_gates", "embed", "build_batch", "argmax"};

bool is_mixer_checkpoint(const std::string& dir) {
    struct stat st;
    return stat((dir + "/config.json").c_str(), &st) == 0 && S_ISREG(st.st_mode);
}

const RegisterModelFormat register_mixer_format(ModelFormat{
    "folder with config.json and model.safetensors", is_mixer_checkpoint,
    [](const std::string& path, const ModelConfig& cfg) -> std::unique_ptr<PagedLm> { return std::make_unique<MixerLm>(path, cfg); }});

}  // namespace

MixerLm::MixerLm(const std::string& dir, const ModelConfig& cfg) : DeviceLm(cfg, class_names) {
    const SafetensorsFile f(dir + "/model.safetensors");
    ms_ = read_mixer_spec_of(dir, f);
    validate_mixer_tensors(ms_, f);  // before any device memory is touched
    f32_ = cfg.compute_f32;
    esz_ = f32_ ? 4 : 2;
    if (f32_) cfg_.kv_f16 = false;
    if (cfg.ep_size > 1) throw std::runtime_error("expert parallelism is not supported for mixer-built decoders");
    open_device();
    spec_.vocab = ms_.vocab;
    runs_ = ms_.runs();
    spec_.layers = (int)runs_.size();
    spec_.hidden = ms_.width;
    // every layer kind of these decoders carries a recurrent state, of which a prompt prefix keeps no copy
    init_pool(cfg_.block_tokens, cfg_.slab_blocks, cfg_.kv_capacity_tokens, cfg_.prefix_capacity_tokens, "recurrent layers");
    init_state_slots(cfg_.state_slots > 0 ? cfg_.state_slots : cfg_.max_batch_lanes);
    spec_.max_context = (int)std::min<int64_t>(pool_->max_blocks() * pool_->block_tokens(), 1 << 30);
    lw_.resize(ms_.layers.size());
    rs_.resize(runs_.size());
    load(f);
    for (int i = 0; i < (int)runs_.size(); ++i) alloc_run(i);
    alloc_activations();
    MK_CUDA(cudaStreamSynchronize(stream_));
}

MixerLm::~MixerLm() {
    if (stream_) cudaStreamSynchronize(stream_);
}

// ---------------------------------------------------------------------------- load

void MixerLm::upload_f32(const std::vector<float>& v, DevBuf& out) {
    out.upload(v.data(), v.size() * 4, stream_);
    MK_CUDA(cudaStreamSynchronize(stream_));
}

void MixerLm::upload_norm(const SafetensorsFile& f, const std::string& name, Norm& out) {
    if (ms_.one_number_norms) upload_f32(std::vector<float>((size_t)ms_.width, f.values(name, {}).at(0)), out.w);
    else upload_f32(f.values(name, {ms_.width}), out.w);
    if (ms_.norm != NormKind::DynTanh) return;
    upload_f32(f.values(name + ".b", {ms_.width}), out.b);
    out.alpha = f.values(name + ".alpha", {}).at(0);
}

void MixerLm::place(const SafetensorsFile& f, const Part& p, int cols, int ld, std::vector<float>& m) {
    const int n = p.cols > 0 ? p.cols : cols, block = p.block > 0 ? p.block : p.rows;
    const std::vector<float> v = f.values(p.name, {p.rows, n});
#pragma omp parallel for
    for (int r = 0; r < p.rows; ++r) {
        int in_block = r % block;
        if (p.turn_from >= 0 && in_block >= p.turn_from) {
            const int i = in_block - p.turn_from, half = p.turn_dims / 2;
            in_block = p.turn_to + (i >= p.turn_dims ? i : (i < half ? 2 * i : 2 * (i - half) + 1));
        }
        const int64_t row = p.at + (int64_t)(r / block) * p.pitch + (int64_t)in_block * p.step;
        memcpy(&m[(size_t)(row * ld + p.col)], &v[(size_t)r * n], (size_t)n * 4);
    }
}

void MixerLm::upload_matrix(const std::vector<float>& m, int64_t rows, int ld, int64_t true_bytes, Dense& out, const std::vector<int64_t>& group_rows,
                            int groups, double share_per_token) {
    out.rows = rows;
    out.ld = ld;
    out.bytes = true_bytes;
    out.n_groups = 1;
    if (groups > 0) {
        out.n_groups = groups;
        out.group_tiles = (int)(rows / groups / 128);
    } else if (group_rows.size() > 1) {
        out.n_groups = (int)group_rows.size();
        int64_t end = 0;
        for (size_t g = 0; g < group_rows.size(); ++g) out.group_end[g] = (int)((end += group_rows[g]) / 128);
    }
    if (f32_) upload_f32(m, out.f32);
    else if (groups > 0) build_bf16_weight_groups(m.data(), rows, ld, groups, out.half, stream_);
    else build_bf16_weight(m.data(), rows, ld, out.half, stream_, group_rows);
    spec_.weight_bytes += out.bytes;
    spec_.weight_bytes_per_token += (int64_t)((double)out.bytes * share_per_token) * passes_;
}

void MixerLm::upload_dense(const SafetensorsFile& f, const std::vector<Part>& parts, int64_t rows, int cols, Dense& out,
                           const std::vector<int64_t>& group_rows, double share_per_token) {
    const int ld = pad_to(cols, 64);
    std::vector<float> m((size_t)(rows * ld), 0.f);
    int64_t bytes = 0;
    for (const Part& p : parts) {
        place(f, p, cols, ld, m);
        bytes += (int64_t)p.rows * (p.cols > 0 ? p.cols : cols) * esz_;
    }
    upload_matrix(m, rows, ld, bytes, out, group_rows, 0, share_per_token);
}

int MixerLm::rope_table(const RotarySpec& r) {
    for (size_t i = 0; i < rope_.size(); ++i)
        if (rope_[i]->spec.same_table(r)) return (int)i;
    auto t = std::make_unique<RopeTable>();
    t->spec = r;
    if (r.dims > 0) {
        // angles in f64, so that a far position is as exact as a near one
        const std::vector<double> freq = rotary_frequencies(r);
        const double amplitude = rotary_amplitude(r);
        const int64_t positions = pool_->max_blocks() * pool_->block_tokens(), half = r.dims / 2;
        std::vector<float> c((size_t)(positions * half)), s((size_t)(positions * half));
#pragma omp parallel for
        for (int64_t p = 0; p < positions; ++p)
            for (int64_t i = 0; i < half; ++i) {
                const double a = (double)p * freq[(size_t)i];
                c[(size_t)(p * half + i)] = (float)(amplitude * std::cos(a));
                s[(size_t)(p * half + i)] = (float)(amplitude * std::sin(a));
            }
        upload_f32(c, t->cos_t);
        upload_f32(s, t->sin_t);
    }
    rope_.push_back(std::move(t));
    return (int)rope_.size() - 1;
}

int MixerLm::geometry_of(const AttentionSpec& a) {
    const int need = std::max(a.dim, a.vdim);
    Geometry g;
    g.heads = a.heads;
    g.kv_heads = a.kv_heads;
    g.chunk = a.chunk;
    g.window = a.window;
    // the tensor-core kernels take rows of 64, 128 or 256; narrower heads are padded with zeros in the pools
    for (int d : {64, 128, 256})
        if (need <= d && !g.tc && attention_tc_supported(a.heads, a.kv_heads, d, cfg_.block_tokens, cfg_.kv_f16)) {
            g.tc = true;
            g.row_width = d;
        }
    if (!g.tc) g.row_width = pad_to(need, 4);
    if (g.row_width > 256) throw std::runtime_error("attention head dimensions above 256 are not supported");
    if (a.heads / a.kv_heads > 64) throw std::runtime_error("more than 64 query heads per key/value head are not supported");
    for (size_t i = 0; i < geo_.size(); ++i)
        if (geo_[i].heads == g.heads && geo_[i].kv_heads == g.kv_heads && geo_[i].row_width == g.row_width && geo_[i].chunk == g.chunk && geo_[i].window == g.window) return (int)i;
    geo_.push_back(std::move(g));
    return (int)geo_.size() - 1;
}

void MixerLm::load(const SafetensorsFile& f) {
    const int C = ms_.width;
    // token tables stay as rows to gather
    auto table = [&](const std::string& name, int64_t cols, DevBuf& out) {
        if (f32_) upload_f32(f.values(name, {ms_.vocab, cols}), out);
        else {
            const std::vector<uint16_t> bits = f.bf16_values(name, {ms_.vocab, cols});
            out.upload(bits.data(), bits.size() * 2, stream_);
            MK_CUDA(cudaStreamSynchronize(stream_));
        }
        spec_.weight_bytes += ms_.vocab * cols * esz_;
    };
    table("embed", C, embed_);
    if (ms_.side_dim > 0) table("side.embed", (int64_t)ms_.layers.size() * ms_.side_dim, side_embed_);
    if (ms_.sinusoid_positions) {
        upload_norm(f, "embed.norm", embed_norm_);
        std::vector<double> freq((size_t)(C + 1) / 2);
        for (size_t i = 0; i < freq.size(); ++i) freq[i] = std::pow(10000.0, -2.0 * (double)i / C);
        position_freq_.upload(freq.data(), freq.size() * 8, stream_);
        MK_CUDA(cudaStreamSynchronize(stream_));
    }
    if (ms_.loop.times > 0) {
        const int second = pad_to(C, 64);  // where the embedding output's columns begin in the input of `loop.in`
        const std::vector<float> w = f.values("loop.in", {C, 2 * C});
        std::vector<float> m((size_t)C * 2 * second, 0.f);
        for (int r = 0; r < C; ++r)
            for (int h = 0; h < 2; ++h) memcpy(&m[((size_t)r * 2 + h) * second], &w[((size_t)r * 2 + h) * C], (size_t)C * 4);
        passes_ = ms_.loop.times;
        upload_matrix(m, C, 2 * second, (int64_t)2 * C * C * esz_, loop_in_, {}, 0);
        upload_f32(f.values("loop.step", {ms_.loop.times, C}), loop_step_);
    }
    for (int l = 0; l < (int)ms_.layers.size(); ++l) {
        if (ms_.layers[(size_t)l].weights_of >= 0) continue;
        passes_ = (int)std::count_if(runs_.begin(), runs_.end(), [&](const LayerRun& r) { return r.layer == l; });
        load_layer(f, l);
    }
    passes_ = 1;
    upload_norm(f, "final.norm", final_norm_);
    upload_dense(f, {{"head", ms_.vocab, 0}}, ms_.vocab, C, head_);
}

void MixerLm::load_layer(const SafetensorsFile& f, int l) {
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    Layer& w = lw_[(size_t)l];
    if (ms_.side_by_side()) return load_side_by_side(f, l);
    if (ms_.norm_place == NormPlace::Output) return load_output_norm(f, l);
    if (ms_.conv_taps > 0) return load_conv_input(f, l);
    const int C = ms_.width;
    const std::string p = "l" + std::to_string(l) + ".", m = p + "mix.";
    upload_norm(f, p + "norm1", w.norm1);
    if (s.kind == MixerKind::Wkv) {
        const int HD = s.wkv.heads * s.wkv.dim, R = s.wkv.rank;
        // r, k, v, g and the decay's low-rank input, each over its own mix of the token and its predecessor
        const int big = pad_to(HD, 128), low = pad_to(R, 128);
        w.c_q = 0; w.c_k = big; w.c_v = 2 * big; w.c_g = 3 * big; w.c_low = 4 * big;
        upload_dense(f, {{m + "r", HD, w.c_q}, {m + "k", HD, w.c_k}, {m + "v", HD, w.c_v}, {m + "g", HD, w.c_g}, {m + "w1", R, w.c_low}}, 4 * (int64_t)big + low, C,
                     w.in, {big, big, big, big, low});
        std::vector<float> mu;
        for (const char* name : {"r", "k", "v", "g", "w"}) {
            const std::vector<float> v = f.values(m + "mu." + name, {C});
            mu.insert(mu.end(), v.begin(), v.end());
        }
        upload_f32(mu, w.mu);
        upload_low_rank(f, m, HD, R, w);
        upload_f32(f.values(m + "u", {s.wkv.heads, s.wkv.dim}), w.bonus);
        upload_f32(f.values(m + "norm", {HD}), w.head_norm);
        upload_dense(f, {{m + "o", C, 0}}, C, HD, w.out);
    } else {
        const AttentionSpec& a = s.attn;
        const DeltaSpec& d = s.delta;
        const std::string L = m + "left.", Rt = m + "right.";
        // every projection of both branches reads the same input: one stacked matrix
        std::vector<Part> parts;
        int at = 0;
        auto part = [&](const std::string& name, int rows) {
            const int here = at;
            parts.push_back({name, rows, here});
            at = pad_to(at + rows, 4);
            return here;
        };
        w.c_q = part(L + "q", a.heads * a.dim);
        w.c_k = part(L + "k", a.kv_heads * a.dim);
        w.c_v = part(L + "v", a.kv_heads * a.vdim);
        w.c_g = part(L + "g", a.heads);
        w.d_q = part(Rt + "q", d.kv_heads * d.dim);
        w.d_k = part(Rt + "k", d.kv_heads * d.dim);
        w.d_v = part(Rt + "v", d.heads * d.vdim);
        w.d_a = part(Rt + "a", d.heads);
        w.d_b = part(Rt + "b", d.heads);
        w.d_g = part(Rt + "g", d.heads * d.vdim);
        upload_dense(f, parts, at, C, w.in);
        upload_f32(f.values(L + "q.norm", {a.dim}), w.q_norm);
        upload_f32(f.values(L + "k.norm", {a.dim}), w.k_norm);
        upload_dense(f, {{L + "o", C, 0}}, C, a.heads * a.vdim, w.out);
        upload_dense(f, {{Rt + "o", C, 0}}, C, d.heads * d.vdim, w.out2);
        upload_f32(f.values(m + "left.out", {C}), w.out_norm);
        upload_f32(f.values(m + "right.out", {C}), w.out2_norm);
        w.geometry = geometry_of(a);
        w.row_width = geo_[(size_t)w.geometry].row_width;
        w.rope = rope_table(a.rot);
        // delta rule
        const int kw = d.kv_heads * d.dim, vw = d.heads * d.vdim, channels = 2 * kw + vw;
        if (d.dim > 256 || d.vdim > 256) throw std::runtime_error("delta-rule head dimensions above 256 are not supported");
        std::vector<float> conv((size_t)channels * d.taps);
        int ch0 = 0;
        for (const auto& part_of : {std::make_pair("q", kw), std::make_pair("k", kw), std::make_pair("v", vw)}) {
            const std::vector<float> t = f.values(Rt + part_of.first + ".conv", {part_of.second, d.taps});
            for (int c = 0; c < part_of.second; ++c)
                for (int j = 0; j < d.taps; ++j) conv[(size_t)j * channels + ch0 + c] = t[(size_t)c * d.taps + j];
            ch0 += part_of.second;
        }
        upload_f32(conv, w.conv);
        upload_f32(f.values(Rt + "dt_bias", {d.heads}), w.dt_bias);
        std::vector<float> decay = f.values(Rt + "A_log", {d.heads});
        for (float& v : decay) v = (float)-std::exp((double)v);
        upload_f32(decay, w.log_decay);
        upload_f32(f.values(Rt + "norm", {d.vdim}), w.head_norm);
    }
    if (s.ff > 0) {
        upload_norm(f, p + "norm2", w.norm2);
        upload_dense(f, {{p + "mlp.gate", s.ff, 0, 2}, {p + "mlp.up", s.ff, 1, 2}}, 2 * (int64_t)s.ff, C, w.gate_up);
        upload_dense(f, {{p + "mlp.down", C, 0}}, C, s.ff, w.down);
    }
    if (ms_.side_dim > 0) {
        upload_dense(f, {{p + "side.gate", ms_.side_dim, 0}}, ms_.side_dim, C, w.side_gate);
        upload_dense(f, {{p + "side.proj", C, 0}}, C, ms_.side_dim, w.side_proj);
        upload_f32(f.values(p + "side.norm", {C}), w.side_norm);
    }
}

// The second half of a low-rank projection and its bias, for the kernels that keep it in f32.
void MixerLm::upload_low_rank(const SafetensorsFile& f, const std::string& prefix, int channels, int rank, Layer& w) {
    const std::vector<float> w2 = f.values(prefix + "w2", {channels, rank});
    std::vector<float> w2t(w2.size());
    for (int c = 0; c < channels; ++c)
        for (int j = 0; j < rank; ++j) w2t[(size_t)j * channels + c] = w2[(size_t)c * rank + j];
    upload_f32(w2t, w.w2t);
    spec_.weight_bytes += (int64_t)channels * rank * 4;
    spec_.weight_bytes_per_token += (int64_t)channels * rank * 4;
    upload_f32(f.values(prefix + "w0", {channels}), w.w0);
}

void MixerLm::alloc_run(int run) {
    const int l = runs_[(size_t)run].layer;
    const MixerLayerSpec& s = ms_.layers[(size_t)l];
    const Layer& w = lw_[(size_t)l];
    RunState& st = rs_[(size_t)run];
    const size_t halves = (size_t)state_slots_->capacity() * 2;
    auto pages = [&](DevBuf& pool, int kv_heads) {
        const int64_t bytes = (int64_t)kv_heads * cfg_.block_tokens * w.row_width * (cfg_.kv_f16 ? 2 : 4);
        pool.alloc((size_t)(pool_->max_blocks() * bytes));
        pool.zero(stream_);
        spec_.kv_bytes_per_token += bytes / cfg_.block_tokens;
    };
    if (s.kind == MixerKind::Wkv || ms_.side_by_side()) st.kept.alloc(halves * (size_t)ms_.width * 4);  // the token shift's row
    if (ms_.conv_taps > 1) st.kept.alloc(halves * (size_t)(ms_.conv_taps - 1) * ms_.width * 4);
    switch (s.kind) {
        case MixerKind::Wkv:
            st.state.alloc(halves * (size_t)s.wkv.heads * s.wkv.dim * linear_state_key_pad(s.wkv.dim) * 4);
            break;
        case MixerKind::Parallel: {
            pages(st.k_pool, s.attn.kv_heads);
            pages(st.v_pool, s.attn.kv_heads);
            const DeltaSpec& d = s.delta;
            st.tail.alloc(halves * (size_t)std::max(1, d.taps - 1) * (2 * (size_t)d.kv_heads * d.dim + (size_t)d.heads * d.vdim) * 4);
            st.state.alloc(halves * (size_t)d.heads * d.vdim * linear_state_key_pad(d.dim) * 4);
            break;
        }
        case MixerKind::ScaledParallel:
            pages(st.k_pool, s.attn.kv_heads);
            pages(st.v_pool, s.attn.kv_heads);
            st.state.alloc(halves * (size_t)s.channel_delta.heads * s.channel_delta.dim * linear_state_key_pad(s.channel_delta.dim) * 4);
            break;
        case MixerKind::Latent: pages(st.k_pool, 1); break;
        case MixerKind::MinGru: st.state.alloc(halves * (size_t)s.gru.width * 4); break;
        case MixerKind::Mlstm:
            st.state.alloc(halves * (size_t)s.mlstm.heads * (s.mlstm.vdim + 1) * linear_state_key_pad(s.mlstm.dim) * 4);
            st.running_max.alloc(halves * (size_t)s.mlstm.heads * 4);
            break;
        case MixerKind::Attention:
            pages(st.k_pool, s.attn.kv_heads);
            pages(st.v_pool, s.attn.kv_heads);
            break;
    }
}

void MixerLm::alloc_activations() {
    const int64_t T = cfg_.max_batch_tokens;
    const int B = cfg_.max_batch_lanes, C = ms_.width;
    int64_t in_rows = 0, mix = 0, a_w = 0, b_w = 0, ff = 0, hd = 0, raw = 0, dqk = 0, dv = 0, dh = 0, attn = 0;
    int64_t q_lat = 0, uq = 0, lat = 0, cat = 0;  // widths of latent attention's rows, and of `out`'s input with both branches
    int lat_ctas = 1;
    int64_t lat_part = 0;
    int64_t mlstm_heads = 0, qkv = 0, removal = 0;
    size_t delta_scratch = 0;
    int64_t pairs = 0, experts = 0, expert_ff = 0, expert_gu = 0;  // routed rows, experts, widths of an expert's activations
    for (size_t l = 0; l < lw_.size(); ++l) {
        const MixerLayerSpec& s = ms_.layers[l];
        const Layer& w = lw_[l];
        in_rows = std::max(in_rows, w.in.rows);
        if (s.ff > 0 && ms_.ff_kind == FfKind::Moe) {
            pairs = std::max(pairs, T * s.moe.top);
            experts = std::max(experts, (int64_t)s.moe.experts);
            in_rows = std::max(in_rows, w.router.rows);
            expert_ff = std::max(expert_ff, (int64_t)w.experts_down.ld);
            expert_gu = std::max(expert_gu, w.experts_gu.rows / std::max(1, s.moe.experts));
        }
        if (s.kind == MixerKind::Mlstm) {
            mlstm_heads = std::max(mlstm_heads, (int64_t)s.mlstm.heads);
            qkv = std::max(qkv, (int64_t)w.c_g);
            b_w = std::max(b_w, (int64_t)s.mlstm.heads * s.mlstm.vdim);
            raw = std::max(raw, (int64_t)s.mlstm.heads * linear_state_raw_width(s.mlstm.vdim));
        } else if (s.kind == MixerKind::Attention) {
            a_w = std::max(a_w, (int64_t)s.attn.heads * s.attn.vdim);
            attn = std::max(attn, (int64_t)s.attn.heads * w.row_width);
        }
        if (ms_.norm_place == NormPlace::Output) {
            ff = std::max(ff, (int64_t)pad_to(s.moe.shared_ff, 64));
            continue;
        }
        if (s.kind == MixerKind::Latent) {
            const LatentSpec& a = s.latent;
            q_lat = std::max(q_lat, (int64_t)w.uq.ld);
            uq = std::max(uq, (int64_t)a.heads * w.q_width);
            lat = std::max(lat, (int64_t)a.heads * w.row_width);
            const LatentGeometry& g = latent_geo_[(size_t)w.geometry];
            if (g.wide) attn = std::max(attn, (int64_t)a.heads * w.q_width);
            lat_ctas = std::max(lat_ctas, g.ctas);
            if (g.tc) lat_part = std::max(lat_part, (int64_t)latent_max_shared_entries(g.ctas) * latent_tc_groups(a.heads) * latent_tc_heads(a.heads) * w.value_width);
        }
        if (ms_.side_by_side()) {
            mix = 2;
            cat = std::max(cat, (int64_t)w.out.ld);
            continue;
        }
        if (ms_.conv_taps > 0) cat = std::max(cat, (int64_t)w.out.ld);
        ff = std::max(ff, (int64_t)s.ff);
        if (s.kind == MixerKind::Wkv) {
            mix = 5;
            const int64_t n = (int64_t)s.wkv.heads * s.wkv.dim;
            hd = std::max(hd, n);
            raw = std::max(raw, n);
            b_w = std::max(b_w, n);
        } else if (s.kind == MixerKind::Parallel) {
            a_w = std::max(a_w, (int64_t)s.attn.heads * s.attn.vdim);
            attn = std::max(attn, (int64_t)s.attn.heads * w.row_width);
            const int64_t n = (int64_t)s.delta.heads * s.delta.vdim;
            b_w = std::max(b_w, n);
            raw = std::max(raw, n);
            dqk = std::max(dqk, (int64_t)s.delta.kv_heads * s.delta.dim);
            dv = std::max(dv, n);
            dh = std::max(dh, (int64_t)s.delta.heads);
        } else if (s.kind == MixerKind::ScaledParallel) {
            attn = std::max(attn, (int64_t)s.attn.heads * w.row_width);
            const int64_t n = (int64_t)s.channel_delta.heads * s.channel_delta.dim;
            removal = std::max(removal, n);
            if (!f32_) delta_scratch = std::max(delta_scratch, channel_delta_chunk_bytes(s.channel_delta.dim, s.channel_delta.heads, (int)T, B));
            hd = std::max(hd, n);
            raw = std::max(raw, n);
        }
    }
    const int64_t ldc = pad_to(C, 64);
    for (DevBuf& x : x_) x.alloc((size_t)(T * C) * 4);
    mixes_.alloc((size_t)(mix * T * ldc) * esz_);
    img_h_.alloc((size_t)(T * ldc) * esz_);
    img_a_.alloc((size_t)(T * pad_to(a_w, 64)) * esz_);
    img_b_.alloc((size_t)(T * pad_to(b_w, 64)) * esz_);
    img_ff_.alloc((size_t)(T * pad_to(ff, 64)) * esz_);
    img_ff_.zero(stream_);  // the gated matmul writes the true columns only
    img_side_.alloc((size_t)(T * pad_to(std::max(ms_.side_dim, 1), 64)) * esz_);
    y_in_.alloc((size_t)(T * std::max<int64_t>(in_rows, ms_.side_dim)) * 4);
    y_a_.alloc((size_t)(T * C) * 4);
    y_b_.alloc((size_t)(T * C) * 4);
    if (f32_) y_gu_.alloc((size_t)std::max(T * 2 * ff, pairs * expert_gu) * 4);
    mlstm_counters_.alloc((size_t)(B * mlstm_heads) * 4);
    mlstm_counters_.zero(stream_);
    if (!f32_) img_qkv_.alloc((size_t)(T * qkv) * 2);
    if (pairs > 0) {
        img_rows_.alloc((size_t)(pairs * ldc) * esz_);
        img_expert_ff_.alloc((size_t)(pairs * expert_ff) * esz_);
        routed_.alloc((size_t)((pairs + T) * C) * 4);
        moe_words_.alloc((size_t)(5 * pairs + 3 * experts + 1 + T) * 4);
        moe_words_.zero(stream_);  // the counts
        moe_.sel = moe_words_.as<int32_t>();
        moe_.rank = moe_.sel + pairs;
        moe_.pos_of_pair = moe_.rank + pairs;
        moe_.count = moe_.pos_of_pair + pairs;
        moe_.counts = (int)experts;
        moe_.offsets = moe_.count + 2 * experts;
        moe_.weight = reinterpret_cast<float*>(moe_.offsets + experts + 1);
        moe_.weight_of_pos = moe_.weight + pairs;
        moe_.shared_gate = moe_.weight_of_pos + pairs;
    }
    decay_.alloc((size_t)(T * hd) * 4);
    removal_.alloc((size_t)(T * removal) * 4);
    delta_scratch_.alloc(delta_scratch);
    raw_.alloc((size_t)(T * raw) * 4);
    q_rot_.alloc((size_t)(T * attn) * 4);
    img_q_.alloc((size_t)(T * q_lat) * esz_);
    img_uq_.alloc((size_t)(T * uq) * esz_);
    q_lat_.alloc((size_t)(T * lat) * 4);
    img_lat_.alloc((size_t)(T * lat) * esz_);
    img_cat_.alloc((size_t)(T * cat) * esz_);
    img_cat_.zero(stream_);  // padding between and behind the two parts meets zero weights
    if (ms_.loop.times > 0) img_loop_.alloc((size_t)(T * loop_in_.ld) * esz_);
    if (lat_part > 0) {
        lat_part_o_.alloc((size_t)lat_part * 4);
        lat_part_ml_.alloc((size_t)lat_part / 64 * 2 * 4);
        lat_counters_.alloc((size_t)latent_max_shared_entries(1) * lat_ctas * 4);
        lat_counters_.zero(stream_);
    }
    attn_.alloc((size_t)(T * attn) * 4);
    dq_.alloc((size_t)(T * dqk) * 4);
    dk_.alloc((size_t)(T * dqk) * 4);
    dv_.alloc((size_t)(T * dv) * 4);
    dbeta_.alloc((size_t)(T * dh) * 4);
    ddecay_.alloc((size_t)(T * dh) * 4);
    if (!f32_)
        for (DevBuf& p : partial_) p.alloc(kSplitScratchBytes);
    size_t extra = (size_t)B * sizeof(StateLane) + 16;
    if (ms_.conv_taps > 0) extra += (size_t)B * sizeof(StateLane) + 48;
    size_t part_o = 0, part_ml = 0, counters = 0;
    for (const Geometry& g : geo_) {
        if (g.tc) {
            const int entries = attention_tc_max_entries(B, g.kv_heads);
            attn_max_entries_ = std::max(attn_max_entries_, entries);
            part_o = std::max(part_o, (size_t)entries * g.kv_heads * 16 * g.row_width * 4);
            part_ml = std::max(part_ml, (size_t)entries * g.kv_heads * 16 * 2 * 4);
            counters = std::max(counters, (size_t)B * g.kv_heads * 4);
            extra += ((size_t)(T + B) * 2 + (size_t)entries * 8 + (size_t)B * 3) * 4 + 64;
        } else {
            extra += (size_t)(T + B) * 8 + 64;
        }
    }
    for (const LatentGeometry& g : latent_geo_) extra += (size_t)latent_max_entries((int)T, g.ctas) * 32 + (size_t)T * 4 + 32;
    extra += wide_.size() * ((size_t)B * sizeof(LaneHeader) + (size_t)(T + B) * 8 + (size_t)T * 4 + (size_t)(pool_->max_blocks() + B) * 4 + 64);
    attn_part_o_.alloc(part_o);
    attn_part_ml_.alloc(part_ml);
    attn_counters_.alloc(counters);
    attn_counters_.zero(stream_);
    alloc_tick(extra);
}

// ---------------------------------------------------------------------------- forward

RowImage MixerLm::image(DevBuf& b, int ld) const {
    RowImage im;
    im.ld = ld;
    if (f32_) im.f = b.as<float>();
    else im.h = b.as<__nv_bfloat16>();
    return im;
}

Shares MixerLm::matmul(const Dense& W, const RowImage& x, int T, DevBuf& y, int scratch) {
    Shares out;
    out.p = y.as<float>();
    out.ld = (int)W.rows;
    const double bytes = (double)W.bytes + (double)esz_ * T * W.ld * W.n_groups + 4.0 * T * W.rows, flops = 2.0 * T * (double)W.rows * W.ld;
    if (f32_) {
        prof_begin(KC_F32_MATMUL, bytes, flops);
        launch_f32_matmul(W.f32.as<float>(), W.rows, W.ld, x.f, T, y.as<float>(), (int)W.rows, W.n_groups, W.group_end, stream_, W.group_tiles);
    } else {
        prof_begin(T <= 64 ? KC_GEMM_NARROW : KC_GEMM, bytes, flops);
        HgemmScratch ws;
        ws.partial = partial_[scratch].as<float>();
        ws.partial_floats = partial_[scratch].size() / 4;
        ws.status = status_.as<int32_t>();
        const int splits = launch_hgemm_tc(W.half, reinterpret_cast<const __half*>(x.h), T, y.as<float>(), (int)W.rows, 1.f, 0.f, ws, stream_, 16);
        if (splits > 1) {
            out.p = ws.partial;
            out.n = splits;
            out.stride = (int64_t)T * W.rows;
        }
    }
    prof_end();
    ++launches_;
    return out;
}

void MixerLm::matmul_scatter(const Dense& W, const RowImage& x, int T, const MatmulScatter& to) {
    const double bytes = (double)W.bytes + (double)esz_ * T * W.ld * W.n_groups + (to.type == MatmulScatter::F32 ? 4.0 : 2.0) * T * W.rows;
    const double flops = 2.0 * T * (double)W.rows * W.ld;
    if (f32_) {
        prof_begin(KC_F32_MATMUL, bytes, flops);
        launch_f32_matmul(W.f32.as<float>(), W.rows, W.ld, x.f, T, nullptr, 0, W.n_groups, W.group_end, stream_, W.group_tiles, 1.f, &to);
    } else {
        prof_begin(T <= 64 ? KC_GEMM_NARROW : KC_GEMM, bytes, flops);
        HgemmScratch ws;
        ws.status = status_.as<int32_t>();
        launch_hgemm_tc_scatter(W.half, reinterpret_cast<const __half*>(x.h), T, to, ws, stream_);
    }
    prof_end();
    ++launches_;
}

void MixerLm::set_norm(RowUpdateArgs& a, const Norm& n) const {
    a.norm = ms_.norm;
    a.norm_eps = ms_.eps;
    a.alpha = n.alpha;
    a.norm_w = n.w.as<float>();
    a.norm_b = n.b.as<float>();
}

// Fills in the residual part of a row update; what is pending is added on the way.
void MixerLm::apply_pending(RowUpdateArgs& a, Pending& p, bool other_buffer) {
    a.x = p.replace ? nullptr : x_[cur_].as<float>();
    a.width = ms_.width;
    a.n_add = p.n;
    for (int i = 0; i < p.n; ++i) {
        a.add[i] = p.y[i];
        a.add_w[i] = p.w[i];
    }
    a.add_bias = p.bias;
    if (p.routed_k > 0) {
        a.routed = routed_.as<float>();
        a.routed_at = p.routed_at;
        a.routed_k = p.routed_k;
    }
    a.add_coef = p.coef;
    a.add_eps = ms_.eps;
    if (p.n > 0) {
        if (other_buffer) cur_ ^= 1;
        a.x_out = x_[cur_].as<float>();
    }
    p = Pending{};
}

void MixerLm::run_wkv(const Tick& t, int run, Pending& pend) {
    const int l = runs_[(size_t)run].layer;
    RunState& st = rs_[(size_t)run];
    const WkvSpec& s = ms_.layers[(size_t)l].wkv;
    Layer& w = lw_[(size_t)l];
    const int T = t.T, C = ms_.width, HD = s.heads * s.dim;
    RowUpdateArgs u;
    u.rows = T;
    apply_pending(u, pend, true);
    set_norm(u, w.norm1);
    u.n_mix = 5;
    u.mu = w.mu.as<float>();
    u.mixes = image(mixes_, w.in.ld);
    u.lanes = state_lanes_;
    u.token_lane = t.bd.token_lane;
    u.kept = st.kept.as<float>();
    prof_begin(KC_ROW_UPDATE, (double)T * C * (8.0 + 4.0 * u.n_add + 5.0 * esz_), 0);
    launch_row_update(u, stream_);
    prof_end();
    const Shares y = matmul(w.in, u.mixes, T, y_in_, 0);
    prof_begin(KC_WKV_DECAY, (double)T * (HD + s.rank) * 4.0 + (double)HD * s.rank * 4.0, 2.0 * T * (double)HD * s.rank);
    launch_wkv_decay(y, w.c_low, T, s.rank, HD, w.w2t.as<float>(), w.w0.as<float>(), decay_.as<float>(), stream_);
    prof_end();
    WkvScanArgs a;
    a.common.lanes = state_lanes_;
    a.common.state = st.state.as<float>();
    a.common.heads = s.heads;
    a.common.dim = a.common.vdim = s.dim;
    a.common.out = raw_.as<float>();
    a.common.norm_w = w.head_norm.as<float>();
    a.common.norm_per_head = 1;
    a.common.eps = ms_.eps;
    a.common.gate = y;
    a.common.gate_col = w.c_g;
    a.rkv = y;
    a.r_col = w.c_q;
    a.k_col = w.c_k;
    a.v_col = w.c_v;
    a.decay = decay_.as<float>();
    a.bonus = w.bonus.as<float>();
    const RowImage img = image(img_b_, w.out.ld);
    const bool finish = short_lanes_ && linear_state_can_finish(s.dim, s.dim);
    if (finish) a.common.image = img;
    prof_begin(KC_WKV_SCAN, (double)T * HD * 20.0 + 8.0 * t.B * HD * s.dim, 8.0 * T * (double)HD * s.dim);
    launch_wkv_scan(a, stream_);
    prof_end();
    launches_ += 3;
    if (!finish) {
        a.common.image = img;
        prof_begin(KC_GATES, (double)T * HD * (8.0 + esz_), 0);
        launch_head_norm_gate(a.common, T, stream_);
        prof_end();
        ++launches_;
    }
    pend.n = 1;
    pend.y[0] = matmul(w.out, img, T, y_a_, 1);
}

void MixerLm::attend(const Tick& t, int run, const AttentionSpec& s, const Shares& y, const std::vector<LmLane>& lanes) {
    const int l = runs_[(size_t)run].layer;
    RunState& st = rs_[(size_t)run];
    Layer& w = lw_[(size_t)l];
    const int T = t.T, D = w.row_width, bt = cfg_.block_tokens;
    const bool whole = s.qk_norm == QkNorm::Whole;
    Geometry& g = geo_[(size_t)w.geometry];
    RopeKvArgs ra;
    ra.q = const_cast<float*>(y.p) + w.c_q;
    ra.k = y.p + w.c_k;
    ra.v = y.p + (s.keys_are_values ? w.c_k : w.c_v);
    ra.ldq = ra.ldk = ra.ldv = y.ld;
    ra.qk_splits = ra.v_splits = y.n;
    ra.qk_split_stride = ra.v_split_stride = y.stride;
    ra.q_out = q_rot_.as<float>();
    ra.ldq_out = s.heads * D;
    ra.q_norm_w = w.q_norm.as<float>();
    ra.k_norm_w = w.k_norm.as<float>();
    ra.norm_eps = ms_.eps;
    if (s.biases) {
        ra.q_bias = w.q_b.as<float>();
        ra.k_bias = w.k_b.as<float>();
        ra.v_bias = (s.keys_are_values ? w.k_b : w.v_b).as<float>();
    }
    if (s.rot.dims > 0) {
        ra.cos_t = rope_[(size_t)w.rope]->cos_t.as<float>();
        ra.sin_t = rope_[(size_t)w.rope]->sin_t.as<float>();
        ra.rotary_dim = s.rot.dims;
        ra.interleaved = s.rot.interleaved ? 1 : 0;
    }
    ra.positions = t.bd.positions;
    ra.slots = t.bd.slots;
    ra.k_pool = st.k_pool.ptr();
    ra.v_pool = st.v_pool.ptr();
    ra.kv_f16 = cfg_.kv_f16 ? 1 : 0;
    ra.T = T;
    ra.q_heads = s.heads;
    ra.kv_heads = s.kv_heads;
    ra.d = s.dim;
    ra.dv = s.vdim;
    ra.d_row = D;
    ra.block_tokens = bt;
    ra.layers = 1;
    ra.layer = 0;
    ra.pool_blocks = pool_->max_blocks();
    // ticks of one-token lanes: the attention kernel prepares its own rows
    const bool fuse_rope = !whole && g.tc && g.plan.n_tiles() == 0 && g.plan.n_entries() > 0 && g.plan.n_dec_lanes() == 0;
    const double kv_esz = cfg_.kv_f16 ? 2.0 : 4.0;
    if (!fuse_rope) {
        prof_begin(KC_ROPE_KV, (double)T * s.heads * (s.dim + D) * 4.0 + (double)T * s.kv_heads * (s.dim + s.vdim + 0.5 * kv_esz * D) * 4.0, 0);
        if (whole) launch_rope_kv_rows(ra, stream_);
        else launch_rope_kv(ra, stream_);
        prof_end();
        ++launches_;
    }
    double kv_tokens = 0, flops = 0;
    for (const LmLane& ln : lanes) {
        const int lo = attention_first_key(ln.start_pos, s.window, s.chunk);
        kv_tokens += (double)ln.start_pos + ln.n_tokens - lo;
        double pairs = (double)ln.n_tokens * (ln.start_pos - lo) + 0.5 * ln.n_tokens * ln.n_tokens;
        if (s.window > 0) {
            pairs = 0;
            for (int k = 0; k < ln.n_tokens; ++k) pairs += ln.start_pos + k + 1 - attention_first_key(ln.start_pos + k, s.window, s.chunk);
        } else if (s.chunk > 0) pairs = std::min(pairs, (double)ln.n_tokens * 0.5 * (s.chunk + 1));
        flops += 2.0 * s.heads * (s.dim + s.vdim) * pairs;
    }
    prof_begin(KC_ATTN, kv_tokens * 2 * s.kv_heads * D * kv_esz + 8.0 * T * s.heads * D, flops);
    if (g.tc) {
        AttnTcArgs ta;
        ta.q = q_rot_.as<float>();
        ta.out = attn_.as<float>();
        ta.k_pool = st.k_pool.ptr();
        ta.v_pool = st.v_pool.ptr();
        ta.hdr = t.bd.hdr;
        ta.tables = t.bd.tables;
        ta.cu_seqlens = t.bd.cu_seqlens;
        ta.tiles = reinterpret_cast<const int32_t*>(t.dp + g.off_tiles);
        ta.entries = reinterpret_cast<const int32_t*>(t.dp + g.off_entries);
        ta.dec_lanes = reinterpret_cast<const int32_t*>(t.dp + g.off_dec);
        ta.n_tiles = g.plan.n_tiles();
        ta.n_entries = g.plan.n_entries();
        ta.n_dec_lanes = g.plan.n_dec_lanes();
        ta.part_o = attn_part_o_.as<float>();
        ta.part_ml = attn_part_ml_.as<float>();
        ta.counters = attn_counters_.as<int32_t>();
        ta.q_heads = s.heads;
        ta.kv_heads = s.kv_heads;
        ta.d = D;
        ta.block_tokens = bt;
        ta.layers = 1;
        ta.pool_blocks = ra.pool_blocks;
        ta.scale = s.scale;
        ta.softcap = s.softcap;
        ta.chunk = s.chunk;
        ta.window = s.window;
        ta.sink = s.sink ? w.sink.as<float>() : nullptr;
        ta.exact_weights = 1;
        if (fuse_rope) {
            ta.fused_rope = 1;
            ta.rk = ra;
        }
        launches_ += launch_paged_attention_tc(ta, stream_);
    } else {
        AttnArgs at;
        at.q = q_rot_.as<float>();
        at.out = attn_.as<float>();
        at.k_pool = st.k_pool.ptr();
        at.v_pool = st.v_pool.ptr();
        at.kv_f16 = ra.kv_f16;
        at.batch = t.bd;
        at.batch.tile_lane = reinterpret_cast<int32_t*>(t.dp + g.off_tile_lane);
        at.batch.tile_row0 = reinterpret_cast<int32_t*>(t.dp + g.off_tile_row);
        at.batch.max_tiles = (int)g.tile_lane.size();
        at.q_heads = s.heads;
        at.kv_heads = s.kv_heads;
        at.d = D;
        at.block_tokens = bt;
        at.layers = 1;
        at.pool_blocks = ra.pool_blocks;
        at.scale = s.scale;
        at.softcap = s.softcap;
        at.chunk = s.chunk;
        at.window = s.window;
        at.sink = s.sink ? w.sink.as<float>() : nullptr;
        at.q_tile = attention_q_tile(s.heads, s.kv_heads);
        launch_paged_attention(at, stream_);
        ++launches_;
    }
    prof_end();
}

void MixerLm::run_parallel(const Tick& t, int run, Pending& pend, const std::vector<LmLane>& lanes) {
    const int l = runs_[(size_t)run].layer;
    RunState& st = rs_[(size_t)run];
    const AttentionSpec& s = ms_.layers[(size_t)l].attn;
    const DeltaSpec& d = ms_.layers[(size_t)l].delta;
    Layer& w = lw_[(size_t)l];
    const int T = t.T, C = ms_.width, D = w.row_width;
    RowUpdateArgs u;
    u.rows = T;
    apply_pending(u, pend, false);
    set_norm(u, w.norm1);
    u.normed = image(img_h_, w.in.ld);
    prof_begin(KC_ROW_UPDATE, (double)T * C * (8.0 + 4.0 * u.n_add + esz_), 0);
    launch_row_update(u, stream_);
    prof_end();
    const Shares y = matmul(w.in, u.normed, T, y_in_, 0);
    ++launches_;

    // ---- attention: head norms, rotation, page write, softmax, head gate
    attend(t, run, s, y, lanes);
    const RowImage img_a = image(img_a_, w.out.ld);
    prof_begin(KC_GATES, (double)T * s.heads * (D * 4.0 + s.vdim * (double)esz_), 0);
    launch_head_gate(attn_.as<float>(), T, s.heads, D, s.vdim, y, w.c_g, img_a, stream_);
    prof_end();

    // ---- gated delta rule
    DeltaPrepArgs dp;
    dp.y = y;
    dp.q_col = w.d_q;
    dp.k_col = w.d_k;
    dp.v_col = w.d_v;
    dp.a_col = w.d_a;
    dp.b_col = w.d_b;
    dp.rows = T;
    dp.heads = d.heads;
    dp.kv_heads = d.kv_heads;
    dp.dim = d.dim;
    dp.vdim = d.vdim;
    dp.taps = d.taps;
    dp.conv = w.conv.as<float>();
    dp.dt_bias = w.dt_bias.as<float>();
    dp.log_decay = w.log_decay.as<float>();
    dp.lanes = state_lanes_;
    dp.token_lane = t.bd.token_lane;
    dp.tail = st.tail.as<float>();
    dp.q = dq_.as<float>();
    dp.k = dk_.as<float>();
    dp.v = dv_.as<float>();
    dp.beta = dbeta_.as<float>();
    dp.decay = ddecay_.as<float>();
    const double channels = 2.0 * d.kv_heads * d.dim + (double)d.heads * d.vdim;
    prof_begin(KC_DELTA_PREP, 8.0 * T * channels, 0);
    launch_delta_prep(dp, stream_);
    prof_end();
    DeltaScanArgs sc;
    sc.common.lanes = state_lanes_;
    sc.common.state = st.state.as<float>();
    sc.common.heads = d.heads;
    sc.common.dim = d.dim;
    sc.common.vdim = d.vdim;
    sc.common.out = raw_.as<float>();
    sc.common.norm_w = w.head_norm.as<float>();
    sc.common.eps = ms_.eps;
    sc.common.gate = y;
    sc.common.gate_col = w.d_g;
    sc.kv_heads = d.kv_heads;
    sc.q = dp.q;
    sc.k = dp.k;
    sc.v = dp.v;
    sc.decay = dp.decay;
    sc.beta = dp.beta;
    const RowImage img_b = image(img_b_, w.out2.ld);
    const bool finish = short_lanes_ && linear_state_can_finish(d.dim, d.vdim);
    if (finish) sc.common.image = img_b;
    const double vw = (double)d.heads * d.vdim;
    prof_begin(KC_DELTA_SCAN, 4.0 * T * (channels + vw) + 8.0 * t.B * vw * d.dim, 8.0 * T * vw * d.dim);
    launch_delta_scan(sc, stream_);
    prof_end();
    launches_ += 3;
    if (!finish) {
        sc.common.image = img_b;
        prof_begin(KC_GATES, T * vw * (8.0 + esz_), 0);
        launch_head_norm_gate(sc.common, T, stream_);
        prof_end();
        ++launches_;
    }
    pend.n = 2;
    pend.y[0] = matmul(w.out, img_a, T, y_a_, 1);
    pend.y[1] = matmul(w.out2, img_b, T, y_b_, 2);
    pend.w[0] = w.out_norm.as<float>();
    pend.w[1] = w.out2_norm.as<float>();
    pend.coef = 0.5f;
}

void MixerLm::run_forward(const std::vector<LmLane>& lanes, KvReservation& r, uint32_t flags) {
    Tick t = stage_tick(lanes, r, flags);
    const int B = t.B, T = t.T, R = t.R, C = ms_.width;
    std::vector<StateLane> halves;
    int longest = 0, first_row = 0;
    for (const LmLane& l : lanes) {
        halves.push_back(StateLane{l.state_in, l.state_out, first_row, l.n_tokens});
        first_row += l.n_tokens;
        longest = std::max(longest, l.n_tokens);
    }
    longest_ = longest;
    short_lanes_ = longest <= kShortLane;
    const size_t off_halves = stage_bytes(t, halves.data(), halves.size() * sizeof(StateLane));
    if (ms_.conv_taps > 0) split_delta_lanes(t, halves);
    std::vector<int32_t> sp((size_t)B), nt((size_t)B), nb((size_t)B);
    for (int i = 0; i < B; ++i) {
        sp[(size_t)i] = lanes[(size_t)i].start_pos;
        nt[(size_t)i] = lanes[(size_t)i].n_tokens;
        nb[(size_t)i] = t.hdr[i].n_blocks;
    }
    for (Geometry& g : geo_) {
        if (g.tc) {
            plan_attention_tc(sp.data(), nt.data(), nb.data(), B, g.heads, g.kv_heads, g.plan, g.chunk, g.window);
            if (g.plan.n_entries() > attn_max_entries_) throw std::runtime_error("attention work list exceeds its scratch");
            g.off_entries = stage_bytes(t, g.plan.entries.data(), g.plan.entries.size() * 4);
            g.off_tiles = stage_bytes(t, g.plan.tiles.data(), g.plan.tiles.size() * 4);
            g.off_dec = stage_bytes(t, g.plan.dec_lanes.data(), g.plan.dec_lanes.size() * 4);
        } else {
            const int q_tile = attention_q_tile(g.heads, g.kv_heads);
            g.tile_lane.clear();
            g.tile_row.clear();
            for (int i = 0; i < B; ++i)
                for (int r0 = 0; r0 < nt[(size_t)i]; r0 += q_tile) {
                    g.tile_lane.push_back(i);
                    g.tile_row.push_back(r0);
                }
            g.off_tile_lane = stage_bytes(t, g.tile_lane.data(), g.tile_lane.size() * 4);
            g.off_tile_row = stage_bytes(t, g.tile_row.data(), g.tile_row.size() * 4);
        }
    }
    if (!latent_geo_.empty()) plan_latent(t, sp, nt, nb, r);
    upload_tick(t, 64, KC_BATCH);
    state_lanes_.lane = reinterpret_cast<const StateLane*>(t.dp + off_halves);
    state_lanes_.lanes = B;
    for (LaneSet* s : {&delta_one_, &delta_rows_, &delta_chunks_}) s->lanes.lane = reinterpret_cast<const StateLane*>(t.dp + s->off);
    // copy-on-write page copies of shared partial tails
    for (const KvCowCopy& c : r.cow_copies())
        for (size_t i = 0; i < rs_.size(); ++i) {
            RunState& st = rs_[i];
            const int l = runs_[i].layer;
            if (st.k_pool.size() == 0) continue;
            const bool latent = st.v_pool.size() == 0;  // one pool: both arguments name it
            launch_cow_copy(st.k_pool.ptr(), latent ? st.k_pool.ptr() : st.v_pool.ptr(), cfg_.kv_f16 ? 1 : 0, c.src_slot, c.dst_slot, c.rows, 1,
                            pool_->max_blocks(), latent ? 1 : ms_.layers[(size_t)l].attn.kv_heads, cfg_.block_tokens, lw_[(size_t)l].row_width, stream_);
            ++launches_;
        }
    cur_ = 0;
    if (moe_.counts > 0) {  // whatever a forward that failed half-way left of its counts
        MK_CUDA(cudaMemsetAsync(moe_.count, 0, (size_t)moe_.counts * 2 * 4, stream_));
        moe_half_ = 0;
    }
    QWeight table;
    table.type = f32_ ? QT_F32 : QT_BF16;
    table.rows = ms_.vocab;
    table.cols = C;
    table.p0 = embed_.ptr();
    prof_begin(KC_EMBED, (4.0 + esz_) * T * C, 0);
    if (ms_.sinusoid_positions) {
        EmbedNormArgs e;
        e.ids = t.ids;
        e.positions = t.bd.positions;
        e.table = embed_.ptr();
        e.table_f32 = f32_ ? 1 : 0;
        e.rows = T;
        e.width = C;
        e.freq = position_freq_.as<double>();
        e.norm_w = embed_norm_.w.as<float>();
        e.eps = ms_.eps;
        e.x = x_[cur_].as<float>();
        if (ms_.loop.times > 0) e.image = image(img_loop_, loop_in_.ld).part(loop_in_.ld / 2, loop_in_.ld / 2);
        launch_embed_norm(e, stream_);
    } else {
        launch_embed(table, t.ids, T, ms_.embedding_scale, x_[cur_].as<float>(), stream_);
    }
    prof_end();
    ++launches_;
    if (capture_) captured_.ensure(runs_.size() * T * C * 4);
    captured_tokens_ = T;

    Pending pend;
    for (int run = 0; run < (int)runs_.size(); ++run) {
        const int l = runs_[(size_t)run].layer;
        const MixerLayerSpec& s = ms_.layers[(size_t)l];
        Layer& w = lw_[(size_t)l];
        if (runs_[(size_t)run].first) begin_pass(t, runs_[(size_t)run].pass, pend);
        if (ms_.side_by_side()) run_side_by_side(t, run, pend, lanes);
        else if (ms_.norm_place == NormPlace::Output) run_output_norm(t, run, pend, lanes);
        else if (ms_.conv_taps > 0) run_conv_input(t, run, pend, lanes);
        else if (s.kind == MixerKind::Wkv) run_wkv(t, run, pend);
        else run_parallel(t, run, pend, lanes);
        if (s.ff > 0 && ms_.norm_place == NormPlace::Input) {
            RowUpdateArgs u;
            u.rows = T;
            apply_pending(u, pend, false);
            set_norm(u, w.norm2);
            u.normed = image(img_h_, w.gate_up.ld);
            prof_begin(KC_ROW_UPDATE, (double)T * C * (8.0 + 4.0 * u.n_add + esz_), 0);
            launch_row_update(u, stream_);
            prof_end();
            const RowImage img = image(img_ff_, w.down.ld);
            GatedAct act;
            act.kind = ms_.ff_kind == FfKind::GatedGelu ? GatedAct::GeluTanh : GatedAct::Silu;
            if (f32_) {
                const Shares gu = matmul(w.gate_up, u.normed, T, y_gu_, 0);
                prof_begin(KC_GATES, 12.0 * T * s.ff, 0);
                launch_gated_act(gu, T, s.ff, img, stream_, act);
                prof_end();
            } else {
                // act(gate) * up in the matmul's epilogue
                prof_begin(T <= 64 ? KC_GEMM_NARROW : KC_GEMM, (double)w.gate_up.bytes + 2.0 * T * C + 2.0 * T * s.ff, 2.0 * T * (double)w.gate_up.rows * w.gate_up.ld);
                HgemmScratch ws;
                ws.status = status_.as<int32_t>();
                launch_hgemm_tc_gated(w.gate_up.half, reinterpret_cast<const __half*>(u.normed.h), T, act, reinterpret_cast<__half*>(img.h), img.ld, ws, stream_);
                prof_end();
            }
            launches_ += 2;
            pend.n = 1;
            pend.y[0] = matmul(w.down, img, T, y_a_, 1);
        }
        if (ms_.side_dim > 0) {
            RowUpdateArgs u;
            u.rows = T;
            apply_pending(u, pend, false);
            u.raw = image(img_h_, w.side_gate.ld);
            prof_begin(KC_ROW_UPDATE, (double)T * C * (8.0 + 4.0 * u.n_add + esz_), 0);
            launch_row_update(u, stream_);
            prof_end();
            const Shares z = matmul(w.side_gate, u.raw, T, y_in_, 0);
            const RowImage img = image(img_side_, w.side_proj.ld);
            prof_begin(KC_GATES, (double)T * ms_.side_dim * (4.0 + 2.0 * esz_), 0);
            launch_side_gate(z, T, ms_.side_dim, t.ids, side_embed_.ptr(), f32_ ? 1 : 0, (int64_t)lw_.size() * ms_.side_dim, l * ms_.side_dim, img, stream_);
            prof_end();
            launches_ += 2;
            pend.n = 1;
            pend.y[0] = matmul(w.side_proj, img, T, y_a_, 1);
            pend.w[0] = w.side_norm.as<float>();
        }
        if (capture_) {
            RowUpdateArgs u;
            u.rows = T;
            apply_pending(u, pend, false);
            launch_row_update(u, stream_);
            ++launches_;
            MK_CUDA(cudaMemcpyAsync(captured_.as<float>() + (size_t)run * T * C, x_[cur_].ptr(), (size_t)T * C * 4, cudaMemcpyDeviceToDevice, stream_));
        }
    }
    if (R > 0 && (flags & (FWD_WANT_LOGITS | FWD_WANT_TOKENS))) {
        // the rows asked for: last residual add, final norm, output projection
        img_h_.ensure((size_t)R * head_.ld * esz_);
        RowUpdateArgs u;
        u.rows = R;
        u.row_index = t.out_rows;
        apply_pending(u, pend, false);
        u.x_out = nullptr;
        set_norm(u, final_norm_);
        u.normed = image(img_h_, head_.ld);
        prof_begin(KC_ROW_UPDATE, (double)R * C * (4.0 + 4.0 * u.n_add + esz_), 0);
        launch_row_update(u, stream_);
        prof_end();
        ++launches_;
        // one buffer receives the logits whatever the row count: no K shares here
        prof_begin(f32_ ? KC_F32_MATMUL : (R <= 64 ? KC_GEMM_NARROW : KC_GEMM), (double)head_.bytes + (double)esz_ * R * C + 4.0 * R * ms_.vocab,
                   2.0 * R * (double)ms_.vocab * C);
        if (f32_) {
            launch_f32_matmul(head_.f32.as<float>(), head_.rows, head_.ld, u.normed.f, R, logits_.as<float>(), ms_.vocab, 1, nullptr, stream_, 0, ms_.logit_scale, nullptr,
                              ms_.logit_softcap);
        } else {
            HgemmScratch ws;
            ws.status = status_.as<int32_t>();
            launch_hgemm_tc(head_.half, reinterpret_cast<const __half*>(u.normed.h), R, logits_.as<float>(), ms_.vocab, ms_.logit_scale, ms_.logit_softcap, ws, stream_, 1);
        }
        prof_end();
        ++launches_;
    }
    finish_tick(t, KC_SAMPLE);
}

// ---------------------------------------------------------------------------- state and taps

void MixerLm::copy_state(int from, int to) {
    MK_CUDA(cudaSetDevice(cfg_.device));
    const size_t halves = (size_t)state_slots_->capacity() * 2;
    for (RunState& st : rs_)
        for (DevBuf* b : {&st.state, &st.kept, &st.tail, &st.running_max}) {
            if (b->size() == 0) continue;
            const size_t n = b->size() / halves;
            MK_CUDA(cudaMemcpyAsync(b->as<uint8_t>() + (size_t)to * n, b->as<uint8_t>() + (size_t)from * n, n, cudaMemcpyDeviceToDevice, stream_));
        }
}

void MixerLm::capture_residuals(bool on) {
    capture_ = on;
    captured_tokens_ = 0;
}

int MixerLm::read_residuals(float* out, int64_t capacity) {
    if (!capture_ || captured_tokens_ == 0) throw std::runtime_error("no forward has left its residual stream");
    const int64_t n = (int64_t)runs_.size() * captured_tokens_ * ms_.width;
    if (out == nullptr || capacity < n) throw std::runtime_error("residual buffer needs " + std::to_string(n) + " floats");
    MK_CUDA(cudaStreamSynchronize(stream_));
    MK_CUDA(cudaMemcpy(out, captured_.ptr(), (size_t)n * 4, cudaMemcpyDeviceToHost));
    return captured_tokens_;
}

}  // namespace mk
