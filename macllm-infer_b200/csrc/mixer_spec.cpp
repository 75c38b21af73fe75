// See mixer_spec.h.
#include "mixer_spec.h"
#include <algorithm>
#include <cmath>
#include <fstream>
#include <map>
#include <sstream>
#include <stdexcept>

namespace mk {

namespace {

std::map<std::string, MixerSpecReader>& readers() {
    static std::map<std::string, MixerSpecReader> all;
    return all;
}

int size_of(const Json& v, int lo = 1, int hi = 1 << 24) {
    const int64_t n = v.integer();
    if (n < lo || n > hi) throw std::runtime_error(v.where() + " is out of range");
    return (int)n;
}

RotarySpec read_rotary(const Json& mixer, int head_dim, RotaryScaling scaling = RotaryScaling::Turns, bool interleaved = true) {
    RotarySpec r;
    r.interleaved = interleaved;
    const Json* rot = mixer.find("rot");
    if (rot == nullptr || rot->is_null()) return r;
    r.dims = size_of(rot->at("dims"), 0, head_dim);
    if (r.dims % 2 != 0) throw std::runtime_error(rot->where() + ".dims must be even");
    r.base = rot->at("base").number();
    if (!(r.base > 0)) throw std::runtime_error(rot->where() + ".base must be positive");
    const Json* s = rot->find("scaling");
    if (s != nullptr && !s->is_null()) {
        if (scaling == RotaryScaling::None) throw std::runtime_error(s->where() + " is not supported here");
        r.scaling = scaling;
        r.factor = s->at("factor").number();
        r.low = s->at(scaling == RotaryScaling::Yarn ? "slow" : "low").number();
        r.high = s->at(scaling == RotaryScaling::Yarn ? "fast" : "high").number();
        r.original = s->at("original").number();
        if (!(r.factor > 0 && r.original > 0)) throw std::runtime_error(s->where() + " needs a positive factor and original context");
        if (scaling == RotaryScaling::Yarn && !(r.low > 0 && r.high > 0 && r.base != 1.0)) throw std::runtime_error(s->where() + " needs positive turns");
    }
    return r;
}

void check_groups(const Json& where, int heads, int kv_heads) {
    if (heads % kv_heads != 0) throw std::runtime_error(where.where() + ": heads must be a multiple of kv_heads");
}

// A size that only a tensor's shape gives.
int matrix_rows(const SafetensorsFile& f, const std::string& name) {
    const StTensor* t = f.find(name);
    if (t == nullptr || t->shape.size() != 2) throw std::runtime_error("tensor `" + name + "` must be a matrix");
    return (int)t->shape[0];
}

// Width of a layer's feed-forward, 0: none.
int read_dense_ff(const Json& layer) {
    const Json* mlp = layer.find("mlp");
    if (mlp == nullptr || mlp->is_null()) return 0;
    if (mlp->at("kind").str() != "dense") throw std::runtime_error(mlp->where() + ".kind `" + mlp->at("kind").str() + "` is not supported");
    return size_of(mlp->at("ff"));
}

// Sizilorn: WKV time-mixing layers and layers that run gated attention beside the gated delta rule, Dynamic Tanh norms, and
// a token input of its own for every layer.
MixerSpec read_sizilorn(const Json& c, const SafetensorsFile& f) {
    MixerSpec s;
    s.arch = "Sizilorn";
    s.vocab = size_of(c.at("vocab"));
    s.width = size_of(c.at("width"));
    s.norm = NormKind::DynTanh;
    s.eps = (float)c.at("norm").at("eps").number();
    if (!(s.eps >= 0.f)) throw std::runtime_error("config norm.eps must not be negative");
    const Json* side = c.find("token_side");
    if (side != nullptr && !side->is_null()) s.side_dim = size_of(side->at("dim"));
    const auto& layers = c.at("layers").items();
    if (layers.empty()) throw std::runtime_error("config lists no layers");
    for (size_t i = 0; i < layers.size(); ++i) {
        const Json& j = layers[i];
        const Json& m = j.at("mixer");
        const std::string type = j.at("type").str();
        MixerLayerSpec l;
        if (type == "wkv") {
            l.kind = MixerKind::Wkv;
            l.wkv.heads = size_of(m.at("heads"));
            l.wkv.dim = size_of(m.at("dim"));
            l.wkv.rank = matrix_rows(f, "l" + std::to_string(i) + ".mix.w1");
        } else if (type == "parallel") {
            l.kind = MixerKind::Parallel;
            const Json& a = m.at("left");
            l.attn.heads = size_of(a.at("heads"));
            l.attn.kv_heads = size_of(a.at("kv_heads"));
            l.attn.dim = size_of(a.at("dim"));
            l.attn.vdim = size_of(a.at("vdim"));
            l.attn.scale = (float)a.at("scale").number();
            l.attn.rot = read_rotary(a, l.attn.dim);
            check_groups(a, l.attn.heads, l.attn.kv_heads);
            const Json& d = m.at("right");
            l.delta.heads = size_of(d.at("heads"));
            l.delta.kv_heads = size_of(d.at("kv_heads"));
            l.delta.dim = size_of(d.at("dim"));
            l.delta.vdim = size_of(d.at("vdim"));
            l.delta.taps = size_of(d.at("conv"));
            check_groups(d, l.delta.heads, l.delta.kv_heads);
        } else {
            throw std::runtime_error(j.where() + ".type `" + type + "` is not a known mixer");
        }
        l.ff = read_dense_ff(j);
        s.layers.push_back(l);
    }
    return s;
}

const RegisterMixerArchitecture register_sizilorn("Sizilorn", read_sizilorn);

float number_of(const Json& v) {
    const double x = v.number();
    if (!std::isfinite(x)) throw std::runtime_error(v.where() + " must be finite");
    return (float)x;
}

// Kunonex: latent attention and minGRU layers, mixer and feed-forward side by side behind one layer norm, token shift in front
// of every mixer, sinusoidal positions, and a run of layers that is passed through several times.
MixerSpec read_kunonex(const Json& c, const SafetensorsFile&) {
    MixerSpec s;
    s.arch = "Kunonex";
    s.vocab = size_of(c.at("vocab"));
    s.width = size_of(c.at("width"));
    s.norm = NormKind::Layer;
    s.ff_kind = FfKind::Poly;
    s.norm_place = NormPlace::Shared;
    s.sinusoid_positions = true;
    s.eps = number_of(c.at("norm").at("eps"));
    if (!(s.eps >= 0.f)) throw std::runtime_error("config norm.eps must not be negative");
    s.logit_scale = number_of(c.at("logit_scale"));
    const auto& layers = c.at("layers").items();
    if (layers.empty()) throw std::runtime_error("config lists no layers");
    for (const Json& j : layers) {
        const Json& m = j.at("mixer");
        const std::string type = j.at("type").str();
        MixerLayerSpec l;
        if (type == "latent_attention") {
            l.kind = MixerKind::Latent;
            l.latent.heads = size_of(m.at("heads"));
            l.latent.dim = size_of(m.at("dim"));
            l.latent.vdim = size_of(m.at("vdim"));
            l.latent.q_rank = size_of(m.at("q_rank"));
            l.latent.kv_rank = size_of(m.at("kv_rank"));
            l.latent.scale = number_of(m.at("scale"));
        } else if (type == "mingru") {
            l.kind = MixerKind::MinGru;
            l.gru.width = size_of(m.at("width"));
        } else {
            throw std::runtime_error(j.where() + ".type `" + type + "` is not a known mixer");
        }
        l.ff = read_dense_ff(j);
        s.layers.push_back(l);
    }
    const Json* loop = c.find("loop");
    if (loop != nullptr && !loop->is_null()) {
        s.loop.start = size_of(loop->at("start"), 0, (int)layers.size() - 1);
        s.loop.stop = size_of(loop->at("stop"), s.loop.start + 1, (int)layers.size());
        s.loop.times = size_of(loop->at("times"), 1, 4096);
    }
    return s;
}

const RegisterMixerArchitecture register_kunonex("Kunonex", read_kunonex);

MoeSpec read_moe(const Json& mlp) {
    if (mlp.at("kind").str() != "moe") throw std::runtime_error(mlp.where() + ".kind `" + mlp.at("kind").str() + "` is not supported");
    auto limit = [](const Json& j) {
        const float v = number_of(j.at("limit"));
        if (!(v >= 0.f)) throw std::runtime_error(j.where() + ".limit must not be negative");
        return v;
    };
    MoeSpec m;
    const Json &r = mlp.at("router"), &e = mlp.at("expert");
    m.experts = size_of(r.at("experts"), 1, 1024);
    m.top = size_of(r.at("top"), 1, std::min(m.experts, 32));
    m.ff = size_of(e.at("ff"));
    m.limit = limit(e);
    const Json* sh = mlp.find("shared");
    if (sh != nullptr && !sh->is_null()) {
        m.shared_ff = size_of(sh->at("ff"));
        m.shared_limit = limit(*sh);
    }
    return m;
}

// Tevanex: mLSTM layers and two kinds of chunked attention over a mixture of experts, norms on what the sublayers give, layers that
// run another layer's tensors again.
MixerSpec read_tevanex(const Json& c, const SafetensorsFile&) {
    MixerSpec s;
    s.arch = "Tevanex";
    s.vocab = size_of(c.at("vocab"));
    s.width = size_of(c.at("width"));
    s.norm = NormKind::Rms;
    s.norm_place = NormPlace::Output;
    s.ff_kind = FfKind::Moe;
    s.eps = number_of(c.at("norm").at("eps"));
    if (!(s.eps >= 0.f)) throw std::runtime_error("config norm.eps must not be negative");
    s.embedding_scale = number_of(c.at("embedding").at("scale"));
    s.residual_mult = number_of(c.at("residual_mult"));
    s.logit_scale = number_of(c.at("logit_scale"));
    s.logit_softcap = number_of(c.at("logit_softcap"));
    if (!(s.logit_softcap > 0.f)) throw std::runtime_error("config.logit_softcap must be positive");
    const auto& layers = c.at("layers").items();
    if (layers.empty()) throw std::runtime_error("config lists no layers");
    for (const Json& j : layers) {
        const Json& m = j.at("mixer");
        const std::string type = j.at("type").str();
        MixerLayerSpec l;
        if (type == "mlstm") {
            l.kind = MixerKind::Mlstm;
            l.mlstm.heads = size_of(m.at("heads"));
            l.mlstm.dim = size_of(m.at("dim"));
            l.mlstm.vdim = size_of(m.at("vdim"));
            l.mlstm.gate_cap = number_of(m.at("gate_cap"));
            if (!(l.mlstm.gate_cap > 0.f)) throw std::runtime_error(m.where() + ".gate_cap must be positive");
        } else if (type == "attention" || type == "attention_2") {
            const bool capped = type == "attention_2";
            l.kind = MixerKind::Attention;
            AttentionSpec& a = l.attn;
            a.heads = size_of(m.at("heads"));
            a.kv_heads = size_of(m.at("kv_heads"));
            a.dim = size_of(m.at("dim"));
            a.vdim = size_of(m.at("vdim"));
            a.scale = number_of(m.at("scale"));
            a.chunk = size_of(m.at("mask").at("size"), 1, 1 << 30);
            a.biases = a.out_bias = true;
            a.qk_norm = QkNorm::Whole;
            a.sink = !capped;
            a.gate = capped ? OutputGate::Value : OutputGate::None;
            a.rot = read_rotary(m, a.dim, capped ? RotaryScaling::Yarn : RotaryScaling::None, capped);
            if (capped) {
                a.softcap = number_of(m.at("softcap"));
                if (!(a.softcap > 0.f)) throw std::runtime_error(m.where() + ".softcap must be positive");
            }
            check_groups(m, a.heads, a.kv_heads);
        } else {
            throw std::runtime_error(j.where() + ".type `" + type + "` is not a known mixer");
        }
        const Json* mlp = j.find("mlp");
        if (mlp != nullptr && !mlp->is_null()) {
            l.moe = read_moe(*mlp);
            l.ff = l.moe.ff;
        }
        const Json* of = j.find("weights_of");
        if (of != nullptr && !of->is_null()) l.weights_of = size_of(*of, 0, (int)layers.size() - 1);
        s.layers.push_back(l);
    }
    for (size_t i = 0; i < s.layers.size(); ++i) {
        // the layer that owns the tensors, through any number of references
        int root = (int)i;
        for (size_t steps = 0; s.layers[(size_t)root].weights_of >= 0; ++steps) {
            if (steps > s.layers.size()) throw std::runtime_error(layers[i].where() + ".weights_of goes round in a circle");
            root = s.layers[(size_t)root].weights_of;
        }
        if (root == (int)i) continue;
        const MixerLayerSpec &a = s.layers[i], &b = s.layers[(size_t)root];
        if (a.kind != b.kind || a.ff != b.ff) throw std::runtime_error(layers[i].where() + ".weights_of names a layer of another kind");
        s.layers[i] = b;
        s.layers[i].weights_of = root;
    }
    return s;
}

const RegisterMixerArchitecture register_tevanex("Tevanex", read_tevanex);

// Mamivik: a short convolution in front of every mixer, windowed attention with shared keys and values beside the delta rule with
// channel gates, and windowed latent attention with a rotated part, a sink and a gate per value.
MixerSpec read_mamivik(const Json& c, const SafetensorsFile& f) {
    MixerSpec s;
    s.arch = "Mamivik";
    s.vocab = size_of(c.at("vocab"));
    s.width = size_of(c.at("width"));
    s.norm = NormKind::Rms;
    s.one_number_norms = true;
    s.ff_kind = FfKind::GatedGelu;
    s.eps = number_of(c.at("norm").at("eps"));
    if (!(s.eps >= 0.f)) throw std::runtime_error("config norm.eps must not be negative");
    s.conv_taps = size_of(c.at("canon").at("taps"), 1, 64);
    const auto& layers = c.at("layers").items();
    if (layers.empty()) throw std::runtime_error("config lists no layers");
    for (const Json& j : layers) {
        const Json& m = j.at("mixer");
        const std::string type = j.at("type").str();
        MixerLayerSpec l;
        if (type == "parallel") {
            l.kind = MixerKind::ScaledParallel;
            l.left_scale = number_of(m.at("left_scale"));
            l.right_scale = number_of(m.at("right_scale"));
            const Json &a = m.at("left"), &d = m.at("right");
            l.attn.heads = size_of(a.at("heads"));
            l.attn.kv_heads = size_of(a.at("kv_heads"));
            check_groups(a, l.attn.heads, l.attn.kv_heads);
            l.attn.dim = size_of(a.at("dim"));
            l.attn.vdim = size_of(a.at("vdim"));
            if (l.attn.vdim != l.attn.dim) throw std::runtime_error(a.where() + ".vdim must be dim, the values being the keys");
            l.attn.scale = number_of(a.at("scale"));
            l.attn.window = size_of(a.at("mask").at("size"), 1, 1 << 30);
            l.attn.biases = l.attn.keys_are_values = true;
            l.attn.qk_norm = QkNorm::None;
            l.attn.gate = OutputGate::None;
            l.attn.rot = read_rotary(a, l.attn.dim, RotaryScaling::None, false);
            l.channel_delta.heads = size_of(d.at("heads"));
            l.channel_delta.dim = size_of(d.at("dim"));
            l.channel_delta.rank = matrix_rows(f, "l" + std::to_string(s.layers.size()) + ".mix.right.w1");
        } else if (type == "latent_attention") {
            l.kind = MixerKind::Latent;
            LatentSpec& a = l.latent;
            a.heads = size_of(m.at("heads"));
            a.dim = size_of(m.at("dim"));
            a.vdim = size_of(m.at("vdim"));
            a.q_rank = size_of(m.at("q_rank"));
            a.kv_rank = size_of(m.at("kv_rank"));
            a.scale = number_of(m.at("scale"));
            a.rot_dim = size_of(m.at("rot_dim"));
            a.rot = read_rotary(m, a.rot_dim, RotaryScaling::Yarn, false);
            a.window = size_of(m.at("mask").at("size"), 1, 1 << 30);
            a.sink = true;
            a.gate = OutputGate::Value;
        } else {
            throw std::runtime_error(j.where() + ".type `" + type + "` is not a known mixer");
        }
        l.ff = read_dense_ff(j);
        s.layers.push_back(l);
    }
    return s;
}

const RegisterMixerArchitecture register_mamivik("Mamivik", read_mamivik);

}  // namespace

RegisterMixerArchitecture::RegisterMixerArchitecture(const std::string& name, MixerSpecReader reader) { readers()[name] = std::move(reader); }

MixerSpec read_mixer_spec(const Json& config, const SafetensorsFile& f) {
    const std::string arch = config.at("architecture").str();
    auto it = readers().find(arch);
    if (it == readers().end()) throw std::runtime_error("architecture `" + arch + "` is not supported");
    return it->second(config, f);
}

MixerSpec read_mixer_spec_of(const std::string& dir, const SafetensorsFile& f) {
    std::ifstream in(dir + "/config.json", std::ios::binary);
    std::stringstream text;
    text << in.rdbuf();
    const std::string s = text.str();
    return read_mixer_spec(Json::parse(s.data(), s.size(), "config"), f);
}

std::vector<std::pair<std::string, std::vector<int64_t>>> mixer_tensors(const MixerSpec& s) {
    std::vector<std::pair<std::string, std::vector<int64_t>>> out;
    const int64_t C = s.width, V = s.vocab;
    auto add = [&](const std::string& name, std::vector<int64_t> shape) { out.emplace_back(name, std::move(shape)); };
    auto norm = [&](const std::string& name) {
        if (s.one_number_norms) add(name, {});
        else add(name, {C});
        if (s.norm == NormKind::DynTanh) {
            add(name + ".b", {C});
            add(name + ".alpha", {});
        }
    };
    add("embed", {V, C});
    if (s.sinusoid_positions) norm("embed.norm");
    if (s.loop.times > 0) {
        add("loop.in", {C, 2 * C});
        add("loop.step", {s.loop.times, C});
    }
    if (s.side_dim > 0) add("side.embed", {V, (int64_t)s.layers.size() * s.side_dim});
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const MixerLayerSpec& l = s.layers[i];
        if (l.weights_of >= 0) continue;
        const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.";
        norm(p + "norm1");
        if (l.kind == MixerKind::Wkv) {
            const int64_t H = l.wkv.heads, D = l.wkv.dim, n = H * D, r = l.wkv.rank;
            for (const char* x : {"r", "k", "v", "g", "w"}) add(m + "mu." + x, {C});
            for (const char* x : {"r", "k", "v", "g"}) add(m + x, {n, C});
            add(m + "w1", {r, C});
            add(m + "w2", {n, r});
            add(m + "w0", {n});
            add(m + "u", {H, D});
            add(m + "norm", {n});
            add(m + "o", {C, n});
        } else if (l.kind == MixerKind::Latent) {
            const LatentSpec& a = l.latent;
            const int64_t kw = (int64_t)a.heads * a.dim, vw = (int64_t)a.heads * a.vdim;
            add(m + "dq", {a.q_rank, C});
            add(m + "dq.norm", {a.q_rank});
            add(m + "uq", {(int64_t)a.heads * (a.dim + a.rot_dim), a.q_rank});
            add(m + "dkv", {a.kv_rank + a.rot_dim, C});
            add(m + "dkv.norm", {a.kv_rank});
            add(m + "uk", {kw, a.kv_rank});
            add(m + "uv", {vw, a.kv_rank});
            if (a.sink) add(m + "sink", {a.heads});
            if (a.gate != OutputGate::None) add(m + "g", {a.gate == OutputGate::Value ? vw : (int64_t)a.heads, C});
            add(m + "o", {C, vw});
        } else if (l.kind == MixerKind::MinGru) {
            const int64_t n = l.gru.width;
            for (const char* x : {"z", "x"}) {
                add(m + x, {n, C});
                add(m + x + ".b", {n});
            }
            add(m + "g", {n, C});
            add(m + "o", {C, n});
        } else if (l.kind == MixerKind::Mlstm) {
            const MlstmSpec& x = l.mlstm;
            const int64_t kw = (int64_t)x.heads * x.dim, vw = (int64_t)x.heads * x.vdim;
            add(m + "q", {kw, C});
            add(m + "k", {kw, C});
            add(m + "v", {vw, C});
            add(m + "g", {vw, C});
            for (const char* gate : {"i", "f"}) {
                add(m + gate, {x.heads, C});
                add(m + gate + ".b", {x.heads});
            }
            add(m + "norm", {vw});
            add(m + "o", {C, vw});
        } else if (l.kind == MixerKind::Attention) {
            const AttentionSpec& a = l.attn;
            const int64_t qw = (int64_t)a.heads * a.dim, kw = (int64_t)a.kv_heads * a.dim, vw = (int64_t)a.kv_heads * a.vdim, ow = (int64_t)a.heads * a.vdim;
            auto linear = [&](const char* name, int64_t rows, int64_t cols) {
                add(m + name, {rows, cols});
                if (a.biases) add(m + name + ".b", {rows});
            };
            linear("q", qw, C);
            linear("k", kw, C);
            linear("v", vw, C);
            add(m + "o", {C, ow});
            if (a.out_bias) add(m + "o.b", {C});
            add(m + "q.norm", {a.qk_norm == QkNorm::Whole ? qw : a.dim});
            add(m + "k.norm", {a.qk_norm == QkNorm::Whole ? kw : a.dim});
            if (a.sink) add(m + "sink", {a.heads});
            if (a.gate != OutputGate::None) add(m + "g", {a.gate == OutputGate::Value ? ow : (int64_t)a.heads, C});
        } else if (l.kind == MixerKind::ScaledParallel) {
            const AttentionSpec& a = l.attn;
            const ChannelDeltaSpec& d = l.channel_delta;
            const int64_t qw = (int64_t)a.heads * a.dim, kw = (int64_t)a.kv_heads * a.dim, n = (int64_t)d.heads * d.dim;
            add(m + "left.q", {qw, C});
            add(m + "left.q.b", {qw});
            add(m + "left.k", {kw, C});
            add(m + "left.k.b", {kw});
            add(m + "left.o", {C, (int64_t)a.heads * a.vdim});
            for (const char* x : {"r", "k", "v", "g", "a"}) add(m + "right." + x, {n, C});
            add(m + "right.a.b", {n});
            add(m + "right.w1", {d.rank, C});
            add(m + "right.w2", {n, d.rank});
            add(m + "right.w0", {n});
            add(m + "right.norm", {n});
            add(m + "right.o", {C, n});
        } else {
            const AttentionSpec& a = l.attn;
            const DeltaSpec& d = l.delta;
            const int64_t qw = (int64_t)a.heads * a.dim, kw = (int64_t)a.kv_heads * a.dim, vw = (int64_t)a.kv_heads * a.vdim;
            add(m + "left.q", {qw, C});
            add(m + "left.k", {kw, C});
            add(m + "left.v", {vw, C});
            add(m + "left.g", {a.heads, C});
            add(m + "left.q.norm", {a.dim});
            add(m + "left.k.norm", {a.dim});
            add(m + "left.o", {C, (int64_t)a.heads * a.vdim});
            add(m + "left.out", {C});
            const int64_t dk = (int64_t)d.kv_heads * d.dim, dv = (int64_t)d.heads * d.vdim;
            add(m + "right.q", {dk, C});
            add(m + "right.k", {dk, C});
            add(m + "right.v", {dv, C});
            add(m + "right.q.conv", {dk, d.taps});
            add(m + "right.k.conv", {dk, d.taps});
            add(m + "right.v.conv", {dv, d.taps});
            for (const char* x : {"a", "b"}) add(m + "right." + x, {d.heads, C});
            for (const char* x : {"A_log", "dt_bias"}) add(m + "right." + x, {d.heads});
            add(m + "right.g", {dv, C});
            add(m + "right.norm", {d.vdim});
            add(m + "right.o", {C, dv});
            add(m + "right.out", {C});
        }
        if (s.side_by_side()) add(p + "shift", {C});
        if (s.conv_taps > 0) add(p + "canon1", {C, s.conv_taps});
        if (l.ff > 0 && s.ff_kind == FfKind::Moe) {
            norm(p + "norm2");
            auto expert = [&](const std::string& name, int64_t ff) {
                add(name + ".gate", {ff, C});
                add(name + ".up", {ff, C});
                add(name + ".down", {C, ff});
            };
            for (int e = 0; e < l.moe.experts; ++e) expert(p + "mlp.e" + std::to_string(e), l.moe.ff);
            add(p + "mlp.router", {l.moe.experts, C});
            if (l.moe.shared_ff > 0) {
                expert(p + "mlp.shared", l.moe.shared_ff);
                add(p + "mlp.shared.sg", {1, C});
            }
        } else if (l.ff > 0) {
            if (!s.side_by_side()) norm(p + "norm2");
            if (s.ff_kind != FfKind::Poly) add(p + "mlp.gate", {l.ff, C});
            add(p + "mlp.up", {l.ff, C});
            add(p + "mlp.down", {C, l.ff});
            if (s.ff_kind == FfKind::Poly) {
                add(p + "mlp.up.b", {l.ff});
                add(p + "mlp.down.b", {C});
                add(p + "mlp.act", {4});
            }
        }
        if (s.side_dim > 0) {
            add(p + "side.gate", {s.side_dim, C});
            add(p + "side.proj", {C, s.side_dim});
            add(p + "side.norm", {C});
        }
    }
    norm("final.norm");
    add("head", {V, C});
    return out;
}

std::vector<LayerRun> MixerSpec::runs() const {
    std::vector<LayerRun> out;
    const int n = (int)layers.size();
    for (int l = 0; l < n;) {
        if (loop.times == 0 || l != loop.start) {
            const int of = layers[(size_t)l].weights_of;
            out.push_back(LayerRun{of >= 0 ? of : l, -1, false});
            ++l;
            continue;
        }
        for (int pass = 0; pass < loop.times; ++pass)
            for (int i = loop.start; i < loop.stop; ++i) out.push_back(LayerRun{i, pass, i == loop.start});
        l = loop.stop;
    }
    return out;
}

MixerAudit validate_mixer_tensors(const MixerSpec& s, const SafetensorsFile& f) {
    MixerAudit a;
    a.tensors_in_file = (int64_t)f.tensors().size();
    for (const auto& t : mixer_tensors(s)) {
        a.parameters += f.require(t.first, t.second).elements();
        ++a.tensors_read;
    }
    return a;
}

std::vector<double> rotary_frequencies(const RotarySpec& r) {
    std::vector<double> f((size_t)(r.dims / 2));
    const double two_pi = 2.0 * std::acos(-1.0);
    double first = 0.0, span = 1.0;  // Yarn: the pair from which frequencies are stretched, and over how many pairs
    if (r.scaling == RotaryScaling::Yarn) {
        auto pair_that_turns = [&](double turns) { return r.dims * std::log(r.original / (two_pi * turns)) / (2.0 * std::log(r.base)); };
        first = std::max(std::floor(pair_that_turns(r.high)), 0.0);
        span = std::max(std::min(std::ceil(pair_that_turns(r.low)), r.dims - 1.0) - first, 0.001);
    }
    for (int i = 0; i < r.dims / 2; ++i) {
        double v = std::pow(r.base, -2.0 * i / r.dims);
        if (r.scaling == RotaryScaling::Yarn) {
            const double stretched = std::min(std::max((i - first) / span, 0.0), 1.0);
            v = v / r.factor * stretched + v * (1.0 - stretched);
        } else if (r.scaling == RotaryScaling::Turns) {
            const double wavelength = two_pi / v;
            if (wavelength > r.original / r.low) {
                v /= r.factor;
            } else if (!(wavelength < r.original / r.high)) {
                const double s = (r.original / wavelength - r.low) / (r.high - r.low);
                v = (1.0 - s) * v / r.factor + s * v;
            }
        }
        f[(size_t)i] = v;
    }
    return f;
}

double rotary_amplitude(const RotarySpec& r) { return r.scaling == RotaryScaling::Yarn ? 0.1 * std::log(r.factor) + 1.0 : 1.0; }

}  // namespace mk
