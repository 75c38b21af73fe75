// Decoders described layer by layer by a config.json: every layer names its sequence mixer, that mixer's sizes and its
// feed-forward.  The reader of one architecture turns its config.json into this description; the executor (mixer_lm.h) and
// the kernels see nothing else of it.
#pragma once
#include "json.h"
#include "safetensors_file.h"
#include <functional>
#include <string>
#include <vector>

namespace mk {

enum class NormKind { None, DynTanh, Layer, Rms };

// How the frequencies of long wavelengths are divided by `factor`, by the turns a pair makes over the original context.
//   Turns: below `low` turns whole, above `high` not at all, in between blended by the number of turns.
//   Yarn:  the same between the pairs that turn `high` and `low` times, blended by the pair's index; cosine and sine are
//          multiplied by 0.1 ln(factor) + 1.
enum class RotaryScaling { None, Turns, Yarn };

// Rotary positions on the first `dims` dimensions of a head; dims = 0: none.
struct RotarySpec {
    int dims = 0;
    double base = 10000.0;
    bool interleaved = true;  // pairs (2i, 2i + 1); false: (i, i + dims / 2)
    RotaryScaling scaling = RotaryScaling::None;
    double factor = 1.0, low = 1.0, high = 1.0, original = 1.0;
    // the same angles and amplitude (the layout of the pairs aside)
    bool same_table(const RotarySpec& o) const {
        return dims == o.dims && base == o.base && scaling == o.scaling &&
               (scaling == RotaryScaling::None || (factor == o.factor && low == o.low && high == o.high && original == o.original));
    }
};
// The frequency of every pair, in radians per position.
std::vector<double> rotary_frequencies(const RotarySpec& r);
// What cosine and sine are multiplied by.
double rotary_amplitude(const RotarySpec& r);

enum class OutputGate { None, Head, Value };     // a sigmoid gate per head, or per value, on what attention gives
enum class QkNorm { None, Head, Whole };         // RMS norm of queries and keys per head, or over all heads at once

// Grouped-query attention; query / key RMS norm before the rotation.
struct AttentionSpec {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 1.f;
    float softcap = 0.f;      // scores pass through softcap * tanh(. / softcap); 0: as they are
    int chunk = 0;            // a position sees the keys of its own chunk only, chunks counted from position 0; 0: all before it
    int window = 0;           // a position sees itself and the window - 1 keys before it; 0: all before it
    bool sink = false;        // one learned term per head in the softmax denominator
    bool biases = false;      // of the query, key and value projections
    bool out_bias = false;    // of the output projection
    bool keys_are_values = false;  // no value projection: the values are the keys before their rotation
    QkNorm qk_norm = QkNorm::Head;
    OutputGate gate = OutputGate::Head;
    RotarySpec rot;
};

// Gated delta rule behind a short causal convolution; head h reads query / key head h / (heads / kv_heads).
struct DeltaSpec {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 1;
};

// Time mixing with a data-dependent decay per key channel and a bonus for the current token.
struct WkvSpec {
    int heads = 0, dim = 0, rank = 0;  // rank of the decay's low-rank projection
};

// The delta rule with a decay and a removal rate per key channel (see ChannelDeltaArgs); square heads.
struct ChannelDeltaSpec {
    int heads = 0, dim = 0, rank = 0;  // rank of the decay's low-rank projection
};

// Attention whose keys and values are two projections of one cached vector of `kv_rank` values per token; queries come from a
// latent of `q_rank` values.  With rot_dim > 0 queries have that many dimensions more per head, and a token has one more key part
// of that width, shared by the heads and cached beside the vector; these dimensions turn with the position, the others do not.
struct LatentSpec {
    int heads = 0, dim = 0, vdim = 0, q_rank = 0, kv_rank = 0;
    float scale = 1.f;
    int rot_dim = 0;
    RotarySpec rot;                      // of the rot_dim dimensions
    int window = 0;                      // as AttentionSpec's
    bool sink = false;
    OutputGate gate = OutputGate::Head;
};

// Element-wise gated recurrence over `width` channels whose gates read the current token only.
struct MinGruSpec {
    int width = 0;
};

// Matrix memory with exponential gates: a log input and a log forget gate per head, held within +-gate_cap, and a running maximum
// that keeps the state in range.
struct MlstmSpec {
    int heads = 0, dim = 0, vdim = 0;
    float gate_cap = 1.f;
};

// Mixture of experts: the `top` experts with the largest sigmoid scores, each reading score * row; gate and up rows held within a
// limit.  A shared expert with a sigmoid gate per token runs beside them (shared_ff = 0: none).
struct MoeSpec {
    int experts = 0, top = 0, ff = 0, shared_ff = 0;
    float limit = 0.f, shared_limit = 0.f;
};

// Parallel: attention and the gated delta rule side by side.  ScaledParallel: attention and the delta rule with channel gates side by
// side, each branch times a constant.
enum class MixerKind { Wkv, Parallel, Latent, MinGru, Mlstm, Attention, ScaledParallel };

// silu(gate) * up; gelu(gate) * up; a cubic of up, every power over its own root mean square; experts
enum class FfKind { Gated, GatedGelu, Poly, Moe };

// Where a layer's norms sit.  Input: in front of the mixer and of the feed-forward.  Shared: one in front of both, which read the
// same row side by side; the mixer's input is mixed with the previous token's normed row (token shift).  Output: on what the mixer
// and the feed-forward give, which read the stream itself.
enum class NormPlace { Input, Shared, Output };

struct MixerLayerSpec {
    MixerKind kind = MixerKind::Wkv;
    WkvSpec wkv;
    AttentionSpec attn;
    DeltaSpec delta;
    LatentSpec latent;
    MinGruSpec gru;
    MlstmSpec mlstm;
    ChannelDeltaSpec channel_delta;
    float left_scale = 1.f, right_scale = 1.f;  // ScaledParallel
    int ff = 0;  // width of the feed-forward (of one expert), 0: the layer has none
    MoeSpec moe;
    int weights_of = -1;  // >= 0: the layer has no tensors and runs that layer's, with a cache and a state of its own
};

// Layers start .. stop - 1 run `times` times in a row, every pass with a cache and a state of its own.  A pass begins with
// x <- W_in [x; x0] + step[pass], x0 being the embedding output.
struct LoopSpec {
    int start = 0, stop = 0, times = 0;  // times = 0: no loop
};

// One execution of a layer: pass < 0 outside of the loop; first: the layer a pass begins with.  `layer` owns the tensors.
struct LayerRun {
    int layer = 0, pass = -1;
    bool first = false;
};

struct MixerSpec {
    std::string arch;
    int vocab = 0, width = 0, side_dim = 0;
    float eps = 1e-6f;
    NormKind norm = NormKind::DynTanh;
    FfKind ff_kind = FfKind::Gated;
    NormPlace norm_place = NormPlace::Input;
    bool side_by_side() const { return norm_place == NormPlace::Shared; }
    bool one_number_norms = false;    // a norm has one weight for all channels
    int conv_taps = 0;                // > 0: the mixers read h + conv(h), a causal convolution per channel behind norm1 (NormPlace::Input)
    bool sinusoid_positions = false;  // added to the embedding, which a norm then follows
    float embedding_scale = 1.f;
    float residual_mult = 1.f;        // of every sublayer's output (NormPlace::Output)
    float logit_scale = 1.f, logit_softcap = 0.f;  // logits <- softcap * tanh(scale * logits / softcap), 0: scale only
    LoopSpec loop;
    std::vector<MixerLayerSpec> layers;
    std::vector<LayerRun> runs() const;  // in the order of execution
};

// Reads `config` (and sizes that only the tensors know) for the architecture it names.
MixerSpec read_mixer_spec(const Json& config, const SafetensorsFile& f);

// Every tensor the executor reads, with its shape.
std::vector<std::pair<std::string, std::vector<int64_t>>> mixer_tensors(const MixerSpec& s);

struct MixerAudit {
    int64_t tensors_in_file = 0, tensors_read = 0, parameters = 0;
};
// Every tensor of the spec present, floating-point and of the expected shape; throws on the first that is not.  Host only, run
// before any device memory is touched.  Tensors the spec does not know are left unread.
MixerAudit validate_mixer_tensors(const MixerSpec& s, const SafetensorsFile& f);

// Reads <dir>/config.json for the checkpoint in `dir`.
MixerSpec read_mixer_spec_of(const std::string& dir, const SafetensorsFile& f);

using MixerSpecReader = std::function<MixerSpec(const Json& config, const SafetensorsFile& f)>;
struct RegisterMixerArchitecture {
    RegisterMixerArchitecture(const std::string& name, MixerSpecReader reader);
};

}  // namespace mk
