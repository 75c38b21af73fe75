// The executor of mixer-built decoders (mixer_spec.h): dense weights from a safetensors checkpoint, K/V or latent pages of the
// layers that attend in the framework's paged pool, recurrent state of the layers that carry one in state slots, and the per-tick
// sequence of kernel launches.  A looped layer has pages and state of its own for every pass.  Sessions, reservations, scheduling, sampling and read-back are those of every other model
// (PagedLm, DeviceLm, Engine).
#pragma once
#include "attention_tc.h"
#include "device_lm.h"
#include "gated_scan.h"
#include "hgemm_tc.h"
#include "latent_attention.h"
#include "linear_state.h"
#include "mixer_ops.h"
#include "mixer_spec.h"
#include "moe_rows.h"

namespace mk {

inline int pad_to(int64_t n, int m) { return (int)((n + m - 1) / m * m); }

constexpr int kShortLane = 4;  // lanes up to this many tokens: the recurrence kernels finish the head rows themselves

class MixerLm : public DeviceLm {
public:
    // `dir` holds config.json and model.safetensors.
    MixerLm(const std::string& dir, const ModelConfig& cfg);
    ~MixerLm() override;
    void capture_residuals(bool on) override;
    int read_residuals(float* out, int64_t capacity) override;

protected:
    void run_forward(const std::vector<LmLane>& lanes, KvReservation& r, uint32_t flags) override;
    void copy_state(int from, int to) override;

private:
    // A dense matrix: a bf16 image for the tensor cores, or f32 values; columns padded to `ld`.
    struct Dense {
        HalfWeight half;
        DevBuf f32;
        int64_t rows = 0;
        int ld = 0;
        int n_groups = 1;
        int group_end[kMaxRowGroups] = {};
        int group_tiles = 0;
        int64_t bytes = 0;  // algorithmic bytes of one pass
    };
    struct Norm {
        float alpha = 1.f;
        DevBuf w, b;
    };
    // Part of a stacked matrix: `rows` rows of tensor `name`, placed from row `at` on, `step` rows apart; with `block` set, runs of
    // `block` rows begin `pitch` rows apart.  Columns from `col` on, `cols` of them (0: the matrix's).  With turn_from >= 0 the rows of a
    // run from turn_from on go to turn_to on, the first turn_dims of them in an order that makes the halves' pairs (i, i + turn_dims / 2)
    // neighbours: a rotation then turns adjacent rows.
    struct Part {
        std::string name;
        int rows;
        int at;
        int step = 1;
        int col = 0, cols = 0;
        int block = 0, pitch = 0;
        int turn_from = -1, turn_to = 0, turn_dims = 0;
    };
    struct Layer {
        Norm norm1, norm2;
        Dense in;          // every projection that reads the mixer's input
        Dense out, out2;   // output projections (attention | the recurrent branch)
        Dense gate_up, down, side_gate, side_proj;
        DevBuf side_norm, out_norm, out2_norm;
        // columns of `in`'s output
        int c_q = 0, c_k = 0, c_v = 0, c_g = 0, c_low = 0;             // WKV (c_q: r) or attention
        int d_q = 0, d_k = 0, d_v = 0, d_a = 0, d_b = 0, d_g = 0;      // delta rule
        // WKV
        DevBuf mu, w2t, w0, bonus, head_norm;   // mu: also the token shift of layers with one norm
        // delta rule
        DevBuf conv, dt_bias, log_decay;
        // attention
        DevBuf q_norm, k_norm;
        int row_width = 0;   // padded width of a head (latent attention: of the cached vector) in the pools
        int geometry = 0, rope = 0;
        // latent attention: queries from their latent, queries to the key latent, values from it, expanded keys and values
        Dense uq, uk, uv, ukv;
        int c_kv = 0;         // column of the key/value latent (c_q: of the query latent)
        int q_width = 0;      // padded width of a query head
        int value_width = 0;  // columns of `row_width` that values come from
        int rot0 = 0, q_rot0 = 0, c_rot = 0;  // rotated part: its column in a page row and in a query head, its projection's column
        int mix_cols = 0;     // columns of the mixer in `out`'s input; the feed-forward's follow
        // delta rule with channel gates (columns d_q: r, d_k, d_v, d_a, d_g, c_low; w2t, w0 as WKV's)
        DevBuf a_b, w2h;
        // the short convolution in front of the mixer, [taps][width]
        DevBuf input_conv;
        // minGRU (columns c_q: z, c_v: x, c_g: g)
        DevBuf z_b, x_b;
        // feed-forward beside the mixer
        int c_ff = 0;
        DevBuf up_b, down_b, poly;
        // biases of the attention projections, a denominator term per head
        DevBuf q_b, k_b, v_b, o_b, sink;
        // mLSTM (columns c_q, c_k, c_v, c_g and these)
        int c_i = 0, c_f = 0;
        DevBuf i_b, f_b;
        // mixture of experts: router rows (the shared expert's gate behind them), gate/up and down matrices of all experts; the
        // shared expert's are gate_up and down
        Dense router, experts_gu, experts_down;
    };
    // What one execution of a layer keeps between forwards: pages, and the two halves of every state slot.
    struct RunState {
        DevBuf k_pool, v_pool;  // latent attention: k_pool only
        DevBuf state, kept, tail, running_max;
    };
    // Layers with the same heads share a tick's attention work list.
    struct Geometry {
        int heads = 0, kv_heads = 0, row_width = 0, chunk = 0, window = 0;
        bool tc = false;
        AttnTcPlan plan;
        size_t off_tiles = 0, off_entries = 0, off_dec = 0;
        std::vector<int32_t> tile_lane, tile_row;
        size_t off_tile_lane = 0, off_tile_row = 0;
    };
    // Latent-attention layers with the same kernel and grid share a tick's work list.
    struct LatentGeometry {
        int ctas = 1;        // CTAs per entry
        bool tc = false;     // tensor-core kernel
        bool wide = false;   // lanes with many tokens run on expanded keys and values
        int window = 0;
        int lanes = 0;       // wide: which of wide_
        LatentPlan plan;
        size_t off_entries = 0, off_rows = 0;
    };
    // The tick's lanes that run on expanded keys and values, of the layers with the same window.
    struct WideLanes {
        int window = 0;
        std::vector<LaneHeader> hdr;          // by lane; table_off: where block 0 would be among the expanded ones
        std::vector<int32_t> tiles, rows, blocks;
        size_t off_hdr = 0, off_tiles = 0, off_rows = 0, off_blocks = 0;
        double keys = 0, pairs = 0;           // of the profile: keys expanded, (query, key) pairs
    };
    struct RopeTable {
        RotarySpec spec;
        DevBuf cos_t, sin_t;
    };
    enum KClass { KC_GEMM = 0, KC_GEMM_NARROW, KC_F32_MATMUL, KC_WKV_SCAN, KC_DELTA_SCAN, KC_ATTN, KC_ROPE_KV, KC_ROW_UPDATE, KC_DELTA_PREP, KC_WKV_DECAY,
                  KC_LATENT_ATTN, KC_MINGRU, KC_LATENT_PREP, KC_LATENT_ROWS, KC_MLSTM_SCAN, KC_MOE_GEMM, KC_MOE_ROUTE, KC_MOE_GATHER, KC_GATES, KC_CHANNEL_GATES, KC_EMBED, KC_BATCH,
                  KC_SAMPLE, KC_COUNT };

    void load(const SafetensorsFile& f);
    void load_layer(const SafetensorsFile& f, int l);
    void load_latent(const SafetensorsFile& f, int l);
    void load_side_by_side(const SafetensorsFile& f, int l);
    void load_output_norm(const SafetensorsFile& f, int l);
    void load_moe(const SafetensorsFile& f, int l);
    void alloc_run(int run);
    void upload_dense(const SafetensorsFile& f, const std::vector<Part>& parts, int64_t rows, int cols, Dense& out,
                      const std::vector<int64_t>& group_rows = {}, double share_per_token = 1.0);
    // `groups` > 0: equal parts with an input each.  share_per_token: how much of it a token's pass reads.
    void upload_matrix(const std::vector<float>& m, int64_t rows, int ld, int64_t true_bytes, Dense& out, const std::vector<int64_t>& group_rows, int groups,
                       double share_per_token = 1.0);
    int passes_ = 1;  // how often a token's pass runs what is being loaded
    void place(const SafetensorsFile& f, const Part& p, int cols, int ld, std::vector<float>& m);
    void upload_f32(const std::vector<float>& v, DevBuf& out);
    void upload_norm(const SafetensorsFile& f, const std::string& name, Norm& out);
    int rope_table(const RotarySpec& r);
    int geometry_of(const AttentionSpec& a);
    void alloc_activations();
    RowImage image(DevBuf& b, int ld) const;
    Shares matmul(const Dense& W, const RowImage& x, int T, DevBuf& y, int scratch);
    void matmul_scatter(const Dense& W, const RowImage& x, int T, const MatmulScatter& to);
    void set_norm(RowUpdateArgs& a, const Norm& n) const;
    int latent_geometry(int ctas, bool tc, bool wide, int window);
    void plan_latent(Tick& t, const std::vector<int32_t>& start, const std::vector<int32_t>& n_tokens, const std::vector<int32_t>& n_blocks, KvReservation& r);

    // Branch outputs not yet added to the residual stream.
    struct Pending {
        int n = 0;
        Shares y[2];
        const float* w[2] = {nullptr, nullptr};
        const float* bias = nullptr;  // of a single branch
        const int32_t* routed_at = nullptr;  // of a single branch: rows of routed_ to add (see RowUpdateArgs)
        int routed_k = 0;
        float coef = 1.f;
        bool replace = false;         // they take the stream's place
    };
    void apply_pending(RowUpdateArgs& a, Pending& p, bool other_buffer);
    void run_wkv(const Tick& t, int run, Pending& p);
    void run_parallel(const Tick& t, int run, Pending& p, const std::vector<LmLane>& lanes);
    // Queries, keys and values out of the projections `y`, page write and attention: leaves the heads' outputs in attn_.
    void attend(const Tick& t, int run, const AttentionSpec& s, const Shares& y, const std::vector<LmLane>& lanes);
    // layers whose mixer reads a short convolution over its norm
    void load_conv_input(const SafetensorsFile& f, int l);
    void run_conv_input(const Tick& t, int run, Pending& p, const std::vector<LmLane>& lanes);
    void run_channel_delta(const Tick& t, int run, const Shares& y, const RowImage& out);
    void split_delta_lanes(Tick& t, const std::vector<StateLane>& lanes);
    void upload_low_rank(const SafetensorsFile& f, const std::string& prefix, int channels, int rank, Layer& w);
    // layers whose mixer and feed-forward read one norm
    void begin_pass(const Tick& t, int pass, Pending& p);
    void run_side_by_side(const Tick& t, int run, Pending& p, const std::vector<LmLane>& lanes);
    // layers whose norms sit on what the sublayers give
    void run_output_norm(const Tick& t, int run, Pending& p, const std::vector<LmLane>& lanes);
    void run_mlstm(const Tick& t, int run, const RowImage& in, const RowImage& out);
    void run_moe(const Tick& t, int layer, Pending& p);
    void run_latent(const Tick& t, int run, const Shares& y, const RowImage& out, const std::vector<LmLane>& lanes);
    void run_latent_wide(const Tick& t, int run, const Shares& y, const RowImage& out);
    void latent_prep_args(const Tick& t, int run, const Shares& y, LatentPrepArgs& p);
    int latent_qkv(const std::string& mix, const LatentSpec& s, Layer& w, std::vector<Part>& parts, int at) const;

    MixerSpec ms_;
    bool f32_ = false;
    int esz_ = 2;  // bytes of a matmul operand
    std::vector<Layer> lw_;
    std::vector<LayerRun> runs_;
    std::vector<RunState> rs_;
    DevBuf embed_, side_embed_, position_freq_, loop_step_, iota_;
    Norm embed_norm_;
    Dense head_, loop_in_;
    Norm final_norm_;
    std::vector<Geometry> geo_;
    std::vector<LatentGeometry> latent_geo_;
    std::vector<WideLanes> wide_;
    std::vector<std::unique_ptr<RopeTable>> rope_;

    // activations of one tick
    DevBuf x_[2], mixes_, img_h_, img_a_, img_b_, img_ff_, img_side_;
    DevBuf y_in_, y_a_, y_b_, y_gu_, decay_, removal_, raw_, q_rot_, attn_, dq_, dk_, dv_, dbeta_, ddecay_;
    // layers with one norm: loop entry, latents, per-head queries, queries and outputs in the latent space, mixer | feed-forward,
    // expanded keys and values (and the vectors they come from)
    DevBuf img_loop_, img_q_, img_uq_, q_lat_, img_lat_, img_cat_, wide_in_, wide_kv_;
    DevBuf lat_part_o_, lat_part_ml_, lat_counters_;
    DevBuf partial_[3];
    // mixture of experts: the tick's routing, rows grouped by expert, their activations and results
    MoeRows moe_;
    int moe_half_ = 0;  // of the counts, alternates from layer to layer
    DevBuf moe_words_, img_rows_, img_expert_ff_, routed_;
    DevBuf mlstm_counters_, img_qkv_;
    DevBuf attn_part_o_, attn_part_ml_, attn_counters_;
    int attn_max_entries_ = 0;
    int cur_ = 0;             // which of x_ holds the residual stream
    StateLanes state_lanes_;  // of the running tick
    // its lanes by the form the delta rule with channel gates takes
    struct LaneSet {
        StateLanes lanes;
        int longest = 0;
        int64_t rows = 0;
        size_t off = 0;
    };
    LaneSet delta_one_, delta_rows_, delta_chunks_;   // one token; row by row; chunks
    DevBuf delta_scratch_;
    bool short_lanes_ = false;
    int longest_ = 0;         // tokens of the longest lane

    bool capture_ = false;
    DevBuf captured_;
    int captured_tokens_ = 0;
};

}  // namespace mk
