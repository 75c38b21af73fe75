// The executor of mixer-built decoders (mixer_spec.h): dense weights from a safetensors checkpoint, K/V pages of the layers
// that attend in the framework's paged pool, recurrent state of the layers that carry one in state slots, and the per-tick
// sequence of kernel launches.  Sessions, reservations, scheduling, sampling and read-back are those of every other model
// (PagedLm, DeviceLm, Engine).
#pragma once
#include "attention_tc.h"
#include "device_lm.h"
#include "hgemm_tc.h"
#include "linear_state.h"
#include "mixer_ops.h"
#include "mixer_spec.h"

namespace mk {

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
        int64_t bytes = 0;  // algorithmic bytes of one pass
    };
    struct Norm {
        float alpha = 1.f;
        DevBuf w, b;
    };
    // Part of a stacked matrix: `rows` rows of tensor `name`, placed from row `at` on, `step` rows apart.
    struct Part {
        std::string name;
        int rows;
        int at;
        int step = 1;
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
        DevBuf mu, w2t, w0, bonus, head_norm, kept;
        // delta rule
        DevBuf conv, dt_bias, log_decay, tail;
        DevBuf state;
        // attention
        DevBuf q_norm, k_norm, k_pool, v_pool;
        int row_width = 0;   // padded width of a head in the pools
        int geometry = 0, rope = 0;
    };
    // Layers with the same heads share a tick's attention work list.
    struct Geometry {
        int heads = 0, kv_heads = 0, row_width = 0;
        bool tc = false;
        AttnTcPlan plan;
        size_t off_tiles = 0, off_entries = 0, off_dec = 0;
        std::vector<int32_t> tile_lane, tile_row;
        size_t off_tile_lane = 0, off_tile_row = 0;
    };
    struct RopeTable {
        RotarySpec spec;
        DevBuf cos_t, sin_t;
    };
    enum KClass { KC_GEMM = 0, KC_GEMM_NARROW, KC_F32_MATMUL, KC_WKV_SCAN, KC_DELTA_SCAN, KC_ATTN, KC_ROPE_KV, KC_ROW_UPDATE, KC_DELTA_PREP, KC_WKV_DECAY,
                  KC_GATES, KC_EMBED, KC_BATCH, KC_SAMPLE, KC_COUNT };

    void load(const SafetensorsFile& f);
    void load_layer(const SafetensorsFile& f, int l);
    void upload_dense(const SafetensorsFile& f, const std::vector<Part>& parts, int64_t rows, int cols, Dense& out,
                      const std::vector<int64_t>& group_rows = {});
    void upload_f32(const std::vector<float>& v, DevBuf& out);
    void upload_norm(const SafetensorsFile& f, const std::string& name, Norm& out);
    int rope_table(const RotarySpec& r);
    int geometry_of(const AttentionSpec& a);
    void alloc_activations();
    RowImage image(DevBuf& b, int ld) const;
    Shares matmul(const Dense& W, const RowImage& x, int T, DevBuf& y, int scratch);
    void set_norm(RowUpdateArgs& a, const Norm& n) const;

    struct Pending;  // branch outputs not yet added to the residual stream
    void apply_pending(RowUpdateArgs& a, Pending& p, bool other_buffer);
    void run_wkv(const Tick& t, int l, Pending& p);
    void run_parallel(const Tick& t, int l, Pending& p, const std::vector<LmLane>& lanes);

    MixerSpec ms_;
    bool f32_ = false;
    int esz_ = 2;  // bytes of a matmul operand
    std::vector<Layer> lw_;
    DevBuf embed_, side_embed_;
    Dense head_;
    Norm final_norm_;
    std::vector<Geometry> geo_;
    std::vector<std::unique_ptr<RopeTable>> rope_;

    // activations of one tick
    DevBuf x_[2], mixes_, img_h_, img_a_, img_b_, img_ff_, img_side_;
    DevBuf y_in_, y_a_, y_b_, y_gu_, decay_, raw_, q_rot_, attn_, dq_, dk_, dv_, dbeta_, ddecay_;
    DevBuf partial_[3];
    DevBuf attn_part_o_, attn_part_ml_, attn_counters_;
    int attn_max_entries_ = 0;
    int cur_ = 0;             // which of x_ holds the residual stream
    StateLanes state_lanes_;  // of the running tick
    bool short_lanes_ = false;

    bool capture_ = false;
    DevBuf captured_;
    int captured_tokens_ = 0;
};

}  // namespace mk
