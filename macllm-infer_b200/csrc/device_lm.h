// What every model on the GPU does around its layers, whatever those are: the stream and its timing events, the pinned
// staging of a tick (lane headers, block tables, token ids, chosen rows, sampling settings and the model's own work lists, in
// one copy), the batch descriptor built from it, token selection from the logits, the way back to the host, and the
// per-kernel-class profile.
#pragma once
#include "device_util.h"
#include "kernels.h"
#include "model_config.h"
#include "paged_lm.h"

namespace mk {

class DeviceLm : public PagedLm {
public:
    ~DeviceLm() override;
    bool device_sampling_covers(float temperature, int top_k) const override { return mk::device_sampling_covers(temperature, top_k, spec_.vocab); }
    float last_forward_ms() const override;
    int64_t launch_count() const override { return launches_; }
    int64_t h2d_bytes() const override { return h2d_bytes_; }
    int64_t d2h_bytes() const override { return d2h_bytes_; }
    void profile_enable(bool on) override;
    std::vector<KernelProfile> profile_query() override;

protected:
    // `profile_classes`: names of the kernel classes prof_begin counts under, in the order of the model's enum.
    DeviceLm(const ModelConfig& cfg, const std::vector<const char*>& profile_classes);
    // Selects the device (throws when there is none: no CPU fallback) and creates the stream and events.
    void open_device();
    // Buffers of a tick: call once the pool exists.  `extra_stage_bytes` is what the model stages on top.
    void alloc_tick(size_t extra_stage_bytes);

    struct Tick {
        int B = 0, T = 0, R = 0;  // lanes, tokens, rows projected to logits
        uint32_t flags = 0;
        uint8_t* hp = nullptr;    // host staging
        uint8_t* dp = nullptr;    // its device copy
        size_t bytes = 0;         // staged so far
        const LaneHeader* hdr = nullptr;  // host copy
        size_t off_tables = 0, off_ids = 0, off_rows = 0, off_sampling = 0;
        BatchDesc bd;
        const uint32_t* ids = nullptr;          // device, after upload_tick
        const int32_t* out_rows = nullptr;      // device: packed index of every row projected to logits [R]
    };
    Tick stage_tick(const std::vector<LmLane>& lanes, KvReservation& r, uint32_t flags);
    // Appends to the staging buffer; returns the offset (16-byte aligned).
    size_t stage_bytes(Tick& t, const void* src, size_t bytes);
    // Starts the tick's clock, copies the staging buffer and expands the batch descriptor.
    void upload_tick(Tick& t, int q_tile, int prof_class);
    // Selects tokens from logits_ (FWD_WANT_TOKENS) and sends the results to pinned memory.
    void finish_tick(const Tick& t, int prof_class);
    void fetch_output(float* logits, uint32_t* tokens) override;
    void device_synchronize() override;
    // Message of a non-zero status word left by a kernel.
    virtual std::string status_message(int32_t status) const;

    void prof_begin(int cls, double bytes, double flops);
    void prof_end();

    ModelConfig cfg_;
    cudaStream_t stream_ = nullptr;
    int64_t launches_ = 0, h2d_bytes_ = 0, d2h_bytes_ = 0;
    bool profiling_ = false;
    DevBuf cu_, pos_, tok_lane_, slots_, last_, tile_lane_, tile_row_, ntiles_, err_;
    DevBuf logits_, tokens_;
    DevBuf status_;  // one word: non-zero when a bounded wait or a device-side check gave up

private:
    void prof_resolve();
    cudaEvent_t ev_start_ = nullptr, ev_stop_ = nullptr;
    bool timed_ = false;
    // profiling: one event pair per launch group, resolved after the tick's barrier
    struct ProfSpan { int cls; double bytes, flops; cudaEvent_t a, b; };
    std::vector<ProfSpan> spans_;
    std::vector<cudaEvent_t> event_pool_;
    std::vector<const char*> prof_names_;
    std::vector<KernelProfile> prof_;
    PinnedBuf stage_host_, out_host_;
    DevBuf stage_dev_, argmax_scratch_;
    int out_lanes_ = 0, out_rows_ = 0;
    uint32_t out_flags_ = 0;
};

}  // namespace mk
