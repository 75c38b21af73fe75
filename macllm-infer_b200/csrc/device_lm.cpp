// See device_lm.h.  Line references are into the reference's sources.
#include "device_lm.h"
#include <cstring>

namespace mk {

DeviceLm::DeviceLm(const ModelConfig& cfg, const std::vector<const char*>& profile_classes) : cfg_(cfg), prof_names_(profile_classes) {}

DeviceLm::~DeviceLm() {
    if (stream_) cudaStreamSynchronize(stream_);
    for (ProfSpan& sp : spans_) {
        cudaEventDestroy(sp.a);
        cudaEventDestroy(sp.b);
    }
    for (cudaEvent_t e : event_pool_) cudaEventDestroy(e);
    if (ev_start_) cudaEventDestroy(ev_start_);
    if (ev_stop_) cudaEventDestroy(ev_stop_);
    if (stream_) cudaStreamDestroy(stream_);
}

void DeviceLm::open_device() {
    int ndev = 0;
    if (cudaGetDeviceCount(&ndev) != cudaSuccess || ndev <= 0) {
        cudaGetLastError();
        throw std::runtime_error("no usable CUDA device: this library has no CPU fallback");
    }
    if (cfg_.device < 0 || cfg_.device >= ndev) throw std::runtime_error("device ordinal out of range");
    MK_CUDA(cudaSetDevice(cfg_.device));
    MK_CUDA(cudaStreamCreateWithFlags(&stream_, cudaStreamNonBlocking));
    MK_CUDA(cudaEventCreate(&ev_start_));
    MK_CUDA(cudaEventCreate(&ev_stop_));
    status_.alloc(4);
    status_.zero(stream_);
}

void DeviceLm::alloc_tick(size_t extra_stage_bytes) {
    const int T = cfg_.max_batch_tokens, B = cfg_.max_batch_lanes;
    cu_.alloc((size_t)(B + 1) * 4);
    pos_.alloc((size_t)T * 4);
    tok_lane_.alloc((size_t)T * 4);
    slots_.alloc((size_t)T * 8);
    last_.alloc((size_t)B * 4);
    tile_lane_.alloc((size_t)(T + B) * 4);
    tile_row_.alloc((size_t)(T + B) * 4);
    ntiles_.alloc(4);
    err_.alloc(4);
    err_.zero(stream_);
    logits_.alloc((size_t)B * spec_.vocab * 4);
    tokens_.alloc((size_t)B * 4);
    argmax_scratch_.alloc(argmax_scratch_bytes(B));
    argmax_scratch_.zero(stream_);
    const size_t bytes = (size_t)B * sizeof(LaneHeader) + (size_t)(pool_->max_blocks() + B) * 4 + (size_t)T * 8 + 128 +
                         (size_t)B * sizeof(LaneSampling) + extra_stage_bytes;
    stage_host_.ensure(bytes);
    stage_dev_.alloc(bytes);
    out_host_.ensure((size_t)B * spec_.vocab * 4 + (size_t)B * 4 + 16);
}

DeviceLm::Tick DeviceLm::stage_tick(const std::vector<LmLane>& lanes, KvReservation& r, uint32_t flags) {
    MK_CUDA(cudaSetDevice(cfg_.device));
    Tick t;
    t.B = (int)lanes.size();
    t.flags = flags;
    bool chosen_rows = false;
    for (const LmLane& l : lanes) {
        t.T += l.n_tokens;
        t.R += l.rows_out();
        chosen_rows |= l.logit_rows != nullptr;
    }
    if (t.B > cfg_.max_batch_lanes) throw std::runtime_error("batch has more lanes than max_batch_lanes");
    if (t.T > cfg_.max_batch_tokens) throw std::runtime_error("batch has more tokens than max_batch_tokens");
    t.hp = stage_host_.as<uint8_t>();
    t.dp = stage_dev_.as<uint8_t>();
    // the per-lane headers, block tables and token ids
    LaneHeader* hdr = reinterpret_cast<LaneHeader*>(t.hp);
    t.hdr = hdr;
    t.off_tables = (size_t)t.B * sizeof(LaneHeader);
    uint32_t* tab = reinterpret_cast<uint32_t*>(t.hp + t.off_tables);
    int n_tab = 0;
    for (int i = 0; i < t.B; ++i) {
        const std::vector<KvBlockId>& blocks = r.lane_blocks((size_t)i);
        hdr[i].start_pos = lanes[(size_t)i].start_pos;
        hdr[i].n_tokens = lanes[(size_t)i].n_tokens;
        hdr[i].table_off = n_tab;
        hdr[i].n_blocks = (int32_t)blocks.size();
        for (const KvBlockId& b : blocks) tab[n_tab++] = b.slot;
    }
    t.off_ids = t.off_tables + (size_t)n_tab * 4;
    uint32_t* ids = reinterpret_cast<uint32_t*>(t.hp + t.off_ids);
    int tpos = 0;
    for (const LmLane& l : lanes) {
        memcpy(ids + tpos, l.ids, (size_t)l.n_tokens * 4);
        tpos += l.n_tokens;
    }
    t.bytes = t.off_ids + (size_t)t.T * 4;
    // rows projected to logits, when they are not simply every lane's last one
    if (chosen_rows) {
        std::vector<int32_t> rows;
        int base = 0;
        for (const LmLane& l : lanes) {
            if (l.logit_rows == nullptr) rows.push_back(base + l.n_tokens - 1);
            else for (int i = 0; i < l.n_logit_rows; ++i) rows.push_back(base + l.logit_rows[i]);
            base += l.n_tokens;
        }
        t.off_rows = rows.empty() ? 0 : stage_bytes(t, rows.data(), rows.size() * 4);
    }
    // per-lane sampling settings, only when some lane does not take the plain argmax
    bool any_stochastic = false;
    for (const LmLane& l : lanes) any_stochastic |= l.temperature > 0.f;
    if (any_stochastic && (flags & FWD_WANT_TOKENS)) {
        std::vector<LaneSampling> sp;
        for (const LmLane& l : lanes) {
            if (!device_sampling_covers(l.temperature, l.top_k))
                throw std::runtime_error("the device sampler covers greedy selection and 1 <= top_k <= 1024");
            sp.push_back(LaneSampling{l.temperature, l.top_k, l.top_p, l.u});
        }
        t.off_sampling = stage_bytes(t, sp.data(), sp.size() * sizeof(LaneSampling));
    }
    // room for the results
    if (flags & FWD_WANT_LOGITS) {
        logits_.ensure((size_t)t.R * spec_.vocab * 4);
        out_host_.ensure((size_t)t.R * spec_.vocab * 4 + (size_t)t.B * 4 + 16);
    }
    return t;
}

size_t DeviceLm::stage_bytes(Tick& t, const void* src, size_t bytes) {
    const size_t at = (t.bytes + 15) / 16 * 16;
    if (at + bytes > stage_host_.size() || at + bytes > stage_dev_.size()) throw std::runtime_error("tick staging buffer is too small");
    if (bytes) memcpy(t.hp + at, src, bytes);
    t.bytes = at + bytes;
    return at;
}

void DeviceLm::upload_tick(Tick& t, int q_tile, int prof_class) {
    if (t.bytes > stage_dev_.size()) throw std::runtime_error("tick staging buffer is too small");
    MK_CUDA(cudaEventRecord(ev_start_, stream_));
    MK_CUDA(cudaMemcpyAsync(stage_dev_.ptr(), t.hp, t.bytes, cudaMemcpyHostToDevice, stream_));
    h2d_bytes_ += (int64_t)t.bytes;
    int tiles = 0;
    for (int i = 0; i < t.B; ++i) tiles += (t.hdr[i].n_tokens + q_tile - 1) / q_tile;
    BatchDesc& bd = t.bd;
    bd.lanes = t.B;
    bd.T = t.T;
    bd.max_tiles = tiles;
    bd.hdr = reinterpret_cast<const LaneHeader*>(t.dp);
    bd.tables = reinterpret_cast<const uint32_t*>(t.dp + t.off_tables);
    bd.cu_seqlens = cu_.as<int32_t>();
    bd.positions = pos_.as<int32_t>();
    bd.token_lane = tok_lane_.as<int32_t>();
    bd.slots = slots_.as<int64_t>();
    bd.last_index = last_.as<int32_t>();
    bd.tile_lane = tile_lane_.as<int32_t>();
    bd.tile_row0 = tile_row_.as<int32_t>();
    bd.n_tiles = ntiles_.as<int32_t>();
    bd.error_flag = err_.as<int32_t>();
    prof_begin(prof_class, 0, 0);
    launch_build_batch(bd, pool_->block_tokens(), q_tile, stream_);
    prof_end();
    ++launches_;
    t.ids = reinterpret_cast<const uint32_t*>(t.dp + t.off_ids);
    t.out_rows = t.off_rows != 0 ? reinterpret_cast<const int32_t*>(t.dp + t.off_rows) : bd.last_index;
}

void DeviceLm::finish_tick(const Tick& t, int prof_class) {
    const int B = t.B;
    if (t.flags & FWD_WANT_TOKENS) {
        prof_begin(prof_class, 4.0 * B * spec_.vocab, 0);
        if (t.off_sampling != 0)
            launch_sample(logits_.as<float>(), B, spec_.vocab, reinterpret_cast<const LaneSampling*>(t.dp + t.off_sampling), tokens_.as<uint32_t>(),
                          status_.as<int32_t>(), stream_);
        else
            launch_argmax(logits_.as<float>(), B, spec_.vocab, tokens_.as<uint32_t>(), argmax_scratch_.ptr(), stream_);
        prof_end();
        ++launches_;
    }
    // results travel to pinned host memory on the same stream; the barrier is in fetch_output
    uint8_t* oh = out_host_.as<uint8_t>();
    const size_t tok_off = (size_t)((t.flags & FWD_WANT_LOGITS) ? t.R : 0) * spec_.vocab * 4;
    if (tok_off) MK_CUDA(cudaMemcpyAsync(oh, logits_.ptr(), tok_off, cudaMemcpyDeviceToHost, stream_));
    if (t.flags & FWD_WANT_TOKENS) MK_CUDA(cudaMemcpyAsync(oh + tok_off, tokens_.ptr(), (size_t)B * 4, cudaMemcpyDeviceToHost, stream_));
    MK_CUDA(cudaMemcpyAsync(oh + tok_off + (size_t)B * 4, err_.ptr(), 4, cudaMemcpyDeviceToHost, stream_));
    MK_CUDA(cudaMemcpyAsync(oh + tok_off + (size_t)B * 4 + 4, status_.ptr(), 4, cudaMemcpyDeviceToHost, stream_));
    d2h_bytes_ += 8 + (int64_t)tok_off + ((t.flags & FWD_WANT_TOKENS) ? (int64_t)B * 4 : 0);
    MK_CUDA(cudaEventRecord(ev_stop_, stream_));
    timed_ = true;
    out_lanes_ = B;
    out_rows_ = t.R;
    out_flags_ = t.flags;
}

std::string DeviceLm::status_message(int32_t status) const {
    if ((status & 0xFFFF0000) == kSampleEmptyStatus)
        return "sampling distribution is empty (lane " + std::to_string(status & 0xFFFF) + ")";  // src/sampling.rs:352-355
    return "a bounded wait inside a kernel gave up (tensor-core matmul pipeline or expert exchange; status " + std::to_string(status) + ")";
}

void DeviceLm::fetch_output(float* logits, uint32_t* tokens) {
    MK_CUDA(cudaStreamSynchronize(stream_));
    if (profiling_) prof_resolve();
    const uint8_t* oh = out_host_.as<uint8_t>();
    const size_t tok_off = (size_t)((out_flags_ & FWD_WANT_LOGITS) ? out_rows_ : 0) * spec_.vocab * 4;
    int32_t flags[2];
    memcpy(flags, oh + tok_off + (size_t)out_lanes_ * 4, 8);
    if (flags[0] != 0) throw std::runtime_error("batch descriptor index out of range on the device (flag " + std::to_string(flags[0]) + ")");
    if (flags[1] != 0) {
        // the status word is sticky on the device: clear it so that the next forward starts clean
        cudaMemsetAsync(status_.ptr(), 0, 4, stream_);
        throw std::runtime_error(status_message(flags[1]));
    }
    if (logits) {
        if (!(out_flags_ & FWD_WANT_LOGITS)) throw std::runtime_error("logits were not requested for this forward");
        memcpy(logits, oh, tok_off);
    }
    if (tokens) {
        if (!(out_flags_ & FWD_WANT_TOKENS)) throw std::runtime_error("tokens were not requested for this forward");
        memcpy(tokens, oh + tok_off, (size_t)out_lanes_ * 4);
    }
}

void DeviceLm::device_synchronize() { MK_CUDA(cudaStreamSynchronize(stream_)); }

float DeviceLm::last_forward_ms() const {
    if (!timed_) return 0.f;
    float ms = 0.f;
    if (cudaEventElapsedTime(&ms, ev_start_, ev_stop_) != cudaSuccess) {
        cudaGetLastError();
        return 0.f;
    }
    return ms;
}

// ---------------------------------------------------------------------------- profiling

void DeviceLm::profile_enable(bool on) {
    profiling_ = on;
    if (!on) return;
    prof_.assign(prof_names_.size(), KernelProfile{});
    for (size_t i = 0; i < prof_.size(); ++i) prof_[i].name = prof_names_[i];
}

void DeviceLm::prof_begin(int cls, double bytes, double flops) {
    if (!profiling_) return;
    ProfSpan sp;
    sp.cls = cls;
    sp.bytes = bytes;
    sp.flops = flops;
    for (cudaEvent_t* e : {&sp.a, &sp.b}) {
        if (event_pool_.empty()) {
            MK_CUDA(cudaEventCreate(e));
        } else {
            *e = event_pool_.back();
            event_pool_.pop_back();
        }
    }
    MK_CUDA(cudaEventRecord(sp.a, stream_));
    spans_.push_back(sp);
}

void DeviceLm::prof_end() {
    if (!profiling_ || spans_.empty()) return;
    MK_CUDA(cudaEventRecord(spans_.back().b, stream_));
}

void DeviceLm::prof_resolve() {
    for (ProfSpan& sp : spans_) {
        float ms = 0.f;
        if (cudaEventElapsedTime(&ms, sp.a, sp.b) == cudaSuccess) {
            KernelProfile& k = prof_[(size_t)sp.cls];
            ++k.launches;
            k.ms += ms;
            k.bytes += sp.bytes;
            k.flops += sp.flops;
        } else {
            cudaGetLastError();
        }
        event_pool_.push_back(sp.a);
        event_pool_.push_back(sp.b);
    }
    spans_.clear();
}

std::vector<PagedLm::KernelProfile> DeviceLm::profile_query() {
    std::vector<KernelProfile> out;
    for (const KernelProfile& k : prof_) if (k.launches > 0) out.push_back(k);
    return out;
}

}  // namespace mk
