// Host bookkeeping of recurrent-state slots.  A model with recurrent layers keeps one fixed-size state per live sequence and
// layer in device memory, as an array of slots; each slot has two halves, so that a forward reads the state of the last
// committed token from one half and writes the next state to the other.  A forward that fails changes nothing: the halves
// trade places only when the forward is committed.  A slot may be handed to another sequence as soon as it is released: all
// device work of a model runs on one stream, so the new owner's first write comes after the old owner's last read, and a
// fresh sequence reads no state at all (its incoming half is -1, which the kernels take as zeros).
#pragma once
#include <memory>
#include <stdexcept>
#include <vector>

namespace mk {

class StateSlots {
public:
    explicit StateSlots(int capacity) : capacity_(capacity) {
        for (int i = capacity; i-- > 0;) free_.push_back(i);
    }
    int capacity() const { return capacity_; }
    int in_use() const { return capacity_ - (int)free_.size(); }
    // -1 when every slot is taken
    int acquire() {
        if (free_.empty()) return -1;
        const int s = free_.back();
        free_.pop_back();
        return s;
    }
    void release(int s) { free_.push_back(s); }

private:
    int capacity_;
    std::vector<int> free_;
};

// One sequence's slot; gives it back on destruction.
class StateLease {
public:
    StateLease(std::shared_ptr<StateSlots> slots, int slot) : slots_(std::move(slots)), slot_(slot) {}
    ~StateLease() { slots_->release(slot_); }
    StateLease(const StateLease&) = delete;
    StateLease& operator=(const StateLease&) = delete;
    // Index (slot * 2 + half) of the half that holds the committed state, and of the half the next forward writes.
    int current() const { return slot_ * 2 + half_; }
    int next() const { return slot_ * 2 + (1 - half_); }
    void flip() { half_ ^= 1; }

private:
    std::shared_ptr<StateSlots> slots_;
    int slot_, half_ = 0;
};

}  // namespace mk
