// The safetensors container: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, data_offsets) and
// the tensor bytes, mapped read-only.  Every offset is checked against the file before a tensor is handed out.
#pragma once
#include <cstdint>
#include <map>
#include <string>
#include <vector>

namespace mk {

enum class StType { F32, F16, BF16, I32, Other };

struct StTensor {
    StType type = StType::Other;
    std::vector<int64_t> shape;
    const uint8_t* data = nullptr;
    int64_t bytes = 0;
    int64_t elements() const {
        int64_t n = 1;
        for (int64_t d : shape) n *= d;
        return n;
    }
};

class SafetensorsFile {
public:
    explicit SafetensorsFile(const std::string& path);
    ~SafetensorsFile();
    SafetensorsFile(const SafetensorsFile&) = delete;
    SafetensorsFile& operator=(const SafetensorsFile&) = delete;

    const std::map<std::string, StTensor>& tensors() const { return tensors_; }
    const StTensor* find(const std::string& name) const;
    // The tensor, with this shape and a floating-point type; throws with the name otherwise.
    const StTensor& require(const std::string& name, const std::vector<int64_t>& shape) const;
    // Its values widened to f32 (exact for every accepted type).
    std::vector<float> values(const std::string& name, const std::vector<int64_t>& shape) const;
    // Its values as bfloat16 bits: as stored for BF16, rounded to nearest even otherwise.
    std::vector<uint16_t> bf16_values(const std::string& name, const std::vector<int64_t>& shape) const;

private:
    std::string path_;
    const uint8_t* map_ = nullptr;
    size_t size_ = 0;
    std::map<std::string, StTensor> tensors_;
};

// Rounds to the nearest bfloat16, ties to even.
uint16_t bf16_bits(float v);

}  // namespace mk
