// See safetensors_file.h.
#include "safetensors_file.h"
#include "json.h"
#include <cuda_fp16.h>
#include <cstring>
#include <fcntl.h>
#include <stdexcept>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

namespace mk {

namespace {

StType type_of(const std::string& s) {
    if (s == "F32") return StType::F32;
    if (s == "F16") return StType::F16;
    if (s == "BF16") return StType::BF16;
    if (s == "I32") return StType::I32;
    return StType::Other;
}

int64_t type_bytes(StType t) { return t == StType::F32 || t == StType::I32 ? 4 : (t == StType::Other ? 0 : 2); }

std::string shape_text(const std::vector<int64_t>& s) {
    std::string out = "[";
    for (size_t i = 0; i < s.size(); ++i) out += (i ? ", " : "") + std::to_string(s[i]);
    return out + "]";
}

}  // namespace

SafetensorsFile::SafetensorsFile(const std::string& path) : path_(path) {
    const int fd = open(path.c_str(), O_RDONLY | O_CLOEXEC | O_NONBLOCK);
    if (fd < 0) throw std::runtime_error("cannot open " + path);
    struct stat st;
    if (fstat(fd, &st) != 0 || !S_ISREG(st.st_mode)) {
        close(fd);
        throw std::runtime_error(path + " is not a regular file");
    }
    size_ = (size_t)st.st_size;
    void* m = size_ >= 8 ? mmap(nullptr, size_, PROT_READ, MAP_PRIVATE, fd, 0) : MAP_FAILED;
    close(fd);
    if (m == MAP_FAILED) throw std::runtime_error(path + " cannot be mapped as a safetensors file");
    map_ = (const uint8_t*)m;
    try {
        uint64_t hn = 0;
        for (int i = 7; i >= 0; --i) hn = (hn << 8) | map_[i];
        if (hn > size_ - 8 || hn > ((uint64_t)256 << 20)) throw std::runtime_error(path + ": safetensors header length is out of range");
        const Json head = Json::parse((const char*)map_ + 8, (size_t)hn, path + " header");
        const uint64_t body = size_ - 8 - hn;
        for (const auto& kv : head.members()) {
            if (kv.first == "__metadata__") continue;
            StTensor t;
            t.type = type_of(kv.second.at("dtype").str());
            int64_t n = 1;
            for (const Json& d : kv.second.at("shape").items()) {
                const int64_t v = d.integer();
                if (v < 0 || (v > 0 && n > ((int64_t)1 << 46) / v)) throw std::runtime_error(path + ": tensor `" + kv.first + "` has an impossible shape");
                n *= v;
                t.shape.push_back(v);
            }
            const auto& off = kv.second.at("data_offsets").items();
            if (off.size() != 2) throw std::runtime_error(path + ": tensor `" + kv.first + "` needs two data offsets");
            const int64_t lo = off[0].integer(), hi = off[1].integer();
            if (lo < 0 || hi < lo || (uint64_t)hi > body) throw std::runtime_error(path + ": tensor `" + kv.first + "` lies outside the file");
            if (t.type != StType::Other && hi - lo != n * type_bytes(t.type))
                throw std::runtime_error(path + ": tensor `" + kv.first + "` has " + std::to_string(hi - lo) + " bytes, its shape needs " +
                                         std::to_string(n * type_bytes(t.type)));
            t.data = map_ + 8 + hn + lo;
            t.bytes = hi - lo;
            tensors_.emplace(kv.first, std::move(t));
        }
    } catch (...) {
        munmap(const_cast<uint8_t*>(map_), size_);
        throw;
    }
}

SafetensorsFile::~SafetensorsFile() {
    if (map_) munmap(const_cast<uint8_t*>(map_), size_);
}

const StTensor* SafetensorsFile::find(const std::string& name) const {
    auto it = tensors_.find(name);
    return it == tensors_.end() ? nullptr : &it->second;
}

const StTensor& SafetensorsFile::require(const std::string& name, const std::vector<int64_t>& shape) const {
    const StTensor* t = find(name);
    if (t == nullptr) throw std::runtime_error("tensor `" + name + "` is missing from " + path_);
    if (t->shape != shape)
        throw std::runtime_error("tensor `" + name + "` has shape " + shape_text(t->shape) + ", expected " + shape_text(shape));
    if (t->type != StType::F32 && t->type != StType::F16 && t->type != StType::BF16)
        throw std::runtime_error("tensor `" + name + "` is not a floating-point tensor");
    return *t;
}

std::vector<float> SafetensorsFile::values(const std::string& name, const std::vector<int64_t>& shape) const {
    const StTensor& t = require(name, shape);
    const int64_t n = t.elements();
    std::vector<float> out((size_t)n);
    if (t.type == StType::F32) {
        memcpy(out.data(), t.data, (size_t)n * 4);
        return out;
    }
    for (int64_t i = 0; i < n; ++i) {
        uint16_t h;
        memcpy(&h, t.data + 2 * i, 2);
        if (t.type == StType::BF16) {
            const uint32_t u = (uint32_t)h << 16;
            memcpy(&out[(size_t)i], &u, 4);
        } else {
            __half_raw r;
            r.x = h;
            out[(size_t)i] = __half2float(__half(r));
        }
    }
    return out;
}

std::vector<uint16_t> SafetensorsFile::bf16_values(const std::string& name, const std::vector<int64_t>& shape) const {
    const StTensor& t = require(name, shape);
    std::vector<uint16_t> out((size_t)t.elements());
    if (t.type == StType::BF16) {
        memcpy(out.data(), t.data, out.size() * 2);
        return out;
    }
    const std::vector<float> v = values(name, shape);
    for (size_t i = 0; i < v.size(); ++i) out[i] = bf16_bits(v[i]);
    return out;
}

uint16_t bf16_bits(float v) {
    uint32_t u;
    memcpy(&u, &v, 4);
    if ((u & 0x7FFFFFFF) > 0x7F800000) return (uint16_t)((u >> 16) | 0x40);  // NaN stays NaN
    return (uint16_t)((u + 0x7FFF + ((u >> 16) & 1)) >> 16);
}

}  // namespace mk
