// Host side of weight loading: named tensors (bf16, fp32 or int32, of a memory-mapped safetensors file or handed
// in one by one) and the cursor that checks shapes and converts rows on the way into the model's layout.
#pragma once
#include <cstdint>
#include <cstring>
#include <fcntl.h>
#include <map>
#include <stdexcept>
#include <string>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>
#include <vector>
#include "json.h"

namespace b200 {

enum class TensorType : int { BF16 = 0, F32 = 1, I32 = 2 };

struct HostTensor {
    TensorType type = TensorType::BF16;
    std::vector<long> shape;
    const uint8_t* data = nullptr;   // into the mapped file, or owned
    std::vector<uint8_t> owned;
    size_t count() const { size_t n = 1; for (long d : shape) n *= (size_t)d; return n; }
    size_t bytes() const { return count() * (type == TensorType::BF16 ? 2 : 4); }
    int integer(size_t i) const { int v; memcpy(&v, data + 4 * i, 4); return v; }
    float value(size_t i) const {
        if (type == TensorType::F32) { float v; memcpy(&v, data + 4 * i, 4); return v; }
        uint16_t h; memcpy(&h, data + 2 * i, 2);
        const uint32_t u = (uint32_t)h << 16;
        float v; memcpy(&v, &u, 4);
        return v;
    }
};

inline uint16_t bf16_bits(float v) {  // nearest, ties to even
    uint32_t u; memcpy(&u, &v, 4);
    if ((u & 0x7fffffffu) > 0x7f800000u) return (uint16_t)(u >> 16 | 0x40);
    return (uint16_t)((u + 0x7fffu + (u >> 16 & 1)) >> 16);
}

class TensorStore {
   public:
    ~TensorStore() { if (map_) munmap(map_, map_len_); }
    void set(const std::string& name, const void* data, TensorType type, const std::vector<long>& shape) {
        HostTensor t;
        t.type = type;
        t.shape = shape;
        const size_t n = t.bytes();
        t.owned.assign(static_cast<const uint8_t*>(data), static_cast<const uint8_t*>(data) + n);
        HostTensor& d = tensors_[name] = std::move(t);
        d.data = d.owned.data();
    }
    // 8-byte little-endian header length, header (JSON: name -> dtype, shape, data_offsets), data
    void open_safetensors(const char* path) {
        const int fd = ::open(path, O_RDONLY);
        if (fd < 0) throw std::runtime_error(std::string("cannot open ") + path);
        struct stat st;
        if (fstat(fd, &st) != 0 || st.st_size < 8) { ::close(fd); throw std::runtime_error(std::string(path) + ": not a safetensors file"); }
        map_len_ = (size_t)st.st_size;
        map_ = mmap(nullptr, map_len_, PROT_READ, MAP_PRIVATE, fd, 0);
        ::close(fd);
        if (map_ == MAP_FAILED) { map_ = nullptr; throw std::runtime_error(std::string("cannot map ") + path); }
        const uint8_t* p = static_cast<const uint8_t*>(map_);
        uint64_t n = 0;
        for (int i = 7; i >= 0; --i) n = n << 8 | p[i];
        if (n > map_len_ - 8) throw std::runtime_error(std::string(path) + ": header beyond the end of the file");
        const Json head = Json::parse(reinterpret_cast<const char*>(p) + 8, reinterpret_cast<const char*>(p) + 8 + n);
        const size_t data_len = map_len_ - 8 - n;
        for (const auto& kv : head.obj) {
            if (kv.first == "__metadata__") continue;
            const std::string& dt = kv.second.string("dtype");
            if (dt != "BF16" && dt != "F32" && dt != "I32") continue;  // (nothing here reads another)
            HostTensor t;
            t.type = dt == "BF16" ? TensorType::BF16 : (dt == "F32" ? TensorType::F32 : TensorType::I32);
            for (const Json& d : kv.second.at("shape").arr) t.shape.push_back((long)d.num);
            const auto& off = kv.second.at("data_offsets").arr;
            if (off.size() != 2) throw std::runtime_error(kv.first + ": bad data_offsets");
            const double b = off[0].num, e = off[1].num;
            if (b < 0 || e < b || e > (double)data_len || (size_t)(e - b) != t.bytes())
                throw std::runtime_error(kv.first + ": data_offsets do not fit the shape or the file");
            t.data = p + 8 + n + (size_t)b;
            tensors_[kv.first] = std::move(t);
        }
    }
    // the tensor, whose shape must be this one; integers: a table of int32 instead of numbers
    const HostTensor& get(const std::string& name, const std::vector<long>& shape, bool integers = false) const {
        auto it = tensors_.find(name);
        if (it == tensors_.end()) throw std::runtime_error("weights: no tensor '" + name + "'");
        if ((it->second.type == TensorType::I32) != integers)
            throw std::runtime_error("weights: '" + name + "' must hold " + (integers ? "int32" : "bf16 or fp32") + " elements");
        if (it->second.shape != shape) {
            std::string s = "weights: '" + name + "' has shape [", w;
            for (long d : it->second.shape) s += std::to_string(d) + ",";
            for (long d : shape) w += std::to_string(d) + ",";
            throw std::runtime_error(s + "], the configuration wants [" + w + "]");
        }
        return it->second;
    }

    // rows of a matrix whose height only its shape gives
    int rows(const std::string& name) const {
        auto it = tensors_.find(name);
        if (it == tensors_.end()) throw std::runtime_error("weights: no tensor '" + name + "'");
        if (it->second.shape.size() != 2 || it->second.shape[0] < 1) throw std::runtime_error("weights: '" + name + "' must be a matrix");
        return (int)it->second.shape[0];
    }

   private:
    std::map<std::string, HostTensor> tensors_;
    void* map_ = nullptr;
    size_t map_len_ = 0;
};

}  // namespace b200
