// Reader for safetensors files, host side of model folders: memory-maps the file and hands out bounds-checked views of its tensors.
// Layout: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets), then the payloads; the offsets
// count from the end of the header.
#pragma once
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstring>
#include <map>
#include <string>
#include <vector>

#include "json.hpp"

namespace qtb {

struct SafeTensor {
    std::string dtype;             // "BF16", "F16", "F32", "I32", ...
    std::vector<uint64_t> shape;   // outermost dimension first
    const uint8_t* data = nullptr;
    uint64_t bytes = 0, elements = 0;
};

inline float half_bits_to_float(uint16_t h) {
    const int e = (h >> 10) & 31, m = h & 1023;
    const float v = e == 31 ? (m ? NAN : INFINITY) : e == 0 ? std::ldexp(static_cast<float>(m), -24) : std::ldexp(static_cast<float>(m | 1024), e - 25);
    return h & 0x8000 ? -v : v;
}

class SafetensorsFile {
  public:
    std::map<std::string, SafeTensor> tensors;
    SafetensorsFile() = default;
    SafetensorsFile(const SafetensorsFile&) = delete;
    SafetensorsFile& operator=(const SafetensorsFile&) = delete;
    ~SafetensorsFile() {
        if (map_ != nullptr) munmap(map_, size_);
    }
    const SafeTensor* find(const std::string& name) const {
        const auto it = tensors.find(name);
        return it == tensors.end() ? nullptr : &it->second;
    }
    // 0 on success, 1 when the file cannot be read, 2 when it is malformed.
    int open(const std::string& path, std::string& why) {
        const int fd = ::open(path.c_str(), O_RDONLY | O_CLOEXEC);
        struct stat st;
        if (fd < 0 || fstat(fd, &st) != 0 || !S_ISREG(st.st_mode)) {
            if (fd >= 0) ::close(fd);
            why = "cannot open " + path;
            return 1;
        }
        size_ = static_cast<size_t>(st.st_size);
        void* p = size_ >= 8 ? mmap(nullptr, size_, PROT_READ, MAP_PRIVATE, fd, 0) : MAP_FAILED;
        ::close(fd);
        if (p == MAP_FAILED) {
            why = path + " cannot be mapped (" + std::to_string(size_) + " bytes)";
            return size_ < 8 ? 2 : 1;
        }
        map_ = static_cast<uint8_t*>(p);
        uint64_t header = 0;
        std::memcpy(&header, map_, 8);
        if (header > size_ - 8) {
            why = path + ": the header does not fit the file";
            return 2;
        }
        JsonValue root;
        if (!JsonReader(reinterpret_cast<const char*>(map_) + 8, header).parse(&root, &why) || !root.is(JsonValue::kObject)) {
            why = path + ": the header is not a JSON object (" + why + ")";
            return 2;
        }
        const uint64_t base = 8 + header, payload = size_ - base;
        for (const auto& f : root.fields) {
            if (f.first == "__metadata__") continue;
            const JsonValue *dt = f.second.get("dtype"), *sh = f.second.get("shape"), *off = f.second.get("data_offsets");
            SafeTensor t;
            uint64_t a = 0, b = 0, d = 0;
            bool good = dt != nullptr && dt->is(JsonValue::kString) && sh != nullptr && sh->is(JsonValue::kArray) && off != nullptr && off->items.size() == 2 &&
                        off->items[0].as_u64(&a) && off->items[1].as_u64(&b) && a <= b && b <= payload;
            t.elements = 1;
            if (good)
                for (const JsonValue& v : sh->items) {
                    good = good && v.as_u64(&d) && (d == 0 || t.elements <= (uint64_t(1) << 48) / d);
                    if (!good) break;
                    t.shape.push_back(d), t.elements *= d;
                }
            if (good) {
                t.dtype = dt->s, t.data = map_ + base + a, t.bytes = b - a;
                const uint64_t width = width_of(t.dtype);
                good = width == 0 || t.elements * width == t.bytes;
            }
            if (!good) {
                why = path + ": malformed entry '" + f.first + "'";
                return 2;
            }
            tensors.emplace(f.first, std::move(t));
        }
        return 0;
    }
    static uint64_t width_of(const std::string& dtype) {
        if (dtype == "BF16" || dtype == "F16") return 2;
        if (dtype == "F32" || dtype == "I32") return 4;
        return 0;
    }
    // Element i of a floating-point tensor.
    static float at(const SafeTensor& t, uint64_t i) {
        if (t.dtype == "F32") {
            float v;
            std::memcpy(&v, t.data + i * 4, 4);
            return v;
        }
        uint16_t h;
        std::memcpy(&h, t.data + i * 2, 2);
        if (t.dtype == "F16") return half_bits_to_float(h);
        const uint32_t u = uint32_t(h) << 16;
        float v;
        std::memcpy(&v, &u, 4);
        return v;
    }
    static bool is_float(const SafeTensor& t) { return t.dtype == "BF16" || t.dtype == "F16" || t.dtype == "F32"; }

  private:
    uint8_t* map_ = nullptr;
    size_t size_ = 0;
};

}  // namespace qtb
