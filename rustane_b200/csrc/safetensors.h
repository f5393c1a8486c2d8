// Reader of a safetensors file (8-byte little-endian header length, JSON header, data), mapped into memory.
#pragma once
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstdint>
#include <cstring>
#include <map>
#include <string>
#include <vector>

#include "json.h"

namespace cd {

struct TensorView {
    std::string dtype;
    std::vector<size_t> shape;
    const unsigned char* data = nullptr;
    size_t bytes = 0;
};

class SafeTensors {
  public:
    SafeTensors() = default;
    SafeTensors(const SafeTensors&) = delete;
    SafeTensors& operator=(const SafeTensors&) = delete;
    ~SafeTensors() {
        if (base_) munmap(base_, size_);
    }
    bool open(const std::string& path, std::string* err) {
        const int fd = ::open(path.c_str(), O_RDONLY);
        if (fd < 0) { *err = "cannot open " + path; return false; }
        struct stat st;
        if (fstat(fd, &st) != 0 || st.st_size < 8) { ::close(fd); *err = path + " is too small for a safetensors file"; return false; }
        size_ = (size_t)st.st_size;
        void* p = mmap(nullptr, size_, PROT_READ, MAP_PRIVATE, fd, 0);
        ::close(fd);
        if (p == MAP_FAILED) { *err = "cannot map " + path; return false; }
        base_ = p;
        const unsigned char* b = static_cast<const unsigned char*>(p);
        uint64_t hlen = 0;
        for (int i = 7; i >= 0; --i) hlen = hlen << 8 | b[i];
        if (hlen > size_ - 8) { *err = path + ": header longer than the file"; return false; }
        const std::string text(reinterpret_cast<const char*>(b + 8), (size_t)hlen);
        JsonValue root;
        if (!JsonReader(text).parse(&root) || root.kind != JsonValue::OBJ) { *err = path + ": malformed header"; return false; }
        const size_t room = size_ - 8 - (size_t)hlen;
        for (const auto& kv : root.obj) {
            if (kv.first == "__metadata__") continue;
            const JsonValue *dt = kv.second.get("dtype"), *sh = kv.second.get("shape"), *of = kv.second.get("data_offsets");
            if (!dt || !sh || !of || of->arr.size() != 2) { *err = path + ": bad entry for " + kv.first; return false; }
            TensorView t;
            t.dtype = dt->str;
            size_t n = 1;
            for (const auto& d : sh->arr) { t.shape.push_back((size_t)d.num); n *= (size_t)d.num; }
            const double lo = of->arr[0].num, hi = of->arr[1].num;
            if (lo < 0 || hi < lo || hi > (double)room) { *err = path + ": " + kv.first + " lies outside the file"; return false; }
            t.data = b + 8 + hlen + (size_t)lo;
            t.bytes = (size_t)(hi - lo);
            const size_t es = t.dtype == "BF16" || t.dtype == "F16" ? 2 : t.dtype == "F32" || t.dtype == "I32" ? 4 : 0;
            if (es && n * es != t.bytes) { *err = path + ": size of " + kv.first + " does not fit its shape"; return false; }
            tensors_[kv.first] = t;
        }
        return true;
    }
    const TensorView* find(const std::string& name) const {
        auto it = tensors_.find(name);
        return it == tensors_.end() ? nullptr : &it->second;
    }

  private:
    void* base_ = nullptr;
    size_t size_ = 0;
    std::map<std::string, TensorView> tensors_;
};

}  // namespace cd
