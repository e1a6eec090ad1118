// Reader of one safetensors file: 8-byte little-endian header length, a JSON header (name -> dtype, shape, data_offsets),
// the data.  Tensors are read on demand; the file is never held in memory as a whole.
#pragma once
#include "json.h"

#include <cstdint>
#include <cstdio>
#include <cstring>
#include <string>
#include <unordered_map>
#include <vector>

namespace tmb {

struct SafeTensor {
    std::string          dtype;
    std::vector<int64_t> shape;
    uint64_t             begin = 0, end = 0;  // bytes from the start of the data
    int64_t              count() const
    {
        int64_t n = 1;
        for (int64_t d : shape) n *= d;
        return n;
    }
};

class SafeTensors {
public:
    ~SafeTensors()
    {
        if (f_) std::fclose(f_);
    }
    bool open(const std::string& path)
    {
        f_ = std::fopen(path.c_str(), "rb");
        if (!f_) return false;
        unsigned char len[8];
        if (std::fread(len, 1, 8, f_) != 8) return false;
        uint64_t n = 0;
        for (int i = 0; i < 8; ++i) n |= (uint64_t)len[i] << (8 * i);
        std::fseek(f_, 0, SEEK_END);
        const uint64_t size = (uint64_t)std::ftell(f_);
        if (n > size - 8) return false;
        std::string head(n, '\0');
        std::fseek(f_, 8, SEEK_SET);
        Json j;
        if (std::fread(&head[0], 1, n, f_) != n || !Json::parse(head, &j) || j.kind != Json::kObject) return false;
        data_ = 8 + n;
        for (const auto& e : j.fields) {
            if (e.first == "__metadata__") continue;
            const Json *dt = e.second.find("dtype"), *sh = e.second.find("shape"), *off = e.second.find("data_offsets");
            if (!dt || !sh || !off || off->items.size() != 2) return false;
            SafeTensor t;
            t.dtype = dt->text;
            for (const Json& d : sh->items) t.shape.push_back((int64_t)d.number);
            t.begin = (uint64_t)off->items[0].number, t.end = (uint64_t)off->items[1].number;
            const uint64_t el = t.dtype == "F32" || t.dtype == "I32" ? 4 : (t.dtype == "BF16" || t.dtype == "F16" ? 2 : 0);
            if (el == 0 || t.end < t.begin || t.end - t.begin != el * (uint64_t)t.count() || data_ + t.end > size) return false;
            table_.emplace(e.first, std::move(t));
        }
        return true;
    }
    const SafeTensor* find(const std::string& name) const
    {
        const auto it = table_.find(name);
        return it == table_.end() ? nullptr : &it->second;
    }
    bool read(const SafeTensor& t, std::vector<unsigned char>& raw)
    {
        raw.resize(t.end - t.begin);
        return std::fseek(f_, (long)(data_ + t.begin), SEEK_SET) == 0 && std::fread(raw.data(), 1, raw.size(), f_) == raw.size();
    }

private:
    std::FILE*                                  f_    = nullptr;
    uint64_t                                    data_ = 0;
    std::unordered_map<std::string, SafeTensor> table_;
};

}  // namespace tmb
