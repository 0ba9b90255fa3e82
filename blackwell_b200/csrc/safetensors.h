// Reader of a safetensors file: an 8-byte little-endian header length, a JSON header {name: {dtype, shape, data_offsets}},
// then the data.  Host only; everything is checked against the file's length.
#pragma once
#include <stdint.h>
#include <stdio.h>
#include <sys/stat.h>

#include <map>
#include <string>
#include <vector>

#include "json.h"

namespace bw {

class SafeTensors {
public:
    struct Entry {
        std::string dtype;
        std::vector<long> shape;
        uint64_t begin = 0, end = 0;   // relative to the data section
        long count() const { long n = 1; for (long d : shape) n *= d; return n; }
    };
    ~SafeTensors() { if (f_) fclose(f_); }

    bool open(const std::string& path, std::string* err) {
        f_ = fopen(path.c_str(), "rb");
        if (!f_) { *err = "cannot open " + path; return false; }
        struct stat st;
        uint64_t n = 0;
        if (fstat(fileno(f_), &st) != 0 || fread(&n, 8, 1, f_) != 1 || n > (uint64_t)st.st_size - 8) {
            *err = path + " is not a safetensors file";
            return false;
        }
        std::string head(n, '\0');
        if (fread(&head[0], 1, n, f_) != n) { *err = "cannot read the header of " + path; return false; }
        data_ = 8 + n;
        const uint64_t room = (uint64_t)st.st_size - data_;
        Json j;
        if (!Json::parse(head.data(), head.size(), &j, err) || j.type != Json::kObject) { *err = path + ": " + *err; return false; }
        for (const auto& kv : j.obj) {
            if (kv.first == "__metadata__") continue;
            const Json *dt = kv.second.get("dtype"), *sh = kv.second.get("shape"), *of = kv.second.get("data_offsets");
            Entry e;
            bool ok = dt && dt->type == Json::kString && sh && sh->type == Json::kArray && of && of->arr.size() == 2 &&
                      of->arr[0].is_int() && of->arr[1].is_int();
            if (ok) {
                e.dtype = dt->str;
                for (const Json& d : sh->arr) {
                    ok = ok && d.is_int() && d.num >= 0;
                    e.shape.push_back((long)d.num);
                }
                ok = ok && of->arr[0].num >= 0 && of->arr[0].num <= of->arr[1].num && of->arr[1].num <= (double)room;
                e.begin = (uint64_t)of->arr[0].num;
                e.end = (uint64_t)of->arr[1].num;
                const int size = e.dtype == "BF16" || e.dtype == "F16" ? 2 : e.dtype == "F32" || e.dtype == "I32" ? 4 : 0;
                ok = ok && (size == 0 || e.end - e.begin == (uint64_t)e.count() * size);
            }
            if (!ok) { *err = path + ": bad entry for " + kv.first; return false; }
            entries_[kv.first] = e;
        }
        return true;
    }
    const Entry* find(const std::string& name) const {
        auto it = entries_.find(name);
        return it == entries_.end() ? nullptr : &it->second;
    }
    // Raw bfloat16 values of a BF16 tensor with the given shape.
    bool read_bf16(const std::string& name, const std::vector<long>& shape, std::vector<uint16_t>* out, std::string* err) {
        const Entry* e = find(name);
        if (!e) { *err = "tensor " + name + " is missing"; return false; }
        if (e->dtype != "BF16" || e->shape != shape) {
            *err = "tensor " + name + ": expected BF16 of shape [";
            for (size_t i = 0; i < shape.size(); ++i) *err += (i ? ", " : "") + std::to_string(shape[i]);
            *err += "]";
            return false;
        }
        out->resize(e->count());
        if (fseek(f_, (long)(data_ + e->begin), SEEK_SET) != 0 || fread(out->data(), 2, out->size(), f_) != out->size()) {
            *err = "cannot read tensor " + name;
            return false;
        }
        return true;
    }

private:
    FILE* f_ = nullptr;
    uint64_t data_ = 0;
    std::map<std::string, Entry> entries_;
};

}  // namespace bw
