#include "safetensors.h"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstring>

#include "json.h"

namespace l2b {

SafeTensorsFile::~SafeTensorsFile() {
    if (base_) munmap(const_cast<uint8_t*>(base_), size_);
    if (fd_ >= 0) close(fd_);
}

bool SafeTensorsFile::open(const std::string& path) {
    fd_ = ::open(path.c_str(), O_RDONLY);
    struct stat st;
    if (fd_ < 0 || fstat(fd_, &st) != 0) {
        err_ = "cannot open " + path;
        return false;
    }
    size_ = (size_t)st.st_size;
    err_ = path + " is not a safetensors file";
    if (size_ < 8) return false;
    void* m = mmap(nullptr, size_, PROT_READ, MAP_PRIVATE, fd_, 0);
    if (m == MAP_FAILED) {
        err_ = "cannot map " + path;
        return false;
    }
    base_ = static_cast<const uint8_t*>(m);
    uint64_t n = 0;
    memcpy(&n, base_, 8);
    if (n > size_ - 8) return false;
    JsonValue dir;
    if (!JsonParser::parse(reinterpret_cast<const char*>(base_ + 8), (size_t)n, dir) || dir.kind != JsonValue::OBJECT) return false;
    const uint64_t room = size_ - 8 - n;
    for (const auto& e : dir.members) {
        if (e.first == "__metadata__") continue;
        const JsonValue *dt = e.second.find("dtype"), *sh = e.second.find("shape"), *of = e.second.find("data_offsets");
        if (!dt || !sh || !of || dt->kind != JsonValue::STRING || sh->kind != JsonValue::ARRAY || of->kind != JsonValue::ARRAY || of->items.size() != 2) return false;
        SafeTensor t;
        t.dtype = dt->str;
        const uint64_t elem = t.dtype == "F64" || t.dtype == "I64" ? 8 : t.dtype == "F32" || t.dtype == "I32" ? 4 : t.dtype == "BF16" || t.dtype == "F16" ? 2 : 1;
        uint64_t count = elem;
        for (const JsonValue& d : sh->items) {
            if (d.kind != JsonValue::NUMBER || d.num < 0 || d.num > 4e9 || (d.num > 0 && count > (uint64_t)(1e15 / d.num))) return false;
            t.shape.push_back((int64_t)d.num);
            count *= (uint64_t)d.num;
        }
        const double lo = of->items[0].num, hi = of->items[1].num;
        if (of->items[0].kind != JsonValue::NUMBER || of->items[1].kind != JsonValue::NUMBER || lo < 0 || hi < lo || hi > (double)room) return false;
        t.nbytes = (uint64_t)hi - (uint64_t)lo;
        if (t.nbytes != count) return false;
        t.data = base_ + 8 + n + (uint64_t)lo;
        tensors_[e.first] = t;
    }
    err_.clear();
    return true;
}

}  // namespace l2b
