// safetensors container reader (host only): an 8-byte little-endian header length, a JSON directory (name -> dtype, shape,
// data_offsets) and the tensor data, over a read-only memory map.
#pragma once
#include <cstdint>
#include <map>
#include <string>
#include <vector>

namespace l2b {

struct SafeTensor {
    std::string dtype;  // "BF16", "F32", ...
    std::vector<int64_t> shape;
    const uint8_t* data = nullptr;
    uint64_t nbytes = 0;
};

class SafeTensorsFile {
public:
    SafeTensorsFile() = default;
    ~SafeTensorsFile();
    SafeTensorsFile(const SafeTensorsFile&) = delete;
    SafeTensorsFile& operator=(const SafeTensorsFile&) = delete;
    // Returns false and sets error() on anything that is not a well-formed file.
    bool open(const std::string& path);
    const std::string& error() const { return err_; }
    const std::map<std::string, SafeTensor>& tensors() const { return tensors_; }

private:
    int fd_ = -1;
    const uint8_t* base_ = nullptr;
    size_t size_ = 0;
    std::map<std::string, SafeTensor> tensors_;
    std::string err_;
};

}  // namespace l2b
