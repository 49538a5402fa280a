// Model folders: config.json and model.safetensors (8-byte little-endian header length, a JSON header of name -> dtype,
// shape, data_offsets, then the data).
#pragma once
#include <cstdint>
#include <fstream>
#include <map>
#include <string>
#include <vector>

namespace vesper::models {

class SafeTensors {
public:
    struct Entry {
        std::string dtype;                    // BF16, F16, F32, I32, I64
        std::vector<int64_t> shape;
        int64_t begin = 0, end = 0;           // byte range in the file
        int64_t numel() const { int64_t n = 1; for (int64_t d : shape) n *= d; return n; }
    };
    explicit SafeTensors(const std::string& path);
    const std::map<std::string, Entry>& entries() const { return entries_; }
    // One tensor's values as fp32 (exact for BF16 / F16 / F32).
    std::vector<float> read(const std::string& name);

private:
    std::ifstream file_;
    std::map<std::string, Entry> entries_;
};

std::string read_text_file(const std::string& path);

}  // namespace vesper::models
