#include <vesper/core/json.h>
#include <vesper/core/tensor.h>
#include <vesper/models/checkpoint.h>

#include <cstring>
#include <sstream>
#include <stdexcept>

namespace vesper::models {

std::string read_text_file(const std::string& path) {
    std::ifstream f(path, std::ios::binary);
    if (!f) throw std::runtime_error("cannot open " + path);
    std::ostringstream o;
    o << f.rdbuf();
    return o.str();
}

SafeTensors::SafeTensors(const std::string& path) : file_(path, std::ios::binary) {
    if (!file_) throw std::runtime_error("cannot open " + path);
    file_.seekg(0, std::ios::end);
    const int64_t size = static_cast<int64_t>(file_.tellg());
    file_.seekg(0);
    unsigned char raw[8] = {};
    file_.read(reinterpret_cast<char*>(raw), 8);
    uint64_t n = 0;
    for (int i = 7; i >= 0; --i) n = n << 8 | raw[i];
    if (!file_ || n > static_cast<uint64_t>(size) - 8) throw std::runtime_error(path + ": not a safetensors file");
    std::string header(n, '\0');
    file_.read(header.data(), static_cast<std::streamsize>(n));
    const Json meta = Json::parse(header);
    const int64_t base = 8 + static_cast<int64_t>(n);
    for (const auto& kv : meta.as_object()) {
        if (kv.first == "__metadata__") continue;
        Entry e;
        e.dtype = kv.second.at("dtype").as_string();
        for (const Json& d : kv.second.at("shape").as_array()) e.shape.push_back(d.as_int());
        const auto& off = kv.second.at("data_offsets").as_array();
        if (off.size() != 2) throw std::runtime_error(path + ": bad data_offsets of " + kv.first);
        e.begin = base + off[0].as_int();
        e.end = base + off[1].as_int();
        if (e.begin < base || e.end < e.begin || e.end > size) throw std::runtime_error(path + ": data of " + kv.first + " lies outside the file");
        entries_[kv.first] = e;
    }
}

std::vector<float> SafeTensors::read(const std::string& name) {
    auto it = entries_.find(name);
    if (it == entries_.end()) throw std::runtime_error("checkpoint has no tensor named " + name);
    const Entry& e = it->second;
    const size_t n = static_cast<size_t>(e.numel());
    const size_t esz = (e.dtype == "BF16" || e.dtype == "F16") ? 2 : (e.dtype == "F32" || e.dtype == "I32") ? 4 : e.dtype == "I64" ? 8 : 0;
    if (esz == 0) throw std::runtime_error("checkpoint tensor " + name + " has unsupported type " + e.dtype);
    if (n * esz != static_cast<size_t>(e.end - e.begin)) throw std::runtime_error("checkpoint tensor " + name + ": size does not match its shape");
    std::vector<char> raw(n * esz);
    file_.clear();
    file_.seekg(e.begin);
    file_.read(raw.data(), static_cast<std::streamsize>(raw.size()));
    if (!file_) throw std::runtime_error("cannot read tensor " + name);
    std::vector<float> out(n);
    for (size_t i = 0; i < n; ++i) {
        const char* p = raw.data() + i * esz;
        if (esz == 2) {
            uint16_t u;
            std::memcpy(&u, p, 2);
            out[i] = e.dtype == "BF16" ? bf16_to_float(u) : fp16_to_float(u);
        } else if (e.dtype == "F32") std::memcpy(&out[i], p, 4);
        else if (esz == 4) { int32_t v; std::memcpy(&v, p, 4); out[i] = static_cast<float>(v); }
        else { int64_t v; std::memcpy(&v, p, 8); out[i] = static_cast<float>(v); }
    }
    return out;
}

}  // namespace vesper::models
