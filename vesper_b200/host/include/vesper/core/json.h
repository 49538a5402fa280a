// A small JSON reader: model configurations and safetensors headers.  Numbers keep their text, so integers are read
// exactly.
#pragma once
#include <cstdint>
#include <map>
#include <string>
#include <vector>

namespace vesper {

class Json {
public:
    enum class Kind { Null, Bool, Number, String, Array, Object };
    static Json parse(const std::string& text);                 // throws std::runtime_error with the byte offset

    Kind kind() const { return kind_; }
    bool is_null() const { return kind_ == Kind::Null; }
    bool has(const std::string& key) const { return kind_ == Kind::Object && object_.count(key) != 0; }
    const Json& at(const std::string& key) const;               // throws when the key is missing
    // The value at key, or Null when the key is missing.
    const Json& get(const std::string& key) const;
    int64_t as_int() const;
    double as_double() const;
    bool as_bool() const;
    const std::string& as_string() const;
    const std::vector<Json>& as_array() const;
    const std::map<std::string, Json>& as_object() const;
    int64_t int_or(const std::string& key, int64_t fallback) const { return has(key) ? at(key).as_int() : fallback; }
    double double_or(const std::string& key, double fallback) const { return has(key) ? at(key).as_double() : fallback; }

private:
    friend struct JsonParser;
    Kind kind_ = Kind::Null;
    bool bool_ = false;
    std::string text_;
    std::vector<Json> array_;
    std::map<std::string, Json> object_;
};

}  // namespace vesper
