#include <vesper/core/json.h>

#include <cctype>
#include <cstdlib>
#include <stdexcept>

namespace vesper {

struct JsonParser {
    const std::string& s;
    size_t i = 0;
    int depth = 0;

    [[noreturn]] void fail(const char* what) const { throw std::runtime_error(std::string("JSON: ") + what + " at byte " + std::to_string(i)); }
    void space() { while (i < s.size() && (s[i] == ' ' || s[i] == '\t' || s[i] == '\n' || s[i] == '\r')) ++i; }
    char peek() { if (i >= s.size()) fail("unexpected end"); return s[i]; }
    void expect(char c) { if (peek() != c) fail("unexpected character"); ++i; }
    bool word(const char* w) {
        const std::string t(w);
        if (s.compare(i, t.size(), t) != 0) return false;
        i += t.size();
        return true;
    }
    static void utf8(std::string& out, unsigned c) {
        if (c < 0x80) out += static_cast<char>(c);
        else if (c < 0x800) { out += static_cast<char>(0xC0 | (c >> 6)); out += static_cast<char>(0x80 | (c & 63)); }
        else if (c < 0x10000) { out += static_cast<char>(0xE0 | (c >> 12)); out += static_cast<char>(0x80 | ((c >> 6) & 63)); out += static_cast<char>(0x80 | (c & 63)); }
        else { out += static_cast<char>(0xF0 | (c >> 18)); out += static_cast<char>(0x80 | ((c >> 12) & 63)); out += static_cast<char>(0x80 | ((c >> 6) & 63)); out += static_cast<char>(0x80 | (c & 63)); }
    }
    unsigned hex4() {
        if (i + 4 > s.size()) fail("short \\u escape");
        unsigned v = 0;
        for (int k = 0; k < 4; ++k) {
            const char c = s[i++];
            if (!std::isxdigit(static_cast<unsigned char>(c))) fail("bad \\u escape");
            v = v * 16 + static_cast<unsigned>(c <= '9' ? c - '0' : (c | 32) - 'a' + 10);
        }
        return v;
    }
    std::string string() {
        expect('"');
        std::string out;
        while (peek() != '"') {
            char c = s[i++];
            if (c != '\\') { out += c; continue; }
            c = peek(); ++i;
            switch (c) {
                case 'n': out += '\n'; break;
                case 't': out += '\t'; break;
                case 'r': out += '\r'; break;
                case 'b': out += '\b'; break;
                case 'f': out += '\f'; break;
                case 'u': {
                    unsigned u = hex4();
                    if (u >= 0xD800 && u < 0xDC00 && i + 1 < s.size() && s[i] == '\\' && s[i + 1] == 'u') {
                        i += 2;
                        u = 0x10000 + ((u - 0xD800) << 10) + (hex4() - 0xDC00);
                    }
                    utf8(out, u);
                    break;
                }
                default: out += c;
            }
        }
        ++i;
        return out;
    }
    Json value() {
        if (++depth > 200) fail("nesting too deep");
        space();
        Json v;
        const char c = peek();
        if (c == '{') {
            v.kind_ = Json::Kind::Object;
            ++i; space();
            if (peek() == '}') ++i;
            else for (;;) {
                space();
                std::string key = string();
                space(); expect(':');
                v.object_[key] = value();
                space();
                if (peek() == ',') { ++i; continue; }
                expect('}');
                break;
            }
        } else if (c == '[') {
            v.kind_ = Json::Kind::Array;
            ++i; space();
            if (peek() == ']') ++i;
            else for (;;) {
                v.array_.push_back(value());
                space();
                if (peek() == ',') { ++i; continue; }
                expect(']');
                break;
            }
        } else if (c == '"') {
            v.kind_ = Json::Kind::String;
            v.text_ = string();
        } else if (word("true")) { v.kind_ = Json::Kind::Bool; v.bool_ = true; }
        else if (word("false")) { v.kind_ = Json::Kind::Bool; }
        else if (word("null")) {}
        else {
            const size_t from = i;
            while (i < s.size() && (std::isalnum(static_cast<unsigned char>(s[i])) || s[i] == '-' || s[i] == '+' || s[i] == '.')) ++i;
            v.kind_ = Json::Kind::Number;
            v.text_ = s.substr(from, i - from);
            char* end = nullptr;
            std::strtod(v.text_.c_str(), &end);
            if (v.text_.empty() || *end) fail("not a value");
        }
        --depth;
        return v;
    }
};

Json Json::parse(const std::string& text) {
    JsonParser p{text};
    Json v = p.value();
    p.space();
    if (p.i != text.size()) p.fail("trailing text");
    return v;
}
const Json& Json::get(const std::string& key) const {
    static const Json null;
    return has(key) ? object_.at(key) : null;
}
const Json& Json::at(const std::string& key) const {
    if (!has(key)) throw std::runtime_error("configuration: missing key '" + key + "'");
    return object_.at(key);
}
int64_t Json::as_int() const {
    if (kind_ != Kind::Number) throw std::runtime_error("configuration: expected a number");
    char* end = nullptr;
    const long long v = std::strtoll(text_.c_str(), &end, 10);
    if (!*end) return v;
    const double d = std::strtod(text_.c_str(), nullptr);
    if (d != static_cast<double>(static_cast<int64_t>(d))) throw std::runtime_error("configuration: expected an integer, found " + text_);
    return static_cast<int64_t>(d);
}
double Json::as_double() const {
    if (kind_ != Kind::Number) throw std::runtime_error("configuration: expected a number");
    return std::strtod(text_.c_str(), nullptr);
}
bool Json::as_bool() const {
    if (kind_ != Kind::Bool) throw std::runtime_error("configuration: expected true or false");
    return bool_;
}
const std::string& Json::as_string() const {
    if (kind_ != Kind::String) throw std::runtime_error("configuration: expected a string");
    return text_;
}
const std::vector<Json>& Json::as_array() const {
    if (kind_ != Kind::Array) throw std::runtime_error("configuration: expected a list");
    return array_;
}
const std::map<std::string, Json>& Json::as_object() const {
    if (kind_ != Kind::Object) throw std::runtime_error("configuration: expected an object");
    return object_;
}

}  // namespace vesper
