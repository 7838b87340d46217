#include "dl/json.h"

#include <charconv>
#include <cmath>
#include <stdexcept>

namespace dl {

struct JsonReader {
    std::string_view s;
    std::size_t at = 0;
    int depth = 0;

    [[noreturn]] void fail(const char* what) const {
        throw std::invalid_argument("JSON: " + std::string(what) + " at byte " + std::to_string(at));
    }
    void space() { while (at < s.size() && (s[at] == ' ' || s[at] == '\t' || s[at] == '\n' || s[at] == '\r')) ++at; }
    char peek() { space(); if (at >= s.size()) fail("unexpected end"); return s[at]; }
    bool take(char c) { if (peek() != c) return false; ++at; return true; }
    void word(std::string_view w) { if (s.substr(at, w.size()) != w) fail("unknown word"); at += w.size(); }

    static void put_utf8(std::string& out, std::uint32_t c) {
        if (c < 0x80) { out += static_cast<char>(c); return; }
        if (c < 0x800) { out += static_cast<char>(0xc0 | (c >> 6)); }
        else if (c < 0x10000) { out += static_cast<char>(0xe0 | (c >> 12)); out += static_cast<char>(0x80 | ((c >> 6) & 0x3f)); }
        else { out += static_cast<char>(0xf0 | (c >> 18)); out += static_cast<char>(0x80 | ((c >> 12) & 0x3f)); out += static_cast<char>(0x80 | ((c >> 6) & 0x3f)); }
        out += static_cast<char>(0x80 | (c & 0x3f));
    }
    std::uint32_t hex4() {
        std::uint32_t v = 0;
        if (at + 4 > s.size()) fail("short escape");
        const auto r = std::from_chars(s.data() + at, s.data() + at + 4, v, 16);
        if (r.ptr != s.data() + at + 4) fail("bad escape");
        at += 4;
        return v;
    }
    std::string string() {
        if (!take('"')) fail("expected a string");
        std::string out;
        while (true) {
            if (at >= s.size()) fail("unterminated string");
            const char c = s[at++];
            if (c == '"') return out;
            if (c != '\\') { out += c; continue; }
            if (at >= s.size()) fail("unterminated string");
            switch (s[at++]) {
            case '"': out += '"'; break;
            case '\\': out += '\\'; break;
            case '/': out += '/'; break;
            case 'b': out += '\b'; break;
            case 'f': out += '\f'; break;
            case 'n': out += '\n'; break;
            case 'r': out += '\r'; break;
            case 't': out += '\t'; break;
            case 'u': {
                std::uint32_t v = hex4();
                if (v >= 0xd800 && v < 0xdc00 && s.substr(at, 2) == "\\u") { at += 2; v = 0x10000 + ((v - 0xd800) << 10) + (hex4() - 0xdc00); }
                put_utf8(out, v);
                break;
            }
            default: fail("bad escape");
            }
        }
    }
    Json value(const std::string& path) {
        if (++depth > 64) fail("nested too deeply");
        Json v;
        v.path_ = path;
        const char c = peek();
        if (c == '{') {
            v.kind_ = Json::Kind::object;
            ++at;
            if (!take('}')) {
                do {
                    space();
                    const std::string key = string();
                    if (!take(':')) fail("expected ':'");
                    v.members_[key] = value(path.empty() ? key : path + "." + key);
                } while (take(','));
                if (!take('}')) fail("expected '}'");
            }
        } else if (c == '[') {
            v.kind_ = Json::Kind::array;
            ++at;
            if (!take(']')) {
                do v.items_.push_back(value(path + "[" + std::to_string(v.items_.size()) + "]")); while (take(','));
                if (!take(']')) fail("expected ']'");
            }
        } else if (c == '"') {
            v.kind_ = Json::Kind::string;
            v.text_ = string();
        } else if (c == 't') { word("true"); v.kind_ = Json::Kind::boolean; v.flag_ = true; }
        else if (c == 'f') { word("false"); v.kind_ = Json::Kind::boolean; }
        else if (c == 'n') { word("null"); }
        else {
            v.kind_ = Json::Kind::number;
            const auto r = std::from_chars(s.data() + at, s.data() + s.size(), v.number_);
            if (r.ec != std::errc{}) fail("bad number");
            at = static_cast<std::size_t>(r.ptr - s.data());
        }
        --depth;
        return v;
    }
};

Json Json::parse(std::string_view text) {
    JsonReader reader{text};
    Json v = reader.value("");
    reader.space();
    if (reader.at != text.size()) reader.fail("text after the value");
    return v;
}

void Json::complain(const char* expected) const {
    throw std::invalid_argument("configuration: '" + (path_.empty() ? std::string("(root)") : path_) + "' must be " + expected);
}
const Json& Json::at(const std::string& key) const {
    if (kind_ != Kind::object) complain("an object");
    const auto found = members_.find(key);
    if (found == members_.end()) throw std::invalid_argument("configuration: '" + (path_.empty() ? key : path_ + "." + key) + "' is missing");
    return found->second;
}
const std::vector<Json>& Json::items() const { if (kind_ != Kind::array) complain("an array"); return items_; }
const std::map<std::string, Json>& Json::members() const { if (kind_ != Kind::object) complain("an object"); return members_; }
double Json::number() const { if (kind_ != Kind::number) complain("a number"); return number_; }
std::int64_t Json::integer() const {
    if (kind_ != Kind::number || number_ != std::floor(number_) || std::fabs(number_) > 9e15) complain("an integer");
    return static_cast<std::int64_t>(number_);
}
std::int64_t Json::positive() const {
    const auto v = integer();
    if (v <= 0) complain("a positive integer");
    return v;
}
const std::string& Json::text() const { if (kind_ != Kind::string) complain("a string"); return text_; }

}  // namespace dl
