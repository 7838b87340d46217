// JSON values of configuration files and safetensors headers.
#pragma once

#include <cstdint>
#include <map>
#include <string>
#include <string_view>
#include <vector>

namespace dl {

// Errors (parse errors, missing keys, wrong types) are std::invalid_argument with the key's path in the text.
class Json {
public:
    enum class Kind { null, boolean, number, string, array, object };
    static Json parse(std::string_view text);

    Kind kind() const { return kind_; }
    bool is_null() const { return kind_ == Kind::null; }
    bool has(const std::string& key) const { return kind_ == Kind::object && members_.count(key) && !members_.at(key).is_null(); }
    const Json& at(const std::string& key) const;          // required member
    const std::vector<Json>& items() const;                // array
    const std::map<std::string, Json>& members() const;    // object
    double number() const;
    std::int64_t integer() const;                          // a number without a fraction
    std::int64_t positive() const;
    const std::string& text() const;

private:
    friend struct JsonReader;
    [[noreturn]] void complain(const char* expected) const;
    Kind kind_ = Kind::null;
    bool flag_ = false;
    double number_ = 0.0;
    std::string text_, path_;
    std::vector<Json> items_;
    std::map<std::string, Json> members_;
};

}  // namespace dl
