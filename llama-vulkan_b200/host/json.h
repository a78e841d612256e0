// A small JSON reader for model configurations, safetensors headers and trace steps.
#ifndef LLAVA_B200_JSON_H
#define LLAVA_B200_JSON_H

#include <string>
#include <utility>
#include <vector>

#include "types.h"

class json_value {
public:
    enum class kind { null, boolean, number, text, array, object };

    // false (with a message) unless the whole text is one JSON value
    static bool parse(const char* text, size_t size, json_value* out, std::string* error);
    static bool parse(const std::string& text, json_value* out, std::string* error) { return parse(text.data(), text.size(), out, error); }

    kind type() const { return type_; }
    bool is_null() const { return type_ == kind::null; }
    bool is_object() const { return type_ == kind::object; }
    bool is_array() const { return type_ == kind::array; }
    bool is_number() const { return type_ == kind::number; }
    bool is_text() const { return type_ == kind::text; }
    bool boolean() const { return number_ != 0; }
    double number() const { return number_; }
    const std::string& text() const { return text_; }
    const std::vector<json_value>& items() const { return items_; }
    const std::vector<std::pair<std::string, json_value>>& members() const { return members_; }
    const json_value* find(const std::string& key) const;     // null when absent (or not an object)
    // a non-negative integer below 2^32 / any finite number / a text; false when it is something else
    bool as_u32(u32* out) const;
    bool as_u64(u64* out) const;
    bool as_float(float* out) const;

private:
    friend struct json_parser;
    kind type_ = kind::null;
    double number_ = 0;
    std::string text_;
    std::vector<json_value> items_;
    std::vector<std::pair<std::string, json_value>> members_;
};

#endif
