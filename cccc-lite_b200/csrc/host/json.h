// A small JSON reader for model configurations, safetensors headers and request lines.
#pragma once

#include <map>
#include <string>
#include <vector>

namespace cccc
{

class Json
{
public:
    enum Type
    {
        NUL,
        BOOL,
        NUMBER,
        STRING,
        ARRAY,
        OBJECT
    };
    // false with *err set on malformed text (or text after the value)
    static bool parse(const std::string& text, Json* out, std::string* err);

    Type type() const { return type_; }
    bool isNull() const { return type_ == NUL; }
    bool has(const std::string& key) const { return type_ == OBJECT && members_.count(key) != 0; }
    const Json& operator[](const std::string& key) const;    // a null value where there is no such member
    const Json& operator[](size_t i) const;
    size_t size() const { return type_ == ARRAY ? items_.size() : members_.size(); }
    const std::map<std::string, Json>& members() const { return members_; }
    bool boolean(bool otherwise = false) const { return type_ == BOOL ? flag_ : otherwise; }
    double number(double otherwise = 0.0) const { return type_ == NUMBER ? number_ : otherwise; }
    const std::string& string() const { return text_; }

private:
    friend class JsonReader;
    Type type_ = NUL;
    bool flag_ = false;
    double number_ = 0.0;
    std::string text_;
    std::vector<Json> items_;
    std::map<std::string, Json> members_;
};

bool readFile(const std::string& path, std::string* out);

}    // namespace cccc
