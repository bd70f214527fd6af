#include "json.h"

#include <cstdio>
#include <cstdlib>

namespace cccc
{

class JsonReader
{
public:
    JsonReader(const std::string& s) : p_(s.c_str()), end_(s.c_str() + s.size()) {}
    bool document(Json* v) { return value(v, 0) && (space(), p_ == end_); }
    size_t at(const std::string& s) const { return (size_t)(p_ - s.c_str()); }

private:
    void space()
    {
        while (p_ < end_ && (*p_ == ' ' || *p_ == '\n' || *p_ == '\t' || *p_ == '\r')) { p_++; }
    }
    bool word(const char* w)
    {
        const char* q = p_;
        for (; *w; w++, q++)
        {
            if (q >= end_ || *q != *w) { return false; }
        }
        p_ = q;
        return true;
    }
    bool value(Json* v, int depth)
    {
        if (depth > 100) { return false; }
        space();
        if (p_ >= end_) { return false; }
        switch (*p_)
        {
        case '{':
            p_++;
            v->type_ = Json::OBJECT;
            space();
            if (p_ < end_ && *p_ == '}') { return p_++, true; }
            for (;;)
            {
                std::string key;
                space();
                if (!text(&key)) { return false; }
                space();
                if (p_ >= end_ || *p_++ != ':') { return false; }
                if (!value(&v->members_[key], depth + 1)) { return false; }
                space();
                if (p_ >= end_) { return false; }
                if (*p_ == '}') { return p_++, true; }
                if (*p_++ != ',') { return false; }
            }
        case '[':
            p_++;
            v->type_ = Json::ARRAY;
            space();
            if (p_ < end_ && *p_ == ']') { return p_++, true; }
            for (;;)
            {
                v->items_.emplace_back();
                if (!value(&v->items_.back(), depth + 1)) { return false; }
                space();
                if (p_ >= end_) { return false; }
                if (*p_ == ']') { return p_++, true; }
                if (*p_++ != ',') { return false; }
            }
        case '"': v->type_ = Json::STRING; return text(&v->text_);
        case 't': v->type_ = Json::BOOL; return v->flag_ = true, word("true");
        case 'f': v->type_ = Json::BOOL; return v->flag_ = false, word("false");
        case 'n': return word("null");
        default: return number(v);
        }
    }
    bool number(Json* v)
    {
        const char* q = p_;
        while (q < end_ && (*q == '-' || *q == '+' || *q == '.' || *q == 'e' || *q == 'E' || (*q >= '0' && *q <= '9'))) { q++; }
        const std::string s(p_, q);
        char* stop = nullptr;
        v->number_ = std::strtod(s.c_str(), &stop);
        if (s.empty() || *stop != '\0') { return false; }
        v->type_ = Json::NUMBER;
        p_ = q;
        return true;
    }
    bool hex4(unsigned int* out)
    {
        if (end_ - p_ < 4) { return false; }
        *out = 0;
        for (int i = 0; i < 4; i++)
        {
            const char c = *p_++;
            unsigned int d;
            if (c >= '0' && c <= '9') { d = (unsigned int)(c - '0'); }
            else if (c >= 'a' && c <= 'f') { d = (unsigned int)(c - 'a') + 10; }
            else if (c >= 'A' && c <= 'F') { d = (unsigned int)(c - 'A') + 10; }
            else { return false; }
            *out = *out * 16 + d;
        }
        return true;
    }
    bool text(std::string* out)
    {
        if (p_ >= end_ || *p_ != '"') { return false; }
        p_++;
        while (p_ < end_ && *p_ != '"')
        {
            if (*p_ != '\\')
            {
                out->push_back(*p_++);
                continue;
            }
            if (++p_ >= end_) { return false; }
            const char c = *p_++;
            unsigned int u, lo;
            switch (c)
            {
            case '"':
            case '\\':
            case '/': out->push_back(c); break;
            case 'b': out->push_back('\b'); break;
            case 'f': out->push_back('\f'); break;
            case 'n': out->push_back('\n'); break;
            case 'r': out->push_back('\r'); break;
            case 't': out->push_back('\t'); break;
            case 'u':
                if (!hex4(&u)) { return false; }
                if (u >= 0xD800 && u < 0xDC00)
                {
                    if (!word("\\u") || !hex4(&lo) || lo < 0xDC00 || lo > 0xDFFF) { return false; }
                    u = 0x10000 + ((u - 0xD800) << 10) + (lo - 0xDC00);
                }
                if (u < 0x80) { out->push_back((char)u); }
                else
                {
                    if (u < 0x800) { out->push_back((char)(0xC0 | (u >> 6))); }
                    else
                    {
                        if (u < 0x10000) { out->push_back((char)(0xE0 | (u >> 12))); }
                        else
                        {
                            out->push_back((char)(0xF0 | (u >> 18)));
                            out->push_back((char)(0x80 | ((u >> 12) & 0x3F)));
                        }
                        out->push_back((char)(0x80 | ((u >> 6) & 0x3F)));
                    }
                    out->push_back((char)(0x80 | (u & 0x3F)));
                }
                break;
            default: return false;
            }
        }
        return p_ < end_ && (p_++, true);
    }
    const char *p_, *end_;
};

bool Json::parse(const std::string& text, Json* out, std::string* err)
{
    *out = Json();
    JsonReader r(text);
    if (r.document(out)) { return true; }
    if (err) { *err = "malformed JSON near byte " + std::to_string(r.at(text)); }
    return false;
}

static const Json kNull;

const Json& Json::operator[](const std::string& key) const
{
    auto it = members_.find(key);
    return type_ == OBJECT && it != members_.end() ? it->second : kNull;
}

const Json& Json::operator[](size_t i) const { return type_ == ARRAY && i < items_.size() ? items_[i] : kNull; }

bool readFile(const std::string& path, std::string* out)
{
    FILE* f = std::fopen(path.c_str(), "rb");
    if (!f) { return false; }
    char buf[1 << 16];
    size_t n;
    out->clear();
    while ((n = std::fread(buf, 1, sizeof(buf), f)) > 0) { out->append(buf, n); }
    const bool ok = !std::ferror(f);
    std::fclose(f);
    return ok;
}

}    // namespace cccc
