#include "tensor_source.h"

#include "json.h"

#include <cmath>
#include <cstring>
#include <fcntl.h>
#include <random>
#include <sys/stat.h>
#include <unistd.h>

namespace cccc
{

namespace
{
bool fail(std::string* err, const std::string& what)
{
    if (err) { *err = what; }
    return false;
}

uint16_t roundBf16(float f)
{
    uint32_t u;
    std::memcpy(&u, &f, 4);
    if ((u & 0x7fffffffu) > 0x7f800000u) { return (uint16_t)((u >> 16) | 0x40u); }
    return (uint16_t)((u + 0x7fffu + ((u >> 16) & 1u)) >> 16);
}

float widenHalf(uint16_t h)
{
    const int e = (h >> 10) & 31, m = h & 1023;
    const float s = (h & 0x8000) ? -1.f : 1.f;
    if (e == 31) { return m ? NAN : s * INFINITY; }
    return e == 0 ? s * std::ldexp((float)m, -24) : s * std::ldexp((float)(m + 1024), e - 25);
}

bool readAt(int fd, uint64_t off, uint64_t len, void* dst)
{
    uint8_t* p = (uint8_t*)dst;
    while (len > 0)
    {
        const ssize_t n = ::pread(fd, p, len > (1ull << 30) ? (1ull << 30) : len, (off_t)off);
        if (n <= 0) { return false; }
        p += n;
        off += (uint64_t)n;
        len -= (uint64_t)n;
    }
    return true;
}

std::string shapeText(const std::vector<int64_t>& s)
{
    std::string t = "[";
    for (size_t i = 0; i < s.size(); i++) { t += (i ? ", " : "") + std::to_string(s[i]); }
    return t + "]";
}

uint64_t elements(const std::vector<int64_t>& s)
{
    uint64_t n = 1;
    for (int64_t d : s) { n *= (uint64_t)d; }
    return n;
}
}    // namespace

SafetensorsFile::~SafetensorsFile()
{
    if (fd_ >= 0) { ::close(fd_); }
}

bool SafetensorsFile::open(const std::string& path, std::string* err)
{
    fd_ = ::open(path.c_str(), O_RDONLY);
    if (fd_ < 0) { return fail(err, "cannot open '" + path + "'"); }
    struct stat st;
    uint8_t head[8];
    if (fstat(fd_, &st) != 0 || st.st_size < 8 || !readAt(fd_, 0, 8, head)) { return fail(err, "'" + path + "' is no safetensors file"); }
    uint64_t len = 0;
    for (int i = 7; i >= 0; i--) { len = len << 8 | head[i]; }
    const uint64_t size = (uint64_t)st.st_size;
    if (len > size - 8) { return fail(err, "'" + path + "' is truncated"); }
    std::string text((size_t)len, '\0');
    Json j;
    std::string e;
    if (!readAt(fd_, 8, len, &text[0]) || !Json::parse(text, &j, &e) || j.type() != Json::OBJECT)
    {
        return fail(err, "'" + path + "': bad header: " + e);
    }
    base_ = 8 + len;
    for (const auto& m : j.members())
    {
        if (m.first == "__metadata__") { continue; }
        Entry t;
        t.dtype = m.second["dtype"].string();
        const Json& s = m.second["shape"];
        for (size_t i = 0; i < s.size(); i++) { t.shape.push_back((int64_t)s[i].number(-1)); }
        const Json& o = m.second["data_offsets"];
        t.begin = (uint64_t)o[(size_t)0].number();
        t.end = (uint64_t)o[(size_t)1].number();
        if (o.size() != 2 || t.begin > t.end || t.end > size - base_) { return fail(err, "'" + path + "': tensor '" + m.first + "' lies outside the file"); }
        entries_[m.first] = t;
    }
    return true;
}

bool SafetensorsFile::readBf16(const std::string& name, const std::vector<int64_t>& shape, std::vector<uint16_t>* out, std::string* err)
{
    auto it = entries_.find(name);
    if (it == entries_.end()) { return fail(err, "tensor '" + name + "' is missing"); }
    const Entry& t = it->second;
    if (t.shape != shape) { return fail(err, "tensor '" + name + "' has shape " + shapeText(t.shape) + ", not " + shapeText(shape)); }
    const uint64_t n = elements(shape), esz = t.dtype == "F32" ? 4 : 2;
    if (t.dtype != "BF16" && t.dtype != "F32" && t.dtype != "F16") { return fail(err, "tensor '" + name + "' has dtype " + t.dtype); }
    if (t.end - t.begin != n * esz) { return fail(err, "tensor '" + name + "' has the wrong size"); }
    out->resize(n);
    if (esz == 2)
    {
        if (!readAt(fd_, base_ + t.begin, n * 2, out->data())) { return fail(err, "cannot read tensor '" + name + "'"); }
        if (t.dtype == "F16")
        {
            for (auto& v : *out) { v = roundBf16(widenHalf(v)); }
        }
        return true;
    }
    std::vector<float> f(n);
    if (!readAt(fd_, base_ + t.begin, n * 4, f.data())) { return fail(err, "cannot read tensor '" + name + "'"); }
    for (uint64_t i = 0; i < n; i++) { (*out)[i] = roundBf16(f[i]); }
    return true;
}

NoiseSource::NoiseSource(uint64_t seed)
{
    std::mt19937_64 rng(seed);
    std::normal_distribution<float> d;
    block_.resize(1 << 18);
    for (auto& v : block_) { v = d(rng); }
}

bool NoiseSource::readBf16(const std::string& name, const std::vector<int64_t>& shape, std::vector<uint16_t>* out, std::string*)
{
    const uint64_t n = elements(shape);
    const bool bias = name.size() > 2 && name.compare(name.size() - 2, 2, ".b") == 0;
    const float s = shape.size() == 2 ? 1.f / std::sqrt((float)shape[1]) : 0.1f, c = shape.size() == 2 || bias ? 0.f : (shape.empty() ? 0.5f : 1.f);
    size_t off = std::hash<std::string>()(name) % block_.size();
    std::vector<uint16_t> bits(block_.size());
    for (size_t i = 0; i < block_.size(); i++) { bits[i] = roundBf16(c + s * block_[i]); }
    out->resize(n);
    for (uint64_t i = 0; i < n;)
    {
        const uint64_t m = std::min<uint64_t>(n - i, block_.size() - off);
        std::memcpy(out->data() + i, bits.data() + off, m * 2);
        i += m;
        off = 0;
    }
    return true;
}

}    // namespace cccc
