// Where a model's tensors come from: a safetensors file, or seeded noise of the right shapes (benchmarks).
#pragma once

#include <cstdint>
#include <map>
#include <string>
#include <vector>

namespace cccc
{

class TensorSource
{
public:
    virtual ~TensorSource() = default;
    virtual bool has(const std::string& name) const = 0;
    // The tensor as BF16 bits, row-major; false with *err set if it is missing or its shape is another.
    virtual bool readBf16(const std::string& name, const std::vector<int64_t>& shape, std::vector<uint16_t>* out, std::string* err) = 0;
};

// An 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets), the data.
// BF16, F32 and F16 tensors are read (rounded to BF16 where they hold more).
class SafetensorsFile : public TensorSource
{
public:
    SafetensorsFile() = default;
    ~SafetensorsFile() override;
    SafetensorsFile(const SafetensorsFile&) = delete;
    SafetensorsFile& operator=(const SafetensorsFile&) = delete;
    bool open(const std::string& path, std::string* err);
    bool has(const std::string& name) const override { return entries_.count(name) != 0; }
    bool readBf16(const std::string& name, const std::vector<int64_t>& shape, std::vector<uint16_t>* out, std::string* err) override;

private:
    struct Entry
    {
        std::string dtype;
        std::vector<int64_t> shape;
        uint64_t begin = 0, end = 0;
    };
    int fd_ = -1;
    uint64_t base_ = 0;
    std::map<std::string, Entry> entries_;
};

// Every tensor exists and holds N(0, 1 / row length) values from one seeded block; vectors near 1.
class NoiseSource : public TensorSource
{
public:
    explicit NoiseSource(uint64_t seed);
    bool has(const std::string&) const override { return true; }
    bool readBf16(const std::string& name, const std::vector<int64_t>& shape, std::vector<uint16_t>* out, std::string* err) override;

private:
    std::vector<float> block_;
};

}    // namespace cccc
