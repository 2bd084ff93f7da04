// Reader of a safetensors file (host only): 8-byte little-endian header length, a JSON header name -> dtype, shape,
// data_offsets, then the data.  The file is mapped; tensors are views into the mapping.
#pragma once

#include <cstdint>
#include <cstring>
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include "json_lite.h"

namespace gptb200 {

struct TensorView {
    std::string dtype;
    std::vector<long long> shape;
    const uint8_t *data = nullptr;
    size_t bytes = 0;
    long long count() const
    {
        long long n = 1;
        for (long long d : shape) n *= d;
        return n;
    }
};

class SafeTensors
{
public:
    explicit SafeTensors(const std::string &path)
    {
        const int fd = open(path.c_str(), O_RDONLY);
        if (fd < 0) throw std::runtime_error("cannot open " + path);
        struct stat st{};
        if (fstat(fd, &st) != 0 || st.st_size < 8) {
            close(fd);
            throw std::runtime_error("not a safetensors file: " + path);
        }
        size_ = static_cast<size_t>(st.st_size);
        void *m = mmap(nullptr, size_, PROT_READ, MAP_PRIVATE, fd, 0);
        close(fd);
        if (m == MAP_FAILED) throw std::runtime_error("cannot map " + path);
        base_ = static_cast<const uint8_t *>(m);
        try {
            read_header(path);
        } catch (...) {
            munmap(const_cast<uint8_t *>(base_), size_);
            throw;
        }
    }
    SafeTensors(const SafeTensors &) = delete;
    SafeTensors &operator=(const SafeTensors &) = delete;
    ~SafeTensors() { munmap(const_cast<uint8_t *>(base_), size_); }

    bool has(const std::string &name) const { return tensors_.count(name) != 0; }
    const TensorView &get(const std::string &name) const
    {
        const auto it = tensors_.find(name);
        if (it == tensors_.end()) throw std::runtime_error("missing tensor '" + name + "'");
        return it->second;
    }
    const std::map<std::string, TensorView> &all() const { return tensors_; }

private:
    void read_header(const std::string &path)
    {
        uint64_t n = 0;
        for (int i = 0; i < 8; ++i) n |= static_cast<uint64_t>(base_[i]) << (8 * i);
        if (n > size_ - 8) throw std::runtime_error("header longer than the file: " + path);
        const Json header = Json::parse(std::string(reinterpret_cast<const char *>(base_ + 8), n));
        const size_t data0 = 8 + static_cast<size_t>(n);
        for (const auto &f : header.fields) {
            if (f.first == "__metadata__") continue;
            TensorView t;
            t.dtype = f.second.str("dtype");
            for (const Json &d : f.second.at("shape").items) t.shape.push_back(static_cast<long long>(d.number));
            const auto &o = f.second.at("data_offsets").items;
            if (o.size() != 2 || o[0].number < 0 || o[1].number < o[0].number || o[1].number > static_cast<double>(size_ - data0))
                throw std::runtime_error("tensor '" + f.first + "' lies outside the file");
            t.data = base_ + data0 + static_cast<size_t>(o[0].number);
            t.bytes = static_cast<size_t>(o[1].number - o[0].number);
            const size_t each = t.dtype == "BF16" || t.dtype == "F16" || t.dtype == "I16" ? 2 : t.dtype == "F32" || t.dtype == "I32" ? 4 : 0;
            if (each && t.bytes != each * static_cast<size_t>(t.count())) throw std::runtime_error("tensor '" + f.first + "': shape and size disagree");
            tensors_[f.first] = t;
        }
    }
    const uint8_t *base_ = nullptr;
    size_t size_ = 0;
    std::map<std::string, TensorView> tensors_;
};

}  // namespace gptb200
