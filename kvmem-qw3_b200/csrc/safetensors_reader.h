// safetensors container reader: maps the file and lists its tensors (an 8-byte little-endian header length, a JSON
// object name -> {dtype, shape, data_offsets}, then the data).  Host code only.
#pragma once

#include "json_reader.h"
#include "qb_internal.h"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <string>
#include <unordered_map>

namespace qbst {

struct Tensor {
    std::string dtype;
    std::vector<uint64_t> shape;
    const uint8_t *data = nullptr;
    uint64_t bytes = 0;
    uint64_t count() const { uint64_t n = 1; for (uint64_t d : shape) n *= d; return n; }
};

class File {
public:
    ~File() { if (base_) munmap(base_, size_); }
    int open(const char *path) {
        const int fd = ::open(path, O_RDONLY);
        if (fd < 0) return qb_fail(QB_ERR_INVALID, "safetensors: cannot open %s", path);
        struct stat st;
        if (fstat(fd, &st) != 0 || st.st_size < 8) { ::close(fd); return qb_fail(QB_ERR_INVALID, "safetensors: %s is too short", path); }
        size_ = (size_t)st.st_size;
        void *p = mmap(nullptr, size_, PROT_READ, MAP_PRIVATE, fd, 0);
        ::close(fd);
        if (p == MAP_FAILED) return qb_fail(QB_ERR_INVALID, "safetensors: cannot map %s", path);
        base_ = p;
        uint64_t hlen = 0;
        memcpy(&hlen, base_, 8);
        if (hlen > size_ - 8) return qb_fail(QB_ERR_INVALID, "safetensors: the header of %s points outside the file", path);
        qbjson::Value root;
        if (!qbjson::Parser((const char *)base_ + 8, (size_t)hlen).parse(root) || root.kind != qbjson::Value::Object)
            return qb_fail(QB_ERR_INVALID, "safetensors: the header of %s is malformed", path);
        const uint64_t room = size_ - 8 - hlen;
        for (const auto &m : root.members) {
            if (m.first == "__metadata__") continue;
            const qbjson::Value *dt = m.second.get("dtype"), *sh = m.second.get("shape"), *off = m.second.get("data_offsets");
            if (!dt || !sh || !off || off->items.size() != 2) return qb_fail(QB_ERR_INVALID, "safetensors: entry %s is malformed", m.first.c_str());
            Tensor t;
            t.dtype = dt->s;
            for (const qbjson::Value &d : sh->items) t.shape.push_back((uint64_t)d.num);
            const uint64_t a = (uint64_t)off->items[0].num, b = (uint64_t)off->items[1].num;
            if (a > b || b > room) return qb_fail(QB_ERR_INVALID, "safetensors: tensor %s points outside the file", m.first.c_str());
            t.data = (const uint8_t *)base_ + 8 + hlen + a;
            t.bytes = b - a;
            tensors_.emplace(m.first, std::move(t));
        }
        return QB_OK;
    }
    const Tensor *find(const std::string &name) const {
        auto it = tensors_.find(name);
        return it == tensors_.end() ? nullptr : &it->second;
    }

private:
    void *base_ = nullptr;
    size_t size_ = 0;
    std::unordered_map<std::string, Tensor> tensors_;
};

}  // namespace qbst
