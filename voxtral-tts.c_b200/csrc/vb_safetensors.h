/*
 * vb_safetensors.h - memory-mapped safetensors file: 8-byte little-endian header length, JSON
 * header (name -> dtype, shape, data_offsets), raw data.
 */
#ifndef VB_SAFETENSORS_H
#define VB_SAFETENSORS_H

#include <stddef.h>
#include <stdint.h>

#include <map>
#include <string>
#include <vector>

namespace vb {

struct Tensor {
    std::string dtype;            /* "BF16", "F32", "I32", ... */
    std::vector<int64_t> shape;
    const void *data = nullptr;   /* into the mapping */
    size_t bytes = 0;
};

class SafeTensors {
public:
    SafeTensors() = default;
    SafeTensors(const SafeTensors &) = delete;
    SafeTensors &operator=(const SafeTensors &) = delete;
    ~SafeTensors();
    bool open(const char *path, std::string *err);
    const Tensor *find(const std::string &name) const;
    size_t count() const { return tensors_.size(); }

private:
    void *map_ = nullptr;
    size_t size_ = 0;
    std::map<std::string, Tensor> tensors_;
};

} // namespace vb

#endif
