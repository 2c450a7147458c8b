/* vb_safetensors.cpp - safetensors reader (vb_safetensors.h). Every offset is checked against the
 * file before a pointer is handed out. */
#include "vb_safetensors.h"

#include <fcntl.h>
#include <string.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include "vb_json.h"

namespace vb {

SafeTensors::~SafeTensors() {
    if (map_) munmap(map_, size_);
}

const Tensor *SafeTensors::find(const std::string &name) const {
    auto it = tensors_.find(name);
    return it == tensors_.end() ? nullptr : &it->second;
}

static size_t dtype_bytes(const std::string &d) {
    if (d == "BF16" || d == "F16" || d == "I16" || d == "U16") return 2;
    if (d == "F32" || d == "I32" || d == "U32") return 4;
    if (d == "F64" || d == "I64" || d == "U64") return 8;
    if (d == "I8" || d == "U8" || d == "BOOL") return 1;
    return 0;
}

bool SafeTensors::open(const char *path, std::string *err) {
    auto fail = [&](const std::string &what) {
        *err = std::string(path) + ": " + what;
        return false;
    };
    const int fd = ::open(path, O_RDONLY);
    if (fd < 0) return fail("cannot be opened");
    struct stat sb;
    if (fstat(fd, &sb) != 0 || sb.st_size < 8) { ::close(fd); return fail("not a safetensors file"); }
    size_ = (size_t)sb.st_size;
    map_ = mmap(nullptr, size_, PROT_READ, MAP_PRIVATE, fd, 0);
    ::close(fd);
    if (map_ == MAP_FAILED) { map_ = nullptr; return fail("cannot be mapped"); }
    const unsigned char *base = (const unsigned char *)map_;
    uint64_t hn = 0;
    for (int i = 7; i >= 0; i--) hn = (hn << 8) | base[i];
    if (hn > size_ - 8) return fail("header longer than the file");
    Json head;
    std::string je;
    if (!json_parse((const char *)base + 8, (size_t)hn, &head, &je) || head.kind != Json::OBJECT) return fail("header: " + je);
    const size_t data0 = 8 + (size_t)hn, data_n = size_ - data0;
    for (const auto &m : head.members) {
        if (m.first == "__metadata__") continue;
        const Json *dt = m.second.get("dtype"), *sh = m.second.get("shape"), *off = m.second.get("data_offsets");
        if (!dt || dt->kind != Json::STRING || !sh || sh->kind != Json::ARRAY || !off || off->items.size() != 2)
            return fail("entry " + m.first + " is incomplete");
        Tensor t;
        t.dtype = dt->text;
        double n = 1.0;
        for (const Json &d : sh->items) { t.shape.push_back((int64_t)d.number); n *= d.number; }
        const double lo = off->items[0].number, hi = off->items[1].number;
        if (lo < 0 || hi < lo || hi > (double)data_n) return fail("entry " + m.first + " lies outside the file");
        const size_t eb = dtype_bytes(t.dtype);
        if (!eb || n * (double)eb != hi - lo) return fail("entry " + m.first + ": size and shape do not agree");
        t.bytes = (size_t)(hi - lo);
        t.data = base + data0 + (size_t)lo;
        tensors_[m.first] = t;
    }
    return true;
}

} // namespace vb
