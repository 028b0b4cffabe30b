#include "safetensors.hpp"
#include "json.hpp"
#include <cerrno>
#include <cstring>
#include <fcntl.h>
#include <stdexcept>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

namespace det {

static size_t element_bytes(const std::string& dtype) {
    if (dtype == "BF16" || dtype == "F16" || dtype == "I16" || dtype == "U16") return 2;
    if (dtype == "F32" || dtype == "I32" || dtype == "U32") return 4;
    if (dtype == "F64" || dtype == "I64" || dtype == "U64") return 8;
    if (dtype == "I8" || dtype == "U8" || dtype == "BOOL") return 1;
    return 0;
}

std::shared_ptr<SafeTensors> SafeTensors::open(const std::string& path) {
    auto fail = [&](const std::string& what) { throw std::runtime_error(path + ": " + what); };
    std::shared_ptr<SafeTensors> f(new SafeTensors());
    const int fd = ::open(path.c_str(), O_RDONLY);
    if (fd < 0) fail(std::strerror(errno));
    struct stat sb;
    if (fstat(fd, &sb) != 0 || sb.st_size < 8) {
        ::close(fd);
        fail("not a safetensors file");
    }
    f->size_ = (size_t)sb.st_size;
    void* p = mmap(nullptr, f->size_, PROT_READ, MAP_PRIVATE, fd, 0);
    ::close(fd);
    if (p == MAP_FAILED) {
        f->size_ = 0;
        fail("mmap failed");
    }
    f->map_ = static_cast<uint8_t*>(p);
    uint64_t n = 0;
    std::memcpy(&n, f->map_, 8);
    if (n > f->size_ - 8) fail("the header runs past the file");
    const Json head = Json::parse(reinterpret_cast<const char*>(f->map_ + 8), (size_t)n);
    if (head.kind != Json::Object) fail("the header is not an object");
    const uint8_t* data = f->map_ + 8 + n;
    const size_t room = f->size_ - 8 - (size_t)n;
    for (const auto& m : head.members) {
        if (m.first == "__metadata__") continue;
        SafeTensor t;
        t.dtype = m.second.string("dtype");
        for (const Json& d : m.second.at("shape").items) {
            if (d.kind != Json::Number || d.num < 0 || d.num > 1e12) fail(m.first + ": bad shape");
            t.shape.push_back((size_t)d.num);
        }
        const Json& off = m.second.at("data_offsets");
        if (off.items.size() != 2 || off.items[0].kind != Json::Number || off.items[1].kind != Json::Number) fail(m.first + ": bad offsets");
        const double a = off.items[0].num, b = off.items[1].num;
        if (a < 0 || b < a || b > (double)room) fail(m.first + ": offsets outside the file");
        t.data = data + (size_t)a;
        t.bytes = (size_t)b - (size_t)a;
        const size_t e = element_bytes(t.dtype);
        if (e == 0) fail(m.first + ": unknown type " + t.dtype);
        if (t.n_elems() * e != t.bytes) fail(m.first + ": size and shape disagree");
        f->tensors_[m.first] = std::move(t);
    }
    return f;
}
SafeTensors::~SafeTensors() {
    if (map_) munmap(map_, size_);
}
const SafeTensor* SafeTensors::find(const std::string& name) const {
    auto it = tensors_.find(name);
    return it == tensors_.end() ? nullptr : &it->second;
}

}  // namespace det
