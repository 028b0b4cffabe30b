// The safetensors container: an 8-byte little-endian header length, a JSON header (name -> dtype, shape, data_offsets), then
// the tensors' bytes.  Read through a memory map.
#pragma once
#include <cstdint>
#include <memory>
#include <string>
#include <unordered_map>
#include <vector>

namespace det {

struct SafeTensor {
    std::string dtype;            // "BF16", "F32", "I32", ...
    std::vector<size_t> shape;    // outermost first
    const uint8_t* data = nullptr;
    size_t bytes = 0;
    size_t n_elems() const {
        size_t n = 1;
        for (size_t d : shape) n *= d;
        return n;
    }
};

class SafeTensors {
  public:
    // Throws std::runtime_error on an unreadable or malformed file (offsets and sizes are checked against the file).
    static std::shared_ptr<SafeTensors> open(const std::string& path);
    ~SafeTensors();
    SafeTensors(const SafeTensors&) = delete;
    SafeTensors& operator=(const SafeTensors&) = delete;
    const SafeTensor* find(const std::string& name) const;
    size_t count() const { return tensors_.size(); }

  private:
    SafeTensors() = default;
    uint8_t* map_ = nullptr;
    size_t size_ = 0;
    std::unordered_map<std::string, SafeTensor> tensors_;
};

}  // namespace det
