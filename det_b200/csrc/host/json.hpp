// A small JSON reader for model folders: config.json and the header of a safetensors file.
#pragma once
#include <cstddef>
#include <string>
#include <utility>
#include <vector>

namespace det {

struct Json {
    enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<Json> items;                              // Array
    std::vector<std::pair<std::string, Json>> members;    // Object, in file order

    // Parses all of `text`; throws std::runtime_error naming the offset on malformed input.
    static Json parse(const char* text, size_t len);
    static Json parse(const std::string& s) { return parse(s.data(), s.size()); }

    const Json* find(const std::string& key) const;        // null when absent (or not an object)
    bool has(const std::string& key) const { const Json* j = find(key); return j && j->kind != Null; }
    // Typed members; throw std::runtime_error naming the key when absent or of another kind.
    const Json& at(const std::string& key) const;
    double number(const std::string& key) const;
    size_t size(const std::string& key) const;             // a non-negative integer
    const std::string& string(const std::string& key) const;
};

}  // namespace det
