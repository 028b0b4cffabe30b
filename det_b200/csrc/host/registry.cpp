#include "registry.hpp"
#include "gguf.hpp"
#include "hybrid.hpp"
#include "qwen35.hpp"
#include <fstream>
#include <sstream>
#include <stdexcept>
#include <sys/stat.h>

namespace det {

static Json read_config(const std::string& dir) {
    std::ifstream f(dir + "/config.json", std::ios::binary);
    if (!f) throw std::runtime_error(dir + "/config.json: cannot be read");
    std::stringstream s;
    s << f.rdbuf();
    try {
        return Json::parse(s.str());
    } catch (const std::exception& ex) {
        throw std::runtime_error(dir + "/config.json: " + ex.what());
    }
}

static std::unique_ptr<Model> open_hybrid(const std::string& path, Backend* bk, const OpenOptions& o) {
    return HybridModel::load_dir(path, read_config(path), bk, o.max_ctx, o.max_batch, o.dtype);
}

const std::vector<Architecture>& architectures() {
    static const std::vector<Architecture> table = {
        {"qwen35", false,
         [](const std::string& path, Backend* bk, const OpenOptions& o) -> std::unique_ptr<Model> {
             std::string err;
             std::unique_ptr<Model> m = Qwen35Model::load(path, bk, o.max_ctx, o.max_batch, err);
             if (!m) throw std::runtime_error(err);
             return m;
         }},
        {"Fazilorn", true, open_hybrid},
        {"Dopipel", true, open_hybrid},
    };
    return table;
}

std::unique_ptr<Model> open_model(const std::string& path, Backend* bk, const OpenOptions& o) {
    struct stat sb;
    if (stat(path.c_str(), &sb) != 0) throw std::runtime_error(path + ": no such file or folder");
    const bool folder = S_ISDIR(sb.st_mode);
    std::string name;
    if (folder) {
        name = read_config(path).string("architecture");
    } else {
        std::string err;
        std::shared_ptr<Gguf> g = Gguf::open(path, err);
        if (!g) throw std::runtime_error(err);
        if (const std::string* a = g->str("general.architecture")) name = *a;
    }
    for (const Architecture& a : architectures())
        if (a.folder == folder && name == a.name) return a.open(path, bk, o);
    throw std::runtime_error(path + ": no model class for architecture '" + name + "'");
}

}  // namespace det
