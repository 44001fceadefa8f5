// A checkpoint folder: config.json as a JSON tree and model.safetensors as a table of named tensors over the mapped file.
#pragma once

#include <map>
#include <memory>
#include <string>
#include <utility>
#include <vector>

#include "common.cuh"

namespace forge {

struct Json {
    enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
    double num = 0;
    bool flag = false;
    std::string str;
    std::vector<Json> items;
    std::vector<std::pair<std::string, Json>> fields;
    const Json* get(const char* key) const {
        for (const auto& f : fields) if (f.first == key) return &f.second;
        return nullptr;
    }
};
int32_t json_parse(const char* text, size_t len, Json* out);

struct TensorView {
    std::string dtype;             // "BF16", "F16", "F32", "I32", ...
    std::vector<int64_t> shape;
    const uint8_t* data = nullptr;
    size_t bytes = 0;
    int64_t count() const { int64_t n = 1; for (int64_t s : shape) n *= s; return n; }
    float at(size_t i) const;      // BF16, F16 and F32
};

class Checkpoint {
public:
    ~Checkpoint();
    int32_t open(const char* dir);
    const Json& config() const { return config_; }
    // null and an error message if it is absent or has another shape ({} = scalar)
    const TensorView* tensor(const std::string& name, const std::vector<int64_t>& shape) const;
    // null if it is absent
    const TensorView* find(const std::string& name) const { auto it = tensors_.find(name); return it == tensors_.end() ? nullptr : &it->second; }
    int64_t parameters() const;

private:
    Json config_;
    std::map<std::string, TensorView> tensors_;
    void* map_ = nullptr;
    size_t map_len_ = 0;
};

}  // namespace forge
