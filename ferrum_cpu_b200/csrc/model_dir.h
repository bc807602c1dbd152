// A model folder: config.json and model.safetensors. Host code only.
#pragma once
#include <cstddef>
#include <cstdint>
#include <map>
#include <string>
#include <utility>
#include <vector>

namespace fc {

// A parsed JSON value. Objects keep their keys in file order.
struct Json {
    enum Kind { Null, Bool, Number, String, Array, Object } kind = Null;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<Json> items;
    std::vector<std::pair<std::string, Json>> members;
    const Json* find(const char* key) const;       // null when absent or not an object
    bool has(const char* key) const { const Json* j = find(key); return j && j->kind != Null; }
};
bool json_parse(const char* text, size_t n, Json* out, std::string* error);

struct TensorView {
    std::string dtype;                  // as the file names it: BF16, F32, F16, I32, ...
    std::vector<int64_t> shape;
    const uint8_t* data = nullptr;      // inside the mapped file
    size_t nbytes = 0;
};

// The folder opened: the configuration parsed, the tensor file mapped and its directory checked (offsets inside the
// file, sizes that agree with shapes and types).
class ModelDir {
public:
    ~ModelDir();
    int open_config(const char* dir);   // config.json only
    int open(const char* dir);          // both
    const TensorView* tensor(const std::string& name) const;
    Json config;
private:
    std::map<std::string, TensorView> tensors_;
    void* map_ = nullptr;
    size_t map_bytes_ = 0;
};

}  // namespace fc
