// Readers of a model folder: config.json (a small JSON tree) and model.safetensors (tensor table + raw data).
#pragma once
#include <stdint.h>

#include <map>
#include <memory>
#include <string>
#include <vector>

#include "common.cuh"

namespace onellm {

struct Json {
    enum Kind { NUL, BOOL, NUMBER, STRING, ARRAY, OBJECT } kind = NUL;
    bool boolean = false;
    double number = 0.0;
    std::string text;
    std::vector<Json> items;
    std::map<std::string, Json> fields;

    // member of an object, NULL when absent (or not an object)
    const Json* find(const char* key) const
    {
        const auto it = fields.find(key);
        return it == fields.end() ? nullptr : &it->second;
    }
    bool is_null() const { return kind == NUL; }
};

// Parses a whole text; ONELLM_ERR_IO with the place in the message when it is not JSON.
int json_parse(const std::string& text, Json* out);
int read_text_file(const std::string& path, std::string* out);

// Required members, reported by `where` (e.g. "layers[2].mixer.left") when missing or of the wrong kind.
int json_object(const Json& j, const char* key, const char* where, const Json** out);
int json_int(const Json& j, const char* key, const char* where, int* out);
int json_float(const Json& j, const char* key, const char* where, double* out);

struct SafeTensor {
    std::string dtype;          // "BF16", "F32", "F16", "I32"
    std::vector<int64_t> shape;
    size_t begin = 0, end = 0;  // bytes inside the data section
};

// An opened .safetensors file: 8-byte little-endian header length, JSON header, data.
class SafeTensors {
  public:
    ~SafeTensors();
    int open(const std::string& path);
    const SafeTensor* find(const std::string& name) const;
    // The raw bytes of a tensor.
    int read(const SafeTensor& t, std::vector<char>* out);

  private:
    std::string path_;
    FILE* f_ = nullptr;
    size_t data_start_ = 0, data_bytes_ = 0;
    std::map<std::string, SafeTensor> tensors_;
};

}  // namespace onellm
