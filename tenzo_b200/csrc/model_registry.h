// Model families and the files they load from: a folder with config.json (its "architecture" names the family) and the
// weights the family expects beside it.
#pragma once
#include <stdint.h>

#include <string>
#include <vector>

#include "../../include/tenzo_ext.h"
#include "json.h"

namespace tz {

class EngineCore;

struct OpenOptions {
    std::string dir;
    tenzo_ext_options_t opt;
    int compute = TENZO_COMPUTE_BF16;
};

struct ModelFamily {
    const char* architecture;
    EngineCore* (*open)(const Json& config, const OpenOptions& o);
};

// A file-scope ModelRegistration in a family's source file makes the family known wherever that file is linked in.
struct ModelRegistration {
    explicit ModelRegistration(const ModelFamily& f);
};
const std::vector<ModelFamily>& model_families();
EngineCore* open_model(const OpenOptions& o);
std::string read_text_file(const std::string& path);      // throws IoError

struct IoError : std::runtime_error { using std::runtime_error::runtime_error; };
struct ParseError : std::runtime_error { using std::runtime_error::runtime_error; };

// model.safetensors: an 8-byte little-endian header length, that many bytes of JSON (name -> dtype, shape, data_offsets),
// then the data. The file stays mapped while the object lives.
struct TensorView {
    std::string dtype;
    std::vector<long long> shape;
    const unsigned char* data = nullptr;
    size_t bytes = 0;
    long long count() const {
        long long n = 1;
        for (long long s : shape) n *= s;
        return n;
    }
};
class SafeTensors {
public:
    explicit SafeTensors(const std::string& path);
    ~SafeTensors();
    SafeTensors(const SafeTensors&) = delete;
    SafeTensors& operator=(const SafeTensors&) = delete;
    const TensorView& at(const std::string& name) const;             // throws ParseError when absent
    const TensorView& bf16(const std::string& name, const std::vector<long long>& shape) const;   // shape entries < 0: any
    std::vector<float> floats(const std::string& name, const std::vector<long long>& shape) const;
    std::map<std::string, TensorView> tensors;

private:
    void* base = nullptr;
    size_t size = 0;
};

}  // namespace tz
