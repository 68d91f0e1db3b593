// Model directories: config.json names the architecture (model_plan.h has the registry and the configuration readers),
// model.safetensors holds the weights — 8 bytes little-endian header length, that many bytes of JSON
// (name -> dtype, shape, data_offsets), then the tensor bytes. The file is mapped; tensors go from the page cache through
// the engine's pinned staging buffers like those of a GGUF file (gguf.cu).
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cmath>
#include <cstring>
#include <fstream>
#include <memory>
#include <sstream>
#include <string>
#include <vector>

#include "engine.h"
#include "model_plan.h"
#include "sp_common.cuh"

using sp::set_error;

namespace {

struct Mapping {
    const uint8_t* p = nullptr;
    size_t n = 0;
    int fd = -1;
    ~Mapping() {
        if (p) munmap((void*)p, n);
        if (fd >= 0) close(fd);
    }
    bool open_file(const std::string& path) {
        fd = ::open(path.c_str(), O_RDONLY);
        struct stat sb;
        if (fd < 0 || fstat(fd, &sb) != 0 || sb.st_size <= 0) return false;
        void* m = mmap(nullptr, (size_t)sb.st_size, PROT_READ, MAP_PRIVATE, fd, 0);
        if (m == MAP_FAILED) return false;
        p = (const uint8_t*)m;
        n = (size_t)sb.st_size;
        return true;
    }
};

int dtype_of(const std::string& s) {
    if (s == "BF16") return sp::T_BF16;
    if (s == "F16") return sp::T_F16;
    if (s == "F32") return sp::T_F32;
    return -1;
}

}  // namespace

// A plan-driven engine without weights from the text of its configuration file.
int sp_engine_from_config_impl(const char* text, size_t n, bool f32, const SpModelDesc& run, sp::Engine** out) {
    sp::Json cfg;
    if (!sp::Json::parse(text, n, &cfg) || cfg.type != sp::Json::OBJ) { set_error("the model configuration is not a JSON object"); return SP_ERR_IO; }
    const sp::Json* arch = cfg.get("architecture");
    if (!arch || arch->type != sp::Json::STR) { set_error("the model configuration names no architecture"); return SP_ERR_ARG; }
    const sp::ArchEntry* a = sp::find_arch(arch->str);
    if (!a || !a->read_plan) { set_error("architecture '" + arch->str + "' is not supported by the CUDA engine"); return SP_ERR_DTYPE; }
    sp::ModelPlan plan;
    const int st = a->read_plan(cfg, &plan);
    if (st != SP_OK) return st;
    if (run.max_ctx <= 0) { set_error("max_ctx must be positive"); return SP_ERR_ARG; }
    *out = new sp::Engine(run, plan, f32);
    return SP_OK;
}

int sp_engine_from_dir_impl(const char* dir, bool f32, const SpModelDesc& run, sp::Engine** out) {
    const std::string base(dir);
    std::ifstream in(base + "/config.json", std::ios::binary);
    if (!in) { set_error("cannot open " + base + "/config.json"); return SP_ERR_IO; }
    std::stringstream ss;
    ss << in.rdbuf();
    const std::string text = ss.str();
    Mapping map;
    if (!map.open_file(base + "/model.safetensors")) { set_error("cannot map " + base + "/model.safetensors"); return SP_ERR_IO; }
    uint64_t hn = 0;
    if (map.n < 8) { set_error("safetensors file truncated"); return SP_ERR_IO; }
    std::memcpy(&hn, map.p, 8);
    sp::Json head;
    if (hn > map.n - 8 || !sp::Json::parse((const char*)map.p + 8, (size_t)hn, &head) || head.type != sp::Json::OBJ) {
        set_error("safetensors header truncated or malformed");
        return SP_ERR_IO;
    }
    sp::Engine* raw = nullptr;
    int st = sp_engine_from_config_impl(text.data(), text.size(), f32, run, &raw);
    if (st != SP_OK) return st;
    std::unique_ptr<sp::Engine> eng(raw);
    const uint64_t data0 = 8 + hn, avail = map.n - data0;
    for (const auto& kv : head.obj) {
        if (kv.first == "__metadata__") continue;
        const sp::Json *dt = kv.second.get("dtype"), *shape = kv.second.get("shape"), *off = kv.second.get("data_offsets");
        if (!dt || dt->type != sp::Json::STR || !shape || shape->type != sp::Json::ARR || !off || off->type != sp::Json::ARR || off->arr.size() != 2) {
            set_error("safetensors entry '" + kv.first + "' is malformed");
            return SP_ERR_IO;
        }
        const int dtype = dtype_of(dt->str);
        if (dtype < 0) {
            if (dt->str == "I32") continue;  // integer tables belong to designs that read them
            set_error("tensor '" + kv.first + "' has unsupported dtype " + dt->str);
            return SP_ERR_DTYPE;
        }
        // sizes and offsets are words of a file: checked before use
        std::vector<int64_t> dims;
        double numel = 1;
        for (const sp::Json& v : shape->arr) {
            if (v.type != sp::Json::NUM || !(v.num >= 1 && v.num <= 1e12) || v.num != std::floor(v.num)) { set_error("tensor '" + kv.first + "' has a bad shape"); return SP_ERR_SHAPE; }
            dims.push_back((int64_t)v.num);
            numel *= v.num;
        }
        const double b = off->arr[0].num, e = off->arr[1].num;
        if (!(b >= 0 && e >= b && e <= (double)avail) || b != std::floor(b) || e != std::floor(e)) { set_error("tensor '" + kv.first + "' data out of file bounds"); return SP_ERR_IO; }
        if (numel * sp::block_bytes(dtype) != e - b) { set_error("tensor '" + kv.first + "' byte count does not match its shape"); return SP_ERR_SHAPE; }
        if (dims.empty()) dims.push_back(1);  // a single number
        if (dims.size() > 2) { set_error("tensor '" + kv.first + "' has more than two dimensions"); return SP_ERR_SHAPE; }
        st = eng->set_tensor(kv.first.c_str(), dtype, dims.data(), (int)dims.size(), map.p + data0 + (size_t)b, (size_t)(e - b));
        if (st != SP_OK) return st;
    }
    st = eng->finalize();
    if (st != SP_OK) return st;
    *out = eng.release();
    return SP_OK;
}
