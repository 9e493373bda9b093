// ---------------------------------------------------------------------------
// model_loader.cu -- model directories read into device memory.
//
// 1. The reference's on-disk format, cdna3::runtime::ModelLoader
// (cdna3-prims/include/cdna3/runtime/model_loader.hpp:83-204).
// A model directory holds meta.json (flat: n_layers, hidden, n_heads,
// n_kv_heads, head_dim, ffn_dim, vocab_size, optional rope_theta, qkv_bias and --
// an extension -- "dtype": "bf16") and one raw little-endian 16-bit file per
// tensor: embed_tokens.bin, lm_head.bin, final_norm.bin and, per layer i,
// layer_<i>_{q,k,v,o}_proj.bin, layer_<i>_{q,k,v}_bias.bin (with qkv_bias),
// layer_<i>_{gate,up,down}_proj.bin, layer_<i>_norm_{attn,mlp}.bin.
// Unlike the reference, which throws, every failure is a status code.
//
// 2. config.json + model.safetensors: config.json's "architecture" names an entry of the
// registry (model.hpp), which lists the tensors it needs with their shapes.  A safetensors
// file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape,
// data_offsets) and the data; it is read through a file mapping.
// ---------------------------------------------------------------------------
#include "common.cuh"
#include "b200p_runtime.h"
#include "model.hpp"
#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <map>
#include <string>
#include <vector>
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

namespace b200p {
namespace { ArchitectureEntry*& registry() { static ArchitectureEntry* head = nullptr; return head; } }
ArchitectureEntry::ArchitectureEntry(const char* name, int (*configure)(b200p_model*, std::vector<TensorWant>*),
                                     int (*build)(struct ::b200p_session*, const b200p_model*))
    : a{name, configure, build}, next(registry()) { registry() = this; }
const Architecture* find_architecture(const std::string& name) {
    for (ArchitectureEntry* e = registry(); e; e = e->next) if (name == e->a.name) return &e->a;
    return nullptr;
}
LlamaCreate& llama_session_create() { static LlamaCreate fn = nullptr; return fn; }
} // namespace b200p

namespace {
using namespace b200p;

// The minimal flat-JSON reader of model_loader.hpp:103-129: "key": value pairs, values kept as text.
bool read_meta(const std::string& path, std::map<std::string, std::string>& kv) {
    FILE* f = std::fopen(path.c_str(), "rb");
    if (!f) return false;
    std::string src;
    char buf[4096];
    size_t n;
    while ((n = std::fread(buf, 1, sizeof buf, f)) > 0) src.append(buf, n);
    std::fclose(f);
    size_t pos = 0;
    while (pos < src.size()) {
        const size_t qs = src.find('"', pos); if (qs == std::string::npos) break;
        const size_t qe = src.find('"', qs + 1); if (qe == std::string::npos) break;
        const std::string key = src.substr(qs + 1, qe - qs - 1);
        const size_t colon = src.find(':', qe); if (colon == std::string::npos) break;
        size_t vs = colon + 1;
        while (vs < src.size() && (src[vs] == ' ' || src[vs] == '\t' || src[vs] == '\n' || src[vs] == '\r')) ++vs;
        std::string val;
        if (vs < src.size() && src[vs] == '"') {
            const size_t ve = src.find('"', vs + 1); if (ve == std::string::npos) break;
            val = src.substr(vs + 1, ve - vs - 1); pos = ve + 1;
        } else {
            size_t ve = vs;
            while (ve < src.size() && src[ve] != ',' && src[ve] != '}' && src[ve] != '\n') ++ve;
            val = src.substr(vs, ve - vs); pos = ve;
            while (!val.empty() && (val.back() == ' ' || val.back() == '\r' || val.back() == '\t')) val.pop_back();
        }
        kv[key] = val;
    }
    return true;
}

int parse_meta(const char* dir, b200p_model_config* c, int* qkv_bias, int* dtype) {
    std::map<std::string, std::string> kv;
    if (!read_meta(std::string(dir) + "/meta.json", kv)) return B200P_E_IO;
    const char* need[] = {"n_layers", "hidden", "n_heads", "n_kv_heads", "head_dim", "ffn_dim", "vocab_size"};
    int* dst[] = {&c->n_layers, &c->hidden, &c->n_heads, &c->n_kv_heads, &c->head_dim, &c->ffn_dim, &c->vocab_size};
    for (int i = 0; i < 7; ++i) {
        auto it = kv.find(need[i]);
        if (it == kv.end()) return B200P_E_IO;
        char* end = nullptr;
        const long v = std::strtol(it->second.c_str(), &end, 10);
        if (end == it->second.c_str() || v <= 0) return B200P_E_IO;
        *dst[i] = int(v);
    }
    c->rope_theta = kv.count("rope_theta") ? std::strtof(kv["rope_theta"].c_str(), nullptr) : 10000.0f;
    if (qkv_bias) *qkv_bias = kv.count("qkv_bias") && (kv["qkv_bias"] == "1" || kv["qkv_bias"] == "true");
    if (dtype) *dtype = (kv.count("dtype") && (kv["dtype"] == "bf16" || kv["dtype"] == "bfloat16")) ? B200P_BF16 : B200P_F16;
    return B200P_OK;
}

// load_tensor (model_loader.hpp:89-98): n_elems raw 16-bit values -> device memory.
int load_tensor(b200p_model* m, const std::string& path, size_t n_elems, const void** out) {
    FILE* f = std::fopen(path.c_str(), "rb");
    if (!f) return B200P_E_IO;
    std::vector<uint16_t> host(n_elems);
    const size_t got = std::fread(host.data(), 2, n_elems, f);
    std::fclose(f);
    if (got != n_elems) return B200P_E_IO;                       // short read
    void* dev = nullptr;
    if (cudaError_t e = cudaMalloc(&dev, n_elems * 2)) return int(e);
    m->owned.push_back(dev);
    if (cudaError_t e = cudaMemcpy(dev, host.data(), n_elems * 2, cudaMemcpyHostToDevice)) return int(e);
    *out = dev;
    return B200P_OK;
}

bool read_text(const std::string& path, std::string* out) {
    FILE* f = std::fopen(path.c_str(), "rb");
    if (!f) return false;
    char buf[65536];
    size_t n;
    while ((n = std::fread(buf, 1, sizeof buf, f)) > 0) out->append(buf, n);
    std::fclose(f);
    return true;
}

int element_bytes(int dtype) { return dtype == B200P_F32 || dtype == B200P_I32 ? 4 : 2; }

size_t element_count(const std::vector<long long>& shape) {
    size_t n = 1;
    for (long long d : shape) n *= size_t(d);
    return n;
}

// A read-only mapping of a whole file.
struct FileMap {
    void* base = MAP_FAILED; size_t bytes = 0;
    explicit FileMap(const std::string& path) {
        const int fd = ::open(path.c_str(), O_RDONLY);
        if (fd < 0) return;
        struct stat sb;
        if (::fstat(fd, &sb) == 0 && sb.st_size > 0) {
            bytes = size_t(sb.st_size);
            base = ::mmap(nullptr, bytes, PROT_READ, MAP_PRIVATE, fd, 0);
        }
        ::close(fd);
    }
    ~FileMap() { if (base != MAP_FAILED) ::munmap(base, bytes); }
    bool ok() const { return base != MAP_FAILED; }
};

// The wanted tensors of a safetensors file into device memory, dtypes as stored.
int load_safetensors(b200p_model* m, const std::string& path, const std::vector<TensorWant>& want) {
    FileMap f(path);
    if (!f.ok() || f.bytes < 8) return B200P_E_IO;
    const unsigned char* p = static_cast<const unsigned char*>(f.base);
    uint64_t hlen = 0;
    for (int i = 0; i < 8; ++i) hlen |= uint64_t(p[i]) << (8 * i);
    if (hlen > f.bytes - 8) return B200P_E_IO;
    Json head;
    if (!Json::parse(reinterpret_cast<const char*>(p + 8), size_t(hlen), &head) || head.kind != Json::Object) return B200P_E_IO;
    const unsigned char* data = p + 8 + hlen;
    const size_t data_bytes = f.bytes - 8 - size_t(hlen);
    for (const TensorWant& t : want) {
        const Json* e = head.get(t.name.c_str());
        const Json *dt = e ? e->get("dtype") : nullptr, *sh = e ? e->get("shape") : nullptr, *off = e ? e->get("data_offsets") : nullptr;
        if (!dt || !sh || !off || off->items.size() != 2) return B200P_E_IO;
        TensorRef r;
        if (dt->str == "BF16") r.dtype = B200P_BF16;
        else if (dt->str == "F16") r.dtype = B200P_F16;
        else if (dt->str == "F32") r.dtype = B200P_F32;
        else if (dt->str == "I32") r.dtype = B200P_I32;
        else return B200P_E_DTYPE;
        for (const Json& d : sh->items) r.shape.push_back((long long)(d.num));
        if (r.shape != t.shape) return B200P_E_DIM;
        const size_t bytes = element_count(r.shape) * element_bytes(r.dtype);
        const double a = off->items[0].num, b = off->items[1].num;
        if (a < 0 || b < a || b > double(data_bytes) || size_t(b) - size_t(a) != bytes) return B200P_E_IO;
        void* dev = nullptr;
        if (cudaError_t ce = cudaMalloc(&dev, bytes ? bytes : 16)) return int(ce);
        m->owned.push_back(dev);
        if (cudaError_t ce = cudaMemcpy(dev, data + size_t(a), bytes, cudaMemcpyHostToDevice)) return int(ce);
        r.dev = dev;
        m->tensors[t.name] = r;
    }
    return B200P_OK;
}

// config.json's text into m->config, m->arch and the architecture's spec.
int configure(b200p_model* m, const char* text, size_t n, std::vector<TensorWant>* want) {
    if (!Json::parse(text, n, &m->config)) return B200P_E_IO;
    const Json* a = m->config.get("architecture");
    if (!a || a->kind != Json::String) return B200P_E_IO;
    m->arch = find_architecture(a->str);
    if (!m->arch) return B200P_E_OP;
    return m->arch->configure(m, want);
}

} // namespace

extern "C" int b200p_model_read_meta(const char* model_dir, b200p_model_config* cfg, int* qkv_bias, int* dtype) {
    if (!model_dir || !cfg) return B200P_E_NULL;
    return parse_meta(model_dir, cfg, qkv_bias, dtype);
}

extern "C" void b200p_model_free(b200p_model* m) {
    if (!m) return;
    for (void* p : m->owned) cudaFree(p);
    delete m;
}

extern "C" b200p_model* b200p_model_load(const char* model_dir, int* status) {
    int dummy; if (!status) status = &dummy;
    *status = B200P_OK;
    if (!model_dir) { *status = B200P_E_NULL; return nullptr; }
    b200p_model* m = new b200p_model();
    std::string text;
    if (read_text(std::string(model_dir) + "/config.json", &text)) {
        std::vector<TensorWant> want;
        int rc = configure(m, text.data(), text.size(), &want);
        if (!rc && sm_count() <= 0) rc = B200P_E_NO_DEVICE;
        if (!rc) rc = load_safetensors(m, std::string(model_dir) + "/model.safetensors", want);
        if (rc) { *status = rc; b200p_model_free(m); return nullptr; }
        return m;
    }
    int bias = 0, dtype = B200P_F16;
    if ((*status = parse_meta(model_dir, &m->w.cfg, &bias, &dtype))) { delete m; return nullptr; }
    if (b200p::sm_count() <= 0) { *status = B200P_E_NO_DEVICE; delete m; return nullptr; }
    m->w.dtype = dtype;
    const b200p_model_config& c = m->w.cfg;
    const size_t H = size_t(c.hidden), F = size_t(c.ffn_dim), V = size_t(c.vocab_size);
    const size_t qd = size_t(c.n_heads) * c.head_dim, kvd = size_t(c.n_kv_heads) * c.head_dim;
    const std::string dir(model_dir);
    auto top = [&](const char* name) { return dir + "/" + name + ".bin"; };
    int rc = load_tensor(m, top("embed_tokens"), V * H, &m->w.embed_tokens);
    if (!rc) rc = load_tensor(m, top("lm_head"), V * H, &m->w.lm_head);
    if (!rc) rc = load_tensor(m, top("final_norm"), H, &m->w.final_norm);
    m->layers.assign(size_t(c.n_layers), b200p_layer_weights{});
    for (int i = 0; i < c.n_layers && !rc; ++i) {
        auto lp = [&](const char* t) { return dir + "/layer_" + std::to_string(i) + "_" + t + ".bin"; };
        b200p_layer_weights& L = m->layers[size_t(i)];
        rc = load_tensor(m, lp("q_proj"), qd * H, &L.Wq);
        if (!rc) rc = load_tensor(m, lp("k_proj"), kvd * H, &L.Wk);
        if (!rc) rc = load_tensor(m, lp("v_proj"), kvd * H, &L.Wv);
        if (!rc) rc = load_tensor(m, lp("o_proj"), H * qd, &L.Wo);
        if (bias) {
            if (!rc) rc = load_tensor(m, lp("q_bias"), qd, &L.bq);
            if (!rc) rc = load_tensor(m, lp("k_bias"), kvd, &L.bk);
            if (!rc) rc = load_tensor(m, lp("v_bias"), kvd, &L.bv);
        }
        if (!rc) rc = load_tensor(m, lp("gate_proj"), F * H, &L.Wgate);
        if (!rc) rc = load_tensor(m, lp("up_proj"), F * H, &L.Wup);
        if (!rc) rc = load_tensor(m, lp("down_proj"), H * F, &L.Wdown);
        if (!rc) rc = load_tensor(m, lp("norm_attn"), H, &L.norm_attn);
        if (!rc) rc = load_tensor(m, lp("norm_mlp"), H, &L.norm_mlp);
    }
    if (rc) { *status = rc; b200p_model_free(m); return nullptr; }
    m->w.layers = m->layers.data();
    return m;
}

extern "C" const b200p_model_weights* b200p_model_weights_of(const b200p_model* m) { return m ? &m->w : nullptr; }

extern "C" b200p_model* b200p_model_create(const char* config_json, int n_tensors, const char* const* names, const void* const* pointers,
                                           const int* dtypes, const int* ranks, const long long* shapes, int* status) {
    int dummy; if (!status) status = &dummy;
    *status = B200P_OK;
    if (!config_json || (n_tensors > 0 && (!names || !pointers || !dtypes || !ranks || !shapes))) { *status = B200P_E_NULL; return nullptr; }
    b200p_model* m = new b200p_model();
    std::vector<TensorWant> want;
    int rc = configure(m, config_json, std::strlen(config_json), &want);
    for (int i = 0; !rc && i < n_tensors; ++i) {
        TensorRef r;
        r.dev = pointers[i]; r.dtype = dtypes[i];
        r.shape.assign(shapes, shapes + ranks[i]);
        shapes += ranks[i];
        if (!r.dev) rc = B200P_E_NULL;
        m->tensors[names[i]] = r;
    }
    for (size_t i = 0; !rc && i < want.size(); ++i) {
        auto it = m->tensors.find(want[i].name);
        if (it == m->tensors.end()) rc = B200P_E_IO;
        else if (it->second.shape != want[i].shape) rc = B200P_E_DIM;
    }
    if (rc) { *status = rc; b200p_model_free(m); return nullptr; }
    return m;
}

extern "C" int b200p_model_describe(const b200p_model* m, char* architecture, int cap, b200p_model_config* cfg) {
    if (!m || !cfg) return B200P_E_NULL;
    *cfg = m->w.cfg;
    if (architecture && cap > 0) {
        std::strncpy(architecture, m->arch ? m->arch->name : "Llama", size_t(cap) - 1);
        architecture[cap - 1] = '\0';
    }
    return B200P_OK;
}
