// A loaded model and the registry of decoder architectures (host only).
//
// b200p_model holds a model's configuration and its tensors in device memory.  Two kinds of directories are read
// (model_loader.cu): the export format of the Llama-style runtime (meta.json + one .bin per tensor), and config.json +
// model.safetensors, whose "architecture" names an entry of the registry.  A decoder registers itself from its own
// translation unit, so a library linked without that unit simply does not know the architecture.
#pragma once
#include "json.hpp"
#include "b200p_runtime.h"
#include <map>
#include <memory>
#include <string>
#include <vector>

namespace b200p {

struct TensorRef {
    const void* dev = nullptr;                 // device memory, row-major
    int dtype = 0;                             // B200P_BF16, B200P_F16, B200P_F32 or B200P_I32
    std::vector<long long> shape;
};

// What a decoder needs: filled by its configure(), used by the loader to find and check the tensors.
struct TensorWant { std::string name; std::vector<long long> shape; };

struct Architecture {
    const char* name;                          // config.json's "architecture"
    // Reads m->config into m->spec and m->w.cfg and lists the tensors.  Host only; a status code.
    int (*configure)(b200p_model* m, std::vector<TensorWant>* tensors);
    // Builds the decoder's part of a session (session.cuh).
    int (*build)(struct ::b200p_session* s, const b200p_model* m);
};

const Architecture* find_architecture(const std::string& name);
struct ArchitectureEntry {                     // static object: registers at load time
    Architecture a;
    ArchitectureEntry* next;
    ArchitectureEntry(const char* name, int (*configure)(b200p_model*, std::vector<TensorWant>*),
                      int (*build)(struct ::b200p_session*, const b200p_model*));
};

// b200p_session_create when the library holds the Llama-style decoder (decoder_gqa.cu sets it), null otherwise.
using LlamaCreate = b200p_session* (*)(const b200p_model_weights*, int, int, int*);
LlamaCreate& llama_session_create();

} // namespace b200p

struct b200p_model {
    b200p_model_weights w{};                   // cfg of every model; the pointer table of Llama-style ones
    std::vector<b200p_layer_weights> layers;
    std::vector<void*> owned;
    const b200p::Architecture* arch = nullptr; // null: the Llama-style decoder of b200p_session_create
    b200p::Json config;
    std::shared_ptr<void> spec;                // the architecture's own configuration
    std::map<std::string, b200p::TensorRef> tensors;
};
