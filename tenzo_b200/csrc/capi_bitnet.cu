// The part of the extern "C" boundary that belongs to the BitNet engine: creation from a tenzo_config_t, its weight setters
// and checkpoint loader, its INT8 KV rows and its measurement aids (reference: include/tenzo.h:92-193).
#include <cstring>
#include <stdexcept>
#include <string>

#include "../../include/tenzo_kernels.h"
#include "capi_common.h"
#include "engine.h"

namespace tz {
tenzo_status_t load_model_files(Engine& e, const char* weights_path, const char* mlir_path);

static Engine& bitnet(tenzo_engine_t engine) {
    Engine* e = dynamic_cast<Engine*>(engine->impl);
    if (!e) throw std::invalid_argument("this call belongs to BitNet engines");
    return *e;
}
}  // namespace tz

using tz::bitnet;
using tz::guarded;
using tz::live;

extern "C" {

tenzo_engine_t tenzo_ext_create_engine(const tenzo_config_t* config, const tenzo_ext_options_t* opt) {
    tenzo_engine_t handle = nullptr;
    guarded([&]() -> tenzo_status_t {
        tenzo_config_t c = config ? *config : tenzo_default_config();
        tenzo_ext_options_t o = opt ? *opt : tenzo_ext_default_options();
        if (c.kv_mode && std::strcmp(c.kv_mode, "int8_fused") != 0 && std::strcmp(c.kv_mode, "paged_int8") != 0)
            throw std::invalid_argument(std::string("kv_mode '") + c.kv_mode + "' is not implemented; only int8_fused and paged_int8");
        int n_dev = 0;
        if (cudaGetDeviceCount(&n_dev) != cudaSuccess || n_dev == 0)
            throw std::runtime_error("no CUDA device is visible; this library has no CPU path");
        tz::Engine* e = new tz::Engine(c, o);
        handle = new tenzo_engine_opaque{e};
        return TENZO_SUCCESS;
    });
    return handle;
}

tenzo_engine_t tenzo_create_engine(const tenzo_config_t* config) { return tenzo_ext_create_engine(config, nullptr); }

tenzo_status_t tenzo_set_layer_weights(tenzo_engine_t engine, int layer_idx, const tenzo_layer_weights_t* weights) {
    if (!live(engine) || !weights) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        if (layer_idx < 0 || layer_idx >= engine->impl->L) throw std::out_of_range("layer index outside [0, num_layers)");
        bitnet(engine).set_layer(layer_idx, *weights);
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_set_final_norm(tenzo_engine_t engine, const float* norm_w) {
    if (!live(engine) || !norm_w) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        bitnet(engine).set_final_norm(norm_w);
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_set_lm_head_f32(tenzo_engine_t engine, const float* embed_w, int, int) {
    if (!live(engine) || !embed_w) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::set_error("the fp32 LM head is outside the quantized decode path; quantise per row and use tenzo_set_lm_head_i8");
    return TENZO_ERROR_UNSUPPORTED;
}

tenzo_status_t tenzo_set_lm_head_i8(tenzo_engine_t engine, const int8_t* embed_w, const float* embed_scales,
                                    int vocab_size, int hidden_size) {
    if (!live(engine) || !embed_w || !embed_scales) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        if (vocab_size != engine->impl->V || hidden_size != engine->impl->h)
            throw std::invalid_argument("LM head shape differs from the engine configuration");
        bitnet(engine).set_lm_head(embed_w, embed_scales);
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_load_model(tenzo_engine_t engine, const char* weights_path, const char* mlir_path) {
    if (!live(engine) || !weights_path || !mlir_path) return TENZO_ERROR_INVALID_ARGUMENT;
    tenzo_status_t inner = TENZO_SUCCESS;
    tenzo_status_t outer = guarded([&]() -> tenzo_status_t {
        inner = tz::load_model_files(bitnet(engine), weights_path, mlir_path);
        return inner;
    });
    return outer;
}

static tenzo_status_t kv_copy(tenzo_engine_t engine, int seq, int layer, void* k, void* v, void* sk, void* sv, int len,
                              bool to_device) {
    if (!live(engine) || !k || !v || !sk || !sv) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        tz::Engine& e = bitnet(engine);
        if (seq < 0 || seq >= e.batch || layer < 0 || layer >= e.L || len < 0 || len > e.cfg.max_seq_len)
            throw std::out_of_range("sequence, layer or length out of range");
        cudaStreamSynchronize(e.stream);
        const int nkv = e.cfg.num_kv_heads;
        if (e.paged) {
            if (to_device) e.reserve_blocks(seq, len);            // an import brings its own blocks
            else if (e.n_blocks[seq] * tz::Engine::kBlock < len) throw std::out_of_range("the sequence holds fewer tokens than asked for");
        }
        const int run = e.paged ? tz::Engine::kBlock : (len > 0 ? len : 1);   // tokens that are contiguous in the cache
        for (int hh = 0; hh < nkv; ++hh) {
            for (int t0 = 0; t0 < len; t0 += run) {
                const size_t n = (size_t)(len - t0 < run ? len - t0 : run);
                const size_t row = e.kv_row(seq, layer, hh, t0);
                const size_t hb = (size_t)hh * len + t0;
                cudaError_t c0, c1, c2, c3;
                if (to_device) {
                    c0 = cudaMemcpy(e.cache_k + row * 128, (const int8_t*)k + hb * 128, n * 128, cudaMemcpyHostToDevice);
                    c1 = cudaMemcpy(e.cache_v + row * 128, (const int8_t*)v + hb * 128, n * 128, cudaMemcpyHostToDevice);
                    c2 = cudaMemcpy(e.scale_k + row, (const float*)sk + hb, n * 4, cudaMemcpyHostToDevice);
                    c3 = cudaMemcpy(e.scale_v + row, (const float*)sv + hb, n * 4, cudaMemcpyHostToDevice);
                } else {
                    c0 = cudaMemcpy((int8_t*)k + hb * 128, e.cache_k + row * 128, n * 128, cudaMemcpyDeviceToHost);
                    c1 = cudaMemcpy((int8_t*)v + hb * 128, e.cache_v + row * 128, n * 128, cudaMemcpyDeviceToHost);
                    c2 = cudaMemcpy((float*)sk + hb, e.scale_k + row, n * 4, cudaMemcpyDeviceToHost);
                    c3 = cudaMemcpy((float*)sv + hb, e.scale_v + row, n * 4, cudaMemcpyDeviceToHost);
                }
                if (c0 != cudaSuccess || c1 != cudaSuccess || c2 != cudaSuccess || c3 != cudaSuccess)
                    throw std::runtime_error("KV copy failed");
            }
        }
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_ext_kv_import(tenzo_engine_t engine, int seq, int layer, const int8_t* k, const int8_t* v,
                                   const float* sk, const float* sv, int len) {
    return kv_copy(engine, seq, layer, (void*)k, (void*)v, (void*)sk, (void*)sv, len, true);
}

tenzo_status_t tenzo_ext_kv_export(tenzo_engine_t engine, int seq, int layer, int8_t* k, int8_t* v, float* sk,
                                   float* sv, int len) {
    return kv_copy(engine, seq, layer, k, v, sk, sv, len, false);
}

float tenzo_ext_bench_gemv_stack(tenzo_engine_t engine, int iters, unsigned long long* launches) {
    if (!live(engine) || iters <= 0) return -1.0f;
    float ms = -1.0f;
    guarded([&]() -> tenzo_status_t {
        ms = bitnet(engine).bench_gemv_stack(iters, launches);
        return TENZO_SUCCESS;
    });
    return ms;
}

int tenzo_ext_persistent_phase_ns(tenzo_engine_t engine, unsigned long long* out8, int reset) {
    if (!live(engine) || !out8) return -1;
    tz::Engine* be = dynamic_cast<tz::Engine*>(engine->impl);
    if (!be) return 0;
    tz::Engine& e = *be;
    if (!e.pc_usable() || !e.pc_phase_ns) return 0;
    cudaStreamSynchronize(e.stream);
    if (cudaMemcpy(out8, e.pc_phase_ns, 8 * sizeof(unsigned long long), cudaMemcpyDeviceToHost) != cudaSuccess) return -1;
    if (reset == 2) {                      // experiments: out8 has room for 72 values, the optional timeline follows the sums
        if (cudaMemcpy(out8, e.pc_phase_ns, 72 * sizeof(unsigned long long), cudaMemcpyDeviceToHost) != cudaSuccess) return -1;
    } else if (reset) {
        cudaMemset(e.pc_phase_ns, 0, 8 * sizeof(unsigned long long));
    }
    return 1;
}

tenzo_status_t tenzo_ext_rope_tables(int max_seq, int head_dim, float rope_theta, float* cos_host, float* sin_host) {
    if (max_seq <= 0 || head_dim <= 0 || (head_dim & 1) || !cos_host || !sin_host) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::rope_tables_host(max_seq, head_dim, rope_theta > 0.0f ? rope_theta : 10000.0f, cos_host, sin_host);
    return TENZO_SUCCESS;
}

}  // extern "C"
