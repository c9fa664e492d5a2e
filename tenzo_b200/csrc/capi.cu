// extern "C" boundary: the fourteen tenzo.h entry points (reference: include/tenzo.h:92-193,
// implemented in src/runtime/TenzoEngine.cpp:2086-2204) and the additive tenzo_ext.h calls.
// No exception crosses this file; failures become the reference's status codes and a message
// retrievable through tenzo_ext_last_error().
#include <cstring>
#include <new>
#include <stdexcept>
#include <string>
#include <vector>

#include "../../include/tenzo.h"
#include "../../include/tenzo_ext.h"
#include "../../include/tenzo_kernels.h"
#include "capi_common.h"
#include "model_registry.h"
#include "sampler.h"

using tz::guarded;
using tz::live;

extern "C" {

const char* tenzo_get_version(void) { return TENZO_VERSION_STRING; }

tenzo_config_t tenzo_default_config(void) {
    tenzo_config_t c;
    c.hidden_size = 2560;
    c.num_q_heads = 20;
    c.num_kv_heads = 5;
    c.head_dim = 128;
    c.num_layers = 30;
    c.ffn_dim = 6912;
    c.vocab_size = 128256;
    c.max_seq_len = 8192;
    c.kv_mode = "int8_fused";
    c.device = "cpu";   // kept for struct-level compatibility (TenzoEngine.cpp:2103); the engine is CUDA regardless
    return c;
}

tenzo_sampling_params_t tenzo_default_sampling_params(void) {
    tenzo_sampling_params_t p;
    p.temperature = 0.7f;
    p.top_p = 0.9f;
    p.top_k = 40;
    p.repetition_penalty = 1.15f;
    return p;
}

tenzo_ext_options_t tenzo_ext_default_options(void) {
    tenzo_ext_options_t o;
    o.batch = 1;
    o.rope_theta = 10000.0f;
    o.use_graph = -1;
    o.use_pdl = -1;
    o.persistent = -1;
    o.attention_mode = -1;
    return o;
}

void tenzo_destroy_engine(tenzo_engine_t engine) {
    if (!engine) return;
    delete engine->impl;
    delete engine;
}

void tenzo_reset(tenzo_engine_t engine) {
    if (!live(engine)) return;
    try {
        engine->impl->reset_kv();                  // TenzoEngine.cpp:213-215, :242-246
    } catch (const std::exception& ex) {
        tz::set_error(ex.what());
    }
}

int tenzo_get_seq_len(tenzo_engine_t engine) { return live(engine) ? engine->impl->seq_len[0] : 0; }

tenzo_status_t tenzo_prefill_token(tenzo_engine_t engine, int token_id) {
    if (!live(engine)) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        if (engine->impl->batch != 1) throw std::invalid_argument("batched engine: use tenzo_ext_prefill_tokens");
        engine->impl->prefill(&token_id);
        return TENZO_SUCCESS;
    });
}

int tenzo_generate_step(tenzo_engine_t engine, int cur_token, const tenzo_sampling_params_t* params,
                        const int* past_tokens, int past_tokens_len) {
    if (!live(engine)) return -1;
    int out = -1;
    tenzo_status_t st = guarded([&]() -> tenzo_status_t {
        tz::EngineCore& e = *engine->impl;
        if (e.batch != 1) throw std::invalid_argument("batched engine: use tenzo_ext_generate_step");
        const tenzo_sampling_params_t p = params ? *params : tenzo_default_sampling_params();   // :1729-1732
        e.generate(&cur_token, &out);
        const bool penalised = p.repetition_penalty != 1.0f && past_tokens && past_tokens_len > 0;
        if (p.temperature > 0.0f || penalised) out = e.sample(p, past_tokens, past_tokens_len);
        return TENZO_SUCCESS;
    });
    return st == TENZO_SUCCESS ? out : -1;
}

// ---------------------------------------------------------------------------------------------
// extension
// ---------------------------------------------------------------------------------------------

tenzo_engine_t tenzo_ext_open_model(const char* model_dir, const tenzo_ext_options_t* opt, int compute) {
    tenzo_engine_t handle = nullptr;
    guarded([&]() -> tenzo_status_t {
        if (!model_dir || (compute != TENZO_COMPUTE_BF16 && compute != TENZO_COMPUTE_F32)) throw std::invalid_argument("bad model folder or compute type");
        int n_dev = 0;
        if (cudaGetDeviceCount(&n_dev) != cudaSuccess || n_dev == 0)
            throw std::runtime_error("no CUDA device is visible; this library has no CPU path");
        tz::OpenOptions o;
        o.dir = model_dir;
        o.opt = opt ? *opt : tenzo_ext_default_options();
        o.compute = compute;
        handle = new tenzo_engine_opaque{tz::open_model(o)};
        return TENZO_SUCCESS;
    });
    return handle;
}

const char* tenzo_ext_architecture(int index) {
    const auto& f = tz::model_families();
    return index >= 0 && index < (int)f.size() ? f[index].architecture : nullptr;
}

tenzo_status_t tenzo_ext_get_config(tenzo_engine_t engine, tenzo_config_t* out) {
    if (!live(engine) || !out) return TENZO_ERROR_INVALID_ARGUMENT;
    *out = engine->impl->cfg;
    return TENZO_SUCCESS;
}

tenzo_status_t tenzo_ext_forward(tenzo_engine_t engine, int seq, const int* tokens, int n, const int* want, int n_want, float* logits) {
    if (!live(engine) || !tokens || n_want < 0 || (n_want > 0 && (!want || !logits))) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        engine->impl->forward(seq, tokens, n, want, n_want, logits);
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_ext_reset_seq(tenzo_engine_t engine, int seq) {
    if (!live(engine) || seq < 0 || seq >= engine->impl->batch) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        engine->impl->reset_seq(seq);
        return TENZO_SUCCESS;
    });
}

int tenzo_ext_batch(tenzo_engine_t engine) { return live(engine) ? engine->impl->batch : 0; }

tenzo_status_t tenzo_ext_prefill_tokens(tenzo_engine_t engine, const int* tokens) {
    if (!live(engine) || !tokens) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        engine->impl->prefill(tokens);
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_ext_generate_step(tenzo_engine_t engine, const int* cur_tokens,
                                       const tenzo_sampling_params_t* params, int* out_tokens) {
    if (!live(engine) || !cur_tokens || !out_tokens) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        if (params && (params->temperature > 0.0f))
            throw std::invalid_argument("batched decode is greedy: pass temperature <= 0 (or NULL params)");
        engine->impl->generate(cur_tokens, out_tokens);
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_ext_decode_greedy(tenzo_engine_t engine, const int* first_tokens, int n_steps, int* out_tokens) {
    if (!live(engine) || !first_tokens || !out_tokens || n_steps < 0) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        tz::EngineCore& e = *engine->impl;
        for (int s = 0; s < e.batch; ++s)
            if (e.seq_len[s] + n_steps > e.cfg.max_seq_len) throw std::out_of_range("n_steps would overflow the KV cache");
        e.decode_greedy(first_tokens, n_steps, out_tokens);
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_ext_kv_fill_random(tenzo_engine_t engine, int len, uint64_t seed) {
    if (!live(engine)) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        tz::EngineCore& e = *engine->impl;
        if (len < 0 || len > e.cfg.max_seq_len) throw std::out_of_range("length outside [0, max_seq_len]");
        e.kv_fill(len, (unsigned long long)seed);
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_ext_set_seq_len(tenzo_engine_t engine, int seq, int len) {
    if (!live(engine)) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::EngineCore& e = *engine->impl;
    if (seq < 0 || seq >= e.batch || len < 0 || len > e.cfg.max_seq_len) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        e.set_seq_len(seq, len);
        return TENZO_SUCCESS;
    });
}

int tenzo_ext_get_seq_len(tenzo_engine_t engine, int seq) {
    if (!live(engine) || seq < 0 || seq >= engine->impl->batch) return 0;
    return engine->impl->seq_len[seq];
}

tenzo_status_t tenzo_ext_read_buffer(tenzo_engine_t engine, int which, int seq, float* dst, size_t count) {
    if (!live(engine) || !dst) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        tz::EngineCore& e = *engine->impl;
        if (seq < 0 || seq >= e.batch) throw std::out_of_range("sequence index out of range");
        size_t n = 0;
        const float* src = e.buffer(which, seq, &n);
        if (count > n) throw std::out_of_range("count exceeds the buffer length");
        cudaStreamSynchronize(e.stream);
        if (cudaMemcpy(dst, src, count * 4, cudaMemcpyDeviceToHost) != cudaSuccess) throw std::runtime_error("read-back failed");
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_ext_write_x(tenzo_engine_t engine, int seq, const float* x) {
    if (!live(engine) || !x) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::EngineCore& e = *engine->impl;
    if (seq < 0 || seq >= e.batch) return TENZO_ERROR_INVALID_ARGUMENT;
    cudaStreamSynchronize(e.stream);
    return cudaMemcpy(e.b_x + (size_t)seq * e.h, x, (size_t)e.h * 4, cudaMemcpyHostToDevice) == cudaSuccess
               ? TENZO_SUCCESS : TENZO_ERROR_UNSUPPORTED;
}

tenzo_status_t tenzo_ext_run_layer(tenzo_engine_t engine, int layer) {
    if (!live(engine)) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        tz::EngineCore& e = *engine->impl;
        if (layer < 0 || layer >= e.L) throw std::out_of_range("layer index outside [0, num_layers)");
        int longest = 1;
        for (int s = 0; s < e.batch; ++s) {
            if (e.seq_len[s] + 1 > e.cfg.max_seq_len) throw std::out_of_range("KV cache is full");
            longest = e.seq_len[s] + 1 > longest ? e.seq_len[s] + 1 : longest;
        }
        e.push_state(nullptr);
        e.prepare_kv(1);
        e.enqueue_layer(layer, longest);
        if (cudaStreamSynchronize(e.stream) != cudaSuccess) throw std::runtime_error("layer execution failed");
        return TENZO_SUCCESS;
    });
}

tenzo_status_t tenzo_ext_synchronize(tenzo_engine_t engine) {
    if (!live(engine)) return TENZO_ERROR_INVALID_ARGUMENT;
    return cudaStreamSynchronize(engine->impl->stream) == cudaSuccess ? TENZO_SUCCESS : TENZO_ERROR_UNSUPPORTED;
}

float tenzo_ext_last_device_ms(tenzo_engine_t engine) { return live(engine) ? engine->impl->last_ms() : -1.0f; }

unsigned long long tenzo_ext_kernel_launches(tenzo_engine_t engine) { return live(engine) ? engine->impl->launches : 0ull; }

tenzo_status_t tenzo_ext_prefill_chunk(tenzo_engine_t engine, const int* tokens, int n) {
    if (!live(engine) || !tokens || n < 0) return TENZO_ERROR_INVALID_ARGUMENT;
    return guarded([&]() -> tenzo_status_t {
        engine->impl->prefill_chunk(tokens, n);
        return TENZO_SUCCESS;
    });
}

int tenzo_ext_sample_pairs(const float* values, const int* indices, int n, const tenzo_sampling_params_t* params, float r) {
    if (!values || n <= 0) return -1;
    const tenzo_sampling_params_t p = params ? *params : tenzo_default_sampling_params();
    return tz::sample_pairs(values, indices, n, p, r);
}

const char* tenzo_ext_last_error(void) { return tz::g_last_error.c_str(); }

}  // extern "C"
