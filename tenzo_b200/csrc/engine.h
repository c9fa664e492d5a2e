// The BitNet engine: state shared between engine.cu (behaviour) and capi_bitnet.cu (its part of the extern "C" boundary).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include <map>
#include <string>
#include <vector>

#include "../../include/tenzo.h"
#include "../../include/tenzo_ext.h"
#include "decode_persistent.h"
#include "engine_core.h"

namespace tz {

void rope_tables_host(int max_seq, int head_dim, float theta, float* cs, float* sn);


struct LayerDev {
    uint8_t* qkv = nullptr;      // q|k|v row blocks back to back, TL1 layout
    uint8_t* o = nullptr;
    uint8_t* gateup = nullptr;   // gate|up
    uint8_t* down = nullptr;
    float s_q = 1, s_k = 1, s_v = 1, s_o = 1, s_gate = 1, s_up = 1, s_down = 1;
    float *in_norm = nullptr, *attn_sub_norm = nullptr, *post_norm = nullptr, *ffn_sub_norm = nullptr;
    bool has_mlp = false, set = false;
};

class Engine final : public EngineCore {
public:
    Engine(const tenzo_config_t& cfg, const tenzo_ext_options_t& opt);
    ~Engine() override;
    void init(const tenzo_config_t& cfg, const tenzo_ext_options_t& opt);

    void set_layer(int l, const tenzo_layer_weights_t& w);
    void set_final_norm(const float* w);
    void set_lm_head(const int8_t* w, const float* scales);

    void enqueue_step(bool with_logits, bool feed_back, int max_len) override;
    void enqueue_layer(int l, int max_len) override;
    void chunk_rows(int seq, const int* tokens, int n) override;
    void rows_logits(const int* want, int n_want, float* host) override;
    const float* buffer(int which, int seq, size_t* count) override;
    void check_device_status(bool force) override;
    bool direct_step(bool with_logits, bool feed_back, int max_len, int longest) override;
    void after_sync() override { pc_check(); }
    void invalidate_graphs() override;
    void kv_fill(int len, unsigned long long seed) override;
    void generate(const int* cur, int* out) override;      // device argmax

    void enqueue_layer(int l, int max_len, bool gemv_only);
    float bench_gemv_stack(int iters, unsigned long long* n_launches);
    void free_prefill_rows();
    void release_all();
    unsigned status_poll = 0;
    size_t kv_row(int seq, int layer, int kvh, int t) const;   // row of a cached token in cache_k/v (x128) and scale_k/v

    float rope_theta = 10000.0f;
    int qd = 0, kvd = 0, ffn = 0;
    std::vector<LayerDev> layers;
    float* final_norm = nullptr;
    int8_t* lm_w = nullptr;
    float* lm_scales = nullptr;

    float *b_qkv = nullptr, *b_attn = nullptr, *b_h1 = nullptr, *b_act = nullptr;
    int8_t *cache_k = nullptr, *cache_v = nullptr;
    float *scale_k = nullptr, *scale_v = nullptr;
    size_t kv_rows_per_seq = 0;
    float *rope_cos = nullptr, *rope_sin = nullptr;
    void *lm_scratch = nullptr, *gemv_ws = nullptr;
    int attention_mode = 0;              // 1: tolerance-mode attention (attention_fast.cu) in the kernel chain
    void* attn_ws = nullptr;
    size_t attn_ws_bytes = 0;
    float *pf_x = nullptr, *pf_qkv = nullptr, *pf_attn = nullptr, *pf_h1 = nullptr, *pf_act = nullptr;   // chunked prefill rows
    int *pf_tokens = nullptr, *pf_pos = nullptr, pf_cap = 0;
    void* pf_ws = nullptr;

    // Single-sequence engines: the whole token as one persistent cooperative kernel (decode_persistent.cu) instead of the
    // kernel chain, whenever the shapes fit it (pc_usable). Its scratch is owned here: zeroed accumulators, the barrier
    // word (only ever grows; pc_bar_base tracks it), status and result words the host can read without a copy.
    int persistent = 0;                  // option / TENZO_PERSISTENT (off unless asked for: measured slower than the kernel chain)
    bool pc_built = false, pc_ok = false;
    int pc_grid = 0;
    PcLayer* pc_layers = nullptr;
    int32_t* pc_acc = nullptr;
    unsigned* pc_bar = nullptr;
    unsigned pc_bar_base = 0;
    int* pc_status = nullptr;
    int* pc_host = nullptr;              // mapped pinned: [0] status mirror, [1] next token
    int* pc_host_dev = nullptr;          // the device's view of it
    LmBest* pc_best = nullptr;
    unsigned long long* pc_phase_ns = nullptr;
    int pc_token_arg = -1, pc_pos_arg = -1;
    int pc_score_cap(int max_len);
    bool pc_usable();                    // builds the layer table on first use; false = use the kernel chain
    void pc_step(bool with_logits, bool feed_back, int max_len);
    void pc_check();                     // after a synchronisation: throws (and re-arms the scratch) if a launch gave up
    void pc_reset_scratch();
};

}  // namespace tz
