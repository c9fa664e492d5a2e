// What every model family shares behind one engine handle: the stream and its events, token / position / logit
// buffers, per-sequence lengths, the KV block manager, one CUDA graph per decode step, the device-resident greedy loop
// and the sampler. A family (BitNet: engine.h, the hybrid decoders: hybrid_engine.h) derives from EngineCore and
// supplies its layers, its caches or recurrent states and its rows-at-a-time prefill.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include <map>
#include <stdexcept>
#include <string>
#include <vector>

#include "../../include/tenzo.h"
#include "../../include/tenzo_ext.h"

namespace tz {

extern thread_local std::string g_last_error;
void set_error(const std::string& m);

struct CudaError : std::runtime_error {
    cudaError_t code;
    CudaError(cudaError_t c, const char* what) : std::runtime_error(std::string(what) + ": " + cudaGetErrorString(c)), code(c) {}
};
#define TZ_CUDA(expr)                                            \
    do {                                                         \
        cudaError_t _e = (expr);                                 \
        if (_e != cudaSuccess) throw tz::CudaError(_e, #expr);   \
    } while (0)
#define TZ_KERNEL(expr)                                                                         \
    do {                                                                                        \
        int _r = (expr);                                                                        \
        if (_r > 0) throw tz::CudaError((cudaError_t)_r, #expr);                                \
        if (_r < 0) throw std::runtime_error(std::string(#expr) + " rejected its arguments");   \
    } while (0)

int env_flag(const char* name, int dflt);
int bucket_for(int len, int max_seq);

// Named ranges around the engine's public operations for timeline tools (the reference marks nothing; its only
// instrumentation is the wall-clock tok/s of its CLI). Off unless TENZO_NVTX=1: a range push is a call into the tools
// interface on every token.
struct NvtxRange {
    bool on;
    explicit NvtxRange(const char* name);
    ~NvtxRange();
};

class EngineCore {
public:
    EngineCore() = default;
    virtual ~EngineCore();
    EngineCore(const EngineCore&) = delete;
    EngineCore& operator=(const EngineCore&) = delete;

    // ---- what a model family supplies ----------------------------------------------------------------------------
    virtual void enqueue_step(bool with_logits, bool feed_back, int max_len) = 0;   // one token of every sequence
    virtual void enqueue_layer(int l, int max_len) = 0;                             // the same for a single layer, on b_x
    virtual void chunk_rows(int seq, const int* tokens, int n) = 0;                 // n consecutive tokens of one sequence
    virtual void rows_logits(const int* want, int n_want, float* host) = 0;         // logits of rows of the last chunk_rows
    virtual const float* buffer(int which, int seq, size_t* count) = 0;             // TENZO_BUF_* of the last step
    virtual void check_device_status(bool force) = 0;                               // throws when a kernel flagged a failure
    virtual bool direct_step(bool, bool, int, int) { return false; }                // a step that bypasses the graph path
    virtual void after_sync() {}
    virtual int step_bucket(int longest) const { return bucket_for(longest, cfg.max_seq_len); }   // part of the graph key
    virtual void invalidate_graphs();
    virtual void reset_seq(int seq);                                                // the sequence starts over
    virtual void reset_kv();                                                        // all of them do
    virtual void set_seq_len(int seq, int len);
    virtual void kv_fill(int len, unsigned long long seed);
    virtual void generate(const int* cur, int* out);                                // device argmax

    // ---- sequencing ------------------------------------------------------------------------------------------------
    void init_core(int batch, int use_graph, int use_pdl);
    void init_core_buffers();                              // token, position and logit buffers, once h and V are known
    void* dalloc(size_t bytes);                            // zeroed, owned by the engine
    void* upload(const void* host, size_t bytes);
    void prefill(const int* tokens);                       // one token per sequence, no logits
    void prefill_chunk(const int* tokens, int n);          // n consecutive tokens of the one sequence, together
    void forward(int seq, const int* tokens, int n, const int* want, int n_want, float* logits);
    void decode_greedy(const int* first, int n_steps, int* out);
    int sample(const tenzo_sampling_params_t& p, const int* past, int n_past);   // on the logits of the last step
    void push_state(const int* tokens);
    void run_step(bool with_logits, bool feed_back);
    void enqueue_advance(bool feed_back);
    float last_ms();
    void release_core();
    void check_tokens(const int* tokens, int n) const;

    // kv_mode "paged_int8" (PagedKVCache + PagedBlockManager of the reference, TenzoEngine.h:117-193): the caches are pools
    // of 16-token blocks [block][layer][kv_head][16][128]; every sequence has a row of the block table. Blocks are taken
    // from the free list on the host before the step that first writes into them (the reference does it inside layer 0,
    // TenzoEngine.cpp:294-300) and the table row is copied to the device ahead of the launch.
    static constexpr int kBlock = 16;
    bool paged = false;
    int total_blocks = 0, table_stride = 0;
    int *d_table = nullptr, *h_table = nullptr;          // [batch][table_stride]; h_table is the pinned master copy
    std::vector<int> free_blocks, n_blocks;              // free list (taken from the back: 0, 1, 2, ... as the reference's)
    bool table_dirty = false;
    void reserve_blocks(int seq, int len);               // the table of `seq` covers tokens [0, len)
    void release_blocks(int seq, int len);               // blocks past token len go back to the free list
    void prepare_kv(int extra);                          // before a step that appends `extra` tokens to every sequence

    tenzo_config_t cfg = {};
    int batch = 1, device = 0, use_graph = 1, use_pdl = 1;
    int h = 0, L = 0, V = 0;
    cudaStream_t stream = nullptr;
    cudaEvent_t ev0 = nullptr, ev1 = nullptr;
    int *d_tokens = nullptr, *d_pos = nullptr, *d_next = nullptr, *d_history = nullptr;
    size_t history_cap = 0;
    float *b_x = nullptr, *b_logits = nullptr;
    void *d_cand = nullptr, *h_cand = nullptr;           // sampler: candidate count + (value, index) pairs
    int* d_sample_past = nullptr;
    size_t sample_past_cap = 0;
    int *h_pin = nullptr, *h_tokens = nullptr, *h_pos = nullptr, *h_next = nullptr;
    std::vector<int> seq_len;
    std::vector<void*> owned;
    std::map<int, cudaGraphExec_t> graphs;
    std::map<int, unsigned long long> graph_kernels;
    unsigned long long launches = 0;
};

}  // namespace tz

struct tenzo_engine_opaque {
    tz::EngineCore* impl;
};
