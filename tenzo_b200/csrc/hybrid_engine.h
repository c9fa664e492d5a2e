// Hybrid decoders: a list of layers, each a mixer (attention, linear recurrence, or two of them side by side) and an
// optional dense feed-forward, on the shared engine (engine_core.h). Sozopel is the design read here; its configuration
// maps onto HybridLayer entries, and everything below works on those.
//
// State of a sequence, allocated once per slot:
//   tails   fp32  inputs that the convolutions reach back to and the token shift's previous input, all layers back to back
//   states  fp32  matrix states of the recurrences, all layers back to back
//   ring    bf16/fp32 keys and values of the last `window` tokens of each attention layer
// Decode advances every slot by one row in place. A chunk (consecutive tokens of one slot) reads the tails while other
// rows of the same launch still need them, so it writes a staging copy that replaces the slot's tails at its end.
#pragma once
#include "engine_core.h"
#include "hybrid_ops.h"
#include "model_registry.h"

namespace tz {

struct DenseWeight {                       // [rows][ld_k] bf16, zero padded
    bf16* w = nullptr;
    int rows = 0, k = 0, ld_k = 0;
};

struct WindowMixer {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 1, window = 0, ring = 0;
    float scale = 1;
    int off_q = 0, off_k = 0, off_v = 0;   // columns of the fused projection
    float *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr;
    DenseWeight o;
    size_t tail = 0;                       // offset into the slot's tails
    void *ring_k = nullptr, *ring_v = nullptr;
    size_t ring_k_stride = 0, ring_v_stride = 0;
    int channels() const { return (heads + kv_heads) * dim + kv_heads * vdim; }
};

struct ScanMixer {
    int heads = 0, dim = 0, vdim = 0, decay_kind = TENZO_DECAY_CONST, rank = 0, norm_per_head = 0;
    float q_scale = 1, k_scale = 1, tau = 1;
    int off_q = 0, off_k = 0, off_v = 0, off_g = 0, off_low = 0;
    float *decay = nullptr, *bias = nullptr, *bonus = nullptr, *norm = nullptr;
    bf16* up = nullptr;
    DenseWeight o;
    size_t state = 0;                      // offset into the slot's states
};

struct HybridLayer {
    bool has_window = false, has_scan = false;
    WindowMixer win;
    ScanMixer scan;
    float norm1 = 1, norm2 = 1;
    float *canon1 = nullptr, *canon2 = nullptr;      // [taps][width]
    size_t tail1 = 0, tail2 = 0, prev = 0;           // offsets into the slot's tails
    float* mu = nullptr;                             // token-shift mixes [n_mix][width]
    int n_mix = 0;
    DenseWeight in;                                  // every projection of the mixer's input, one product
    int n_seg = 1, seg_end[8] = {0};
    float *left_out = nullptr, *right_out = nullptr; // norms of the two outputs of a side-by-side mixer
    bool has_mlp = false;
    DenseWeight up, down;
    float act_pos = 0, act_neg = 0;
};

class HybridEngine final : public EngineCore {
public:
    HybridEngine(const Json& config, const OpenOptions& o);
    ~HybridEngine() override;

    void enqueue_step(bool with_logits, bool feed_back, int max_len) override;
    void enqueue_layer(int l, int max_len) override;
    void chunk_rows(int seq, const int* tokens, int n) override;
    void rows_logits(const int* want, int n_want, float* host) override;
    const float* buffer(int which, int seq, size_t* count) override;
    void check_device_status(bool force) override;
    int step_bucket(int) const override { return 0; }          // no launch depends on the context length
    void reset_seq(int seq) override;
    void reset_kv() override;
    void set_seq_len(int seq, int len) override;

private:
    struct Rows {                            // activations of M rows; decode and chunk each have their own set
        int cap = 0;
        float* x = nullptr;                  // residual
        void *in = nullptr, *mix_a = nullptr, *mix_b = nullptr, *act = nullptr;
        float *row_inv = nullptr, *proj = nullptr, *ya = nullptr, *yb = nullptr;
        std::vector<void*> owned;
    };
    struct Pending {                         // what the next row kernel adds to the residual
        const float *y0 = nullptr, *y1 = nullptr, *w0 = nullptr, *w1 = nullptr;
    };
    struct Pass {                            // one walk through the layers
        Rows* rows;
        int M, decode, seq, pos0;
        const int *tokens, *pos;
        bool embed = true;
        Pending add;
    };

    void init(const Json& config, const OpenOptions& o);
    void load(const Json& config, const std::string& dir);
    void read_window(WindowMixer& m, const Json& mix);
    void alloc_rows(Rows& r, int cap);
    void free_rows(Rows& r);
    RowsArgs row_args(Pass& p, float gain, const float* conv, size_t tail);
    void run_rows(Pass& p, RowsArgs& a);
    void run_gemm(Pass& p, const void* a, const DenseWeight& w, void* c, int ld_c, const HybridLayer* mixes = nullptr, const HybridLayer* act = nullptr);
    void run_layer(Pass& p, int l);
    void upload_weight(DenseWeight& d, int row0, const SafeTensors& st, const std::string& name, int rows, int k);
    DenseWeight make_weight(int rows, int k);
    float* upload_floats(const std::vector<float>& v);
    float* conv_weights(const SafeTensors& st, const std::string& name, int channels, int taps);

    bool f32 = false;
    int taps = 1, n_pos = 0;
    float eps = 0, final_gain = 1;
    std::vector<HybridLayer> layers;
    bf16 *embed = nullptr, *pos_table = nullptr;
    DenseWeight head;
    size_t tail_floats = 0, state_floats = 0;          // per slot
    float *tails = nullptr, *tail_stage = nullptr, *states = nullptr;
    int max_proj = 0, max_in = 0, max_mix = 0, max_ff = 0;   // row widths over the layers
    int max_seg = 1;
    Rows dec, chunk;
    int *chunk_tokens = nullptr, *chunk_pos = nullptr;
    void *lin_q = nullptr, *lin_k = nullptr, *lin_v = nullptr;
    float *w_rows = nullptr, *o_rows = nullptr, *scan_part = nullptr;
    void *gemm_ws = nullptr, *argmax_ws = nullptr, *logit_in = nullptr;
    float* want_logits = nullptr;
    unsigned status_poll = 0;
};

}  // namespace tz
