// Hybrid decoders: a list of layers, each a mixer (attention, linear recurrence, or two of them side by side) and an
// optional feed-forward (dense or a mixture of experts), on the shared engine (engine_core.h). A design (Sozopel:
// hybrid_sozopel.cu, Tigitar: hybrid_tigitar.cu) maps its configuration and weights onto HybridLayer entries, and
// everything below works on those.
//
// State of a sequence, allocated once per slot:
//   tails   fp32  inputs that the convolutions reach back to and the token shift's previous input, all layers back to back
//   states  fp32  matrix states of the recurrences and the delta rule's convolution inputs, all layers back to back
//   rings   bf16/fp32 keys and values, or latents, of the last `window` tokens of each attention layer; a latent layer may
//           read another one's ring, which then reaches as far back as the widest window among its readers
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

struct DeltaMixer {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 1;
    int off_q = 0, off_k = 0, off_v = 0, off_g = 0, off_a = 0, off_b = 0;
    float *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr, *a_log = nullptr, *dt_bias = nullptr, *norm = nullptr;
    DenseWeight o;
    size_t state = 0, tail = 0;            // offsets into the slot's states
    int channels() const { return 2 * kv_heads * dim + heads * vdim; }
};

struct LatentCache {                       // of a layer that makes its own latents
    int rank = 0, rot = 0, ring = 0, lin = 0;      // lin: which pair of chunk buffers
    bool borrowed = false;
    double* freq = nullptr;
    void *ring_c = nullptr, *ring_r = nullptr;
    size_t ring_c_stride = 0, ring_r_stride = 0;
    int ld_c() const { return round_up(rank, 64); }
    int rot8() const { return round_up(rot, 8); }
};

struct LatentMixer {
    int heads = 0, dim = 0, vdim = 0, window = 0, cache = 0;
    bool owner = false;
    float scale = 1;
    int off_q = 0, off_dkv = 0;
    float* norm = nullptr;
    bf16* kv = nullptr;                    // key rows of all heads, then value rows, padded as tenzo_latent_attention_args has them
    DenseWeight o;                         // columns of a head padded to vdim8
    int dim8() const { return round_up(dim, 8); }
    int vdim8() const { return round_up(vdim, 8); }
};

struct ExpertMlp {
    int experts = 0, top = 0, ff = 0;
    DenseWeight router, up, down;          // up: gate and up rows of all experts interleaved, expert after expert; down likewise
    float* correction = nullptr;
};

struct HybridLayer {
    bool has_window = false, has_scan = false, has_delta = false, has_latent = false;
    WindowMixer win;
    ScanMixer scan;
    DeltaMixer delta;
    LatentMixer lat;
    float norm1 = 1, norm2 = 1;                      // gains of the norms in front of the two sublayers,
    float *norm1_w = nullptr, *norm2_w = nullptr;    // per channel when the design has them so,
    float *post1_w = nullptr, *post2_w = nullptr;    // and of the norms behind them, when it has any
    float *canon1 = nullptr, *canon2 = nullptr;      // [taps][width]
    size_t tail1 = 0, tail2 = 0, prev = 0;           // offsets into the slot's tails
    float* mu = nullptr;                             // token-shift mixes [n_mix][width]
    int n_mix = 0;
    DenseWeight in;                                  // every projection of the mixer's input, one product
    int n_seg = 1, seg_end[8] = {0};
    float *left_out = nullptr, *right_out = nullptr; // norms of the two outputs of a side-by-side mixer
    bool has_mlp = false;
    DenseWeight up, down;
    int up_epilogue = TENZO_GEMM_XIELU;              // GLU: `up` holds gate and up rows interleaved
    float act_pos = 0, act_neg = 0;
    ExpertMlp moe;                                   // instead of up and down, when it has experts
};

class HybridEngine final : public EngineCore {
public:
    using Loader = void (HybridEngine::*)(const Json& config, const SafeTensors& st);
    HybridEngine(const Json& config, const OpenOptions& o, Loader load);
    ~HybridEngine() override;
    // A loader fills the sizes (h, V, n_pos, L, eps, ...), the layers and the weights, and reserves the slots' state.
    void load_sozopel(const Json& config, const SafeTensors& st);      // hybrid_sozopel.cu
    void load_tigitar(const Json& config, const SafeTensors& st);      // hybrid_tigitar.cu

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
        float* q_abs = nullptr;              // latent attention, decode
        void* lat = nullptr;
        int *chosen = nullptr, *slot = nullptr, *row_of = nullptr, *group_off = nullptr;      // experts: routing,
        float *weight = nullptr, *ye = nullptr;                                               // outputs of all pairs,
        void *gathered = nullptr, *act_e = nullptr;                                           // their inputs and activations
        std::vector<void*> owned;
    };
    struct Pending {                         // what the next row kernel adds to the residual
        const float *y0 = nullptr, *y1 = nullptr, *w0 = nullptr, *w1 = nullptr;
        const int* slot = nullptr;
        const float* weight = nullptr;
        int n_y = 0;
    };
    struct Piece {                           // of a fused projection: tensor, rows, where its first column goes
        std::string name;
        int rows;
        int* off;
    };
    struct Pass {                            // one walk through the layers
        Rows* rows;
        int M, decode, seq, pos0;
        const int *tokens, *pos;
        bool embed = true;
        Pending add;
    };

    void init(const Json& config, const OpenOptions& o, Loader load);
    void start_layers(int n);                          // sizes are known: the layer list and what depends on the width
    size_t take_tail(size_t floats);                   // 16-byte pieces of the slot's tails / states
    size_t take_state(size_t floats);
    void fuse_inputs(HybridLayer& y, const std::vector<Piece>& pieces, int align, const SafeTensors& st);
    void read_window(WindowMixer& m, const Json& mix);
    void read_delta(HybridLayer& y, const Json& mix, const SafeTensors& st, const std::string& pre);
    void read_latent(int l, const Json& config, const SafeTensors& st, const std::string& pre, std::vector<int>& cache_of);
    void read_glu(DenseWeight& up, DenseWeight& down, int index, int ff, const SafeTensors& st, const std::string& pre);
    void alloc_rows(Rows& r, int cap);
    void free_rows(Rows& r);
    RowsArgs row_args(Pass& p, float gain, const float* gain_w, const float* conv, size_t tail);
    void run_rows(Pass& p, RowsArgs& a);
    GemmArgs gemm_args(Pass& p, const void* a, const DenseWeight& w, void* c, int ld_c);
    void run_gemm(const GemmArgs& g);
    void run_head(Pass& p, const void* rows, float* logits);
    void run_window(Pass& p, HybridLayer& y);
    void run_scan(Pass& p, HybridLayer& y);
    void run_delta(Pass& p, HybridLayer& y);
    void run_latent(Pass& p, HybridLayer& y);
    void run_experts(Pass& p, HybridLayer& y);
    void run_layer(Pass& p, int l);
    void run_final(Pass& p);
    void grow_chunk(int rows);
    void upload_weight(DenseWeight& d, int row0, const SafeTensors& st, const std::string& name, int rows, int k);
    DenseWeight make_weight(int rows, int k);
    float* upload_floats(const std::vector<float>& v);
    float* conv_weights(const SafeTensors& st, const std::string& name, int channels, int taps);

    bool f32 = false;
    int taps = 1, n_pos = 0;
    float eps = 0, final_gain = 1, logit_cap = 0;      // logit_cap 0: none
    float* final_gain_w = nullptr;
    std::vector<HybridLayer> layers;
    std::vector<LatentCache> caches;
    bf16 *embed = nullptr, *pos_table = nullptr;
    DenseWeight head;
    size_t tail_floats = 0, state_floats = 0;          // per slot
    float *tails = nullptr, *tail_stage = nullptr, *states = nullptr;
    int max_proj = 0, max_in = 0, max_mix = 0, max_ff = 0;   // row widths over the layers
    int max_seg = 1;
    int max_top = 0, max_experts = 0, max_expert_ff = 0;     // 0: no mixture of experts
    size_t max_lat = 0;                                      // heads * ld_c over the latent layers
    Rows dec, chunk;
    int *chunk_tokens = nullptr, *chunk_pos = nullptr;
    void *lin_q = nullptr, *lin_k = nullptr, *lin_v = nullptr;
    float *w_rows = nullptr, *o_rows = nullptr, *scan_part = nullptr, *delta_work = nullptr;
    std::vector<void*> lin_c, lin_r;                         // latent rows of a chunk, a pair per cache that is borrowed and one for the others
    void* lat_kv = nullptr;
    void *gemm_ws = nullptr, *argmax_ws = nullptr, *logit_in = nullptr;
    float* want_logits = nullptr;
    unsigned status_poll = 0;
};

}  // namespace tz
