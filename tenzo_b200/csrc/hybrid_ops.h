// Building blocks of decoders that mix attention with recurrent layers: row kernels (embedding, residual sums, RMS norm,
// causal convolution over time), bf16-weight matrix products, sliding-window attention and linear recurrences. Every
// constant is a field of the argument structs, so another design of this kind composes the same pieces.
//
// Two storage types: activations that enter a matrix product and cached keys/values are bf16 (`f32` = 0) or fp32
// (`f32` = 1); weights of matrix products are bf16 in both. Everything else (residual, norms, scores, states, decays)
// is fp32 always, and the fp32 path uses plain FMA arithmetic, no reduced-precision matrix mode.
//
// Rows: a "decode" launch has one row per sequence (row b belongs to sequence b and its per-sequence state at
// b * seq_stride); a "chunk" launch has M consecutive tokens of one sequence, whose carried state is read from *_in and
// written to *_out (a staging area: other rows of the launch may still read *_in).
//
// Launchers return 0 or a cudaError_t / negative code (TZ_KERNEL).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace tz {

using bf16 = __nv_bfloat16;
constexpr int kMaxTaps = 16;
constexpr int kMaxHeadDim = 256;

static inline int round_up(int v, int m) { return (v + m - 1) / m * m; }

// ---- rows.cu -----------------------------------------------------------------------------------------------------
// x = source; h = x / rms(x) * gain; y = h + conv(h); out = y (or the token-shift mixes of y), padded rows of ld_out.
struct RowsArgs {
    // source: tokens != null -> embed[token] + pos_table[pos]; else x_in, plus y0 (one addend) or, with y1,
    // 0.5 * (y0 / rms(y0) * w0 + y1 / rms(y1) * w1)
    const int *tokens = nullptr, *pos = nullptr;
    const bf16 *embed = nullptr, *pos_table = nullptr;
    int vocab = 0, n_pos = 0;
    const float *x_in = nullptr, *y0 = nullptr, *y1 = nullptr, *w0 = nullptr, *w1 = nullptr;
    int ld_y = 0;
    float* x_out = nullptr;                // [M][width], not x_in
    int width = 0, M = 0;
    float eps = 0, gain = 1;
    const float* conv_w = nullptr;         // [taps][width] or null
    int taps = 1;
    const float* tail_in = nullptr;        // [taps-1][width] per sequence: the last inputs of the convolution, oldest first
    float* tail_out = nullptr;
    const float* mu = nullptr;             // [n_mix][width]: out s = y + (y_prev - y) * mu_s
    int n_mix = 0;
    const float* prev_in = nullptr;        // [width] per sequence: y of the token before
    float* prev_out = nullptr;
    size_t seq_stride = 0;                 // floats between the states of two sequences
    int decode = 0;
    void* out = nullptr;                   // [max(n_mix,1)][M][ld_out]
    int ld_out = 0;
    int f32 = 0, use_pdl = 0;
};
int launch_rows(const RowsArgs& a, cudaStream_t st);

// ---- gemm.cu / gemm_umma.cu ------------------------------------------------------------------------------------------
// C[m][n] = sum_k A_seg[m][k] W[n][k]; W bf16 [n_rows][ld_k] with ld_k a multiple of 64, zero padded; A rows of ld_k.
// Rows of W in segment s (seg_end[s-1] <= n < seg_end[s]) multiply the A matrix at a + s * a_seg_stride elements.
enum { GEMM_STORE = 0, GEMM_XIELU = 1 };
struct GemmArgs {
    const void* a = nullptr;
    const bf16* w = nullptr;
    int M = 0, N = 0, ld_k = 0;
    int n_seg = 1, seg_end[8] = {0};
    size_t a_seg_stride = 0;
    int epilogue = GEMM_STORE;
    float act_pos = 0, act_neg = 0;        // xIELU: z > 0: pos z^2 + z/2, else neg (exp(z) - 1 - z) + z/2
    void* c = nullptr;                     // GEMM_STORE: float [M][ld_c]; GEMM_XIELU: activation type [M][ld_c]
    int ld_c = 0;
    int f32 = 0, use_pdl = 0;
    void* workspace = nullptr;             // split-K partial tiles (zeroed once at allocation)
    size_t workspace_bytes = 0;
};
int launch_gemm(const GemmArgs& a, cudaStream_t st);
int launch_gemm_umma(const GemmArgs& a, cudaStream_t st);       // bf16, M >= 16
bool gemm_umma_applicable(const GemmArgs& a);
constexpr int kGemmUmmaMinRows = 16;
size_t gemm_workspace_bytes();
int gemm_umma_take_timeouts();

// Row-wise argmax of fp32 logits, first maximum wins.
int launch_argmax(const float* logits, int vocab, int rows, int* out, void* scratch, cudaStream_t st);
size_t argmax_scratch_bytes(int rows);

// ---- window_attention.cu -----------------------------------------------------------------------------------------------
// Causal sliding-window attention over grouped heads after a short causal convolution on q, k, v channels, linear distance
// bias; the softmax denominator carries the extra constant `sink`. The last `window`
// keys and values of a sequence live in a ring: slot = position % ring.
struct WindowAttnArgs {
    const float* q = nullptr;              // projections of the M rows (row stride ld), before the convolution
    const float* k = nullptr;
    const float* v = nullptr;
    int ld = 0;
    const float *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr;    // [taps][channels]
    int taps = 1;
    const float* tail_in = nullptr;        // [taps-1][q|k|v channels] per sequence
    float* tail_out = nullptr;
    size_t tail_seq_stride = 0;
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 1, slope_base = 8;       // slope_h = 2^(-slope_base (h+1) / heads)
    float sink = 1;                        // 0: an ordinary softmax
    int window = 0, ring = 0;              // ring >= min(window, longest sequence)
    void *ring_k = nullptr, *ring_v = nullptr;   // [kv_heads][ring][ld_dim / ld_vdim] per sequence, ld = round_up(.., 8)
    size_t ring_k_stride = 0, ring_v_stride = 0; // elements between two sequences
    const int* pos = nullptr;              // decode: position of every row
    int pos0 = 0;                          // chunk: position of the first row
    int M = 0, decode = 0;
    void* out = nullptr;                   // [M][ld_out] activation type, head after head
    int ld_out = 0;
    // chunk scratch: convolved queries [M][heads][ld_dim], and keys / values [kv_heads][history + M][ld]
    void *lin_q = nullptr, *lin_k = nullptr, *lin_v = nullptr;
    int f32 = 0, use_pdl = 0;
};
int launch_window_attention(const WindowAttnArgs& a, cudaStream_t st, unsigned long long* n_kernels);

// ---- linear_scan.cu --------------------------------------------------------------------------------------------------------
// S_t = diag(w_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t, or (bonus u) o_t = (S_{t-1} + diag(u) k_t v_t^T)^T q_t; then per head
// o / rms(o) * norm * silu(g).
enum { DECAY_CONST = 0, DECAY_SIGMOID_ROOT = 1, DECAY_EXP_EXP = 2 };
struct ScanArgs {
    const float *q = nullptr, *k = nullptr, *v = nullptr, *g = nullptr;     // row stride ld
    int ld = 0;
    float q_scale = 1, k_scale = 1;
    int heads = 0, dim = 0, vdim = 0;
    int decay_kind = DECAY_CONST;
    const float* decay = nullptr;          // DECAY_CONST: [heads]
    // low-rank gate: z = up . f(low) + bias; SIGMOID_ROOT: f = identity, w = sigmoid(z)^(1/tau); EXP_EXP: f = tanh, w = exp(-exp(z))
    const float* low = nullptr;            // [M] rows (stride ld) of `rank` values
    const bf16* up = nullptr;              // [heads*dim][rank]
    const float* bias = nullptr;           // [heads*dim]
    int rank = 0;
    float tau = 1;
    const float* bonus = nullptr;          // [heads*dim] or null
    const float* norm = nullptr;           // [vdim] shared or [heads*vdim], or null
    int norm_per_head = 0;
    float eps = 0;
    float* state = nullptr;                // [heads][dim][ld_v] per sequence, ld_v = round_up(vdim, 4)
    size_t state_seq_stride = 0;
    int M = 0, decode = 0;
    void* out = nullptr;                   // [M][ld_out] activation type
    int ld_out = 0;
    // chunk scratch
    float* w_rows = nullptr;               // [M][heads*dim] decays
    float* o_rows = nullptr;               // [M][heads*vdim]
    float* part = nullptr;                 // scan_part_floats()
    int f32 = 0, use_pdl = 0;
};
int launch_scan(const ScanArgs& a, cudaStream_t st, unsigned long long* n_kernels);
size_t scan_part_floats(int M, int heads, int dim, int vdim);

}  // namespace tz
