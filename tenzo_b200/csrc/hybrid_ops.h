// Building blocks of decoders that mix attention with recurrent layers: row kernels (embedding, residual sums, RMS norm,
// causal convolution over time), bf16-weight matrix products, sliding-window attention and linear recurrences. The
// argument structs are those of the flat C calls (include/tenzo_kernels.h); every constant is a field, so another design
// of this kind composes the same pieces. Launchers return 0, a cudaError_t or a negative code (TZ_KERNEL).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../../include/tenzo_kernels.h"

namespace tz {

using bf16 = __nv_bfloat16;
constexpr int kMaxTaps = 16;
constexpr int kMaxHeadDim = 256;
constexpr int kMaxLatentRank = 1024;

static inline int round_up(int v, int m) { return (v + m - 1) / m * m; }

// The C structs with neutral defaults.
struct RowsArgs : tenzo_rows_args {
    RowsArgs() : tenzo_rows_args{} { gain = 1; taps = 1; }
};
struct GemmArgs : tenzo_gemm_args {
    GemmArgs() : tenzo_gemm_args{} { n_seg = 1; }
};
struct WindowAttnArgs : tenzo_window_attention_args {
    WindowAttnArgs() : tenzo_window_attention_args{} { taps = 1; scale = 1; slope_base = 8; sink = 1; }
};
struct ScanArgs : tenzo_scan_args {
    ScanArgs() : tenzo_scan_args{} { q_scale = k_scale = tau = 1; }
};

struct DeltaArgs : tenzo_delta_args {
    DeltaArgs() : tenzo_delta_args{} { taps = 1; q_scale = 1; unit_eps = 1e-6f; }
};
struct LatentAttnArgs : tenzo_latent_attention_args {
    LatentAttnArgs() : tenzo_latent_attention_args{} { scale = 1; }
};
struct RouteArgs : tenzo_route_args {
    RouteArgs() : tenzo_route_args{} {}
};

// Attention of M rows of one sequence over linear keys and values in the storage type: row hist + t belongs to query t, rows
// before hist are older tokens. A key is d1 elements of its head's row followed by d2 elements that all heads share.
struct LinearAttn {
    const void* q = nullptr;                             // [M][heads][d1 + d2]
    const void *k = nullptr, *k2 = nullptr, *v = nullptr;
    size_t k_row = 0, k_head = 0, k2_row = 0, v_row = 0, v_head = 0;      // elements between rows / heads, multiples of 8
    int d1 = 0, d2 = 0, dv = 0, vdim = 0;                // d1, d2, dv multiples of 8, padding zero; vdim columns are stored
    int heads = 1, group = 1, M = 0, hist = 0, window = 1;     // group: query heads per key head
    float scale = 1, slope_base = 0, sink = 0;           // as in tenzo_window_attention_args
    void* out = nullptr;                                 // storage type, head h of row t at t * ld_out + h * out_head
    int ld_out = 0, out_head = 0, f32 = 0;
};

int launch_rows(const RowsArgs& a, cudaStream_t st, unsigned long long* n_kernels);                       // rows.cu
int launch_gemm(const GemmArgs& a, cudaStream_t st, unsigned long long* n_kernels);                       // gemm.cu
int launch_gemm_umma(const GemmArgs& a, cudaStream_t st);                                                 // gemm_umma.cu
bool gemm_umma_applicable(const GemmArgs& a);
constexpr int kGemmUmmaMinRows = 16;
int launch_window_attention(const WindowAttnArgs& a, cudaStream_t st, unsigned long long* n_kernels);     // window_attention.cu
int launch_linear_attention(const LinearAttn& a, cudaStream_t st);                                        // linear_attention.cu
int launch_scan(const ScanArgs& a, cudaStream_t st, unsigned long long* n_kernels);                       // linear_scan.cu
int launch_scan_gate(const ScanArgs& a, cudaStream_t st, unsigned long long* n_kernels);                  // its last step: M, heads, vdim, o_rows, norm, g, ld, eps, out
int launch_delta(const DeltaArgs& a, cudaStream_t st, unsigned long long* n_kernels);                     // delta_rule.cu
int launch_latent_attention(const LatentAttnArgs& a, cudaStream_t st, unsigned long long* n_kernels);     // latent_attention.cu
int launch_route(const RouteArgs& a, cudaStream_t st, unsigned long long* n_kernels);                     // route.cu

// Row-wise argmax of fp32 logits, first maximum wins (gemm.cu).
int launch_argmax(const float* logits, int vocab, int rows, int* out, void* scratch, cudaStream_t st);
size_t argmax_scratch_bytes(int rows);

}  // namespace tz
