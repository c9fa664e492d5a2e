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

int launch_rows(const RowsArgs& a, cudaStream_t st, unsigned long long* n_kernels);                       // rows.cu
int launch_gemm(const GemmArgs& a, cudaStream_t st);                                                      // gemm.cu
int launch_gemm_umma(const GemmArgs& a, cudaStream_t st);                                                 // gemm_umma.cu
bool gemm_umma_applicable(const GemmArgs& a);
constexpr int kGemmUmmaMinRows = 16;
int launch_window_attention(const WindowAttnArgs& a, cudaStream_t st, unsigned long long* n_kernels);     // window_attention.cu
int launch_scan(const ScanArgs& a, cudaStream_t st, unsigned long long* n_kernels);                       // linear_scan.cu

// Row-wise argmax of fp32 logits, first maximum wins (gemm.cu).
int launch_argmax(const float* logits, int vocab, int rows, int* out, void* scratch, cudaStream_t st);
size_t argmax_scratch_bytes(int rows);

}  // namespace tz
