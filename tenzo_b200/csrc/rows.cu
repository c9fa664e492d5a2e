// Row kernels of the hybrid decoders: residual update, RMS norm with one gain or a gain per channel, causal convolution over
// time on every channel, and the token-shift mixes of a time-mixing layer (tenzo_rows_args).
//
// Decode, and rows that carry nothing from one to the next: one CTA per row does all of it; a thread keeps its columns in
// registers, with the convolution's weights and the carried inputs fetched before the kernel waits for its producer (the
// launch that wrote them lies a whole step back).
// Rows without convolution and mixes (designs that have none) take a kernel of 256 threads and 16-byte pieces instead.
// Chunk (and decode of rows wider than that): one kernel updates the residual and leaves each row's inverse RMS, a second
// one walks tiles of rows per channel with the convolution's inputs in registers.
#include "hybrid_common.cuh"

namespace tz {

constexpr int kStepThreads = 1024, kStepTaps = 4, kStepMaxCols = 4;
constexpr int kNormThreads = 256, kConvThreads = 128, kConvRows = 16;

// Sums of two values over the block, the same bits in every thread. scratch: 2 * 32 floats, not reused by the next call.
__device__ __forceinline__ float2 block_sum2(float2 v, float2* scratch) {
    const int lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    v.x = warp_sum(v.x);
    v.y = warp_sum(v.y);
    if (lane == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    const float2 p = lane < nw ? scratch[lane] : make_float2(0.0f, 0.0f);
    return make_float2(warp_sum(p.x), warp_sum(p.y));
}

struct RowSource {                              // where a row's residual comes from
    const RowsArgs& a;
    const bf16 *e = nullptr, *p = nullptr;
    const float *x = nullptr, *y0 = nullptr, *y1 = nullptr, *yw = nullptr;
    const int* ys = nullptr;
    bool normed = false;                        // the addends are normed
    __device__ __forceinline__ RowSource(const RowsArgs& args, int t) : a(args) {
        if (a.tokens) {
            const int tok = min(max(a.tokens[t], 0), a.vocab - 1);
            e = static_cast<const bf16*>(a.embed) + (size_t)tok * a.width;
            if (a.pos_table) p = static_cast<const bf16*>(a.pos_table) + (size_t)min(max(a.pos[t], 0), a.n_pos - 1) * a.width;
        } else {
            x = a.x_in + (size_t)t * a.width;
            y1 = a.y1 ? a.y1 + (size_t)t * a.ld_y : nullptr;
            normed = a.w0 != nullptr;
            if (a.y_slot) {
                ys = a.y_slot + (size_t)t * a.n_y;
                yw = a.y_weight + (size_t)t * a.n_y;
                y0 = a.y0;
            } else if (a.y0) {
                y0 = a.y0 + (size_t)t * a.ld_y;
            }
        }
    }
    __device__ __forceinline__ float first(int c) const {
        if (!ys) return y0[c];
        float v = 0.0f;
        for (int j = 0; j < a.n_y; ++j) v = fmaf(yw[j], y0[(size_t)ys[j] * a.ld_y + c], v);
        return v;
    }
    // without normed addends
    __device__ __forceinline__ float plain(int c) const {
        if (e) return p ? to_f(e[c]) + to_f(p[c]) : to_f(e[c]);
        return y0 && !normed ? x[c] + first(c) : x[c];
    }
};

// CPT columns per thread: c = threadIdx.x + i * kStepThreads.
template <typename T, int CPT>
__global__ void __launch_bounds__(kStepThreads) rows_step_kernel(const RowsArgs a) {
    __shared__ float2 s_red[2][32];
    const int row = blockIdx.x, width = a.width, taps = a.conv_w ? a.taps : 1, nt = taps - 1;
    const size_t off = (size_t)row * a.seq_stride;
    // w[3] belongs to the current input, u[0..2] are the three before it; both are zero beyond the convolution's reach
    float w[CPT][kStepTaps], u[CPT][kStepTaps - 1], prev[CPT];
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
        const int c = threadIdx.x + i * kStepThreads;
        const bool in = c < width;
#pragma unroll
        for (int j = 0; j < kStepTaps; ++j) w[i][j] = in && a.conv_w && j >= kStepTaps - taps ? a.conv_w[(size_t)(j - kStepTaps + taps) * width + c] : 0.0f;
#pragma unroll
        for (int j = 0; j < kStepTaps - 1; ++j)
            u[i][j] = in && j >= kStepTaps - 1 - nt ? a.tail_in[off + (size_t)(j - (kStepTaps - 1 - nt)) * width + c] : 0.0f;
        prev[i] = in && a.mu ? a.prev_in[off + c] : 0.0f;
    }
    pdl_wait();
    pdl_launch_dependents();
    const RowSource src(a, row);
    float x[CPT], l[CPT], r[CPT];
    float2 q = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
        const int c = threadIdx.x + i * kStepThreads;
        x[i] = l[i] = r[i] = 0.0f;
        if (c >= width) continue;
        x[i] = src.plain(c);
        if (src.normed) {
            l[i] = src.first(c);
            q.x = fmaf(l[i], l[i], q.x);
            if (src.y1) {
                r[i] = src.y1[c];
                q.y = fmaf(r[i], r[i], q.y);
            }
        }
    }
    if (src.normed) {
        q = block_sum2(q, s_red[0]);
        const float i0 = 1.0f / sqrtf(q.x / (float)width + a.eps), i1 = 1.0f / sqrtf(q.y / (float)width + a.eps);
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
            const int c = threadIdx.x + i * kStepThreads;
            if (c >= width) continue;
            const float v = l[i] * i0 * a.w0[c];
            x[i] += src.y1 ? 0.5f * (v + r[i] * i1 * a.w1[c]) : v;
        }
    }
    q = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
        const int c = threadIdx.x + i * kStepThreads;
        if (c < width) a.x_out[(size_t)row * width + c] = x[i];
        q.x = fmaf(x[i], x[i], q.x);
    }
    q = block_sum2(q, s_red[1]);
    const float inv = 1.0f / sqrtf(q.x / (float)width + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + (size_t)row * a.ld_out;
    const size_t mix_stride = (size_t)a.M * a.ld_out;
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
        const int c = threadIdx.x + i * kStepThreads;
        if (c >= width) continue;
        const float h = x[i] * inv * (a.gain_w ? a.gain * a.gain_w[c] : a.gain);
        float z = 0.0f;
#pragma unroll
        for (int j = 0; j < kStepTaps - 1; ++j) z = fmaf(w[i][j], u[i][j], z);
        const float y = h + fmaf(w[i][kStepTaps - 1], h, z);
        if (a.mu) {
            for (int s = 0; s < a.n_mix; ++s) out[s * mix_stride + c] = from_f<T>(fmaf(prev[i] - y, a.mu[(size_t)s * width + c], y));
            a.prev_out[off + c] = y;
        } else {
            out[c] = from_f<T>(y);
        }
#pragma unroll
        for (int j = 0; j < kStepTaps - 1; ++j) {                // the tail moves up by one
            const int k = j - (kStepTaps - 1 - nt);
            if (k >= 0) a.tail_out[off + (size_t)k * width + c] = j + 1 < kStepTaps - 1 ? u[i][j + 1] : h;
        }
    }
}

// Rows without convolution and mixes, four columns at a time: NV pieces per thread, weights fetched ahead of the wait.
constexpr int kPlainThreads = 256;

__device__ __forceinline__ float sum4(const float4& a, const float4& b) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w))); }
__device__ __forceinline__ float4 fma4(float s, const float4& a, const float4& b) {
    return make_float4(fmaf(s, a.x, b.x), fmaf(s, a.y, b.y), fmaf(s, a.z, b.z), fmaf(s, a.w, b.w));
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, const float4& v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(reinterpret_cast<const uint32_t&>(lo), reinterpret_cast<const uint32_t&>(hi));
}

template <typename T, int NV>
__global__ void __launch_bounds__(kPlainThreads) rows_plain_kernel(const RowsArgs a) {
    __shared__ float2 s_red[2][32];
    const int t = blockIdx.x, width = a.width;
    float4 w[NV], g[NV], x[NV], y[NV];
    const float4 one = make_float4(1, 1, 1, 1), zero = make_float4(0, 0, 0, 0);
    auto at = [&](int i) { return (threadIdx.x + i * kPlainThreads) * 4; };
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        w[i] = a.w0 && at(i) < width ? *reinterpret_cast<const float4*>(a.w0 + at(i)) : one;
        g[i] = a.gain_w && at(i) < width ? *reinterpret_cast<const float4*>(a.gain_w + at(i)) : one;
        x[i] = y[i] = zero;
    }
    pdl_wait();
    pdl_launch_dependents();
    if (a.tokens) {
        const bf16* e = static_cast<const bf16*>(a.embed) + (size_t)min(max(a.tokens[t], 0), a.vocab - 1) * width;
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (at(i) < width) {
                const uint2 u = *reinterpret_cast<const uint2*>(e + at(i));
                bf16x2_to_f(u.x, x[i].x, x[i].y);
                bf16x2_to_f(u.y, x[i].z, x[i].w);
            }
    } else {
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (at(i) < width) x[i] = *reinterpret_cast<const float4*>(a.x_in + (size_t)t * width + at(i));
        if (a.y_slot) {
            for (int j = 0; j < a.n_y; ++j) {
                const float s = a.y_weight[(size_t)t * a.n_y + j];
                const float* src = a.y0 + (size_t)a.y_slot[(size_t)t * a.n_y + j] * a.ld_y;
#pragma unroll
                for (int i = 0; i < NV; ++i)
                    if (at(i) < width) y[i] = fma4(s, *reinterpret_cast<const float4*>(src + at(i)), y[i]);
            }
        } else if (a.y0) {
#pragma unroll
            for (int i = 0; i < NV; ++i)
                if (at(i) < width) y[i] = *reinterpret_cast<const float4*>(a.y0 + (size_t)t * a.ld_y + at(i));
        }
    }
    float inv = 1.0f;
    if (a.w0 && !a.tokens) {
        float q = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i) q += sum4(y[i], y[i]);
        q = block_sum2(make_float2(q, 0.0f), s_red[0]).x;
        inv = 1.0f / sqrtf(q / (float)width + a.eps);
    }
    float q = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        x[i].x += y[i].x * inv * w[i].x; x[i].y += y[i].y * inv * w[i].y; x[i].z += y[i].z * inv * w[i].z; x[i].w += y[i].w * inv * w[i].w;
        q += sum4(x[i], x[i]);
        if (at(i) < width) *reinterpret_cast<float4*>(a.x_out + (size_t)t * width + at(i)) = x[i];
    }
    q = block_sum2(make_float2(q, 0.0f), s_red[1]).x;
    inv = 1.0f / sqrtf(q / (float)width + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + (size_t)t * a.ld_out;
#pragma unroll
    for (int i = 0; i < NV; ++i)
        if (at(i) < width) {
            const float s = inv * a.gain;
            store4(out + at(i), make_float4(x[i].x * s * g[i].x, x[i].y * s * g[i].y, x[i].z * s * g[i].z, x[i].w * s * g[i].w));
        }
}

// Residual and inverse RMS of a row.
__global__ void __launch_bounds__(kNormThreads) rows_norm_kernel(const RowsArgs a) {
    __shared__ float2 s_red[2][32];
    const int t = blockIdx.x, width = a.width;
    pdl_wait();
    pdl_launch_dependents();
    const RowSource src(a, t);
    float i0 = 0.0f, i1 = 0.0f;
    float2 q = make_float2(0.0f, 0.0f);
    if (src.normed) {
#pragma unroll 4
        for (int c = threadIdx.x; c < width; c += kNormThreads) {
            const float u = src.first(c), v = src.y1 ? src.y1[c] : 0.0f;
            q.x = fmaf(u, u, q.x);
            q.y = fmaf(v, v, q.y);
        }
        q = block_sum2(q, s_red[0]);
        i0 = 1.0f / sqrtf(q.x / (float)width + a.eps);
        i1 = 1.0f / sqrtf(q.y / (float)width + a.eps);
    }
    q = make_float2(0.0f, 0.0f);
    float* xo = a.x_out + (size_t)t * width;
#pragma unroll 4
    for (int c = threadIdx.x; c < width; c += kNormThreads) {
        float x = src.plain(c);
        if (src.normed) {
            const float v = src.first(c) * i0 * a.w0[c];
            x += src.y1 ? 0.5f * (v + src.y1[c] * i1 * a.w1[c]) : v;
        }
        xo[c] = x;
        q.x = fmaf(x, x, q.x);
    }
    q = block_sum2(q, s_red[1]);
    if (threadIdx.x == 0) a.row_inv[t] = 1.0f / sqrtf(q.x / (float)width + a.eps);
}

// Convolution and mixes over kConvRows rows of one channel per thread; decode: one row, with its own carried state.
// NT: taps rounded up to 4 or 16.
template <typename T, bool DECODE, int NT>
__global__ void __launch_bounds__(kConvThreads) rows_conv_kernel(const RowsArgs a) {
    const int c = blockIdx.x * kConvThreads + threadIdx.x, width = a.width, taps = a.conv_w ? a.taps : 1, nt = taps - 1;
    pdl_wait();
    pdl_launch_dependents();
    if (c >= width) return;
    const int t0 = blockIdx.y * (DECODE ? 1 : kConvRows), n_rows = DECODE ? 1 : min(kConvRows, a.M - t0);
    const size_t off = DECODE ? (size_t)t0 * a.seq_stride : 0;
    const float* tail_in = a.tail_in + off;
    const float gain = a.gain_w ? a.gain * a.gain_w[c] : a.gain;
    // input of the convolution at row t: from the launch, or from the carried rows before it
    auto input = [&](int t) {
        const int rel = DECODE ? t - t0 : t;
        if (rel < 0) return rel >= -nt ? tail_in[(size_t)(nt + rel) * width + c] : 0.0f;
        return a.x_out[(size_t)t * width + c] * a.row_inv[t] * gain;
    };
    const bool lead = a.mu && !DECODE && t0 > 0;                 // the shift starts from the row before, recomputed
    const int start = lead ? -1 : 0;
    float w[NT], u[NT];                                          // w[NT-1] belongs to the current row
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        w[j] = a.conv_w && j >= NT - taps ? a.conv_w[(size_t)(j - NT + taps) * width + c] : 0.0f;
        u[j] = a.conv_w && j > NT - taps ? input(t0 + start - NT + j) : 0.0f;
    }
    float prev = a.mu && !lead ? a.prev_in[off + c] : 0.0f, in[kConvRows + 1];
#pragma unroll
    for (int i = 0; i <= (DECODE ? 0 : kConvRows); ++i) in[i] = start + i < n_rows ? input(t0 + start + i) : 0.0f;
    T* out = reinterpret_cast<T*>(a.out);
    const size_t mix_stride = (size_t)a.M * a.ld_out;
#pragma unroll
    for (int k = 0; k <= (DECODE ? 0 : kConvRows); ++k) {
        const int i = start + k;
        if (i >= n_rows) break;
#pragma unroll
        for (int j = 0; j + 1 < NT; ++j) u[j] = u[j + 1];
        u[NT - 1] = in[k];
        float z = 0.0f;
#pragma unroll
        for (int j = 0; j < NT; ++j) z = fmaf(w[j], u[j], z);
        const float y = in[k] + z;
        if (i >= 0) {
            const size_t row = (size_t)(t0 + i) * a.ld_out + c;
            if (a.mu) {
                for (int s = 0; s < a.n_mix; ++s) out[s * mix_stride + row] = from_f<T>(fmaf(prev - y, a.mu[(size_t)s * width + c], y));
            } else {
                out[row] = from_f<T>(y);
            }
        }
        prev = y;
    }
    if (DECODE || t0 + n_rows == a.M) {                          // the state after the last row
        if (a.mu) a.prev_out[off + c] = prev;
        float last[NT];
#pragma unroll
        for (int j = 0; j < NT; ++j) last[j] = j < nt ? input(t0 + n_rows - nt + j) : 0.0f;
#pragma unroll
        for (int j = 0; j < NT; ++j)
            if (j < nt) a.tail_out[off + (size_t)j * width + c] = last[j];
    }
}

int launch_rows(const RowsArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    if (a.M <= 0) return 0;
    if (a.taps < 1 || a.taps > kMaxTaps || a.width <= 0 || a.n_mix > 8) return -1;
    if ((a.y_slot && (!a.y_weight || a.n_y < 1)) || (a.y1 && !a.w0)) return -1;
    const bool alone = a.decode || (!a.conv_w && !a.mu);          // no row looks at another one of the launch
    if (!a.conv_w && !a.mu && !a.y1 && !a.pos_table && a.width <= 16 * kPlainThreads && a.width % 4 == 0 && a.ld_out % 4 == 0 && a.ld_y % 4 == 0) {
        auto go = [&](auto kernel) { return launch_kernel(kernel, dim3(a.M), dim3(kPlainThreads), 0, st, a.use_pdl, 1, a); };
        *n_kernels += 1;
        const int nv = (a.width + 4 * kPlainThreads - 1) / (4 * kPlainThreads);
        if (a.f32) return nv == 1 ? go(rows_plain_kernel<float, 1>) : nv == 2 ? go(rows_plain_kernel<float, 2>) : nv == 3 ? go(rows_plain_kernel<float, 3>) : go(rows_plain_kernel<float, 4>);
        return nv == 1 ? go(rows_plain_kernel<bf16, 1>) : nv == 2 ? go(rows_plain_kernel<bf16, 2>) : nv == 3 ? go(rows_plain_kernel<bf16, 3>) : go(rows_plain_kernel<bf16, 4>);
    }
    if (alone && a.width <= kStepThreads * kStepMaxCols && a.taps <= kStepTaps) {
        auto go = [&](auto kernel) { return launch_kernel(kernel, dim3(a.M), dim3(kStepThreads), 0, st, a.use_pdl, 1, a); };
        *n_kernels += 1;
        const int cols = (a.width + kStepThreads - 1) / kStepThreads;
        if (a.f32) return cols == 1 ? go(rows_step_kernel<float, 1>) : cols == 2 ? go(rows_step_kernel<float, 2>) : go(rows_step_kernel<float, 4>);
        return cols == 1 ? go(rows_step_kernel<bf16, 1>) : cols == 2 ? go(rows_step_kernel<bf16, 2>) : go(rows_step_kernel<bf16, 4>);
    }
    if (!a.row_inv) return -1;
    *n_kernels += 2;
    if (int rc = launch_kernel(rows_norm_kernel, dim3(a.M), dim3(kNormThreads), 0, st, a.use_pdl, 1, a)) return rc;
    const dim3 grid((a.width + kConvThreads - 1) / kConvThreads, a.decode ? a.M : (a.M + kConvRows - 1) / kConvRows);
    auto go = [&](auto kernel) { return launch_kernel(kernel, grid, dim3(kConvThreads), 0, st, a.use_pdl, 1, a); };
    if (a.taps <= 4) {
        if (a.f32) return a.decode ? go(rows_conv_kernel<float, true, 4>) : go(rows_conv_kernel<float, false, 4>);
        return a.decode ? go(rows_conv_kernel<bf16, true, 4>) : go(rows_conv_kernel<bf16, false, 4>);
    }
    if (a.f32) return a.decode ? go(rows_conv_kernel<float, true, kMaxTaps>) : go(rows_conv_kernel<float, false, kMaxTaps>);
    return a.decode ? go(rows_conv_kernel<bf16, true, kMaxTaps>) : go(rows_conv_kernel<bf16, false, kMaxTaps>);
}

}  // namespace tz

extern "C" int tenzo_cuda_rows(const tenzo_rows_args* args, void* stream) {
    if (!args) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::RowsArgs a;
    static_cast<tenzo_rows_args&>(a) = *args;
    unsigned long long n = 0;
    return tz::launch_rows(a, static_cast<cudaStream_t>(stream), &n);
}
