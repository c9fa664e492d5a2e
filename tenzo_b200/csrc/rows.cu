// Row kernels of the hybrid decoders: residual update, RMS norm with one gain, causal convolution over time on every
// channel, and the token-shift mixes of a time-mixing layer, in one pass over the residual.
//
// A CTA owns TR consecutive rows (one row in decode) and keeps their normalised inputs in shared memory, plus the rows
// before them that the convolution and the shift reach back to. Those halo rows are recomputed from the residual
// source instead of being exchanged between CTAs, which is why the updated residual goes to a second buffer; before the
// first row of the launch they come from the sequence's carried state.
#include "hybrid_common.cuh"

namespace tz {

constexpr int kRowThreads = 512;

struct RowsLaunch {
    RowsArgs a;
    int TR, halo;
};

__device__ __forceinline__ float rows_source(const RowsArgs& a, int t, int c, float inv0, float inv1, int tok, int p) {
    if (a.tokens) return to_f(static_cast<const bf16*>(a.embed)[(size_t)tok * a.width + c]) + to_f(static_cast<const bf16*>(a.pos_table)[(size_t)p * a.width + c]);
    float x = a.x_in[(size_t)t * a.width + c];
    if (a.y1) {
        const float l = a.y0[(size_t)t * a.ld_y + c] * inv0 * a.w0[c], r = a.y1[(size_t)t * a.ld_y + c] * inv1 * a.w1[c];
        x += 0.5f * (l + r);
    } else if (a.y0) {
        x += a.y0[(size_t)t * a.ld_y + c];
    }
    return x;
}

// Sum over the group's threads: a warp (chunk launches: one warp per row) or the whole block (decode).
template <bool DECODE>
__device__ __forceinline__ float group_sum(float v, float* scratch) {
    return DECODE ? block_sum(v, scratch) : warp_sum(v);
}

// NT: taps rounded up to 4 or 16.
template <typename T, bool DECODE, int NT>
__global__ void __launch_bounds__(kRowThreads) rows_kernel(const RowsLaunch L) {
    extern __shared__ float s_h[];                      // [halo + TR][width]
    __shared__ float s_red[kRowThreads / 32];
    const RowsArgs& a = L.a;
    const int width = a.width, halo = L.halo;
    const int t0 = blockIdx.x * L.TR, n_rows = min(L.TR, a.M - t0);
    pdl_wait();
    pdl_launch_dependents();
    const float* tail_in = a.tail_in;
    const float* prev_in = a.prev_in;
    float *tail_out = a.tail_out, *prev_out = a.prev_out;
    if (DECODE) {
        const size_t off = (size_t)blockIdx.x * a.seq_stride;
        tail_in += off; tail_out += off;
        if (prev_in) { prev_in += off; prev_out += off; }
    }
    const int lane_g = DECODE ? threadIdx.x : (threadIdx.x & 31), size_g = DECODE ? kRowThreads : 32;
    const int groups = DECODE ? 1 : kRowThreads / 32, group = DECODE ? 0 : threadIdx.x >> 5;
    const float inv_w = 1.0f / (float)width;
    // rows of this launch: residual, norm
    for (int r = group; r < halo + n_rows; r += groups) {
        const int t = t0 - halo + r;
        if (DECODE ? r < halo : t < 0) continue;
        int tok = 0, p = 0;
        if (a.tokens) {
            tok = min(max(a.tokens[t], 0), a.vocab - 1);
            p = min(max(a.pos[t], 0), a.n_pos - 1);
        }
        float inv0 = 0.0f, inv1 = 0.0f;
        if (a.y1) {
            float q0 = 0.0f, q1 = 0.0f;
            for (int c = lane_g; c < width; c += size_g) {
                const float u = a.y0[(size_t)t * a.ld_y + c], v = a.y1[(size_t)t * a.ld_y + c];
                q0 = fmaf(u, u, q0);
                q1 = fmaf(v, v, q1);
            }
            q0 = group_sum<DECODE>(q0, s_red);
            q1 = group_sum<DECODE>(q1, s_red);
            inv0 = 1.0f / sqrtf(q0 * inv_w + a.eps);
            inv1 = 1.0f / sqrtf(q1 * inv_w + a.eps);
        }
        float* hrow = s_h + (size_t)r * width;
        float q = 0.0f;
#pragma unroll 4
        for (int c = lane_g; c < width; c += size_g) {
            const float x = rows_source(a, t, c, inv0, inv1, tok, p);
            q = fmaf(x, x, q);
            hrow[c] = x;
            if (r >= halo) a.x_out[(size_t)t * width + c] = x;
        }
        q = group_sum<DECODE>(q, s_red);
        const float inv = 1.0f / sqrtf(q * inv_w + a.eps);
        for (int c = lane_g; c < width; c += size_g) hrow[c] = hrow[c] * inv * a.gain;   // a thread rescales what it stored
    }
    // rows before the launch, from the carried state
    const int taps = a.conv_w ? a.taps : 1, nt = taps - 1;
    for (int r = 0; r < halo; ++r) {
        const int t = DECODE ? r - halo : t0 - halo + r;        // relative to the launch's first row
        if (t >= 0) break;
        if (t < -nt) continue;                                   // only the shift's own state reaches there
        for (int c = threadIdx.x; c < width; c += kRowThreads) s_h[(size_t)r * width + c] = tail_in[(size_t)(nt + t) * width + c];
    }
    __syncthreads();
    // convolution, mixes
    T* out = reinterpret_cast<T*>(a.out);
    const size_t mix_stride = (size_t)a.M * a.ld_out;
    const bool lead = a.mu && !DECODE && t0 > 0;                 // the shift starts from the row before, recomputed
    for (int c = threadIdx.x; c < width; c += kRowThreads) {
        // w[NT-1] belongs to the current row; u holds the last NT inputs, those before the convolution's reach as zero
        float w[NT], u[NT];
        const int start = lead ? -1 : 0;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const bool in = j >= NT - taps;
            w[j] = in && a.conv_w ? a.conv_w[(size_t)(j - NT + taps) * width + c] : 0.0f;
            u[j] = j > NT - taps && a.conv_w ? s_h[(size_t)max(0, halo + start - NT + j) * width + c] : 0.0f;
        }
        float prev = a.mu && !lead ? prev_in[c] : 0.0f;
        for (int i = start; i < n_rows; ++i) {
#pragma unroll
            for (int j = 0; j + 1 < NT; ++j) u[j] = u[j + 1];
            u[NT - 1] = s_h[(size_t)(halo + i) * width + c];
            float y = u[NT - 1];
            if (a.conv_w) {
                float z = 0.0f;
#pragma unroll
                for (int j = 0; j < NT; ++j) z = fmaf(w[j], u[j], z);
                y += z;
            }
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
        if (t0 + n_rows == a.M || DECODE) {                      // the state after the last row
            if (a.mu) prev_out[c] = prev;
            for (int i = 0; i < nt; ++i)                         // rows n_rows - nt .. n_rows - 1 relative to the tile
                tail_out[(size_t)i * width + c] = s_h[(size_t)(halo + n_rows - nt + i) * width + c];
        }
    }
}

int launch_rows(const RowsArgs& a, cudaStream_t st) {
    if (a.M <= 0) return 0;
    if (a.taps < 1 || a.taps > kMaxTaps || a.width <= 0 || a.n_mix > 8) return -1;
    RowsLaunch L;
    L.a = a;
    const int nt = a.conv_w ? a.taps - 1 : 0;
    L.halo = a.decode ? nt : nt + (a.mu ? 1 : 0);
    const size_t row_bytes = (size_t)a.width * 4;
    L.TR = 1;
    if (!a.decode)
        while (L.TR < 8 && (L.halo + 2 * L.TR) * row_bytes <= 108 * 1024) L.TR *= 2;
    const size_t smem = (L.halo + L.TR) * row_bytes;
    if (smem > 220 * 1024) return -1;
    const dim3 grid((a.M + L.TR - 1) / L.TR);
    auto go = [&](auto kernel) {
        if (int rc = allow_smem(kernel, smem)) return rc;
        return launch_kernel(kernel, grid, dim3(kRowThreads), smem, st, a.use_pdl, 1, L);
    };
    if (a.taps <= 4) {
        if (a.f32) return a.decode ? go(rows_kernel<float, true, 4>) : go(rows_kernel<float, false, 4>);
        return a.decode ? go(rows_kernel<bf16, true, 4>) : go(rows_kernel<bf16, false, 4>);
    }
    if (a.f32) return a.decode ? go(rows_kernel<float, true, kMaxTaps>) : go(rows_kernel<float, false, kMaxTaps>);
    return a.decode ? go(rows_kernel<bf16, true, kMaxTaps>) : go(rows_kernel<bf16, false, kMaxTaps>);
}

}  // namespace tz

extern "C" int tenzo_cuda_rows(const tenzo_rows_args* args, void* stream) {
    if (!args) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::RowsArgs a;
    static_cast<tenzo_rows_args&>(a) = *args;
    return tz::launch_rows(a, static_cast<cudaStream_t>(stream));
}
