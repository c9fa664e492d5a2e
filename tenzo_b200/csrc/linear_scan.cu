// Linear recurrences with a decaying matrix state (ScanArgs): retention (a constant per head), gated linear attention (a
// decay per key channel and token, read after the update) and RWKV-style time mixing (the same decay shape, read before
// the update with a bonus for the current token). States, decays and sums are fp32.
//
// Decode: one CTA per (head, sequence); the state is fetched before the kernel waits for its producer - the kernel that
// wrote it lies several launches back - and normalisation, weight and gate are applied on the way out.
// Chunk: rows are cut into blocks of kScanBlock. The blocks' own states from zero and their decay products are formed in
// parallel, a short pass carries the state across blocks, and every block is then walked from its true starting
// state. Products of decays only ever multiply states, so small decays underflow harmlessly.
#include "hybrid_common.cuh"

namespace tz {

constexpr int kScanThreads = 256, kScanBlock = 64;

// decay of channel ch (head * dim + d) for one row of low-rank values (fp32 in `low`, already through tanh if asked for)
__device__ __forceinline__ float scan_decay(const ScanArgs& a, int ch, const float* low) {
    if (a.decay_kind == TENZO_DECAY_CONST) return a.decay[ch / a.dim];
    float z = a.bias[ch];
    const bf16* u = static_cast<const bf16*>(a.up) + (size_t)ch * a.rank;
    for (int r = 0; r < a.rank; ++r) z = fmaf(to_f(u[r]), low[r], z);
    return a.decay_kind == TENZO_DECAY_SIGMOID_ROOT ? expf(-softplus_neg(z) / a.tau) : expf(-expf(z));
}

// ---- decode --------------------------------------------------------------------------------------------------------------
constexpr int kScanPre = 8;                              // state rows of a thread that are fetched ahead

template <typename T>
__global__ void __launch_bounds__(kScanThreads) scan_decode_kernel(const ScanArgs a) {
    extern __shared__ float sm[];
    const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
    const int ldv = (a.vdim + 3) & ~3, nc = ldv / 4;
    int nc2 = 1;
    while (nc2 < nc) nc2 *= 2;
    const int col = tid & (nc2 - 1), rg = tid / nc2, n_rg = kScanThreads / nc2;   // vdim <= 256: at least four row groups
    const bool live = col < nc;
    float4* S = reinterpret_cast<float4*>(a.state + (size_t)seq * a.state_seq_stride + (size_t)head * a.dim * ldv) + col;
    float4 pre[kScanPre];
#pragma unroll
    for (int i = 0; i < kScanPre; ++i) {
        const int r = rg + i * n_rg;
        if (live && r < a.dim) pre[i] = S[(size_t)r * nc];
    }
    float* s_q = sm;                                     // [dim]
    float* s_k = s_q + a.dim;
    float* s_w = s_k + a.dim;
    float* s_u = s_w + a.dim;                            // bonus
    float* s_low = s_u + a.dim;                          // [rank]
    float* s_v = s_low + a.rank;                         // [ldv]
    float* s_o = sm + ((4 * a.dim + a.rank + ldv + 3) & ~3);    // [n_rg][ldv]
    float* s_red = s_o + n_rg * ldv;                     // [8]
    pdl_wait();
    pdl_launch_dependents();
    const size_t row = (size_t)seq * a.ld;
    for (int i = tid; i < a.rank; i += kScanThreads) {
        const float l = a.low[row + i];
        s_low[i] = a.decay_kind == TENZO_DECAY_EXP_EXP ? tanhf(l) : l;
    }
    for (int i = tid; i < a.dim; i += kScanThreads) {
        s_q[i] = a.q[row + head * a.dim + i] * a.q_scale;
        s_k[i] = a.k[row + head * a.dim + i] * a.k_scale;
        s_u[i] = a.bonus ? a.bonus[head * a.dim + i] : 0.0f;
    }
    for (int i = tid; i < ldv; i += kScanThreads) s_v[i] = i < a.vdim ? a.v[row + head * a.vdim + i] : 0.0f;
    __syncthreads();
    for (int i = tid; i < a.dim; i += kScanThreads) s_w[i] = scan_decay(a, head * a.dim + i, s_low);
    __syncthreads();
    float o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    if (live) {
        const float v[4] = {s_v[col * 4], s_v[col * 4 + 1], s_v[col * 4 + 2], s_v[col * 4 + 3]};
        auto step = [&](int r, const float4& sv) {
            const float w = s_w[r], k = s_k[r], q = s_q[r], u = s_u[r];
            const float s[4] = {sv.x, sv.y, sv.z, sv.w};
            float n[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float kv = k * v[j];
                n[j] = fmaf(w, s[j], kv);
                o[j] = fmaf(q, a.bonus ? fmaf(u, kv, s[j]) : n[j], o[j]);
            }
            S[(size_t)r * nc] = make_float4(n[0], n[1], n[2], n[3]);
        };
#pragma unroll
        for (int i = 0; i < kScanPre; ++i)
            if (rg + i * n_rg < a.dim) step(rg + i * n_rg, pre[i]);
        for (int r = rg + kScanPre * n_rg; r < a.dim; r += n_rg) step(r, S[(size_t)r * nc]);
#pragma unroll
        for (int j = 0; j < 4; ++j) s_o[rg * ldv + col * 4 + j] = o[j];
    }
    __syncthreads();
    float q = 0.0f;
    for (int d = tid; d < a.vdim; d += kScanThreads) {
        float t = 0.0f;
        for (int r = 0; r < n_rg; ++r) t += s_o[r * ldv + d];
        s_v[d] = t;
        q = fmaf(t, t, q);
    }
    q = block_sum(q, s_red);
    const float inv = 1.0f / sqrtf(q / (float)a.vdim + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + (size_t)seq * a.ld_out + head * a.vdim;
    for (int d = tid; d < a.vdim; d += kScanThreads) {
        float y = s_v[d] * inv;
        if (a.norm) y *= a.norm[(a.norm_per_head ? head * a.vdim : 0) + d];
        out[d] = from_f<T>(y * silu_f(a.g[row + head * a.vdim + d]));
    }
}

// ---- chunk ---------------------------------------------------------------------------------------------------------------
// Decays of all rows and channels. One CTA per row.
__global__ void __launch_bounds__(256) scan_decay_rows_kernel(const ScanArgs a) {
    extern __shared__ float s_low[];
    const size_t t = blockIdx.x;
    for (int i = threadIdx.x; i < a.rank; i += 256) {
        const float l = a.low[t * a.ld + i];
        s_low[i] = a.decay_kind == TENZO_DECAY_EXP_EXP ? tanhf(l) : l;
    }
    __syncthreads();
    const int n = a.heads * a.dim;
    for (int ch = threadIdx.x; ch < n; ch += 256) a.w_rows[t * n + ch] = scan_decay(a, ch, s_low);
}

// A block of rows for 16 value columns of one head, 32 threads: lane = 4 * column pair + key slice; a key slice owns the
// rows 4 * (slice + 4 j) .. + 3 of the state, so that the four slices read adjacent 16-byte pieces of k, q and w.
// Pass 1 (OUT = 0) starts from zero and leaves the block's own state and decay products, pass 2 (OUT = 1) starts
// from the state before the block and writes the outputs.
constexpr int kScanCols = 32;                            // columns per CTA (two warps of 16)

template <int KJ, bool OUT>
__global__ void __launch_bounds__(64) scan_block_kernel(const ScanArgs a, int n_blocks, float* own, float* prod, const float* start) {
    constexpr int KD = KJ * 16, kScanTile = KJ > 8 ? 8 : 16;   // padded key dimension, rows staged at a time
    __shared__ __align__(16) float s_k[kScanTile][KD], s_q[OUT ? kScanTile : 1][KD], s_w[kScanTile][KD];
    __shared__ __align__(16) float s_v[kScanTile][kScanCols];
    const int head = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int slice = lane & 3, c0 = blockIdx.x * kScanCols + warp * 16 + (lane >> 2) * 2;
    const int ldv = (a.vdim + 3) & ~3;
    const int t_begin = b * kScanBlock, t_end = min(a.M, t_begin + kScanBlock);
    float S[2][KJ * 4], P[OUT ? 1 : KJ * 4], U[OUT ? KJ * 4 : 1];
#pragma unroll
    for (int j = 0; j < KJ * 4; ++j) {
        const int d = 4 * (slice + 4 * (j >> 2)) + (j & 3);
#pragma unroll
        for (int c = 0; c < 2; ++c)
            S[c][j] = OUT && d < a.dim && c0 + c < a.vdim ? start[((size_t)b * a.heads + head) * a.dim * ldv + (size_t)d * ldv + c0 + c] : 0.0f;
        if (!OUT) P[OUT ? 0 : j] = 1.0f;
        if (OUT) U[OUT ? j : 0] = a.bonus && d < a.dim ? a.bonus[head * a.dim + d] : 0.0f;
    }
    const float w_const = a.decay_kind == TENZO_DECAY_CONST ? a.decay[head] : 0.0f;
    for (int tb = t_begin; tb < t_end; tb += kScanTile) {
        const int nt = min(kScanTile, t_end - tb);
        __syncthreads();
        for (int i = tid; i < nt * KD; i += 64) {
            const int r = i / KD, d = i - r * KD;
            const size_t row = (size_t)(tb + r) * a.ld + head * a.dim + d;
            const bool in = d < a.dim;
            s_k[r][d] = in ? a.k[row] * a.k_scale : 0.0f;
            if (OUT) s_q[OUT ? r : 0][d] = in ? a.q[row] * a.q_scale : 0.0f;
            s_w[r][d] = in ? (a.decay_kind == TENZO_DECAY_CONST ? w_const : a.w_rows[(size_t)(tb + r) * a.heads * a.dim + head * a.dim + d]) : 0.0f;
        }
        for (int i = tid; i < nt * kScanCols; i += 64) {
            const int r = i / kScanCols, c = i - r * kScanCols, vc = blockIdx.x * kScanCols + c;
            s_v[r][c] = vc < a.vdim ? a.v[(size_t)(tb + r) * a.ld + head * a.vdim + vc] : 0.0f;
        }
        __syncthreads();
        for (int r = 0; r < nt; ++r) {
            const float2 v = *reinterpret_cast<const float2*>(&s_v[r][warp * 16 + (lane >> 2) * 2]);
            float o0 = 0.0f, o1 = 0.0f;
#pragma unroll
            for (int jj = 0; jj < KJ; ++jj) {
                const int d = 4 * (slice + 4 * jj);
                const float4 k4 = *reinterpret_cast<const float4*>(&s_k[r][d]), w4 = *reinterpret_cast<const float4*>(&s_w[r][d]);
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, ww[4] = {w4.x, w4.y, w4.z, w4.w};
                float qq[4] = {};
                if (OUT) {
                    const float4 q4 = *reinterpret_cast<const float4*>(&s_q[OUT ? r : 0][d]);
                    qq[0] = q4.x; qq[1] = q4.y; qq[2] = q4.z; qq[3] = q4.w;
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int j = jj * 4 + i;
                    const float kv0 = kk[i] * v.x, kv1 = kk[i] * v.y;
                    if (OUT && a.bonus) {
                        o0 = fmaf(qq[i], fmaf(U[OUT ? j : 0], kv0, S[0][j]), o0);
                        o1 = fmaf(qq[i], fmaf(U[OUT ? j : 0], kv1, S[1][j]), o1);
                    }
                    S[0][j] = fmaf(ww[i], S[0][j], kv0);
                    S[1][j] = fmaf(ww[i], S[1][j], kv1);
                    if (OUT && !a.bonus) {
                        o0 = fmaf(qq[i], S[0][j], o0);
                        o1 = fmaf(qq[i], S[1][j], o1);
                    }
                    if (!OUT) P[OUT ? 0 : j] *= ww[i];
                }
            }
            if (OUT) {
                o0 += __shfl_xor_sync(0xffffffffu, o0, 1);
                o1 += __shfl_xor_sync(0xffffffffu, o1, 1);
                o0 += __shfl_xor_sync(0xffffffffu, o0, 2);
                o1 += __shfl_xor_sync(0xffffffffu, o1, 2);
                float* o = a.o_rows + (size_t)(tb + r) * a.heads * a.vdim + head * a.vdim + c0;
                if (slice == 0 && c0 < a.vdim) o[0] = o0;
                if (slice == 1 && c0 + 1 < a.vdim) o[1] = o1;
            }
        }
    }
    if (!OUT) {
#pragma unroll
        for (int j = 0; j < KJ * 4; ++j) {
            const int d = 4 * (slice + 4 * (j >> 2)) + (j & 3);
            if (d >= a.dim) continue;
            float* dst = own + ((size_t)b * a.heads + head) * a.dim * ldv + (size_t)d * ldv + c0;
            if (c0 < a.vdim) dst[0] = S[0][j];
            if (c0 + 1 < a.vdim) dst[1] = S[1][j];
            if (blockIdx.x == 0 && tid < 4) prod[((size_t)b * a.heads + head) * a.dim + d] = P[OUT ? 0 : j];
        }
    }
}

// own[b] becomes the state before block b; the state after the last block goes back to the sequence.
__global__ void __launch_bounds__(256) scan_carry_kernel(const ScanArgs a, int n_blocks, float* own, const float* prod) {
    const int ldv = (a.vdim + 3) & ~3;
    const size_t n = (size_t)a.heads * a.dim * ldv, i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= n || (int)(i % ldv) >= a.vdim) return;
    const size_t row = i / ldv;
    float s = a.state[i];
    for (int b = 0; b < n_blocks; ++b) {
        const float mine = own[(size_t)b * n + i];
        own[(size_t)b * n + i] = s;
        s = fmaf(prod[(size_t)b * a.heads * a.dim + row], s, mine);
    }
    a.state[i] = s;
}

// Per head: o / rms(o) * norm * silu(g). One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) scan_gate_kernel(const ScanArgs a) {
    const int wid = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (wid >= a.M * a.heads) return;
    const int t = wid / a.heads, head = wid - t * a.heads;
    const float* o = a.o_rows + (size_t)t * a.heads * a.vdim + head * a.vdim;
    float v[kMaxHeadDim / 32], q = 0.0f;
#pragma unroll
    for (int i = 0; i < kMaxHeadDim / 32; ++i) {
        v[i] = i * 32 + lane < a.vdim ? o[i * 32 + lane] : 0.0f;
        q = fmaf(v[i], v[i], q);
    }
    q = warp_sum(q);
    const float inv = 1.0f / sqrtf(q / (float)a.vdim + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + (size_t)t * a.ld_out + head * a.vdim;
#pragma unroll
    for (int i = 0; i < kMaxHeadDim / 32; ++i) {
        const int d = i * 32 + lane;
        if (d >= a.vdim) continue;
        float y = v[i] * inv;
        if (a.norm) y *= a.norm[(a.norm_per_head ? head * a.vdim : 0) + d];
        out[d] = from_f<T>(y * silu_f(a.g[(size_t)t * a.ld + head * a.vdim + d]));
    }
}

int launch_scan(const ScanArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    if (a.M <= 0) return 0;
    if (a.dim < 1 || a.dim > kMaxHeadDim || a.vdim < 1 || a.vdim > kMaxHeadDim || a.heads < 1) return -1;
    const int rank = a.decay_kind == TENZO_DECAY_CONST ? 0 : a.rank;
    ScanArgs p = a;
    p.rank = rank;
    const int ldv = round_up(a.vdim, 4);
    if (a.decode) {
        int nc2 = 1;
        while (nc2 < ldv / 4) nc2 *= 2;
        const size_t smem = 4 * (size_t)(((4 * a.dim + rank + ldv + 3) & ~3) + kScanThreads / nc2 * ldv + 8);
        const dim3 grid(a.heads, a.M);
        *n_kernels += 1;
        auto go = [&](auto kernel) {
            if (int rc = allow_smem(kernel, smem)) return rc;
            return launch_kernel(kernel, grid, dim3(kScanThreads), smem, st, a.use_pdl, 1, p);
        };
        return a.f32 ? go(scan_decode_kernel<float>) : go(scan_decode_kernel<bf16>);
    }
    const int n_blocks = (a.M + kScanBlock - 1) / kScanBlock;
    float* own = a.part;
    float* prod = own + (size_t)n_blocks * a.heads * a.dim * ldv;
    if (rank) {
        scan_decay_rows_kernel<<<a.M, 256, rank * 4, st>>>(p);
        *n_kernels += 1;
    }
    const dim3 grid((a.vdim + kScanCols - 1) / kScanCols, a.heads, n_blocks);
    auto blocks = [&](auto k1, auto k2) {
        k1<<<grid, 64, 0, st>>>(p, n_blocks, own, prod, nullptr);
        scan_carry_kernel<<<(unsigned)(((size_t)a.heads * a.dim * ldv + 255) / 256), 256, 0, st>>>(p, n_blocks, own, prod);
        k2<<<grid, 64, 0, st>>>(p, n_blocks, nullptr, nullptr, own);
    };
    if (a.dim <= 32) blocks(scan_block_kernel<2, false>, scan_block_kernel<2, true>);
    else if (a.dim <= 64) blocks(scan_block_kernel<4, false>, scan_block_kernel<4, true>);
    else if (a.dim <= 128) blocks(scan_block_kernel<8, false>, scan_block_kernel<8, true>);
    else blocks(scan_block_kernel<16, false>, scan_block_kernel<16, true>);
    const unsigned gate_ctas = (unsigned)(((size_t)a.M * a.heads + 7) / 8);
    if (a.f32) scan_gate_kernel<float><<<gate_ctas, 256, 0, st>>>(p);
    else scan_gate_kernel<bf16><<<gate_ctas, 256, 0, st>>>(p);
    *n_kernels += 4;
    return (int)cudaGetLastError();
}

}  // namespace tz

extern "C" int tenzo_cuda_linear_scan(const tenzo_scan_args* args, void* stream) {
    if (!args) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::ScanArgs a;
    static_cast<tenzo_scan_args&>(a) = *args;
    unsigned long long n = 0;
    return tz::launch_scan(a, static_cast<cudaStream_t>(stream), &n);
}

extern "C" size_t tenzo_cuda_linear_scan_part_floats(int M, int heads, int dim, int vdim) {
    const size_t blocks = (M + tz::kScanBlock - 1) / tz::kScanBlock;
    return blocks * heads * dim * (size_t)(tz::round_up(vdim, 4) + 1);
}
