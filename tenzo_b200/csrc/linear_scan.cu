// Linear recurrences with a decaying matrix state (ScanArgs): retention (a constant per head), gated linear attention (a
// decay per key channel and token, read after the update) and RWKV-style time mixing (the same decay shape, read before
// the update with a bonus for the current token). States, decays and sums are fp32.
//
// Decode: one CTA per (head, sequence); the state is fetched before the kernel waits for its producer - the kernel that
// wrote it lies several launches back - and normalisation, weight and gate are applied on the way out.
// Chunk: rows are cut into blocks of kScanBlock. The blocks' own states from zero and their decay products are formed in
// parallel, a short pass carries the state across blocks, and every block is then walked from its true starting
// state. Products of decays only ever multiply states, so small decays underflow harmlessly.
#include <type_traits>

#include "hybrid_common.cuh"

namespace tz {

constexpr int kScanThreads = 256, kScanBlock = 64;

// decay from the gate's value
__device__ __forceinline__ float gate_decay(int kind, float z, float tau) {
    return kind == TENZO_DECAY_SIGMOID_ROOT ? expf(-softplus_neg(z) / tau) : expf(-expf(z));
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
    float* s_low = s_u + a.dim;                          // [rank, padded to 8]
    float* s_v = s_low + ((a.rank + 7) & ~7);            // [ldv]
    float* s_o = sm + ((4 * a.dim + ((a.rank + 7) & ~7) + ldv + 3) & ~3);   // [n_rg][ldv]
    float* s_red = s_o + n_rg * ldv;                     // [8]
    // low-rank gate: four lanes per channel, 16-byte pieces of its row; the first two are fetched ahead as well
    const bool gated = a.decay_kind != TENZO_DECAY_CONST;
    const int rank8 = (a.rank + 7) & ~7, sub = tid & 3;
    const bf16* up = static_cast<const bf16*>(a.up) + (size_t)head * a.dim * rank8;
    uint4 gate[2] = {};
#pragma unroll
    for (int i = 0; i < 2; ++i)
        if (gated && tid / 4 < a.dim && (sub + 4 * i) * 8 < rank8) gate[i] = *reinterpret_cast<const uint4*>(up + (size_t)(tid / 4) * rank8 + (sub + 4 * i) * 8);
    pdl_wait();
    pdl_launch_dependents();
    const size_t row = (size_t)seq * a.ld;
    for (int i = tid; i < rank8; i += kScanThreads) {
        const float l = i < a.rank ? a.low[row + i] : 0.0f;
        s_low[i] = a.decay_kind == TENZO_DECAY_EXP_EXP ? tanhf(l) : l;
    }
    for (int i = tid; i < a.dim; i += kScanThreads) {
        s_q[i] = a.q[row + head * a.dim + i] * a.q_scale;
        s_k[i] = a.k[row + head * a.dim + i] * a.k_scale;
        s_u[i] = a.bonus ? a.bonus[head * a.dim + i] : 0.0f;
    }
    for (int i = tid; i < ldv; i += kScanThreads) s_v[i] = i < a.vdim ? a.v[row + head * a.vdim + i] : 0.0f;
    __syncthreads();
    if (gated) {
        for (int d0 = 0; d0 < a.dim; d0 += kScanThreads / 4) {          // uniform trips: the exchanges are warp-wide
            const int d = d0 + tid / 4;
            float z = 0.0f;
            if (d < a.dim)
                for (int i = 0; (sub + 4 * i) * 8 < rank8; ++i) {
                    const int c = (sub + 4 * i) * 8;
                    float u[8];
                    if (d0 == 0 && i < 2) unpack8(i ? gate[1] : gate[0], u); else load8(up + (size_t)d * rank8 + c, u);
#pragma unroll
                    for (int j = 0; j < 8; ++j) z = fmaf(u[j], s_low[c + j], z);
                }
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            z += __shfl_xor_sync(0xffffffffu, z, 2);
            if (sub == 0 && d < a.dim) s_w[d] = gate_decay(a.decay_kind, z + a.bias[head * a.dim + d], a.tau);
        }
    } else {
        for (int i = tid; i < a.dim; i += kScanThreads) s_w[i] = a.decay[head];
    }
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
// Decays of all rows and channels: 64 channels x 32 rows per CTA, 32 of the rank at a time in shared memory.
__global__ void __launch_bounds__(256) scan_decay_rows_kernel(const ScanArgs a) {
    __shared__ float s_up[32][65], s_low[32][33];
    const int n = a.heads * a.dim, rank8 = (a.rank + 7) & ~7, tid = threadIdx.x;
    const int c = tid & 63, r0 = (tid >> 6) * 8, ch0 = blockIdx.x * 64, t0 = blockIdx.y * 32;
    float z[8] = {};
    for (int k0 = 0; k0 < a.rank; k0 += 32) {
        for (int i = tid; i < 64 * 32; i += 256) {
            const int k = i & 31, cc = i >> 5;
            s_up[k][cc] = ch0 + cc < n && k0 + k < a.rank ? to_f(static_cast<const bf16*>(a.up)[(size_t)(ch0 + cc) * rank8 + k0 + k]) : 0.0f;
        }
        for (int i = tid; i < 32 * 32; i += 256) {
            const int k = i & 31, r = i >> 5;
            const float l = t0 + r < a.M && k0 + k < a.rank ? a.low[(size_t)(t0 + r) * a.ld + k0 + k] : 0.0f;
            s_low[r][k] = a.decay_kind == TENZO_DECAY_EXP_EXP ? tanhf(l) : l;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < 32; ++k)
#pragma unroll
            for (int r = 0; r < 8; ++r) z[r] = fmaf(s_up[k][c], s_low[r0 + r][k], z[r]);
        __syncthreads();
    }
    if (ch0 + c >= n) return;
#pragma unroll
    for (int r = 0; r < 8; ++r)
        if (t0 + r0 + r < a.M) a.w_rows[(size_t)(t0 + r0 + r) * n + ch0 + c] = gate_decay(a.decay_kind, z[r] + a.bias[ch0 + c], a.tau);
}

// A block of rows for 32 value columns of one head, 64 threads: lane = 4 * column pair + key slice; a key slice owns the
// rows 4 * (slice + 4 j) .. + 3 of the state, so that the four slices read adjacent 16-byte pieces of k, q and w. Rows are
// staged by asynchronous copies, one tile ahead.
// Pass 1 (OUT = 0) starts from zero and leaves the block's own state and decay products, pass 2 (OUT = 1) starts
// from the state before the block and writes the outputs. WC: the decay is one constant per head.
constexpr int kScanCols = 32;

struct ScanBlockLaunch {
    ScanArgs a;
    float *own, *prod;
    const float* start;
    int vec_k, vec_v;            // key / value rows can be copied 16 bytes at a time
};

template <int KJ, bool OUT, bool WC>
struct ScanBlockShape {
    static constexpr int KD = KJ * 16, TILE = KJ > 8 ? 8 : 16;            // padded key size, rows per tile
    static constexpr int K = 0, Q = TILE * KD, W = Q + (OUT ? TILE * KD : 0), V = W + (WC ? 0 : TILE * KD), FLOATS = V + TILE * kScanCols;
};

__device__ __forceinline__ void async_copy(float* dst, const float* src, int vec) {
    if (vec) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}
// `rows` x `cols` floats, destination rows of ld_dst
__device__ __forceinline__ void async_tile(float* dst, int ld_dst, const float* src, size_t ld_src, int rows, int cols, int vec) {
    const int step = vec ? 4 : 1, per = cols / step;
    for (int i = threadIdx.x; i < rows * per; i += 64) {
        const int r = i / per, c = (i - r * per) * step;
        async_copy(dst + r * ld_dst + c, src + (size_t)r * ld_src + c, vec);
    }
}

template <int KJ, bool OUT, bool WC>
__global__ void __launch_bounds__(64) scan_block_kernel(const ScanBlockLaunch L) {
    using S = ScanBlockShape<KJ, OUT, WC>;
    constexpr int KD = S::KD, TILE = S::TILE;
    extern __shared__ __align__(16) float smem[];
    const ScanArgs& a = L.a;
    const int head = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int slice = lane & 3, cl = warp * 16 + (lane >> 2) * 2, c0 = blockIdx.x * kScanCols + cl;
    const int ldv = (a.vdim + 3) & ~3, n = a.heads * a.dim;
    const int t_begin = b * kScanBlock, t_end = min(a.M, t_begin + kScanBlock);
    const int v_cols = min(kScanCols, a.vdim - (int)blockIdx.x * kScanCols);
    for (int i = tid; i < 2 * S::FLOATS / 4; i += 64) reinterpret_cast<float4*>(smem)[i] = make_float4(0, 0, 0, 0);     // padding
    float st[2][KJ * 4], P[OUT ? 1 : KJ * 4], U[OUT ? KJ * 4 : 1];
#pragma unroll
    for (int j = 0; j < KJ * 4; ++j) {
        const int d = 4 * (slice + 4 * (j >> 2)) + (j & 3);
#pragma unroll
        for (int c = 0; c < 2; ++c)
            st[c][j] = OUT && d < a.dim && c0 + c < a.vdim ? L.start[((size_t)b * a.heads + head) * a.dim * ldv + (size_t)d * ldv + c0 + c] : 0.0f;
        if (!OUT) P[OUT ? 0 : j] = 1.0f;
        if (OUT) U[OUT ? j : 0] = a.bonus && d < a.dim ? a.bonus[head * a.dim + d] : 0.0f;
    }
    const float w_const = WC ? a.decay[head] : 0.0f;
    auto stage = [&](int tb, float* buf) {
        const int nt = min(TILE, t_end - tb);
        async_tile(buf + S::K, KD, a.k + (size_t)tb * a.ld + head * a.dim, a.ld, nt, a.dim, L.vec_k);
        if (OUT) async_tile(buf + S::Q, KD, a.q + (size_t)tb * a.ld + head * a.dim, a.ld, nt, a.dim, L.vec_k);
        if (!WC) async_tile(buf + S::W, KD, a.w_rows + (size_t)tb * n + head * a.dim, n, nt, a.dim, L.vec_k);
        async_tile(buf + S::V, kScanCols, a.v + (size_t)tb * a.ld + head * a.vdim + blockIdx.x * kScanCols, a.ld, nt, v_cols, L.vec_v);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    __syncthreads();
    stage(t_begin, smem);
    int flip = 0;
    for (int tb = t_begin; tb < t_end; tb += TILE, flip ^= 1) {
        const int nt = min(TILE, t_end - tb);
        if (tb + TILE < t_end) {
            stage(tb + TILE, smem + (flip ^ 1) * S::FLOATS);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* buf = smem + flip * S::FLOATS;
        for (int r = 0; r < nt; ++r) {
            float2 v = *reinterpret_cast<const float2*>(buf + S::V + r * kScanCols + cl);
            v.x *= a.k_scale;
            v.y *= a.k_scale;
            float o0[2] = {}, o1[2] = {};
#pragma unroll
            for (int jj = 0; jj < KJ; ++jj) {
                const int d = r * KD + 4 * (slice + 4 * jj);
                const float4 k4 = *reinterpret_cast<const float4*>(buf + S::K + d);
                const float4 w4 = WC ? make_float4(w_const, w_const, w_const, w_const) : *reinterpret_cast<const float4*>(buf + S::W + d);
                const float4 q4 = OUT ? *reinterpret_cast<const float4*>(buf + S::Q + d) : make_float4(0, 0, 0, 0);
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, ww[4] = {w4.x, w4.y, w4.z, w4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int j = jj * 4 + i;
                    const float kv0 = kk[i] * v.x, kv1 = kk[i] * v.y;
                    if (OUT && a.bonus) {
                        o0[i & 1] = fmaf(qq[i], fmaf(U[OUT ? j : 0], kv0, st[0][j]), o0[i & 1]);
                        o1[i & 1] = fmaf(qq[i], fmaf(U[OUT ? j : 0], kv1, st[1][j]), o1[i & 1]);
                    }
                    st[0][j] = fmaf(ww[i], st[0][j], kv0);
                    st[1][j] = fmaf(ww[i], st[1][j], kv1);
                    if (OUT && !a.bonus) {
                        o0[i & 1] = fmaf(qq[i], st[0][j], o0[i & 1]);
                        o1[i & 1] = fmaf(qq[i], st[1][j], o1[i & 1]);
                    }
                    if (!OUT) P[OUT ? 0 : j] *= ww[i];
                }
            }
            if (OUT) {
                float s0 = o0[0] + o0[1], s1 = o1[0] + o1[1];
                s0 += __shfl_xor_sync(0xffffffffu, s0, 1);
                s1 += __shfl_xor_sync(0xffffffffu, s1, 1);
                s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
                s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
                float* o = a.o_rows + (size_t)(tb + r) * a.heads * a.vdim + head * a.vdim + c0;
                if (slice == 0 && c0 < a.vdim) o[0] = s0 * a.q_scale;
                if (slice == 1 && c0 + 1 < a.vdim) o[1] = s1 * a.q_scale;
            }
        }
        __syncthreads();                                     // the tile is free for the copies after next
    }
    if (!OUT) {
#pragma unroll
        for (int j = 0; j < KJ * 4; ++j) {
            const int d = 4 * (slice + 4 * (j >> 2)) + (j & 3);
            if (d >= a.dim) continue;
            float* dst = L.own + ((size_t)b * a.heads + head) * a.dim * ldv + (size_t)d * ldv + c0;
            if (c0 < a.vdim) dst[0] = st[0][j];
            if (c0 + 1 < a.vdim) dst[1] = st[1][j];
            if (blockIdx.x == 0 && tid < 4) L.prod[((size_t)b * a.heads + head) * a.dim + d] = P[OUT ? 0 : j];
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
    for (int b0 = 0; b0 < n_blocks; b0 += 8) {                // eight blocks' values in flight
        float mine[8], p[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            mine[u] = b0 + u < n_blocks ? own[(size_t)(b0 + u) * n + i] : 0.0f;
            p[u] = b0 + u < n_blocks ? prod[(size_t)(b0 + u) * a.heads * a.dim + row] : 0.0f;
        }
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (b0 + u < n_blocks) {
                own[(size_t)(b0 + u) * n + i] = s;
                s = fmaf(p[u], s, mine[u]);
            }
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

int launch_scan_gate(const ScanArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    const unsigned ctas = (unsigned)(((size_t)a.M * a.heads + 7) / 8);
    if (a.f32) scan_gate_kernel<float><<<ctas, 256, 0, st>>>(a);
    else scan_gate_kernel<bf16><<<ctas, 256, 0, st>>>(a);
    *n_kernels += 1;
    return (int)cudaGetLastError();
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
        const size_t smem = 4 * (size_t)(((4 * a.dim + round_up(rank, 8) + ldv + 3) & ~3) + kScanThreads / nc2 * ldv + 8);
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
        scan_decay_rows_kernel<<<dim3((a.heads * a.dim + 63) / 64, (a.M + 31) / 32), 256, 0, st>>>(p);
        *n_kernels += 1;
    }
    auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    ScanBlockLaunch L = {p, own, prod, own, 0, 0};
    L.vec_k = a.dim % 4 == 0 && a.ld % 4 == 0 && aligned(a.q) && aligned(a.k) && aligned(a.w_rows);
    L.vec_v = a.vdim % 4 == 0 && a.ld % 4 == 0 && aligned(a.v);
    const dim3 grid((a.vdim + kScanCols - 1) / kScanCols, a.heads, n_blocks);
    auto blocks = [&](auto kj, auto wc) {
        constexpr int KJ = decltype(kj)::value;
        constexpr bool WC = decltype(wc)::value;
        const size_t s1 = 8 * ScanBlockShape<KJ, false, WC>::FLOATS, s2 = 8 * ScanBlockShape<KJ, true, WC>::FLOATS;
        if (int rc = allow_smem(scan_block_kernel<KJ, false, WC>, s1)) return rc;
        if (int rc = allow_smem(scan_block_kernel<KJ, true, WC>, s2)) return rc;
        scan_block_kernel<KJ, false, WC><<<grid, 64, s1, st>>>(L);
        scan_carry_kernel<<<(unsigned)(((size_t)a.heads * a.dim * ldv + 255) / 256), 256, 0, st>>>(p, n_blocks, own, prod);
        scan_block_kernel<KJ, true, WC><<<grid, 64, s2, st>>>(L);
        return (int)cudaGetLastError();
    };
    auto sized = [&](auto kj) { return rank ? blocks(kj, std::false_type()) : blocks(kj, std::true_type()); };
    const int rc = a.dim <= 32 ? sized(std::integral_constant<int, 2>()) : a.dim <= 64 ? sized(std::integral_constant<int, 4>())
                 : a.dim <= 128 ? sized(std::integral_constant<int, 8>()) : sized(std::integral_constant<int, 16>());
    if (rc) return rc;
    *n_kernels += 3;
    return launch_scan_gate(p, st, n_kernels);
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
