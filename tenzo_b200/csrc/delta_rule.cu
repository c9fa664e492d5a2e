// Gated delta rule (DeltaArgs): short convolutions with silu on q, k, v, unit q and k, one decay and one step size per head,
// and a matrix state that is decayed, corrected towards v along k, then read. State, decays, step sizes and sums are fp32.
//
// With S the state before a token, a = S^T k and b = S^T q give everything of that token in one pass over the state:
// u = beta (v - g a), o = g b + (k.q) u, and the new state is g S + k u^T.
//
// Decode: one CTA per (head, sequence), its part of the state fetched before the kernel waits for its producer. Inputs of the
// convolutions are kept in rows by position modulo taps, so that heads that share q and k can read the older rows while
// one of them stores the newest.
// Chunk: rows are taken eight at a time. Within a block the values u solve a unit lower triangular system whose matrix
// (step sizes, decays between the rows, k.k) does not depend on the state; a preparation kernel inverts it for every block
// and head in parallel, next to the convolved rows. One kernel then walks the blocks: sixteen products with the state, the
// 8 x 8 solutions, the outputs, the update. Decays appear only as products over a range of rows, never as quotients.
#include "hybrid_common.cuh"

namespace tz {

constexpr int kDeltaThreads = 256;
constexpr int kDeltaBlock = 8, kDeltaCols = 8, kDeltaStages = 4, kDeltaBlockThreads = 64;
constexpr int kDeltaCoef = 2 * kDeltaBlock * kDeltaBlock + 2 * kDeltaBlock;   // inverse * beta, read-out, decays from the start, to the end

__device__ __forceinline__ float softplus_f(float z) { return softplus_neg(-z); }
__device__ __forceinline__ float head_log_decay(const DeltaArgs& a, int head, float z) { return -expf(a.a_log[head]) * softplus_f(z + a.dt_bias[head]); }

// ---- decode --------------------------------------------------------------------------------------------------------------
// The older inputs' part of one channel's convolution at position pos; rows of the tail that no token of the sequence has
// written are zero.
__device__ __forceinline__ float conv_before(const float* w, int ch, int n_ch, int taps, const float* tail, int tail_ld, int pos) {
    float y = 0.0f;
    int slot = pos % taps;
    for (int j = 1; j < taps; ++j) {
        slot = slot == 0 ? taps - 1 : slot - 1;
        y = fmaf(w[(size_t)(taps - 1 - j) * n_ch + ch], tail[(size_t)slot * tail_ld], y);
    }
    return y;
}

// THREADS 256 or 512, whichever lets a thread hold its part of the state in kPre pieces for most sizes.
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS, 1024 / THREADS) delta_decode_kernel(const DeltaArgs a) {
    extern __shared__ float sm[];
    constexpr int kPre = 8;                              // float4 pieces of the state that are fetched ahead
    __shared__ float s_red[4][THREADS / 32];
    const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int ldv = (a.vdim + 3) & ~3, nc = ldv / 4;
    int nc2 = 1;
    while (nc2 < nc) nc2 *= 2;
    const int col = tid & (nc2 - 1), rg = tid / nc2, n_rg = THREADS / nc2;
    const bool live = col < nc;
    float4* S = reinterpret_cast<float4*>(a.state + (size_t)seq * a.state_seq_stride + (size_t)head * a.dim * ldv) + col;
    float4 pre[kPre];
#pragma unroll
    for (int i = 0; i < kPre; ++i) {
        const int r = rg + i * n_rg;
        if (live && r < a.dim) pre[i] = S[(size_t)r * nc];
    }
    float* s_q = sm;                                     // [dim]
    float* s_k = s_q + a.dim;                            // [dim]
    float* s_u = sm + ((2 * a.dim + 3) & ~3);            // [ldv]
    float* s_a = s_u + ldv;                              // [n_rg][ldv]
    float* s_b = s_a + n_rg * ldv;
    const int group = a.heads / a.kv_heads, kvh = head / group;
    const int n_q = a.kv_heads * a.dim, n_v = a.heads * a.vdim, n_ch = 2 * n_q + n_v;
    // the position and the convolutions' older inputs were written a whole step ago, like the state
    const int pos = a.pos[seq], chq = kvh * a.dim + tid, chv = head * a.vdim + tid;
    float* tail = a.tail + (size_t)seq * a.tail_seq_stride;
    float* newest = tail + (size_t)(pos % a.taps) * n_ch;
    const bool has_q = tid < a.dim, has_v = tid < a.vdim;  // head sizes are at most one thread per element
    const size_t last = a.taps - 1;
    float q = 0.0f, k = 0.0f, v = 0.0f, wq = 0.0f, wk = 0.0f, wv = 0.0f, gain = 0.0f, uq = 0.0f, uk = 0.0f, uv = 0.0f, gate = 0.0f;
    if (has_q) {
        wq = a.conv_q[last * n_q + chq];
        wk = a.conv_k[last * n_q + chq];
        q = conv_before(a.conv_q, chq, n_q, a.taps, tail + chq, n_ch, pos);
        k = conv_before(a.conv_k, chq, n_q, a.taps, tail + n_q + chq, n_ch, pos);
    }
    if (has_v) {
        wv = a.conv_v[last * n_v + chv];
        gain = a.norm[tid];
        v = conv_before(a.conv_v, chv, n_v, a.taps, tail + 2 * n_q + chv, n_ch, pos);
    }
    pdl_wait();
    pdl_launch_dependents();
    const size_t row = (size_t)seq * a.ld;
    if (has_q) {
        uq = a.q[row + chq];
        uk = a.k[row + chq];
    }
    if (has_v) {
        uv = a.v[row + chv];
        gate = a.g[row + chv];
    }
    const float g = expf(head_log_decay(a, head, a.a[row + head])), beta = sigmoid_f(a.b[row + head]);
    if (has_q) {
        q = silu_f(fmaf(wq, uq, q));
        k = silu_f(fmaf(wk, uk, k));
        if (head % group == 0) {
            newest[chq] = uq;
            newest[n_q + chq] = uk;
        }
    }
    if (has_v) {
        v = silu_f(fmaf(wv, uv, v));
        newest[2 * n_q + chv] = uv;
    }
    const float qq = warp_sum(q * q), kk = warp_sum(k * k), qk = warp_sum(q * k);
    if (lane == 0) { s_red[0][warp] = qq; s_red[1][warp] = kk; s_red[2][warp] = qk; }
    __syncthreads();
    float sums[3];
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        sums[i] = 0.0f;
#pragma unroll
        for (int w = 0; w < THREADS / 32; ++w) sums[i] += s_red[i][w];
    }
    const float iq = a.q_scale / sqrtf(sums[0] + a.unit_eps), ik = 1.0f / sqrtf(sums[1] + a.unit_eps), kq = sums[2] * iq * ik;
    if (has_q) { s_q[tid] = q * iq; s_k[tid] = k * ik; }
    __syncthreads();
    if (live) {
        float pa[4] = {}, pb[4] = {};
        auto step = [&](int r, const float4& s4) {
            const float kr = s_k[r], qr = s_q[r], s[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                pa[j] = fmaf(kr, s[j], pa[j]);
                pb[j] = fmaf(qr, s[j], pb[j]);
            }
        };
#pragma unroll
        for (int i = 0; i < kPre; ++i)
            if (rg + i * n_rg < a.dim) step(rg + i * n_rg, pre[i]);
        for (int r = rg + kPre * n_rg; r < a.dim; r += n_rg) step(r, S[(size_t)r * nc]);
        *reinterpret_cast<float4*>(s_a + rg * ldv + col * 4) = make_float4(pa[0], pa[1], pa[2], pa[3]);
        *reinterpret_cast<float4*>(s_b + rg * ldv + col * 4) = make_float4(pb[0], pb[1], pb[2], pb[3]);
    }
    __syncthreads();
    float o = 0.0f;
    if (tid < ldv) {
        float sa = 0.0f, sb = 0.0f;
        for (int r = 0; r < n_rg; ++r) {
            sa += s_a[r * ldv + tid];
            sb += s_b[r * ldv + tid];
        }
        const float u = has_v ? beta * (v - g * sa) : 0.0f;
        s_u[tid] = u;
        if (has_v) o = fmaf(g, sb, kq * u);
    }
    const float oo = warp_sum(o * o);
    if (lane == 0) s_red[3][warp] = oo;
    __syncthreads();
    if (has_v) {
        float t = 0.0f;
#pragma unroll
        for (int w = 0; w < THREADS / 32; ++w) t += s_red[3][w];
        const float y = o * (1.0f / sqrtf(t / (float)a.vdim + a.eps)) * gain;
        reinterpret_cast<T*>(a.out)[(size_t)seq * a.ld_out + chv] = from_f<T>(y * silu_f(gate));
    }
    if (live) {
        const float4 u = *reinterpret_cast<const float4*>(s_u + col * 4);
        auto update = [&](int r, const float4& s) {
            const float kr = s_k[r];
            S[(size_t)r * nc] = make_float4(fmaf(g, s.x, kr * u.x), fmaf(g, s.y, kr * u.y), fmaf(g, s.z, kr * u.z), fmaf(g, s.w, kr * u.w));
        };
#pragma unroll
        for (int i = 0; i < kPre; ++i)
            if (rg + i * n_rg < a.dim) update(rg + i * n_rg, pre[i]);
        for (int r = rg + kPre * n_rg; r < a.dim; r += n_rg) update(r, S[(size_t)r * nc]);
    }
}

// ---- chunk ---------------------------------------------------------------------------------------------------------------
struct DeltaLaunch {
    DeltaArgs a;
    int dp, vp;                  // padded head sizes: delta_padded(), a multiple of kDeltaCols
    float *kq, *v, *coef, *o;    // [block][kv_head][8 k, 8 q][dp], [block][head][8][vp], [block][head][kDeltaCoef], [M][heads*vdim]
};

// One CTA per (block of rows, kv head). Convolutions: a thread per channel, the block's rows and the taps - 1 inputs before
// them in registers; then a warp per row. NT: taps rounded up to 4 or 16.
template <int NT>
__global__ void __launch_bounds__(kDeltaThreads) delta_prepare_kernel(const DeltaLaunch L) {
    extern __shared__ float sm[];
    __shared__ float s_kk[8][9], s_qk[8][9], s_sys[8][64], s_gl[8][8], s_beta[8][8];
    const DeltaArgs& a = L.a;
    const int b = blockIdx.x, kvh = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, dp = L.dp;
    const int t0 = b * kDeltaBlock, group = a.heads / a.kv_heads, taps = a.taps;
    const int n_q = a.kv_heads * a.dim, n_v = a.heads * a.vdim, n_ch = 2 * n_q + n_v;
    float* s_k = sm;                                     // [8][dp]
    float* s_q = sm + 8 * dp;
    for (int i = tid; i < 2 * dp + group * L.vp; i += kDeltaThreads) {
        // channel `ch` of `nch` with its input at src, its place among the tail's channels and its destination rows
        const float *src, *w;
        float* dst;
        int ch, nch, first, ld;
        bool ok;
        if (i < 2 * dp) {
            const int d = i < dp ? i : i - dp;
            ok = d < a.dim; ch = kvh * a.dim + d; nch = n_q; ld = dp;
            src = i < dp ? a.q : a.k; w = i < dp ? a.conv_q : a.conv_k; first = i < dp ? 0 : n_q;
            dst = (i < dp ? s_q : s_k) + d;
        } else {
            const int x = i - 2 * dp, h = kvh * group + x / L.vp, d = x % L.vp;
            ok = d < a.vdim; ch = h * a.vdim + d; nch = n_v; ld = L.vp;
            src = a.v; w = a.conv_v; first = 2 * n_q;
            dst = L.v + ((size_t)b * a.heads + h) * 8 * L.vp + d;
        }
        float wt[NT], u[NT + 7];                         // u[NT - 1 + r] is row t0 + r, wt[NT - 1] belongs to the row itself
#pragma unroll
        for (int j = 0; j < NT; ++j) wt[j] = ok && j >= NT - taps ? w[(size_t)(j - NT + taps) * nch + ch] : 0.0f;
#pragma unroll
        for (int j = 0; j < NT + 7; ++j) {
            const int r = t0 + j - (NT - 1), p = a.pos0 + r;
            u[j] = 0.0f;
            if (ok && j >= NT - taps && r < a.M) {
                if (r >= 0) u[j] = src[(size_t)r * a.ld + ch];
                else if (p >= 0) u[j] = a.tail[(size_t)(p % taps) * n_ch + first + ch];
            }
        }
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            float y = 0.0f;
#pragma unroll
            for (int j = 0; j < NT; ++j) y = fmaf(wt[j], u[j + r], y);
            dst[r * ld] = t0 + r < a.M ? silu_f(y) : 0.0f;
        }
    }
    __syncthreads();
    float* out = L.kq + ((size_t)b * a.kv_heads + kvh) * 16 * dp;
    {
        float qq = 0.0f, kk = 0.0f;
        for (int d = lane; d < dp; d += 32) {
            qq = fmaf(s_q[warp * dp + d], s_q[warp * dp + d], qq);
            kk = fmaf(s_k[warp * dp + d], s_k[warp * dp + d], kk);
        }
        const float iq = a.q_scale / sqrtf(warp_sum(qq) + a.unit_eps), ik = 1.0f / sqrtf(warp_sum(kk) + a.unit_eps);
        for (int d = lane; d < dp; d += 32) {
            const float q = s_q[warp * dp + d] * iq, k = s_k[warp * dp + d] * ik;
            s_q[warp * dp + d] = q;
            s_k[warp * dp + d] = k;
            out[warp * dp + d] = k;
            out[(8 + warp) * dp + d] = q;
        }
    }
    __syncthreads();
    {                                                    // row `warp` against all rows
        float kkj[8] = {}, qkj[8] = {};
        for (int d = lane; d < dp; d += 32) {
            const float k = s_k[warp * dp + d], q = s_q[warp * dp + d];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float kj = s_k[j * dp + d];
                kkj[j] = fmaf(k, kj, kkj[j]);
                qkj[j] = fmaf(q, kj, qkj[j]);
            }
        }
        int j;
        const float kk = group_sums<8, 32>(kkj, lane, j), qk = group_sums<8, 32>(qkj, lane, j);
        if ((lane & 3) == 0) { s_kk[warp][j] = kk; s_qk[warp][j] = qk; }
    }
    __syncthreads();
    for (int hh = warp; hh < group; hh += 8) {
        const int h = kvh * group + hh;
        float* c = L.coef + ((size_t)b * a.heads + h) * kDeltaCoef;
        if (lane < 8) {
            const int r = b * kDeltaBlock + lane;        // rows past the end change nothing
            s_gl[warp][lane] = r < a.M ? head_log_decay(a, h, a.a[(size_t)r * a.ld + h]) : 0.0f;
            s_beta[warp][lane] = r < a.M ? sigmoid_f(a.b[(size_t)r * a.ld + h]) : 0.0f;
        }
        __syncwarp();
        for (int e = lane; e < 64; e += 32) {
            const int i = e >> 3, j = e & 7;
            float s = 0.0f;
            for (int m = j + 1; m <= i; ++m) s += s_gl[warp][m];
            const float d = expf(s);
            s_sys[warp][e] = j < i ? s_beta[warp][i] * d * s_kk[i][j] : 0.0f;
            c[64 + e] = j <= i ? d * s_qk[i][j] : 0.0f;
        }
        __syncwarp();
        if (lane < 8) {                                  // column `lane` of the inverse of (1 + system), times beta
            float x[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                float y = i == lane ? 1.0f : 0.0f;
#pragma unroll
                for (int j = 0; j < i; ++j) y = fmaf(-s_sys[warp][i * 8 + j], x[j], y);
                x[i] = y;
                c[i * 8 + lane] = y * s_beta[warp][lane];
            }
            float from = 0.0f, to = 0.0f;
            for (int m = 0; m <= lane; ++m) from += s_gl[warp][m];
            for (int m = lane + 1; m < 8; ++m) to += s_gl[warp][m];
            c[128 + lane] = expf(from);
            c[136 + lane] = expf(to);
        }
        __syncwarp();
    }
}

// Eight value columns of one head, four per warp. Half a warp shares a pair of columns, lane l of it holding the state's rows
// 4 (l + 16 j) .. + 3 of both; once the products are summed, eight lanes stand for the block's eight rows of one column.
template <int KJ>
__global__ void __launch_bounds__(kDeltaBlockThreads) delta_block_kernel(const DeltaLaunch L) {
    constexpr int DP = 64 * KJ, V = 16 * DP, C = V + 8 * kDeltaCols, FLOATS = C + kDeltaCoef;
    extern __shared__ __align__(16) float smem[];
    const DeltaArgs& a = L.a;
    const int head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, l = lane & 15, r = lane & 7;
    const int cl = (tid >> 5) * 4 + (lane >> 3), c = blockIdx.x * kDeltaCols + cl;              // column whose row r this lane finishes
    const int cs = blockIdx.x * kDeltaCols + (tid >> 5) * 4 + (lane >> 4) * 2;                  // first column of its part of the state
    const int group = a.heads / a.kv_heads, kvh = head / group, ldv = (a.vdim + 3) & ~3, nv = a.heads * a.vdim;
    const int n_blocks = (a.M + kDeltaBlock - 1) / kDeltaBlock;
    auto stage = [&](int b) {
        if (b < n_blocks) {
            float* dst = smem + (b % kDeltaStages) * FLOATS;
            const float* kq = L.kq + ((size_t)b * a.kv_heads + kvh) * 16 * DP;
#pragma unroll
            for (int i = 0; i < 4 * DP / kDeltaBlockThreads; ++i) cp16(dst + 4 * (tid + i * kDeltaBlockThreads), kq + 4 * (tid + i * kDeltaBlockThreads));
            if (tid < 16) cp16(dst + V + 4 * tid, L.v + (((size_t)b * a.heads + head) * 8 + tid / 2) * L.vp + blockIdx.x * kDeltaCols + (tid & 1) * 4);
            else if (tid < 16 + kDeltaCoef / 4) cp16(dst + C + 4 * (tid - 16), L.coef + ((size_t)b * a.heads + head) * kDeltaCoef + 4 * (tid - 16));
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int b = 0; b + 1 < kDeltaStages; ++b) stage(b);
    float s[2][KJ * 4];
    auto place = [&](int x, int j) { return ((size_t)head * a.dim + 4 * (l + 16 * (j >> 2)) + (j & 3)) * ldv + cs + x; };
    auto exists = [&](int x, int j) { return cs + x < a.vdim && 4 * (l + 16 * (j >> 2)) + (j & 3) < a.dim; };
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int j = 0; j < KJ * 4; ++j) s[x][j] = exists(x, j) ? a.state[place(x, j)] : 0.0f;
    for (int b = 0; b < n_blocks; ++b) {
        asm volatile("cp.async.wait_group %0;" ::"n"(kDeltaStages - 2) : "memory");
        __syncthreads();                                 // the block is here, and the stage before it is free
        stage(b + kDeltaStages - 1);
        const float* buf = smem + (b % kDeltaStages) * FLOATS;
        const float *sk = buf + 4 * l, *sq = sk + 8 * DP, *co = buf + C;
        float pa[16], pb[16];                            // [column][row]
        float4 kr[KJ > 2 ? 1 : 8][KJ];                   // the block's keys, for the update, where registers allow it
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            float ka[2] = {}, qb[2] = {};
#pragma unroll
            for (int j = 0; j < KJ; ++j) {
                const float4 k4 = *reinterpret_cast<const float4*>(sk + t * DP + 64 * j), q4 = *reinterpret_cast<const float4*>(sq + t * DP + 64 * j);
                if (KJ <= 2) kr[KJ > 2 ? 0 : t][j] = k4;
                const float kf[4] = {k4.x, k4.y, k4.z, k4.w}, qf[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        ka[x] = fmaf(kf[i], s[x][4 * j + i], ka[x]);
                        qb[x] = fmaf(qf[i], s[x][4 * j + i], qb[x]);
                    }
            }
            pa[t] = ka[0]; pa[8 + t] = ka[1];
            pb[t] = qb[0]; pb[8 + t] = qb[1];
            if (KJ > 2) asm volatile("" ::: "memory");   // otherwise the loads of all rows are moved ahead, and spilled
        }
        int which;                                       // = l: column l / 8 of the pair, row l % 8
        const float at = group_sums<16, 16>(pa, lane, which), bt = group_sums<16, 16>(pb, lane, which);
        const float from = co[128 + r], x = buf[V + r * kDeltaCols + cl] - from * at;
        const float4 i0 = *reinterpret_cast<const float4*>(co + r * 8), i1 = *reinterpret_cast<const float4*>(co + r * 8 + 4);
        const float4 p0 = *reinterpret_cast<const float4*>(co + 64 + r * 8), p1 = *reinterpret_cast<const float4*>(co + 64 + r * 8 + 4);
        const float inv[8] = {i0.x, i0.y, i0.z, i0.w, i1.x, i1.y, i1.z, i1.w}, p[8] = {p0.x, p0.y, p0.z, p0.w, p1.x, p1.y, p1.z, p1.w};
        float u[2] = {}, o[2] = {from * bt, 0.0f};
#pragma unroll
        for (int t = 0; t < 8; ++t) u[t & 1] = fmaf(inv[t], __shfl_sync(0xffffffffu, x, t, 8), u[t & 1]);
        const float ur = u[0] + u[1], wr = ur * co[136 + r], decay = co[128 + 7];
#pragma unroll
        for (int y = 0; y < 2; ++y)
#pragma unroll
            for (int j = 0; j < KJ * 4; ++j) s[y][j] *= decay;
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            o[t & 1] = fmaf(p[t], __shfl_sync(0xffffffffu, ur, t, 8), o[t & 1]);
            const float w0 = __shfl_sync(0xffffffffu, wr, t, 16), w1 = __shfl_sync(0xffffffffu, wr, 8 + t, 16);
            if (KJ > 2) asm volatile("" ::: "memory");
#pragma unroll
            for (int j = 0; j < KJ; ++j) {
                const float4 k4 = KJ <= 2 ? kr[KJ > 2 ? 0 : t][j] : *reinterpret_cast<const float4*>(sk + t * DP + 64 * j);
                const float kf[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    s[0][4 * j + i] = fmaf(kf[i], w0, s[0][4 * j + i]);
                    s[1][4 * j + i] = fmaf(kf[i], w1, s[1][4 * j + i]);
                }
            }
        }
        const int row = b * kDeltaBlock + r;
        if (c < a.vdim && row < a.M) L.o[(size_t)row * nv + head * a.vdim + c] = o[0] + o[1];
    }
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int j = 0; j < KJ * 4; ++j)
            if (exists(x, j)) a.state[place(x, j)] = s[x][j];
    // the convolutions' last inputs; the preparation kernel has read the older ones
    if (blockIdx.x == 0) {
        const int n_q = a.kv_heads * a.dim, n_ch = 2 * n_q + nv;
        for (int t = max(0, a.M - a.taps); t < a.M; ++t) {
            float* to = a.tail + (size_t)((a.pos0 + t) % a.taps) * n_ch;
            const size_t row = (size_t)t * a.ld;
            if (head % group == 0)
                for (int d = tid; d < a.dim; d += kDeltaBlockThreads) {
                    to[kvh * a.dim + d] = a.q[row + kvh * a.dim + d];
                    to[n_q + kvh * a.dim + d] = a.k[row + kvh * a.dim + d];
                }
            for (int d = tid; d < a.vdim; d += kDeltaBlockThreads) to[2 * n_q + head * a.vdim + d] = a.v[row + head * a.vdim + d];
        }
    }
}

static int delta_padded(int dim) { return dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

static size_t delta_work_floats(int M, int heads, int kv_heads, int dp, int vp, int vdim, DeltaLaunch* L, float* work) {
    const size_t blocks = (M + kDeltaBlock - 1) / kDeltaBlock;
    const size_t kq = blocks * kv_heads * 16 * dp, v = blocks * heads * 8 * vp, coef = blocks * heads * kDeltaCoef;
    if (L) { L->kq = work; L->v = work + kq; L->coef = L->v + v; L->o = L->coef + coef; }
    return kq + v + coef + (size_t)M * heads * vdim;
}

int launch_delta(const DeltaArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    if (a.M <= 0) return 0;
    if (a.dim < 1 || a.dim > kMaxHeadDim || a.vdim < 1 || a.vdim > kMaxHeadDim || a.kv_heads < 1 || a.heads < 1 || a.heads % a.kv_heads ||
        a.taps < 1 || a.taps > kMaxTaps || !a.norm) return -1;
    if (a.decode) {
        const int ldv = round_up(a.vdim, 4);
        int nc2 = 1;
        while (nc2 < ldv / 4) nc2 *= 2;
        const int threads = (size_t)a.dim * nc2 <= 8 * 256 ? 256 : 512;
        const size_t smem = 4 * (size_t)(round_up(2 * a.dim, 4) + ldv + 2 * (threads / nc2) * ldv);
        *n_kernels += 1;
        auto go = [&](auto kernel) {
            if (int rc = allow_smem(kernel, smem)) return rc;
            return launch_kernel(kernel, dim3(a.heads, a.M), dim3(threads), smem, st, a.use_pdl, 1, a);
        };
        if (threads == 256) return a.f32 ? go(delta_decode_kernel<float, 256>) : go(delta_decode_kernel<bf16, 256>);
        return a.f32 ? go(delta_decode_kernel<float, 512>) : go(delta_decode_kernel<bf16, 512>);
    }
    DeltaLaunch L;
    L.a = a;
    L.dp = delta_padded(a.dim);
    L.vp = round_up(a.vdim, kDeltaCols);
    delta_work_floats(a.M, a.heads, a.kv_heads, L.dp, L.vp, a.vdim, &L, a.work);
    const dim3 blocks((a.M + kDeltaBlock - 1) / kDeltaBlock, a.kv_heads);
    if (a.taps <= 4) delta_prepare_kernel<4><<<blocks, kDeltaThreads, 64 * (size_t)L.dp, st>>>(L);
    else delta_prepare_kernel<kMaxTaps><<<blocks, kDeltaThreads, 64 * (size_t)L.dp, st>>>(L);
    const dim3 grid(L.vp / kDeltaCols, a.heads);
    auto go = [&](auto kernel) {
        const size_t smem = 4 * (size_t)kDeltaStages * (16 * L.dp + 8 * kDeltaCols + kDeltaCoef);
        if (int rc = allow_smem(kernel, smem)) return rc;
        kernel<<<grid, kDeltaBlockThreads, smem, st>>>(L);
        return (int)cudaGetLastError();
    };
    const int rc = L.dp == 64 ? go(delta_block_kernel<1>) : L.dp == 128 ? go(delta_block_kernel<2>) : go(delta_block_kernel<4>);
    if (rc) return rc;
    ScanArgs s;                                          // per head: o / rms(o) * norm * silu(g)
    s.M = a.M; s.heads = a.heads; s.vdim = a.vdim; s.o_rows = L.o; s.eps = a.eps; s.norm = a.norm;
    s.g = a.g; s.ld = a.ld; s.out = a.out; s.ld_out = a.ld_out; s.f32 = a.f32;
    *n_kernels += 2;
    return launch_scan_gate(s, st, n_kernels);
}

}  // namespace tz

extern "C" int tenzo_cuda_delta_rule(const tenzo_delta_args* args, void* stream) {
    if (!args) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::DeltaArgs a;
    static_cast<tenzo_delta_args&>(a) = *args;
    unsigned long long n = 0;
    return tz::launch_delta(a, static_cast<cudaStream_t>(stream), &n);
}

extern "C" size_t tenzo_cuda_delta_rule_work_floats(int M, int heads, int kv_heads, int dim, int vdim) {
    return tz::delta_work_floats(M, heads, kv_heads, tz::delta_padded(dim), tz::round_up(vdim, tz::kDeltaCols), vdim, nullptr, nullptr);
}
