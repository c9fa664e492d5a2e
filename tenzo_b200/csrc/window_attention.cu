// Sliding-window attention over grouped heads with a short convolution on q, k, v, a linear distance bias and a sink term
// in the softmax denominator (WindowAttnArgs). Scores, weights and sums are fp32.
//
// Decode: a thread-block cluster per (kv head, sequence). Every CTA convolves the head's channels, takes a slice of the
// cached keys, and the partial softmaxes meet in the first CTA through distributed shared memory. The new token's key
// and value are used from registers / shared memory; the first CTA appends them to the ring and shifts the convolution
// tails once the whole cluster has read them.
// Chunk: a preparation kernel convolves all rows and lays the window's history and the new rows out back to back, the
// ring is brought up to date from that, and the attention proper runs over the linear layout.
#include <cooperative_groups.h>

#include "hybrid_common.cuh"

namespace cg = cooperative_groups;

namespace tz {

int launch_window_flash(const WindowAttnArgs& a, int hist, cudaStream_t st);     // window_attention_mma.cu: bf16, tensor cores
bool window_flash_applicable(const WindowAttnArgs& a);

constexpr int kWaThreads = 256, kWaWarps = 8, kWaSeg = 256;

__device__ __forceinline__ float head_slope(const WindowAttnArgs& a, int h) {
    return a.slope_base == 0.0f ? 0.0f : exp2f(-a.slope_base * (float)(h + 1) / (float)a.heads);
}

// y = sum_j w[j] u_(t-taps+1+j) for one channel; `cur` is u_t, older values from the tail
__device__ __forceinline__ float conv_step(const float* w, int ch, int n_ch, int taps, const float* tail, int tail_ld, float cur) {
    float y = w[(size_t)(taps - 1) * n_ch + ch] * cur;
    for (int j = 0; j + 1 < taps; ++j) y = fmaf(w[(size_t)j * n_ch + ch], tail[(size_t)j * tail_ld], y);
    return y;
}

struct WaDecodeLaunch {
    WindowAttnArgs a;
    int ldd, ldv, group;         // padded row lengths, query heads per kv head
    int nvc;                     // value chunks of 8 per lane group, rounded up to a power of two
};

// GQ query heads at a time.
template <typename T, int GQ>
__global__ void __launch_bounds__(kWaThreads) window_decode_kernel(const WaDecodeLaunch L) {
    extern __shared__ float sm[];
    const WindowAttnArgs& a = L.a;
    cg::cluster_group cluster = cg::this_cluster();
    const int rank = (int)cluster.block_rank(), n_rank = (int)cluster.num_blocks();
    const int kvh = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int ldd = L.ldd, ldv = L.ldv, group = L.group;
    float* s_q = sm;                                     // [group][ldd]
    float* s_k = s_q + group * ldd;                      // [ldd] the new key
    float* s_v = s_k + ldd;                              // [ldv]
    float* s_p = s_v + ldv;                              // [GQ][kWaSeg]
    float* s_acc = s_p + GQ * kWaSeg;                    // [kWaWarps][GQ][ldv] per-warp value sums; [0] holds the CTA's sum
    float* s_ml = s_acc + kWaWarps * GQ * ldv;           // [2][GQ] running maximum and denominator of this CTA
    float* s_red = s_ml + 2 * GQ;                        // [32]
    pdl_wait();
    pdl_launch_dependents();
    const int pos = a.pos[seq];
    const int n_q = a.heads * a.dim, n_k = a.kv_heads * a.dim, n_v = a.kv_heads * a.vdim, n_ch = n_q + n_k + n_v;
    const float* tail = a.tail_in + (size_t)seq * a.tail_seq_stride;
    float* tail_out = a.tail_out + (size_t)seq * a.tail_seq_stride;
    const float *pq = a.q + (size_t)seq * a.ld, *pk = a.k + (size_t)seq * a.ld, *pv = a.v + (size_t)seq * a.ld;

    for (int i = tid; i < group * ldd; i += kWaThreads) {
        const int g = i / ldd, d = i - g * ldd, ch = (kvh * group + g) * a.dim + d;
        // the query as the storage type holds it, times the scale
        s_q[i] = d < a.dim ? to_f(from_f<T>(conv_step(a.conv_q, ch, n_q, a.taps, tail + ch, n_ch, pq[ch]))) * a.scale : 0.0f;
    }
    for (int d = tid; d < ldd; d += kWaThreads) {
        const int ch = kvh * a.dim + d;
        s_k[d] = d < a.dim ? to_f(from_f<T>(conv_step(a.conv_k, ch, n_k, a.taps, tail + n_q + ch, n_ch, pk[ch]))) : 0.0f;
    }
    for (int d = tid; d < ldv; d += kWaThreads) {
        const int ch = kvh * a.vdim + d;
        s_v[d] = d < a.vdim ? to_f(from_f<T>(conv_step(a.conv_v, ch, n_v, a.taps, tail + n_q + n_k + ch, n_ch, pv[ch]))) : 0.0f;
    }
    __syncthreads();

    T* ring_k = reinterpret_cast<T*>(a.ring_k) + (size_t)seq * a.ring_k_stride + (size_t)kvh * a.ring * ldd;
    T* ring_v = reinterpret_cast<T*>(a.ring_v) + (size_t)seq * a.ring_v_stride + (size_t)kvh * a.ring * ldv;
    const int first = max(0, pos - a.window + 1), n_keys = pos - first;      // cached keys; the new one comes on top
    const int per = (n_keys + n_rank - 1) / n_rank, j0 = min(n_keys, rank * per), j1 = min(n_keys, j0 + per);
    const int nvc = L.nvc, kpi = 32 / nvc, vc = lane & (nvc - 1), vk = lane / nvc;   // value chunk and key of this lane

    for (int q0 = 0; q0 < group; q0 += GQ) {
        float m[GQ], l[GQ], acc[GQ][8];
#pragma unroll
        for (int g = 0; g < GQ; ++g) {
            m[g] = -INFINITY; l[g] = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[g][i] = 0.0f;
        }
        const bool has_new = rank == 0;
        const int total = j1 - j0 + (has_new ? 1 : 0);   // key index total-1 of rank 0 is the new token
        for (int sb = 0; sb < total; sb += kWaSeg) {
            const int ns = min(kWaSeg, total - sb);
            // scores: eight lanes per key, 16 bytes of it per lane and step
            for (int kk = warp * 4 + (lane >> 3); kk < ns; kk += kWaWarps * 4) {
                const int j = sb + kk;
                const bool fresh = has_new && j == total - 1;
                const int p = fresh ? pos : first + j0 + j;
                const T* krow = ring_k + (size_t)(p % a.ring) * ldd;
                float s[GQ];
#pragma unroll
                for (int g = 0; g < GQ; ++g) s[g] = 0.0f;
                for (int c = (lane & 7) * 8; c < ldd; c += 64) {
                    float kf[8];
                    if (fresh) load8(s_k + c, kf); else load8(krow + c, kf);
#pragma unroll
                    for (int g = 0; g < GQ; ++g)
                        if (q0 + g < group) {
                            float qf[8];
                            load8(s_q + (q0 + g) * ldd + c, qf);
#pragma unroll
                            for (int i = 0; i < 8; ++i) s[g] = fmaf(qf[i], kf[i], s[g]);
                        }
                }
                const unsigned mask = 0xffu << (lane & 24);       // the eight lanes of this key
#pragma unroll
                for (int g = 0; g < GQ; ++g) {
                    s[g] += __shfl_xor_sync(mask, s[g], 4);
                    s[g] += __shfl_xor_sync(mask, s[g], 2);
                    s[g] += __shfl_xor_sync(mask, s[g], 1);
                    if ((lane & 7) == 0 && q0 + g < group)
                        s_p[g * kWaSeg + kk] = s[g] - head_slope(a, kvh * group + q0 + g) * (float)(pos - p);
                }
            }
            __syncthreads();
            // softmax over the segment: warp g handles query g (GQ <= 8 = warps)
            if (warp < GQ && q0 + warp < group) {
                float mx = -INFINITY;
                for (int i = lane; i < ns; i += 32) mx = fmaxf(mx, s_p[warp * kWaSeg + i]);
                mx = warp_max(mx);
                float sum = 0.0f;
                for (int i = lane; i < ns; i += 32) {
                    const float e = expf(s_p[warp * kWaSeg + i] - mx);
                    s_p[warp * kWaSeg + i] = e;
                    sum += e;
                }
                sum = warp_sum(sum);
                if (lane == 0) { s_ml[warp] = mx; s_ml[GQ + warp] = sum; }
            }
            __syncthreads();
            float f_new[GQ];
#pragma unroll
            for (int g = 0; g < GQ; ++g) {
                f_new[g] = 0.0f;
                if (q0 + g >= group) continue;
                const float ms = s_ml[g], mn = fmaxf(m[g], ms), f_old = expf(m[g] - mn);      // expf(-inf) = 0
                f_new[g] = expf(ms - mn);
                l[g] = l[g] * f_old + s_ml[GQ + g] * f_new[g];
                m[g] = mn;
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[g][i] *= f_old;
            }
            for (int kk = warp * kpi + vk; kk < ns; kk += kWaWarps * kpi) {
                const int j = sb + kk;
                const bool fresh = has_new && j == total - 1;
                const int p = fresh ? pos : first + j0 + j;
                if (vc * 8 >= ldv) continue;
                float vf[8];
                if (fresh) load8(s_v + vc * 8, vf); else load8(ring_v + (size_t)(p % a.ring) * ldv + vc * 8, vf);
#pragma unroll
                for (int g = 0; g < GQ; ++g) {
                    if (q0 + g >= group) continue;
                    const float w = s_p[g * kWaSeg + kk] * f_new[g];
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[g][i] = fmaf(w, vf[i], acc[g][i]);
                }
            }
            __syncthreads();
        }
        // value sums: across the key groups of a warp, then across warps
#pragma unroll
        for (int g = 0; g < GQ; ++g)
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                for (int mm = nvc; mm < 32; mm <<= 1) acc[g][i] += __shfl_xor_sync(0xffffffffu, acc[g][i], mm);
                if (vk == 0 && vc * 8 < ldv) s_acc[((size_t)warp * GQ + g) * ldv + vc * 8 + i] = acc[g][i];
            }
        if (tid == 0) {
#pragma unroll
            for (int g = 0; g < GQ; ++g) { s_ml[g] = m[g]; s_ml[GQ + g] = l[g]; }
        }
        __syncthreads();
        for (int i = tid; i < GQ * ldv; i += kWaThreads) {
            float t = 0.0f;
#pragma unroll
            for (int w = 0; w < kWaWarps; ++w) t += s_acc[(size_t)w * GQ * ldv + i];
            s_acc[i] = t;
        }
        cluster.sync();
        if (rank == 0) {
            T* out = reinterpret_cast<T*>(a.out) + (size_t)seq * a.ld_out;
            for (int i = tid; i < GQ * ldv; i += kWaThreads) {
                const int g = i / ldv, d = i - g * ldv;
                if (q0 + g >= group || d >= a.vdim) continue;
                float mx = a.sink > 0.0f ? 0.0f : -1e30f;     // the sink is a score of 0
                for (int r = 0; r < n_rank; ++r) mx = fmaxf(mx, cluster.map_shared_rank(s_ml, r)[g]);
                float den = a.sink * expf(-mx), num = 0.0f;
                for (int r = 0; r < n_rank; ++r) {
                    const float* ml = cluster.map_shared_rank(s_ml, r);
                    const float f = expf(ml[g] - mx);
                    den = fmaf(ml[GQ + g], f, den);
                    num = fmaf(cluster.map_shared_rank(s_acc, r)[i], f, num);
                }
                out[(size_t)(kvh * group + q0 + g) * a.vdim + d] = from_f<T>(num / den);
            }
        }
        cluster.sync();                                       // partials are read; the buffers may be reused
    }
    if (rank == 0) {
        const int slot = pos % a.ring;
        for (int d = tid; d < a.dim; d += kWaThreads) ring_k[(size_t)slot * ldd + d] = from_f<T>(s_k[d]);
        for (int d = tid; d < a.vdim; d += kWaThreads) ring_v[(size_t)slot * ldv + d] = from_f<T>(s_v[d]);
        auto shift = [&](int ch, float cur) {
            for (int j = 0; j + 2 < a.taps; ++j) tail_out[(size_t)j * n_ch + ch] = tail[(size_t)(j + 1) * n_ch + ch];
            if (a.taps > 1) tail_out[(size_t)(a.taps - 2) * n_ch + ch] = cur;
        };
        for (int i = tid; i < group * a.dim; i += kWaThreads) shift(kvh * group * a.dim + i, pq[kvh * group * a.dim + i]);
        for (int d = tid; d < a.dim; d += kWaThreads) shift(n_q + kvh * a.dim + d, pk[kvh * a.dim + d]);
        for (int d = tid; d < a.vdim; d += kWaThreads) shift(n_q + n_k + kvh * a.vdim + d, pv[kvh * a.vdim + d]);
    }
}

// ---- chunk ---------------------------------------------------------------------------------------------------------------
struct WaChunkLaunch {
    WindowAttnArgs a;
    int ldd, ldv, group, hist;
};

// Rows 0..hist-1 of lin_k / lin_v come from the ring, the M new rows from the convolution; queries get the storage type.
// One CTA per row of the linear layout.
template <typename T>
__global__ void __launch_bounds__(256) window_prepare_kernel(const WaChunkLaunch L) {
    const WindowAttnArgs& a = L.a;
    const int row = blockIdx.x, ldd = L.ldd, ldv = L.ldv, total = L.hist + a.M;
    const int n_q = a.heads * a.dim, n_k = a.kv_heads * a.dim, n_v = a.kv_heads * a.vdim, n_ch = n_q + n_k + n_v;
    T *lin_q = reinterpret_cast<T*>(a.lin_q), *lin_k = reinterpret_cast<T*>(a.lin_k), *lin_v = reinterpret_cast<T*>(a.lin_v);
    if (row < L.hist) {
        const int slot = (a.pos0 - L.hist + row) % a.ring;
        for (int i = threadIdx.x; i < a.kv_heads * ldd; i += 256) {
            const int h = i / ldd, d = i - h * ldd;
            lin_k[((size_t)h * total + row) * ldd + d] = reinterpret_cast<const T*>(a.ring_k)[((size_t)h * a.ring + slot) * ldd + d];
        }
        for (int i = threadIdx.x; i < a.kv_heads * ldv; i += 256) {
            const int h = i / ldv, d = i - h * ldv;
            lin_v[((size_t)h * total + row) * ldv + d] = reinterpret_cast<const T*>(a.ring_v)[((size_t)h * a.ring + slot) * ldv + d];
        }
        return;
    }
    const int t = row - L.hist, nt = a.taps - 1;
    auto conv = [&](const float* src, const float* w, int nch, int ch, int tail_ch) {
        float y = 0.0f;
        for (int j = 0; j < a.taps; ++j) {
            const int u = t - nt + j;
            const float v = u >= 0 ? src[(size_t)u * a.ld + ch] : a.tail_in[(size_t)(nt + u) * n_ch + tail_ch];
            y = fmaf(w[(size_t)j * nch + ch], v, y);
        }
        return y;
    };
    for (int i = threadIdx.x; i < a.heads * ldd; i += 256) {
        const int h = i / ldd, d = i - h * ldd, ch = h * a.dim + d;
        lin_q[((size_t)t * a.heads + h) * ldd + d] = from_f<T>(d < a.dim ? conv(a.q, a.conv_q, n_q, ch, ch) : 0.0f);
    }
    for (int i = threadIdx.x; i < a.kv_heads * ldd; i += 256) {
        const int h = i / ldd, d = i - h * ldd, ch = h * a.dim + d;
        lin_k[((size_t)h * total + row) * ldd + d] = from_f<T>(d < a.dim ? conv(a.k, a.conv_k, n_k, ch, n_q + ch) : 0.0f);
    }
    for (int i = threadIdx.x; i < a.kv_heads * ldv; i += 256) {
        const int h = i / ldv, d = i - h * ldv, ch = h * a.vdim + d;
        lin_v[((size_t)h * total + row) * ldv + d] = from_f<T>(d < a.vdim ? conv(a.v, a.conv_v, n_v, ch, n_q + n_k + ch) : 0.0f);
    }
    if (t == a.M - 1)
        for (int j = 0; j < nt; ++j) {
            const int u = a.M - nt + j;
            for (int ch = threadIdx.x; ch < n_ch; ch += 256) {
                float v;
                if (u < 0) v = a.tail_in[(size_t)(nt + u) * n_ch + ch];
                else if (ch < n_q) v = a.q[(size_t)u * a.ld + ch];
                else if (ch < n_q + n_k) v = a.k[(size_t)u * a.ld + ch - n_q];
                else v = a.v[(size_t)u * a.ld + ch - n_q - n_k];
                a.tail_out[(size_t)j * n_ch + ch] = v;
            }
        }
}

// The last min(M, ring) new rows go into the ring. One CTA per row.
template <typename T>
__global__ void __launch_bounds__(256) window_ring_kernel(const WaChunkLaunch L, int rows) {
    const WindowAttnArgs& a = L.a;
    const int t = a.M - rows + blockIdx.x, total = L.hist + a.M, slot = (a.pos0 + t) % a.ring, ldd = L.ldd, ldv = L.ldv;
    for (int i = threadIdx.x; i < a.kv_heads * ldd; i += 256) {
        const int h = i / ldd, d = i - h * ldd;
        reinterpret_cast<T*>(a.ring_k)[((size_t)h * a.ring + slot) * ldd + d] = reinterpret_cast<const T*>(a.lin_k)[((size_t)h * total + L.hist + t) * ldd + d];
    }
    for (int i = threadIdx.x; i < a.kv_heads * ldv; i += 256) {
        const int h = i / ldv, d = i - h * ldv;
        reinterpret_cast<T*>(a.ring_v)[((size_t)h * a.ring + slot) * ldv + d] = reinterpret_cast<const T*>(a.lin_v)[((size_t)h * total + L.hist + t) * ldv + d];
    }
}

// Plain FMA attention: a CTA takes eight consecutive queries of one head, a warp one of them; 32 keys at a time in shared
// memory, lanes over keys for the scores and over value columns for the sums.
constexpr int kWaQ = 8, kWaMaxCols = kMaxHeadDim / 32;

template <typename T>
__global__ void __launch_bounds__(kWaThreads) window_chunk_kernel(const WaChunkLaunch L) {
    extern __shared__ float sm[];
    const WindowAttnArgs& a = L.a;
    const int ldd = L.ldd, ldv = L.ldv, total = L.hist + a.M, h = blockIdx.y, kvh = h / L.group;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int kstride = ldd + 1;                            // odd: lanes hit different banks
    float* s_k = sm;                                        // [32][ldd + 1]
    float* s_v = s_k + 32 * kstride;                        // [32][ldv]
    float* s_q = s_v + 32 * ldv;                            // [kWaQ][ldd]
    const int t = blockIdx.x * kWaQ + warp, i = L.hist + t;  // linear index of this warp's query
    const bool live = t < a.M;
    for (int d = lane; d < ldd; d += 32)
        s_q[warp * ldd + d] = live ? to_f(reinterpret_cast<const T*>(a.lin_q)[((size_t)t * a.heads + h) * ldd + d]) * a.scale : 0.0f;
    const float slope = head_slope(a, h);
    float m = a.sink > 0.0f ? 0.0f : -1e30f, l = a.sink, acc[kWaMaxCols];   // the sink is a score of 0
#pragma unroll
    for (int c = 0; c < kWaMaxCols; ++c) acc[c] = 0.0f;
    const int i_last = L.hist + min(a.M, (int)(blockIdx.x + 1) * kWaQ) - 1;
    const int first = max(0, L.hist + (int)blockIdx.x * kWaQ - a.window + 1);
    for (int k0 = first; k0 <= i_last; k0 += 32) {
        __syncthreads();
        for (int e = threadIdx.x; e < 32 * ldd; e += kWaThreads) {
            const int r = e / ldd, d = e - r * ldd;
            s_k[r * kstride + d] = k0 + r < total ? to_f(reinterpret_cast<const T*>(a.lin_k)[((size_t)kvh * total + k0 + r) * ldd + d]) : 0.0f;
        }
        for (int e = threadIdx.x; e < 32 * ldv; e += kWaThreads) {
            const int r = e / ldv;
            s_v[e] = k0 + r < total ? to_f(reinterpret_cast<const T*>(a.lin_v)[((size_t)kvh * total + k0) * ldv + e]) : 0.0f;
        }
        __syncthreads();
        const int j = k0 + lane, dist = i - j;
        float s = 0.0f;
        for (int d = 0; d < ldd; ++d) s = fmaf(s_q[warp * ldd + d], s_k[lane * kstride + d], s);
        s = live && dist >= 0 && dist < a.window ? s - slope * (float)dist : -INFINITY;
        const float mn = fmaxf(m, warp_max(s)), f = expf(m - mn), p = expf(s - mn);
        l = l * f + warp_sum(p);
        m = mn;
#pragma unroll
        for (int c = 0; c < kWaMaxCols; ++c) acc[c] *= f;
        for (int r = 0; r < 32; ++r) {
            const float pr = __shfl_sync(0xffffffffu, p, r);
#pragma unroll
            for (int c = 0; c < kWaMaxCols; ++c)
                if (c * 32 + lane < ldv) acc[c] = fmaf(pr, s_v[r * ldv + c * 32 + lane], acc[c]);
        }
    }
    if (!live) return;
    T* out = reinterpret_cast<T*>(a.out) + (size_t)t * a.ld_out + (size_t)h * a.vdim;
#pragma unroll
    for (int c = 0; c < kWaMaxCols; ++c)
        if (c * 32 + lane < a.vdim) out[c * 32 + lane] = from_f<T>(acc[c] / l);
}

template <typename T>
static int window_attention(const WindowAttnArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    const int ldd = round_up(a.dim, 8), ldv = round_up(a.vdim, 8), group = a.heads / a.kv_heads;
    if (a.decode) {
        WaDecodeLaunch L;
        L.a = a; L.ldd = ldd; L.ldv = ldv; L.group = group;
        L.nvc = 1;
        while (L.nvc * 8 < ldv) L.nvc *= 2;
        // slices of about 256 keys, at most eight CTAs
        int cl = 1;
        while (cl < 8 && a.ring > 256 * cl) cl *= 2;
        auto go = [&](auto kernel, int GQ) {
            const size_t smem = 4 * ((size_t)group * ldd + ldd + ldv + GQ * kWaSeg + (size_t)kWaWarps * GQ * ldv + 2 * GQ + 32);
            if (smem > 220 * 1024) return -1;
            if (int rc = allow_smem(kernel, smem)) return rc;
            return launch_kernel(kernel, dim3(cl, a.kv_heads, a.M), dim3(kWaThreads), smem, st, a.use_pdl, cl, L);
        };
        *n_kernels += 1;
        if (group == 1) return go(window_decode_kernel<T, 1>, 1);
        if (group == 2) return go(window_decode_kernel<T, 2>, 2);
        if (group <= 4) return go(window_decode_kernel<T, 4>, 4);
        return go(window_decode_kernel<T, 8>, 8);
    }
    WaChunkLaunch L;
    L.a = a; L.ldd = ldd; L.ldv = ldv; L.group = group;
    L.hist = a.pos0 < a.window - 1 ? a.pos0 : a.window - 1;
    window_prepare_kernel<T><<<L.hist + a.M, 256, 0, st>>>(L);
    const int rows = a.M < a.ring ? a.M : a.ring;
    window_ring_kernel<T><<<rows, 256, 0, st>>>(L, rows);
    *n_kernels += 3;
    if (!a.f32 && window_flash_applicable(a)) return launch_window_flash(a, L.hist, st);
    const size_t smem = 4 * ((size_t)32 * (ldd + 1) + 32 * ldv + kWaQ * ldd);
    if (int rc = allow_smem(window_chunk_kernel<T>, smem)) return rc;
    window_chunk_kernel<T><<<dim3((a.M + kWaQ - 1) / kWaQ, a.heads), kWaThreads, smem, st>>>(L);
    return (int)cudaGetLastError();
}

int launch_window_attention(const WindowAttnArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    if (a.M <= 0) return 0;
    if (a.dim > kMaxHeadDim || a.vdim > kMaxHeadDim || a.taps < 1 || a.taps > kMaxTaps || a.window < 1 || a.ring < 1 || a.kv_heads < 1 ||
        a.heads % a.kv_heads) return -1;
    return a.f32 ? window_attention<float>(a, st, n_kernels) : window_attention<bf16>(a, st, n_kernels);
}

}  // namespace tz

extern "C" int tenzo_cuda_window_attention(const tenzo_window_attention_args* args, void* stream) {
    if (!args) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::WindowAttnArgs a;
    static_cast<tenzo_window_attention_args&>(a) = *args;
    unsigned long long n = 0;
    return tz::launch_window_attention(a, static_cast<cudaStream_t>(stream), &n);
}
