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

constexpr int kWaThreads = 256, kWaWarps = 8, kWaSeg = 256;

// y = sum_j w[j] u_(t-taps+1+j) for one channel; `cur` is u_t, older values from the tail
__device__ __forceinline__ float conv_step(const float* w, int ch, int n_ch, int taps, const float* tail, int tail_ld, float cur) {
    float y = w[(size_t)(taps - 1) * n_ch + ch] * cur;
    for (int j = 0; j + 1 < taps; ++j) y = fmaf(w[(size_t)j * n_ch + ch], tail[(size_t)j * tail_ld], y);
    return y;
}

struct WaDecodeLaunch {
    WindowAttnArgs a;
    int ldd, ldv, group;         // padded row lengths, query heads per kv head
    int nvc;                     // value chunks of 8 per key, rounded up to a power of two
};

__device__ __forceinline__ void load_raw(const bf16* p, uint4 (&r)[1]) { r[0] = *reinterpret_cast<const uint4*>(p); }
__device__ __forceinline__ void load_raw(const float* p, uint4 (&r)[2]) {
    r[0] = reinterpret_cast<const uint4*>(p)[0];
    r[1] = reinterpret_cast<const uint4*>(p)[1];
}
__device__ __forceinline__ void raw_floats(const uint4 (&r)[1], float (&f)[8]) { unpack8(r[0], f); }
__device__ __forceinline__ void raw_floats(const uint4 (&r)[2], float (&f)[8]) {
    const uint32_t b[8] = {r[0].x, r[0].y, r[0].z, r[0].w, r[1].x, r[1].y, r[1].z, r[1].w};
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(b[i]);
}

// GQ query heads at a time (1, 2 or 4); LK lanes share a key, eight elements each. A lane's piece of the queries is in
// registers, and the rows of several keys are requested before the first is used.
template <typename T, int GQ, int LK>
__global__ void __launch_bounds__(kWaThreads, 2) window_decode_kernel(const WaDecodeLaunch L) {
    extern __shared__ float sm[];
    constexpr int RAW = sizeof(T) / 2;                   // 16-byte words of eight elements
    constexpr int KU = (GQ == 4 ? 4 : 8) / RAW, VU = KU, KW = 32 / LK;   // rows in flight per lane, keys per warp and trip
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
    pdl_wait();
    pdl_launch_dependents();
    const int pos = a.pos[seq];
    const int n_q = a.heads * a.dim, n_k = a.kv_heads * a.dim, n_v = a.kv_heads * a.vdim, n_ch = n_q + n_k + n_v;
    const float* tail = a.tail_in + (size_t)seq * a.tail_seq_stride;
    float* tail_out = a.tail_out + (size_t)seq * a.tail_seq_stride;
    const float *pq = a.q + (size_t)seq * a.ld, *pk = a.k + (size_t)seq * a.ld, *pv = a.v + (size_t)seq * a.ld;

    for (int i = tid; i < (group + 1) * ldd + ldv; i += kWaThreads) {
        // the convolved vectors as the storage type holds them; queries times the scale
        float y = 0.0f;
        if (i < group * ldd) {
            const int g = i / ldd, d = i - g * ldd, ch = (kvh * group + g) * a.dim + d;
            if (d < a.dim) y = to_f(from_f<T>(conv_step(a.conv_q, ch, n_q, a.taps, tail + ch, n_ch, pq[ch]))) * a.scale;
        } else if (i < (group + 1) * ldd) {
            const int d = i - group * ldd, ch = kvh * a.dim + d;
            if (d < a.dim) y = to_f(from_f<T>(conv_step(a.conv_k, ch, n_k, a.taps, tail + n_q + ch, n_ch, pk[ch])));
        } else {
            const int d = i - (group + 1) * ldd, ch = kvh * a.vdim + d;
            if (d < a.vdim) y = to_f(from_f<T>(conv_step(a.conv_v, ch, n_v, a.taps, tail + n_q + n_k + ch, n_ch, pv[ch])));
        }
        sm[i] = y;                                       // s_q, s_k and s_v lie back to back
    }
    __syncthreads();

    T* ring_k = reinterpret_cast<T*>(a.ring_k) + (size_t)seq * a.ring_k_stride + (size_t)kvh * a.ring * ldd;
    T* ring_v = reinterpret_cast<T*>(a.ring_v) + (size_t)seq * a.ring_v_stride + (size_t)kvh * a.ring * ldv;
    const int first = max(0, pos - a.window + 1), n_keys = pos - first;      // cached keys; the new one comes on top
    const int per = (n_keys + n_rank - 1) / n_rank, j0 = min(n_keys, rank * per), j1 = min(n_keys, j0 + per);
    const int slot0 = (first + j0) % a.ring;                                   // slot of this CTA's first key
    const int nvc = L.nvc, kpi = 32 / nvc, vc = lane & (nvc - 1), vk = lane / nvc;   // value chunk and key of this lane
    const int kc = (lane & (LK - 1)) * 8, kg = lane / LK;                       // key piece and key of this lane
    auto slot_of = [&](int j) { const int s = slot0 + j; return s >= a.ring ? s - a.ring : s; };

    for (int q0 = 0; q0 < group; q0 += GQ) {
        float qf[GQ][8];
#pragma unroll
        for (int g = 0; g < GQ; ++g)
#pragma unroll
            for (int i = 0; i < 8; ++i) qf[g][i] = q0 + g < group && kc < ldd ? s_q[(q0 + g) * ldd + kc + i] : 0.0f;
        int mine = 0;                                     // the query whose score this lane ends up with
        {
            float none[GQ] = {};
            group_sums<GQ, LK>(none, lane, mine);
        }
        const float slope = head_slope(a.slope_base, a.heads, kvh * group + q0 + mine);
        float m[GQ], l[GQ], acc[GQ][8];
#pragma unroll
        for (int g = 0; g < GQ; ++g) {
            m[g] = -INFINITY; l[g] = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[g][i] = 0.0f;
        }
        const int total = j1 - j0 + (rank == 0 ? 1 : 0), fresh = rank == 0 ? total - 1 : -1;   // rank 0 also takes the new token
        for (int sb = 0; sb < total; sb += kWaSeg) {
            const int ns = min(kWaSeg, total - sb);
            // scores. Every lane of a warp makes the same trips, so the exchanges are warp-wide.
            for (int b = warp * KW; b < ns; b += kWaWarps * KW * KU) {
                uint4 raw[KU][RAW];
#pragma unroll
                for (int x = 0; x < KU; ++x) {
                    const int kk = b + x * kWaWarps * KW + kg, j = sb + kk;
                    if (kk < ns && j != fresh && kc < ldd) load_raw(ring_k + (size_t)slot_of(j) * ldd + kc, raw[x]);
                }
#pragma unroll
                for (int x = 0; x < KU; ++x) {
                    const int kk = b + x * kWaWarps * KW + kg, j = sb + kk;
                    float s[GQ];
#pragma unroll
                    for (int g = 0; g < GQ; ++g) s[g] = 0.0f;
                    if (kk < ns && kc < ldd) {
                        float kf[8];
                        if (j == fresh) load8(s_k + kc, kf); else raw_floats(raw[x], kf);
#pragma unroll
                        for (int g = 0; g < GQ; ++g)
#pragma unroll
                            for (int i = 0; i < 8; ++i) s[g] = fmaf(qf[g][i], kf[i], s[g]);
                    }
                    int which;
                    const float t = group_sums<GQ, LK>(s, lane, which);
                    // distance to the new token, whose own is 0
                    if (kk < ns && (lane & (LK / GQ - 1)) == 0) s_p[which * kWaSeg + kk] = t - slope * (float)(j == fresh ? 0 : n_keys - j0 - j);
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
            if (vc * 8 < ldv)
                for (int b = warp * kpi + vk; b < ns; b += kWaWarps * kpi * VU) {
                    uint4 raw[VU][RAW];
#pragma unroll
                    for (int x = 0; x < VU; ++x) {
                        const int kk = b + x * kWaWarps * kpi, j = sb + kk;
                        if (kk < ns && j != fresh) load_raw(ring_v + (size_t)slot_of(j) * ldv + vc * 8, raw[x]);
                    }
#pragma unroll
                    for (int x = 0; x < VU; ++x) {
                        const int kk = b + x * kWaWarps * kpi, j = sb + kk;
                        if (kk >= ns) continue;
                        float vf[8];
                        if (j == fresh) load8(s_v + vc * 8, vf); else raw_floats(raw[x], vf);
#pragma unroll
                        for (int g = 0; g < GQ; ++g) {
                            const float w = q0 + g < group ? s_p[g * kWaSeg + kk] * f_new[g] : 0.0f;
#pragma unroll
                            for (int i = 0; i < 8; ++i) acc[g][i] = fmaf(w, vf[i], acc[g][i]);
                        }
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
        // every CTA of the cluster finishes a slice of the outputs
        T* out = reinterpret_cast<T*>(a.out) + (size_t)seq * a.ld_out;
        for (int i = rank * kWaThreads + tid; i < GQ * ldv; i += n_rank * kWaThreads) {
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

// Convolved rows in the storage type: queries to lin_q, keys and values behind the history in lin_k / lin_v. A thread owns
// one channel of kPrepRows rows, with the convolution's inputs in registers. NT: taps rounded up to 4 or 16.
constexpr int kPrepRows = 16, kPrepThreads = 128;

template <typename T, int NT>
__global__ void __launch_bounds__(kPrepThreads) window_prepare_kernel(const WaChunkLaunch L) {
    const WindowAttnArgs& a = L.a;
    const int n_q = a.heads * a.dim, n_k = a.kv_heads * a.dim, n_v = a.kv_heads * a.vdim, n_ch = n_q + n_k + n_v, nt = a.taps - 1;
    const int ch = blockIdx.x * kPrepThreads + threadIdx.x, t0 = blockIdx.y * kPrepRows, n_rows = min(kPrepRows, a.M - t0), total = L.hist + a.M;
    if (ch >= n_ch) return;
    const float *src, *w;
    T* dst;                                                  // row t at dst + t * step
    size_t step;
    int local, nch, d, size, ld;
    if (ch < n_q) {
        local = ch; nch = n_q; size = a.dim; ld = L.ldd; src = a.q; w = a.conv_q;
        dst = reinterpret_cast<T*>(a.lin_q) + (size_t)(local / size) * ld;
        step = (size_t)a.heads * ld;
    } else if (ch < n_q + n_k) {
        local = ch - n_q; nch = n_k; size = a.dim; ld = L.ldd; src = a.k; w = a.conv_k;
        dst = reinterpret_cast<T*>(a.lin_k) + ((size_t)(local / size) * total + L.hist) * ld;
        step = ld;
    } else {
        local = ch - n_q - n_k; nch = n_v; size = a.vdim; ld = L.ldv; src = a.v; w = a.conv_v;
        dst = reinterpret_cast<T*>(a.lin_v) + ((size_t)(local / size) * total + L.hist) * ld;
        step = ld;
    }
    d = local % size;
    dst += d;
    const int pad = d == size - 1 ? ld - size : 0;           // the last channel also zeroes the padding behind it
    auto input = [&](int t) { return t >= 0 ? src[(size_t)t * a.ld + local] : t >= -nt ? a.tail_in[(size_t)(nt + t) * n_ch + ch] : 0.0f; };
    float wt[NT], u[NT], in[kPrepRows];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        wt[j] = j >= NT - a.taps ? w[(size_t)(j - NT + a.taps) * nch + local] : 0.0f;
        u[j] = j > NT - a.taps ? input(t0 - NT + j) : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < kPrepRows; ++i) in[i] = i < n_rows ? input(t0 + i) : 0.0f;
#pragma unroll
    for (int i = 0; i < kPrepRows; ++i) {
        if (i >= n_rows) break;
#pragma unroll
        for (int j = 0; j + 1 < NT; ++j) u[j] = u[j + 1];
        u[NT - 1] = in[i];
        float y = 0.0f;
#pragma unroll
        for (int j = 0; j < NT; ++j) y = fmaf(wt[j], u[j], y);
        T* o = dst + (size_t)(t0 + i) * step;
        o[0] = from_f<T>(y);
        for (int k = 1; k <= pad; ++k) o[k] = from_f<T>(0.0f);
    }
    if (t0 + n_rows == a.M)
        for (int j = 0; j < nt; ++j) a.tail_out[(size_t)j * n_ch + ch] = input(a.M - nt + j);
}

// Rows between the ring and the linear layout, 16 bytes per thread: TO_RING = 0 brings the history in front of the new rows,
// TO_RING = 1 puts the last `rows` of them into the ring (a separate launch: the history is read first).
template <typename T, bool TO_RING>
__global__ void __launch_bounds__(256) window_ring_kernel(const WaChunkLaunch L, int rows) {
    const WindowAttnArgs& a = L.a;
    constexpr int E = 16 / sizeof(T);
    const int row = blockIdx.x, total = L.hist + a.M;
    const int lin = TO_RING ? total - rows + row : row, slot = (a.pos0 - L.hist + lin) % a.ring;
    const int kc = L.ldd / E, vc = L.ldv / E;
    for (int i = threadIdx.x; i < a.kv_heads * (kc + vc); i += 256) {
        const bool is_k = i < a.kv_heads * kc;
        const int n = is_k ? kc : vc, x = is_k ? i : i - a.kv_heads * kc, h = x / n, c = x - h * n, ld = n * E;
        T* l = reinterpret_cast<T*>(is_k ? a.lin_k : a.lin_v) + ((size_t)h * total + lin) * ld;
        T* r = reinterpret_cast<T*>(is_k ? a.ring_k : a.ring_v) + ((size_t)h * a.ring + slot) * ld;
        if (TO_RING) reinterpret_cast<uint4*>(r)[c] = reinterpret_cast<const uint4*>(l)[c];
        else reinterpret_cast<uint4*>(l)[c] = reinterpret_cast<const uint4*>(r)[c];
    }
}

template <typename T>
static int window_attention(const WindowAttnArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    const int ldd = round_up(a.dim, 8), ldv = round_up(a.vdim, 8), group = a.heads / a.kv_heads;
    if (a.decode) {
        WaDecodeLaunch L;
        L.a = a; L.ldd = ldd; L.ldv = ldv; L.group = group;
        L.nvc = 1;
        while (L.nvc * 8 < ldv) L.nvc *= 2;
        // slices of at least 64 keys, at most eight CTAs, more than one only while the grid is small
        int cl = 1;
        while (cl < 8 && a.ring > 128 * cl && (long long)cl * a.kv_heads * a.M < 4 * 148) cl *= 2;
        auto go = [&](auto kernel, int GQ) {
            const size_t smem = 4 * ((size_t)group * ldd + ldd + ldv + GQ * kWaSeg + (size_t)kWaWarps * GQ * ldv + 2 * GQ);
            if (smem > 220 * 1024) return -1;
            if (int rc = allow_smem(kernel, smem)) return rc;
            return launch_kernel(kernel, dim3(cl, a.kv_heads, a.M), dim3(kWaThreads), smem, st, a.use_pdl, cl, L);
        };
        *n_kernels += 1;
        auto heads_at_once = [&](auto one, auto two, auto four) { return group == 1 ? go(one, 1) : group == 2 ? go(two, 2) : go(four, 4); };
        if (ldd > 128) return heads_at_once(window_decode_kernel<T, 1, 32>, window_decode_kernel<T, 2, 32>, window_decode_kernel<T, 4, 32>);
        if (ldd > 64) return heads_at_once(window_decode_kernel<T, 1, 16>, window_decode_kernel<T, 2, 16>, window_decode_kernel<T, 4, 16>);
        return heads_at_once(window_decode_kernel<T, 1, 8>, window_decode_kernel<T, 2, 8>, window_decode_kernel<T, 4, 8>);
    }
    WaChunkLaunch L;
    L.a = a; L.ldd = ldd; L.ldv = ldv; L.group = group;
    L.hist = a.pos0 < a.window - 1 ? a.pos0 : a.window - 1;
    const dim3 grid((a.heads * a.dim + a.kv_heads * (a.dim + a.vdim) + kPrepThreads - 1) / kPrepThreads, (a.M + kPrepRows - 1) / kPrepRows);
    if (a.taps <= 4) window_prepare_kernel<T, 4><<<grid, kPrepThreads, 0, st>>>(L);
    else window_prepare_kernel<T, kMaxTaps><<<grid, kPrepThreads, 0, st>>>(L);
    if (L.hist > 0) window_ring_kernel<T, false><<<L.hist, 256, 0, st>>>(L, L.hist);
    const int rows = a.M < a.ring ? a.M : a.ring;
    window_ring_kernel<T, true><<<rows, 256, 0, st>>>(L, rows);
    *n_kernels += L.hist > 0 ? 4 : 3;
    LinearAttn n;
    n.q = a.lin_q;
    n.k = a.lin_k; n.k_row = ldd; n.k_head = (size_t)(L.hist + a.M) * ldd;
    n.v = a.lin_v; n.v_row = ldv; n.v_head = (size_t)(L.hist + a.M) * ldv;
    n.d1 = ldd; n.dv = ldv; n.vdim = a.vdim;
    n.heads = a.heads; n.group = group; n.M = a.M; n.hist = L.hist; n.window = a.window;
    n.scale = a.scale; n.slope_base = a.slope_base; n.sink = a.sink;
    n.out = a.out; n.ld_out = a.ld_out; n.out_head = a.vdim; n.f32 = a.f32;
    return launch_linear_attention(n, st);
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
