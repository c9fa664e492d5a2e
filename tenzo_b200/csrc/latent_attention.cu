// Sliding-window attention over a shared latent (LatentAttnArgs): the cache holds one normed latent and one rotated key part
// per token, every head makes its unrotated key and its value from the latent. Scores, weights and sums are fp32.
//
// Decode never expands the cache: a head's key matrix is moved to the query (q_h W_uk,h, latent_absorb_kernel), which then
// scores the latents themselves, the weighted sum of latents is the heads' common value, and the value matrix follows as
// a product with one segment per head. All heads of a sequence share every key, so a CTA takes 16 heads at once on
// mma.sync (bf16) or eight with FMA arithmetic (fp32), and a thread-block cluster splits the keys.
// Chunk: history and new rows side by side, keys and values of all heads in one product, then attention over linear rows.
// A layer that borrows another one's cache finds that layer's new rows already there, in both forms.
#include <cooperative_groups.h>

#include "hybrid_common.cuh"

namespace cg = cooperative_groups;

namespace tz {

constexpr int kLtThreads = 256, kLtTile = 64, kLtHeads = 16, kLtFmaHeads = 8, kLtFmaTile = 32, kLtAbsorbRows = 4;

struct LatentLaunch {
    LatentAttnArgs a;
    int dim8, rot8, vdim8, ld_c, hist;       // hist: rows of the ring in front of the new ones in lin_c / lin_r
};

// cos and sin of position * freq; the angle is reduced in 64 bits
__device__ __forceinline__ void rotation(double freq, int pos, float& c, float& s) {
    const double x = freq * (double)pos;
    sincosf((float)(x - 6.283185307179586 * rint(x * 0.15915494309189535)), &s, &c);
}

// One token's cache row from its projection: the normed latent and the rotated key part, padding zero. All threads of the CTA.
template <typename T>
__device__ __forceinline__ void latent_row(const LatentLaunch& L, const float* src, int pos, T* c, T* r, float* scratch) {
    const LatentAttnArgs& a = L.a;
    float q = 0.0f;
    for (int i = threadIdx.x; i < a.rank; i += kLtThreads) q = fmaf(src[i], src[i], q);
    q = block_sum(q, scratch);
    const float inv = 1.0f / sqrtf(q / (float)a.rank + a.eps);
    for (int i = threadIdx.x; i < L.ld_c; i += kLtThreads) c[i] = from_f<T>(i < a.rank ? src[i] * inv * a.norm[i] : 0.0f);
    const int half = a.rot / 2;
    for (int i = threadIdx.x; i < half; i += kLtThreads) {
        float cs, sn;
        rotation(a.freq[i], pos, cs, sn);
        const float u = src[a.rank + i], v = src[a.rank + half + i];
        r[i] = from_f<T>(u * cs - v * sn);
        r[half + i] = from_f<T>(v * cs + u * sn);
    }
    for (int i = a.rot + threadIdx.x; i < L.rot8; i += kLtThreads) r[i] = from_f<T>(0.0f);
}

// ---- decode --------------------------------------------------------------------------------------------------------------
// The new tokens' cache rows, sequences `first`, `first` + `step`, .. below `end`.
template <typename T>
__device__ __forceinline__ void append_rows(const LatentLaunch& L, int first, int end, int step, float* scratch) {
    const LatentAttnArgs& a = L.a;
    for (int m = first; m < end; m += step) {
        const int pos = a.pos[m];
        const size_t slot = pos % a.ring;
        latent_row<T>(L, a.dkv + (size_t)m * a.ld, pos, static_cast<T*>(a.ring_c) + (size_t)m * a.ring_c_stride + slot * L.ld_c,
                      static_cast<T*>(a.ring_r) + (size_t)m * a.ring_r_stride + slot * L.rot8, scratch);
    }
}

// 128 columns of the latent for one head and up to MR sequences: 16 threads over the columns, 16 slices of the head's rows.
// One more head index, when the layer owns its cache, appends the new tokens' rows to the rings.
template <typename T, int MR>
__global__ void __launch_bounds__(kLtThreads) latent_absorb_kernel(const LatentLaunch L) {
    extern __shared__ float sm[];
    const LatentAttnArgs& a = L.a;
    const int h = blockIdx.y, tid = threadIdx.x, cc = (tid & 15) * 8, ds = tid >> 4, c0 = blockIdx.x * 128 + cc;
    const int m0 = blockIdx.z * MR, nm = min(MR, a.M - m0);
    const bool product = h < a.heads, live = product && c0 < L.ld_c;
    const bf16* w = static_cast<const bf16*>(a.w_kv) + (size_t)(product ? h : 0) * L.dim8 * L.ld_c + c0;
    constexpr int kPre = 8;
    uint4 pre[kPre];
#pragma unroll
    for (int i = 0; i < kPre; ++i)
        if (live && ds + 16 * i < a.dim) pre[i] = ld_stream_u4(w + (size_t)(ds + 16 * i) * L.ld_c);
    pdl_wait();
    pdl_launch_dependents();
    if (!product) {
        append_rows<T>(L, m0 + blockIdx.x, m0 + nm, gridDim.x, sm);
        return;
    }
    float* s_q = sm;                                     // [MR][dim8]
    float* s_part = sm + MR * L.dim8;                    // [8][MR][128]
    for (int i = tid; i < MR * L.dim8; i += kLtThreads) {
        const int m = i / L.dim8, d = i - m * L.dim8;
        s_q[i] = m < nm && d < a.dim ? a.q[(size_t)(m0 + m) * a.ld + (size_t)h * (a.dim + a.rot) + d] : 0.0f;
    }
    __syncthreads();
    float acc[MR][8] = {};
    auto step = [&](const uint4& wv, int d) {
        float f[8];
        unpack8(wv, f);
#pragma unroll
        for (int m = 0; m < MR; ++m) {
            const float q = s_q[m * L.dim8 + d];
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[m][j] = fmaf(q, f[j], acc[m][j]);
        }
    };
    if (live) {
#pragma unroll
        for (int i = 0; i < kPre; ++i)
            if (ds + 16 * i < a.dim) step(pre[i], ds + 16 * i);
        for (int d = ds + 16 * kPre; d < a.dim; d += 16) step(ld_stream_u4(w + (size_t)d * L.ld_c), d);
    }
#pragma unroll
    for (int m = 0; m < MR; ++m) {                       // the two slices of a warp meet in its lower half
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[m][j] += __shfl_xor_sync(0xffffffffu, acc[m][j], 16);
        if ((ds & 1) == 0) {
            float4* p = reinterpret_cast<float4*>(s_part + ((ds >> 1) * MR + m) * 128 + cc);
            p[0] = make_float4(acc[m][0], acc[m][1], acc[m][2], acc[m][3]);
            p[1] = make_float4(acc[m][4], acc[m][5], acc[m][6], acc[m][7]);
        }
    }
    __syncthreads();
    for (int i = tid; i < nm * 128; i += kLtThreads) {
        const int m = i >> 7, c = i & 127;
        if (blockIdx.x * 128 + c >= L.ld_c) continue;
        float t = 0.0f;
#pragma unroll
        for (int s = 0; s < 8; ++s) t += s_part[(s * MR + m) * 128 + c];
        a.q_abs[((size_t)(m0 + m) * a.heads + h) * L.ld_c + blockIdx.x * 128 + c] = t;
    }
}

// The same for many sequences with bf16 arithmetic, on tensor cores: 64 sequences x 128 columns of one head per CTA, a warp
// 16 x 64 of them. The head's rows are in shared memory before the wait.
constexpr int kLaM = 64, kLaN = 128, kLaW = kLaN + 8, kLaMinRows = 12;

__global__ void __launch_bounds__(kLtThreads) latent_absorb_mma_kernel(const LatentLaunch L) {
    extern __shared__ __align__(16) unsigned char smem[];
    const LatentAttnArgs& a = L.a;
    const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, c0 = blockIdx.x * kLaN, m0 = blockIdx.z * kLaM, m_end = min(a.M, m0 + kLaM);
    const int dp = (a.dim + 15) & ~15, qs = dp + 8;
    bf16 *s_w = reinterpret_cast<bf16*>(smem), *s_q = s_w + dp * kLaW;       // [dp][136], [64][qs]
    if (h < a.heads) {
        const bf16* w = static_cast<const bf16*>(a.w_kv) + (size_t)h * L.dim8 * L.ld_c + c0;
        for (int i = tid; i < dp * (kLaN / 8); i += kLtThreads) {
            const int d = i / (kLaN / 8), c = (i - d * (kLaN / 8)) * 8;
            if (d < a.dim && c0 + c < L.ld_c) cp16(s_w + d * kLaW + c, w + (size_t)d * L.ld_c + c);
            else *reinterpret_cast<uint4*>(s_w + d * kLaW + c) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    pdl_wait();
    pdl_launch_dependents();
    if (h >= a.heads) {
        append_rows<bf16>(L, m0 + blockIdx.x + gridDim.x * (h - a.heads), m_end, gridDim.x * (gridDim.y - a.heads), reinterpret_cast<float*>(smem));
        return;
    }
    for (int m = warp; m < kLaM; m += kLtThreads / 32)
        for (int d = lane; d < dp; d += 32)
            s_q[m * qs + d] = __float2bfloat16_rn(m0 + m < m_end && d < a.dim ? a.q[(size_t)(m0 + m) * a.ld + (size_t)h * (a.dim + a.rot) + d] : 0.0f);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int rt = (warp & 3) * 16, ch = (warp >> 2) * 64, g = lane >> 2, t4 = lane & 3;
    const uint32_t aq = smem_addr(s_q) + 2 * ((rt + (lane & 15)) * qs + (lane >> 4) * 8);
    const uint32_t bw = smem_addr(s_w) + 2 * (((lane & 7) + ((lane >> 3) & 1) * 8) * kLaW + ch + (lane >> 4) * 8);
    float acc[8][4] = {};
    for (int k = 0; k < dp; k += 16) {
        uint32_t q[4];
        ldsm4(q, aq + 2 * k);
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            uint32_t b[4];
            ldsm4t(b, bw + 2 * (k * kLaW + n * 16));
            mma_bf16(acc[2 * n], q, b[0], b[1]);
            mma_bf16(acc[2 * n + 1], q, b[2], b[3]);
        }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int m = m0 + rt + g + e * 8, c = c0 + ch + n * 8 + t4 * 2;
            if (m < m_end && c < L.ld_c) *reinterpret_cast<float2*>(a.q_abs + ((size_t)m * a.heads + h) * L.ld_c + c) = make_float2(acc[n][2 * e], acc[n][2 * e + 1]);
        }
}

// element d of a head's query against a cache row: the absorbed part, then the rotated part, times the scale
__device__ __forceinline__ float latent_query(const LatentLaunch& L, int seq, int h, int d, int pos) {
    const LatentAttnArgs& a = L.a;
    if (h >= a.heads) return 0.0f;
    if (d < L.ld_c) return a.q_abs[((size_t)seq * a.heads + h) * L.ld_c + d] * a.scale;
    d -= L.ld_c;
    if (d >= a.rot) return 0.0f;
    const int half = a.rot / 2, i = d < half ? d : d - half;
    const float* q = a.q + (size_t)seq * a.ld + (size_t)h * (a.dim + a.rot) + a.dim;
    float cs, sn;
    rotation(a.freq[i], pos, cs, sn);
    const float u = q[i], v = q[half + i];
    return (d < half ? u * cs - v * sn : v * cs + u * sn) * a.scale;
}

// Partial sums of the cluster's CTAs, [heads of the CTA][ld_c] with maximum and denominator, into the sums of latents.
template <typename T>
__device__ __forceinline__ void latent_merge(const LatentLaunch& L, cg::cluster_group& cluster, int seq, int h0, int nh, float* s_acc, float* s_ml) {
    const LatentAttnArgs& a = L.a;
    const int rank = (int)cluster.block_rank(), n_rank = (int)cluster.num_blocks();
    cluster.sync();
    for (int i = rank * (int)blockDim.x + threadIdx.x; i < nh * L.ld_c; i += n_rank * (int)blockDim.x) {
        const int h = i / L.ld_c, d = i - h * L.ld_c;
        if (h0 + h >= a.heads) continue;
        float mx = -1e30f;
        for (int r = 0; r < n_rank; ++r) mx = fmaxf(mx, cluster.map_shared_rank(s_ml, r)[h]);
        float den = 0.0f, num = 0.0f;
        for (int r = 0; r < n_rank; ++r) {
            const float* ml = cluster.map_shared_rank(s_ml, r);
            const float f = expf(ml[h] - mx);
            den = fmaf(ml[nh + h], f, den);
            num = fmaf(cluster.map_shared_rank(s_acc, r)[i], f, num);
        }
        static_cast<T*>(a.lat)[((size_t)(h0 + h) * a.M + seq) * L.ld_c + d] = from_f<T>(num / den);
    }
    cluster.sync();                                       // nobody leaves while its sums are read
}

// FMA arithmetic: a warp per head, lanes over 32 keys for the scores and over the latent's columns for the sums.
template <typename T, int NC>
__global__ void __launch_bounds__(kLtThreads) latent_decode_kernel(const LatentLaunch L) {
    extern __shared__ float sm[];
    __shared__ float s_ml[2 * kLtFmaHeads];
    const LatentAttnArgs& a = L.a;
    cg::cluster_group cluster = cg::this_cluster();
    const int rank = (int)cluster.block_rank(), n_rank = (int)cluster.num_blocks();
    const int h0 = blockIdx.y * kLtFmaHeads, seq = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int ldk = L.ld_c + L.rot8, ks = ldk + 1;       // odd row length: lanes hit different banks
    float* s_q = sm;                                     // [heads][ldk]
    float* s_k = s_q + kLtFmaHeads * ldk;                // [keys][ks]; the sums at the end
    pdl_wait();
    pdl_launch_dependents();
    const int pos = a.pos[seq], n_keys = min(pos + 1, a.window), first = pos + 1 - n_keys;
    for (int i = tid; i < kLtFmaHeads * ldk; i += kLtThreads) s_q[i] = latent_query(L, seq, h0 + i / ldk, i % ldk, pos);
    const T* rc = static_cast<const T*>(a.ring_c) + (size_t)seq * a.ring_c_stride;
    const T* rr = static_cast<const T*>(a.ring_r) + (size_t)seq * a.ring_r_stride;
    const int per = (n_keys + n_rank - 1) / n_rank, j0 = min(n_keys, rank * per), j1 = min(n_keys, j0 + per);
    float m = -1e30f, l = 0.0f, acc[NC] = {};
    for (int t0 = j0; t0 < j1; t0 += kLtFmaTile) {
        __syncthreads();
        for (int i = tid; i < kLtFmaTile * ldk; i += kLtThreads) {
            const int r = i / ldk, d = i - r * ldk;
            const size_t slot = (first + t0 + r) % a.ring;
            s_k[r * ks + d] = t0 + r >= j1 ? 0.0f : to_f(d < L.ld_c ? rc[slot * L.ld_c + d] : rr[slot * L.rot8 + d - L.ld_c]);
        }
        __syncthreads();
        float s = 0.0f;
        for (int d = 0; d < ldk; ++d) s = fmaf(s_q[warp * ldk + d], s_k[lane * ks + d], s);
        if (t0 + lane >= j1) s = -INFINITY;
        const float mn = fmaxf(m, warp_max(s)), f = expf(m - mn), p = expf(s - mn);
        l = l * f + warp_sum(p);
        m = mn;
#pragma unroll
        for (int c = 0; c < NC; ++c) acc[c] *= f;
        for (int r = 0; r < kLtFmaTile; ++r) {
            const float pr = __shfl_sync(0xffffffffu, p, r);
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (c * 32 + lane < L.ld_c) acc[c] = fmaf(pr, s_k[r * ks + c * 32 + lane], acc[c]);
        }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < NC; ++c)
        if (c * 32 + lane < L.ld_c) s_k[warp * L.ld_c + c * 32 + lane] = acc[c];
    if (lane == 0) { s_ml[warp] = m; s_ml[kLtFmaHeads + warp] = l; }
    latent_merge<T>(L, cluster, seq, h0, kLtFmaHeads, s_k, s_ml);
}

// bf16 cache on tensor cores: tiles of 64 keys for 16 heads, 16 warps. Scores: a warp takes eight keys and half of the
// elements, whose query fragments stay in its registers; softmax: a warp per head; sums: 16-column blocks over the warps.
// The weights enter the second product as the sum of two bf16 values, so that rounding them costs nothing visible.
constexpr int kLmThreads = 512;
constexpr float kLog2e = 1.4426950408889634f;             // scores here are in powers of two

struct LatentSmem {
    int ks;                                              // elements of a padded row
    size_t k, s, p, bytes;
    __host__ __device__ LatentSmem(int ld_c, int rot8) {
        ks = ld_c + (rot8 + 31) / 32 * 32 + 8;
        k = 0;                                           // [2][64][ks] bf16, the queries [16][ks] at first in the second; the sums at the end
        s = k + (size_t)2 * kLtTile * ks * 2;            // [2 halves][16][68] fp32 scores
        p = s + (size_t)2 * kLtHeads * 68 * 4;           // [2: value, rest][16][72] bf16 weights
        bytes = p + (size_t)2 * kLtHeads * 72 * 2;
    }
};

// NP: 16-column blocks of the latent per warp; PH: 32-element steps per half.
template <int NP, int PH>
__global__ void __launch_bounds__(kLmThreads, 1) latent_decode_mma_kernel(const LatentLaunch L) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float s_f[kLtHeads], s_ml[2 * kLtHeads];
    const LatentAttnArgs& a = L.a;
    const LatentSmem o(L.ld_c, L.rot8);
    cg::cluster_group cluster = cg::this_cluster();
    const int rank = (int)cluster.block_rank(), n_rank = (int)cluster.num_blocks();
    const int h0 = blockIdx.y * kLtHeads, seq = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    const int ks = o.ks, ldk = ks - 8, n_step = ldk / 32;
    const int kg = warp & 7, half = warp >> 3, p0 = half ? PH : 0, n_p = min(PH, n_step - p0);      // this warp's keys and steps
    bf16 *s_k = reinterpret_cast<bf16*>(smem + o.k), *s_q = s_k + kLtTile * ks, *s_p = reinterpret_cast<bf16*>(smem + o.p);
    float* s_s = reinterpret_cast<float*>(smem + o.s);
    for (int i = tid; i < kLtTile; i += kLmThreads)      // padding behind the rotated part
        for (int x = 0; x < 2; ++x)
            for (int c = L.ld_c + L.rot8; c < ks; c += 8) *reinterpret_cast<uint4*>(s_k + (size_t)(x * kLtTile + i) * ks + c) = make_uint4(0, 0, 0, 0);
    pdl_wait();
    pdl_launch_dependents();
    const int pos = a.pos[seq], n_keys = min(pos + 1, a.window), first = pos + 1 - n_keys;
    const bf16* rc = static_cast<const bf16*>(a.ring_c) + (size_t)seq * a.ring_c_stride;
    const bf16* rr = static_cast<const bf16*>(a.ring_r) + (size_t)seq * a.ring_r_stride;
    const int per = (n_keys + n_rank - 1) / n_rank, j0 = min(n_keys, rank * per), j1 = min(n_keys, j0 + per);
    const int n_tiles = (j1 - j0 + kLtTile - 1) / kLtTile, slot0 = (first + j0) % a.ring;
    const uint32_t c_bytes = 2 * L.ld_c, r_bytes = 2 * L.rot8, sk = smem_addr(s_k);
    const char *rc8 = reinterpret_cast<const char*>(rc) + lane * 16, *rr8 = reinterpret_cast<const char*>(rr) + lane * 16;
    auto copy = [](uint32_t dst, const char* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); };
    auto fetch = [&](int tile) {                         // a warp takes whole rows; rows past the end repeat the last one
#pragma unroll
        for (int i = 0; i < kLtTile * 32 / kLmThreads; ++i) {
            const int r = warp + i * (kLmThreads / 32);
            int slot = slot0 + min(tile * kLtTile + r, j1 - j0 - 1);
            if (slot >= a.ring) slot -= a.ring;
            const uint32_t dst = sk + 2 * ((tile & 1) * kLtTile + r) * ks + lane * 16;
            const char* src = rc8 + (size_t)slot * c_bytes;
            for (uint32_t c = 0; c + lane * 16 < c_bytes; c += 512) copy(dst + c, src + c);
            if (lane * 16 < r_bytes) copy(dst + c_bytes, rr8 + (size_t)slot * r_bytes);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (n_tiles > 0) fetch(0);
    // the queries: absorbed part four elements at a time, rotated part a pair at a time, padding
    const float scale = a.scale * kLog2e;
    const int c4 = L.ld_c / 4, pairs = a.rot / 2, pad = ldk - L.ld_c - a.rot;
#pragma unroll 4
    for (int i = tid; i < kLtHeads * c4; i += kLmThreads) {
        const int h = i / c4, d = (i - h * c4) * 4;
        const float4 v = h0 + h < a.heads ? *reinterpret_cast<const float4*>(a.q_abs + ((size_t)seq * a.heads + h0 + h) * L.ld_c + d) : make_float4(0, 0, 0, 0);
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x * scale, v.y * scale), hi = __floats2bfloat162_rn(v.z * scale, v.w * scale);
        *reinterpret_cast<uint2*>(s_q + h * ks + d) = make_uint2(reinterpret_cast<const uint32_t&>(lo), reinterpret_cast<const uint32_t&>(hi));
    }
    for (int i = tid; i < kLtHeads * pairs; i += kLmThreads) {
        const int h = i / pairs, f = i - h * pairs;
        float u = 0.0f, v = 0.0f, cs, sn;
        if (h0 + h < a.heads) {
            const float* x = a.q + (size_t)seq * a.ld + (size_t)(h0 + h) * (a.dim + a.rot) + a.dim;
            u = x[f];
            v = x[pairs + f];
        }
        rotation(a.freq[f], pos, cs, sn);
        s_q[h * ks + L.ld_c + f] = __float2bfloat16_rn((u * cs - v * sn) * scale);
        s_q[h * ks + L.ld_c + pairs + f] = __float2bfloat16_rn((v * cs + u * sn) * scale);
    }
    for (int i = tid; i < kLtHeads * pad; i += kLmThreads) s_q[(i / pad) * ks + ldk - pad + i % pad] = __float2bfloat16_rn(0.0f);
    __syncthreads();
    uint32_t q[PH][2][4];
    const uint32_t aq = smem_addr(s_q) + 2 * ((lane & 15) * ks + (lane >> 4) * 8), ap = smem_addr(s_p) + 2 * ((lane & 15) * 72 + (lane >> 4) * 8);
#pragma unroll
    for (int i = 0; i < PH; ++i)
        if (i < n_p) {
            ldsm4(q[i][0], aq + 2 * (p0 + i) * 32);
            ldsm4(q[i][1], aq + 2 * ((p0 + i) * 32 + 16));
        }
    __syncthreads();                                     // the queries' place becomes the second stage
    float m = -1e30f, l = 0.0f, acc[NP][2][4] = {};      // m, l: head `warp`
    const int n_pair = L.ld_c / 16;
    for (int tile = 0; tile < n_tiles; ++tile) {
        if (tile + 1 < n_tiles) {
            fetch(tile + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t bk = smem_addr(s_k + (tile & 1) * kLtTile * ks), kr = bk + 2 * ((kg * 8 + (lane & 7)) * ks + (lane >> 3) * 8 + p0 * 32);
        float sc[2][4] = {};
#pragma unroll
        for (int i = 0; i < PH; ++i)
            if (i < n_p) {
                uint32_t b[4];
                ldsm4(b, kr + 64 * i);
                mma_bf16(sc[0], q[i][0], b[0], b[1]);
                mma_bf16(sc[1], q[i][1], b[2], b[3]);
            }
#pragma unroll
        for (int i = 0; i < 4; ++i) s_s[(half * kLtHeads + g + (i >> 1) * 8) * 68 + kg * 8 + t4 * 2 + (i & 1)] = sc[0][i] + sc[1][i];
        __syncthreads();
        {
            const int left = j1 - j0 - tile * kLtTile;   // keys of this tile
            const float *s0 = s_s + warp * 68, *s1 = s_s + (kLtHeads + warp) * 68;
            const float v0 = lane < left ? s0[lane] + s1[lane] : -INFINITY, v1 = lane + 32 < left ? s0[lane + 32] + s1[lane + 32] : -INFINITY;
            const float mn = fmaxf(m, warp_max(fmaxf(v0, v1))), f = exp2f(m - mn), e0 = exp2f(v0 - mn), e1 = exp2f(v1 - mn);
            l = l * f + warp_sum(e0 + e1);
            m = mn;
            const bf16 b0 = __float2bfloat16_rn(e0), b1 = __float2bfloat16_rn(e1);
            s_p[warp * 72 + lane] = b0;
            s_p[warp * 72 + 32 + lane] = b1;
            s_p[(kLtHeads + warp) * 72 + lane] = __float2bfloat16_rn(e0 - __bfloat162float(b0));
            s_p[(kLtHeads + warp) * 72 + 32 + lane] = __float2bfloat16_rn(e1 - __bfloat162float(b1));
            if (lane == 0) s_f[warp] = f;
        }
        __syncthreads();
        const float f0 = s_f[g], f1 = s_f[g + 8];
#pragma unroll
        for (int i = 0; i < NP; ++i)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                acc[i][x][0] *= f0; acc[i][x][1] *= f0;
                acc[i][x][2] *= f1; acc[i][x][3] *= f1;
            }
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {
            uint32_t p[4], rest[4];
            ldsm4(p, ap + 2 * kt * 16);
            ldsm4(rest, ap + 2 * (kLtHeads * 72 + kt * 16));
#pragma unroll
            for (int i = 0; i < NP; ++i) {
                const int pair = warp + i * 16;
                if (pair >= n_pair) break;
                uint32_t b[4];
                ldsm4t(b, bk + 2 * ((kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ks + pair * 16 + (lane >> 4) * 8));
                mma_bf16(acc[i][0], p, b[0], b[1]);
                mma_bf16(acc[i][1], p, b[2], b[3]);
                mma_bf16(acc[i][0], rest, b[0], b[1]);
                mma_bf16(acc[i][1], rest, b[2], b[3]);
            }
        }
        __syncthreads();                                  // the stage and the weights may be overwritten
    }
    float* s_acc = reinterpret_cast<float*>(s_k);         // [16][ld_c]
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int pair = warp + i * 16;
        if (pair >= n_pair) break;
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int e = 0; e < 4; ++e) s_acc[(g + (e >> 1) * 8) * L.ld_c + pair * 16 + x * 8 + t4 * 2 + (e & 1)] = acc[i][x][e];
    }
    if (lane == 0) { s_ml[warp] = m / kLog2e; s_ml[kLtHeads + warp] = l; }
    latent_merge<bf16>(L, cluster, seq, h0, kLtHeads, s_acc, s_ml);
}

// ---- chunk ---------------------------------------------------------------------------------------------------------------
// One CTA per row: the M new rows (queries with their rotated part; cache row when the layer owns its cache), then the
// history rows from the ring.
template <typename T>
__global__ void __launch_bounds__(kLtThreads) latent_rows_kernel(const LatentLaunch L) {
    extern __shared__ float sm[];
    const LatentAttnArgs& a = L.a;
    const int t = blockIdx.x, tid = threadIdx.x;
    if (t >= a.M) {
        const int row = t - a.M;
        const size_t slot = (a.pos0 - L.hist + row) % a.ring;
        constexpr int E = 16 / sizeof(T);
        const uint4 *c = reinterpret_cast<const uint4*>(static_cast<const T*>(a.ring_c) + slot * L.ld_c), *r = reinterpret_cast<const uint4*>(static_cast<const T*>(a.ring_r) + slot * L.rot8);
        uint4 *dc = reinterpret_cast<uint4*>(static_cast<T*>(a.lin_c) + (size_t)row * L.ld_c), *dr = reinterpret_cast<uint4*>(static_cast<T*>(a.lin_r) + (size_t)row * L.rot8);
        for (int i = tid; i < L.ld_c / E; i += kLtThreads) dc[i] = c[i];
        for (int i = tid; i < L.rot8 / E; i += kLtThreads) dr[i] = r[i];
        return;
    }
    const int pos = a.pos0 + t, half = a.rot / 2, dq = a.dim + a.rot, lq = L.dim8 + L.rot8;
    float* s_cs = sm + 32;                               // [2][half]
    for (int i = tid; i < half; i += kLtThreads) rotation(a.freq[i], pos, s_cs[i], s_cs[half + i]);
    __syncthreads();
    const float* q = a.q + (size_t)t * a.ld;
    T* out = static_cast<T*>(a.lin_q) + (size_t)t * a.heads * lq;
    for (int i = tid; i < a.heads * lq; i += kLtThreads) {
        const int h = i / lq, d = i - h * lq, e = d - L.dim8;
        const float* qh = q + (size_t)h * dq;
        float v = 0.0f;
        if (e < 0) {
            if (d < a.dim) v = qh[d];
        } else if (e < a.rot) {
            const int f = e < half ? e : e - half;
            const float x = qh[a.dim + f], y = qh[a.dim + half + f], cs = s_cs[f], sn = s_cs[half + f];
            v = e < half ? x * cs - y * sn : y * cs + x * sn;
        }
        out[i] = from_f<T>(v);
    }
    if (a.dkv)
        latent_row<T>(L, a.dkv + (size_t)t * a.ld, pos, static_cast<T*>(a.lin_c) + (size_t)(L.hist + t) * L.ld_c, static_cast<T*>(a.lin_r) + (size_t)(L.hist + t) * L.rot8, sm);
}

// The last `rows` rows go into the ring (a launch of its own: the history is read first).
template <typename T>
__global__ void __launch_bounds__(128) latent_ring_kernel(const LatentLaunch L, int rows) {
    const LatentAttnArgs& a = L.a;
    constexpr int E = 16 / sizeof(T);
    const size_t lin = (size_t)L.hist + a.M - rows + blockIdx.x, slot = (a.pos0 + a.M - rows + blockIdx.x) % a.ring;
    uint4 *c = reinterpret_cast<uint4*>(static_cast<T*>(a.ring_c) + slot * L.ld_c), *r = reinterpret_cast<uint4*>(static_cast<T*>(a.ring_r) + slot * L.rot8);
    const uint4 *sc = reinterpret_cast<const uint4*>(static_cast<const T*>(a.lin_c) + lin * L.ld_c), *sr = reinterpret_cast<const uint4*>(static_cast<const T*>(a.lin_r) + lin * L.rot8);
    for (int i = threadIdx.x; i < L.ld_c / E; i += 128) c[i] = sc[i];
    for (int i = threadIdx.x; i < L.rot8 / E; i += 128) r[i] = sr[i];
}

template <typename T>
static int latent_decode(const LatentLaunch& L, cudaStream_t st, unsigned long long* n_kernels) {
    const LatentAttnArgs& a = L.a;
    auto absorb = [&](auto kernel, int rows, size_t smem, int append) {
        if (int rc = allow_smem(kernel, smem)) return rc;
        return launch_kernel(kernel, dim3((L.ld_c + 127) / 128, a.heads + (a.dkv ? append : 0), (a.M + rows - 1) / rows), dim3(kLtThreads), smem, st, a.use_pdl, 1, L);
    };
    auto fma_smem = [&](int rows) { return 4 * ((size_t)rows * L.dim8 + 8 * rows * 128); };
    const int dp = round_up(a.dim, 16);
    const int rc0 = a.M == 1                           ? absorb(latent_absorb_kernel<T, 1>, 1, fma_smem(1), 1)
                    : sizeof(T) == 4 || a.M < kLaMinRows ? absorb(latent_absorb_kernel<T, kLtAbsorbRows>, kLtAbsorbRows, fma_smem(kLtAbsorbRows), 1)
                                                         : absorb(latent_absorb_mma_kernel, kLaM, 2 * ((size_t)dp * kLaW + kLaM * (dp + 8)), 4);
    if (rc0) return rc0;
    const LatentSmem o(L.ld_c, L.rot8);
    const bool mma = sizeof(T) == 2 && L.ld_c <= 512 && o.bytes <= 220 * 1024;
    const int per_cta = mma ? kLtHeads : kLtFmaHeads, tiles = (a.heads + per_cta - 1) / per_cta;
    int cl = 1;                                          // slices of at least 64 keys, more than one only while SMs are free
    while (cl < 8 && a.ring > 64 * cl && (long long)2 * cl * tiles * a.M <= 148) cl *= 2;
    const dim3 grid(cl, tiles, a.M);
    auto go = [&](auto kernel, size_t smem, int threads = kLtThreads) {
        if (smem > 220 * 1024) return -1;
        if (int rc = allow_smem(kernel, smem)) return rc;
        return launch_kernel(kernel, grid, dim3(threads), smem, st, a.use_pdl, cl, L);
    };
    int rc;
    if (mma) {
        const int steps = (o.ks - 8) / 32;               // of 32 elements, over two halves
        rc = L.ld_c <= 256 ? (steps <= 6 ? go(latent_decode_mma_kernel<1, 3>, o.bytes, kLmThreads) : go(latent_decode_mma_kernel<1, 8>, o.bytes, kLmThreads))
                           : (steps <= 18 ? go(latent_decode_mma_kernel<2, 9>, o.bytes, kLmThreads) : go(latent_decode_mma_kernel<2, 12>, o.bytes, kLmThreads));
    } else {
        const int ldk = L.ld_c + L.rot8;
        const size_t smem = 4 * ((size_t)kLtFmaHeads * ldk + kLtFmaTile * (ldk + 1));
        rc = L.ld_c <= 128 ? go(latent_decode_kernel<T, 4>, smem) : L.ld_c <= 256 ? go(latent_decode_kernel<T, 8>, smem)
             : L.ld_c <= 512 ? go(latent_decode_kernel<T, 16>, smem) : go(latent_decode_kernel<T, 32>, smem);
    }
    if (rc) return rc;
    *n_kernels += 2;
    GemmArgs p;                                          // values: one segment per head
    p.a = a.lat; p.w = static_cast<const bf16*>(a.w_kv) + (size_t)a.heads * L.dim8 * L.ld_c;
    p.M = a.M; p.N = a.heads * L.vdim8; p.ld_k = L.ld_c;
    p.seg_rows = L.vdim8; p.a_seg_stride = (size_t)a.M * L.ld_c;
    p.epilogue = TENZO_GEMM_CAST; p.c = a.out; p.ld_c = a.ld_out;
    p.f32 = a.f32; p.use_pdl = a.use_pdl; p.workspace = a.workspace; p.workspace_bytes = a.workspace_bytes;
    return launch_gemm(p, st, n_kernels);
}

template <typename T>
static int latent_chunk(LatentLaunch& L, cudaStream_t st, unsigned long long* n_kernels) {
    const LatentAttnArgs& a = L.a;
    L.hist = a.pos0 < a.ring - 1 ? a.pos0 : a.ring - 1;
    const size_t smem = 4 * (32 + (size_t)a.rot);
    latent_rows_kernel<T><<<a.M + (a.dkv ? L.hist : 0), kLtThreads, smem, st>>>(L);
    *n_kernels += 1;
    if (a.dkv) {
        const int rows = a.M < a.ring ? a.M : a.ring;
        latent_ring_kernel<T><<<rows, 128, 0, st>>>(L, rows);
        *n_kernels += 1;
    }
    if (cudaError_t e = cudaGetLastError()) return (int)e;
    const int hist = a.pos0 < a.window - 1 ? a.pos0 : a.window - 1, skip = L.hist - hist;     // the cache may reach further back
    const int nk = a.heads * L.dim8, n = nk + a.heads * L.vdim8;
    GemmArgs p;
    p.a = static_cast<const T*>(a.lin_c) + (size_t)skip * L.ld_c; p.w = a.w_kv;
    p.M = hist + a.M; p.N = n; p.ld_k = L.ld_c; p.seg_end[0] = n;
    p.epilogue = TENZO_GEMM_CAST; p.c = a.kv; p.ld_c = n;
    p.f32 = a.f32; p.workspace = a.workspace; p.workspace_bytes = a.workspace_bytes;
    if (int rc = launch_gemm(p, st, n_kernels)) return rc;
    LinearAttn y;
    y.q = a.lin_q;
    y.k = a.kv; y.k_row = n; y.k_head = L.dim8;
    y.k2 = static_cast<const T*>(a.lin_r) + (size_t)skip * L.rot8; y.k2_row = L.rot8;
    y.v = static_cast<const T*>(a.kv) + nk; y.v_row = n; y.v_head = L.vdim8;
    y.d1 = L.dim8; y.d2 = L.rot8; y.dv = L.vdim8; y.vdim = L.vdim8;      // padded value columns are zero, and stored
    y.heads = a.heads; y.M = a.M; y.hist = hist; y.window = a.window; y.scale = a.scale;
    y.out = a.out; y.ld_out = a.ld_out; y.out_head = L.vdim8; y.f32 = a.f32;
    *n_kernels += 1;
    return launch_linear_attention(y, st);
}

int launch_latent_attention(const LatentAttnArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    if (a.M <= 0) return 0;
    if (a.heads < 1 || a.dim < 1 || a.rot < 2 || a.rot % 2 || a.vdim < 1 || a.vdim > kMaxHeadDim || a.dim > kMaxHeadDim || a.rot > kMaxHeadDim || a.rank < 1 ||
        a.rank > kMaxLatentRank || a.window < 1 || a.ring < 1 || !a.w_kv || !a.freq || (a.dkv && !a.norm)) return -1;
    LatentLaunch L;
    L.a = a;
    L.dim8 = round_up(a.dim, 8); L.rot8 = round_up(a.rot, 8); L.vdim8 = round_up(a.vdim, 8); L.ld_c = round_up(a.rank, 64); L.hist = 0;
    if (a.decode) return a.f32 ? latent_decode<float>(L, st, n_kernels) : latent_decode<bf16>(L, st, n_kernels);
    return a.f32 ? latent_chunk<float>(L, st, n_kernels) : latent_chunk<bf16>(L, st, n_kernels);
}

}  // namespace tz

extern "C" int tenzo_cuda_latent_attention(const tenzo_latent_attention_args* args, void* stream) {
    if (!args) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::LatentAttnArgs a;
    static_cast<tenzo_latent_attention_args&>(a) = *args;
    unsigned long long n = 0;
    return tz::launch_latent_attention(a, static_cast<cudaStream_t>(stream), &n);
}
