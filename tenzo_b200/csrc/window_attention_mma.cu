// Sliding-window attention over the linear layout of a chunk (LinearAttn) with bf16 storage, on tensor cores (mma.sync
// m16n8k16).
//
// A CTA takes 64 consecutive queries of one head, a warp 16 of them; tiles of 64 keys stream through two shared-memory
// stages. Scores and softmax are fp32. The weights enter the second product as the sum of two bf16 values (the rounded
// weight and its remainder), so that rounding them costs nothing visible.
#include "hybrid_common.cuh"

namespace tz {

constexpr int kWfQ = 64, kWfK = 64, kWfThreads = 128;

struct WfLaunch {
    LinearAttn a;
    int dp, vp;                              // head sizes padded to 32 / 16
};

// two floats as bf16 (x in the low half), and what the rounding dropped
__device__ __forceinline__ uint32_t pack_split(float x, float y, uint32_t& rest) {
    const bf16 bx = __float2bfloat16_rn(x), by = __float2bfloat16_rn(y);
    const bf16 rx = __float2bfloat16_rn(x - __bfloat162float(bx)), ry = __float2bfloat16_rn(y - __bfloat162float(by));
    rest = (uint32_t)__bfloat16_as_ushort(ry) << 16 | __bfloat16_as_ushort(rx);
    return (uint32_t)__bfloat16_as_ushort(by) << 16 | __bfloat16_as_ushort(bx);
}

// KT: 16-wide steps of the key size (even), VT: 8-wide blocks of the value size (even).
template <int KT, int VT>
__global__ void __launch_bounds__(kWfThreads) window_flash_kernel(const WfLaunch L) {
    extern __shared__ __align__(16) unsigned char smem[];
    const LinearAttn& a = L.a;
    const int d1 = a.d1 / 8, ldd = a.d1 + a.d2, ldv = a.dv, ks = L.dp + 8, vs = L.vp + 8, total = a.hist + a.M;
    const int h = blockIdx.y, kvh = h / a.group, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    bf16* s_k = reinterpret_cast<bf16*>(smem);               // [2][64][ks]
    bf16* s_v = s_k + 2 * kWfK * ks;                         // [2][64][vs]
    const bf16* gk = static_cast<const bf16*>(a.k) + (size_t)kvh * a.k_head;
    const bf16* gk2 = static_cast<const bf16*>(a.k2);
    const bf16* gv = static_cast<const bf16*>(a.v) + (size_t)kvh * a.v_head;
    for (int i = tid; i < 2 * kWfK * (ks + vs) / 8; i += kWfThreads) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);   // padding
    __syncthreads();

    const int q0 = blockIdx.x * kWfQ, row0 = q0 + warp * 16;  // this warp's queries
    uint32_t qf[KT][4];
#pragma unroll
    for (int kt = 0; kt < KT; ++kt)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int t = row0 + g + (i & 1) * 8, c = kt * 16 + t4 * 2 + (i >> 1) * 8;
            qf[kt][i] = t < a.M && c < ldd ? *reinterpret_cast<const uint32_t*>(static_cast<const bf16*>(a.q) + ((size_t)t * a.heads + h) * ldd + c) : 0u;
        }

    const int i_first = a.hist + q0, i_last = a.hist + min(a.M, q0 + kWfQ) - 1;      // linear places of the CTA's queries
    const int k_first = max(0, i_first - a.window + 1) / kWfK * kWfK;
    const int n_tiles = (i_last - k_first) / kWfK + 1;
    auto fetch = [&](int tile) {
        const int k0 = k_first + tile * kWfK;
        bf16 *dk = s_k + (tile & 1) * kWfK * ks, *dv = s_v + (tile & 1) * kWfK * vs;
        for (int i = tid; i < kWfK * (ldd / 8); i += kWfThreads) {
            const int r = i / (ldd / 8), c = i - r * (ldd / 8);
            const size_t row = min(k0 + r, total - 1);
            cp16(dk + r * ks + c * 8, c < d1 ? gk + row * a.k_row + c * 8 : gk2 + row * a.k2_row + (c - d1) * 8);
        }
        for (int i = tid; i < kWfK * (ldv / 8); i += kWfThreads) {
            const int r = i / (ldv / 8), c = i - r * (ldv / 8);
            cp16(dv + r * vs + c * 8, gv + (size_t)min(k0 + r, total - 1) * a.v_row + c * 8);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const float log2e = 1.4426950408889634f;
    const float scale = a.scale * log2e, slope = (a.slope_base == 0.0f ? 0.0f : exp2f(-a.slope_base * (float)(h + 1) / (float)a.heads)) * log2e;
    float m[2], l[2] = {0.0f, 0.0f}, o[VT][4];
    m[0] = m[1] = a.sink > 0.0f ? 0.0f : -1e30f;
#pragma unroll
    for (int v = 0; v < VT; ++v) o[v][0] = o[v][1] = o[v][2] = o[v][3] = 0.0f;

    fetch(0);
    for (int tile = 0; tile < n_tiles; ++tile) {
        if (tile + 1 < n_tiles) {
            fetch(tile + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int k0 = k_first + tile * kWfK, w_first = a.hist + row0, w_last = w_first + 15;
        // a warp skips tiles that none of its queries sees
        if (row0 < a.M && k0 <= w_last && k0 + kWfK - 1 > w_first - a.window) {
            const uint32_t bk = smem_addr(s_k + (tile & 1) * kWfK * ks), bv = smem_addr(s_v + (tile & 1) * kWfK * vs);
            float s[8][4];
#pragma unroll
            for (int n = 0; n < 8; ++n) {
                s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.0f;
#pragma unroll
                for (int kt = 0; kt < KT; kt += 2) {
                    if (kt * 16 >= L.dp) break;
                    uint32_t b[4];
                    ldsm4(b, bk + 2 * ((n * 8 + (lane & 7)) * ks + kt * 16 + (lane >> 3) * 8));
                    mma_bf16(s[n], qf[kt], b[0], b[1]);
                    mma_bf16(s[n], qf[kt + 1], b[2], b[3]);
                }
            }
            const bool edge = k0 + kWfK - 1 > w_first || k0 <= w_last - a.window;
            float mx[2] = {m[0], m[1]};
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int dist = w_first + g + (i >> 1) * 8 - (k0 + n * 8 + t4 * 2 + (i & 1));
                    float x = fmaf(s[n][i], scale, -slope * (float)dist);
                    if (edge && (dist < 0 || dist >= a.window)) x = -INFINITY;
                    s[n][i] = x;
                    mx[i >> 1] = fmaxf(mx[i >> 1], x);
                }
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                const float f = exp2f(m[r] - mx[r]);
                m[r] = mx[r];
                l[r] *= f;
#pragma unroll
                for (int v = 0; v < VT; ++v) {
                    o[v][2 * r] *= f;
                    o[v][2 * r + 1] *= f;
                }
            }
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) {                  // 16 keys at a time
                uint32_t p[4], rest[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int n = 2 * kt + (i >> 1), r = i & 1;
                    const float x = exp2f(s[n][2 * r] - m[r]), y = exp2f(s[n][2 * r + 1] - m[r]);
                    l[r] += x + y;
                    p[i] = pack_split(x, y, rest[i]);
                }
#pragma unroll
                for (int v = 0; v < VT; v += 2) {
                    if (v * 8 >= L.vp) break;
                    uint32_t b[4];
                    ldsm4t(b, bv + 2 * ((kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + v * 8 + (lane >> 4) * 8));
                    mma_bf16(o[v], p, b[0], b[1]);
                    mma_bf16(o[v], rest, b[0], b[1]);
                    mma_bf16(o[v + 1], p, b[2], b[3]);
                    mma_bf16(o[v + 1], rest, b[2], b[3]);
                }
            }
        }
        __syncthreads();                                      // the stage is free for the fetch after next
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        const int t = row0 + g + r * 8;
        if (t >= a.M) continue;
        const float inv = 1.0f / (l[r] + (a.sink > 0.0f ? a.sink * exp2f(-m[r]) : 0.0f));
        bf16* out = reinterpret_cast<bf16*>(a.out) + (size_t)t * a.ld_out + (size_t)h * a.out_head;
#pragma unroll
        for (int v = 0; v < VT; ++v)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int d = v * 8 + t4 * 2 + i;
                if (d < a.vdim) out[d] = __float2bfloat16_rn(o[v][2 * r + i] * inv);
            }
    }
}

bool window_flash_applicable(const LinearAttn& a) { return a.d1 + a.d2 <= 256 && a.vdim <= 128 && a.M >= 16; }

int launch_window_flash(const LinearAttn& a, cudaStream_t st) {
    WfLaunch L;
    L.a = a;
    L.dp = round_up(a.d1 + a.d2, 32); L.vp = round_up(a.vdim, 16);
    const size_t smem = (size_t)2 * 2 * kWfK * (L.dp + 8 + L.vp + 8);
    const dim3 grid((a.M + kWfQ - 1) / kWfQ, a.heads);
    auto go = [&](auto kernel) {
        if (int rc = allow_smem(kernel, smem)) return rc;
        kernel<<<grid, kWfThreads, smem, st>>>(L);
        return (int)cudaGetLastError();
    };
    if (L.dp <= 64) return L.vp <= 64 ? go(window_flash_kernel<4, 8>) : go(window_flash_kernel<4, 16>);
    if (L.dp <= 128) return L.vp <= 64 ? go(window_flash_kernel<8, 8>) : go(window_flash_kernel<8, 16>);
    if (L.dp <= 192) return L.vp <= 64 ? go(window_flash_kernel<12, 8>) : go(window_flash_kernel<12, 16>);
    return L.vp <= 64 ? go(window_flash_kernel<16, 8>) : go(window_flash_kernel<16, 16>);
}

}  // namespace tz
