// Sliding-window attention of a chunk's rows over keys and values that lie in memory row after row (LinearAttn): bf16 rows
// go to the tensor cores (window_attention_mma.cu) where the head sizes allow it, the plain FMA form below does the rest.
#include "hybrid_common.cuh"

namespace tz {

int launch_window_flash(const LinearAttn& a, cudaStream_t st);       // window_attention_mma.cu
bool window_flash_applicable(const LinearAttn& a);

// A CTA takes eight consecutive queries of one head, a warp one of them; 32 keys at a time in shared memory, lanes over keys
// for the scores and over value columns for the sums.
constexpr int kLaThreads = 256, kLaQ = 8, kLaMaxCols = kMaxHeadDim / 32;

template <typename T>
__global__ void __launch_bounds__(kLaThreads) linear_attention_kernel(const LinearAttn a) {
    extern __shared__ float sm[];
    const int ldd = a.d1 + a.d2, ldv = a.dv, total = a.hist + a.M, h = blockIdx.y, kvh = h / a.group;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int kstride = ldd + 1;                            // odd: lanes hit different banks
    const T *gk = static_cast<const T*>(a.k) + (size_t)kvh * a.k_head, *gk2 = static_cast<const T*>(a.k2), *gv = static_cast<const T*>(a.v) + (size_t)kvh * a.v_head;
    float* s_k = sm;                                        // [32][ldd + 1]
    float* s_v = s_k + 32 * kstride;                        // [32][ldv]
    float* s_q = s_v + 32 * ldv;                            // [kLaQ][ldd]
    const int t = blockIdx.x * kLaQ + warp, i = a.hist + t;  // linear index of this warp's query
    const bool live = t < a.M;
    for (int d = lane; d < ldd; d += 32)
        s_q[warp * ldd + d] = live ? to_f(static_cast<const T*>(a.q)[((size_t)t * a.heads + h) * ldd + d]) * a.scale : 0.0f;
    const float slope = head_slope(a.slope_base, a.heads, h);
    float m = a.sink > 0.0f ? 0.0f : -1e30f, l = a.sink, acc[kLaMaxCols];   // the sink is a score of 0
#pragma unroll
    for (int c = 0; c < kLaMaxCols; ++c) acc[c] = 0.0f;
    const int i_last = a.hist + min(a.M, (int)(blockIdx.x + 1) * kLaQ) - 1;
    const int first = max(0, a.hist + (int)blockIdx.x * kLaQ - a.window + 1);
    for (int k0 = first; k0 <= i_last; k0 += 32) {
        __syncthreads();
        for (int e = threadIdx.x; e < 32 * ldd; e += kLaThreads) {
            const int r = e / ldd, d = e - r * ldd;
            const size_t row = k0 + r;
            s_k[r * kstride + d] = k0 + r >= total ? 0.0f : to_f(d < a.d1 ? gk[row * a.k_row + d] : gk2[row * a.k2_row + d - a.d1]);
        }
        for (int e = threadIdx.x; e < 32 * ldv; e += kLaThreads) {
            const int r = e / ldv, d = e - r * ldv;
            s_v[e] = k0 + r < total ? to_f(gv[(size_t)(k0 + r) * a.v_row + d]) : 0.0f;
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
        for (int c = 0; c < kLaMaxCols; ++c) acc[c] *= f;
        for (int r = 0; r < 32; ++r) {
            const float pr = __shfl_sync(0xffffffffu, p, r);
#pragma unroll
            for (int c = 0; c < kLaMaxCols; ++c)
                if (c * 32 + lane < ldv) acc[c] = fmaf(pr, s_v[r * ldv + c * 32 + lane], acc[c]);
        }
    }
    if (!live) return;
    T* out = static_cast<T*>(a.out) + (size_t)t * a.ld_out + (size_t)h * a.out_head;
#pragma unroll
    for (int c = 0; c < kLaMaxCols; ++c)
        if (c * 32 + lane < a.vdim) out[c * 32 + lane] = from_f<T>(acc[c] / l);
}

template <typename T>
static int linear_attention(const LinearAttn& a, cudaStream_t st) {
    const int ldd = a.d1 + a.d2;
    const size_t smem = 4 * ((size_t)32 * (ldd + 1) + 32 * a.dv + kLaQ * ldd);
    if (int rc = allow_smem(linear_attention_kernel<T>, smem)) return rc;
    linear_attention_kernel<T><<<dim3((a.M + kLaQ - 1) / kLaQ, a.heads), kLaThreads, smem, st>>>(a);
    return (int)cudaGetLastError();
}

int launch_linear_attention(const LinearAttn& a, cudaStream_t st) {
    if (a.d1 % 8 || a.d2 % 8 || a.dv % 8 || a.d1 + a.d2 > 2 * kMaxHeadDim || a.dv > kMaxHeadDim || (a.d2 && !a.k2)) return -1;
    if (a.f32) return linear_attention<float>(a, st);
    return window_flash_applicable(a) ? launch_window_flash(a, st) : linear_attention<bf16>(a, st);
}

}  // namespace tz
