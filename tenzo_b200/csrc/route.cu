// Choice of experts (RouteArgs): sigmoid scores, the `top` largest of score + correction per row, weights are the chosen
// scores themselves, and the (row, choice) pairs in order of their expert, which is how the grouped products take them.
// Few rows: one CTA does all of it. Many: a warp per row chooses, then a CTA per expert collects its pairs in row order.
#include "hybrid_common.cuh"

namespace tz {

constexpr int kRouteThreads = 1024, kRouteSmallPairs = 1024;

// A warp chooses for row m; s: [E] scratch of the warp. Choice scores are kept as integers in the order of the floats, 0 for
// an expert that is taken (what a score that is not a number becomes may be any other value).
__device__ __forceinline__ unsigned ordered(float v) {
    const unsigned b = __float_as_uint(v);
    return max(b ^ ((b >> 31) ? 0xffffffffu : 0x80000000u), 1u);
}

__device__ __forceinline__ void choose(const RouteArgs& a, int m, unsigned* s) {
    const int lane = threadIdx.x & 31;
    const float* z = a.logits + (size_t)m * a.ld;
    for (int e = lane; e < a.experts; e += 32) s[e] = ordered(sigmoid_f(z[e]) + (a.correction ? a.correction[e] : 0.0f));
    __syncwarp();
    for (int j = 0; j < a.top; ++j) {
        unsigned best = 0;
        int at = 0x7fffffff;
        for (int e = lane; e < a.experts; e += 32)
            if (s[e] > best) { best = s[e]; at = e; }
        const unsigned top = __reduce_max_sync(0xffffffffu, best);
        at = (int)__reduce_min_sync(0xffffffffu, best == top ? (unsigned)at : 0x7fffffffu);      // equal scores: the lower index
        if (lane == 0) {
            a.chosen[(size_t)m * a.top + j] = at;
            a.weight[(size_t)m * a.top + j] = sigmoid_f(z[at]);
            s[at] = 0;
        }
        __syncwarp();
    }
}

// Pairs of expert e, in order: their places start after those of the experts before it. One warp.
__device__ __forceinline__ void place_pairs(const RouteArgs& a, int e, const int* chosen, int n) {
    const int lane = threadIdx.x & 31;
    int before = 0, mine = 0;
    for (int p0 = 0; p0 < n; p0 += 32) {
        const int c = p0 + lane < n ? chosen[p0 + lane] : a.experts;
        before += __popc(__ballot_sync(0xffffffffu, c < e));
        mine += __popc(__ballot_sync(0xffffffffu, c == e));
    }
    if (lane == 0) {
        a.group_off[e] = before;
        if (e == a.experts - 1) a.group_off[a.experts] = n;
    }
    if (!mine) return;
    int at = before;
    for (int p0 = 0; p0 < n; p0 += 32) {
        const bool hit = p0 + lane < n && chosen[p0 + lane] == e;
        const unsigned b = __ballot_sync(0xffffffffu, hit);
        if (hit) {
            const int slot = at + __popc(b & ((1u << lane) - 1));
            a.slot[p0 + lane] = slot;
            a.row_of[slot] = (p0 + lane) / a.top;
        }
        at += __popc(b);
    }
}

__global__ void __launch_bounds__(kRouteThreads) route_small_kernel(const RouteArgs a) {
    extern __shared__ unsigned sm[];
    __shared__ int s_chosen[kRouteSmallPairs];
    const int warp = threadIdx.x >> 5, nw = blockDim.x >> 5, n = a.M * a.top;
    pdl_wait();
    pdl_launch_dependents();
    for (int m = warp; m < a.M; m += nw) choose(a, m, sm + (size_t)warp * a.experts);
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x) s_chosen[i] = a.chosen[i];
    __syncthreads();
    for (int e = warp; e < a.experts; e += nw) place_pairs(a, e, s_chosen, n);
}

__global__ void __launch_bounds__(256) route_choose_kernel(const RouteArgs a) {
    extern __shared__ unsigned sm[];
    const int m = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (m < a.M) choose(a, m, sm + (size_t)(threadIdx.x >> 5) * a.experts);
}

// One CTA per expert: counts, then places, 1024 pairs at a time.
__global__ void __launch_bounds__(kRouteThreads) route_place_kernel(const RouteArgs a) {
    __shared__ int s_less[32], s_mine[32];
    const int e = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = a.M * a.top;
    int less = 0;
    for (int p = tid; p < n; p += kRouteThreads) less += a.chosen[p] < e;
    less = warp_sum_i(less);
    if (lane == 0) s_less[warp] = less;
    __syncthreads();
    int at = warp_sum_i(s_less[lane]);
    if (tid == 0) {
        a.group_off[e] = at;
        if (e == a.experts - 1) a.group_off[a.experts] = n;
    }
    for (int p0 = 0; p0 < n; p0 += kRouteThreads) {
        const int p = p0 + tid;
        const bool hit = p < n && a.chosen[p] == e;
        const unsigned b = __ballot_sync(0xffffffffu, hit);
        if (lane == 0) s_mine[warp] = __popc(b);
        __syncthreads();
        const int c = s_mine[lane], total = warp_sum_i(c), before = warp_sum_i(lane < warp ? c : 0);
        if (hit) {
            const int slot = at + before + __popc(b & ((1u << lane) - 1));
            a.slot[p] = slot;
            a.row_of[slot] = p / a.top;
        }
        at += total;
        __syncthreads();
    }
}

int launch_route(const RouteArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    if (a.M <= 0) return 0;
    if (a.experts < 1 || a.top < 1 || a.top > a.experts || a.experts > 4096 || !a.logits || !a.chosen || !a.weight || !a.slot || !a.row_of || !a.group_off) return -1;
    if ((long long)a.M * a.top <= kRouteSmallPairs) {
        // enough warps for the rows and the experts, as far as their scratch fits
        int nw = (a.M > a.experts ? a.M : a.experts);
        if (nw > 32) nw = 32;
        while (nw > 1 && (size_t)nw * a.experts * 4 > 40 * 1024) nw /= 2;
        *n_kernels += 1;
        return launch_kernel(route_small_kernel, dim3(1), dim3(32 * nw), (size_t)nw * a.experts * 4, st, a.use_pdl, 1, a);
    }
    const size_t smem = (size_t)8 * a.experts * 4;
    if (int rc = allow_smem(route_choose_kernel, smem)) return rc;
    route_choose_kernel<<<(a.M + 7) / 8, 256, smem, st>>>(a);
    route_place_kernel<<<a.experts, kRouteThreads, 0, st>>>(a);
    *n_kernels += 2;
    return (int)cudaGetLastError();
}

}  // namespace tz

extern "C" int tenzo_cuda_route(const tenzo_route_args* args, void* stream) {
    if (!args) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::RouteArgs a;
    static_cast<tenzo_route_args&>(a) = *args;
    unsigned long long n = 0;
    return tz::launch_route(a, static_cast<cudaStream_t>(stream), &n);
}
