// Matrix products with bf16 weights for the hybrid decoders: few rows (decode) as a weight-streaming GEMV, many fp32 rows
// as a tiled FMA product; many bf16 rows go to the tensor cores (gemm_umma.cu). Also the greedy argmax over fp32 logits.
#include "hybrid_common.cuh"
#include "lm_head.cuh"

namespace tz {

constexpr int kGemvThreads = 256, kGemvWarps = kGemvThreads / 32, kGemvMaxRows = 8;

template <typename T>
__device__ __forceinline__ void gemm_store(const GemmArgs& a, int m, int n, float v) {
    const size_t at = (size_t)m * a.ld_c + n;
    switch (a.epilogue) {
        case TENZO_GEMM_XIELU: reinterpret_cast<T*>(a.c)[at] = from_f<T>(xielu_f(v, a.act_pos, a.act_neg)); break;
        case TENZO_GEMM_CAST: reinterpret_cast<T*>(a.c)[at] = from_f<T>(v); break;
        case TENZO_GEMM_SOFTCAP: reinterpret_cast<float*>(a.c)[at] = soft_cap_f(v, a.cap); break;
        default: reinterpret_cast<float*>(a.c)[at] = v;
    }
}
__device__ __forceinline__ bool gemm_is_glu(const GemmArgs& a) { return a.epilogue == TENZO_GEMM_GLU_RELU || a.epilogue == TENZO_GEMM_GLU_SILU; }

__device__ __forceinline__ int gemm_segment(const GemmArgs& a, int n) {
    if (a.seg_rows > 0) return n / a.seg_rows;
    int s = 0;
    while (s + 1 < a.n_seg && n >= a.seg_end[s]) ++s;
    return s;
}

// One warp per output column n (= weight row), all MR activation rows at once. The first 2048 weights of the row are in
// registers before the kernel waits for its producer: weights do not depend on it. Grouped form: blockIdx.y is the row, and
// which matrix it multiplies is only known after the wait. GLU: neighbouring warps hold a gate and its up value.
template <typename T, int MR>
__global__ void __launch_bounds__(kGemvThreads) gemv_kernel(const GemmArgs a) {
    __shared__ float s_glu[kGemvWarps][MR];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n = blockIdx.x * kGemvWarps + warp;
    bool live = n < a.N;
    const bf16* wrow = static_cast<const bf16*>(a.w) + (size_t)(live ? n : 0) * a.ld_k;
    const int chunks = a.ld_k / 8;
    constexpr int kPre = 8;
    uint4 pre[kPre];
    auto fetch = [&]() {
#pragma unroll
        for (int i = 0; i < kPre; ++i)
            if (live && i * 32 + lane < chunks) pre[i] = ld_stream_u4(wrow + (size_t)(i * 32 + lane) * 8);
    };
    if (!a.group_off) fetch();
    pdl_wait();
    pdl_launch_dependents();
    const T* x = reinterpret_cast<const T*>(a.a);
    int row0 = 0;
    if (a.group_off) {
        row0 = blockIdx.y;
        int g = 0;
        for (int e0 = 0; e0 < a.n_group; e0 += 32) g += __popc(__ballot_sync(0xffffffffu, e0 + lane < a.n_group && a.group_off[e0 + lane + 1] <= row0));
        live = live && g < a.n_group;
        wrow += (size_t)(g < a.n_group ? g : 0) * a.N * a.ld_k;
        x += (size_t)(a.a_index ? a.a_index[row0] : row0) * a.ld_k;
        fetch();
    } else if (live) {
        x += (size_t)gemm_segment(a, n) * a.a_seg_stride;
    }
    float acc[MR];
#pragma unroll
    for (int m = 0; m < MR; ++m) acc[m] = 0.0f;
    const int n_rows = a.group_off ? 1 : a.M;
    if (live) {
    auto step = [&](const uint4& wv, int ch) {
        float w[8];
        unpack8(wv, w);
#pragma unroll
        for (int m = 0; m < MR; ++m) {
            if (m < n_rows) {
                float xv[8];
                load8(x + (size_t)m * a.ld_k + (size_t)ch * 8, xv);
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[m] = fmaf(w[j], xv[j], acc[m]);
            }
        }
    };
#pragma unroll
    for (int i = 0; i < kPre; ++i)
        if (i * 32 + lane < chunks) step(pre[i], i * 32 + lane);
    for (int ch = kPre * 32 + lane; ch < chunks; ch += 4 * 32) {
        uint4 w[4];
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (ch + u * 32 < chunks) w[u] = ld_stream_u4(wrow + (size_t)(ch + u * 32) * 8);
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (ch + u * 32 < chunks) step(w[u], ch + u * 32);
    }
#pragma unroll
    for (int m = 0; m < MR; ++m) acc[m] = warp_sum(acc[m]);
    }
    if (gemm_is_glu(a)) {
        if (lane == 0) {
#pragma unroll
            for (int m = 0; m < MR; ++m) s_glu[warp][m] = acc[m];
        }
        __syncthreads();
        if ((warp & 1) == 0 && lane < n_rows && live) {
            const float g = s_glu[warp][lane < MR ? lane : 0], u = s_glu[warp + 1][lane < MR ? lane : 0];
            reinterpret_cast<T*>(a.c)[(size_t)(row0 + lane) * a.ld_c + n / 2] = from_f<T>(glu_f(a.epilogue, g, u));
        }
    } else if (live && lane == 0) {
#pragma unroll
        for (int m = 0; m < MR; ++m)
            if (m < n_rows) gemm_store<T>(a, row0 + m, n, acc[m]);
    }
}

// 64 x 64 output tile, 16-wide K steps, 4 x 4 outputs per thread. Grouped form: blockIdx.z is the group, tiles past its rows
// leave at once.
template <typename T>
__global__ void __launch_bounds__(256) gemm_fma_kernel(const GemmArgs a) {
    __shared__ float s_a[16][68], s_w[16][68];
    const int n0 = blockIdx.x * 64, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    pdl_wait();
    pdl_launch_dependents();
    const int first = a.group_off ? a.group_off[blockIdx.z] : 0, m_end = a.group_off ? min(a.M, a.group_off[blockIdx.z + 1]) : a.M;
    const int m0 = first + blockIdx.y * 64;
    if (m0 >= m_end) return;
    const bf16* w = static_cast<const bf16*>(a.w) + (a.group_off ? (size_t)blockIdx.z * a.N * a.ld_k : 0);
    // a segment border inside the tile: columns of both segments are computed from their own A, tile by tile of 64 columns
    const int s_first = gemm_segment(a, n0), s_last = gemm_segment(a, min(n0 + 63, a.N - 1));
    for (int seg = s_first; seg <= s_last; ++seg) {
        const T* x = reinterpret_cast<const T*>(a.a) + (size_t)seg * a.a_seg_stride;
        float acc[4][4] = {};
        for (int k0 = 0; k0 < a.ld_k; k0 += 16) {
            {
                const int r = tid >> 2, kk = (tid & 3) * 4;
                const int m = m0 + r, n = n0 + r;
                const size_t src = (size_t)(m < m_end && a.a_index ? a.a_index[m] : m) * a.ld_k;
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    s_a[kk + j][r] = m < m_end ? to_f(x[src + k0 + kk + j]) : 0.0f;
                    s_w[kk + j][r] = n < a.N ? to_f(w[(size_t)n * a.ld_k + k0 + kk + j]) : 0.0f;
                }
            }
            __syncthreads();
#pragma unroll
            for (int k = 0; k < 16; ++k) {
                const float4 av = *reinterpret_cast<const float4*>(&s_a[k][ty * 4]), wv = *reinterpret_cast<const float4*>(&s_w[k][tx * 4]);
                const float af[4] = {av.x, av.y, av.z, av.w}, wf[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(af[i], wf[j], acc[i][j]);
            }
            __syncthreads();
        }
        if (gemm_is_glu(a)) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; j += 2) {
                    const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
                    if (m < m_end && n < a.N && gemm_segment(a, n) == seg)
                        reinterpret_cast<T*>(a.c)[(size_t)m * a.ld_c + n / 2] = from_f<T>(glu_f(a.epilogue, acc[i][j], acc[i][j + 1]));
                }
            continue;
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
                if (m < m_end && n < a.N && gemm_segment(a, n) == seg) gemm_store<T>(a, m, n, acc[i][j]);
            }
    }
}

// Rows of a grouped product side by side: dst[m] = src[index[m]], 16 bytes per thread and trip.
struct GatherArgs { uint4* dst; const uint4* src; const int* index; int a_rows, chunks; };
__global__ void __launch_bounds__(256) gather_rows_kernel(const GatherArgs g) {
    pdl_wait();
    pdl_launch_dependents();
    const int r = min(max(g.index[blockIdx.x], 0), g.a_rows - 1);
    for (int i = threadIdx.x; i < g.chunks; i += 256) g.dst[(size_t)blockIdx.x * g.chunks + i] = g.src[(size_t)r * g.chunks + i];
}

template <typename T>
static int launch_gemv(const GemmArgs& a, cudaStream_t st) {
    const dim3 grid((a.N + kGemvWarps - 1) / kGemvWarps, a.group_off ? a.M : 1), block(kGemvThreads);
    auto go = [&](auto kernel) { return launch_kernel(kernel, grid, block, 0, st, a.use_pdl, 1, a); };
    if (a.M == 1 || a.group_off) return go(gemv_kernel<T, 1>);
    if (a.M == 2) return go(gemv_kernel<T, 2>);
    if (a.M <= 4) return go(gemv_kernel<T, 4>);
    return go(gemv_kernel<T, 8>);
}

int launch_gemm(const GemmArgs& a, cudaStream_t st, unsigned long long* n_kernels) {
    if (a.M <= 0 || a.N <= 0) return 0;
    if (a.ld_k % 64 || a.n_seg < 1 || a.n_seg > 8 || a.seg_rows < 0) return -1;
    const bool glu = a.epilogue == TENZO_GEMM_GLU_RELU || a.epilogue == TENZO_GEMM_GLU_SILU, grouped = a.group_off != nullptr;
    if ((glu && (a.N % 2 || a.seg_rows % 2)) || (grouped && (a.n_group < 1 || a.n_seg != 1 || a.seg_rows)) || (a.a_index && !grouped)) return -1;
    *n_kernels += 1;
    if (!a.f32 && gemm_umma_applicable(a)) {
        if (!a.a_index) return launch_gemm_umma(a, st);
        *n_kernels += 1;
        const GatherArgs g = {static_cast<uint4*>(a.a_gather), static_cast<const uint4*>(a.a), a.a_index, a.a_rows, a.ld_k / 8};
        if (int rc = launch_kernel(gather_rows_kernel, dim3(a.M), dim3(256), 0, st, a.use_pdl, 1, g)) return rc;
        GemmArgs p = a;
        p.a = a.a_gather;
        p.a_index = nullptr;
        return launch_gemm_umma(p, st);
    }
    if (a.f32 && a.M > (grouped ? 8 * kGemvMaxRows : kGemvMaxRows)) {
        gemm_fma_kernel<float><<<dim3((a.N + 63) / 64, (a.M + 63) / 64, grouped ? a.n_group : 1), 256, 0, st>>>(a);
        return (int)cudaGetLastError();
    }
    if (grouped) return a.M > 65535 ? -1 : a.f32 ? launch_gemv<float>(a, st) : launch_gemv<bf16>(a, st);
    *n_kernels += (a.M - 1) / kGemvMaxRows;
    // groups of up to eight rows; the weights of the second group come from L2
    for (int m0 = 0; m0 < a.M; m0 += kGemvMaxRows) {
        GemmArgs p = a;
        p.M = a.M - m0 < kGemvMaxRows ? a.M - m0 : kGemvMaxRows;
        const size_t es = a.f32 ? 4 : 2, cs = a.epilogue == TENZO_GEMM_STORE || a.epilogue == TENZO_GEMM_SOFTCAP ? 4 : es;
        p.a = static_cast<const char*>(a.a) + (size_t)m0 * a.ld_k * es;
        p.c = static_cast<char*>(a.c) + (size_t)m0 * a.ld_c * cs;
        if (int rc = a.f32 ? launch_gemv<float>(p, st) : launch_gemv<bf16>(p, st)) return rc;
    }
    return 0;
}

// ---- greedy argmax ------------------------------------------------------------------------------------------------------
constexpr int kArgmaxSplits = 64;

__device__ __forceinline__ LmBest block_best(LmBest b) {
    __shared__ LmBest s[8];
#pragma unroll
    for (int m = 16; m > 0; m >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, b.val, m);
        const int i = __shfl_xor_sync(0xffffffffu, b.idx, m);
        if (better(v, i, b.val, b.idx)) { b.val = v; b.idx = i; }
    }
    if ((threadIdx.x & 31) == 0) s[threadIdx.x >> 5] = b;
    __syncthreads();
    if (threadIdx.x == 0)
        for (int w = 1; w < (int)(blockDim.x >> 5); ++w)
            if (better(s[w].val, s[w].idx, b.val, b.idx)) b = s[w];
    return b;
}

__global__ void __launch_bounds__(256) argmax_part_kernel(const float* __restrict__ logits, int vocab, LmBest* part) {
    const float* row = logits + (size_t)blockIdx.y * vocab;
    LmBest b = {-INFINITY, 0x7fffffff};
    for (int i = blockIdx.x * 256 + threadIdx.x; i < vocab; i += gridDim.x * 256)
        if (better(row[i], i, b.val, b.idx)) { b.val = row[i]; b.idx = i; }
    b = block_best(b);
    if (threadIdx.x == 0) part[(size_t)blockIdx.y * gridDim.x + blockIdx.x] = b;
}

__global__ void __launch_bounds__(64) argmax_finish_rows_kernel(const LmBest* part, int n, int* out) {
    LmBest b = {-INFINITY, 0x7fffffff};
    for (int i = threadIdx.x; i < n; i += 64) {
        const LmBest p = part[(size_t)blockIdx.x * n + i];
        if (better(p.val, p.idx, b.val, b.idx)) b = p;
    }
    b = block_best(b);
    if (threadIdx.x == 0) out[blockIdx.x] = b.idx == 0x7fffffff ? 0 : b.idx;
}

size_t argmax_scratch_bytes(int rows) { return (size_t)rows * kArgmaxSplits * sizeof(LmBest); }

int launch_argmax(const float* logits, int vocab, int rows, int* out, void* scratch, cudaStream_t st) {
    int splits = (vocab + 1023) / 1024;
    if (splits > kArgmaxSplits) splits = kArgmaxSplits;
    argmax_part_kernel<<<dim3(splits, rows), 256, 0, st>>>(logits, vocab, static_cast<LmBest*>(scratch));
    argmax_finish_rows_kernel<<<rows, 64, 0, st>>>(static_cast<const LmBest*>(scratch), splits, out);
    return (int)cudaGetLastError();
}

}  // namespace tz

extern "C" int tenzo_cuda_gemm(const tenzo_gemm_args* args, void* stream) {
    if (!args) return TENZO_ERROR_INVALID_ARGUMENT;
    tz::GemmArgs a;
    static_cast<tenzo_gemm_args&>(a) = *args;
    unsigned long long n = 0;
    return tz::launch_gemm(a, static_cast<cudaStream_t>(stream), &n);
}
