// Device helpers of the hybrid-decoder kernels.
#pragma once
#include "../../include/tenzo.h"
#include "common.cuh"
#include "hybrid_ops.h"

namespace tz {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ void bf16x2_to_f(uint32_t u, float& lo, float& hi) {
    lo = __uint_as_float(u << 16);
    hi = __uint_as_float(u & 0xffff0000u);
}
__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
    bf16x2_to_f(u.x, f[0], f[1]); bf16x2_to_f(u.y, f[2], f[3]); bf16x2_to_f(u.z, f[4], f[5]); bf16x2_to_f(u.w, f[6], f[7]);
}
// eight consecutive elements, 16-byte aligned
__device__ __forceinline__ void load8(const bf16* p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }
// ln(1 + e^-z), stable on both sides
__device__ __forceinline__ float softplus_neg(float z) { return fmaxf(-z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap_f(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float glu_f(int epilogue, float gate, float up) {
    return (epilogue == TENZO_GEMM_GLU_RELU ? fmaxf(gate, 0.0f) : silu_f(gate)) * up;
}
__device__ __forceinline__ float xielu_f(float z, float pos, float neg) {
    return 0.5f * z + (z > 0.0f ? pos * z * z : neg * (expm1f(z) - z));
}

// slope of head h's linear distance bias
__device__ __forceinline__ float head_slope(float slope_base, int heads, int h) {
    return slope_base == 0.0f ? 0.0f : exp2f(-slope_base * (float)(h + 1) / (float)heads);
}

// Sums of GQ values over groups of LK lanes: halves of the values travel while there are several, so that the total is
// GQ - 1 + log2(LK / GQ) exchanges. The lane is left with the sum of value `which`.
template <int GQ, int LK>
__device__ __forceinline__ float group_sums(float (&s)[GQ], int lane, int& which) {
    which = 0;
    int m = LK / 2;
#pragma unroll
    for (int n = GQ; n > 1; n >>= 1, m >>= 1) {
        const bool up = lane & m;
#pragma unroll
        for (int i = 0; i < n / 2; ++i) {
            const float send = up ? s[i] : s[i + n / 2], keep = up ? s[i + n / 2] : s[i];
            s[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
        }
        if (up) which += n / 2;
    }
#pragma unroll
    for (; m > 0; m >>= 1) s[0] += __shfl_xor_sync(0xffffffffu, s[0], m);
    return s[0];
}

// mma.sync pieces: 8 x 8 tiles of bf16 from shared memory, 16 x 8 x 16 products, 16-byte asynchronous copies
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}

template <typename K, typename A>
static inline int launch_kernel(K kernel, dim3 grid, dim3 block, size_t smem, cudaStream_t st, int use_pdl, int cluster_x, const A& args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (use_pdl) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster_x > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = (unsigned)cluster_x;
        attr[n].val.clusterDim.y = 1;
        attr[n++].val.clusterDim.z = 1;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    return (int)cudaLaunchKernelEx(&cfg, kernel, args);
}
// Dynamic shared memory above 48 KB has to be asked for per kernel.
template <typename K>
static inline int allow_smem(K kernel, size_t bytes) {
    return bytes > 48 * 1024 ? (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) : 0;
}

}  // namespace tz
