// bf16 matrix product on tcgen05 (kind::f16, fp32 accumulators in tensor memory) for 16 or more rows.
//
// The weight matrix is the MMA's M operand: a tile is 128 weight rows x up to 256 activation rows, so one kernel covers
// batched decode (few activation rows, the weights read once) and prefill. Persistent CTAs walk the work units; warp 0
// loads both K-major operands by TMA (128-byte swizzle, 64 values of K per stage), warp 1 issues the MMAs, warps 2-5
// run the epilogue of one unit out of one half of tensor memory while the MMAs of the next fill the other half.
//
// When the tiles alone would leave most SMs idle, K is split: every unit stores its partial tile to the workspace, and
// the CTA that finishes a tile last adds the partials in split order (a counter decides, nobody waits), so results do
// not depend on timing.
#include <algorithm>
#include <cmath>

#include "hybrid_common.cuh"
#include "umma.cuh"

namespace tz {

constexpr int kGuThreads = 192, kGuStages = 4, kGuKc = 64, kGuRows = 128, kGuMaxN = 256;
constexpr int kGuSplitTiles = 148, kGuMaxSplit = 16;         // split K only below this many tiles

__device__ int g_gu_timeouts = 0;

struct GuLaunch {
    GemmArgs a;
    int n_tiles, m_tiles, n_split, n_box, tmem_half, chunks, chunks_per_split, a_seg_rows;
    float* partial;              // [tile][split][n_box][128]
    unsigned* counters;          // [tile]
};

struct GuSmem {
    static __host__ __device__ int stage_bytes(int n_box) { return (kGuRows + n_box) * 128; }
    static constexpr int n_bars = 2 * kGuStages + 4;
    static __host__ __device__ size_t bytes(int n_box) { return 1024 + (size_t)kGuStages * stage_bytes(n_box) + 8 * n_bars + 64; }
};

__device__ __forceinline__ void umma_bf16(uint32_t tmem_d, uint64_t da, uint64_t db, uint32_t idesc, uint32_t accumulate) {
    asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
                 ::"r"(tmem_d), "l"(da), "l"(db), "r"(idesc), "r"(accumulate) : "memory");
}

// Sixteen rows of column n, rows m0 .. below m_end. All lanes of the warp call it (the two halves of a GLU pair are neighbours).
__device__ __forceinline__ void gu_store16(const GemmArgs& a, int n, int m0, int m_end, const float (&v)[16]) {
    if (a.epilogue == TENZO_GEMM_GLU_RELU || a.epilogue == TENZO_GEMM_GLU_SILU) {
        const bool up = threadIdx.x & 1;                       // the even lane finishes eight rows, the odd one the others
        float g[8], u[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float other = __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + 8], 1);
            g[i] = up ? other : v[i];
            u[i] = up ? v[i + 8] : other;
        }
        if (n >= a.N) return;
        bf16* c = reinterpret_cast<bf16*>(a.c) + n / 2;
        const int m1 = m0 + (up ? 8 : 0);
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (m1 + i < m_end) c[(size_t)(m1 + i) * a.ld_c] = __float2bfloat16_rn(glu_f(a.epilogue, g[i], u[i]));
        return;
    }
    if (n >= a.N) return;
    if (a.epilogue == TENZO_GEMM_XIELU || a.epilogue == TENZO_GEMM_CAST) {
        bf16* c = reinterpret_cast<bf16*>(a.c) + n;
        const bool act = a.epilogue == TENZO_GEMM_XIELU;
#pragma unroll
        for (int i = 0; i < 16; ++i)
            if (m0 + i < m_end) c[(size_t)(m0 + i) * a.ld_c] = __float2bfloat16_rn(act ? xielu_f(v[i], a.act_pos, a.act_neg) : v[i]);
    } else {
        float* c = reinterpret_cast<float*>(a.c) + n;
        const bool cap = a.epilogue == TENZO_GEMM_SOFTCAP;
#pragma unroll
        for (int i = 0; i < 16; ++i)
            if (m0 + i < m_end) c[(size_t)(m0 + i) * a.ld_c] = cap ? soft_cap_f(v[i], a.cap) : v[i];
    }
}

// A unit of work: a weight tile against a tile of activation rows, over a part of K.
struct GuUnit {
    int row_w, row_a, n0;        // first row of the weight tile and of the activation tile in their tensor maps; its first column
    int m0, m_end;               // first output row, end of the rows that may be stored
    int split, tile;
};
// Unit u of the launch, false past the last one. Every role walks its units in ascending order; in the grouped form the
// number of row tiles of a group is read as the walk reaches it.
struct GuWalk {
    int g = 0, base = 0, lo = 0, hi = -1;
    __device__ __forceinline__ bool at(const GuLaunch& L, int u, GuUnit& o) {
        const GemmArgs& a = L.a;
        if (!a.group_off) {
            if (u >= L.n_tiles * L.m_tiles * L.n_split) return false;
            // consecutive units share the activation rows
            const int nt = (u / L.n_split) % L.n_tiles, mt = u / (L.n_split * L.n_tiles);
            o.split = u % L.n_split;
            o.tile = mt * L.n_tiles + nt;
            o.n0 = o.row_w = nt * kGuRows;
            int seg = 0;
            if (a.seg_rows > 0) seg = o.row_w / a.seg_rows;
            else
                while (seg + 1 < a.n_seg && o.row_w >= a.seg_end[seg]) ++seg;
            o.row_a = seg * L.a_seg_rows + mt * L.n_box;
            o.m0 = mt * L.n_box;
            o.m_end = a.M;
            return true;
        }
        for (;; ++g, hi = -1) {
            if (g >= a.n_group) return false;
            if (hi < 0) {
                lo = a.group_off[g];
                hi = min(a.M, a.group_off[g + 1]);
            }
            const int n = (hi - lo + L.n_box - 1) / L.n_box * L.n_tiles;
            if (u < base + n) break;
            base += n;
        }
        const int nt = (u - base) % L.n_tiles, mt = (u - base) / L.n_tiles;
        o.split = o.tile = 0;
        o.n0 = nt * kGuRows;
        o.row_w = g * a.N + o.n0;
        o.row_a = o.m0 = lo + mt * L.n_box;
        o.m_end = hi;
        return true;
    }
};

__global__ void __launch_bounds__(kGuThreads, 1) gemm_umma_kernel(const GuLaunch L, const __grid_constant__ CUtensorMap wmap,
                                                                  const __grid_constant__ CUtensorMap amap) {
    extern __shared__ unsigned char smem_raw[];
    const uint32_t base_off = ((smem_addr(smem_raw) + 1023u) & ~1023u) - smem_addr(smem_raw);
    unsigned char* stages = smem_raw + base_off;
    const int N = L.n_box, stage_bytes = GuSmem::stage_bytes(N);
    uint64_t* bars = reinterpret_cast<uint64_t*>(stages + (size_t)kGuStages * stage_bytes);
    uint64_t *bar_full = bars, *bar_empty = bars + kGuStages, *bar_acc_full = bars + 2 * kGuStages, *bar_acc_empty = bar_acc_full + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + GuSmem::n_bars);
    int* s_last = reinterpret_cast<int*>(tmem_slot + 1);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;

    if (tid == 0) {
        for (int s = 0; s < kGuStages; ++s) { mbar_init(&bar_full[s], 1); mbar_init(&bar_empty[s], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&bar_acc_full[i], 1); mbar_init(&bar_acc_empty[i], 4); }
        mbar_init_fence();
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(tmem_slot)), "r"(2 * L.tmem_half) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(tmem_slot);
    pdl_wait();
    pdl_launch_dependents();
    bool timed_out = false;

    GuWalk walk;
    GuUnit t = {};
    auto k_begin = [&]() { return t.split * L.chunks_per_split; };
    auto k_end = [&]() { return min(L.chunks, k_begin() + L.chunks_per_split); };

    if (warp == 0) {
        if (lane == 0) {
            int it = 0;
            for (int u = blockIdx.x; !timed_out && walk.at(L, u, t); u += gridDim.x) {
                for (int j = k_begin(); j < k_end(); ++j, ++it) {
                    const int s = it % kGuStages, use = it / kGuStages;
                    if (use > 0 && !mbar_spin_bounded(&bar_empty[s], (unsigned)(use - 1) & 1u)) { timed_out = true; break; }
                    unsigned char* sp = stages + (size_t)s * stage_bytes;
                    mbar_expect_tx(&bar_full[s], (unsigned)stage_bytes);
                    tma_load_2d(sp, &wmap, j * kGuKc, t.row_w, &bar_full[s]);
                    tma_load_2d(sp + kGuRows * 128, &amap, j * kGuKc, t.row_a, &bar_full[s]);
                }
            }
            if (timed_out)                                     // shared memory must outlive the copies in flight
                for (int j = it > kGuStages ? it - kGuStages : 0; j < it; ++j) mbar_spin_bounded(&bar_full[j % kGuStages], (unsigned)(j / kGuStages) & 1u);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            // d = f32, a = b = bf16, both K-major, N at bit 17 (>>3), M at bit 24 (>>4)
            const uint32_t idesc0 = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kGuRows >> 4) << 24);
            int it = 0, n = 0;
            for (int u = blockIdx.x; !timed_out && walk.at(L, u, t); u += gridDim.x, ++n) {
                const int half = n & 1, use_acc = n >> 1;
                if (use_acc > 0 && !mbar_spin_bounded(&bar_acc_empty[half], (unsigned)(use_acc - 1) & 1u)) { timed_out = true; break; }
                tc_fence_after();
                const uint32_t d = tmem_base + (uint32_t)(half * L.tmem_half);
                const uint32_t idesc = idesc0 | ((uint32_t)(min(N, (t.m_end - t.m0 + 15) & ~15) >> 3) << 17);      // only rows that exist
                uint32_t acc = 0;
                for (int j = k_begin(); j < k_end(); ++j, ++it) {
                    const int s = it % kGuStages, use = it / kGuStages;
                    if (!mbar_spin_bounded(&bar_full[s], (unsigned)use & 1u)) { timed_out = true; break; }
                    tc_fence_after();
                    const uint32_t sa = smem_addr(stages + (size_t)s * stage_bytes);
                    const uint64_t da = umma_desc_sw128(sa), db = umma_desc_sw128(sa + kGuRows * 128);
#pragma unroll
                    for (int k4 = 0; k4 < kGuKc / 16; ++k4) {
                        umma_bf16(d, da + (uint64_t)(2 * k4), db + (uint64_t)(2 * k4), idesc, acc);
                        acc = 1;
                    }
                    umma_commit(&bar_empty[s]);
                }
                umma_commit(&bar_acc_full[half]);
            }
        }
    } else {
        const int q = warp & 3, row = 32 * q + lane;
        int n = 0;
        for (int u = blockIdx.x; walk.at(L, u, t); u += gridDim.x, ++n) {
            const int half = n & 1, use_acc = n >> 1;
            bool ok = true;
            if (lane == 0) ok = mbar_spin_bounded(&bar_acc_full[half], (unsigned)use_acc & 1u);
            ok = __shfl_sync(0xffffffffu, ok, 0);
            // a give-up is only flagged: the four warps keep the same barrier sequence whatever each of them saw
            if (!ok) timed_out = true;
            tc_fence_after();
            const uint32_t d = tmem_base + ((uint32_t)(32 * q) << 16) + (uint32_t)(half * L.tmem_half);
            const int n_row = t.n0 + row, m0 = t.m0, tile = t.tile;
            float* part = L.n_split > 1 ? L.partial + ((size_t)tile * L.n_split + t.split) * N * kGuRows : nullptr;
            for (int c0 = 0; c0 < N && m0 + c0 < t.m_end; c0 += 16) {
                uint32_t r[16];
                float v[16];
                tmem_ld16(d + (uint32_t)c0, r);
#pragma unroll
                for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
                if (part) {
#pragma unroll
                    for (int i = 0; i < 16; ++i) __stcg(part + (size_t)(c0 + i) * kGuRows + row, v[i]);
                } else {
                    gu_store16(L.a, n_row, m0 + c0, t.m_end, v);
                }
            }
            tc_fence_before();
            if (lane == 0) mbar_arrive(&bar_acc_empty[half]);
            if (part) {
                __threadfence();
                named_barrier_sync(1, 128);
                if (tid == 64) *s_last = atomicAdd(&L.counters[tile], 1u) == (unsigned)(L.n_split - 1);
                named_barrier_sync(1, 128);
                if (*s_last) {
                    __threadfence();
                    const float* base = L.partial + (size_t)tile * L.n_split * N * kGuRows + row;
                    for (int c0 = 0; c0 < N && m0 + c0 < L.a.M; c0 += 16) {
                        float v[16] = {};
                        for (int s = 0; s < L.n_split; ++s)
#pragma unroll
                            for (int i = 0; i < 16; ++i) v[i] += __ldcg(base + ((size_t)s * N + c0 + i) * kGuRows);
                        gu_store16(L.a, n_row, m0 + c0, t.m_end, v);
                    }
                    if (tid == 64) L.counters[tile] = 0;      // ready for the next launch
                }
                named_barrier_sync(1, 128);                     // s_last is reused
            }
        }
    }
    if (timed_out) atomicExch(&g_gu_timeouts, 1);
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(2 * L.tmem_half) : "memory");
    }
}

constexpr size_t kGuCounterBytes = 4096;
constexpr size_t kGuWorkspaceBytes = kGuCounterBytes + (size_t)kGuSplitTiles * kGuMaxN * kGuRows * 4;

bool gemm_umma_applicable(const GemmArgs& a) {
    if (a.f32 || a.M < kGemmUmmaMinRows || a.ld_k % kGuKc || !a.workspace) return false;
    if (a.group_off) return !a.a_index || a.a_gather;
    if (a.seg_rows > 0) return a.seg_rows % kGuRows == 0 && a.a_seg_stride % a.ld_k == 0;
    for (int s = 0; s + 1 < a.n_seg; ++s)
        if (a.seg_end[s] % kGuRows) return false;
    return a.n_seg == 1 || a.a_seg_stride % a.ld_k == 0;
}

int launch_gemm_umma(const GemmArgs& a, cudaStream_t st) {
    GuLaunch L;
    L.a = a;
    // grouped: equal tiles that cover a group somewhat larger than the mean
    const int mean = a.group_off ? std::max(1, a.M / a.n_group) : 0, rows = a.group_off ? std::min(a.M, mean + 2 * (int)std::sqrt((double)mean)) : a.M;
    L.n_box = a.group_off ? round_up((rows + (rows + kGuMaxN - 1) / kGuMaxN - 1) / ((rows + kGuMaxN - 1) / kGuMaxN), 16) : std::min(kGuMaxN, round_up(rows, 16));
    L.tmem_half = 32;
    while (L.tmem_half < L.n_box) L.tmem_half *= 2;
    L.n_tiles = (a.N + kGuRows - 1) / kGuRows;
    L.m_tiles = (a.M + L.n_box - 1) / L.n_box;
    L.chunks = a.ld_k / kGuKc;
    const int n_seg = a.seg_rows > 0 ? (a.N + a.seg_rows - 1) / a.seg_rows : a.n_seg;
    L.a_seg_rows = n_seg > 1 ? (int)(a.a_seg_stride / a.ld_k) : 0;
    const int tiles = a.group_off ? L.n_tiles * (L.m_tiles + a.n_group) : L.n_tiles * L.m_tiles;      // grouped: at most
    int split = 1;
    if (!a.group_off && tiles <= kGuSplitTiles / 2 && tiles * sizeof(unsigned) <= kGuCounterBytes)
        split = std::max(1, std::min({kGuMaxSplit, kGuSplitTiles / tiles, L.chunks / 2}));
    L.chunks_per_split = (L.chunks + split - 1) / split;
    L.n_split = (L.chunks + L.chunks_per_split - 1) / L.chunks_per_split;
    L.counters = static_cast<unsigned*>(a.workspace);
    L.partial = reinterpret_cast<float*>(static_cast<char*>(a.workspace) + kGuCounterBytes);
    if (L.n_split > 1 && kGuCounterBytes + (size_t)tiles * L.n_split * L.n_box * kGuRows * 4 > a.workspace_bytes) return -1;
    CUtensorMap wmap, amap;
    if (int rc = encode_2d(&wmap, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, a.w, (uint64_t)a.ld_k, (uint64_t)a.N * (a.group_off ? a.n_group : 1), (uint64_t)a.ld_k * 2, kGuKc, kGuRows,
                           CU_TENSOR_MAP_SWIZZLE_128B)) return rc;
    const uint64_t a_rows = n_seg > 1 ? (uint64_t)(n_seg - 1) * L.a_seg_rows + a.M : (uint64_t)a.M;
    if (int rc = encode_2d(&amap, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, a.a, (uint64_t)a.ld_k, a_rows, (uint64_t)a.ld_k * 2, kGuKc, (uint32_t)L.n_box,
                           CU_TENSOR_MAP_SWIZZLE_128B)) return rc;
    const size_t smem = GuSmem::bytes(L.n_box);
    cudaError_t e = cudaFuncSetAttribute(gemm_umma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)std::min(148, tiles * L.n_split));
    cfg.blockDim = dim3(kGuThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = a.use_pdl ? 1 : 0;
    return (int)cudaLaunchKernelEx(&cfg, gemm_umma_kernel, L, wmap, amap);
}

}  // namespace tz

extern "C" size_t tenzo_cuda_gemm_workspace_bytes(void) { return tz::kGuWorkspaceBytes; }

extern "C" int tenzo_cuda_gemm_take_timeouts(void) {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, tz::g_gu_timeouts, sizeof v) != cudaSuccess) return -1;
    if (v) cudaMemcpyToSymbol(tz::g_gu_timeouts, &zero, sizeof zero);
    return v;
}
