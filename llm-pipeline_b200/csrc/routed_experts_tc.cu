// The experts' products for steps of many rows on the fifth-generation tensor cores (bfloat16).
//
//   sort:    one block puts the (token, choice) pairs in the order of their experts; every expert's run starts at a
//            multiple of 128 rows, so tile t is rows 128 t .. 128 t + 127 and has one expert. The places between an expert's
//            last pair and the next tile hold -1. Which place within its run a pair gets depends on the order of atomic
//            adds, but a row's result does not depend on its place.
//   gather:  the tokens' rows are copied into that order, so that a tile's rows are one TMA box.
//   products: persistent blocks, a tile of 128 rows by 256 weight rows at a time, as in gemm_tc.cu: one thread feeds a ring
//            of stages with TMA, one issues tcgen05.mma into one of two accumulators in tensor memory, four warps empty the
//            other. First product: the expert's up rows (or 128 gate rows and 128 up rows) with the activation and the
//            choice's weight as it is stored (y, bfloat16, in sorted order). Second product: y against the expert's down
//            rows, float32 at the pair's own place.
//   combine: out[token] = sum of its pairs' rows in the order of its choices.
//
// Every wait is bounded, as in gemm_tc.cu: when one runs out, *error_flag becomes 1 and the kernel returns in order.
#include "routed_experts.cuh"
#include "tcgen05.cuh"

namespace {

constexpr int MT_ROWS = 128;
constexpr int MT_COLS = 256;          // weight rows of a tile
constexpr int MT_BK = 64;
constexpr int MT_STAGES = 4;
constexpr int MT_THREADS = 192;

// One block. Shared: counts [E], cursor [E].
__global__ void __launch_bounds__(1024) moe_sort_kernel(const int* __restrict__ ids, int pairs, int E, int rows, int* __restrict__ sorted_pair,
                                                        int* __restrict__ tile_expert, int* __restrict__ num_tiles) {
    extern __shared__ int ms_smem[];
    __shared__ int warp_sums[32], carry;
    pdl_wait();
    pdl_trigger();
    int* counts = ms_smem;
    int* cursor = ms_smem + E;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    for (int e = tid; e < E; e += blockDim.x) counts[e] = 0;
    for (int i = tid; i < rows; i += blockDim.x) sorted_pair[i] = -1;
    if (tid == 0) carry = 0;
    __syncthreads();
    for (int i = tid; i < pairs; i += blockDim.x) {
        const int e = ids[i];
        if (e < E) atomicAdd(&counts[e], 1);             // identity experts (ids from E on) take no part
    }
    __syncthreads();
    for (int e0 = 0; e0 < E; e0 += blockDim.x) {         // first tile of every expert: a scan over the experts' tile counts
        const int e = e0 + tid;
        const int n = e < E ? counts[e] : 0;
        const int t = (n + MT_ROWS - 1) / MT_ROWS;
        int x = t;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int y = __shfl_up_sync(0xffffffffu, x, o);
            if (lane >= o) x += y;
        }
        if (lane == 31) warp_sums[warp] = x;
        __syncthreads();
        if (warp == 0) {
            int s = warp_sums[lane];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int y = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += y;
            }
            warp_sums[lane] = s;
        }
        __syncthreads();
        const int first = carry + x - t + (warp > 0 ? warp_sums[warp - 1] : 0);
        if (e < E) {
            cursor[e] = first * MT_ROWS;
            for (int k = 0; k < t; ++k) tile_expert[first + k] = e;
        }
        __syncthreads();
        if (tid == 0) carry += warp_sums[31];
        __syncthreads();
    }
    if (tid == 0) *num_tiles = carry;
    for (int i = tid; i < pairs; i += blockDim.x) {
        const int e = ids[i];
        if (e < E) sorted_pair[atomicAdd(&cursor[e], 1)] = i;
    }
}

// A warp per sorted row: the row of the pair's token.
__global__ void __launch_bounds__(128) moe_gather_kernel(const bf16* __restrict__ h, const int* __restrict__ sorted_pair,
                                                         const int* __restrict__ num_tiles, int top, int K, bf16* __restrict__ x) {
    pdl_wait();
    pdl_trigger();
    const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= *num_tiles * MT_ROWS) return;
    const int pair = sorted_pair[row];
    if (pair < 0) return;
    const uint4* src = reinterpret_cast<const uint4*>(h + (size_t)(pair / top) * K);
    uint4* dst = reinterpret_cast<uint4*>(x + (size_t)row * K);
#pragma unroll 4
    for (int i = lane; i < K / 8; i += 32) dst[i] = src[i];
}

struct MoeTcArgs {
    const int* sorted_pair; const int* tile_expert; const int* num_tiles;
    const float* wts;
    bf16* y;                  // first product's result [sorted rows, cols]
    float* out;               // second product's result [pairs, cols]
    int K, cols, form;
    float limit;
    int* error_flag;
};

template <bool FIRST, bool GATED>
__global__ void __launch_bounds__(MT_THREADS, 1)
moe_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b, const MoeTcArgs a) {
    extern __shared__ unsigned char mt_raw[];
    constexpr uint32_t A_BYTES = MT_ROWS * 128, B_BYTES = MT_COLS * 128, STAGE_BYTES = A_BYTES + B_BYTES;
    constexpr int OUT_COLS = GATED ? MT_COLS / 2 : MT_COLS;      // output columns of a tile
    __shared__ __align__(8) uint64_t full_bar[MT_STAGES], empty_bar[MT_STAGES], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_slot;
    const uint32_t raw_addr = tc_smem_u32(mt_raw);
    unsigned char* tiles = mt_raw + (((raw_addr + 1023u) & ~1023u) - raw_addr);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
#pragma unroll
        for (int s = 0; s < MT_STAGES; ++s) {
            mbar_init(&full_bar[s], 1);
            mbar_init(&empty_bar[s], 1);
        }
        mbar_init(&acc_full[0], 1);
        mbar_init(&acc_full[1], 1);
        mbar_init(&acc_empty[0], 4);
        mbar_init(&acc_empty[1], 4);
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(tc_smem_u32(&tmem_slot)), "r"(2u * MT_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    const uint32_t tmem_base = tmem_slot;
    pdl_wait();                                                  // what the kernels before wrote is complete
    pdl_trigger();
    const int m_tiles = *a.num_tiles, n_tiles = (a.cols + OUT_COLS - 1) / OUT_COLS;
    const int total = m_tiles * n_tiles;                         // in the order of the experts: what runs at one time shares rows and weights
    const int kblocks = (a.K + MT_BK - 1) / MT_BK;
    const int w_rows = (GATED ? 2 : 1) * a.cols;                 // weight rows of an expert

    if (warp == 0) {
        if (lane == 0) {
            int it = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
                const int m = tile / n_tiles, c0 = (tile % n_tiles) * OUT_COLS;
                const int b0 = a.tile_expert[m] * w_rows + c0;
                for (int kb = 0; kb < kblocks; ++kb, ++it) {
                    const int s = it % MT_STAGES;
                    if (it >= MT_STAGES && !mbar_wait(&empty_bar[s], ((it / MT_STAGES) - 1) & 1, a.error_flag)) { ok = false; break; }
                    mbar_expect_tx(&full_bar[s], STAGE_BYTES);
                    unsigned char* stage = tiles + (size_t)s * STAGE_BYTES;
                    tma_load_2d(stage, &map_a, kb * MT_BK, m * MT_ROWS, &full_bar[s]);
                    tma_load_2d(stage + A_BYTES, &map_b, kb * MT_BK, b0, &full_bar[s]);
                    if (GATED) tma_load_2d(stage + A_BYTES + B_BYTES / 2, &map_b, kb * MT_BK, b0 + a.cols, &full_bar[s]);
                }
            }
            // the copies of the last stages are over before the block may end
            for (int k = it > MT_STAGES ? it - MT_STAGES : 0; k < it; ++k) mbar_wait(&full_bar[k % MT_STAGES], (k / MT_STAGES) & 1, a.error_flag);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            int it = 0, n = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x, ++n) {
                const int c0 = (tile % n_tiles) * OUT_COLS;
                // a last tile of at most half the columns takes half the product (its other weight rows are another expert's)
                const uint32_t idesc = !GATED && a.cols - c0 <= MT_COLS / 2 ? umma_idesc(MT_ROWS, MT_COLS / 2) : umma_idesc(MT_ROWS, MT_COLS);
                const int acc = n & 1;
                if (n >= 2 && !mbar_wait(&acc_empty[acc], ((n >> 1) - 1) & 1, a.error_flag)) { ok = false; break; }
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                const uint32_t d_addr = tmem_base + (uint32_t)(acc * MT_COLS);
                for (int kb = 0; kb < kblocks; ++kb, ++it) {
                    const int s = it % MT_STAGES;
                    if (!mbar_wait(&full_bar[s], (it / MT_STAGES) & 1, a.error_flag)) { ok = false; break; }
                    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                    const uint32_t a_addr = tc_smem_u32(tiles + (size_t)s * STAGE_BYTES);
                    const uint64_t desc_a = umma_desc(a_addr), desc_b = umma_desc(a_addr + A_BYTES);
#pragma unroll
                    for (int k = 0; k < MT_BK / 16; ++k) umma_f16(d_addr, desc_a + 2 * k, desc_b + 2 * k, idesc, (kb | k) != 0 ? 1u : 0u);
                    umma_commit(&empty_bar[s]);
                }
                if (ok) umma_commit(&acc_full[acc]);
            }
        }
    } else {
        const int quarter = warp & 3;
        int n = 0;
        for (int tile = blockIdx.x; tile < total; tile += gridDim.x, ++n) {
            const int acc = n & 1;
            const int m = tile / n_tiles, c0 = (tile % n_tiles) * OUT_COLS;
            const int row = m * MT_ROWS + quarter * 32 + lane;
            const int pair = a.sorted_pair[row];
            const float w = FIRST && pair >= 0 ? a.wts[pair] : 0.f;
            if (!mbar_wait(&acc_full[acc], (n >> 1) & 1, a.error_flag)) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            const uint32_t t0 = tmem_base + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(acc * MT_COLS);
            const int cols = min(OUT_COLS, a.cols - c0);
#pragma unroll 4
            for (int c = 0; c < cols; c += 16) {
                float v[16];
                tmem_ld_16(t0 + (uint32_t)c, v);
                if (GATED) {
                    float u[16];
                    tmem_ld_16(t0 + (uint32_t)(OUT_COLS + c), u);
#pragma unroll
                    for (int j = 0; j < 16; ++j) v[j] = expert_act(v[j], u[j], w, a.limit, a.form);
                } else if (FIRST) {
#pragma unroll
                    for (int j = 0; j < 16; ++j) v[j] = expert_act(0.f, v[j], w, a.limit, EXPERT_FORM_UNGATED);
                }
                if (pair < 0) continue;
                if (FIRST) {
                    bf16* dst = a.y + (size_t)row * a.cols + c0 + c;
#pragma unroll
                    for (int j = 0; j < 16; j += 8) {            // the widths are multiples of 8
                        if (c + j < cols) {
                            const __nv_bfloat162 h0 = __floats2bfloat162_rn(v[j], v[j + 1]), h1 = __floats2bfloat162_rn(v[j + 2], v[j + 3]);
                            const __nv_bfloat162 h2 = __floats2bfloat162_rn(v[j + 4], v[j + 5]), h3 = __floats2bfloat162_rn(v[j + 6], v[j + 7]);
                            *reinterpret_cast<uint4*>(dst + j) = make_uint4(*reinterpret_cast<const unsigned*>(&h0), *reinterpret_cast<const unsigned*>(&h1),
                                                                           *reinterpret_cast<const unsigned*>(&h2), *reinterpret_cast<const unsigned*>(&h3));
                        }
                    }
                } else {
                    float* dst = a.out + (size_t)pair * a.cols + c0 + c;
#pragma unroll
                    for (int j = 0; j < 16; j += 4)
                        if (c + j < cols) *reinterpret_cast<float4*>(dst + j) = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(tc_smem_u32(&acc_empty[acc])) : "memory");
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem_base), "r"(2u * MT_COLS) : "memory");
    }
}

// A thread takes four entries of a token's row.
__global__ void __launch_bounds__(256) moe_combine4_kernel(const float4* __restrict__ pair_out, float4* __restrict__ out, int top, int Hd4,
                                                           size_t total, const int* __restrict__ ids, const float* __restrict__ wts,
                                                           const bf16* __restrict__ h, int E) {
    pdl_wait();
    pdl_trigger();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t n = i / Hd4, c = i % Hd4;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < top; ++k) {
        const size_t pair = n * top + k;
        float4 v;
        if (ids[pair] < E) {
            v = pair_out[pair * Hd4 + c];
        } else {                                         // identity expert: the weighted input
            const float w = wts[pair];
            const bf16* x = h + i * 4;
            v = make_float4(w * to_float(x[0]), w * to_float(x[1]), w * to_float(x[2]), w * to_float(x[3]));
        }
        s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
    }
    out[i] = s;
}

template <bool FIRST, bool GATED>
int launch_moe_tc(const bf16* A, long rows_a, const bf16* B, long rows_b, const MoeTcArgs& a, long tiles_max, cudaStream_t stream) {
    CUtensorMap map_a, map_b;
    if (llmp_matrix_tensor_map(A, rows_a, a.K, a.K, MT_ROWS, &map_a) ||
        llmp_matrix_tensor_map(B, rows_b, a.K, a.K, GATED ? MT_COLS / 2 : MT_COLS, &map_b)) return 1;
    constexpr size_t smem = (size_t)MT_STAGES * (MT_ROWS + MT_COLS) * 128 + 1024;
    LLMP_ALLOW_SMEM((moe_tc_kernel<FIRST, GATED>), smem);
    const int out_cols = GATED ? MT_COLS / 2 : MT_COLS;
    const long tiles = tiles_max * ((a.cols + out_cols - 1) / out_cols);
    const int sms = llmp_sm_count();
    llmp_launch_dependent(moe_tc_kernel<FIRST, GATED>, dim3((unsigned)(tiles < sms ? tiles : sms)), dim3(MT_THREADS), smem, stream, map_a, map_b, a);
    return 0;
}

}  // namespace

LLMP_API int llmp_expert_tc_supports(int Hd, int F) { return Hd % 8 == 0 && F % 8 == 0; }

// Rows of the sorted order for `pairs` pairs among E experts (every expert's run padded to a multiple of 128).
LLMP_API long llmp_expert_tc_rows(int pairs, int E) {
    const long tiles = (pairs + MT_ROWS - 1) / MT_ROWS + (E < pairs ? E : pairs);
    return tiles * MT_ROWS;
}

// ints: int32 scratch [1 + rows / 128 + rows]; x: bf16 [rows, Hd]; y: bf16 [rows, F]; pair_out: float32 [pairs, Hd].
LLMP_API int llmp_expert_tc(const void* h, const void* w_first, const void* w_down, const int* ids, const float* wts, float limit, int* ints,
                            void* x, void* y, float* pair_out, float* out, int N, int top, int Hd, int F, int E, int form, int identity,
                            int* error_flag, cudaStream_t stream) {
    if (N <= 0) return 0;
    LLMP_REQUIRE(llmp_expert_tc_supports(Hd, F) && top > 0 && E > 0 && E <= 8192 && error_flag && pair_out,
                 "expert_tc: sizes width=%d ff=%d experts=%d are not served", Hd, F, E);
    LLMP_REQUIRE(((size_t)h | (size_t)w_first | (size_t)w_down | (size_t)x | (size_t)y | (size_t)pair_out | (size_t)out) % 16 == 0,
                 "expert_tc: operands must be 16-byte aligned");
    (void)identity;
    const int pairs = N * top;
    const long rows = llmp_expert_tc_rows(pairs, E), tiles_max = rows / MT_ROWS;
    int* num_tiles = ints;
    int* tile_expert = ints + 1;
    int* sorted_pair = tile_expert + tiles_max;
    const size_t sort_smem = 2 * (size_t)E * sizeof(int);
    LLMP_ALLOW_SMEM(moe_sort_kernel, sort_smem);
    llmp_launch_dependent(moe_sort_kernel, dim3(1), dim3(1024), sort_smem, stream, ids, pairs, E, (int)rows, sorted_pair,
                          tile_expert, num_tiles);
    llmp_launch_dependent(moe_gather_kernel, dim3((unsigned)(rows / 4)), dim3(128), 0, stream, (const bf16*)h, (const int*)sorted_pair,
                          (const int*)num_tiles, top, Hd, (bf16*)x);
    MoeTcArgs a;
    a.sorted_pair = sorted_pair; a.tile_expert = tile_expert; a.num_tiles = num_tiles; a.wts = wts; a.y = (bf16*)y; a.out = pair_out;
    a.form = form; a.limit = limit; a.error_flag = error_flag;
    a.K = Hd; a.cols = F;
    const bool gated = form != EXPERT_FORM_UNGATED;
    const int rc = gated ? launch_moe_tc<true, true>((const bf16*)x, rows, (const bf16*)w_first, (long)E * 2 * F, a, tiles_max, stream)
                         : launch_moe_tc<true, false>((const bf16*)x, rows, (const bf16*)w_first, (long)E * F, a, tiles_max, stream);
    if (rc) return rc;
    a.K = F; a.cols = Hd;
    if (launch_moe_tc<false, false>((const bf16*)y, rows, (const bf16*)w_down, (long)E * Hd, a, tiles_max, stream)) return 1;
    const size_t total = (size_t)N * (Hd / 4);
    llmp_launch_dependent(moe_combine4_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream, (const float4*)pair_out, (float4*)out,
                          top, Hd / 4, total, ids, wts, (const bf16*)h, E);
    return llmp_check_launch("expert_tc");
}
