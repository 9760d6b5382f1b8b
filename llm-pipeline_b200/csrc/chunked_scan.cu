// The recurrences of state_space.cu for the many tokens of a prompt portion, in chunks on the tensor cores (bfloat16 path).
//
//   S_t = a_t S_(t-1) + w_t b_t x_t^T,   y_t = S_t^T c_t + skip x_t
// with b, c of N entries, x of P and the scalar a_t = exp(l_t): the state-space recurrence (l_t = -exp(A_log) w_t with
// w_t = softplus(dt + bias)), or one with a constant decay per head and w_t = 1 (retention: keys, queries, values). With
// L_i the sum of l over the chunk's tokens up to i and S the state before the chunk, a chunk of up to 128 tokens is
//   y_i = exp(L_i) S^T c_i + sum_(j <= i) (c_i . b_j) exp(L_i - L_j) w_j x_j + skip x_i
//   S' = exp(L_last) S + sum_j exp(L_last - L_j) w_j b_j x_j^T
// Three launches, every chunk of every request side by side in the first and the third:
//   1. each chunk's own sum over j (the second term of S'), float32, to scratch;
//   2. along the chunks of a request: scratch becomes the state before each chunk; the last state goes to the slot;
//   3. the outputs.
// b, c, x are bfloat16 (projections and short convolutions); decays, step sizes, scores and their weights, states and sums
// are float32. Where a float32 number enters a product it is split into two bfloat16 halves (16 bits of mantissa) and both
// are multiplied. Nothing of a chunk depends on other requests; chunks are counted from a portion's first token.
#include "common.cuh"

namespace {

constexpr int CS_TOKENS = 128;        // tokens of a chunk
constexpr int CS_COLS = 64;           // columns of x a block takes
constexpr int CS_XS = CS_COLS + 8;    // entries of a row of x in shared memory
constexpr int CS_THREADS = 256;

struct ChunkArgs {
    const bf16* b; const bf16* c; const bf16* x; long row_t;
    const float* dt; long dt_t; const float* dt_bias; const float* a_log; const float* d_skip;   // null with constant decays
    const float* log_decay;                                                                      // [H], or null
    const int* chunks;                // [chunks][2]: first row, tokens
    float* sums; float* gains;        // [chunks][H][N][P], [chunks][H]
    float* y; long y_t;
    int H, G, N, P;
};

__device__ __forceinline__ unsigned cs_smem(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cs_copy16(void* dst, const void* src, bool valid) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(cs_smem(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cs_wait() { asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;\n" ::: "memory"); }
__device__ __forceinline__ void cs_ld4(unsigned (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(cs_smem(p)) : "memory");
}
__device__ __forceinline__ void cs_ld4_t(unsigned (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(cs_smem(p)) : "memory");
}
__device__ __forceinline__ void cs_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two floats as a pair of bfloat16, and what that leaves of them as another pair.
__device__ __forceinline__ void cs_split(float u, float v, unsigned& hi, unsigned& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(u, v);
    const __nv_bfloat162 l = __floats2bfloat162_rn(u - __low2float(h), v - __high2float(h));
    hi = *reinterpret_cast<const unsigned*>(&h);
    lo = *reinterpret_cast<const unsigned*>(&l);
}

__device__ __forceinline__ float cs_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// cum[t]: the sum of the log decays up to and with token t; w[t]: the input's factor (0 past the chunk's tokens).
__device__ __forceinline__ void chunk_weights(const ChunkArgs& a, int h, int row0, int cnt, float* cum, float* w, float* part) {
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5;
    float l = 0.f;
    if (t < CS_TOKENS) {
        float wt = 0.f;
        if (t < cnt) {
            if (a.log_decay) {
                l = a.log_decay[h];
                wt = 1.f;
            } else {
                wt = cs_softplus(a.dt[(size_t)(row0 + t) * a.dt_t + h] + a.dt_bias[h]);
                l = -expf(a.a_log[h]) * wt;
            }
        }
        w[t] = wt;
        if (a.log_decay) {
            cum[t] = l = (float)min(t + 1, cnt) * a.log_decay[h];
        } else {
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, l, o);
                if (lane >= o) l += up;
            }
            if (lane == 31) part[warp] = l;
        }
    }
    __syncthreads();
    if (t < CS_TOKENS && !a.log_decay) {
        for (int k = 0; k < warp; ++k) l += part[k];
        cum[t] = l;
    }
    __syncthreads();
}

// rows [cnt of CS_TOKENS][n] of a bfloat16 matrix into shared memory with `stride` entries a row; the rest is zero
__device__ __forceinline__ void chunk_rows(bf16* dst, int stride, const bf16* src, long row_t, int cnt, int n, int pad_to) {
    const int pieces = pad_to >> 3;
    for (int i = threadIdx.x; i < CS_TOKENS * pieces; i += CS_THREADS) {
        const int t = i / pieces, e = (i % pieces) * 8;
        const bool valid = t < cnt && e < n;
        cs_copy16(dst + t * stride + e, valid ? src + (size_t)t * row_t + e : src, valid);
    }
}

// ---- 1: sums[chunk][h] = sum_j exp(L_last - L_j) w_j b_j x_j^T ---------------------------------------------------------
__global__ void __launch_bounds__(CS_THREADS) chunk_sums_kernel(const ChunkArgs a) {
    extern __shared__ __align__(16) unsigned char cs_raw[];
    __shared__ float cum[CS_TOKENS], w[CS_TOKENS], part[4];
    const int chunk = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * CS_COLS;
    const int row0 = a.chunks[2 * chunk], cnt = a.chunks[2 * chunk + 1];
    const int N = a.N, P = a.P, ns = N + 8, g = h / (a.H / a.G);
    bf16* bs = reinterpret_cast<bf16*>(cs_raw);                   // [CS_TOKENS][ns]
    bf16* xh = bs + CS_TOKENS * ns;                               // [CS_TOKENS][CS_XS]: the scaled x, its two halves
    bf16* xl = xh + CS_TOKENS * CS_XS;
    chunk_rows(bs, ns, a.b + (size_t)row0 * a.row_t + (size_t)g * N, a.row_t, cnt, N, N);
    chunk_weights(a, h, row0, cnt, cum, w, part);
    const float last = cum[CS_TOKENS - 1];
    if (threadIdx.x == 0 && blockIdx.z == 0) a.gains[(size_t)chunk * a.H + h] = expf(last);
    const int ncols = min(CS_COLS, P - j0);
    const bf16* x = a.x + (size_t)row0 * a.row_t + (size_t)h * P + j0;
    for (int i = threadIdx.x; i < CS_TOKENS * (CS_COLS / 8); i += CS_THREADS) {
        const int t = i / (CS_COLS / 8), e = (i % (CS_COLS / 8)) * 8;
        uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
        if (t < cnt && e < ncols) {
            const uint4 raw = *reinterpret_cast<const uint4*>(x + (size_t)t * a.row_t + e);
            const __nv_bfloat162* v = reinterpret_cast<const __nv_bfloat162*>(&raw);
            const float f = expf(last - cum[t]) * w[t];
            cs_split(__low2float(v[0]) * f, __high2float(v[0]) * f, hi.x, lo.x);
            cs_split(__low2float(v[1]) * f, __high2float(v[1]) * f, hi.y, lo.y);
            cs_split(__low2float(v[2]) * f, __high2float(v[2]) * f, hi.z, lo.z);
            cs_split(__low2float(v[3]) * f, __high2float(v[3]) * f, hi.w, lo.w);
        }
        *reinterpret_cast<uint4*>(xh + t * CS_XS + e) = hi;
        *reinterpret_cast<uint4*>(xl + t * CS_XS + e) = lo;
    }
    cs_wait();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, q = lane >> 3, r = lane & 7;
    const int steps = (cnt + 15) >> 4;
    float* out = a.sums + ((size_t)chunk * a.H + h) * N * P + j0;
    // an item is 16 rows of the state and half of the block's columns
    for (int item = warp; item < (N >> 4) * 2; item += CS_THREADS / 32) {
        const int m0 = (item >> 1) * 16, n0 = (item & 1) * (CS_COLS / 2);
        if (n0 >= ncols) continue;
        float acc[4][4] = {};
        for (int k = 0; k < steps; ++k) {
            unsigned at[4];
            cs_ld4_t(at, bs + (k * 16 + (q >> 1) * 8 + r) * ns + m0 + (q & 1) * 8);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                unsigned bh[4], bl[4];
                const int at_x = (k * 16 + (q & 1) * 8 + r) * CS_XS + n0 + n * 16 + (q >> 1) * 8;
                cs_ld4_t(bh, xh + at_x);
                cs_ld4_t(bl, xl + at_x);
                cs_mma(acc[2 * n], at, bh[0], bh[1]);
                cs_mma(acc[2 * n + 1], at, bh[2], bh[3]);
                cs_mma(acc[2 * n], at, bl[0], bl[1]);
                cs_mma(acc[2 * n + 1], at, bl[2], bl[3]);
            }
        }
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            const int col = n0 + n * 8 + (lane & 3) * 2;
            if (col >= ncols) continue;
            float* o = out + (size_t)(m0 + (lane >> 2)) * P + col;
            *reinterpret_cast<float2*>(o) = make_float2(acc[n][0], acc[n][1]);
            *reinterpret_cast<float2*>(o + (size_t)8 * P) = make_float2(acc[n][2], acc[n][3]);
        }
    }
}

// ---- 2: along a request's chunks, sums becomes the state before each chunk ---------------------------------------------
__global__ void __launch_bounds__(256) chunk_states_kernel(float* sums, const float* gains, const int* requests, float* state, long state_slot,
                                                           long state_half, const int* q_start, const int* slots, const int* positions,
                                                           int H, int per) {
    const int r = requests[3 * blockIdx.z], first = requests[3 * blockIdx.z + 1], count = requests[3 * blockIdx.z + 2];
    const int h = blockIdx.y, i = (blockIdx.x * 256 + threadIdx.x) * 4;        // per = N P entries of a head's state
    if (i >= per) return;
    const int begin = q_start[r], p0 = positions[begin], last = p0 + q_start[r + 1] - begin - 1;
    float* slot = state + (size_t)slots[r] * state_slot + (size_t)h * per + i;
    float4 S = *reinterpret_cast<const float4*>(slot + ((p0 + 1) & 1) * state_half);
    const size_t step = (size_t)H * per;
    float* at = sums + ((size_t)first * H + h) * per + i;
    constexpr int AHEAD = 4;
    float4 next[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
        if (k < count) next[k] = *reinterpret_cast<const float4*>(at + k * step);
    for (int c = 0; c < count; c += AHEAD) {
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            if (c + k >= count) break;
            const float4 own = next[k];
            if (c + k + AHEAD < count) next[k] = *reinterpret_cast<const float4*>(at + (c + k + AHEAD) * step);
            const float g = gains[(size_t)(first + c + k) * H + h];
            *reinterpret_cast<float4*>(at + (c + k) * step) = S;
            S = make_float4(fmaf(g, S.x, own.x), fmaf(g, S.y, own.y), fmaf(g, S.z, own.z), fmaf(g, S.w, own.w));
        }
    }
    *reinterpret_cast<float4*>(slot + (last & 1) * state_half) = S;
}

// ---- 3: outputs --------------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(CS_THREADS) chunk_outputs_kernel(const ChunkArgs a) {
    extern __shared__ __align__(16) unsigned char cs_raw[];
    __shared__ float cum[CS_TOKENS], w[CS_TOKENS], part[4];
    const int chunk = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * CS_COLS;
    const int row0 = a.chunks[2 * chunk], cnt = a.chunks[2 * chunk + 1];
    const int N = a.N, P = a.P, ns = N + 8, g = h / (a.H / a.G);
    const int ncols = min(CS_COLS, P - j0);
    bf16* cs = reinterpret_cast<bf16*>(cs_raw);                   // [CS_TOKENS][ns]
    bf16* sh = cs + CS_TOKENS * ns;                               // first [N][CS_XS] twice: the state's two halves
    bf16* sl = sh + N * CS_XS;
    bf16* bs = sh;                                                // then [CS_TOKENS][ns] and [CS_TOKENS][CS_XS]: b and x
    bf16* xs = bs + CS_TOKENS * ns;
    chunk_rows(cs, ns, a.c + (size_t)row0 * a.row_t + (size_t)g * N, a.row_t, cnt, N, N);
    const float* S = a.sums + ((size_t)chunk * a.H + h) * N * P + j0;
    for (int i = threadIdx.x; i < N * (CS_COLS / 4); i += CS_THREADS) {
        const int n = i / (CS_COLS / 4), e = (i % (CS_COLS / 4)) * 4;
        uint2 hi = make_uint2(0, 0), lo = hi;
        if (e < ncols) {
            const float4 v = *reinterpret_cast<const float4*>(S + (size_t)n * P + e);
            cs_split(v.x, v.y, hi.x, lo.x);
            cs_split(v.z, v.w, hi.y, lo.y);
        }
        *reinterpret_cast<uint2*>(sh + n * CS_XS + e) = hi;
        *reinterpret_cast<uint2*>(sl + n * CS_XS + e) = lo;
    }
    chunk_weights(a, h, row0, cnt, cum, w, part);
    cs_wait();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, q = lane >> 3, r = lane & 7;
    const int i0 = warp * 16, ia = i0 + (lane >> 2), ib = ia + 8;
    const bool busy = i0 < cnt;
    float o[8][4] = {};
    if (busy) {
        for (int k = 0; k < N; k += 16) {
            unsigned ac[4];
            cs_ld4(ac, cs + (i0 + (q & 1) * 8 + r) * ns + k + (q >> 1) * 8);
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                unsigned bh[4], bl[4];
                const int at = (k + (q & 1) * 8 + r) * CS_XS + n * 16 + (q >> 1) * 8;
                cs_ld4_t(bh, sh + at);
                cs_ld4_t(bl, sl + at);
                cs_mma(o[2 * n], ac, bh[0], bh[1]);
                cs_mma(o[2 * n + 1], ac, bh[2], bh[3]);
                cs_mma(o[2 * n], ac, bl[0], bl[1]);
                cs_mma(o[2 * n + 1], ac, bl[2], bl[3]);
            }
        }
        const float ea = expf(cum[ia]), eb = expf(cum[ib]);
#pragma unroll
        for (int n = 0; n < 8; ++n) { o[n][0] *= ea; o[n][1] *= ea; o[n][2] *= eb; o[n][3] *= eb; }
    }
    __syncthreads();                                              // the state's place is free
    chunk_rows(bs, ns, a.b + (size_t)row0 * a.row_t + (size_t)g * N, a.row_t, cnt, N, N);
    chunk_rows(xs, CS_XS, a.x + (size_t)row0 * a.row_t + (size_t)h * P + j0, a.row_t, cnt, ncols, CS_COLS);
    cs_wait();
    __syncthreads();
    if (!busy) return;
    const float ca = cum[ia], cb = cum[ib];
    for (int t0 = 0; t0 <= i0; t0 += 64) {                        // 64 tokens of the chunk at a time, those not after the warp's rows
        float s[8][4] = {};
        const int pairs = min(4, (i0 + 16 - t0 + 15) >> 4);       // runs of 16 tokens that some row sees
        for (int k = 0; k < N; k += 16) {
            unsigned ac[4];
            cs_ld4(ac, cs + (i0 + (q & 1) * 8 + r) * ns + k + (q >> 1) * 8);
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                if (n >= pairs) break;
                unsigned b[4];
                cs_ld4(b, bs + (t0 + n * 16 + (q >> 1) * 8 + r) * ns + k + (q & 1) * 8);
                cs_mma(s[2 * n], ac, b[0], b[1]);
                cs_mma(s[2 * n + 1], ac, b[2], b[3]);
            }
        }
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            const int j = t0 + n * 8 + (lane & 3) * 2;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float cj = cum[j + e], wj = w[j + e];
                s[n][e] = j + e <= ia ? s[n][e] * (expf(ca - cj) * wj) : 0.f;
                s[n][2 + e] = j + e <= ib ? s[n][2 + e] * (expf(cb - cj) * wj) : 0.f;
            }
        }
#pragma unroll
        for (int m = 0; m < 4; ++m) {
            if (m >= pairs) break;
            unsigned ph[4], pl[4];
            cs_split(s[2 * m][0], s[2 * m][1], ph[0], pl[0]);
            cs_split(s[2 * m][2], s[2 * m][3], ph[1], pl[1]);
            cs_split(s[2 * m + 1][0], s[2 * m + 1][1], ph[2], pl[2]);
            cs_split(s[2 * m + 1][2], s[2 * m + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                unsigned b[4];
                cs_ld4_t(b, xs + (t0 + m * 16 + (q & 1) * 8 + r) * CS_XS + n * 16 + (q >> 1) * 8);
                cs_mma(o[2 * n], ph, b[0], b[1]);
                cs_mma(o[2 * n + 1], ph, b[2], b[3]);
                cs_mma(o[2 * n], pl, b[0], b[1]);
                cs_mma(o[2 * n + 1], pl, b[2], b[3]);
            }
        }
    }
    const float skip = a.d_skip ? a.d_skip[h] : 0.f;
    float* y = a.y + (size_t)row0 * a.y_t + (size_t)h * P + j0;
#pragma unroll
    for (int n = 0; n < 8; ++n) {
        const int col = n * 8 + (lane & 3) * 2;
        if (col >= ncols) continue;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = e ? ib : ia;
            if (i >= cnt) continue;
            const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(xs + i * CS_XS + col);
            *reinterpret_cast<float2*>(y + (size_t)i * a.y_t + col) =
                make_float2(fmaf(skip, __low2float(x), o[n][2 * e]), fmaf(skip, __high2float(x), o[n][2 * e + 1]));
        }
    }
}

}  // namespace

// chunks [n_chunks][2]: (first row, tokens); requests [n_requests][3]: (request, its first chunk, its chunks). sums and gains:
// scratch of n_chunks H N P and n_chunks H floats. With log_decay ([H]) the decays are constants and dt .. d_skip null.
LLMP_API int llmp_chunked_scan(const void* b, const void* c, const void* x, long row_t, const float* dt, long dt_t, const float* dt_bias,
                               const float* a_log, const float* d_skip, const float* log_decay, float* state, long state_slot, long state_half,
                               const int* q_start, const int* slots, const int* positions, const int* chunks, int n_chunks,
                               const int* requests, int n_requests, float* sums, float* gains, float* y, long y_t, int H, int G, int N, int P,
                               cudaStream_t stream) {
    if (n_chunks <= 0 || n_requests <= 0) return 0;
    LLMP_REQUIRE(H > 0 && G > 0 && H % G == 0 && H <= 65535 && n_requests <= 65535, "chunked_scan: %d heads in %d groups", H, G);
    LLMP_REQUIRE(N % 16 == 0 && N >= 16 && N <= 256 && P % 16 == 0 && P >= 16, "chunked_scan: no form for a state of %d x %d", N, P);
    LLMP_REQUIRE(((uintptr_t)b | (uintptr_t)c | (uintptr_t)x) % 16 == 0 && row_t % 8 == 0, "chunked_scan: rows are not in 16-byte pieces");
    LLMP_REQUIRE(((uintptr_t)state | (uintptr_t)sums) % 16 == 0 && state_slot % 4 == 0 && state_half % 4 == 0, "chunked_scan: states are not in 16-byte pieces");
    LLMP_REQUIRE((uintptr_t)y % 8 == 0 && y_t % 2 == 0, "chunked_scan: output rows are not in 8-byte pieces");
    ChunkArgs a;
    a.b = (const bf16*)b; a.c = (const bf16*)c; a.x = (const bf16*)x; a.row_t = row_t;
    a.dt = dt; a.dt_t = dt_t; a.dt_bias = dt_bias; a.a_log = a_log; a.d_skip = d_skip; a.log_decay = log_decay;
    a.chunks = chunks; a.sums = sums; a.gains = gains; a.y = y; a.y_t = y_t; a.H = H; a.G = G; a.N = N; a.P = P;
    const dim3 grid(n_chunks, H, (P + CS_COLS - 1) / CS_COLS);
    const size_t rows = (size_t)CS_TOKENS * (N + 8) * 2, cols = (size_t)CS_TOKENS * CS_XS * 2, states = (size_t)N * CS_XS * 4;
    const size_t smem1 = rows + 2 * cols, smem3 = rows + (states > rows + cols ? states : rows + cols);
    LLMP_ALLOW_SMEM(chunk_sums_kernel, smem1);
    LLMP_ALLOW_SMEM(chunk_outputs_kernel, smem3);
    chunk_sums_kernel<<<grid, CS_THREADS, smem1, stream>>>(a);
    const int per = N * P;
    chunk_states_kernel<<<dim3((per / 4 + 255) / 256, H, n_requests), 256, 0, stream>>>(sums, gains, requests, state, state_slot, state_half,
                                                                                        q_start, slots, positions, H, per);
    chunk_outputs_kernel<<<grid, CS_THREADS, smem3, stream>>>(a);
    return llmp_check_launch("chunked_scan");
}
