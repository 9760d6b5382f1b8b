// Time mixing with a matrix state per head whose rows decay channel by channel (the "wkv" mixer).
//
// Per head, with r_t, k_t, w_t [d] (receptance, key, decay in (0, 1)), v_t [d] and a bonus u [d]; S [d, d] (key channel,
// value channel), zero before the first token:
//   o_t[j] = sum_c r_t[c] (S[c, j] + u[c] k_t[c] v_t[j]);      S[c, j] <- w_t[c] S[c, j] + k_t[c] v_t[j]
//
// wkv_shift:  the mixes x_t + (x_(t-1) - x_t) mu_s of every token's row with the row before it, one matrix per s. The row
//             before a step's first token lies in the request's slot.
// wkv_decay:  the decays exp(-exp(W2 tanh(low) + w0)) from the float32 rows `low` of the first step of their projection.
// wkv_scan:   the recurrence; a block per (request, head, 16 value columns).
// wkv_gate:   every head's o divided by its root mean square, times a weight per channel and silu of the gate.
//
// A request's state is one float32 vector [shift piece | scan piece], each piece two copies that take turns by the parity
// of the last position written: a step of one token never overwrites what it read. Everything is float32.
#include "common.cuh"

namespace {

// ---- the mixes with the row before -----------------------------------------------------------------------------------
struct ShiftArgs {
    const float* x; const float* mu;                     // [tokens, D], [k, D]
    float* state; long state_slot; long state_half;      // copy: [D]
    const int* q_start; const int* slots; const int* positions; const int* token_request;
    void* out; long out_block; int D, k;                 // [k, tokens, D]
};

template <typename T> __device__ __forceinline__ void shift_store4(T* p, float4 v);
template <> __device__ __forceinline__ void shift_store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void shift_store4<bf16>(bf16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}

// A thread takes one place (or, VEC, four) of a token's row. The thread of a request's first token of the step also moves
// that place's state on: it reads the copy first, so the copies may coincide (a step of an even number of tokens).
template <typename T, bool VEC>
__global__ void wkv_shift_kernel(const ShiftArgs a) {
    pdl_wait();                                          // what the kernels before wrote is complete
    pdl_trigger();
    const int n = blockIdx.x;
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * (VEC ? 4 : 1);
    if (c >= a.D) return;
    const int r = a.token_request[n], pos = a.positions[n], begin = a.q_start[r];
    const float* row = a.x + (size_t)n * a.D + c;
    float* slot = a.state + (size_t)a.slots[r] * a.state_slot + c;
    if (VEC) {
        const float4 x = *reinterpret_cast<const float4*>(row);
        float4 p = make_float4(0.f, 0.f, 0.f, 0.f);
        if (n > begin) p = *reinterpret_cast<const float4*>(row - a.D);
        else if (pos > 0) p = *reinterpret_cast<const float4*>(slot + ((pos - 1) & 1) * a.state_half);
        if (n == begin) {
            const int count = a.q_start[r + 1] - begin;
            *reinterpret_cast<float4*>(slot + ((pos + count - 1) & 1) * a.state_half) =
                *reinterpret_cast<const float4*>(row + (size_t)(count - 1) * a.D);
        }
        const float4 dx = make_float4(p.x - x.x, p.y - x.y, p.z - x.z, p.w - x.w);
        for (int s = 0; s < a.k; ++s) {
            const float4 m = *reinterpret_cast<const float4*>(a.mu + (size_t)s * a.D + c);
            shift_store4(reinterpret_cast<T*>(a.out) + (size_t)s * a.out_block + (size_t)n * a.D + c,
                         make_float4(fmaf(dx.x, m.x, x.x), fmaf(dx.y, m.y, x.y), fmaf(dx.z, m.z, x.z), fmaf(dx.w, m.w, x.w)));
        }
    } else {
        const float x = row[0];
        const float p = n > begin ? row[-a.D] : (pos > 0 ? slot[((pos - 1) & 1) * a.state_half] : 0.f);
        if (n == begin) {
            const int count = a.q_start[r + 1] - begin;
            slot[((pos + count - 1) & 1) * a.state_half] = row[(size_t)(count - 1) * a.D];
        }
        for (int s = 0; s < a.k; ++s)
            reinterpret_cast<T*>(a.out)[(size_t)s * a.out_block + (size_t)n * a.D + c] = from_float<T>(fmaf(p - x, a.mu[(size_t)s * a.D + c], x));
    }
}

// ---- decays ----------------------------------------------------------------------------------------------------------
constexpr int WD_TOKENS = 16;
constexpr int WD_RANK = 64;                              // entries of `low` staged at a time

// A thread takes a channel and WD_TOKENS tokens: out[t, c] = exp(-exp(w0[c] + sum_i tanh(low[t, i]) w2t[i, c])).
__global__ void __launch_bounds__(128) wkv_decay_kernel(const float* __restrict__ low, long low_t, const float* __restrict__ w2t,
                                                        const float* __restrict__ w0, float* __restrict__ out, int N, int C, int rank) {
    __shared__ __align__(16) float tl[WD_RANK][WD_TOKENS];
    pdl_wait();
    pdl_trigger();
    const int t0 = blockIdx.x * WD_TOKENS, c = blockIdx.y * blockDim.x + threadIdx.x;
    const int cnt = min(WD_TOKENS, N - t0);
    float acc[WD_TOKENS];
    const float base = c < C ? w0[c] : 0.f;
#pragma unroll
    for (int t = 0; t < WD_TOKENS; ++t) acc[t] = base;
    for (int i0 = 0; i0 < rank; i0 += WD_RANK) {
        const int ni = min(WD_RANK, rank - i0);
        __syncthreads();
        for (int e = threadIdx.x; e < ni * WD_TOKENS; e += blockDim.x) {
            const int t = e / ni, i = e % ni;
            tl[i][t] = t < cnt ? tanhf(low[(size_t)(t0 + t) * low_t + i0 + i]) : 0.f;
        }
        __syncthreads();
        if (c < C) {
            const float* w = w2t + (size_t)i0 * C + c;
#pragma unroll 8
            for (int i = 0; i < ni; ++i) {
                const float wv = w[(size_t)i * C];
#pragma unroll
                for (int t4 = 0; t4 < WD_TOKENS / 4; ++t4) {
                    const float4 v = *reinterpret_cast<const float4*>(&tl[i][t4 * 4]);
                    acc[t4 * 4] = fmaf(v.x, wv, acc[t4 * 4]); acc[t4 * 4 + 1] = fmaf(v.y, wv, acc[t4 * 4 + 1]);
                    acc[t4 * 4 + 2] = fmaf(v.z, wv, acc[t4 * 4 + 2]); acc[t4 * 4 + 3] = fmaf(v.w, wv, acc[t4 * 4 + 3]);
                }
            }
        }
    }
    if (c >= C) return;
#pragma unroll
    for (int t = 0; t < WD_TOKENS; ++t)
        if (t < cnt) out[(size_t)(t0 + t) * C + c] = expf(-expf(acc[t]));
}

// ---- the recurrence --------------------------------------------------------------------------------------------------
constexpr int WK_THREADS = 128;
constexpr int WK_COLS = 16;       // value columns of a block: a warp has four, a half-warp two
constexpr int WK_CHUNK = 8;       // tokens of a stage
constexpr int WK_STAGES = 4;

struct WkvArgs {
    const float* r; const float* k; const float* v; long rkv_t;     // [tokens, H d] each, one stride
    const float* w; long w_t;                                        // [tokens, H d]
    const float* u;                                                  // [H, d]
    float* state; long state_slot; long state_half;                  // a copy: [H][column blocks][2 NR][128] (see below)
    const int* q_start; const int* slots; const int* positions;
    float* o; long o_t;                                              // [tokens, H d]
    int H, d, vec;
};

__device__ __forceinline__ void wk_cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void wk_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

template <int NR> __device__ __forceinline__ void wk_rows(const float* p, float (&v)[NR]) {
    if constexpr (NR % 4 == 0) {
#pragma unroll
        for (int i = 0; i < NR / 4; ++i) {
            const float4 t = *reinterpret_cast<const float4*>(p + 4 * i);
            v[4 * i] = t.x; v[4 * i + 1] = t.y; v[4 * i + 2] = t.z; v[4 * i + 3] = t.w;
        }
    } else if constexpr (NR == 2) {
        const float2 t = *reinterpret_cast<const float2*>(p);
        v[0] = t.x; v[1] = t.y;
    } else {
#pragma unroll
        for (int i = 0; i < NR; ++i) v[i] = p[i];
    }
}

// A block owns (request, head, 16 value columns) and walks the request's tokens in order. A half-warp owns two columns; its
// lane l holds their rows l NR .. l NR + NR - 1 in registers (16 NR >= d; rows past d stay zero because their keys are).
// Nothing of a token's read-out feeds the recurrence, so the sums over the lanes of a chunk of 8 tokens are taken
// together: 16 values (token, column) a lane, halved with every exchange, until each lane holds the value it stores.
// The tokens' inputs come through a ring of stages of one chunk (asynchronous copies, one barrier a chunk).
// In the slot a copy of the state is kept in the order in which the threads hold it: entry e = 2 i + column (i the row
// within the lane) of thread t of column block b of head h at ((h blocks + b) 2 NR + e) 128 + t.
template <int NR>
__global__ void __launch_bounds__(WK_THREADS) wkv_scan_kernel(const WkvArgs a) {
    constexpr int DP = 16 * NR;                          // rows with padding
    constexpr int ROW = 3 * DP + WK_COLS;                // r, k, w, this block's v
    extern __shared__ __align__(16) float wk_smem[];
    float* us = wk_smem;                                 // [DP]
    float* ring = us + DP;                               // [WK_STAGES][WK_CHUNK][ROW]
    pdl_wait();
    pdl_trigger();
    const int q = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
    const int begin = a.q_start[q], end = a.q_start[q + 1];
    if (end <= begin) return;
    const int tid = threadIdx.x, lane = tid & 31, l16 = lane & 15;
    const int d = a.d, j0 = b * WK_COLS;
    const int ncols = min(WK_COLS, d - j0);
    const int col = (tid >> 4) * 2;                      // this thread's first column within the block
    const int p0 = a.positions[begin];
    float* slot = a.state + (size_t)a.slots[q] * a.state_slot + ((size_t)h * gridDim.z + b) * (2 * NR) * WK_THREADS + tid;
    const float* rd = slot + ((p0 + 1) & 1) * a.state_half;
    float* wr = slot + ((p0 + end - begin - 1) & 1) * a.state_half;
    float S[NR][2];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        S[i][0] = rd[(size_t)(2 * i) * WK_THREADS];
        S[i][1] = rd[(size_t)(2 * i + 1) * WK_THREADS];
    }
    for (int i = tid; i < DP; i += WK_THREADS) us[i] = i < d ? a.u[(size_t)h * d + i] : 0.f;
    if (d < DP || ncols < WK_COLS)
        for (int i = tid; i < WK_STAGES * WK_CHUNK * ROW; i += WK_THREADS) ring[i] = 0.f;       // the padding stays as it is now
    __syncthreads();
    const int chunks = (end - begin + WK_CHUNK - 1) / WK_CHUNK;
    auto issue = [&](int s) {
        if (s < chunks) {
            float* base = ring + (size_t)(s % WK_STAGES) * WK_CHUNK * ROW;
            const int t0 = begin + s * WK_CHUNK, cnt = min(WK_CHUNK, end - t0);
            const int unit = a.vec ? 4 : 1, du = d / unit, per = 3 * du + ncols / unit;      // pieces of a row of r, k, w; of a token
            for (int x = lane; x < per; x += 32) {       // a lane's pieces are the same for all tokens; a warp takes every fourth token
                const int which = (x >= du) + (x >= 2 * du) + (x >= 3 * du);
                const int at = (x - which * du) * unit;
                const float* src = (which == 0 ? a.r : which == 1 ? a.k : which == 2 ? a.w : a.v + j0) + (size_t)h * d + at;
                const long stride = which == 2 ? a.w_t : a.rkv_t;
                for (int tt = tid >> 5; tt < cnt; tt += WK_THREADS / 32) {
                    float* dst = base + (size_t)tt * ROW + which * DP + at;
                    if (a.vec) wk_cp16(dst, src + (size_t)(t0 + tt) * stride);
                    else wk_cp4(dst, src + (size_t)(t0 + tt) * stride);
                }
            }
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    float ul[NR];
    wk_rows<NR>(us + l16 * NR, ul);
#pragma unroll
    for (int s = 0; s < WK_STAGES - 1; ++s) issue(s);
    for (int s = 0; s < chunks; ++s) {
        asm volatile("cp.async.wait_group %0;\n" ::"n"(WK_STAGES - 2) : "memory");
        __syncthreads();                                 // stage s is here for everyone; everyone has left stage s - 1
        issue(s + WK_STAGES - 1);                        // into the buffer of stage s - 1
        const float* base = ring + (size_t)(s % WK_STAGES) * WK_CHUNK * ROW;
        const int t0 = begin + s * WK_CHUNK, cnt = min(WK_CHUNK, end - t0);
        auto token = [&](const float* cur, float& o0, float& o1) {
            float r[NR], k[NR], w[NR];
            wk_rows<NR>(cur + l16 * NR, r);
            wk_rows<NR>(cur + DP + l16 * NR, k);
            wk_rows<NR>(cur + 2 * DP + l16 * NR, w);
            const float2 v = *reinterpret_cast<const float2*>(cur + 3 * DP + col);
            float ruk = 0.f;
            o0 = o1 = 0.f;
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                ruk = fmaf(r[i], ul[i] * k[i], ruk);
                o0 = fmaf(r[i], S[i][0], o0);
                o1 = fmaf(r[i], S[i][1], o1);
                S[i][0] = fmaf(w[i], S[i][0], k[i] * v.x);
                S[i][1] = fmaf(w[i], S[i][1], k[i] * v.y);
            }
            o0 = fmaf(ruk, v.x, o0);
            o1 = fmaf(ruk, v.y, o1);
        };
        if (cnt == WK_CHUNK) {
            float acc[2 * WK_CHUNK];                     // (token tt, column c) at 2 tt + c
#pragma unroll
            for (int tt = 0; tt < WK_CHUNK; ++tt) token(base + (size_t)tt * ROW, acc[2 * tt], acc[2 * tt + 1]);
            // lane l16 ends with the sum of value l16: bit m of the lane chooses the half that keeps going
#pragma unroll
            for (int m = 8; m > 0; m >>= 1) {
                const bool up = l16 & m;
#pragma unroll
                for (int i = 0; i < m; ++i) {
                    const float give = up ? acc[i] : acc[i + m], keep = up ? acc[i + m] : acc[i];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, m);
                }
            }
            const int j = col + (l16 & 1);
            if (j < ncols) a.o[(size_t)(t0 + (l16 >> 1)) * a.o_t + (size_t)h * d + j0 + j] = acc[0];
        } else {
            for (int tt = 0; tt < cnt; ++tt) {
                float o0, o1;
                token(base + (size_t)tt * ROW, o0, o1);
#pragma unroll
                for (int m = 8; m > 0; m >>= 1) {
                    o0 += __shfl_xor_sync(0xffffffffu, o0, m);
                    o1 += __shfl_xor_sync(0xffffffffu, o1, m);
                }
                if (l16 < 2 && col + l16 < ncols) a.o[(size_t)(t0 + tt) * a.o_t + (size_t)h * d + j0 + col + l16] = l16 ? o1 : o0;
            }
        }
    }
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        wr[(size_t)(2 * i) * WK_THREADS] = S[i][0];
        wr[(size_t)(2 * i + 1) * WK_THREADS] = S[i][1];
    }
}

int wkv_rows_per_lane(int d) {
    int nr = 1;
    while (16 * nr < d) nr *= 2;
    return nr;
}

// ---- the heads' norm and the gate ------------------------------------------------------------------------------------
// A warp per (token, head): out = o / sqrt(mean(o^2) + eps) * weight[channel] * silu(gate).
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(bf16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

template <typename T>
__global__ void wkv_gate_kernel(const float* __restrict__ o, long o_t, const float* __restrict__ gate, long gate_t,
                                const float* __restrict__ weight, T* __restrict__ out, long out_t, long items, int H, int d, float eps) {
    pdl_wait();
    pdl_trigger();
    const long item = (long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= items) return;
    const int lane = threadIdx.x & 31;
    const size_t t = (size_t)(item / H);
    const int c0 = (int)(item % H) * d;
    const float* y = o + t * o_t + c0;
    const float* z = gate + t * gate_t + c0;
    T* dst = out + t * out_t + c0;
    float ss = 0.f;
    if ((d & 1) == 0 && d <= 256 && ((o_t | gate_t | out_t) & 1) == 0) {      // pairs, the row in registers
        float2 v[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 2 * (lane + 32 * i);
            v[i] = c < d ? *reinterpret_cast<const float2*>(y + c) : make_float2(0.f, 0.f);
            ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, ss));
        }
        ss = warp_sum(ss);
        const float f = 1.f / sqrtf(ss / (float)d + eps);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 2 * (lane + 32 * i);
            if (c < d) {
                const float2 zz = *reinterpret_cast<const float2*>(z + c), w = *reinterpret_cast<const float2*>(weight + c0 + c);
                const float a = v[i].x * f * w.x * (zz.x / (1.f + expf(-zz.x))), b = v[i].y * f * w.y * (zz.y / (1.f + expf(-zz.y)));
                store2(dst + c, a, b);
            }
        }
        return;
    }
    for (int c = lane; c < d; c += 32) ss = fmaf(y[c], y[c], ss);
    ss = warp_sum(ss);
    const float f = 1.f / sqrtf(ss / (float)d + eps);
    for (int c = lane; c < d; c += 32) dst[c] = from_float<T>(y[c] * f * weight[c0 + c] * (z[c] / (1.f + expf(-z[c]))));
}

}  // namespace

LLMP_API int llmp_wkv_shift(const float* x, const float* mu, float* state, long state_slot, long state_half, const int* q_start,
                            const int* slots, const int* positions, const int* token_request, void* out, int out_dtype, int N, int D,
                            int k, cudaStream_t stream) {
    if (N <= 0) return 0;
    LLMP_REQUIRE(D > 0 && k > 0, "wkv_shift: bad sizes width=%d mixes=%d", D, k);
    ShiftArgs a;
    a.x = x; a.mu = mu; a.state = state; a.state_slot = state_slot; a.state_half = state_half; a.q_start = q_start; a.slots = slots;
    a.positions = positions; a.token_request = token_request; a.out = out; a.out_block = (long)N * D; a.D = D; a.k = k;
    const bool vec = D % 4 == 0 && state_slot % 4 == 0 && state_half % 4 == 0 && ((size_t)x | (size_t)mu | (size_t)state | (size_t)out) % 16 == 0;
    const int per = vec ? D / 4 : D;
    const int threads = per >= 256 ? 256 : 128;
    const dim3 grid(N, (per + threads - 1) / threads);
    void (*kernel)(const ShiftArgs) = out_dtype == LLMP_BF16 ? (vec ? wkv_shift_kernel<bf16, true> : wkv_shift_kernel<bf16, false>)
                                                             : (vec ? wkv_shift_kernel<float, true> : wkv_shift_kernel<float, false>);
    llmp_launch_dependent(kernel, grid, dim3(threads), 0, stream, a);
    return llmp_check_launch("wkv_shift");
}

LLMP_API int llmp_wkv_decay(const float* low, long low_t, const float* w2t, const float* w0, float* out, int N, int C, int rank,
                            cudaStream_t stream) {
    if (N <= 0) return 0;
    LLMP_REQUIRE(C > 0 && rank > 0 && (C + 127) / 128 <= 65535, "wkv_decay: bad sizes channels=%d rank=%d", C, rank);
    llmp_launch_dependent(wkv_decay_kernel, dim3((N + WD_TOKENS - 1) / WD_TOKENS, (C + 127) / 128), dim3(128), 0, stream, low, low_t, w2t, w0,
                          out, N, C, rank);
    return llmp_check_launch("wkv_decay");
}

// Entries of one copy of the recurrence's state (0: heads of this size are not served).
LLMP_API long llmp_wkv_state_entries(int H, int d) {
    if (H <= 0 || d <= 0 || d > 256) return 0;
    return (long)H * ((d + WK_COLS - 1) / WK_COLS) * 2 * wkv_rows_per_lane(d) * WK_THREADS;
}

LLMP_API int llmp_wkv_scan(const float* r, const float* k, const float* v, long rkv_t, const float* w, long w_t, const float* u, float* state,
                           long state_slot, long state_half, const int* q_start, const int* slots, const int* positions, float* o,
                           long o_t, int R, int H, int d, cudaStream_t stream) {
    if (R <= 0) return 0;
    LLMP_REQUIRE(H > 0 && H <= 65535 && d > 0 && d <= 256, "wkv_scan: %d heads of %d channels are not served", H, d);
    LLMP_REQUIRE(state_half >= llmp_wkv_state_entries(H, d), "wkv_scan: the state's copies are too small");
    WkvArgs a;
    a.r = r; a.k = k; a.v = v; a.rkv_t = rkv_t; a.w = w; a.w_t = w_t; a.u = u; a.state = state; a.state_slot = state_slot;
    a.state_half = state_half; a.q_start = q_start; a.slots = slots; a.positions = positions; a.o = o; a.o_t = o_t; a.H = H; a.d = d;
    a.vec = d % 4 == 0 && rkv_t % 4 == 0 && w_t % 4 == 0 && ((size_t)r | (size_t)k | (size_t)v | (size_t)w) % 16 == 0;
    const int nr = wkv_rows_per_lane(d);
    const size_t smem = sizeof(float) * ((size_t)16 * nr + (size_t)WK_STAGES * WK_CHUNK * (48 * nr + WK_COLS));
    const dim3 grid(R, H, (d + WK_COLS - 1) / WK_COLS);
#define LLMP_WKV(NR)                                                                             \
    if (nr == NR) {                                                                              \
        LLMP_ALLOW_SMEM(wkv_scan_kernel<NR>, smem);                                              \
        llmp_launch_dependent(wkv_scan_kernel<NR>, grid, dim3(WK_THREADS), smem, stream, a);     \
    } else
    LLMP_WKV(1) LLMP_WKV(2) LLMP_WKV(4) LLMP_WKV(8) LLMP_WKV(16) {}
#undef LLMP_WKV
    return llmp_check_launch("wkv_scan");
}

LLMP_API int llmp_wkv_gate(const float* o, long o_t, const float* gate, long gate_t, const float* weight, void* out, int out_dtype, long out_t,
                           int N, int H, int d, float eps, cudaStream_t stream) {
    if (N <= 0) return 0;
    LLMP_REQUIRE(H > 0 && d > 0, "wkv_gate: bad sizes heads=%d dim=%d", H, d);
    const long items = (long)N * H;
    const dim3 grid((unsigned)((items + 3) / 4));
    if (out_dtype == LLMP_BF16)
        llmp_launch_dependent(wkv_gate_kernel<bf16>, grid, dim3(128), 0, stream, o, o_t, gate, gate_t, weight, (bf16*)out, out_t, items, H, d, eps);
    else
        llmp_launch_dependent(wkv_gate_kernel<float>, grid, dim3(128), 0, stream, o, o_t, gate, gate_t, weight, (float*)out, out_t, items, H, d, eps);
    return llmp_check_launch("wkv_gate");
}
