// Time mixing with a matrix state per head whose rows decay channel by channel (the "wkv" mixer).
//
// Per head, with r_t, k_t, w_t [d] (receptance, key, decay in (0, 1)), v_t [d] and a bonus u [d]; S [d, d] (key channel,
// value channel), zero before the first token:
//   o_t[j] = sum_c r_t[c] (S[c, j] + u[c] k_t[c] v_t[j]);      S[c, j] <- w_t[c] S[c, j] + k_t[c] v_t[j]
//
// wkv_shift:  the mixes x_t + (x_(t-1) - x_t) mu_s of every token's row with the row before it, one matrix per s. The row
//             before a step's first token lies in the request's slot.
// wkv_decay:  the decays exp(-exp(W2 tanh(low) + w0)) from the float32 rows `low` of the first step of their projection.
// wkv_scan:   the recurrence; a block per (request, head, 32 value columns), long prompts in segments side by side.
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
constexpr int WK_COLS = 32;       // value columns of a block: a half-warp has four
constexpr int WK_CHUNK = 8;       // tokens of a stage
constexpr int WK_STAGES = 4;

struct WkvArgs {
    const float* r; const float* k; const float* v; long rkv_t;     // [tokens, H d] each, one stride
    const float* w; long w_t;                                        // [tokens, H d]
    const float* u;                                                  // [H, d]
    float* state; long state_slot; long state_half;                  // a copy: [H][column blocks][4 NR][128] (see below)
    const int* q_start; const int* slots; const int* positions;
    float* o; long o_t;                                              // [tokens, H d]
    float* ends; float* decays; int seg_tokens, segments;            // segments: [requests][segments][a copy], [requests][segments][H][16 NR]
    int H, d, vec, blocks;                                           // blocks: column blocks of a head
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

// A block owns (request, head, 32 value columns) and walks the request's tokens in order. A half-warp owns four columns;
// its lane l holds their rows l NR .. l NR + NR - 1 in registers (16 NR >= d; rows past d stay zero because their keys
// are). Nothing of a token's read-out feeds the recurrence, so the sums over the lanes of a chunk of 8 tokens are taken
// together: 32 values (token, column) a lane, halved with every exchange, until each lane holds the two it stores.
// The tokens' inputs come through a ring of stages of one chunk (asynchronous copies, one barrier a chunk).
// A copy of the state is kept in the order in which the threads hold it: entry e = 4 i + column (i the row within the lane)
// of thread t of column block b of head h at ((h blocks + b) 4 NR + e) 128 + t.
//
// The recurrence is linear in its state, so a long prompt can be cut into segments of `seg_tokens` that run side by side
// (blockIdx.z also counts segments). MODE 0: a segment after the first starts from zero, and every segment leaves its end
// state and the products of its decays. MODE 1, for the segments after the first: the state a segment really starts
// from, folded from the earlier segments' ends, adds (the decays since the segment's start, times r)^T state to the
// segment's read-outs; the last segment's block writes the request's state.
template <int NR, int MODE>
__global__ void __launch_bounds__(WK_THREADS) wkv_scan_kernel(const WkvArgs a) {
    constexpr int DP = 16 * NR;                          // rows with padding
    constexpr int ROW = 3 * DP + WK_COLS;                // r, k, w, this block's v
    constexpr int E = 4 * NR;                            // state entries of a thread
    extern __shared__ __align__(16) float wk_smem[];
    float* us = wk_smem;                                 // [DP]
    float* ring = us + DP;                               // [WK_STAGES][WK_CHUNK][ROW]
    pdl_wait();
    pdl_trigger();
    const int q = blockIdx.x, h = blockIdx.y, b = blockIdx.z % a.blocks;
    const int seg = blockIdx.z / a.blocks + (MODE == 1 ? 1 : 0);
    const int req_begin = a.q_start[q], req_end = a.q_start[q + 1];
    const int begin = req_begin + seg * a.seg_tokens;    // without segments seg is 0 and seg_tokens covers every request
    const int end = min(req_end, begin + a.seg_tokens);
    if (end <= begin) return;
    const int tid = threadIdx.x, lane = tid & 31, l16 = lane & 15;
    const int d = a.d, j0 = b * WK_COLS;
    const int ncols = min(WK_COLS, d - j0);
    const int col = (tid >> 4) * 4;                      // this thread's first column within the block
    const int p0 = a.positions[req_begin];
    const size_t place = ((size_t)h * a.blocks + b) * E * WK_THREADS + tid;
    const size_t copy = (size_t)a.H * a.blocks * E * WK_THREADS;
    float* slot = a.state + (size_t)a.slots[q] * a.state_slot + place;
    float* wr = slot + ((p0 + req_end - req_begin - 1) & 1) * a.state_half;
    float* ends = a.ends + (size_t)q * a.segments * copy + place;                        // segment s at ends + s * copy
    float* decays = a.decays + ((size_t)q * a.segments * a.H + h) * DP + l16 * NR;       // segment s at decays + s * H * DP
    float S[NR][4], p[NR];                               // p: products of the decays since the segment's start
#pragma unroll
    for (int i = 0; i < NR; ++i) p[i] = 1.f;
    if (MODE == 1) {
        // the state this segment starts from: the first segment's end, then the later ones before this one
#pragma unroll
        for (int e = 0; e < E; ++e) S[e >> 2][e & 3] = ends[(size_t)e * WK_THREADS];
        for (int s = 1; s < seg; ++s) {
            float f[NR];
            wk_rows<NR>(decays + (size_t)s * a.H * DP, f);
#pragma unroll
            for (int e = 0; e < E; ++e) S[e >> 2][e & 3] = fmaf(f[e >> 2], S[e >> 2][e & 3], ends[s * copy + (size_t)e * WK_THREADS]);
        }
        if (end == req_end) {
            float f[NR];
            wk_rows<NR>(decays + (size_t)seg * a.H * DP, f);
#pragma unroll
            for (int e = 0; e < E; ++e)
                wr[(size_t)e * WK_THREADS] = fmaf(f[e >> 2], S[e >> 2][e & 3], ends[seg * copy + (size_t)e * WK_THREADS]);
        }
    } else if (seg == 0) {
        const float* rd = slot + ((p0 + 1) & 1) * a.state_half;
#pragma unroll
        for (int e = 0; e < E; ++e) S[e >> 2][e & 3] = rd[(size_t)e * WK_THREADS];
    } else {
#pragma unroll
        for (int e = 0; e < E; ++e) S[e >> 2][e & 3] = 0.f;
    }
    for (int i = tid; i < DP; i += WK_THREADS) us[i] = i < d ? a.u[(size_t)h * d + i] : 0.f;
    if (d < DP || ncols < WK_COLS)
        for (int i = tid; i < WK_STAGES * WK_CHUNK * ROW; i += WK_THREADS) ring[i] = 0.f;       // the padding stays as it is now
    __syncthreads();
    const int chunks = (end - begin + WK_CHUNK - 1) / WK_CHUNK;
    // a lane's pieces of a token (16 bytes where all rows allow it) are the same for all tokens; a warp takes every fourth token
    const int unit = a.vec ? 4 : 1, du = d / unit, per = 3 * du + (MODE == 1 ? 0 : ncols / unit);
    auto issue = [&](int s) {
        if (s < chunks) {
            float* base = ring + (size_t)(s % WK_STAGES) * WK_CHUNK * ROW;
            const int t0 = begin + s * WK_CHUNK, cnt = min(WK_CHUNK, end - t0);
            for (int x = lane; x < per; x += 32) {
                const int which = (x >= du) + (x >= 2 * du) + (x >= 3 * du);
                if (MODE == 1 && which == 1) continue;   // the correction reads no keys
                const int at = (x - which * du) * unit;
                const float* src = (which == 0 ? a.r : which == 1 ? a.k : which == 2 ? a.w : a.v + j0) + (size_t)h * d + at;
                const long stride = which == 2 ? a.w_t : a.rkv_t;
                float* dst = base + which * DP + at;
#pragma unroll
                for (int tt0 = 0; tt0 < WK_CHUNK; tt0 += WK_THREADS / 32) {
                    const int tt = tt0 + (tid >> 5);
                    if (tt < cnt) {
                        if (a.vec) wk_cp16(dst + (size_t)tt * ROW, src + (size_t)(t0 + tt) * stride);
                        else wk_cp4(dst + (size_t)tt * ROW, src + (size_t)(t0 + tt) * stride);
                    }
                }
            }
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    float ul[NR];
    wk_rows<NR>(us + l16 * NR, ul);
#pragma unroll
    for (int s = 0; s < WK_STAGES - 1; ++s) issue(s);
    struct Inputs { float r[NR], k[NR], w[NR]; float4 v; };
    auto fetch = [&](const float* cur, Inputs& x) {
        wk_rows<NR>(cur + l16 * NR, x.r);
        wk_rows<NR>(cur + 2 * DP + l16 * NR, x.w);
        if (MODE == 0) {
            wk_rows<NR>(cur + DP + l16 * NR, x.k);
            x.v = *reinterpret_cast<const float4*>(cur + 3 * DP + col);
        }
    };
    auto token = [&](const Inputs& x, float (&o)[4]) {
        if (MODE == 1) {
            o[0] = o[1] = o[2] = o[3] = 0.f;
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const float rp = x.r[i] * p[i];
                p[i] *= x.w[i];
#pragma unroll
                for (int c = 0; c < 4; ++c) o[c] = fmaf(rp, S[i][c], o[c]);
            }
            return;
        }
        const float v[4] = {x.v.x, x.v.y, x.v.z, x.v.w};
        float ruk = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) ruk = fmaf(x.r[i], ul[i] * x.k[i], ruk);
#pragma unroll
        for (int c = 0; c < 4; ++c) o[c] = ruk * v[c];
#pragma unroll
        for (int i = 0; i < NR; ++i) {
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                o[c] = fmaf(x.r[i], S[i][c], o[c]);
                S[i][c] = fmaf(x.w[i], S[i][c], x.k[i] * v[c]);
            }
            p[i] *= x.w[i];
        }
    };
    float* out = a.o + (size_t)h * d + j0;
    for (int s = 0; s < chunks; ++s) {
        asm volatile("cp.async.wait_group %0;\n" ::"n"(WK_STAGES - 2) : "memory");
        __syncthreads();                                 // stage s is here for everyone; everyone has left stage s - 1
        const float* base = ring + (size_t)(s % WK_STAGES) * WK_CHUNK * ROW;
        const int t0 = begin + s * WK_CHUNK, cnt = min(WK_CHUNK, end - t0);
        if (cnt == WK_CHUNK) {
            float acc[4 * WK_CHUNK];                     // (token tt, column c) at 4 tt + c
            Inputs x[2];
            fetch(base, x[0]);
            issue(s + WK_STAGES - 1);                    // into the buffer of stage s - 1
            // lane l16 ends with values 2 l16 and 2 l16 + 1: token l16 / 2, columns 2 (l16 & 1) and the next
            const int jo = col + 2 * (l16 & 1);
            float* dst = out + (size_t)(t0 + (l16 >> 1)) * a.o_t + jo;
            float old0 = 0.f, old1 = 0.f;
            if (MODE == 1) {
                if (jo < ncols) old0 = dst[0];
                if (jo + 1 < ncols) old1 = dst[1];
            }
#pragma unroll
            for (int tt = 0; tt < WK_CHUNK; ++tt) {
                if (tt + 1 < WK_CHUNK) fetch(base + (size_t)(tt + 1) * ROW, x[(tt + 1) & 1]);      // a token ahead of the sums
                float o[4];
                token(x[tt & 1], o);
#pragma unroll
                for (int c = 0; c < 4; ++c) acc[4 * tt + c] = o[c];
            }
            // bit m / 2 of the lane chooses the half that keeps going
#pragma unroll
            for (int m = 16; m > 1; m >>= 1) {
                const bool up = l16 & (m >> 1);
#pragma unroll
                for (int i = 0; i < m; ++i) {
                    const float give = up ? acc[i] : acc[i + m], keep = up ? acc[i + m] : acc[i];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, m >> 1);
                }
            }
            if (jo < ncols) dst[0] = acc[0] + old0;
            if (jo + 1 < ncols) dst[1] = acc[1] + old1;
        } else {
            issue(s + WK_STAGES - 1);
            for (int tt = 0; tt < cnt; ++tt) {
                Inputs x;
                fetch(base + (size_t)tt * ROW, x);
                float o[4];
                token(x, o);
#pragma unroll
                for (int m = 8; m > 0; m >>= 1) {
#pragma unroll
                    for (int c = 0; c < 4; ++c) o[c] += __shfl_xor_sync(0xffffffffu, o[c], m);
                }
                if (l16 < 4 && col + l16 < ncols) {
                    float* dst = out + (size_t)(t0 + tt) * a.o_t + col + l16;
                    const float sum = l16 == 0 ? o[0] : l16 == 1 ? o[1] : l16 == 2 ? o[2] : o[3];
                    *dst = MODE == 1 ? *dst + sum : sum;
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    if (MODE == 1) return;
    if (seg > 0 || end < req_end) {                      // one of several segments
        float* to = ends + seg * copy;
#pragma unroll
        for (int e = 0; e < E; ++e) to[(size_t)e * WK_THREADS] = S[e >> 2][e & 3];
        if (b == 0 && tid < 16) {
#pragma unroll
            for (int i = 0; i < NR; ++i) decays[(size_t)seg * a.H * DP + i] = p[i];
        }
        return;
    }
#pragma unroll
    for (int e = 0; e < E; ++e) wr[(size_t)e * WK_THREADS] = S[e >> 2][e & 3];
}

int wkv_rows_per_lane(int d) {
    int nr = 1;
    while (16 * nr < d) nr *= 2;
    return nr;
}

// ---- the heads' norm and the gate ------------------------------------------------------------------------------------
// out = o / sqrt(mean(o^2) + eps) * weight[channel] * silu(gate), the mean over the channels of a head. VEC: `group` lanes (a
// power of two) share a head of at most 4 `group` channels, a lane has four of them; else a warp per (token, head).
template <typename T, bool VEC>
__global__ void wkv_gate_kernel(const float* __restrict__ o, long o_t, const float* __restrict__ gate, long gate_t,
                                const float* __restrict__ weight, T* __restrict__ out, long out_t, long items, int H, int d, int group, float eps) {
    pdl_wait();
    pdl_trigger();
    const long item = ((long)blockIdx.x * blockDim.x + threadIdx.x) / group;
    const int lane = threadIdx.x % group;
    const bool valid = item < items;
    const size_t t = valid ? (size_t)(item / H) : 0;
    const int c0 = valid ? (int)(item % H) * d : 0;
    if (VEC) {
        const int c = lane * 4;
        const bool mine = valid && c < d;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f), z = v, w = v;
        if (mine) {
            v = *reinterpret_cast<const float4*>(o + t * o_t + c0 + c);
            z = *reinterpret_cast<const float4*>(gate + t * gate_t + c0 + c);
            w = *reinterpret_cast<const float4*>(weight + c0 + c);
        }
        float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
        for (int m = group >> 1; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
        const float f = 1.f / sqrtf(ss / (float)d + eps);
        if (mine)
            shift_store4(out + t * out_t + c0 + c, make_float4(v.x * f * w.x * (z.x / (1.f + expf(-z.x))), v.y * f * w.y * (z.y / (1.f + expf(-z.y))),
                                                              v.z * f * w.z * (z.z / (1.f + expf(-z.z))), v.w * f * w.w * (z.w / (1.f + expf(-z.w)))));
        return;
    }
    if (!valid) return;
    const float* y = o + t * o_t + c0;
    const float* z = gate + t * gate_t + c0;
    T* dst = out + t * out_t + c0;
    float ss = 0.f;
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
    return (long)H * ((d + WK_COLS - 1) / WK_COLS) * 4 * wkv_rows_per_lane(d) * WK_THREADS;
}

// Float32 scratch of a scan in `segments` segments per request.
LLMP_API long llmp_wkv_scratch(int R, int H, int d, int segments) {
    return (long)R * segments * (llmp_wkv_state_entries(H, d) + (long)H * 16 * wkv_rows_per_lane(d));
}

// segments > 1: requests are cut into that many segments of seg_tokens (they must cover the longest), with `scratch` of
// llmp_wkv_scratch floats.
LLMP_API int llmp_wkv_scan(const float* r, const float* k, const float* v, long rkv_t, const float* w, long w_t, const float* u, float* state,
                           long state_slot, long state_half, const int* q_start, const int* slots, const int* positions, float* o,
                           long o_t, int R, int H, int d, int segments, int seg_tokens, float* scratch, cudaStream_t stream) {
    if (R <= 0) return 0;
    LLMP_REQUIRE(H > 0 && H <= 65535 && d > 0 && d <= 256, "wkv_scan: %d heads of %d channels are not served", H, d);
    LLMP_REQUIRE(state_half >= llmp_wkv_state_entries(H, d), "wkv_scan: the state's copies are too small");
    WkvArgs a;
    a.r = r; a.k = k; a.v = v; a.rkv_t = rkv_t; a.w = w; a.w_t = w_t; a.u = u; a.state = state; a.state_slot = state_slot;
    a.state_half = state_half; a.q_start = q_start; a.slots = slots; a.positions = positions; a.o = o; a.o_t = o_t; a.H = H; a.d = d;
    a.vec = d % 4 == 0 && rkv_t % 4 == 0 && w_t % 4 == 0 && ((size_t)r | (size_t)k | (size_t)v | (size_t)w) % 16 == 0;
    const int nr = wkv_rows_per_lane(d);
    a.blocks = (d + WK_COLS - 1) / WK_COLS;
    const bool cut = segments > 1;
    LLMP_REQUIRE(!cut || (scratch && (size_t)scratch % 16 == 0 && seg_tokens > 0 && seg_tokens % WK_CHUNK == 0 && (long)segments * a.blocks <= 65535),
                 "wkv_scan: segments need scratch and a length that is a multiple of %d", WK_CHUNK);
    a.segments = cut ? segments : 1;
    a.seg_tokens = cut ? seg_tokens : 0x3fffffff;
    a.ends = scratch;
    a.decays = cut ? scratch + (size_t)R * segments * llmp_wkv_state_entries(H, d) : nullptr;
    const size_t smem = sizeof(float) * ((size_t)16 * nr + (size_t)WK_STAGES * WK_CHUNK * (48 * nr + WK_COLS));
    const dim3 grid(R, H, a.blocks * a.segments), later(R, H, a.blocks * (a.segments - 1));
#define LLMP_WKV(NR)                                                                                        \
    if (nr == NR) {                                                                                         \
        LLMP_ALLOW_SMEM((wkv_scan_kernel<NR, 0>), smem);                                                    \
        llmp_launch_dependent(wkv_scan_kernel<NR, 0>, grid, dim3(WK_THREADS), smem, stream, a);             \
        if (cut) {                                                                                          \
            LLMP_ALLOW_SMEM((wkv_scan_kernel<NR, 1>), smem);                                                \
            llmp_launch_dependent(wkv_scan_kernel<NR, 1>, later, dim3(WK_THREADS), smem, stream, a);        \
        }                                                                                                   \
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
    int group = 32;
    const bool vec = d % 4 == 0 && d <= 128 && o_t % 4 == 0 && gate_t % 4 == 0 && out_t % 4 == 0 &&
                     ((size_t)o | (size_t)gate | (size_t)weight | (size_t)out) % 16 == 0;
    if (vec) for (group = 1; 4 * group < d;) group *= 2;
    const dim3 grid((unsigned)((items * group + 127) / 128));
#define LLMP_WKV_GATE(T, VEC) \
    llmp_launch_dependent(wkv_gate_kernel<T, VEC>, grid, dim3(128), 0, stream, o, o_t, gate, gate_t, weight, (T*)out, out_t, items, H, d, group, eps)
    if (out_dtype == LLMP_BF16) { if (vec) LLMP_WKV_GATE(bf16, true); else LLMP_WKV_GATE(bf16, false); }
    else { if (vec) LLMP_WKV_GATE(float, true); else LLMP_WKV_GATE(float, false); }
#undef LLMP_WKV_GATE
    return llmp_check_launch("wkv_gate");
}
