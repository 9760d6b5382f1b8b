// Softmax attention with grouped key/value heads whose scores are capped and lose a distance bias, over a sliding
// window that keeps the first tokens, with a sink in the denominator and a gate on the output.
//
// With H query heads, G key/value heads (head h uses key/value head h / (H / G)), keys of d and values of dv entries,
// for the token at position i and a key at position j <= i:
//   seen(i, j) = i - j < window  or  j < keep_first                     (window 0: every j <= i)
//   and, with a chunk size n > 0, i / n = j / n (whole division)
//   s = (q . k) * scale;  s <- cap * tanh(s / cap) if cap > 0;  s <- s - slope[h] * (i - j)  if slopes are given
//   p_j = exp(s_j) / (exp(sink[h]) + sum_seen exp(s_j))                 (without a sink: the plain softmax)
//   o_h = sum_j p_j v_j;   o_h <- o_h * sigmoid(gate)  if a gate is given (a number per channel, or one per head)
// Scores, the cap, the bias, the softmax and the weighted sums are float32.
//
// capped_qkv_post: adds the projections' biases to the float32 product [q | k | v], divides every value head by its
// root mean square (if asked), writes the queries in the compute type and the token's cache rows [k | v] per key/value
// head into its page slot.
//
// capped_rows_post: the same step for designs that norm the whole rows of q and of k (before they are cut into heads) and
// may rotate them: q and k divided by their root mean square times a weight per entry, the first rot entries of every head
// rotated by the token's angles, values as projected (from their own columns, or the projected keys themselves).
//
// capped_attention (any sizes, float32 or bfloat16): a block per (token, key/value head, up to 8 heads of the group), a
// warp per query head. Keys are walked in tiles of 32 aligned to key 0; tiles that hold no key the token sees are
// skipped, and rows of keys it does not see are never read (their pages may be gone). A row's operations depend on its
// position alone, not on the step.
#include "common.cuh"

namespace {

constexpr int CA_KEYS = 32;
constexpr int CA_WARPS = 8;

template <typename T>
__global__ void capped_qkv_post_kernel(const float* __restrict__ qkv, long qkv_t, const void* __restrict__ bias, int bias_bf16,
                                       float v_eps, int v_norm, T* __restrict__ q_out, long q_out_t, const int* __restrict__ slots,
                                       T* __restrict__ pages, int page_size, int H, int G, int d, int dv) {
    pdl_wait();                                    // what the kernels before wrote is complete
    pdl_trigger();
    const int n = blockIdx.x;
    const float* row = qkv + (size_t)n * qkv_t;
    const int slot = slots ? slots[n] : -1;
    const int rs = d + dv;
    T* page_row = nullptr;
    if (pages && slot >= 0) page_row = pages + (((size_t)(slot / page_size) * G) * page_size + slot % page_size) * rs;
    const size_t head_stride = (size_t)page_size * rs;
    for (int i = threadIdx.x; i < (H + G) * d; i += blockDim.x) {
        const int head = i / d, c = i % d;
        const float v = row[i] + (bias ? load_as_float(bias, bias_bf16, i) : 0.f);
        if (head < H) q_out[(size_t)n * q_out_t + i] = from_float<T>(v);
        else if (page_row) page_row[(size_t)(head - H) * head_stride + c] = from_float<T>(v);
    }
    if (!page_row) return;
    // values: a warp per key/value head in turn
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    const int v_at = (H + G) * d;
    for (int g = warp; g < G; g += nw) {
        float ss = 0.f;
        for (int c = lane; c < dv; c += 32) {
            const float v = row[v_at + g * dv + c] + (bias ? load_as_float(bias, bias_bf16, v_at + g * dv + c) : 0.f);
            ss = fmaf(v, v, ss);
        }
        ss = warp_sum(ss);
        const float f = v_norm ? 1.f / sqrtf(ss / (float)dv + v_eps) : 1.f;
        for (int c = lane; c < dv; c += 32) {
            const float v = row[v_at + g * dv + c] + (bias ? load_as_float(bias, bias_bf16, v_at + g * dv + c) : 0.f);
            page_row[(size_t)g * head_stride + d + c] = from_float<T>(v * f);
        }
    }
}

struct RowsPostArgs {
    const float* proj; long proj_t;           // [tokens, q | k | ..]
    const float* qw; const float* kw;         // [H d], [G d]: weights of the row norms
    float eps;
    const float* cos_t; const float* sin_t;   // [tokens, rot / 2] or null
    int rot, interleaved;
    void* q_out; long q_out_t;
    const int* slots; void* pages;            // null: the queries alone
    int page_size, H, G, d, dv;
    int v_at;                                 // first column of the values
};

// Entry i of a row whose heads have d entries, normed by f and w, rotated within its head.
__device__ __forceinline__ float rows_entry(const RowsPostArgs& a, const float* row, const float* w, float f, const float* cs, const float* sn,
                                            int i) {
    const float v = row[i] * f * w[i];
    const int c = i % a.d;
    if (c >= a.rot) return v;
    const int half = a.rot >> 1;
    const bool first = a.interleaved ? !(c & 1) : c < half;
    const int at = a.interleaved ? c >> 1 : (first ? c : c - half);
    const int other = i + (a.interleaved ? (first ? 1 : -1) : (first ? half : -half));
    const float o = row[other] * f * w[other];
    return first ? v * cs[at] - o * sn[at] : v * cs[at] + o * sn[at];
}

template <typename T> __device__ __forceinline__ void rows_store4(T* p, float4 v);
template <> __device__ __forceinline__ void rows_store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void rows_store4<bf16>(bf16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}

// A block per token. VEC: pieces of four entries (d, dv, rot multiples of 4, and rot / 2 too in the half-split layout).
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) capped_rows_post_kernel(const RowsPostArgs a) {
    __shared__ float scratch[32];
    pdl_wait();                                    // what the kernels before wrote is complete
    pdl_trigger();
    const int n = blockIdx.x;
    const float* row = a.proj + (size_t)n * a.proj_t;
    const int slot = a.pages ? a.slots[n] : -1;
    const int nq = a.H * a.d, nk = a.pages ? a.G * a.d : 0, nv = a.pages ? a.G * a.dv : 0;
    float sq = 0.f, sk = 0.f;
    if (VEC) {
        for (int i = threadIdx.x * 4; i < nq + nk; i += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(row + i);
            const float s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
            if (i < nq) sq += s; else sk += s;
        }
    } else {
        for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
            const float v = row[i];
            if (i < nq) sq = fmaf(v, v, sq); else sk = fmaf(v, v, sk);
        }
    }
    sq = block_sum(sq, scratch);
    const float fq = 1.f / sqrtf(sq / (float)nq + a.eps);
    float fk = 0.f;
    if (nk > 0) {
        sk = block_sum(sk, scratch);
        fk = 1.f / sqrtf(sk / (float)nk + a.eps);
    }
    const int half = a.rot >> 1;
    const float* cs = a.cos_t ? a.cos_t + (size_t)n * half : nullptr;
    const float* sn = a.sin_t ? a.sin_t + (size_t)n * half : nullptr;
    T* qo = reinterpret_cast<T*>(a.q_out) + (size_t)n * a.q_out_t;
    const int rs = a.d + a.dv;
    T* page_row = nullptr;
    if (slot >= 0) page_row = reinterpret_cast<T*>(a.pages) + (((size_t)(slot / a.page_size) * a.G) * a.page_size + slot % a.page_size) * rs;
    const size_t head_stride = (size_t)a.page_size * rs;
    if (VEC) {
        for (int i = threadIdx.x * 4; i < nq + nk + nv; i += blockDim.x * 4) {
            if (i >= nq && !page_row) return;
            if (i >= nq + nk) {                    // values as projected
                const int j = i - nq - nk;
                rows_store4(page_row + (size_t)(j / a.dv) * head_stride + a.d + j % a.dv, *reinterpret_cast<const float4*>(row + a.v_at + j));
                continue;
            }
            const bool is_q = i < nq;
            const int j = is_q ? i : i - nq, c = j % a.d;
            const float f = is_q ? fq : fk;
            float4 v = *reinterpret_cast<const float4*>(row + i);
            const float4 w = *reinterpret_cast<const float4*>((is_q ? a.qw : a.kw) + j);
            v = make_float4(v.x * f * w.x, v.y * f * w.y, v.z * f * w.z, v.w * f * w.w);
            if (c < a.rot && !a.interleaved) {     // the piece of the pairs' other entries lies rot / 2 before or behind
                const bool first = c < half;
                const int at = first ? c : c - half, to = first ? half : -half;
                const float4 ov = *reinterpret_cast<const float4*>(row + i + to), ow = *reinterpret_cast<const float4*>((is_q ? a.qw : a.kw) + j + to);
                const float4 co = *reinterpret_cast<const float4*>(cs + at), si = *reinterpret_cast<const float4*>(sn + at);
                const float fs = first ? -f : f;
                v = make_float4(v.x * co.x + ov.x * fs * ow.x * si.x, v.y * co.y + ov.y * fs * ow.y * si.y, v.z * co.z + ov.z * fs * ow.z * si.z,
                                v.w * co.w + ov.w * fs * ow.w * si.w);
            } else if (c < a.rot) {
                const float2 co = *reinterpret_cast<const float2*>(cs + (c >> 1)), si = *reinterpret_cast<const float2*>(sn + (c >> 1));
                v = make_float4(v.x * co.x - v.y * si.x, v.y * co.x + v.x * si.x, v.z * co.y - v.w * si.y, v.w * co.y + v.z * si.y);
            }
            if (is_q) rows_store4(qo + j, v);
            else rows_store4(page_row + (size_t)(j / a.d) * head_stride + c, v);
        }
    } else {
        for (int i = threadIdx.x; i < nq; i += blockDim.x) qo[i] = from_float<T>(rows_entry(a, row, a.qw, fq, cs, sn, i));
        if (!page_row) return;
        for (int i = threadIdx.x; i < nk; i += blockDim.x)
            page_row[(size_t)(i / a.d) * head_stride + i % a.d] = from_float<T>(rows_entry(a, row + nq, a.kw, fk, cs, sn, i));
        for (int i = threadIdx.x; i < nv; i += blockDim.x)
            page_row[(size_t)(i / a.dv) * head_stride + a.d + i % a.dv] = from_float<T>(row[a.v_at + i]);
    }
}

struct CappedArgs {
    const void* q; long q_t;                  // [tokens, H d]
    const void* pages;                        // [page, kv head, token in page, d + dv]
    const int* tables; int width;
    const int* token_request; const int* positions;
    const float* slopes;                      // [H] or null
    const float* sink;                        // [H] or null
    const float* gate; long gate_t;           // float32 [tokens, H dv] (a view), [tokens, H] with gate_heads, or null
    int gate_heads;
    void* out; long out_t;                    // [tokens, H dv]
    int H, G, d, dv, page_size, window, keep, chunk;
    float scale, cap;
};

template <typename T, int NO>
__global__ void __launch_bounds__(CA_WARPS * 32) capped_attention_kernel(const CappedArgs a) {
    extern __shared__ float smem[];
    const int d = a.d, dv = a.dv, rs = a.d + a.dv;
    const int ks = d | 1;                                    // odd row stride: the lanes of a warp hit different banks
    float* Ks = smem;                                        // [CA_KEYS][ks]
    float* Vs = Ks + CA_KEYS * ks;                           // [CA_KEYS][dv]
    float* qs = Vs + CA_KEYS * dv;                           // [CA_WARPS][d]
    float* ps = qs + CA_WARPS * d;                           // [CA_WARPS][CA_KEYS]
    const int n = blockIdx.x;
    const int hpg = a.H / a.G;
    const int chunks = (hpg + CA_WARPS - 1) / CA_WARPS;
    const int g = blockIdx.y / chunks;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int hl = (blockIdx.y % chunks) * CA_WARPS + warp;
    const bool active = hl < hpg;
    const int h = g * hpg + hl;
    const int pos = a.positions[n];
    const int* table = a.tables + (size_t)a.token_request[n] * a.width;
    const T* pages = reinterpret_cast<const T*>(a.pages);
    int lo_w = a.window > 0 ? max(0, pos - a.window + 1) : 0;             // first key of the window (and of the chunk)
    if (a.chunk > 0) lo_w = max(lo_w, pos / a.chunk * a.chunk);
    const int keep_end = min(a.keep, lo_w);                               // kept keys before the window: [0, keep_end)
    float slope = 0.f, m_run = -INFINITY, l_run = 0.f;
    if (active) {
        const T* q = reinterpret_cast<const T*>(a.q) + (size_t)n * a.q_t + (size_t)h * d;
        for (int i = lane; i < d; i += 32) qs[warp * d + i] = to_float(q[i]);
        if (a.slopes) slope = a.slopes[h];
        if (a.sink) { m_run = a.sink[h]; l_run = 1.f; }
    }
    float o[NO];
#pragma unroll
    for (int i = 0; i < NO; ++i) o[i] = 0.f;
    for (int k0 = 0; k0 <= pos; k0 += CA_KEYS) {
        if (k0 >= keep_end && k0 + CA_KEYS <= lo_w) {        // the tile lies between the kept keys and the window
            k0 = (lo_w / CA_KEYS) * CA_KEYS - CA_KEYS;
            continue;
        }
        __syncthreads();
        for (int j = warp; j < CA_KEYS; j += CA_WARPS) {     // a warp copies a key's row
            const int key = k0 + j;
            const bool seen = key <= pos && (key >= lo_w || key < keep_end);
            if (seen) {
                const int page = table[key / a.page_size];
                const T* row = pages + (((size_t)page * a.G + g) * a.page_size + key % a.page_size) * rs;
                for (int i = lane; i < d; i += 32) Ks[j * ks + i] = to_float(row[i]);
                for (int i = lane; i < dv; i += 32) Vs[j * dv + i] = to_float(row[d + i]);
            } else {
                for (int i = lane; i < d; i += 32) Ks[j * ks + i] = 0.f;
                for (int i = lane; i < dv; i += 32) Vs[j * dv + i] = 0.f;
            }
        }
        __syncthreads();
        if (!active) continue;
        const int key = k0 + lane;
        const bool valid = key <= pos && (key >= lo_w || key < keep_end);
        float s = 0.f;
        const float* kr = Ks + lane * ks;
        const float* qw = qs + warp * d;
        for (int i = 0; i < d; ++i) s = fmaf(qw[i], kr[i], s);
        s *= a.scale;
        if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
        s -= slope * (float)(pos - key);
        s = valid ? s : -INFINITY;
        const float m_new = fmaxf(m_run, warp_max(s));       // finite: a tile that is walked holds a key the token sees
        const float p = valid ? expf(s - m_new) : 0.f;
        const float alpha = expf(m_run - m_new);             // 0 at the first tile without a sink (m_run = -inf)
        l_run = l_run * alpha + warp_sum(p);
        m_run = m_new;
        ps[warp * CA_KEYS + lane] = p;
        __syncwarp();
#pragma unroll
        for (int i = 0; i < NO; ++i) {
            const int c = lane + 32 * i;
            if (c < dv) {
                float acc = o[i] * alpha;
                for (int j = 0; j < CA_KEYS; ++j) acc = fmaf(ps[warp * CA_KEYS + j], Vs[j * dv + c], acc);
                o[i] = acc;
            }
        }
        __syncwarp();
    }
    if (!active) return;
    const float inv = 1.f / l_run;
    T* dst = reinterpret_cast<T*>(a.out) + (size_t)n * a.out_t + (size_t)h * dv;
    const float* gate = a.gate ? a.gate + (size_t)n * a.gate_t + (a.gate_heads ? (size_t)h : (size_t)h * dv) : nullptr;
#pragma unroll
    for (int i = 0; i < NO; ++i) {
        const int c = lane + 32 * i;
        if (c < dv) {
            float v = o[i] * inv;
            if (gate) v = v / (1.f + expf(-gate[a.gate_heads ? 0 : c]));
            dst[c] = from_float<T>(v);
        }
    }
}

template <typename T>
int launch_capped(const CappedArgs& a, int N, cudaStream_t stream) {
    const size_t smem = ((size_t)CA_KEYS * ((a.d | 1) + a.dv) + (size_t)CA_WARPS * a.d + CA_WARPS * CA_KEYS) * sizeof(float);
    LLMP_REQUIRE(smem <= 200 * 1024, "capped_attention: heads of %d + %d entries do not fit shared memory", a.d, a.dv);
    const int hpg = a.H / a.G;
    const long blocks_y = (long)a.G * ((hpg + CA_WARPS - 1) / CA_WARPS);
    LLMP_REQUIRE(blocks_y <= 65535, "capped_attention: too many heads %d", a.H);
    dim3 grid(N, (unsigned)blocks_y);
#define LLMP_CA_LAUNCH(NO)                                                         \
    do {                                                                           \
        LLMP_ALLOW_SMEM((capped_attention_kernel<T, NO>), smem);                   \
        capped_attention_kernel<T, NO><<<grid, CA_WARPS * 32, smem, stream>>>(a);  \
    } while (0)
    if (a.dv <= 64) LLMP_CA_LAUNCH(2);
    else if (a.dv <= 128) LLMP_CA_LAUNCH(4);
    else if (a.dv <= 256) LLMP_CA_LAUNCH(8);
    else LLMP_CA_LAUNCH(16);
#undef LLMP_CA_LAUNCH
    return llmp_check_launch("capped_attention");
}

}  // namespace

LLMP_API int llmp_capped_qkv_post(const float* qkv, long qkv_t, const void* bias, int bias_dtype, float v_eps, int v_norm, void* q_out,
                                  int dtype, long q_out_t, const int* slots, void* pages, int page_size, int N, int H, int G, int d,
                                  int dv, cudaStream_t stream) {
    if (N <= 0) return 0;
    LLMP_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0, "capped_qkv_post: bad sizes heads=%d kv=%d dim=%d vdim=%d", H, G, d, dv);
    LLMP_REQUIRE(pages == nullptr || page_size > 0, "capped_qkv_post: pages without a page size");
    if (dtype == LLMP_F32)
        llmp_launch_dependent(capped_qkv_post_kernel<float>, dim3(N), dim3(256), 0, stream, qkv, qkv_t, bias, (int)(bias_dtype == LLMP_BF16), v_eps, v_norm, (float*)q_out,
                                                             q_out_t, slots, (float*)pages, page_size, H, G, d, dv);
    else
        llmp_launch_dependent(capped_qkv_post_kernel<bf16>, dim3(N), dim3(256), 0, stream, qkv, qkv_t, bias, (int)(bias_dtype == LLMP_BF16), v_eps, v_norm, (bf16*)q_out,
                                                            q_out_t, slots, (bf16*)pages, page_size, H, G, d, dv);
    return llmp_check_launch("capped_qkv_post");
}

LLMP_API int llmp_capped_rows_post(const float* proj, long proj_t, const float* qw, const float* kw, float eps, const float* cos_t,
                                   const float* sin_t, int rot, int interleaved, void* q_out, int dtype, long q_out_t, const int* slots,
                                   void* pages, int page_size, int v_at, int N, int H, int G, int d, int dv, cudaStream_t stream) {
    if (N <= 0) return 0;
    LLMP_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0 && qw && (!pages || (kw && slots && page_size > 0)),
                 "capped_rows_post: bad sizes heads=%d kv=%d dim=%d vdim=%d", H, G, d, dv);
    LLMP_REQUIRE(rot >= 0 && rot <= d && rot % 2 == 0 && (rot == 0 || (cos_t && sin_t)), "capped_rows_post: a rotation of %d entries needs its tables", rot);
    RowsPostArgs a;
    a.proj = proj; a.proj_t = proj_t; a.qw = qw; a.kw = kw; a.eps = eps; a.cos_t = cos_t; a.sin_t = sin_t; a.rot = rot; a.interleaved = interleaved;
    a.q_out = q_out; a.q_out_t = q_out_t; a.slots = slots; a.pages = pages; a.page_size = page_size; a.H = H; a.G = G; a.d = d; a.dv = dv; a.v_at = v_at;
    const bool vec = d % 4 == 0 && dv % 4 == 0 && rot % 4 == 0 && (rot == 0 || interleaved || rot % 8 == 0) && proj_t % 4 == 0 && v_at % 4 == 0 && q_out_t % 4 == 0 &&
                     ((size_t)proj | (size_t)qw | (size_t)kw | (size_t)cos_t | (size_t)sin_t | (size_t)q_out | (size_t)pages) % 16 == 0;
    void (*kernel)(const RowsPostArgs) = dtype == LLMP_F32 ? (vec ? capped_rows_post_kernel<float, true> : capped_rows_post_kernel<float, false>)
                                                           : (vec ? capped_rows_post_kernel<bf16, true> : capped_rows_post_kernel<bf16, false>);
    llmp_launch_dependent(kernel, dim3(N), dim3(256), 0, stream, a);
    return llmp_check_launch("capped_rows_post");
}

LLMP_API int llmp_capped_attention(const void* q, long q_t, const void* pages, int dtype, const int* tables, int width,
                                   const int* token_request, const int* positions, const float* slopes, const float* sink,
                                   const float* gate, long gate_t, int gate_heads, void* out, long out_t, int N, int H, int G, int d,
                                   int dv, int page_size, int window, int keep, int chunk, float scale, float cap, cudaStream_t stream) {
    if (N <= 0) return 0;
    LLMP_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && dv > 0 && dv <= 512 && page_size > 0 && width > 0 && window >= 0 && keep >= 0 && chunk >= 0,
                 "capped_attention: bad sizes heads=%d kv=%d dim=%d vdim=%d page=%d width=%d", H, G, d, dv, page_size, width);
    CappedArgs a;
    a.gate_heads = gate_heads; a.chunk = chunk;
    a.q = q; a.q_t = q_t; a.pages = pages; a.tables = tables; a.width = width; a.token_request = token_request; a.positions = positions;
    a.slopes = slopes; a.sink = sink; a.gate = gate; a.gate_t = gate_t; a.out = out; a.out_t = out_t;
    a.H = H; a.G = G; a.d = d; a.dv = dv; a.page_size = page_size; a.window = window; a.keep = keep; a.scale = scale; a.cap = cap;
    return dtype == LLMP_F32 ? launch_capped<float>(a, N, stream) : launch_capped<bf16>(a, N, stream);
}
