// Hyper-connections: the residual stream as several copies ("streams") of the hidden state that a sublayer reads and
// writes through small learned matrices. One kernel does what lies between two sublayers, per row (token):
//   y_j  = addend_j, or addend_j / sqrt(mean(addend_j^2) + eps_j) * w_j    (j = 0, 1: one or two addends)
//   y    = (f_0 y_0 + f_1 y_1) * scale[column]                               (scale: optional)
//   x_t <- sum_s mix[s, t] x_s + out[t] y                                    (all streams at once from the old ones; with `mix`)
//   u    = sum_s in[s] x_s                                                   (without `in`: the sum of the streams)
//   h    = u / sqrt(mean(u^2) + eps) * w                                     (without `w`: u itself; optional)
// The streams, every statistic and every sum are float32. Streams that are still all equal are read from one row
// (src_s = 0). With `rows` the chosen rows alone are computed and the streams stay as they are.
#include "common.cuh"

namespace {

struct StreamArgs {
    const float* src; long src_t, src_s;          // x_s of token t at src + t src_t + s src_s
    float* dst;                                   // [tokens][S][H], or null
    const void* y[2]; int y_bf16[2]; const float* yw[2]; float yeps[2], yf[2];
    const float* scale; const float* mix; const float* out_w; const float* in_w;
    const void* w; int w_bf16; float eps;
    void* out; int out_bf16;
    const int* rows; int S, H;
};

constexpr int HC_MAX_STREAMS = 16;

// Any sizes: a block per row, the combined row in shared memory.
__global__ void stream_step_kernel(const StreamArgs a) {
    extern __shared__ float u_row[];
    __shared__ float scratch[32];
    __shared__ float coef[HC_MAX_STREAMS * HC_MAX_STREAMS + 2 * HC_MAX_STREAMS];
    pdl_wait();
    pdl_trigger();
    const int H = a.H, S = a.S;
    const int m = blockIdx.x, r = a.rows ? a.rows[m] : m;
    float* mix = coef;
    float* ow = coef + HC_MAX_STREAMS * HC_MAX_STREAMS;
    float* iw = ow + HC_MAX_STREAMS;
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix[i] = a.mix ? a.mix[i] : 0.f;
    for (int i = threadIdx.x; i < S; i += blockDim.x) {
        ow[i] = a.mix ? a.out_w[i] : 0.f;
        iw[i] = a.in_w ? a.in_w[i] : 1.f;
    }
    __syncthreads();
    float f[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        f[j] = a.yf[j];
        if (a.y[j] && a.yw[j]) {
            float ss = 0.f;
            for (int c = threadIdx.x; c < H; c += blockDim.x) {
                const float v = load_as_float(a.y[j], a.y_bf16[j], (size_t)r * H + c);
                ss = fmaf(v, v, ss);
            }
            ss = block_sum(ss, scratch);
            f[j] *= rsqrtf(ss / (float)H + a.yeps[j]);
        }
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float x[HC_MAX_STREAMS];
        for (int s = 0; s < S; ++s) x[s] = a.src[(size_t)r * a.src_t + (size_t)s * a.src_s + c];
        float u = 0.f;
        if (a.mix) {
            float y = 0.f;
#pragma unroll
            for (int j = 0; j < 2; ++j)
                if (a.y[j]) {
                    const float v = load_as_float(a.y[j], a.y_bf16[j], (size_t)r * H + c) * f[j];
                    y += a.yw[j] ? v * a.yw[j][c] : v;
                }
            if (a.scale) y *= a.scale[c];
            for (int t = 0; t < S; ++t) {
                float v = ow[t] * y;
                for (int s = 0; s < S; ++s) v = fmaf(mix[s * S + t], x[s], v);
                if (a.dst) a.dst[((size_t)r * S + t) * H + c] = v;
                u = fmaf(iw[t], v, u);
            }
        } else {
            for (int s = 0; s < S; ++s) u = fmaf(iw[s], x[s], u);
        }
        u_row[c] = u;
        ss = fmaf(u, u, ss);
    }
    if (!a.out) return;
    float g = 1.f;
    if (a.w) g = rsqrtf(block_sum(ss, scratch) / (float)H + a.eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = a.w ? u_row[c] * g * load_as_float(a.w, a.w_bf16, c) : u_row[c];
        if (a.out_bf16) reinterpret_cast<bf16*>(a.out)[(size_t)m * H + c] = __float2bfloat16_rn(v);
        else reinterpret_cast<float*>(a.out)[(size_t)m * H + c] = v;
    }
}

__device__ __forceinline__ float4 hc_load4(const void* p, int is_bf16, size_t i4) {
    if (!is_bf16) return reinterpret_cast<const float4*>(p)[i4];
    const uint2 raw = reinterpret_cast<const uint2*>(p)[i4];
    const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), hi = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    return make_float4(__low2float(lo), __high2float(lo), __low2float(hi), __high2float(hi));
}
__device__ __forceinline__ void hc_store4(void* p, int is_bf16, size_t i4, float4 v) {
    if (!is_bf16) { reinterpret_cast<float4*>(p)[i4] = v; return; }
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    reinterpret_cast<uint2*>(p)[i4] = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}
__device__ __forceinline__ float4 hc_fma4(float k, float4 v, float4 acc) {
    return make_float4(fmaf(k, v.x, acc.x), fmaf(k, v.y, acc.y), fmaf(k, v.z, acc.z), fmaf(k, v.w, acc.w));
}
__device__ __forceinline__ float4 hc_mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float hc_sq4(float4 v, float ss) { return fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, fmaf(v.x, v.x, ss)))); }

// The same in 16-byte accesses with all streams of the thread's columns in registers, which are loaded before anything is
// summed: S streams (a template parameter), NP pieces of four columns a thread.
template <int S, int NP>
__global__ void __launch_bounds__(512) stream_step_rows_kernel(const StreamArgs a) {
    __shared__ float scratch[2][32];
    pdl_wait();
    pdl_trigger();
    const int H4 = a.H >> 2;
    const int m = blockIdx.x, r = a.rows ? a.rows[m] : m;
    float4 x[NP][S], y[NP][2];
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int p = 0; p < NP; ++p) {
        const int i = threadIdx.x + p * blockDim.x;
        y[p][0] = y[p][1] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int s = 0; s < S; ++s) x[p][s] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < H4) {
            if (a.y[0]) y[p][0] = hc_load4(a.y[0], a.y_bf16[0], (size_t)r * H4 + i);
            if (a.y[1]) y[p][1] = hc_load4(a.y[1], a.y_bf16[1], (size_t)r * H4 + i);
#pragma unroll
            for (int s = 0; s < S; ++s) x[p][s] = *reinterpret_cast<const float4*>(a.src + (size_t)r * a.src_t + (size_t)s * a.src_s + 4 * i);
        }
        s0 = hc_sq4(y[p][0], s0);
        s1 = hc_sq4(y[p][1], s1);
    }
    float f0 = a.yf[0], f1 = a.yf[1];
    if (a.yw[0] || a.yw[1]) {                      // both sums in one exchange
        s0 = warp_sum(s0);
        s1 = warp_sum(s1);
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
        if (lane == 0) { scratch[0][warp] = s0; scratch[1][warp] = s1; }
        __syncthreads();
        s0 = warp_sum(lane < nw ? scratch[0][lane] : 0.f);
        s1 = warp_sum(lane < nw ? scratch[1][lane] : 0.f);
        if (a.yw[0]) f0 *= rsqrtf(s0 / (float)a.H + a.yeps[0]);
        if (a.yw[1]) f1 *= rsqrtf(s1 / (float)a.H + a.yeps[1]);
    }
    float4 u[NP];
    float ss = 0.f;
    constexpr int KEPT = S <= 4 ? S : 0;           // the matrix in registers where it is small
    float in_w[S], out_w[S], mix[KEPT * KEPT + 1];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        in_w[s] = a.in_w ? a.in_w[s] : 1.f;
        out_w[s] = a.mix ? a.out_w[s] : 0.f;
    }
#pragma unroll
    for (int k = 0; k < KEPT * KEPT; ++k) mix[k] = a.mix ? a.mix[k] : 0.f;
#pragma unroll
    for (int p = 0; p < NP; ++p) {
        const int i = threadIdx.x + p * blockDim.x;
        u[p] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i >= H4) continue;
        if (a.mix) {
            float4 v = make_float4(y[p][0].x * f0, y[p][0].y * f0, y[p][0].z * f0, y[p][0].w * f0);
            if (a.yw[0]) v = hc_mul4(v, reinterpret_cast<const float4*>(a.yw[0])[i]);
            if (a.y[1]) {
                float4 v1 = make_float4(y[p][1].x * f1, y[p][1].y * f1, y[p][1].z * f1, y[p][1].w * f1);
                if (a.yw[1]) v1 = hc_mul4(v1, reinterpret_cast<const float4*>(a.yw[1])[i]);
                v.x += v1.x; v.y += v1.y; v.z += v1.z; v.w += v1.w;
            }
            if (a.scale) v = hc_mul4(v, reinterpret_cast<const float4*>(a.scale)[i]);
#pragma unroll
            for (int t = 0; t < S; ++t) {
                float4 n = make_float4(out_w[t] * v.x, out_w[t] * v.y, out_w[t] * v.z, out_w[t] * v.w);
#pragma unroll
                for (int s = 0; s < S; ++s) n = hc_fma4(KEPT ? mix[s * KEPT + t] : a.mix[s * S + t], x[p][s], n);
                if (a.dst) *reinterpret_cast<float4*>(a.dst + ((size_t)r * S + t) * a.H + 4 * i) = n;
                u[p] = hc_fma4(in_w[t], n, u[p]);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) u[p] = hc_fma4(in_w[s], x[p][s], u[p]);
        }
        ss = hc_sq4(u[p], ss);
    }
    if (!a.out) return;
    float g = 1.f;
    if (a.w) {
        __syncthreads();                           // the first exchange's sums have been read
        g = rsqrtf(block_sum(ss, scratch[0]) / (float)a.H + a.eps);
    }
#pragma unroll
    for (int p = 0; p < NP; ++p) {
        const int i = threadIdx.x + p * blockDim.x;
        if (i >= H4) continue;
        float4 v = make_float4(u[p].x * g, u[p].y * g, u[p].z * g, u[p].w * g);
        if (a.w) v = hc_mul4(v, hc_load4(a.w, a.w_bf16, i));
        hc_store4(a.out, a.out_bf16, (size_t)m * H4 + i, v);
    }
}

template <int S> bool launch_rows(const StreamArgs& a, int M, cudaStream_t stream) {
    const int H4 = a.H / 4;
    auto threads_for = [](int n) { return (n + 31) / 32 * 32; };
    // the same shape for few and many rows: a row's sums never depend on how many rows a step has
    if (H4 <= 512) {
        llmp_launch_dependent(stream_step_rows_kernel<S, 1>, dim3(M), dim3(threads_for(H4)), 0, stream, a);
        return true;
    }
    if constexpr (S <= 8) {
        if (H4 <= 1024) {
            llmp_launch_dependent(stream_step_rows_kernel<S, 2>, dim3(M), dim3(threads_for((H4 + 1) / 2)), 0, stream, a);
            return true;
        }
    }
    if constexpr (S <= 4) {
        if (H4 <= 2048) {
            llmp_launch_dependent(stream_step_rows_kernel<S, 4>, dim3(M), dim3(threads_for((H4 + 3) / 4)), 0, stream, a);
            return true;
        }
    }
    return false;
}

}  // namespace

LLMP_API int llmp_stream_step(const float* src, long src_t, long src_s, float* dst, const void* y0, int y0_dtype, const float* yw0,
                              float yeps0, float yf0, const void* y1, int y1_dtype, const float* yw1, float yeps1, float yf1,
                              const float* scale, const float* mix, const float* out_w, const float* in_w, const void* w, int w_dtype,
                              float eps, void* out, int out_dtype, const int* rows, int M, int S, int H, cudaStream_t stream) {
    if (M <= 0) return 0;
    LLMP_REQUIRE(H > 0 && (size_t)H * 4 <= 200 * 1024 && S > 0 && S <= HC_MAX_STREAMS, "stream_step: %d streams of width %d", S, H);
    LLMP_REQUIRE(!mix || out_w, "stream_step: an update needs the weights its addend enters with");
    LLMP_REQUIRE(!(rows && dst), "stream_step: chosen rows leave the streams as they are");
    StreamArgs a;
    a.src = src; a.src_t = src_t; a.src_s = src_s; a.dst = dst;
    a.y[0] = y0; a.y_bf16[0] = y0_dtype == LLMP_BF16; a.yw[0] = yw0; a.yeps[0] = yeps0; a.yf[0] = yf0;
    a.y[1] = y1; a.y_bf16[1] = y1_dtype == LLMP_BF16; a.yw[1] = yw1; a.yeps[1] = yeps1; a.yf[1] = yf1;
    a.scale = scale; a.mix = mix; a.out_w = out_w; a.in_w = in_w;
    a.w = w; a.w_bf16 = w_dtype == LLMP_BF16; a.eps = eps; a.out = out; a.out_bf16 = out_dtype == LLMP_BF16;
    a.rows = rows; a.S = S; a.H = H;
    auto aligned = [](const void* q, int bf) { return q == nullptr || ((size_t)q % (bf ? 8 : 16)) == 0; };
    if (H % 4 == 0 && src_t % 4 == 0 && src_s % 4 == 0 && aligned(src, 0) && aligned(dst, 0) && aligned(y0, a.y_bf16[0]) &&
        aligned(y1, a.y_bf16[1]) && aligned(yw0, 0) && aligned(yw1, 0) && aligned(scale, 0) && aligned(w, a.w_bf16) &&
        aligned(out, a.out_bf16)) {
        bool done = false;
        switch (S) {
            case 1: done = launch_rows<1>(a, M, stream); break;
            case 2: done = launch_rows<2>(a, M, stream); break;
            case 3: done = launch_rows<3>(a, M, stream); break;
            case 4: done = launch_rows<4>(a, M, stream); break;
            case 5: done = launch_rows<5>(a, M, stream); break;
            case 6: done = launch_rows<6>(a, M, stream); break;
            case 8: done = launch_rows<8>(a, M, stream); break;
        }
        if (done) return llmp_check_launch("stream_step");
    }
    const size_t smem = (size_t)H * sizeof(float);
    LLMP_ALLOW_SMEM(stream_step_kernel, smem);
    llmp_launch_dependent(stream_step_kernel, dim3(M), dim3(H >= 2048 ? 512 : 128), smem, stream, a);
    return llmp_check_launch("stream_step");
}
