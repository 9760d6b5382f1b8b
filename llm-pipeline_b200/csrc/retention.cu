// Rows of retention's queries and keys: the first `rot` entries of every head turn by the token's position (entry i with
// i + rot / 2, the half-split layout; cos and sin float32 [tokens, rot / 2]), and the heads from `scaled_from` on (the keys)
// are scaled by `factor` after the rotation. In place (float32), or into bfloat16 rows of their own together with `extra`
// further columns as they are (the values), or both.
#include "common.cuh"

namespace {

struct RotateArgs {
    float* x; long x_t; bf16* typed; long typed_t;
    const float* cos; const float* sin;
    int rot, heads, scaled_from, dim, extra, in_place;
    float factor;
};

__global__ void rotate_heads_kernel(const RotateArgs a) {
    const int n = blockIdx.x, half = a.rot >> 1, per = half + a.dim - a.rot;       // pairs, then single entries, of a head
    float* row = a.x + (size_t)n * a.x_t;
    bf16* typed = a.typed ? a.typed + (size_t)n * a.typed_t : nullptr;
    for (int i = threadIdx.x; i < a.heads * per; i += blockDim.x) {
        const int h = i / per, j = i % per;
        const float f = h >= a.scaled_from ? a.factor : 1.f;
        const size_t head = (size_t)h * a.dim;
        if (j < half) {
            const float c = a.cos[(size_t)n * half + j], s = a.sin[(size_t)n * half + j];
            const float u = row[head + j], v = row[head + j + half];
            const float p = (u * c - v * s) * f, q = (v * c + u * s) * f;
            if (a.in_place) { row[head + j] = p; row[head + j + half] = q; }
            if (typed) { typed[head + j] = __float2bfloat16_rn(p); typed[head + j + half] = __float2bfloat16_rn(q); }
        } else {
            const size_t at = head + a.rot + j - half;
            const float p = row[at] * f;
            if (a.in_place && h >= a.scaled_from) row[at] = p;
            if (typed) typed[at] = __float2bfloat16_rn(p);
        }
    }
    if (typed)
        for (int i = threadIdx.x; i < a.extra; i += blockDim.x) typed[(size_t)a.heads * a.dim + i] = __float2bfloat16_rn(row[(size_t)a.heads * a.dim + i]);
}

__device__ __forceinline__ float4 rt_load(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void rt_store(float* row, bf16* typed, size_t at, float4 v, bool in_place) {
    if (in_place) *reinterpret_cast<float4*>(row + at) = v;
    if (typed) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(typed + at) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
    }
}

// The same with four entries (pairs) a thread and step: rot / 2 and dim are multiples of 4.
__global__ void __launch_bounds__(512) rotate_heads_by_4_kernel(const RotateArgs a) {
    pdl_wait();
    pdl_trigger();
    const int n = blockIdx.x, half = a.rot >> 1, h4 = half >> 2, per = h4 + ((a.dim - a.rot) >> 2);
    float* row = a.x + (size_t)n * a.x_t;
    bf16* typed = a.typed ? a.typed + (size_t)n * a.typed_t : nullptr;
    for (int i = threadIdx.x; i < a.heads * per; i += blockDim.x) {
        const int h = i / per, j = i % per;
        const float f = h >= a.scaled_from ? a.factor : 1.f;
        const size_t head = (size_t)h * a.dim;
        if (j < h4) {
            const float4 c = rt_load(a.cos + (size_t)n * half + 4 * j), s = rt_load(a.sin + (size_t)n * half + 4 * j);
            const size_t at = head + 4 * j;
            const float4 u = rt_load(row + at), v = rt_load(row + at + half);
            rt_store(row, typed, at, make_float4((u.x * c.x - v.x * s.x) * f, (u.y * c.y - v.y * s.y) * f, (u.z * c.z - v.z * s.z) * f,
                                                 (u.w * c.w - v.w * s.w) * f), a.in_place);
            rt_store(row, typed, at + half, make_float4((v.x * c.x + u.x * s.x) * f, (v.y * c.y + u.y * s.y) * f, (v.z * c.z + u.z * s.z) * f,
                                                        (v.w * c.w + u.w * s.w) * f), a.in_place);
        } else {
            const size_t at = head + a.rot + 4 * (j - h4);
            const float4 v = rt_load(row + at);
            rt_store(row, typed, at, make_float4(v.x * f, v.y * f, v.z * f, v.w * f), a.in_place);
        }
    }
    if (typed)
        for (int i = threadIdx.x; i < a.extra >> 2; i += blockDim.x) {
            const size_t at = (size_t)a.heads * a.dim + 4 * i;
            rt_store(row, typed, at, rt_load(row + at), false);
        }
}

}  // namespace

LLMP_API int llmp_rotate_heads(float* x, long x_t, void* typed, long typed_t, int in_place, const float* cos, const float* sin, int rot, int heads,
                               int scaled_from, int dim, int extra, float factor, int tokens, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    LLMP_REQUIRE(heads > 0 && dim > 0 && extra >= 0 && rot >= 0 && rot % 2 == 0 && rot <= dim && (rot == 0 || (cos && sin)),
                 "rotate_heads: %d rotated entries of heads of %d", rot, dim);
    const RotateArgs a = {x, x_t, (bf16*)typed, typed_t, cos, sin, rot, heads, scaled_from, dim, extra, in_place, factor};
    const bool by4 = rot % 8 == 0 && dim % 4 == 0 && extra % 4 == 0 && x_t % 4 == 0 && typed_t % 4 == 0 && (uintptr_t)x % 16 == 0 &&
                     (uintptr_t)typed % 8 == 0 && ((uintptr_t)cos | (uintptr_t)sin) % 16 == 0;
    if (by4) {
        const int work = heads * (dim - rot / 2) / 4;
        llmp_launch_dependent(rotate_heads_by_4_kernel, dim3(tokens), dim3(work >= 512 ? 512 : (work + 31) / 32 * 32), 0, stream, a);
        return llmp_check_launch("rotate_heads");
    }
    const int work = heads * (dim - rot / 2);
    rotate_heads_kernel<<<tokens, work >= 512 ? 512 : (work + 31) / 32 * 32, 0, stream>>>(a);
    return llmp_check_launch("rotate_heads");
}
