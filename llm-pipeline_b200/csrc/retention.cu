// Rows of retention's queries and keys, in place: the first `rot` entries of every head turn by the token's position (entry i
// with i + rot / 2, the half-split layout; cos and sin float32 [tokens, rot / 2]), and the second half of the heads (the keys)
// is scaled by `factor` after the rotation.
#include "common.cuh"

namespace {

__global__ void rotate_heads_kernel(float* __restrict__ x, long x_t, const float* __restrict__ cos, const float* __restrict__ sin, int rot,
                                    int heads, int scaled_from, int dim, float factor) {
    const int n = blockIdx.x, half = rot >> 1, per = half + dim - rot;       // pairs, then single entries, of a head
    float* row = x + (size_t)n * x_t;
    for (int i = threadIdx.x; i < heads * per; i += blockDim.x) {
        const int h = i / per, j = i % per;
        const float f = h >= scaled_from ? factor : 1.f;
        float* head = row + (size_t)h * dim;
        if (j < half) {
            const float c = cos[(size_t)n * half + j], s = sin[(size_t)n * half + j];
            const float u = head[j], v = head[j + half];
            head[j] = (u * c - v * s) * f;
            head[j + half] = (v * c + u * s) * f;
        } else if (h >= scaled_from) {
            head[rot + j - half] *= f;
        }
    }
}

}  // namespace

LLMP_API int llmp_rotate_heads(float* x, long x_t, const float* cos, const float* sin, int rot, int heads, int scaled_from, int dim,
                               float factor, int tokens, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    LLMP_REQUIRE(heads > 0 && dim > 0 && rot >= 0 && rot % 2 == 0 && rot <= dim && (rot == 0 || (cos && sin)),
                 "rotate_heads: %d rotated entries of heads of %d", rot, dim);
    const int work = heads * (dim - rot / 2);
    rotate_heads_kernel<<<tokens, work >= 512 ? 512 : (work + 31) / 32 * 32, 0, stream>>>(x, x_t, cos, sin, rot, heads, scaled_from, dim, factor);
    return llmp_check_launch("rotate_heads");
}
