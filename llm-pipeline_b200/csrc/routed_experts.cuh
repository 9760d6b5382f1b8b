// What the kernels of the routed experts share.
#pragma once
#include "common.cuh"

// form 0: clamped, the weight on the input; form 1: silu(g) u, the weight on the output; form 2: max(u, 0)^2 without a
// gate, the weight on the output
#define EXPERT_FORM_UNGATED 2
__device__ __forceinline__ float expert_act(float g, float u, float w, float limit, int form) {
    if (form == EXPERT_FORM_UNGATED) { u = fmaxf(u, 0.f); return w * (u * u); }
    if (form == 1) return w * (g / (1.f + expf(-g))) * u;
    g = fminf(w * g, limit);
    u = fminf(fmaxf(w * u, -limit), limit);
    return g * (1.f / (1.f + expf(-1.702f * g))) * (u + 1.f);
}
