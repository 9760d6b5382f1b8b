// The recurrences of state_space.cu for steps in which every request brings one token.
//   S <- a S + k v^T,   y = S^T q      with a scalar a per head
// A block takes one (request, head): its state [N, P] is read and written once, in 16-byte pieces whose lines are whole (a
// warp's lanes lie along a row), and the sums over the rows are added in shared memory. The state lives in the request's
// slot as two copies that take turns by the parity of the position; nothing of this step writes the copy that is read, so
// its loads are in flight before the kernel waits for the one before it. Two forms:
//   state space:  a = exp(-exp(A_log) dt), k = dt B, v = x, q = C, y + D x leaves float32
//   retention:    constant a; q and k are turned by the token's position and k scaled (the rows come as the product left
//                 them); the head's y is divided by its root mean square, times silu(gate), and leaves in the compute type
#include "common.cuh"

namespace {

constexpr int ST_THREADS = 256;
constexpr int ST_AHEAD = 16;             // 16-byte pieces of the state a thread has in flight

struct StepArgs {
    const float* q; const float* k; const float* v; long row_t;      // [rows, ..]: C, B, x or queries, keys, values
    const float* gate; long gate_t;                                  // retention
    const float* dt; long dt_t; const float* dt_bias; const float* a_log; const float* d_skip;   // state space
    const float* decay;                                              // retention: [2][H], the constants and what their float leaves
    const float* cos; const float* sin; int rot; float k_scale, eps;
    float* state; long state_slot; long state_half; const int* slots; const int* positions;
    void* out; long out_t;
    int H, G, N, P;
};

__device__ __forceinline__ float st_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

template <typename T, bool RETENTION>
__global__ void __launch_bounds__(ST_THREADS) state_step_kernel(const StepArgs a) {
    extern __shared__ __align__(16) float st_smem[];
    __shared__ float scratch[32];
    const int r = blockIdx.x, h = blockIdx.y;
    const int N = a.N, P = a.P, lanes = P >> 2, groups = ST_THREADS / lanes;      // threads along a row, rows at a time
    const int col = threadIdx.x % lanes, row = threadIdx.x / lanes;
    const bool busy = row < groups;
    float* qs = st_smem;                           // [N]
    float* ks = qs + N;                            // [N]
    float* ys = st_smem + ((2 * N + 3) & ~3);      // [groups][P]
    const int pos = a.positions[r];
    float* slot = a.state + (size_t)a.slots[r] * a.state_slot + (size_t)h * N * P + 4 * col;
    const float* rd = slot + ((pos + 1) & 1) * a.state_half;
    float* wr = slot + (pos & 1) * a.state_half;
    float4 S[ST_AHEAD];
#pragma unroll
    for (int i = 0; i < ST_AHEAD; ++i) {
        const int n = row + i * groups;
        if (busy && n < N) S[i] = *reinterpret_cast<const float4*>(rd + (size_t)n * P);
    }
    pdl_wait();
    pdl_trigger();
    const int g = h / (a.H / a.G);
    const float* q = a.q + (size_t)r * a.row_t + (size_t)g * N;
    const float* k = a.k + (size_t)r * a.row_t + (size_t)g * N;
    float decay, decay_lo = 0.f, in = 1.f;
    if constexpr (RETENTION) {
        decay = a.decay[h];
        decay_lo = a.decay[a.H + h];
        const int half = a.rot >> 1;
        const float* cs = a.cos + (size_t)r * half;
        const float* sn = a.sin + (size_t)r * half;
        for (int i = threadIdx.x; i < 2 * N; i += ST_THREADS) {
            const bool key = i >= N;
            const int c = key ? i - N : i;
            const float* x = key ? k : q;
            float v = x[c];
            if (c < half) v = v * cs[c] - x[c + half] * sn[c];
            else if (c < a.rot) v = v * cs[c - half] + x[c - half] * sn[c - half];
            (key ? ks : qs)[c] = key ? v * a.k_scale : v;
        }
    } else {
        in = st_softplus(a.dt[(size_t)r * a.dt_t + h] + a.dt_bias[h]);
        decay = expf(-expf(a.a_log[h]) * in);
        for (int i = threadIdx.x; i < N; i += ST_THREADS) { qs[i] = q[i]; ks[i] = k[i]; }
    }
    const float* vr = a.v + (size_t)r * a.row_t + (size_t)h * P + 4 * col;         // rows need no alignment
    const float4 v = make_float4(vr[0] * in, vr[1] * in, vr[2] * in, vr[3] * in);
    __syncthreads();
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int n0 = row; n0 < N; n0 += ST_AHEAD * groups) {
        if (!busy) break;
        if (n0 != row) {
#pragma unroll
            for (int i = 0; i < ST_AHEAD; ++i)
                if (n0 + i * groups < N) S[i] = *reinterpret_cast<const float4*>(rd + (size_t)(n0 + i * groups) * P);
        }
#pragma unroll
        for (int i = 0; i < ST_AHEAD; ++i) {
            const int n = n0 + i * groups;
            if (n >= N) continue;
            const float kn = ks[n], qn = qs[n];
            float4 s = S[i];
            float4 add = make_float4(kn * v.x, kn * v.y, kn * v.z, kn * v.w);
            if constexpr (RETENTION)
                add = make_float4(fmaf(decay_lo, s.x, add.x), fmaf(decay_lo, s.y, add.y), fmaf(decay_lo, s.z, add.z), fmaf(decay_lo, s.w, add.w));
            s = make_float4(fmaf(decay, s.x, add.x), fmaf(decay, s.y, add.y), fmaf(decay, s.z, add.z), fmaf(decay, s.w, add.w));
            *reinterpret_cast<float4*>(wr + (size_t)n * P) = s;
            y = make_float4(fmaf(qn, s.x, y.x), fmaf(qn, s.y, y.y), fmaf(qn, s.z, y.z), fmaf(qn, s.w, y.w));
        }
    }
    if (busy) *reinterpret_cast<float4*>(ys + (size_t)row * P + 4 * col) = y;
    __syncthreads();
    float ss = 0.f;
    for (int p = threadIdx.x; p < P; p += ST_THREADS) {
        float sum = 0.f;
        for (int i = 0; i < groups; ++i) sum += ys[i * P + p];
        if constexpr (RETENTION) {
            ys[p] = sum;                           // the first group's place: this thread alone reads and writes the column
            ss = fmaf(sum, sum, ss);
        } else {
            reinterpret_cast<float*>(a.out)[(size_t)r * a.out_t + (size_t)h * P + p] =
                fmaf(a.d_skip[h], a.v[(size_t)r * a.row_t + (size_t)h * P + p], sum);
        }
    }
    if constexpr (RETENTION) {
        const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)P + a.eps);
        for (int p = threadIdx.x; p < P; p += ST_THREADS) {
            const float z = a.gate[(size_t)r * a.gate_t + (size_t)h * P + p];
            reinterpret_cast<T*>(a.out)[(size_t)r * a.out_t + (size_t)h * P + p] = from_float<T>(ys[p] * inv * z * (1.f / (1.f + expf(-z))));
        }
    }
}

int check_step(const StepArgs& a, int R, const char* what, size_t& smem) {
    LLMP_REQUIRE(a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.H <= 65535 && a.N > 0 && a.P % 4 == 0 && a.P >= 4 && a.P <= 4 * ST_THREADS,
                 "%s: bad sizes heads=%d groups=%d state=%d x %d", what, a.H, a.G, a.N, a.P);
    LLMP_REQUIRE((uintptr_t)a.state % 16 == 0 && a.state_slot % 4 == 0 && a.state_half % 4 == 0, "%s: the state is not in 16-byte pieces", what);
    const int groups = ST_THREADS / (a.P / 4);
    smem = ((size_t)((2 * a.N + 3) & ~3) + (size_t)groups * a.P) * sizeof(float);
    LLMP_REQUIRE(smem <= 200 * 1024, "%s: a state of %d rows does not fit shared memory", what, a.N);
    return 0;
}

}  // namespace

LLMP_API int llmp_ssd_step(const float* xbc, long xbc_t, const float* dt, long dt_t, const float* dt_bias, const float* a_log,
                           const float* d_skip, float* state, long state_slot, long state_half, const int* slots, const int* positions,
                           float* y, long y_t, int R, int H, int G, int N, int P, cudaStream_t stream) {
    if (R <= 0) return 0;
    StepArgs a = {};
    a.v = xbc; a.k = xbc + (size_t)H * P; a.q = a.k + (size_t)G * N; a.row_t = xbc_t;
    a.dt = dt; a.dt_t = dt_t; a.dt_bias = dt_bias; a.a_log = a_log; a.d_skip = d_skip;
    a.state = state; a.state_slot = state_slot; a.state_half = state_half; a.slots = slots; a.positions = positions;
    a.out = y; a.out_t = y_t; a.H = H; a.G = G; a.N = N; a.P = P;
    size_t smem = 0;
    if (check_step(a, R, "ssd_step", smem)) return 1;
    LLMP_ALLOW_SMEM((state_step_kernel<float, false>), smem);
    llmp_launch_dependent(state_step_kernel<float, false>, dim3(R, H), dim3(ST_THREADS), smem, stream, a);
    return llmp_check_launch("ssd_step");
}

// q, k [rows, H N] and v, gate [rows, H P] with one stride, q and k before their rotation; out [rows, H P].
LLMP_API int llmp_retention_step(const float* q, const float* k, const float* v, const float* gate, long row_t, const float* cos, const float* sin,
                                 int rot, float k_scale, const float* decay, float eps, float* state, long state_slot, long state_half,
                                 const int* slots, const int* positions, void* out, int out_dtype, long out_t, int R, int H, int N, int P,
                                 cudaStream_t stream) {
    if (R <= 0) return 0;
    LLMP_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= N && (rot == 0 || (cos && sin)), "retention_step: %d rotated entries of heads of %d", rot, N);
    StepArgs a = {};
    a.q = q; a.k = k; a.v = v; a.row_t = row_t; a.gate = gate; a.gate_t = row_t; a.decay = decay;
    a.cos = cos; a.sin = sin; a.rot = rot; a.k_scale = k_scale; a.eps = eps;
    a.state = state; a.state_slot = state_slot; a.state_half = state_half; a.slots = slots; a.positions = positions;
    a.out = out; a.out_t = out_t; a.H = H; a.G = H; a.N = N; a.P = P;
    size_t smem = 0;
    if (check_step(a, R, "retention_step", smem)) return 1;
    if (out_dtype == LLMP_BF16) {
        LLMP_ALLOW_SMEM((state_step_kernel<bf16, true>), smem);
        llmp_launch_dependent(state_step_kernel<bf16, true>, dim3(R, H), dim3(ST_THREADS), smem, stream, a);
    } else {
        LLMP_ALLOW_SMEM((state_step_kernel<float, true>), smem);
        llmp_launch_dependent(state_step_kernel<float, true>, dim3(R, H), dim3(ST_THREADS), smem, stream, a);
    }
    return llmp_check_launch("retention_step");
}
