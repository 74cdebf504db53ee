// gla.cu -- gated linear attention: per head a [D, V] matrix S with a decay per key channel,
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   alpha = sigmoid(z)^(1/tau),  z = A2 (A1 h) + b,
// followed by an RMS norm of each head's o over V and the gate silu(W_g h).  q carries the factor D^(-1/2).  The recurrence, its
// decays and the norm are f32 whatever the model's dtype; q, k, v, the gate and A1 h come from the layer's input projection.
//
// gla_recurrent walks the tokens one by one (any sizes, both dtypes; a decode step is T = 1).
#include "layered.h"
#include "epilogue_math.cuh"
#include "pdl.cuh"
#include <math.h>

namespace spt {

namespace {

constexpr int kRecTokens = 16;         // tokens staged in shared memory at a time
constexpr int kRecWarps = 8;

// log alpha = log(sigmoid(z)) / tau
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return (fminf(z, 0.0f) - log1pf(expf(-fabsf(z)))) * inv_tau; }

// A CTA owns 32 columns of one (sequence, head)'s state: lane = column, warp w the DPW rows w * DPW ...  Each warp sums its rows'
// share of o; the eight shares are added in warp order once per block of staged tokens.
template <typename T, int DPW>
__global__ void __launch_bounds__(kRecWarps * 32) gla_recurrent_kernel(const GlaArgs a, float* __restrict__ o) {
    extern __shared__ float sm[];
    const int D = a.D, V = a.V, R = a.R;
    float* qs = sm;                                   // [tokens][D]
    float* ks = qs + kRecTokens * D;
    float* al = ks + kRecTokens * D;
    float* vs = al + kRecTokens * D;                  // [tokens][32]
    float* part = vs + kRecTokens * 32;               // [warps][tokens][32]
    float* as = part + kRecWarps * kRecTokens * 32;   // [tokens][R]
    pdl_release();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int v0 = blockIdx.x * 32, b = blockIdx.y / a.H, h = blockIdx.y % a.H;
    const int col = v0 + lane;
    float* st = a.state ? a.state + (size_t)blockIdx.y * D * V : nullptr;
    float s[DPW];
    pdl_acquire();
#pragma unroll
    for (int i = 0; i < DPW; i++) {
        const int d = warp * DPW + i;
        s[i] = st && d < D && col < V ? st[(size_t)d * V + col] : 0.0f;
    }
    const T* in = static_cast<const T*>(a.in) + (size_t)b * a.T * a.ld;
    const float qsc = 1.0f / sqrtf((float)D), inv_tau = 1.0f / a.tau;
    for (int t0 = 0; t0 < a.T; t0 += kRecTokens) {
        const int n = min(kRecTokens, a.T - t0);
        for (int i = tid; i < n * R; i += blockDim.x) { const int t = i / R; as[i] = (float)in[(size_t)(t0 + t) * a.ld + a.c_a + (i - t * R)]; }
        for (int i = tid; i < n * 32; i += blockDim.x) {
            const int t = i >> 5, c = v0 + (i & 31);
            vs[i] = c < V ? (float)in[(size_t)(t0 + t) * a.ld + a.c_v + h * V + c] : 0.0f;
        }
        __syncthreads();
        for (int i = tid; i < n * D; i += blockDim.x) {
            const int t = i / D, d = i - t * D;
            const T* row = in + (size_t)(t0 + t) * a.ld;
            qs[i] = (float)row[a.c_q + h * D + d] * qsc;
            ks[i] = (float)row[a.c_k + h * D + d];
            const float* w = a.a2 + (size_t)(h * D + d) * R;
            float z = a.a2_b[h * D + d];
            for (int r = 0; r < R; r++) z = fmaf(as[t * R + r], __ldg(w + r), z);
            al[i] = expf(log_decay(z, inv_tau));
        }
        __syncthreads();
        for (int t = 0; t < n; t++) {
            const float v = vs[t * 32 + lane];
            const int base = t * D + warp * DPW;
            float acc = 0.0f;
#pragma unroll
            for (int i = 0; i < DPW; i++) {
                if (warp * DPW + i < D) {
                    s[i] = fmaf(s[i], al[base + i], ks[base + i] * v);
                    acc = fmaf(s[i], qs[base + i], acc);
                }
            }
            part[(warp * kRecTokens + t) * 32 + lane] = acc;
        }
        __syncthreads();
        for (int i = tid; i < n * 32; i += blockDim.x) {
            float sum = 0.0f;
#pragma unroll
            for (int w = 0; w < kRecWarps; w++) sum += part[w * kRecTokens * 32 + i];
            const int t = i >> 5, c = v0 + (i & 31);
            if (c < V) o[((size_t)b * a.T + t0 + t) * a.H * V + h * V + c] = sum;
        }
        // the next block's staging writes as / vs / qs only after every warp is past its token loop (the barrier above)
    }
    if (st) {
#pragma unroll
        for (int i = 0; i < DPW; i++) {
            const int d = warp * DPW + i;
            if (d < D && col < V) st[(size_t)d * V + col] = s[i];
        }
    }
}

// out = o / sqrt(mean(o^2) + eps) * w * silu(g): one warp per (token, head); the last head's warp zeroes the row's padding
template <typename T>
__global__ void __launch_bounds__(256) gla_norm_gate_kernel(const GlaArgs a, const float* __restrict__ o) {
    pdl_release();
    const int lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    pdl_acquire();
    if (item >= (long long)a.B * a.T * a.H) return;
    const long long row = item / a.H;
    const int h = (int)(item % a.H), V = a.V;
    const float* src = o + (size_t)row * a.H * V + h * V;
    float sq = 0.0f;
    for (int i = lane; i < V; i += 32) sq = fmaf(src[i], src[i], sq);
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, s);
    const float inv = 1.0f / sqrtf(sq / (float)V + a.eps);
    const T* g = static_cast<const T*>(a.in) + (size_t)row * a.ld + a.c_g + h * V;
    T* out = static_cast<T*>(a.out) + (size_t)row * a.ld_out;
    for (int i = lane; i < V; i += 32) out[h * V + i] = (T)(src[i] * inv * a.head_norm[i] * silu_exact((float)g[i]));
    if (h == a.H - 1) for (int i = a.H * V + lane; i < a.ld_out; i += 32) out[i] = (T)0.0f;
}

template <typename T, int DPW>
int launch_recurrent(const GlaArgs& a, float* o, bool dependent) {
    const size_t smem = (size_t)kRecTokens * (3 * a.D + 32 + kRecWarps * 32 + a.R) * sizeof(float);
    if (smem > 200 * 1024) return fail("gla: key size %d with a decay rank of %d does not fit shared memory", a.D, a.R);
    auto kern = gla_recurrent_kernel<T, DPW>;
    static size_t granted = 48 * 1024;
    if (smem > granted) { SPT_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); granted = smem; }
    SPT_CUDA(launch_dependent(kern, dim3(ceil_div(a.V, 32), a.B * a.H), dim3(kRecWarps * 32), smem, dependent, 1, a, o));
    note_submit();
    return 0;
}

template <typename T>
int recurrent_t(const GlaArgs& a, float* o, bool dependent) {
    const int per = ceil_div(a.D, kRecWarps);
    if (per <= 4) return launch_recurrent<T, 4>(a, o, dependent);
    if (per <= 8) return launch_recurrent<T, 8>(a, o, dependent);
    if (per <= 16) return launch_recurrent<T, 16>(a, o, dependent);
    if (per <= 32) return launch_recurrent<T, 32>(a, o, dependent);
    if (per <= 64) return launch_recurrent<T, 64>(a, o, dependent);
    return fail("gla: key size %d is larger than 512", a.D);
}

}  // namespace

int gla_norm_gate(const GlaArgs& a, const float* o, bool dependent) {
    const long long items = (long long)a.B * a.T * a.H;
    const dim3 grid((unsigned)((items + 7) / 8)), block(256);
    if (a.dtype == BF16) SPT_CUDA(launch_dependent(gla_norm_gate_kernel<__nv_bfloat16>, grid, block, 0, dependent, 1, a, o));
    else SPT_CUDA(launch_dependent(gla_norm_gate_kernel<float>, grid, block, 0, dependent, 1, a, o));
    note_submit();
    return 0;
}

int gla_recurrent(const GlaArgs& a, float* o_scratch, bool dependent) {
    if (a.B * a.H > 65535) return fail("gla: batch x heads exceeds one launch");
    if (a.dtype == BF16 ? recurrent_t<__nv_bfloat16>(a, o_scratch, dependent) : recurrent_t<float>(a, o_scratch, dependent)) return 1;
    return gla_norm_gate(a, o_scratch, dependent);
}

bool gla_chunked_supported(const GlaArgs&) { return false; }
size_t gla_chunked_state_bytes(const GlaArgs&) { return 0; }
size_t gla_chunked_decay_bytes(const GlaArgs&) { return 0; }
int gla_chunked(const GlaArgs&, float*, float*) { return fail("gla: no chunked kernel"); }

}  // namespace spt
