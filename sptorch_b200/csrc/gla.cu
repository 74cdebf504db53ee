// gla.cu -- gated linear attention: per head a [D, V] matrix S with a decay per key channel,
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   alpha = sigmoid(z)^(1/tau),  z = A2 (A1 h) + b,
// followed by an RMS norm of each head's o over V and the gate silu(W_g h).  q carries the factor D^(-1/2).  The recurrence, its
// decays and the norm are f32 whatever the model's dtype; q, k, v, the gate and A1 h come from the layer's input projection.
//
// gla_recurrent walks the tokens one by one (any sizes, both dtypes; one token per sequence has a kernel of
// its own); gla_chunked takes bf16 prompts in chunks.
#include "layered.h"
#include "epilogue_math.cuh"
#include "pdl.cuh"
#include <math.h>
#include <cooperative_groups.h>

namespace spt {

namespace {

constexpr int kRecTokens = 16;         // tokens staged in shared memory at a time
constexpr int kRecWarps = 8;

// log alpha = log(sigmoid(z)) / tau
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return (fminf(z, 0.0f) - log1pf(expf(-fabsf(z)))) * inv_tau; }

// A CTA owns 32 columns of one (sequence, head)'s state: lane = column, warp w the DPW rows w * DPW ...  Each warp sums its rows'
// share of o; the eight shares are added in warp order once per block of staged tokens.
// FUSED (at most kRecTokens tokens): the CTAs of a (sequence, head) are one cluster; they exchange their columns' sums of squares through
// distributed shared memory and write the normed, gated heads themselves instead of o.
template <typename T, int DPW, bool FUSED>
__global__ void __launch_bounds__(kRecWarps * 32) gla_recurrent_kernel(const GlaArgs a, float* __restrict__ o) {
    __shared__ float sq_sh[kRecTokens];
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
            if constexpr (FUSED) {                         // a warp holds the 32 columns of one token
                vs[i] = sum;                               // v of this element has been used up (the barrier above)
                float sq = sum * sum;                      // columns past V are zero
#pragma unroll
                for (int w = 16; w > 0; w >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, w);
                if (lane == 0) sq_sh[t] = sq;
            } else if (c < V) o[((size_t)b * a.T + t0 + t) * a.H * V + h * V + c] = sum;
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
    if constexpr (FUSED) {
        namespace cg = cooperative_groups;
        cg::cluster_group cluster = cg::this_cluster();
        const int parts = gridDim.x;
        if (parts > 1) cluster.sync(); else __syncthreads();
        T* out = static_cast<T*>(a.out) + (size_t)b * a.T * a.ld_out;
        for (int i = tid; i < a.T * 32; i += blockDim.x) {
            const int t = i >> 5, c = v0 + (i & 31);
            float sq = 0.0f;
            for (int r = 0; r < parts; r++) sq += parts > 1 ? cluster.map_shared_rank(sq_sh, r)[t] : sq_sh[t];
            const float inv = 1.0f / sqrtf(sq / (float)V + a.eps);
            if (c < V) out[(size_t)t * a.ld_out + h * V + c] = (T)(vs[i] * inv * a.head_norm[c] * silu_exact((float)in[(size_t)t * a.ld + a.c_g + h * V + c]));
            else if (h == a.H - 1 && h * V + c < a.ld_out) out[(size_t)t * a.ld_out + h * V + c] = (T)0.0f;
        }
        if (h == a.H - 1 && v0 + 32 >= V)              // padding of the output row that lies past this CTA's columns
            for (int i = tid; i < a.T * 8; i += blockDim.x) { const int c = h * V + v0 + 32 + (i & 7); if (c < a.ld_out) out[(size_t)(i >> 3) * a.ld_out + c] = (T)0.0f; }
        if (parts > 1) cluster.sync();                  // no CTA leaves while its sums may still be read
    }
}

// One token per sequence, V a multiple of four: a CTA owns a whole head.  Thread = (row group, four columns); its rows of the state are
// requested before the programmatic-launch wait (the step before wrote them), pass through registers once and go back; the row groups'
// shares of o meet in shared memory, where norm and gate finish the head.  HBM bytes: 8 D V per head.
template <typename T, int NR>
__global__ void __launch_bounds__(NR > 16 ? 512 : 256) gla_step_kernel(const GlaArgs a) {
    extern __shared__ float sm[];
    __shared__ float red[16];
    pdl_release();
    const int D = a.D, V = a.V, R = a.R, c4n = V / 4, rgs = blockDim.x / c4n;
    const int D4 = (D + 3) / 4 * 4;
    float* qs = sm;                                   // [D4]
    float* ks = qs + D4;
    float* al = ks + D4;
    float* as = al + D4;                              // [R]
    float* part = as + (R + 3) / 4 * 4;               // [row groups][V]
    const int tid = threadIdx.x, bh = blockIdx.x, b = bh / a.H, h = bh - b * a.H, rg = tid / c4n, c = (tid - rg * c4n) * 4;
    const bool mine = rg < rgs;
    float* st = a.state + (size_t)bh * D * V + c;
    float4 s[NR];
#pragma unroll
    for (int i = 0; i < NR; i++) { const int d = rg + i * rgs; if (mine && d < D) s[i] = *reinterpret_cast<const float4*>(st + (size_t)d * V); }
    pdl_acquire();
    const T* in = static_cast<const T*>(a.in) + (size_t)b * a.ld;
    const float qsc = 1.0f / sqrtf((float)D), inv_tau = 1.0f / a.tau;
    for (int r = tid; r < R; r += blockDim.x) as[r] = (float)in[a.c_a + r];
    for (int d = tid; d < D; d += blockDim.x) { qs[d] = (float)in[a.c_q + h * D + d] * qsc; ks[d] = (float)in[a.c_k + h * D + d]; }
    float v[4] = {0, 0, 0, 0};
    if (mine) {
#pragma unroll
        for (int j = 0; j < 4; j++) v[j] = (float)in[a.c_v + h * V + c + j];
    }
    __syncthreads();
    for (int d = tid; d < D; d += blockDim.x) {
        const float* w = a.a2 + (size_t)(h * D + d) * R;
        float z = a.a2_b[h * D + d];
#pragma unroll 8
        for (int r = 0; r < R; r++) z = fmaf(as[r], __ldg(w + r), z);
        al[d] = expf(log_decay(z, inv_tau));
    }
    __syncthreads();
    float4 acc = make_float4(0, 0, 0, 0);
#pragma unroll
    for (int i = 0; i < NR; i++) {
        const int d = rg + i * rgs;
        if (mine && d < D) {
            const float f = al[d], k = ks[d], q = qs[d];
            s[i].x = fmaf(s[i].x, f, k * v[0]); s[i].y = fmaf(s[i].y, f, k * v[1]); s[i].z = fmaf(s[i].z, f, k * v[2]); s[i].w = fmaf(s[i].w, f, k * v[3]);
            *reinterpret_cast<float4*>(st + (size_t)d * V) = s[i];
            acc.x = fmaf(s[i].x, q, acc.x); acc.y = fmaf(s[i].y, q, acc.y); acc.z = fmaf(s[i].z, q, acc.z); acc.w = fmaf(s[i].w, q, acc.w);
        }
    }
    if (mine) *reinterpret_cast<float4*>(part + rg * V + c) = acc;
    __syncthreads();
    float sq = 0.0f;
    for (int i = tid; i < V; i += blockDim.x) {
        float o = 0.0f;
        for (int r = 0; r < rgs; r++) o += part[r * V + i];
        part[i] = o;                                  // only this thread reads column i
        sq = fmaf(o, o, sq);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if ((tid & 31) == 0) red[tid >> 5] = sq;
    __syncthreads();
    float tot = 0.0f;
    for (int w = 0; w < (int)blockDim.x / 32; w++) tot += red[w];
    const float inv = 1.0f / sqrtf(tot / (float)V + a.eps);
    T* out = static_cast<T*>(a.out) + (size_t)b * a.ld_out;
    for (int i = tid; i < V; i += blockDim.x) out[h * V + i] = (T)(part[i] * inv * a.head_norm[i] * silu_exact((float)in[a.c_g + h * V + i]));
    if (h == a.H - 1) for (int i = a.H * V + tid; i < a.ld_out; i += blockDim.x) out[i] = (T)0.0f;
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

// ---------------- prompts: chunks of kChunk tokens on the tensor cores ----------------
// With b_t the running sum of log2 alpha inside a chunk (b_t <= 0, per key channel) and S the state before the chunk:
//   o_t = (q_t 2^(b_t))^T S + sum_(s <= t) A[t][s] v_s,    A[t][s] = sum_d q_t[d] k_s[d] 2^(b_t[d] - b_s[d])
//   S'  = diag(2^(b_C)) S + sum_s (k_s 2^(b_C - b_s)) v_s^T
// Chunks are independent except through S, so three launches do a prompt: the chunks' own sums U = sum_s (k_s 2^(b_C - b_s)) v_s^T
// (gla_chunk_state_kernel), a scan over the chunks that turns U into the state before each (gla_scan_kernel), and the outputs with head
// norm and gate (gla_chunk_out_kernel).  (This is the chunkwise form of "Gated Linear Attention Transformers with Hardware-Efficient
// Training", Yang, Wang, Shen, Panda, Kim.)  Every exponent that is evaluated is <= 0: A is taken as a binary tree of blocks -- rows
// 32..63 against columns 0..31, then the two such halves of each 32, then of each 16 -- each relative to the last token r before its rows
// (2^(b_t - b_r) 2^(b_r - b_s)), and pair by pair inside the 8 x 8 blocks on the diagonal, so a strong decay underflows where the product is
// nothing and never overflows.
// Products run as mma.sync on TF32 with each f32 operand split into two TF32 parts (hi hi + hi lo + lo hi: 21 mantissa bits); v comes
// in bf16 and needs no split.  The tiles are 64 rows and the operands are scaled element by element on their way into the fragments,
// so there is no operand for tcgen05 to fetch from shared memory as it lies there; the kernels are bound by that work and by HBM.
constexpr int kChunk = 64;
constexpr int kChunkThreads = 512;    // sixteen warps: the phases are chains of dependent work, two such CTAs an SM keep it busy

__device__ __forceinline__ float exp2_fast(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// x = hi + lo: hi keeps the ten upper mantissa bits; the tensor core reads the upper ten of lo's
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi));
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct ChunkArgs { GlaArgs a; float *u, *dec; int nc; };

// rows of bf16 -> f32 tile [kChunk][PITCH], zero outside n rows and w columns (up to WP columns).  Eight columns at a time where aligned:
// request() starts the loads (all tiles of a kernel before the first is stored), store() widens them into shared memory.
template <int PITCH, int WP>
struct TileLoad {
    static constexpr int PER = WP / 8, TURNS = (kChunk * PER + kChunkThreads - 1) / kChunkThreads;
    uint4 raw[TURNS];
    __device__ __forceinline__ void request(const __nv_bfloat16* src, long long ld, int n, int w, bool vec) {
#pragma unroll
        for (int i0 = 0; i0 < TURNS; i0++) {
            const int i = i0 * kChunkThreads + (int)threadIdx.x, t = i / PER, c = (i % PER) * 8;
            raw[i0] = make_uint4(0, 0, 0, 0);
            if (vec && t < n && c < w) raw[i0] = __ldg(reinterpret_cast<const uint4*>(src + (size_t)t * ld + c));
        }
    }
    __device__ __forceinline__ void store(float* dst, const __nv_bfloat16* src, long long ld, int n, int w, float f, bool vec) const {
        if (vec) {
#pragma unroll
            for (int i0 = 0; i0 < TURNS; i0++) {
                const int i = i0 * kChunkThreads + (int)threadIdx.x, t = i / PER, c = (i % PER) * 8;
                if (kChunk * PER % kChunkThreads == 0 || i < kChunk * PER) {
                    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw[i0]);
#pragma unroll
                    for (int j = 0; j < 4; j += 2) {
                        const float2 x = bf16x2_to_float2(h[j]), y = bf16x2_to_float2(h[j + 1]);
                        *reinterpret_cast<float4*>(dst + t * PITCH + c + 2 * j) = make_float4(x.x * f, x.y * f, y.x * f, y.y * f);
                    }
                }
            }
        } else {
            for (int i = threadIdx.x; i < kChunk * WP; i += kChunkThreads) {
                const int t = i / WP, c = i % WP;
                dst[t * PITCH + c] = t < n && c < w ? (float)src[(size_t)t * ld + c] * f : 0.0f;
            }
        }
    }
};

// log2 of the decay: 1 + e with e = exp(-|z|) loses e's low bits, so a small e takes the series of log(1 + e) (next term e^5 / 5)
__device__ __forceinline__ float log2_decay(float z, float inv_tau) {
    const float e = exp2_fast(-1.4426950408889634f * fabsf(z));
    float lg;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(lg) : "f"(1.0f + e));
    const float series = e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 0.33333334f), -0.5f), 1.0f) * 1.4426950408889634f;
    return (fminf(z, 0.0f) * 1.4426950408889634f - (e < 0.03f ? series : lg)) * inv_tau;
}

// DP / VP: dim and vdim rounded up to the sizes the kernels are built for; padding columns are zeros
template <int DP, int VP>
struct ChunkSmem {
    static constexpr int LDK = DP + 8, LDQ = DP + 4, LDV = VP + 8, LDA = 68;      // = 8 / 4 / 8 / 4 (mod 32)
    static constexpr int kStateFloats = kChunk * (2 * LDK + LDV) + 4 * DP;        // + R (kChunk + DP) for the decay projection
    static constexpr int kOutFloats = kChunk * (3 * LDQ + LDV + LDA) + 4 * kChunk;
};

template <int DP, int VP>
__global__ void __launch_bounds__(kChunkThreads) gla_chunk_state_kernel(const ChunkArgs p) {
    extern __shared__ __align__(16) float sm[];
    using L = ChunkSmem<DP, VP>;
    constexpr int LDK = L::LDK, LDV = L::LDV;
    const GlaArgs& a = p.a;
    const int D = a.D, V = a.V, R = a.R;
    float* bs = sm;                               // [kChunk][LDK]: log2 decays, then their running sums
    float* ks = bs + kChunk * LDK;                // [kChunk][LDK]
    float* vs = ks + kChunk * LDK;                // [kChunk][LDV]
    float* seg = vs + kChunk * LDV;               // [4][DP]
    float* a1s = seg + 4 * DP;                    // [R][kChunk]
    float* a2s = a1s + R * kChunk;                // [R][DP]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
    const int chunk = blockIdx.x, bh = blockIdx.y, b = bh / a.H, h = bh - b * a.H;
    const int t0 = chunk * kChunk, n = min(kChunk, a.T - t0);
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + ((size_t)b * a.T + t0) * a.ld;
    const bool vec = D % 8 == 0 && V % 8 == 0;
    TileLoad<LDK, DP> tk;
    TileLoad<LDV, VP> tv;
    tk.request(in + a.c_k + h * D, a.ld, n, D, vec);
    tv.request(in + a.c_v + h * V, a.ld, n, V, vec);
    for (int i = tid; i < kChunk * R; i += kChunkThreads) { const int t = i % kChunk, r = i / kChunk; a1s[i] = t < n ? (float)in[(size_t)t * a.ld + a.c_a + r] : 0.0f; }
    for (int i = tid; i < DP * R; i += kChunkThreads) { const int d = i % DP, r = i / DP; a2s[i] = d < D ? __ldg(a.a2 + (size_t)(h * D + d) * R + r) : 0.0f; }
    tk.store(ks, in + a.c_k + h * D, a.ld, n, D, 1.0f, vec);
    tv.store(vs, in + a.c_v + h * V, a.ld, n, V, 1.0f, vec);
    __syncthreads();
    // log2 alpha of four tokens per turn of a thread; padding tokens and channels decay by nothing
    const float inv_tau = 1.0f / a.tau;
#pragma unroll 1
    for (int i = tid; i < kChunk / 4 * DP; i += kChunkThreads) {
        const int d = i % DP, t = i / DP * 4;
        const float bias = d < D ? a.a2_b[h * D + d] : 0.0f;
        float z[4] = {bias, bias, bias, bias};
#pragma unroll 4
        for (int r = 0; r < R; r++) {
            const float w = a2s[r * DP + d];
            const float4 x = *reinterpret_cast<const float4*>(a1s + r * kChunk + t);
            z[0] = fmaf(x.x, w, z[0]); z[1] = fmaf(x.y, w, z[1]); z[2] = fmaf(x.z, w, z[2]); z[3] = fmaf(x.w, w, z[3]);
        }
#pragma unroll
        for (int j = 0; j < 4; j++) bs[(t + j) * LDK + d] = d < D && t + j < n ? log2_decay(z[j], inv_tau) : 0.0f;
    }
    __syncthreads();
    // running sums: four segments of 16 tokens side by side, then the segments' totals on top
    for (int i = tid; i < 4 * DP; i += kChunkThreads) {
        const int d = i % DP, s = i / DP;
        float sum = 0.0f;
#pragma unroll
        for (int t = 0; t < 16; t++) { float& x = bs[(s * 16 + t) * LDK + d]; sum += x; x = sum; }
        seg[i] = sum;
    }
    __syncthreads();
    {
        float* dec = p.dec + ((size_t)bh * p.nc + chunk) * kChunk * D;
        constexpr int STEP = kChunkThreads / DP;                       // tokens per turn (4, 8 or 16); a thread keeps its channel
        const int d = tid % DP;
        float off[5];
        off[0] = 0.0f;
#pragma unroll
        for (int j = 0; j < 4; j++) off[j + 1] = off[j] + seg[j * DP + d];
#pragma unroll
        for (int t1 = 0; t1 < kChunk; t1 += STEP) {
            const int t = t1 + tid / DP;
            const float bt = bs[t * LDK + d] + off[t1 >> 4];           // STEP divides 16: the segment does not depend on the thread
            if (d < D) dec[(size_t)t * D + d] = bt;
            ks[t * LDK + d] *= exp2_fast(fminf(off[4] - bt, 0.0f));
        }
    }
    __syncthreads();
    // U[d][v] = sum_t ks[t][d] vs[t][v]: blocks of 16 channels x 32 values dealt over the warps
    float* u = p.u + ((size_t)bh * p.nc + chunk) * D * V;
    constexpr int MB = DP / 16, NB = VP / 32;
    for (int blk = warp; blk < MB * NB; blk += kChunkThreads / 32) {
        const int m0 = blk % MB * 16, n0 = blk / MB * 32;
        if (m0 >= D || n0 >= V) continue;
        float acc[4][4] = {};
        const float *kp = ks + q4 * LDK + m0 + g, *vp = vs + q4 * LDV + n0 + g;
#pragma unroll 2
        for (int k = 0; k < kChunk; k += 8, kp += 8 * LDK, vp += 8 * LDV) {
            uint32_t hi[4], lo[4];
            split_tf32(kp[0], hi[0], lo[0]);
            split_tf32(kp[8], hi[1], lo[1]);
            split_tf32(kp[4 * LDK], hi[2], lo[2]);
            split_tf32(kp[4 * LDK + 8], hi[3], lo[3]);
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const uint32_t b0 = __float_as_uint(vp[8 * j]), b1 = __float_as_uint(vp[4 * LDV + 8 * j]);
                mma_tf32(acc[j], lo, b0, b1);
                mma_tf32(acc[j], hi, b0, b1);
            }
        }
        const bool even = V % 2 == 0;
#pragma unroll
        for (int j = 0; j < 4; j++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int d = m0 + g + e * 8, v = n0 + 8 * j + 2 * q4;
                if (d < D && v < V) {
                    if (even) *reinterpret_cast<float2*>(u + (size_t)d * V + v) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
                    else { u[(size_t)d * V + v] = acc[j][2 * e]; if (v + 1 < V) u[(size_t)d * V + v + 1] = acc[j][2 * e + 1]; }
                }
            }
    }
}

// u[c] <- the state before chunk c; state <- the state behind the last one.  A thread owns W neighbouring values (W = 4 where V is a
// multiple of four), eight chunks in flight.
template <int W>
__global__ void __launch_bounds__(256) gla_scan_kernel(const ChunkArgs p) {
    struct alignas(4 * W) Vec { float v[W]; };
    const GlaArgs& a = p.a;
    const int DV = a.D * a.V;
    const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * W;
    if (i >= (long long)a.B * a.H * DV) return;
    const int bh = (int)(i / DV), e = (int)(i - (long long)bh * DV), d = e / a.V;
    float* u = p.u + (size_t)bh * p.nc * DV + e;
    const float* last = p.dec + ((size_t)bh * p.nc * kChunk + kChunk - 1) * a.D + d;
    Vec s;
#pragma unroll
    for (int w = 0; w < W; w++) s.v[w] = 0.0f;
    if (a.state) s = *reinterpret_cast<const Vec*>(a.state + i);
    for (int c0 = 0; c0 < p.nc; c0 += 8) {
        Vec x[8];
        float f[8];
#pragma unroll
        for (int j = 0; j < 8; j++)
            if (c0 + j < p.nc) { x[j] = *reinterpret_cast<const Vec*>(u + (size_t)(c0 + j) * DV); f[j] = last[(size_t)(c0 + j) * kChunk * a.D]; }
#pragma unroll
        for (int j = 0; j < 8; j++)
            if (c0 + j < p.nc) {
                *reinterpret_cast<Vec*>(u + (size_t)(c0 + j) * DV) = s;
                const float g = exp2_fast(f[j]);
#pragma unroll
                for (int w = 0; w < W; w++) s.v[w] = fmaf(s.v[w], g, x[j].v[w]);
            }
    }
    if (a.state) *reinterpret_cast<Vec*>(a.state + i) = s;
}

// One block of A: rows r0 .. r0 + 15 (ROWS8: only the lower eight of the fragment, rows r0 .. r0 + 7), columns c0 .. c0 + 8 NTILES - 1, all
// before row `ref + 1`; exponents relative to token ref.
template <int DP, int NTILES, bool ROWS8>
__device__ __forceinline__ void a_block(const float* qs, const float* ks, const float* bs, float* as, int r0, int c0, int ref, int g, int q4) {
    constexpr int LD = DP + 4, LDA = 68;
    float acc[NTILES][4] = {};
    const float *qp = qs + (r0 + g) * LD + q4, *bq = bs + (r0 + g) * LD + q4, *br = bs + ref * LD + q4, *kp = ks + (c0 + g) * LD + q4, *bk = bs + (c0 + g) * LD + q4;
#pragma unroll 2
    for (int k = 0; k < DP; k += 8) {
        const float f0 = br[k], f1 = br[k + 4];
        uint32_t ah[4] = {0, 0, 0, 0}, al[4] = {0, 0, 0, 0};
        split_tf32(qp[k] * exp2_fast(bq[k] - f0), ah[0], al[0]);
        split_tf32(qp[k + 4] * exp2_fast(bq[k + 4] - f1), ah[2], al[2]);
        if (!ROWS8) {
            split_tf32(qp[8 * LD + k] * exp2_fast(bq[8 * LD + k] - f0), ah[1], al[1]);
            split_tf32(qp[8 * LD + k + 4] * exp2_fast(bq[8 * LD + k + 4] - f1), ah[3], al[3]);
        }
#pragma unroll
        for (int j = 0; j < NTILES; j++) {
            uint32_t h0, l0, h1, l1;
            split_tf32(kp[8 * j * LD + k] * exp2_fast(f0 - bk[8 * j * LD + k]), h0, l0);
            split_tf32(kp[8 * j * LD + k + 4] * exp2_fast(f1 - bk[8 * j * LD + k + 4]), h1, l1);
            mma_tf32(acc[j], al, h0, h1);
            mma_tf32(acc[j], ah, l0, l1);
            mma_tf32(acc[j], ah, h0, h1);
        }
    }
#pragma unroll
    for (int j = 0; j < NTILES; j++) {
        float* o = as + (r0 + g) * LDA + c0 + 8 * j + 2 * q4;
        o[0] = acc[j][0]; o[1] = acc[j][1];
        if (!ROWS8) { o[8 * LDA] = acc[j][2]; o[8 * LDA + 1] = acc[j][3]; }
    }
}

// Warps are 4 (16 rows each) x 4 (quarters of the values), NT 8-column tiles each.
template <int DP, int VP>
__global__ void __launch_bounds__(kChunkThreads, ChunkSmem<DP, VP>::kOutFloats * 4 <= 113 * 1024 ? 2 : 1) gla_chunk_out_kernel(const ChunkArgs p) {
    extern __shared__ __align__(16) float sm[];
    using L = ChunkSmem<DP, VP>;
    constexpr int LD = L::LDQ, LDV = L::LDV, LDA = L::LDA, NT = VP / 32;
    const GlaArgs& a = p.a;
    const int D = a.D, V = a.V;
    float* bs = sm;                               // [kChunk][LD]: running sums of the log2 decays
    float* ks = bs + kChunk * LD;                 // [kChunk][LD]
    float* qs = ks + kChunk * LD;                 // [kChunk][LD]: q D^(-1/2), later times 2^b
    // SS: the state's tile fits the values' place.  S is then copied there while A is computed, and v -- kept in registers meanwhile --
    // goes where b and k lay.  Otherwise S comes straight from global memory into the fragments.  Either way the place next to A holds
    // the normed output at the end.
    constexpr bool SS = DP <= kChunk && LDV <= 2 * LD;
    float* xs = qs + kChunk * LD;                 // [kChunk][LDV]: S or v, then the output
    float* vs = SS ? sm : xs;
    float* as = xs + kChunk * LDV;                // [kChunk][LDA]: A
    float* red = as + kChunk * LDA;               // [4][kChunk]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
    const int chunk = blockIdx.x, bh = blockIdx.y, b = bh / a.H, h = bh - b * a.H;
    const int t0 = chunk * kChunk, n = min(kChunk, a.T - t0);
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + ((size_t)b * a.T + t0) * a.ld;
    const bool vec = D % 8 == 0 && V % 8 == 0;
    const float* dec = p.dec + ((size_t)bh * p.nc + chunk) * kChunk * D;
    const bool carried = chunk > 0 || a.state;
    const float* u = p.u + ((size_t)bh * p.nc + chunk) * D * V;
    TileLoad<LDV, VP> tv;
    {
        constexpr int TURNS = kChunk * DP / 4 / kChunkThreads;
        TileLoad<LD, DP> tq, tk;
        float4 bd[TURNS];
#pragma unroll
        for (int i0 = 0; i0 < TURNS; i0++) {
            const int i = i0 * kChunkThreads + tid, t = i / (DP / 4), d = i % (DP / 4) * 4;      // DP >= 32: the turns are full
            bd[i0] = D % 4 == 0 && d < D ? __ldg(reinterpret_cast<const float4*>(dec + (size_t)t * D + d)) : make_float4(0, 0, 0, 0);
        }
        tq.request(in + a.c_q + h * D, a.ld, n, D, vec);
        tk.request(in + a.c_k + h * D, a.ld, n, D, vec);
        tv.request(in + a.c_v + h * V, a.ld, n, V, vec);
#pragma unroll
        for (int i0 = 0; i0 < TURNS; i0++) {
            const int i = i0 * kChunkThreads + tid;
            if (D % 4 == 0) *reinterpret_cast<float4*>(bs + i / (DP / 4) * LD + i % (DP / 4) * 4) = bd[i0];
        }
        if (D % 4) for (int i = tid; i < kChunk * DP; i += kChunkThreads) { const int t = i / DP, d = i % DP; bs[t * LD + d] = d < D ? dec[(size_t)t * D + d] : 0.0f; }
        tq.store(qs, in + a.c_q + h * D, a.ld, n, D, 1.0f / sqrtf((float)D), vec);
        tk.store(ks, in + a.c_k + h * D, a.ld, n, D, 1.0f, vec);
        if (!SS) tv.store(vs, in + a.c_v + h * V, a.ld, n, V, 1.0f, vec);
        if (SS && carried) {
            if (V % 4 == 0) {
                for (int i = tid; i < DP * (VP / 4); i += kChunkThreads) {
                    const int d = i / (VP / 4), v = i % (VP / 4) * 4;
                    float* dst = xs + d * LDV + v;
                    if (d < D && v < V) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(u + (size_t)d * V + v) : "memory");
                    else *reinterpret_cast<float4*>(dst) = make_float4(0, 0, 0, 0);
                }
                asm volatile("cp.async.commit_group;" ::: "memory");
            } else
                for (int i = tid; i < DP * VP; i += kChunkThreads) { const int d = i / VP, v = i % VP; xs[d * LDV + v] = d < D && v < V ? u[(size_t)d * V + v] : 0.0f; }
        }
    }
    for (int i = tid; i < kChunk * LDA / 4; i += kChunkThreads) reinterpret_cast<float4*>(as)[i] = make_float4(0, 0, 0, 0);
    __syncthreads();

    // A: four tasks of the 32-row block and two of the 16-row blocks (16 rows x 16 columns each), four 8 x 8 blocks, and the 288 pairs of
    // the diagonal blocks in nine turns of a warp
    int pair_turn = 0, pair_last = 0;             // this warp's turns
    if (warp < 4) a_block<DP, 2, false>(qs, ks, bs, as, 32 + 16 * (warp >> 1), 16 * (warp & 1), 31, g, q4);
    else if (warp < 6) a_block<DP, 2, false>(qs, ks, bs, as, warp == 4 ? 16 : 48, warp == 4 ? 0 : 32, warp == 4 ? 15 : 47, g, q4);
    else if (warp < 10) a_block<DP, 1, true>(qs, ks, bs, as, 16 * (warp - 6) + 8, 16 * (warp - 6), 16 * (warp - 6) + 7, g, q4);
    else { const int w = warp - 10; pair_turn = w < 3 ? 2 * w : w + 3; pair_last = w < 3 ? pair_turn + 2 : pair_turn + 1; }
#pragma unroll 1
    for (; pair_turn < pair_last; pair_turn++) {
        // turn i covers pairs 32 i ..: pair e of the eight diagonal blocks' 8 * 36, row-major inside a block's triangle
        const int e = pair_turn * 32 + lane, blk = e / 36, f = e - blk * 36;
        const int t = f < 1 ? 0 : f < 3 ? 1 : f < 6 ? 2 : f < 10 ? 3 : f < 15 ? 4 : f < 21 ? 5 : f < 28 ? 6 : 7, s = f - t * (t + 1) / 2;
        const int rt = (blk * 8 + t) * LD, rs = (blk * 8 + s) * LD;
        float acc = 0.0f;
#pragma unroll 4
        for (int d = 0; d < DP; d += 4) {
            const float4 x = *reinterpret_cast<const float4*>(qs + rt + d), y = *reinterpret_cast<const float4*>(ks + rs + d);
            const float4 u = *reinterpret_cast<const float4*>(bs + rt + d), w = *reinterpret_cast<const float4*>(bs + rs + d);
            acc = fmaf(x.x * y.x, exp2_fast(u.x - w.x), acc); acc = fmaf(x.y * y.y, exp2_fast(u.y - w.y), acc);
            acc = fmaf(x.z * y.z, exp2_fast(u.z - w.z), acc); acc = fmaf(x.w * y.w, exp2_fast(u.w - w.w), acc);
        }
        as[(blk * 8 + t) * LDA + blk * 8 + s] = acc;
    }
    const int wm = warp >> 2, wn = warp & 3, first = wn * NT;
    float acc[NT][4] = {};
    float cur[NT][2], nxt[NT][2];
    auto fetch = [&](int k, float (&x)[NT][2]) {
#pragma unroll
        for (int j = 0; j < NT; j++) {
            const int v = (first + j) * 8 + g;
#pragma unroll
            for (int e = 0; e < 2; e++) { const int d = k + q4 + 4 * e; x[j][e] = v < V && d < D ? __ldg(u + (size_t)d * V + v) : 0.0f; }
        }
    };
    if (!SS && carried) { fetch(0, cur); fetch(8, nxt); }
    __syncthreads();
#pragma unroll
    for (int i0 = 0; i0 < kChunk * DP / 4; i0 += kChunkThreads) {
        const int i = i0 + tid, o = i / (DP / 4) * LD + i % (DP / 4) * 4;
        float4 x = *reinterpret_cast<const float4*>(qs + o);
        const float4 e = *reinterpret_cast<const float4*>(bs + o);
        x.x *= exp2_fast(e.x); x.y *= exp2_fast(e.y); x.z *= exp2_fast(e.z); x.w *= exp2_fast(e.w);
        *reinterpret_cast<float4*>(qs + o) = x;
    }
    if (SS) asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (SS) tv.store(vs, in + a.c_v + h * V, a.ld, n, V, 1.0f, vec);          // over b and k, which are done; read behind the next barrier
    if (carried) {
        // (q 2^b) S
        const float* qp = qs + (wm * 16 + g) * LD + q4;
#pragma unroll 2
        for (int k = 0; k < DP; k += 8) {
            float far[NT][2];                              // S two steps ahead
            if (!SS && k + 16 < DP) fetch(k + 16, far);
            if (SS) {
                const float* sp = xs + (k + q4) * LDV + first * 8 + g;
#pragma unroll
                for (int j = 0; j < NT; j++) { cur[j][0] = sp[8 * j]; cur[j][1] = sp[4 * LDV + 8 * j]; }
            }
            uint32_t ah[4], al[4];
#pragma unroll
            for (int e = 0; e < 4; e++) split_tf32(qp[(e & 1) * 8 * LD + k + (e >> 1) * 4], ah[e], al[e]);
#pragma unroll
            for (int j = 0; j < NT; j++) {
                uint32_t h0, l0, h1, l1;
                split_tf32(cur[j][0], h0, l0); split_tf32(cur[j][1], h1, l1);
                mma_tf32(acc[j], al, h0, h1); mma_tf32(acc[j], ah, l0, l1); mma_tf32(acc[j], ah, h0, h1);
            }
            if (!SS && k + 8 < DP) {
#pragma unroll
                for (int j = 0; j < NT; j++) { cur[j][0] = nxt[j][0]; cur[j][1] = nxt[j][1]; nxt[j][0] = far[j][0]; nxt[j][1] = far[j][1]; }
            }
        }
    }
    if (SS) __syncthreads();
    // A v up to the diagonal
    {
        const float *ap = as + (wm * 16 + g) * LDA + q4, *vp = vs + q4 * LDV + first * 8 + g;
#pragma unroll 2
        for (int k = 0; k < wm * 16 + 16; k += 8) {
            uint32_t ah[4], al[4];
#pragma unroll
            for (int e = 0; e < 4; e++) split_tf32(ap[(e & 1) * 8 * LDA + k + (e >> 1) * 4], ah[e], al[e]);
#pragma unroll
            for (int j = 0; j < NT; j++) {
                const uint32_t b0 = __float_as_uint(vp[k * LDV + 8 * j]), b1 = __float_as_uint(vp[(k + 4) * LDV + 8 * j]);
                mma_tf32(acc[j], al, b0, b1); mma_tf32(acc[j], ah, b0, b1);
            }
        }
    }
    // head norm over V and gate; a row's values lie with four warps
#pragma unroll
    for (int r = 0; r < 2; r++) {
        float sq = 0.0f;
#pragma unroll
        for (int j = 0; j < NT; j++) { sq = fmaf(acc[j][2 * r], acc[j][2 * r], sq); sq = fmaf(acc[j][2 * r + 1], acc[j][2 * r + 1], sq); }
        sq += __shfl_xor_sync(0xffffffffu, sq, 1);
        sq += __shfl_xor_sync(0xffffffffu, sq, 2);
        if (q4 == 0) red[wn * kChunk + wm * 16 + r * 8 + g] = sq;
    }
    __syncthreads();
    // normed rows through shared memory, so that gate and output are read and written sixteen bytes at a time
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int t = wm * 16 + r * 8 + g;
        const float inv = 1.0f / sqrtf((red[t] + red[kChunk + t] + red[2 * kChunk + t] + red[3 * kChunk + t]) / (float)V + a.eps);
#pragma unroll
        for (int j = 0; j < NT; j++)
            *reinterpret_cast<float2*>(xs + t * LDV + (first + j) * 8 + 2 * q4) = make_float2(acc[j][2 * r] * inv, acc[j][2 * r + 1] * inv);
    }
    __syncthreads();
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + ((size_t)b * a.T + t0) * a.ld_out + h * V;
    const __nv_bfloat16* gate = in + a.c_g + h * V;
    if (vec) {
        constexpr int PER = VP / 8;
#pragma unroll 2
        for (int i = tid; i < kChunk * PER; i += kChunkThreads) {
            const int t = i / PER, c = i % PER * 8;
            if (t >= n || c >= V) continue;
            const uint4 gr = __ldg(reinterpret_cast<const uint4*>(gate + (size_t)t * a.ld + c));
            const __nv_bfloat162* gh = reinterpret_cast<const __nv_bfloat162*>(&gr);
            const float* xr = xs + t * LDV + c;
            uint4 o4;
            __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o4);
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const float2 gg = bf16x2_to_float2(gh[j]), x = *reinterpret_cast<const float2*>(xr + 2 * j), w = __ldg(reinterpret_cast<const float2*>(a.head_norm + c + 2 * j));
                oh[j] = __floats2bfloat162_rn(x.x * w.x * silu_fast(gg.x), x.y * w.y * silu_fast(gg.y));
            }
            *reinterpret_cast<uint4*>(out + (size_t)t * a.ld_out + c) = o4;
        }
    } else
        for (int i = tid; i < n * V; i += kChunkThreads) {
            const int t = i / V, c = i - t * V;
            out[(size_t)t * a.ld_out + c] = __float2bfloat16_rn(xs[t * LDV + c] * a.head_norm[c] * silu_fast((float)gate[(size_t)t * a.ld + c]));
        }
    if (h == a.H - 1)                             // the padding of the output rows
        for (int i = tid; i < n * 8; i += kChunkThreads) { const int c = V + (i & 7); if (h * V + c < a.ld_out) out[(size_t)(i >> 3) * a.ld_out + c] = __float2bfloat16_rn(0.0f); }
}

template <int DP, int VP>
int launch_chunked(const ChunkArgs& p) {
    using L = ChunkSmem<DP, VP>;
    static size_t granted = 0;
    const size_t s1 = (L::kStateFloats + (size_t)p.a.R * (kChunk + DP)) * sizeof(float), s2 = L::kOutFloats * sizeof(float);
    if (s1 > granted) {
        SPT_CUDA(cudaFuncSetAttribute(gla_chunk_state_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1));
        SPT_CUDA(cudaFuncSetAttribute(gla_chunk_out_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2));
        granted = s1;
    }
    const dim3 grid(p.nc, p.a.B * p.a.H);
    gla_chunk_state_kernel<DP, VP><<<grid, kChunkThreads, s1, rt().stream>>>(p);
    SPT_LAUNCH_CHECK("gla_chunk_state");
    const long long elems = (long long)p.a.B * p.a.H * p.a.D * p.a.V;
    if (p.a.V % 4 == 0) gla_scan_kernel<4><<<(unsigned)((elems / 4 + 255) / 256), 256, 0, rt().stream>>>(p);
    else gla_scan_kernel<1><<<(unsigned)((elems + 255) / 256), 256, 0, rt().stream>>>(p);
    SPT_LAUNCH_CHECK("gla_scan");
    gla_chunk_out_kernel<DP, VP><<<grid, kChunkThreads, s2, rt().stream>>>(p);
    SPT_LAUNCH_CHECK("gla_chunk_out");
    return 0;
}
template <int DP>
int launch_chunked_v(const ChunkArgs& p) {
    return p.a.V <= 64 ? launch_chunked<DP, 64>(p) : p.a.V <= 128 ? launch_chunked<DP, 128>(p) : launch_chunked<DP, 256>(p);
}

// few tokens and at most eight CTAs (a portable cluster) per head: norm and gate in the same launch
// ... while the launch is short: with many CTAs the clusters hold their SMs longer than the second launch costs (64 sequences x 16 heads of
// 64 x 128: 57 us fused, 37 us in two launches; 8 sequences: 13 and 14)
bool recurrent_fuses(const GlaArgs& a) { return a.T <= kRecTokens && a.V <= 256 && (long long)a.B * a.H * ceil_div(a.V, 32) <= 8ll * rt().sm_count; }

template <typename T, int DPW>
int launch_recurrent(const GlaArgs& a, float* o, bool dependent) {
    const size_t smem = (size_t)kRecTokens * (3 * a.D + 32 + kRecWarps * 32 + a.R) * sizeof(float);
    if (smem > 200 * 1024) return fail("gla: key size %d with a decay rank of %d does not fit shared memory", a.D, a.R);
    const bool fused = recurrent_fuses(a);
    auto kern = fused ? gla_recurrent_kernel<T, DPW, true> : gla_recurrent_kernel<T, DPW, false>;
    static size_t granted = 48 * 1024;
    if (smem > granted) {
        SPT_CUDA(cudaFuncSetAttribute(gla_recurrent_kernel<T, DPW, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        SPT_CUDA(cudaFuncSetAttribute(gla_recurrent_kernel<T, DPW, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        granted = smem;
    }
    SPT_CUDA(launch_dependent(kern, dim3(ceil_div(a.V, 32), a.B * a.H), dim3(kRecWarps * 32), smem, dependent, fused ? ceil_div(a.V, 32) : 1, a, o));
    note_submit();
    return 0;
}

// rows of the state per thread of the one-token kernel with `threads` threads; 0: it does not take this layer
int step_rows(const GlaArgs& a, int threads) {
    if (a.T != 1 || !a.state || a.V % 4 || a.V > 1024 || a.V / 4 > threads) return 0;
    return ceil_div(a.D, threads / (a.V / 4));
}

template <typename T>
int step_t(const GlaArgs& a, bool dependent) {
    const int small = step_rows(a, 256), threads = small <= 16 ? 256 : 512, rows = threads == 256 ? small : step_rows(a, 512);
    const size_t smem = ((size_t)3 * ((a.D + 3) / 4 * 4) + (a.R + 3) / 4 * 4 + (size_t)threads / (a.V / 4) * a.V) * sizeof(float);
    const dim3 grid(a.B * a.H), block(threads);
    if (rows <= 4) SPT_CUDA(launch_dependent(gla_step_kernel<T, 4>, grid, block, smem, dependent, 1, a));
    else if (rows <= 8) SPT_CUDA(launch_dependent(gla_step_kernel<T, 8>, grid, block, smem, dependent, 1, a));
    else if (rows <= 16 && threads == 256) SPT_CUDA(launch_dependent(gla_step_kernel<T, 16>, grid, block, smem, dependent, 1, a));
    else SPT_CUDA(launch_dependent(gla_step_kernel<T, 24>, grid, block, smem, dependent, 1, a));
    note_submit();
    return 0;
}
bool step_takes(const GlaArgs& a) {
    const int small = step_rows(a, 256), wide = step_rows(a, 512);
    return (small > 0 && small <= 16) || (wide > 8 && wide <= 24);
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
    if (step_takes(a)) return a.dtype == BF16 ? step_t<__nv_bfloat16>(a, dependent) : step_t<float>(a, dependent);
    if (a.dtype == BF16 ? recurrent_t<__nv_bfloat16>(a, o_scratch, dependent) : recurrent_t<float>(a, o_scratch, dependent)) return 1;
    return recurrent_fuses(a) ? 0 : gla_norm_gate(a, o_scratch, dependent);
}

bool gla_chunked_supported(const GlaArgs& a) { return a.dtype == BF16 && a.T > kRecTokens && a.D <= 128 && a.V <= 256 && a.R <= 64 && a.B * a.H <= 65535; }
static size_t chunks_of(const GlaArgs& a) { return (size_t)a.B * a.H * ceil_div(a.T, kChunk); }
size_t gla_chunked_state_bytes(const GlaArgs& a) { return chunks_of(a) * a.D * a.V * sizeof(float); }
size_t gla_chunked_decay_bytes(const GlaArgs& a) { return chunks_of(a) * kChunk * a.D * sizeof(float); }

int gla_chunked(const GlaArgs& a, float* u_scratch, float* dec_scratch) {
    const ChunkArgs p = {a, u_scratch, dec_scratch, ceil_div(a.T, kChunk)};
    return a.D <= 32 ? launch_chunked_v<32>(p) : a.D <= 64 ? launch_chunked_v<64>(p) : launch_chunked_v<128>(p);
}

}  // namespace spt
