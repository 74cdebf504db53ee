// gla.cu -- gated linear attention: per head a [D, V] matrix S with a decay per key channel,
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   alpha = sigmoid(z)^(1/tau),  z = A2 (A1 h) + b,
// followed by an RMS norm of each head's o over V and the gate silu(W_g h).  q carries the factor D^(-1/2).  The recurrence, its
// decays and the norm are f32 whatever the model's dtype; q, k, v, the gate and A1 h come from the layer's input projection.
//
// gla_recurrent walks the tokens one by one (any sizes, both dtypes; a decode step is T = 1); gla_chunked takes bf16 prompts in chunks.
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

// ---------------- prompts: chunks of kChunk tokens on the tensor cores ----------------
// With b_t the running sum of log2 alpha inside a chunk (b_t <= 0, per key channel) and S the state before the chunk:
//   o_t = (q_t 2^(b_t))^T S + sum_(s <= t) A[t][s] v_s,    A[t][s] = sum_d q_t[d] k_s[d] 2^(b_t[d] - b_s[d])
//   S'  = diag(2^(b_C)) S + sum_s (k_s 2^(b_C - b_s)) v_s^T
// Chunks are independent except through S, so three launches do a prompt: the chunks' own sums U = sum_s (k_s 2^(b_C - b_s)) v_s^T
// (gla_chunk_state_kernel), a scan over the chunks that turns U into the state before each (gla_scan_kernel), and the outputs with head
// norm and gate (gla_chunk_out_kernel).  (This is the chunkwise form of "Gated Linear Attention Transformers with Hardware-Efficient
// Training", Yang, Wang, Shen, Panda, Kim.)  Every exponent that is evaluated is <= 0: A is taken in 16 x 16 blocks, off the diagonal
// relative to the last token before the row block (2^(b_t - b_r) 2^(b_r - b_s)), on the diagonal pair by pair, so a strong decay
// underflows where the product is nothing and never overflows.
// Products run as mma.sync on TF32 with each f32 operand split into two TF32 parts (hi hi + hi lo + lo hi: 21 mantissa bits); v comes
// in bf16 and needs no split.  The tiles are 64 rows and the operands are scaled element by element on their way into the fragments,
// so there is no operand for tcgen05 to fetch from shared memory as it lies there; the kernels are bound by that work and by HBM.
constexpr int kChunk = 64;
constexpr int kChunkThreads = 256;

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

__host__ __device__ constexpr int round_up(int n, int m) { return (n + m - 1) / m * m; }
// row pitches of shared-memory tiles: = 4 (mod 32) where fragments take rows by lane / 4 and columns by lane % 4, = 8 where the other way round
__host__ __device__ constexpr int pitch4(int n) { return round_up(n, 32) + 4; }
__host__ __device__ constexpr int pitch8(int n) { return round_up(n, 32) + 8; }

struct ChunkArgs { GlaArgs a; float *u, *dec; int nc; };

// rows of bf16 -> f32 tile [kChunk][pitch], zero outside n rows and w columns (up to wp columns); eight columns at a time where aligned
__device__ __forceinline__ void load_tile(float* dst, int pitch, const __nv_bfloat16* src, long long ld, int n, int w, int wp, float f, bool vec) {
    if (vec) {
        const int per = wp / 8;
        for (int i = threadIdx.x; i < kChunk * per; i += kChunkThreads) {
            const int t = i / per, c = (i - t * per) * 8;
            uint4 raw = make_uint4(0, 0, 0, 0);
            if (t < n && c < w) raw = *reinterpret_cast<const uint4*>(src + (size_t)t * ld + c);
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const float2 x = bf16x2_to_float2(h[j]), y = bf16x2_to_float2(h[j + 1]);
                *reinterpret_cast<float4*>(dst + t * pitch + c + 2 * j) = make_float4(x.x * f, x.y * f, y.x * f, y.y * f);
            }
        }
    } else {
        for (int i = threadIdx.x; i < kChunk * wp; i += kChunkThreads) {
            const int t = i / wp, c = i - t * wp;
            dst[t * pitch + c] = t < n && c < w ? (float)src[(size_t)t * ld + c] * f : 0.0f;
        }
    }
}

__global__ void __launch_bounds__(kChunkThreads) gla_chunk_state_kernel(const ChunkArgs p) {
    extern __shared__ __align__(16) float sm[];
    const GlaArgs& a = p.a;
    const int D = a.D, V = a.V, R = a.R, Dp = round_up(D, 16), Vp = round_up(V, 8);
    const int ldk = pitch8(Dp), ldv = pitch8(Vp);
    float* bs = sm;                               // [kChunk][ldk]: log2 decays, then their running sums
    float* ks = bs + kChunk * ldk;                // [kChunk][ldk]
    float* vs = ks + kChunk * ldk;                // [kChunk][ldv]
    float* a1s = vs + kChunk * ldv;               // [kChunk][R]
    float* a2s = a1s + kChunk * R;                // [R][Dp]
    float* seg = a2s + R * Dp;                    // [4][Dp]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
    const int chunk = blockIdx.x, bh = blockIdx.y, b = bh / a.H, h = bh - b * a.H;
    const int t0 = chunk * kChunk, n = min(kChunk, a.T - t0);
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + ((size_t)b * a.T + t0) * a.ld;
    const bool vec = D % 8 == 0 && V % 8 == 0;
    for (int i = tid; i < kChunk * R; i += kChunkThreads) { const int t = i / R; a1s[i] = t < n ? (float)in[(size_t)t * a.ld + a.c_a + (i - t * R)] : 0.0f; }
    for (int i = tid; i < D * R; i += kChunkThreads) { const int d = i / R, r = i - d * R; a2s[r * Dp + d] = a.a2[(size_t)(h * D) * R + i]; }
    load_tile(ks, ldk, in + a.c_k + h * D, a.ld, n, D, Dp, 1.0f, vec);
    load_tile(vs, ldv, in + a.c_v + h * V, a.ld, n, V, Vp, 1.0f, vec);
    __syncthreads();
    // log2 alpha of four tokens per turn of a thread; padding tokens and channels decay by nothing
    const float to_log2 = 1.4426950408889634f, inv_tau = 1.0f / a.tau;
    for (int i = tid; i < kChunk / 4 * Dp; i += kChunkThreads) {
        const int d = i % Dp, t = i / Dp * 4;
        float z[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        if (d < D) {
            const float bias = a.a2_b[h * D + d];
#pragma unroll
            for (int j = 0; j < 4; j++) z[j] = bias;
            for (int r = 0; r < R; r++) {
                const float w = a2s[r * Dp + d];
#pragma unroll
                for (int j = 0; j < 4; j++) z[j] = fmaf(a1s[(t + j) * R + r], w, z[j]);
            }
        }
#pragma unroll
        for (int j = 0; j < 4; j++) bs[(t + j) * ldk + d] = d < D && t + j < n ? log_decay(z[j], inv_tau) * to_log2 : 0.0f;
    }
    __syncthreads();
    // running sums: four segments of 16 tokens side by side, then the segments' totals on top
    for (int i = tid; i < 4 * Dp; i += kChunkThreads) {
        const int d = i % Dp, s = i / Dp;
        float sum = 0.0f;
#pragma unroll
        for (int t = 0; t < 16; t++) { float& x = bs[(s * 16 + t) * ldk + d]; sum += x; x = sum; }
        seg[s * Dp + d] = sum;
    }
    __syncthreads();
    for (int i = tid; i < kChunk * Dp; i += kChunkThreads) {
        const int d = i % Dp, t = i / Dp, s = t >> 4;
        float off = 0.0f, tot = 0.0f;
#pragma unroll
        for (int j = 0; j < 4; j++) { const float x = seg[j * Dp + d]; if (j < s) off += x; tot += x; }
        const float bt = bs[t * ldk + d] + off;
        if (d < D) p.dec[(((size_t)bh * p.nc + chunk) * kChunk + t) * D + d] = bt;
        ks[t * ldk + d] *= exp2_fast(fminf(tot - bt, 0.0f));
    }
    __syncthreads();
    // U[d][v] = sum_t ks[t][d] vs[t][v]: blocks of 16 channels x 64 values dealt over the warps
    float* u = p.u + ((size_t)bh * p.nc + chunk) * D * V;
    const int mb = Dp / 16, nt = Vp / 8, nb = (nt + 7) / 8;
    for (int blk = warp; blk < mb * nb; blk += kChunkThreads / 32) {
        const int m0 = blk % mb * 16, n0 = blk / mb * 64;
        float acc[8][4] = {};
        for (int k = 0; k < kChunk; k += 8) {
            uint32_t hi[4], lo[4];
            split_tf32(ks[(k + q4) * ldk + m0 + g], hi[0], lo[0]);
            split_tf32(ks[(k + q4) * ldk + m0 + g + 8], hi[1], lo[1]);
            split_tf32(ks[(k + q4 + 4) * ldk + m0 + g], hi[2], lo[2]);
            split_tf32(ks[(k + q4 + 4) * ldk + m0 + g + 8], hi[3], lo[3]);
#pragma unroll
            for (int j = 0; j < 8; j++) {
                const int c = n0 + 8 * j;
                if (c < Vp) {
                    const uint32_t b0 = __float_as_uint(vs[(k + q4) * ldv + c + g]), b1 = __float_as_uint(vs[(k + q4 + 4) * ldv + c + g]);
                    mma_tf32(acc[j], hi, b0, b1);
                    mma_tf32(acc[j], lo, b0, b1);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int d = m0 + g + (e >> 1) * 8, v = n0 + 8 * j + 2 * q4 + (e & 1);
                if (d < D && v < V) u[(size_t)d * V + v] = acc[j][e];
            }
    }
}

// u[c] <- the state before chunk c; state <- the state behind the last one.  One thread per element, eight chunks in flight.
__global__ void __launch_bounds__(256) gla_scan_kernel(const ChunkArgs p) {
    const GlaArgs& a = p.a;
    const int DV = a.D * a.V;
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= (long long)a.B * a.H * DV) return;
    const int bh = (int)(i / DV), e = (int)(i - (long long)bh * DV), d = e / a.V;
    float* u = p.u + (size_t)bh * p.nc * DV + e;
    const float* last = p.dec + ((size_t)bh * p.nc * kChunk + kChunk - 1) * a.D + d;
    float s = a.state ? a.state[i] : 0.0f;
    for (int c0 = 0; c0 < p.nc; c0 += 8) {
        float x[8], f[8];
#pragma unroll
        for (int j = 0; j < 8; j++)
            if (c0 + j < p.nc) { x[j] = u[(size_t)(c0 + j) * DV]; f[j] = last[(size_t)(c0 + j) * kChunk * a.D]; }
#pragma unroll
        for (int j = 0; j < 8; j++)
            if (c0 + j < p.nc) { u[(size_t)(c0 + j) * DV] = s; s = fmaf(s, exp2_fast(f[j]), x[j]); }
    }
    if (a.state) a.state[i] = s;
}

// Warps are 2 (halves of the rows) x 4 (quarters of the values); NT: the most 8-column tiles a warp owns (V <= 32 NT).
template <int NT>
__global__ void __launch_bounds__(kChunkThreads) gla_chunk_out_kernel(const ChunkArgs p) {
    extern __shared__ __align__(16) float sm[];
    const GlaArgs& a = p.a;
    const int D = a.D, V = a.V, Dp = round_up(D, 16), Vp = round_up(V, 8);
    const int ld = pitch4(Dp), ldv = pitch8(Vp);
    constexpr int lda = 68;
    float* bs = sm;                               // [kChunk][ld]: running sums of the log2 decays
    float* qs = bs + kChunk * ld;                 // [kChunk][ld]: q D^(-1/2), later times 2^b
    float* ks = qs + kChunk * ld;
    float* vs = ks + kChunk * ld;                 // [kChunk][ldv]
    float* as = vs + kChunk * ldv;                // [kChunk][lda]: A
    float* red = as + kChunk * lda;               // [4][kChunk]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
    const int chunk = blockIdx.x, bh = blockIdx.y, b = bh / a.H, h = bh - b * a.H;
    const int t0 = chunk * kChunk, n = min(kChunk, a.T - t0);
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + ((size_t)b * a.T + t0) * a.ld;
    const bool vec = D % 8 == 0 && V % 8 == 0;
    const float* dec = p.dec + ((size_t)bh * p.nc + chunk) * kChunk * D;
    for (int i = tid; i < kChunk * Dp; i += kChunkThreads) { const int t = i / Dp, d = i - t * Dp; bs[t * ld + d] = d < D ? dec[(size_t)t * D + d] : 0.0f; }
    load_tile(qs, ld, in + a.c_q + h * D, a.ld, n, D, Dp, 1.0f / sqrtf((float)D), vec);
    load_tile(ks, ld, in + a.c_k + h * D, a.ld, n, D, Dp, 1.0f, vec);
    load_tile(vs, ldv, in + a.c_v + h * V, a.ld, n, V, Vp, 1.0f, vec);
    for (int i = tid; i < kChunk * lda; i += kChunkThreads) as[i] = 0.0f;
    __syncthreads();

    if (warp < 4) {
        // diagonal block `warp`: its 136 pairs (t, s <= t) one by one, four channels at a time
        const int r0 = warp * 16;
#pragma unroll 1
        for (int pr = lane; pr < 136; pr += 32) {
            int t = (int)((sqrtf(8.0f * pr + 1.0f) - 1.0f) * 0.5f);
            while ((t + 1) * (t + 2) / 2 <= pr) t++;
            while (t * (t + 1) / 2 > pr) t--;
            const int s = pr - t * (t + 1) / 2;
            const float *qt = qs + (r0 + t) * ld, *bt = bs + (r0 + t) * ld, *kt = ks + (r0 + s) * ld, *bk = bs + (r0 + s) * ld;
            float acc = 0.0f;
            for (int d = 0; d < Dp; d += 4) {
                const float4 x = *reinterpret_cast<const float4*>(qt + d), y = *reinterpret_cast<const float4*>(kt + d);
                const float4 u = *reinterpret_cast<const float4*>(bt + d), w = *reinterpret_cast<const float4*>(bk + d);
                acc = fmaf(x.x * y.x, exp2_fast(u.x - w.x), acc); acc = fmaf(x.y * y.y, exp2_fast(u.y - w.y), acc);
                acc = fmaf(x.z * y.z, exp2_fast(u.z - w.z), acc); acc = fmaf(x.w * y.w, exp2_fast(u.w - w.w), acc);
            }
            as[(r0 + t) * lda + r0 + s] = acc;
        }
    } else {
        // the six blocks below the diagonal, each as two halves of eight columns: twelve tasks over four warps
#pragma unroll 1
        for (int task = warp - 4; task < 12; task += 4) {
            const int blk = task >> 1, i = blk == 0 ? 1 : blk < 3 ? 2 : 3, j = blk == 0 ? 0 : blk < 3 ? blk - 1 : blk - 3;
            const int r0 = 16 * i, c0 = 16 * j + 8 * (task & 1);
            const float* br = bs + (r0 - 1) * ld;                       // the last token before the row block
            float acc[4] = {};
            for (int k = 0; k < Dp; k += 8) {
                uint32_t ah[4], al[4], bh_[2], bl[2];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int t = r0 + g + (e & 1) * 8, d = k + q4 + (e >> 1) * 4;
                    split_tf32(qs[t * ld + d] * exp2_fast(bs[t * ld + d] - br[d]), ah[e], al[e]);
                }
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int s = c0 + g, d = k + q4 + e * 4;
                    split_tf32(ks[s * ld + d] * exp2_fast(br[d] - bs[s * ld + d]), bh_[e], bl[e]);
                }
                mma_tf32(acc, al, bh_[0], bh_[1]);
                mma_tf32(acc, ah, bl[0], bl[1]);
                mma_tf32(acc, ah, bh_[0], bh_[1]);
            }
#pragma unroll
            for (int e = 0; e < 4; e++) as[(r0 + g + (e >> 1) * 8) * lda + c0 + 2 * q4 + (e & 1)] = acc[e];
        }
    }
    __syncthreads();
    for (int i = tid; i < kChunk * Dp; i += kChunkThreads) { const int t = i / Dp, d = i - t * Dp; qs[t * ld + d] *= exp2_fast(bs[t * ld + d]); }
    __syncthreads();

    const int wm = warp >> 2, wn = warp & 3, nt_all = Vp / 8, per = (nt_all + 3) / 4, first = wn * per, mine = max(0, min(per, nt_all - first));
    float acc[2][NT][4] = {};
    if (chunk > 0 || a.state) {
        // (q 2^b) S: S straight from global memory into the fragments, the next eight channels in flight
        const float* u = p.u + ((size_t)bh * p.nc + chunk) * D * V;
        float cur[NT][2], nxt[NT][2];
        auto fetch = [&](int k, float (&x)[NT][2]) {
#pragma unroll
            for (int j = 0; j < NT; j++) {
                const int v = (first + j) * 8 + g;
#pragma unroll
                for (int e = 0; e < 2; e++) { const int d = k + q4 + 4 * e; x[j][e] = j < mine && v < V && d < D ? u[(size_t)d * V + v] : 0.0f; }
            }
        };
        fetch(0, cur);
        for (int k = 0; k < Dp; k += 8) {
            if (k + 8 < Dp) fetch(k + 8, nxt);
            uint32_t ah[2][4], al[2][4];
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
                for (int e = 0; e < 4; e++) split_tf32(qs[(wm * 32 + i * 16 + g + (e & 1) * 8) * ld + k + q4 + (e >> 1) * 4], ah[i][e], al[i][e]);
#pragma unroll
            for (int j = 0; j < NT; j++) {
                if (j < mine) {
                    uint32_t h0, l0, h1, l1;
                    split_tf32(cur[j][0], h0, l0); split_tf32(cur[j][1], h1, l1);
#pragma unroll
                    for (int i = 0; i < 2; i++) { mma_tf32(acc[i][j], al[i], h0, h1); mma_tf32(acc[i][j], ah[i], l0, l1); mma_tf32(acc[i][j], ah[i], h0, h1); }
                }
            }
#pragma unroll
            for (int j = 0; j < NT; j++) { cur[j][0] = nxt[j][0]; cur[j][1] = nxt[j][1]; }
        }
    }
    // A v up to the diagonal
    for (int k = 0; k < wm * 32 + 32; k += 8) {
        uint32_t ah[2][4], al[2][4];
#pragma unroll
        for (int i = 0; i < 2; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) split_tf32(as[(wm * 32 + i * 16 + g + (e & 1) * 8) * lda + k + q4 + (e >> 1) * 4], ah[i][e], al[i][e]);
#pragma unroll
        for (int j = 0; j < NT; j++) {
            if (j < mine) {
                const int c = (first + j) * 8 + g;
                const uint32_t b0 = __float_as_uint(vs[(k + q4) * ldv + c]), b1 = __float_as_uint(vs[(k + q4 + 4) * ldv + c]);
#pragma unroll
                for (int i = 0; i < 2; i++)
                    if (k < wm * 32 + i * 16 + 16) { mma_tf32(acc[i][j], al[i], b0, b1); mma_tf32(acc[i][j], ah[i], b0, b1); }
            }
        }
    }
    // head norm over V and gate; a row's values lie with four warps
#pragma unroll
    for (int i = 0; i < 2; i++)
#pragma unroll
        for (int r = 0; r < 2; r++) {
            float sq = 0.0f;
#pragma unroll
            for (int j = 0; j < NT; j++) { sq = fmaf(acc[i][j][2 * r], acc[i][j][2 * r], sq); sq = fmaf(acc[i][j][2 * r + 1], acc[i][j][2 * r + 1], sq); }
            sq += __shfl_xor_sync(0xffffffffu, sq, 1);
            sq += __shfl_xor_sync(0xffffffffu, sq, 2);
            if (q4 == 0) red[wn * kChunk + wm * 32 + i * 16 + r * 8 + g] = sq;
        }
    __syncthreads();
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + ((size_t)b * a.T + t0) * a.ld_out + h * V;
    const __nv_bfloat16* gate = in + a.c_g + h * V;
    const bool even = V % 2 == 0;
#pragma unroll
    for (int i = 0; i < 2; i++)
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int t = wm * 32 + i * 16 + r * 8 + g;
            if (t >= n) continue;
            const float inv = 1.0f / sqrtf((red[t] + red[kChunk + t] + red[2 * kChunk + t] + red[3 * kChunk + t]) / (float)V + a.eps);
#pragma unroll
            for (int j = 0; j < NT; j++) {
                const int v = (first + j) * 8 + 2 * q4;
                if (j >= mine || v >= V) continue;
                const float x = acc[i][j][2 * r] * inv * a.head_norm[v];
                if (even) {
                    const float y = acc[i][j][2 * r + 1] * inv * a.head_norm[v + 1];
                    const float2 gg = bf16x2_to_float2(*reinterpret_cast<const __nv_bfloat162*>(gate + (size_t)t * a.ld + v));
                    *reinterpret_cast<__nv_bfloat162*>(out + (size_t)t * a.ld_out + v) = __floats2bfloat162_rn(x * silu_fast(gg.x), y * silu_fast(gg.y));
                } else {
                    out[(size_t)t * a.ld_out + v] = __float2bfloat16_rn(x * silu_fast((float)gate[(size_t)t * a.ld + v]));
                    if (v + 1 < V) out[(size_t)t * a.ld_out + v + 1] = __float2bfloat16_rn(acc[i][j][2 * r + 1] * inv * a.head_norm[v + 1] * silu_fast((float)gate[(size_t)t * a.ld + v + 1]));
                }
            }
        }
    if (h == a.H - 1)                             // the padding of the output rows
        for (int i = tid; i < n * 8; i += kChunkThreads) { const int c = V + (i & 7); if (h * V + c < a.ld_out) out[(size_t)(i >> 3) * a.ld_out + c] = __float2bfloat16_rn(0.0f); }
}

size_t chunk_state_smem(const GlaArgs& a) {
    const int Dp = round_up(a.D, 16), Vp = round_up(a.V, 8);
    return ((size_t)kChunk * (2 * pitch8(Dp) + pitch8(Vp) + a.R) + (size_t)a.R * Dp + 4 * Dp) * sizeof(float);
}
size_t chunk_out_smem(const GlaArgs& a) {
    const int Dp = round_up(a.D, 16), Vp = round_up(a.V, 8);
    return ((size_t)kChunk * (3 * pitch4(Dp) + pitch8(Vp) + 68) + 4 * kChunk) * sizeof(float);
}
constexpr size_t kMaxSmem = 227 * 1024;

template <int NT>
int launch_chunk_out(const ChunkArgs& p) {
    auto kern = gla_chunk_out_kernel<NT>;
    const size_t smem = chunk_out_smem(p.a);
    static size_t granted = 48 * 1024;
    if (smem > granted) { SPT_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); granted = smem; }
    kern<<<dim3(p.nc, p.a.B * p.a.H), kChunkThreads, smem, rt().stream>>>(p);
    SPT_LAUNCH_CHECK("gla_chunk_out");
    return 0;
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

bool gla_chunked_supported(const GlaArgs& a) {
    return a.dtype == BF16 && a.D <= 128 && a.V <= 256 && a.B * a.H <= 65535 && chunk_state_smem(a) <= kMaxSmem && chunk_out_smem(a) <= kMaxSmem;
}
static size_t chunks_of(const GlaArgs& a) { return (size_t)a.B * a.H * ceil_div(a.T, kChunk); }
size_t gla_chunked_state_bytes(const GlaArgs& a) { return chunks_of(a) * a.D * a.V * sizeof(float); }
size_t gla_chunked_decay_bytes(const GlaArgs& a) { return chunks_of(a) * kChunk * a.D * sizeof(float); }

int gla_chunked(const GlaArgs& a, float* u_scratch, float* dec_scratch) {
    const ChunkArgs p = {a, u_scratch, dec_scratch, ceil_div(a.T, kChunk)};
    const size_t smem = chunk_state_smem(a);
    static size_t granted = 48 * 1024;
    if (smem > granted) { SPT_CUDA(cudaFuncSetAttribute(gla_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); granted = smem; }
    gla_chunk_state_kernel<<<dim3(p.nc, a.B * a.H), kChunkThreads, smem, rt().stream>>>(p);
    SPT_LAUNCH_CHECK("gla_chunk_state");
    const long long elems = (long long)a.B * a.H * a.D * a.V;
    gla_scan_kernel<<<(unsigned)((elems + 255) / 256), 256, 0, rt().stream>>>(p);
    SPT_LAUNCH_CHECK("gla_scan");
    const int nt = ceil_div(ceil_div(a.V, 8), 4);
    return nt <= 2 ? launch_chunk_out<2>(p) : nt <= 4 ? launch_chunk_out<4>(p) : launch_chunk_out<8>(p);
}

}  // namespace spt
