// latent_attention.cu -- attention whose keys and values are projections of one cached latent per position.
//
// A position keeps the row [c | kr]: its RMS-normed latent c (kv values) and one rotated key part kr (rot values) that all heads share.
// Head h scores a key with (qn . W_uk,h c + qr . kr) * scale and takes its value from W_uv,h c.  Since W_uk,h and W_uv,h are linear,
//   qn . (W_uk,h c) = (W_uk,h^T qn) . c      and      sum_j p_j W_uv,h c_j = W_uv,h (sum_j p_j c_j),
// so a few query tokens attend over the cached rows themselves ("absorbed": H * (kv + rot) values read once per position instead of
// H * (D + V) expanded ones), while a prompt expands keys and values with one GEMM and runs the fused kernel (attention_fused.cu).
// Scores, softmax weights and the weighted sum are f32; positions and angles come from an f32 table evaluated in f64 on the host.
#include "layered.h"
#include "pdl.cuh"
#include <math.h>
#include <cooperative_groups.h>

namespace spt {

namespace {

__device__ __forceinline__ float block_sum(float v, float* sh) {        // 128 threads; every thread gets the sum
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
    __syncthreads();
    return (sh[0] + sh[1]) + (sh[2] + sh[3]);
}

__device__ __forceinline__ float sigmoid_exact(float z) { return 1.0f / (1.0f + expf(-z)); }

// One CTA per token: RMS norm of the query latent into cq; RMS norm of the latent and rotation of the key part into the cached row.
template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentArgs a) {
    __shared__ float sh[4];
    pdl_release();
    const int m = blockIdx.x, b = m / a.T, tid = threadIdx.x;
    pdl_acquire();
    const int pos = (a.pos_dev ? a.pos_dev[0] : a.first) + (m - b * a.T);
    const T* in = static_cast<const T*>(a.in) + (size_t)m * a.ld_in;
    {
        float sq = 0.0f;
        for (int i = tid; i < a.q_rank; i += 128) { const float v = (float)in[a.c_dq + i]; sq = fmaf(v, v, sq); }
        const float inv = 1.0f / sqrtf(block_sum(sq, sh) / (float)a.q_rank + a.eps);
        T* cq = static_cast<T*>(a.cq) + (size_t)m * a.ld_cq;
        for (int i = tid; i < a.ld_cq; i += 128) cq[i] = (T)(i < a.q_rank ? (float)in[a.c_dq + i] * inv * a.dq_norm[i] : 0.0f);
    }
    T* row = static_cast<T*>(a.rows) + (size_t)b * a.seq_stride + (size_t)pos * a.row;
    const T* kv = in + a.c_dkv;
    float sq = 0.0f;
    for (int i = tid; i < a.kv; i += 128) { const float v = (float)kv[i]; sq = fmaf(v, v, sq); }
    const float inv = 1.0f / sqrtf(block_sum(sq, sh) / (float)a.kv + a.eps);
    for (int i = tid; i < a.kv8; i += 128) row[i] = (T)(i < a.kv ? (float)kv[i] * inv * a.dkv_norm[i] : 0.0f);
    const T* kr = kv + a.kv;
    const int half = a.rope_dims / 2;
    for (int i = tid; i < a.row - a.kv8; i += 128) {
        float v = i < a.rot ? (float)kr[i] : 0.0f;
        if (i < a.rope_dims) {
            const float2 cs = a.angles[(size_t)pos * half + (i >> 1)];
            const float o = (float)kr[i ^ 1];
            v = (i & 1) ? v * cs.x + o * cs.y : v * cs.x - o * cs.y;
        }
        row[a.kv8 + i] = (T)v;
    }
}

// eight bf16 at a time
struct Eight { float v[8]; };
__device__ __forceinline__ Eight load_eight(const __nv_bfloat16* p) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
    Eight e;
#pragma unroll
    for (int i = 0; i < 4; i++) { const float2 f = bf16x2_to_float2(h[i]); e.v[2 * i] = f.x; e.v[2 * i + 1] = f.y; }
    return e;
}
__device__ __forceinline__ void store_eight(__nv_bfloat16* p, const Eight& e) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; i++) h[i] = __floats2bfloat162_rn(e.v[2 * i], e.v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
}
__device__ __forceinline__ void rotate_eight(Eight& e, const float2* cs) {      // four pairs by four angles (16-byte aligned)
#pragma unroll
    for (int i = 0; i < 4; i += 2) {
        const float4 c = __ldg(reinterpret_cast<const float4*>(cs + i));
        const float u0 = e.v[2 * i] * c.x - e.v[2 * i + 1] * c.y, v0 = e.v[2 * i + 1] * c.x + e.v[2 * i] * c.y;
        const float u1 = e.v[2 * i + 2] * c.z - e.v[2 * i + 3] * c.w, v1 = e.v[2 * i + 3] * c.z + e.v[2 * i + 2] * c.w;
        e.v[2 * i] = u0; e.v[2 * i + 1] = v0; e.v[2 * i + 2] = u1; e.v[2 * i + 3] = v1;
    }
}

// The same as latent_prep_kernel for bf16 sizes that are multiples of eight: one warp per token, the row in registers.  NQ / NK: groups
// of eight per lane of the query latent and of the latent.
template <int NQ, int NK>
__global__ void __launch_bounds__(128) latent_prep_vec_kernel(const LatentArgs a) {
    pdl_release();
    const int m = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31, b = m / a.T;
    pdl_acquire();
    if (m >= a.B * a.T) return;
    const int pos = (a.pos_dev ? a.pos_dev[0] : a.first) + (m - b * a.T);
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + (size_t)m * a.ld_in;
    const int nq = a.q_rank / 8, nk = a.kv / 8, nr = a.rot / 8;
    Eight q[NQ], c[NK], r = {};
    float sq = 0.0f, sc = 0.0f;
#pragma unroll
    for (int i = 0; i < NQ; i++) if (i * 32 + lane < nq) q[i] = load_eight(in + a.c_dq + (i * 32 + lane) * 8);
#pragma unroll
    for (int i = 0; i < NK; i++) if (i * 32 + lane < nk) c[i] = load_eight(in + a.c_dkv + (i * 32 + lane) * 8);
    if (lane < nr) r = load_eight(in + a.c_dkv + a.kv + lane * 8);
#pragma unroll
    for (int i = 0; i < NQ; i++) if (i * 32 + lane < nq) {
#pragma unroll
        for (int j = 0; j < 8; j++) sq = fmaf(q[i].v[j], q[i].v[j], sq);
    }
#pragma unroll
    for (int i = 0; i < NK; i++) if (i * 32 + lane < nk) {
#pragma unroll
        for (int j = 0; j < 8; j++) sc = fmaf(c[i].v[j], c[i].v[j], sc);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) { sq += __shfl_xor_sync(0xffffffffu, sq, o); sc += __shfl_xor_sync(0xffffffffu, sc, o); }
    const float iq = 1.0f / sqrtf(sq / (float)a.q_rank + a.eps), ic = 1.0f / sqrtf(sc / (float)a.kv + a.eps);
    __nv_bfloat16* cq = static_cast<__nv_bfloat16*>(a.cq) + (size_t)m * a.ld_cq;
    __nv_bfloat16* row = static_cast<__nv_bfloat16*>(a.rows) + (size_t)b * a.seq_stride + (size_t)pos * a.row;
    auto scaled = [](Eight e, float inv, const float* w) {
        const float4 w0 = __ldg(reinterpret_cast<const float4*>(w)), w1 = __ldg(reinterpret_cast<const float4*>(w + 4));
        const float ww[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
        for (int j = 0; j < 8; j++) e.v[j] = e.v[j] * inv * ww[j];
        return e;
    };
#pragma unroll
    for (int i = 0; i < NQ; i++) if (i * 32 + lane < nq) store_eight(cq + (i * 32 + lane) * 8, scaled(q[i], iq, a.dq_norm + (i * 32 + lane) * 8));
#pragma unroll
    for (int i = 0; i < NK; i++) if (i * 32 + lane < nk) store_eight(row + (i * 32 + lane) * 8, scaled(c[i], ic, a.dkv_norm + (i * 32 + lane) * 8));
    if (lane < nr) {
        if (lane * 8 < a.rope_dims) rotate_eight(r, a.angles + (size_t)pos * (a.rope_dims / 2) + lane * 4);
        store_eight(row + a.kv8 + lane * 8, r);
    }
}

bool vec_sizes(const LatentArgs& a) {
    return a.dtype == BF16 && a.q_rank % 8 == 0 && a.kv % 8 == 0 && a.rot % 8 == 0 && a.rope_dims % 8 == 0 && a.D % 8 == 0 && a.rot <= 256;
}

// rotation of every head's rot part in place, four pairs per thread
__global__ void __launch_bounds__(256) latent_rope_q_vec_kernel(const LatentArgs a) {
    const int per = a.rope_dims / 8;
    const long long idx = (long long)blockIdx.x * 256 + threadIdx.x;
    if (idx >= (long long)a.B * a.T * a.H * per) return;
    const int e = (int)(idx % per);
    const long long mh = idx / per, m = mh / a.H;
    const int h = (int)(mh - m * a.H), pos = (a.pos_dev ? a.pos_dev[0] : a.first) + (int)(m % a.T);
    __nv_bfloat16* p = static_cast<__nv_bfloat16*>(a.q) + m * a.ld_q + (long long)h * (a.D + a.rot) + a.D + 8 * e;
    Eight v = load_eight(p);
    rotate_eight(v, a.angles + (size_t)pos * (a.rope_dims / 2) + 4 * e);
    store_eight(p, v);
}

// rotation of neighbouring pairs of every head's rot part, in place
template <typename T>
__global__ void __launch_bounds__(256) latent_rope_q_kernel(const LatentArgs a) {
    const int half = a.rope_dims / 2;
    const long long idx = (long long)blockIdx.x * 256 + threadIdx.x;
    if (idx >= (long long)a.B * a.T * a.H * half) return;
    const int pr = (int)(idx % half);
    const long long mh = idx / half;
    const int h = (int)(mh % a.H);
    const long long m = mh / a.H;
    const int pos = (a.pos_dev ? a.pos_dev[0] : a.first) + (int)(m % a.T);
    const float2 cs = a.angles[(size_t)pos * half + pr];
    T* p = static_cast<T*>(a.q) + m * a.ld_q + (long long)h * (a.D + a.rot) + a.D + 2 * pr;
    const float u = (float)p[0], v = (float)p[1];
    p[0] = (T)(u * cs.x - v * cs.y);
    p[1] = (T)(v * cs.x + u * cs.y);
}

// qabs[m][h] = [W_uk,h^T qn | rotated qr]: one thread per column of the row, the head's query in shared memory
template <typename T>
__global__ void __launch_bounds__(128) latent_absorb_kernel(const LatentArgs a) {
    extern __shared__ float qs[];                        // [D + rot]
    pdl_release();
    const int h = blockIdx.y, m = blockIdx.z, c = blockIdx.x * 128 + threadIdx.x;
    pdl_acquire();
    const T* q = static_cast<const T*>(a.q) + (size_t)m * a.ld_q + (size_t)h * (a.D + a.rot);
    for (int i = threadIdx.x; i < a.D + a.rot; i += 128) qs[i] = (float)q[i];
    __syncthreads();
    if (c >= a.row) return;
    float v = 0.0f;
    if (c < a.kv) {
        const T* w = static_cast<const T*>(a.w_uk) + (size_t)h * a.D * a.ld_w + c;
        for (int d = 0; d < a.D; d++) v = fmaf(qs[d], (float)w[(size_t)d * a.ld_w], v);
    } else if (c >= a.kv8 && c - a.kv8 < a.rot) {
        const int i = c - a.kv8;
        v = qs[a.D + i];
        if (i < a.rope_dims) {
            const int pos = (a.pos_dev ? a.pos_dev[0] : a.first) + m % a.T;
            const float2 cs = a.angles[(size_t)pos * (a.rope_dims / 2) + (i >> 1)];
            const float o = qs[a.D + (i ^ 1)];
            v = (i & 1) ? v * cs.x + o * cs.y : v * cs.x - o * cs.y;
        }
    }
    static_cast<float*>(a.qabs)[((size_t)m * a.H + h) * a.row + c] = v;
}

// One CTA per (head, token): four warps share the keys 0 .. pos, each with a running (maximum, sum, weighted latent); merged at the
// end in warp order.  NV: columns of a row per lane (32 * NV >= row).
template <typename T, int NV>
__global__ void __launch_bounds__(128) latent_rows_kernel(const LatentArgs a) {
    extern __shared__ float acc_sh[];                    // [4][32 * NV] weighted latents
    __shared__ float m_sh[4], l_sh[4];
    pdl_release();
    const int h = blockIdx.x, mt = blockIdx.y, b = mt / a.T, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_acquire();
    const int n = (a.pos_dev ? a.pos_dev[0] : a.first) + (mt - b * a.T) + 1;
    const T* rows = static_cast<const T*>(a.rows) + (size_t)b * a.seq_stride;
    const float* qp = static_cast<const float*>(a.qabs) + ((size_t)mt * a.H + h) * a.row;
    float q[NV], o[NV];
#pragma unroll
    for (int i = 0; i < NV; i++) { const int c = i * 32 + lane; q[i] = c < a.row ? qp[c] : 0.0f; o[i] = 0.0f; }
    float mx = -INFINITY, l = 0.0f;
    for (int p = warp; p < n; p += 4) {
        const T* r = rows + (size_t)p * a.row;
        float k[NV], s = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; i++) { const int c = i * 32 + lane; k[i] = c < a.row ? (float)r[c] : 0.0f; s = fmaf(q[i], k[i], s); }
#pragma unroll
        for (int w = 16; w > 0; w >>= 1) s += __shfl_xor_sync(0xffffffffu, s, w);
        s *= a.scale;
        const float mn = fmaxf(mx, s), corr = expf(mx - mn), e = expf(s - mn);
        l = l * corr + e;
#pragma unroll
        for (int i = 0; i < NV; i++) o[i] = fmaf(o[i], corr, e * k[i]);
        mx = mn;
    }
    if (lane == 0) { m_sh[warp] = mx; l_sh[warp] = l; }
#pragma unroll
    for (int i = 0; i < NV; i++) acc_sh[warp * 32 * NV + i * 32 + lane] = o[i];
    __syncthreads();
    float tm = fmaxf(fmaxf(m_sh[0], m_sh[1]), fmaxf(m_sh[2], m_sh[3])), tl = 0.0f, f[4];
#pragma unroll
    for (int w = 0; w < 4; w++) { f[w] = m_sh[w] == -INFINITY ? 0.0f : expf(m_sh[w] - tm); tl += l_sh[w] * f[w]; }
    const float inv = 1.0f / tl;
    float* out = static_cast<float*>(a.olat) + ((size_t)mt * a.H + h) * a.kv8;
    for (int c = threadIdx.x; c < a.kv8; c += 128) {
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < 4; w++) v = fmaf(acc_sh[w * 32 * NV + c], f[w], v);
        out[c] = v * inv;
    }
}

// out[m][h*V + v] = sigmoid(gate) * sum_c W_uv[h*V + v][c] olat[m][h][c]: one warp per value, eight per CTA
template <typename T>
__global__ void __launch_bounds__(256) latent_value_kernel(const LatentArgs a) {
    pdl_release();
    const int m = blockIdx.y, lane = threadIdx.x & 31, i = blockIdx.x * 8 + (threadIdx.x >> 5);
    pdl_acquire();
    if (i >= a.ld_out) return;
    T* out = static_cast<T*>(a.out) + (size_t)m * a.ld_out;
    if (i >= a.H * a.V) { if (lane == 0) out[i] = (T)0.0f; return; }
    const int h = i / a.V;
    const T* w = static_cast<const T*>(a.w_uv) + (size_t)i * a.ld_w;
    const float* ol = static_cast<const float*>(a.olat) + ((size_t)m * a.H + h) * a.kv8;
    float s = 0.0f;
    for (int c = lane; c < a.kv; c += 32) s = fmaf((float)w[c], ol[c], s);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) {
        const float g = (float)static_cast<const T*>(a.in)[(size_t)m * a.ld_in + a.c_g + h];
        out[i] = (T)(s * sigmoid_exact(g));
    }
}

// ---------------- few tokens, bf16: attention over the cached rows on the tensor cores ----------------
// A cluster of `splits` CTAs owns one token and sixteen heads; each CTA walks its part of the positions in tiles of 64 cached rows
// (cp.async, two tiles in flight).  Per tile: scores [16 heads x 64 keys] = Q rows^T, sixteen warps taking eight keys and half of
// the columns each; an online softmax by one warp per head; O [16 x kv] += P rows, the warps taking kv / 16 columns each, with P as the sum of two bf16 numbers (16
// mantissa bits).  The cluster's parts meet through distributed shared memory, every CTA merging a slice of the columns.  A row is read
// from HBM once for all heads: 2 (kv + rot) bytes per position and sixteen heads.  mma.sync m16n8k16: sixteen heads are a sixteenth of a
// tcgen05 tile's rows, and the kernel streams the cache at a few FLOP per byte.
// NTW: 8-column tiles of the latent per warp (kv8 <= 128 NTW).
constexpr int kLdThreads = 512, kLdKeys = 64, kLdP = 72, kLdS = 68;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

__host__ __device__ constexpr int ld_pitch(int row) { return (row + 31) / 32 * 32 + 8; }      // an odd number of 16-byte units: ldmatrix without conflicts
inline size_t latent_decode_smem(int row) {
    return (size_t)(2 * kLdKeys + 16) * ld_pitch(row) * 2 + 2 * 16 * kLdP * 2 + (size_t)2 * 16 * kLdS * 4 + 3 * 16 * 4;
}

template <int NTW>
__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_kernel(const LatentArgs a, int splits, int groups) {
    extern __shared__ __align__(16) uint8_t raw[];
    const int pitch = ld_pitch(a.row), wide = pitch - 8;
    __nv_bfloat16* tile = reinterpret_cast<__nv_bfloat16*>(raw);                // [2][64][pitch]
    __nv_bfloat16* qs = tile + 2 * kLdKeys * pitch;                             // [16][pitch]
    __nv_bfloat16* ph = qs + 16 * pitch;                                        // [2][16][kLdP]: softmax weights, upper and lower half
    float* ss = reinterpret_cast<float*>(ph + 2 * 16 * kLdP);                   // [2][16][kLdS]: scores over either half of the columns
    float* corr_s = ss + 2 * 16 * kLdS;                                             // [16]
    float* m_s = corr_s + 16;                                                   // [16]
    float* l_s = m_s + 16;                                                      // [16]
    float* o_s = reinterpret_cast<float*>(raw);                                 // [16][kv8 + 4], over the tiles once they are done
    pdl_release();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
    const int rank = blockIdx.x % splits, item = blockIdx.x / splits, hg = item % groups, mt = item / groups, b = mt / a.T;
    const int pos0 = a.pos_dev ? a.pos_dev[0] : a.first, n = pos0 + (mt - b * a.T) + 1;
    const int part = ((n + splits - 1) / splits + kLdKeys - 1) / kLdKeys * kLdKeys, lo = min(n, rank * part), hi = min(n, lo + part);
    const __nv_bfloat16* rows = static_cast<const __nv_bfloat16*>(a.rows) + (size_t)b * a.seq_stride;
    const int per_row = a.row / 8;
    auto load = [&](int stage, int k0) {
        __nv_bfloat16* dst = tile + stage * kLdKeys * pitch;
#pragma unroll
        for (int r = 0; r < kLdKeys / 16; r++) {                                // a warp copies four rows
            const int k = warp + 16 * r;
            const bool live = k0 + k < hi;
            const __nv_bfloat16* src = rows + (size_t)(k0 + k) * a.row;
            const uint32_t d = smem_addr(dst + k * pitch);
            for (int c = lane * 8; c < a.row; c += 256) {
                if (live) cp_async16(d + c * 2, src + c);
                else *reinterpret_cast<uint4*>(dst + k * pitch + c) = make_uint4(0, 0, 0, 0);
            }
        }
    };
    // rows before this step's tokens were written by earlier steps: the first tile may be requested before the kernels ahead are done
    const bool early = lo + kLdKeys <= pos0 && lo < hi;
    if (early) load(0, lo);
    for (int i = tid; i < (2 * kLdKeys + 16) * (wide - a.row); i += kLdThreads) {       // columns past the row: zero in every tile and in Q
        const int r = i / (wide - a.row), c = a.row + i % (wide - a.row);
        tile[r * pitch + c] = __float2bfloat16_rn(0.0f);
    }
    pdl_acquire();
    if (!early && lo < hi) load(0, lo);
    asm volatile("cp.async.commit_group;" ::: "memory");
    // Q: absorbed part as it is, rotated part rotated to the token's position; missing heads of the last group are zero
    for (int i = tid; i < 16 * per_row; i += kLdThreads) {
        const int r = i / per_row, c = (i - r * per_row) * 8, h = hg * 16 + r;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (h < a.H) {
            if (c < a.kv8) v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.qabs) + ((size_t)mt * a.H + h) * a.kv8 + c);
            else {
                const __nv_bfloat16* qr = static_cast<const __nv_bfloat16*>(a.q) + (size_t)mt * a.ld_q + (size_t)h * (a.D + a.rot) + a.D;
                __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const int e = c - a.kv8 + 2 * j;
                    float x = e < a.rot ? __bfloat162float(qr[e]) : 0.0f, y = e + 1 < a.rot ? __bfloat162float(qr[e + 1]) : 0.0f;
                    if (e < a.rope_dims) {
                        const float2 cs = a.angles[(size_t)(n - 1) * (a.rope_dims / 2) + (e >> 1)];
                        const float u = x * cs.x - y * cs.y;
                        y = y * cs.x + x * cs.y; x = u;
                    }
                    o[j] = __floats2bfloat162_rn(x, y);
                }
            }
        }
        *reinterpret_cast<uint4*>(qs + r * pitch + c) = v;
    }
    float acc[NTW][4];
#pragma unroll
    for (int j = 0; j < NTW; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) acc[j][e] = 0.0f;
    const float scale = a.scale * 1.4426950408889634f;
    const int srow = warp, sk = lane * 2;                                       // softmax: one warp per head, two keys per lane
    float m = -INFINITY, l = 0.0f;
    int stage = 0;
    for (int k0 = lo; k0 < hi; k0 += kLdKeys, stage ^= 1) {
        if (k0 != lo) __syncthreads();                                          // the other stage's readers are done
        if (k0 + kLdKeys < hi) load(stage ^ 1, k0 + kLdKeys);
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const __nv_bfloat16* tl = tile + stage * kLdKeys * pitch;
        {
            float s0[4] = {0, 0, 0, 0}, s1[4] = {0, 0, 0, 0};
            const int nt = warp & 7, half = warp >> 3, kmid = (wide / 32 + 1) / 2 * 32;
            const uint32_t qa = smem_addr(qs + (lane & 15) * pitch + (lane >> 4) * 8), ka = smem_addr(tl + (nt * 8 + (lane & 7)) * pitch + (lane >> 3) * 8);
#pragma unroll 4
            for (int k = half ? kmid : 0; k < (half ? wide : kmid); k += 32) {
                uint32_t x[4], y[4], kb[4];
                ldsm4(x, qa + k * 2); ldsm4(y, qa + k * 2 + 32); ldsm4(kb, ka + k * 2);
                mma_bf16(s0, x, kb[0], kb[1]);
                mma_bf16(s1, y, kb[2], kb[3]);
            }
            float* so = ss + (half * 16 + g) * kLdS + nt * 8 + 2 * q4;
            *reinterpret_cast<float2*>(so) = make_float2((s0[0] + s1[0]) * scale, (s0[1] + s1[1]) * scale);
            *reinterpret_cast<float2*>(so + 8 * kLdS) = make_float2((s0[2] + s1[2]) * scale, (s0[3] + s1[3]) * scale);
        }
        __syncthreads();
        {
            const float2 sa = *reinterpret_cast<const float2*>(ss + srow * kLdS + sk), sb = *reinterpret_cast<const float2*>(ss + (16 + srow) * kLdS + sk);
            const float x = k0 + sk < hi ? sa.x + sb.x : -INFINITY, y = k0 + sk + 1 < hi ? sa.y + sb.y : -INFINITY;
            float mx = fmaxf(m, fmaxf(x, y));
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float corr = ex2(m - mx);                                     // first tile: 2^(-inf) = 0
            const float e0 = ex2(x - mx), e1 = ex2(y - mx);
            const __nv_bfloat162 hi2 = __floats2bfloat162_rn(e0, e1);
            const float2 f = bf16x2_to_float2(hi2);
            const __nv_bfloat162 lo2 = __floats2bfloat162_rn(e0 - f.x, e1 - f.y);
            float sum = e0 + e1;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l = l * corr + sum; m = mx;
            *reinterpret_cast<__nv_bfloat162*>(ph + srow * kLdP + sk) = hi2;
            *reinterpret_cast<__nv_bfloat162*>(ph + (16 + srow) * kLdP + sk) = lo2;
            if (lane == 0) corr_s[srow] = corr;
        }
        __syncthreads();
        {
            const float f0 = corr_s[g], f1 = corr_s[g + 8];
#pragma unroll
            for (int j = 0; j < NTW; j++) { acc[j][0] *= f0; acc[j][1] *= f0; acc[j][2] *= f1; acc[j][3] *= f1; }
            const uint32_t pa = smem_addr(ph + (lane & 15) * kLdP + (lane >> 4) * 8), va = smem_addr(tl + (lane & 15) * pitch + warp * NTW * 8 + (lane >> 4) * 8);
#pragma unroll
            for (int k = 0; k < kLdKeys; k += 16) {
                uint32_t x[4], y[4];
                ldsm4(x, pa + k * 2); ldsm4(y, pa + 16 * kLdP * 2 + k * 2);
#pragma unroll
                for (int j = 0; j < NTW; j += 2) {
                    if (warp * NTW * 8 + j * 8 < a.kv8) {
                        uint32_t vb[4];
                        ldsm4_trans(vb, va + (k * pitch + j * 8) * 2);
                        mma_bf16(acc[j], x, vb[0], vb[1]); mma_bf16(acc[j], y, vb[0], vb[1]);
                        mma_bf16(acc[j + 1], x, vb[2], vb[3]); mma_bf16(acc[j + 1], y, vb[2], vb[3]);
                    }
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int lo_ = a.kv8 + 4;
#pragma unroll
    for (int j = 0; j < NTW; j++) {
        const int c = (warp * NTW + j) * 8 + 2 * q4;
        if (c < a.kv8) {
            *reinterpret_cast<float2*>(o_s + g * lo_ + c) = make_float2(acc[j][0], acc[j][1]);
            *reinterpret_cast<float2*>(o_s + (g + 8) * lo_ + c) = make_float2(acc[j][2], acc[j][3]);
        }
    }
    if (lane == 0) { m_s[srow] = m; l_s[srow] = l; }
    namespace cg = cooperative_groups;
    cg::cluster_group cluster = cg::this_cluster();
    if (splits > 1) cluster.sync(); else __syncthreads();
    // this CTA's slice of the columns, over all parts
    const int slice = (a.kv8 / 8 + splits - 1) / splits * 8, c0 = rank * slice, c1 = min(a.kv8, c0 + slice);
    const int w2 = max(0, c1 - c0) / 2;
    for (int i = tid; i < 16 * w2; i += kLdThreads) {
        const int r = i / w2, c = c0 + (i - r * w2) * 2, h = hg * 16 + r;
        if (h >= a.H) continue;
        float tm = -INFINITY, tl = 0.0f;
        float2 t = make_float2(0.0f, 0.0f);
        for (int s = 0; s < splits; s++) tm = fmaxf(tm, splits > 1 ? cluster.map_shared_rank(m_s, s)[r] : m_s[r]);
        for (int s = 0; s < splits; s++) {
            const float* om = splits > 1 ? cluster.map_shared_rank(o_s, s) : o_s;
            const float ms = splits > 1 ? cluster.map_shared_rank(m_s, s)[r] : m_s[r], ls = splits > 1 ? cluster.map_shared_rank(l_s, s)[r] : l_s[r];
            const float f = ms == -INFINITY ? 0.0f : ex2(ms - tm);
            const float2 v = *reinterpret_cast<const float2*>(om + r * lo_ + c);
            tl = fmaf(ls, f, tl); t.x = fmaf(v.x, f, t.x); t.y = fmaf(v.y, f, t.y);
        }
        const float inv = 1.0f / tl;
        *reinterpret_cast<__nv_bfloat162*>(static_cast<__nv_bfloat16*>(a.olat) + ((size_t)mt * a.H + h) * a.kv8 + c) = __floats2bfloat162_rn(t.x * inv, t.y * inv);
    }
    if (splits > 1) cluster.sync();                     // no CTA leaves while its shared memory may still be read
}

template <int NTW>
int launch_latent_decode(const LatentArgs& a, bool dependent) {
    auto kern = latent_decode_kernel<NTW>;
    const size_t smem = latent_decode_smem(a.row);
    static size_t granted = 48 * 1024;
    if (smem > granted) { SPT_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); granted = smem; }
    const int groups = ceil_div(a.H, 16), items = a.B * a.T * groups;
    // the widest split whose clusters are all resident at once and leave every CTA a tile: a CTA fills its SM, and how many clusters of 2,
    // 4, 8 such CTAs fit depends on how the SMs are grouped
    static int fits[4] = {0, -1, -1, -1};
    static size_t fits_smem = 0;
    if (fits_smem != smem) {
        fits_smem = smem;
        for (int k = 1; k < 4; k++) {
            cudaLaunchConfig_t cfg = {};
            cfg.gridDim = dim3(8 * 148); cfg.blockDim = dim3(kLdThreads); cfg.dynamicSmemBytes = smem;
            cudaLaunchAttribute at[1];
            at[0].id = cudaLaunchAttributeClusterDimension; at[0].val.clusterDim.x = 1u << k; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
            cfg.attrs = at; cfg.numAttrs = 1;
            int c = 0;
            if (cudaOccupancyMaxActiveClusters(&c, kern, &cfg) != cudaSuccess) { cudaGetLastError(); c = 0; }
            fits[k] = c;
        }
    }
    int splits = 1;
    for (int k = 1; k < 4; k++)
        if (items <= fits[k] && a.capacity > (1 << (k - 1)) * kLdKeys) splits = 1 << k;
    SPT_CUDA(launch_dependent(kern, dim3(items * splits), dim3(kLdThreads), smem, dependent, splits, a, splits, groups));
    note_submit();
    return 0;
}

template <typename T, int NV>
int launch_rows(const LatentArgs& a, bool dependent) {
    const size_t smem = (size_t)4 * 32 * NV * sizeof(float);
    SPT_CUDA(launch_dependent(latent_rows_kernel<T, NV>, dim3(a.H, a.B * a.T), dim3(128), smem, dependent, 1, a));
    note_submit();
    return 0;
}

template <typename T>
int absorbed_t(const LatentArgs& a, bool dependent) {
    const int M = a.B * a.T;
    if (M > 65535) return fail("latent attention: %d tokens exceed one launch", M);
    {
        const dim3 grid(ceil_div(a.row, 128), a.H, M);
        SPT_CUDA(launch_dependent(latent_absorb_kernel<T>, grid, dim3(128), (size_t)(a.D + a.rot) * sizeof(float), dependent, 1, a));
        note_submit();
    }
    const int per = ceil_div(a.row, 32);
    int rc;
    if (per <= 4) rc = launch_rows<T, 4>(a, dependent);
    else if (per <= 8) rc = launch_rows<T, 8>(a, dependent);
    else if (per <= 20) rc = launch_rows<T, 20>(a, dependent);
    else if (per <= 40) rc = launch_rows<T, 40>(a, dependent);
    else return fail("latent attention: rows of %d values are larger than 1280", a.row);
    if (rc) return rc;
    SPT_CUDA(launch_dependent(latent_value_kernel<T>, dim3(ceil_div(a.ld_out, 8), M), dim3(256), 0, dependent, 1, a));
    note_submit();
    return 0;
}

}  // namespace

int latent_prep(const LatentArgs& a, bool dependent) {
    const dim3 grid(a.B * a.T), block(128);
    const int nq = ceil_div(a.q_rank, 256), nk = ceil_div(a.kv, 256);
    if (vec_sizes(a) && nq <= 8 && nk <= 4) {
        const dim3 rows(ceil_div(a.B * a.T, 4));
        if (nq <= 2 && nk <= 1) SPT_CUDA(launch_dependent(latent_prep_vec_kernel<2, 1>, rows, block, 0, dependent, 1, a));
        else if (nq <= 4 && nk <= 2) SPT_CUDA(launch_dependent(latent_prep_vec_kernel<4, 2>, rows, block, 0, dependent, 1, a));
        else SPT_CUDA(launch_dependent(latent_prep_vec_kernel<8, 4>, rows, block, 0, dependent, 1, a));
        note_submit();
        return 0;
    }
    if (a.dtype == BF16) SPT_CUDA(launch_dependent(latent_prep_kernel<__nv_bfloat16>, grid, block, 0, dependent, 1, a));
    else SPT_CUDA(launch_dependent(latent_prep_kernel<float>, grid, block, 0, dependent, 1, a));
    note_submit();
    return 0;
}

int latent_rope_q(const LatentArgs& a) {
    const long long work = (long long)a.B * a.T * a.H * (a.rope_dims / 2);
    if (work == 0) return 0;
    if (vec_sizes(a)) {
        latent_rope_q_vec_kernel<<<(unsigned)((work / 4 + 255) / 256), 256, 0, rt().stream>>>(a);
        SPT_LAUNCH_CHECK("latent_rope_q");
        return 0;
    }
    const unsigned grid = (unsigned)((work + 255) / 256);
    if (a.dtype == BF16) latent_rope_q_kernel<__nv_bfloat16><<<grid, 256, 0, rt().stream>>>(a);
    else latent_rope_q_kernel<float><<<grid, 256, 0, rt().stream>>>(a);
    SPT_LAUNCH_CHECK("latent_rope_q");
    return 0;
}

int latent_attention_absorbed(const LatentArgs& a, bool dependent) {
    return a.dtype == BF16 ? absorbed_t<__nv_bfloat16>(a, dependent) : absorbed_t<float>(a, dependent);
}

bool latent_decode_supported(const LatentArgs& a) {
    return a.dtype == BF16 && a.kv8 <= 512 && latent_decode_smem(a.row) <= 227 * 1024;
}

int latent_decode(const LatentArgs& a, bool dependent) {
    const int tiles = a.kv8 / 8;
    return tiles <= 32 ? launch_latent_decode<2>(a, dependent) : launch_latent_decode<4>(a, dependent);
}

}  // namespace spt
