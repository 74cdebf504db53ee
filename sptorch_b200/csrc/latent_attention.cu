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
    a.qabs[((size_t)m * a.H + h) * a.row + c] = v;
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
    const float* qp = a.qabs + ((size_t)mt * a.H + h) * a.row;
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
    float* out = a.olat + ((size_t)mt * a.H + h) * a.kv8;
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
    const float* ol = a.olat + ((size_t)m * a.H + h) * a.kv8;
    float s = 0.0f;
    for (int c = lane; c < a.kv; c += 32) s = fmaf((float)w[c], ol[c], s);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) {
        const float g = (float)static_cast<const T*>(a.in)[(size_t)m * a.ld_in + a.c_g + h];
        out[i] = (T)(s * sigmoid_exact(g));
    }
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
    if (a.dtype == BF16) SPT_CUDA(launch_dependent(latent_prep_kernel<__nv_bfloat16>, grid, block, 0, dependent, 1, a));
    else SPT_CUDA(launch_dependent(latent_prep_kernel<float>, grid, block, 0, dependent, 1, a));
    note_submit();
    return 0;
}

int latent_rope_q(const LatentArgs& a) {
    const long long work = (long long)a.B * a.T * a.H * (a.rope_dims / 2);
    if (work == 0) return 0;
    const unsigned grid = (unsigned)((work + 255) / 256);
    if (a.dtype == BF16) latent_rope_q_kernel<__nv_bfloat16><<<grid, 256, 0, rt().stream>>>(a);
    else latent_rope_q_kernel<float><<<grid, 256, 0, rt().stream>>>(a);
    SPT_LAUNCH_CHECK("latent_rope_q");
    return 0;
}

int latent_attention_absorbed(const LatentArgs& a, bool dependent) {
    return a.dtype == BF16 ? absorbed_t<__nv_bfloat16>(a, dependent) : absorbed_t<float>(a, dependent);
}

}  // namespace spt
