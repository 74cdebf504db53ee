// window_attention.cu -- softmax attention over cached keys and values, in the form a layer of a list-built model may ask for:
//   query head h reads key/value head h / (H / G);  score(i, j) = q_i . k_j * scale - slope_h (i - j);  position i sees the last
//   `window` positions up to i itself;  the concatenated heads are multiplied element by element with sigmoid(gate).
// q, k and v pass a short causal convolution over time on their way from the projection (every channel by itself; the last projected
// rows of a sequence are kept in a ring, slot = position % taps), q is then multiplied by a factor that depends on its position.
// A position keeps the row [keys of G heads | values of G heads], every head padded to eight elements with zeros.
//
// Three paths: prompts of bf16 models run the fused tcgen05 kernel (attention_fused.cu) behind window_prep; a few tokens of a bf16 model
// run window_decode, whose warps each own sixteen keys at a time on mma.sync; everything else (f32, head sizes the others do not take)
// runs the plain kernel.  Scores, softmax weights (in P V the sum of two bf16 numbers) and sums are f32 in all of them.
#include "layered.h"
#include "pdl.cuh"
#include <math.h>
#include <cooperative_groups.h>

namespace spt {

namespace {

// ---------------- convolution, position factor, cached rows ----------------
// the projected value of column `col` at token t of sequence b (t < 0: before this call's first token, at position pos0)
template <typename T>
__device__ __forceinline__ float projected(const WindowArgs& a, int b, int t, int pos0, int col) {
    if (t >= 0) return (float)static_cast<const T*>(a.in)[((size_t)b * a.T + t) * a.ld_in + col];
    const int p = pos0 + t;
    return p < 0 ? 0.0f : (float)static_cast<const T*>(a.ring)[((size_t)b * a.taps + p % a.taps) * a.ring_cols + col];
}
template <typename T>
__device__ __forceinline__ float convolved(const WindowArgs& a, int b, int t, int pos0, int col) {
    if (a.taps == 0) return projected<T>(a, b, t, pos0, col);
    float s = 0.0f;
    for (int j = 0; j < a.taps; j++) s = fmaf(a.conv[(size_t)j * a.ring_cols + col], projected<T>(a, b, t - a.taps + 1 + j, pos0, col), s);
    return s;
}

// One CTA per token, any sizes.
template <typename T>
__global__ void __launch_bounds__(128) window_prep_kernel(const WindowArgs a) {
    pdl_release();
    const int m = blockIdx.x, b = m / a.T, t = m - b * a.T;
    pdl_acquire();
    const int pos0 = a.pos_dev ? a.pos_dev[0] : a.first, pos = pos0 + t;
    const int nq = a.H * a.D8, nk = a.G * a.D8, n = nq + (a.own_kv ? a.row : 0);
    const float temp = a.temp ? a.temp[pos] : 1.0f;
    T* q = static_cast<T*>(a.q) + (size_t)m * nq;
    T* row = static_cast<T*>(a.rows) + (size_t)b * a.seq_stride + (size_t)pos * a.row;
    for (int i = threadIdx.x; i < n; i += 128) {
        const int e = i < nq ? i : i - nq, size8 = i < nq || e < nk ? a.D8 : a.V8, size = i < nq || e < nk ? a.D : a.V;
        const int first = i < nq ? a.c_q : e < nk ? a.c_k : a.c_v, o = i >= nq && e >= nk ? e - nk : e, h = o / size8, d = o - h * size8;
        float v = d < size ? convolved<T>(a, b, t, pos0, first + h * size + d) : 0.0f;
        if (i < nq) q[i] = (T)(v * temp);
        else row[e] = (T)v;
    }
}

__device__ __forceinline__ void unpack(uint4 raw, float (&f)[8]) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; i++) { const float2 v = bf16x2_to_float2(h[i]); f[2 * i] = v.x; f[2 * i + 1] = v.y; }
}
__device__ __forceinline__ void load_taps(const float* w, float (&f)[8]) {
    const float4 x = __ldg(reinterpret_cast<const float4*>(w)), y = __ldg(reinterpret_cast<const float4*>(w + 4));
    f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w; f[4] = y.x; f[5] = y.y; f[6] = y.z; f[7] = y.w;
}

constexpr int kPrepTokens = 16;

// bf16, head sizes multiples of eight: a thread takes eight channels of kPrepTokens consecutive tokens, the rows before the current one in
// registers.  Bytes per token and channel: 2 read (and the taps - 1 rows ahead of a run), 2 written.
template <int TAPS>
__global__ void __launch_bounds__(128) window_prep_vec_kernel(const WindowArgs a) {
    const int nq = a.H * a.D, c = (blockIdx.x * 128 + threadIdx.x) * 8, cols = nq + (a.own_kv ? a.row : 0);
    pdl_release();
    pdl_acquire();
    if (c >= cols) return;
    const int b = blockIdx.z, t0 = blockIdx.y * kPrepTokens, t1 = min(a.T, t0 + kPrepTokens);
    const int pos0 = a.pos_dev ? a.pos_dev[0] : a.first;
    float w[TAPS][8], u[TAPS][8];                               // u[j]: the row j - (TAPS - 1) tokens from the current one
#pragma unroll
    for (int j = 0; j < TAPS; j++) load_taps(a.conv + (size_t)j * a.ring_cols + c, w[j]);
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + (size_t)b * a.T * a.ld_in + c;
#pragma unroll
    for (int j = 0; j < TAPS - 1; j++) {
        const int t = t0 - (TAPS - 1) + j, p = pos0 + t;
        uint4 raw = make_uint4(0, 0, 0, 0);
        if (t >= 0) raw = *reinterpret_cast<const uint4*>(in + (size_t)t * a.ld_in);
        else if (p >= 0) raw = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.ring) + ((size_t)b * TAPS + p % TAPS) * a.ring_cols + c);
        unpack(raw, u[j + 1]);
    }
    const bool is_q = c < nq;
    __nv_bfloat16* dst = is_q ? static_cast<__nv_bfloat16*>(a.q) + (size_t)b * a.T * nq + c : static_cast<__nv_bfloat16*>(a.rows) + (size_t)b * a.seq_stride + (size_t)pos0 * a.row + (c - nq);
    const int ld = is_q ? nq : a.row;
#pragma unroll 4
    for (int t = t0; t < t1; t++) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; j++)
#pragma unroll
            for (int i = 0; i < 8; i++) u[j][i] = u[j + 1][i];
        unpack(*reinterpret_cast<const uint4*>(in + (size_t)t * a.ld_in), u[TAPS - 1]);
        const float f = is_q && a.temp ? __ldg(a.temp + pos0 + t) : 1.0f;
        uint4 o;
        __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int i = 0; i < 8; i += 2) {
            float x = 0.0f, y = 0.0f;
#pragma unroll
            for (int j = 0; j < TAPS; j++) { x = fmaf(w[j][i], u[j][i], x); y = fmaf(w[j][i + 1], u[j][i + 1], y); }
            oh[i / 2] = __floats2bfloat162_rn(x * f, y * f);
        }
        *reinterpret_cast<uint4*>(dst + (size_t)t * ld) = o;
    }
}

// The projected rows the next call's convolutions look back at: the last taps - 1 tokens of this one, each in its slot of the ring.  A
// launch behind the convolutions, because a slot may still hold a row they read.
template <typename T>
__global__ void __launch_bounds__(128) window_tail_kernel(const WindowArgs a, int keep) {
    pdl_release();
    const int b = blockIdx.x / keep, t = a.T - keep + blockIdx.x % keep;
    pdl_acquire();
    const int pos = (a.pos_dev ? a.pos_dev[0] : a.first) + t;
    const T* src = static_cast<const T*>(a.in) + ((size_t)b * a.T + t) * a.ld_in;
    T* dst = static_cast<T*>(a.ring) + ((size_t)b * a.taps + pos % a.taps) * a.ring_cols;
    for (int i = threadIdx.x; i < a.ring_cols; i += 128) dst[i] = src[i];
}

// ---------------- any sizes: plain kernel ----------------
__device__ __forceinline__ float sigmoid_exact(float z) { return 1.0f / (1.0f + expf(-z)); }

// One CTA per (token, head): four warps share the visible keys, each with a running (maximum, sum, weighted values); merged at the end in
// warp order.  NV: values per lane (32 NV >= V).
template <typename T, int NV>
__global__ void __launch_bounds__(128) window_plain_kernel(const WindowArgs a) {
    extern __shared__ float dyn_f[];                     // [D8] query, then [4][32 * NV] weighted values
    __shared__ float m_sh[4], l_sh[4];
    pdl_release();
    const int mt = blockIdx.x / a.H, h = blockIdx.x - mt * a.H, b = mt / a.T, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* qs = dyn_f;
    float* acc_sh = dyn_f + a.D8;
    pdl_acquire();
    const int pos = (a.pos_dev ? a.pos_dev[0] : a.first) + (mt - b * a.T), lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const int g = h / (a.H / a.G);
    const T* krow = static_cast<const T*>(a.rows) + (size_t)b * a.seq_stride + (size_t)g * a.D8;
    const T* vrow = static_cast<const T*>(a.rows) + (size_t)b * a.seq_stride + (size_t)a.G * a.D8 + (size_t)g * a.V8;
    for (int i = threadIdx.x; i < a.D; i += 128) qs[i] = (float)static_cast<const T*>(a.q)[((size_t)mt * a.H + h) * a.D8 + i];
    __syncthreads();
    const float slope = a.slopes ? a.slopes[h] : 0.0f;
    float o[NV], mx = -INFINITY, l = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; i++) o[i] = 0.0f;
    for (int p = lo + warp; p <= pos; p += 4) {
        const T* k = krow + (size_t)p * a.row;
        const T* v = vrow + (size_t)p * a.row;
        float s = 0.0f;
        for (int i = lane; i < a.D; i += 32) s = fmaf(qs[i], (float)k[i], s);
#pragma unroll
        for (int w = 16; w > 0; w >>= 1) s += __shfl_xor_sync(0xffffffffu, s, w);
        s = s * a.scale - slope * (float)(pos - p);
        const float mn = fmaxf(mx, s), corr = expf(mx - mn), e = expf(s - mn);
        l = l * corr + e;
#pragma unroll
        for (int i = 0; i < NV; i++) { const int c = i * 32 + lane; o[i] = fmaf(o[i], corr, c < a.V ? e * (float)v[c] : 0.0f); }
        mx = mn;
    }
    if (lane == 0) { m_sh[warp] = mx; l_sh[warp] = l; }
#pragma unroll
    for (int i = 0; i < NV; i++) acc_sh[warp * 32 * NV + i * 32 + lane] = o[i];
    __syncthreads();
    const float tm = fmaxf(fmaxf(m_sh[0], m_sh[1]), fmaxf(m_sh[2], m_sh[3]));
    float tl = 0.0f, f[4];
#pragma unroll
    for (int w = 0; w < 4; w++) { f[w] = m_sh[w] == -INFINITY ? 0.0f : expf(m_sh[w] - tm); tl += l_sh[w] * f[w]; }
    const float inv = 1.0f / tl;
    for (int c = threadIdx.x; c < a.V; c += 128) {
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < 4; w++) v = fmaf(acc_sh[w * 32 * NV + c], f[w], v);
        v *= inv;
        if (a.gate) v *= sigmoid_exact((float)static_cast<const T*>(a.gate)[(size_t)mt * a.ld_out + h * a.V + c]);
        static_cast<T*>(a.out)[(size_t)mt * a.ld_out + h * a.V + c] = (T)v;
    }
}

// ---------------- few tokens, bf16, on the tensor cores ----------------
// A cluster of `splits` CTAs owns one token and up to sixteen query heads of one key/value head.  Every warp of the cluster walks the
// visible keys sixteen at a time, all by itself: keys and values go from global memory straight into mma.sync fragments (a sum over k
// does not care about the order of k, and a column of the output may stand for any value dimension, so 16-byte loads of consecutive
// elements serve as they are), with its own running (maximum, sum, output).  The warps' parts meet in shared memory, the CTAs' through
// distributed shared memory, in a fixed order.  HBM bytes: (D + V) * 2 per visible position and key/value head, read once.
// FRESH (one token per sequence): the CTA convolves its heads' query, key and value itself and writes the new cached row and the ring.
//   S: k slot (lane l = 4 g + t; elements 8 t .. 8 t + 7 of a 32-element slice) as in linear_few_rows.cu;  scores: row = query head, column = key
//   P V: k = keys, n-tile j, column g = value dimension 64 (j / 8) + 8 g + j % 8
// NS: 32-element slices of D; NB: 64-element blocks of V.
__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = bf16x2_to_float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h); lo = *reinterpret_cast<const uint32_t*>(&l);
}

constexpr int kWdHeads = 16;
__host__ __device__ constexpr int wd_q_pitch(int ns) { return ns * 32 + 8; }
__host__ __device__ constexpr int wd_o_pitch(int nb) { return nb * 64 + 4; }
template <int NS, int NB>
constexpr size_t wd_smem(int warps, int heads) {
    return (size_t)kWdHeads * wd_q_pitch(NS) * 2 + (size_t)(NS * 32 + NB * 64) * 2 + (size_t)warps * kWdHeads * 8 + kWdHeads * 4 + (size_t)warps * heads * wd_o_pitch(NB) * 4;
}

template <int NS, int NB, bool FRESH, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) window_decode_kernel(const WindowArgs a, int splits, int hgroups) {
    extern __shared__ __align__(16) uint8_t raw[];
    constexpr int QP = wd_q_pitch(NS), OP = wd_o_pitch(NB);
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(raw);                  // [16][QP]
    __nv_bfloat16* kf = qs + kWdHeads * QP;                                     // the new key and value (FRESH)
    __nv_bfloat16* vf = kf + NS * 32;
    float* m_s = reinterpret_cast<float*>(vf + NB * 64);                        // [WARPS][16]
    float* l_s = m_s + WARPS * kWdHeads;
    float* f0_s = l_s + WARPS * kWdHeads;                                       // [16]: warp 0's factor
    float* o_s = f0_s + kWdHeads;                                               // [WARPS][heads][OP]
    pdl_release();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int rank = blockIdx.x % splits, item = blockIdx.x / splits, R = a.H / a.G;
    const int hg = item % hgroups, gg = item / hgroups % a.G, mt = item / hgroups / a.G, b = mt / a.T;
    const int h0 = gg * R + hg * kWdHeads, heads = min(kWdHeads, R - hg * kWdHeads), heads_max = min(kWdHeads, R);
    const int pos0 = a.pos_dev ? a.pos_dev[0] : a.first, pos = pos0 + (mt - b * a.T), lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const __nv_bfloat16* krow = static_cast<const __nv_bfloat16*>(a.rows) + (size_t)b * a.seq_stride + (size_t)gg * a.D;
    const __nv_bfloat16* vrow = static_cast<const __nv_bfloat16*>(a.rows) + (size_t)b * a.seq_stride + (size_t)a.G * a.D + (size_t)gg * a.V;
    const bool fresh_kv = FRESH && a.own_kv;                 // the row of position `pos` is not in the cache yet
    uint4 kr[2][NS], vr[4][NB];
    const uint4 zero4 = make_uint4(0, 0, 0, 0);
    // keys k0 + g and k0 + 8 + g; values of keys k0 + 2t, 2t + 1, 2t + 8, 2t + 9.  Positions past `last` are not read.
    auto fetch_keys = [&](int k0, int last) {
#pragma unroll
        for (int n = 0; n < 2; n++) {
            const int p = k0 + 8 * n + g;
#pragma unroll
            for (int s = 0; s < NS; s++) kr[n][s] = p <= last && 32 * s + 8 * t < a.D ? *reinterpret_cast<const uint4*>(krow + (size_t)p * a.row + 32 * s + 8 * t) : zero4;
        }
    };
    auto fetch_values = [&](int k0, int last) {
#pragma unroll
        for (int n = 0; n < 4; n++) {
            const int p = k0 + 2 * t + (n & 1) + 8 * (n >> 1);
#pragma unroll
            for (int s = 0; s < NB; s++) vr[n][s] = p <= last && 64 * s + 8 * g < a.V ? *reinterpret_cast<const uint4*>(vrow + (size_t)p * a.row + 64 * s + 8 * g) : zero4;
        }
    };
    const int step = splits * WARPS * 16, first = lo + (rank * WARPS + warp) * 16;
    const int last = fresh_kv ? pos - 1 : pos;               // what the cache holds
    // rows before this step's tokens were written by earlier steps: they may be requested before the kernels ahead are done
    const bool early = first + 15 < pos0;
    if (early && first <= pos) { fetch_keys(first, last); fetch_values(first, last); }
    if constexpr (FRESH) {
        // this CTA's share of the convolutions, eight channels per thread: heads' queries, then (own_kv) the key and the value.  Everything
        // but the newest projected row is there already, so only its product is left for after the wait.
        const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + (size_t)mt * a.ld_in;
        __nv_bfloat16* ring = a.taps ? static_cast<__nv_bfloat16*>(a.ring) + (size_t)b * a.taps * a.ring_cols : nullptr;
        const int nq = heads * a.D, nk = fresh_kv ? a.D : 0, nv = fresh_kv ? a.V : 0;
        bool acquired = false;
        for (int i = tid * 8; i < nq + nk + nv || !acquired; i += WARPS * 256) {
            const bool live = i < nq + nk + nv, is_q = i < nq;
            const int col = is_q ? a.c_q + h0 * a.D + i : i < nq + nk ? a.c_k + gg * a.D + (i - nq) : a.c_v + gg * a.V + (i - nq - nk);
            float sum[8] = {0, 0, 0, 0, 0, 0, 0, 0}, w[8] = {1, 1, 1, 1, 1, 1, 1, 1}, u[8];
            if (live && a.taps) {
#pragma unroll 4
                for (int j = 1; j < a.taps; j++)
                    if (pos - j >= 0) {
                        load_taps(a.conv + (size_t)(a.taps - 1 - j) * a.ring_cols + col, w);
                        unpack(*reinterpret_cast<const uint4*>(ring + (size_t)((pos - j) % a.taps) * a.ring_cols + col), u);
#pragma unroll
                        for (int e = 0; e < 8; e++) sum[e] = fmaf(w[e], u[e], sum[e]);
                    }
                load_taps(a.conv + (size_t)(a.taps - 1) * a.ring_cols + col, w);
            }
            const float factor = is_q && a.temp ? a.temp[pos] : 1.0f;
            if (!acquired) { pdl_acquire(); acquired = true; }
            if (!live) break;
            const uint4 now = *reinterpret_cast<const uint4*>(in + col);
            unpack(now, u);
            uint4 o;
            __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
            for (int e = 0; e < 8; e += 2) oh[e / 2] = __floats2bfloat162_rn(fmaf(w[e], u[e], sum[e]) * factor, fmaf(w[e + 1], u[e + 1], sum[e + 1]) * factor);
            // no CTA reads this slot of the ring in this step
            if (a.taps && rank == 0 && (is_q || hg == 0)) *reinterpret_cast<uint4*>(ring + (size_t)(pos % a.taps) * a.ring_cols + col) = now;
            if (is_q) { const int r = i / a.D; *reinterpret_cast<uint4*>(qs + r * QP + i - r * a.D) = o; }
            else {
                *reinterpret_cast<uint4*>(i < nq + nk ? kf + (i - nq) : vf + (i - nq - nk)) = o;
                if (rank == 0 && hg == 0)
                    *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.rows) + (size_t)b * a.seq_stride + (size_t)pos * a.row + (i < nq + nk ? gg * a.D + (i - nq) : a.G * a.D + gg * a.V + (i - nq - nk))) = o;
            }
        }
        if (!early && first <= pos) { fetch_keys(first, last); fetch_values(first, last); }
        // the rest of Q: missing heads and columns
        for (int i = tid; i < kWdHeads * QP; i += WARPS * 32) { const int r = i / QP; if (r >= heads || i - r * QP >= a.D) qs[i] = __float2bfloat16_rn(0.0f); }
    } else {
        pdl_acquire();
        if (!early && first <= pos) { fetch_keys(first, last); fetch_values(first, last); }
        for (int i = tid; i < kWdHeads * (QP / 8); i += WARPS * 32) {
            const int r = i / (QP / 8), c = (i - r * (QP / 8)) * 8;
            *reinterpret_cast<uint4*>(qs + r * QP + c) = r < heads && c < a.D ? *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q) + ((size_t)mt * a.H + h0 + r) * a.D + c) : zero4;
        }
    }
    __syncthreads();
    float acc[8 * NB][4];
#pragma unroll
    for (int j = 0; j < 8 * NB; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) acc[j][e] = 0.0f;
    const float kLog2e = 1.4426950408889634f, scale = a.scale * kLog2e;
    const float sl0 = a.slopes && g < heads ? a.slopes[h0 + g] * kLog2e : 0.0f, sl1 = a.slopes && g + 8 < heads ? a.slopes[h0 + g + 8] * kLog2e : 0.0f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    for (int k0 = first; k0 <= pos; k0 += step) {
        if (fresh_kv && pos - k0 < 16) {                     // the newest position takes its row from shared memory
            const int d = pos - k0;
#pragma unroll
            for (int n = 0; n < 2; n++)
                if (8 * n + g == d) {
#pragma unroll
                    for (int s = 0; s < NS; s++) if (32 * s + 8 * t < a.D) kr[n][s] = *reinterpret_cast<const uint4*>(kf + 32 * s + 8 * t);
                }
#pragma unroll
            for (int n = 0; n < 4; n++)
                if (2 * t + (n & 1) + 8 * (n >> 1) == d) {
#pragma unroll
                    for (int s = 0; s < NB; s++) if (64 * s + 8 * g < a.V) vr[n][s] = *reinterpret_cast<const uint4*>(vf + 64 * s + 8 * g);
                }
        }
        float s[2][4] = {{0, 0, 0, 0}, {0, 0, 0, 0}};
#pragma unroll
        for (int i = 0; i < NS; i++) {
            const uint4 x = *reinterpret_cast<const uint4*>(qs + g * QP + 32 * i + 8 * t), y = *reinterpret_cast<const uint4*>(qs + (g + 8) * QP + 32 * i + 8 * t);
#pragma unroll
            for (int n = 0; n < 2; n++) {
                mma_bf16(s[n], x.x, y.x, x.y, y.y, kr[n][i].x, kr[n][i].y);
                mma_bf16(s[n], x.z, y.z, x.w, y.w, kr[n][i].z, kr[n][i].w);
            }
        }
        if (k0 + step <= pos) fetch_keys(k0 + step, last);         // in flight while the softmax and P V run
        // scores of heads g (entries 0, 1) and g + 8 (2, 3), keys k0 + 8 n + 2 t + {0, 1}
        float mx0 = m0, mx1 = m1;
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int back = pos - (k0 + 8 * n + 2 * t + e);
                const bool seen = back >= 0;                 // the window's far edge is where the walk begins
                s[n][e] = seen ? fmaf(s[n][e], scale, -sl0 * (float)back) : -INFINITY;
                s[n][2 + e] = seen ? fmaf(s[n][2 + e], scale, -sl1 * (float)back) : -INFINITY;
                mx0 = fmaxf(mx0, s[n][e]); mx1 = fmaxf(mx1, s[n][2 + e]);
            }
#pragma unroll
        for (int o = 1; o < 4; o <<= 1) { mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, o)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, o)); }
        // key k0 is visible to every head: the maxima are finite from here on
        const float c0 = ex2(m0 - mx0), c1 = ex2(m1 - mx1);
        m0 = mx0; m1 = mx1;
        uint32_t ph[4], pl[4];
        l0 *= c0; l1 *= c1;
#pragma unroll
        for (int n = 0; n < 2; n++) {
            const float e0 = ex2(s[n][0] - m0), e1 = ex2(s[n][1] - m0), e2 = ex2(s[n][2] - m1), e3 = ex2(s[n][3] - m1);
            l0 += e0 + e1; l1 += e2 + e3;
            split2(e0, e1, ph[2 * n], pl[2 * n]); split2(e2, e3, ph[2 * n + 1], pl[2 * n + 1]);
        }
#pragma unroll
        for (int j = 0; j < 8 * NB; j++) { acc[j][0] *= c0; acc[j][1] *= c0; acc[j][2] *= c1; acc[j][3] *= c1; }
#pragma unroll
        for (int sb = 0; sb < NB; sb++) {
            const uint32_t* v0 = reinterpret_cast<const uint32_t*>(&vr[0][sb]);
            const uint32_t* v1 = reinterpret_cast<const uint32_t*>(&vr[1][sb]);
            const uint32_t* v2 = reinterpret_cast<const uint32_t*>(&vr[2][sb]);
            const uint32_t* v3 = reinterpret_cast<const uint32_t*>(&vr[3][sb]);
#pragma unroll
            for (int j = 0; j < 8; j++) {
                const uint32_t sel = j & 1 ? 0x7632 : 0x5410;
                const uint32_t b0 = __byte_perm(v0[j / 2], v1[j / 2], sel), b1 = __byte_perm(v2[j / 2], v3[j / 2], sel);
                mma_bf16(acc[8 * sb + j], ph[0], ph[1], ph[2], ph[3], b0, b1);
                mma_bf16(acc[8 * sb + j], pl[0], pl[1], pl[2], pl[3], b0, b1);
            }
        }
        if (k0 + step <= pos) fetch_values(k0 + step, last);
    }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) { l0 += __shfl_xor_sync(0xffffffffu, l0, o); l1 += __shfl_xor_sync(0xffffffffu, l1, o); }
    if (t == 0) {
        m_s[warp * kWdHeads + g] = m0; m_s[warp * kWdHeads + g + 8] = m1;
        l_s[warp * kWdHeads + g] = l0; l_s[warp * kWdHeads + g + 8] = l1;
    }
    // accumulator column 2 t + e of n-tile j is value dimension 64 (j / 8) + 8 (2 t + e) + j % 8
#pragma unroll
    for (int r = 0; r < 2; r++)
        if (g + 8 * r < heads_max) {
            float* dst = o_s + ((size_t)warp * heads_max + g + 8 * r) * OP;
#pragma unroll
            for (int sb = 0; sb < NB; sb++)
#pragma unroll
                for (int e = 0; e < 2; e++)
#pragma unroll
                    for (int q = 0; q < 8; q += 4)
                        *reinterpret_cast<float4*>(dst + 64 * sb + 8 * (2 * t + e) + q) =
                            make_float4(acc[8 * sb + q][2 * r + e], acc[8 * sb + q + 1][2 * r + e], acc[8 * sb + q + 2][2 * r + e], acc[8 * sb + q + 3][2 * r + e]);
        }
    namespace cg = cooperative_groups;
    cg::cluster_group cluster = cg::this_cluster();
    __syncthreads();
    // the CTA's own warps first: every warp's factor against the CTA's maximum, then the sums, which land in warp 0's slots
    if (tid < kWdHeads) {
        float tm = -INFINITY, tl = 0.0f;
#pragma unroll
        for (int w = 0; w < WARPS; w++) tm = fmaxf(tm, m_s[w * kWdHeads + tid]);
#pragma unroll
        for (int w = 0; w < WARPS; w++) {
            const float x = m_s[w * kWdHeads + tid], f = x == -INFINITY ? 0.0f : ex2(x - tm);
            tl = fmaf(l_s[w * kWdHeads + tid], f, tl);
            if (w > 0) m_s[w * kWdHeads + tid] = f; else f0_s[tid] = f;
        }
        m_s[tid] = tm; l_s[tid] = tl;
    }
    __syncthreads();
    for (int i = tid * 4; i < heads * a.V; i += WARPS * 128) {
        const int r = i / a.V, c = i - r * a.V;
        float4 v = make_float4(0, 0, 0, 0);
#pragma unroll
        for (int w = 0; w < WARPS; w++) {
            const float f = w > 0 ? m_s[w * kWdHeads + r] : f0_s[r];
            const float4 x = *reinterpret_cast<const float4*>(o_s + ((size_t)w * heads_max + r) * OP + c);
            v.x = fmaf(x.x, f, v.x); v.y = fmaf(x.y, f, v.y); v.z = fmaf(x.z, f, v.z); v.w = fmaf(x.w, f, v.w);
        }
        *reinterpret_cast<float4*>(o_s + (size_t)r * OP + c) = v;              // this thread was the only reader of its columns
    }
    if (splits > 1) cluster.sync(); else __syncthreads();
    const int quads = heads * a.V / 4, per = (quads + splits - 1) / splits, i1 = min(quads, (rank + 1) * per);
    for (int i = rank * per + tid; i < i1; i += WARPS * 32) {
        const int r = i * 4 / a.V, c = i * 4 - r * a.V;
        float tm = -INFINITY, tl = 0.0f, ms[8];
        float4 v = make_float4(0, 0, 0, 0);
#pragma unroll
        for (int s = 0; s < 8; s++) { ms[s] = s < splits ? (splits > 1 ? cluster.map_shared_rank(m_s, s) : m_s)[r] : -INFINITY; tm = fmaxf(tm, ms[s]); }
#pragma unroll
        for (int s = 0; s < 8; s++)
            if (s < splits) {
                const float f = ms[s] == -INFINITY ? 0.0f : ex2(ms[s] - tm);
                const float4 x = *reinterpret_cast<const float4*>((splits > 1 ? cluster.map_shared_rank(o_s, s) : o_s) + (size_t)r * OP + c);
                tl = fmaf((splits > 1 ? cluster.map_shared_rank(l_s, s) : l_s)[r], f, tl);
                v.x = fmaf(x.x, f, v.x); v.y = fmaf(x.y, f, v.y); v.z = fmaf(x.z, f, v.z); v.w = fmaf(x.w, f, v.w);
            }
        const float inv = 1.0f / tl;
        const size_t at = (size_t)mt * a.ld_out + (size_t)(h0 + r) * a.V + c;
        float y[4] = {v.x * inv, v.y * inv, v.z * inv, v.w * inv};
        if (a.gate) {
            const uint2 graw = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(a.gate) + at);
            const float2 g0 = bf16x2_to_float2(*reinterpret_cast<const __nv_bfloat162*>(&graw.x)), g1 = bf16x2_to_float2(*reinterpret_cast<const __nv_bfloat162*>(&graw.y));
            y[0] *= 1.0f / (1.0f + __expf(-g0.x)); y[1] *= 1.0f / (1.0f + __expf(-g0.y)); y[2] *= 1.0f / (1.0f + __expf(-g1.x)); y[3] *= 1.0f / (1.0f + __expf(-g1.y));
        }
        uint2 o;
        *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(y[0], y[1]);
        *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(y[2], y[3]);
        *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(a.out) + at) = o;
    }
    if (splits > 1) cluster.sync();                        // no CTA leaves while its shared memory may still be read
}

template <int NS, int NB, bool FRESH, int WARPS>
int launch_decode(const WindowArgs& a, bool dependent, int splits) {
    auto kern = window_decode_kernel<NS, NB, FRESH, WARPS>;
    const int R = a.H / a.G, hgroups = ceil_div(R, kWdHeads);
    const size_t smem = wd_smem<NS, NB>(WARPS, R < kWdHeads ? R : kWdHeads);
    static size_t granted = 48 * 1024;
    if (smem > granted) { SPT_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); granted = smem; }
    SPT_CUDA(launch_dependent(kern, dim3(a.B * a.T * a.G * hgroups * splits), dim3(WARPS * 32), smem, dependent, splits, a, splits, hgroups));
    note_submit();
    return 0;
}

template <int NS, int NB>
int choose_decode(const WindowArgs& a, bool fresh, bool dependent) {
    // Wide CTAs split over a cluster while all of them fit the SMs at once, narrow ones (several per SM) when the items fill the GPU
    const int items = a.B * a.T * a.G * ceil_div(a.H / a.G, kWdHeads);
    const int span = a.window > 0 && a.window < a.capacity ? a.window : a.capacity;
    if (items * 2 > rt().sm_count || span <= 64)
        return fresh ? launch_decode<NS, NB, true, 4>(a, dependent, 1) : launch_decode<NS, NB, false, 4>(a, dependent, 1);
    int splits = 1;
    while (splits < 8 && items * splits * 2 <= rt().sm_count && span > splits * 128) splits *= 2;
    return fresh ? launch_decode<NS, NB, true, 8>(a, dependent, splits) : launch_decode<NS, NB, false, 8>(a, dependent, splits);
}

template <typename T, int NV>
int launch_plain(const WindowArgs& a, bool dependent) {
    auto kern = window_plain_kernel<T, NV>;
    const size_t smem = ((size_t)a.D8 + 4 * 32 * NV) * sizeof(float);
    const long long ctas = (long long)a.B * a.T * a.H;
    if (ctas > INT32_MAX) return fail("window attention: %lld (token, head) pairs exceed one launch", ctas);
    SPT_CUDA(launch_dependent(kern, dim3((unsigned)ctas), dim3(128), smem, dependent, 1, a));
    note_submit();
    return 0;
}

template <typename T>
int plain_t(const WindowArgs& a, bool dependent) {
    if (a.V <= 64) return launch_plain<T, 2>(a, dependent);
    if (a.V <= 128) return launch_plain<T, 4>(a, dependent);
    if (a.V <= 256) return launch_plain<T, 8>(a, dependent);
    if (a.V <= kWindowMaxHead) return launch_plain<T, 32>(a, dependent);
    return fail("window attention: values of %d are larger than %d", a.V, kWindowMaxHead);
}

bool vectors(const WindowArgs& a) { return a.dtype == BF16 && a.D % 8 == 0 && a.V % 8 == 0 && a.c_q == 0 && (!a.own_kv || (a.c_k == a.H * a.D && a.c_v == a.c_k + a.G * a.D)); }

}  // namespace

// projections -> convolved queries (times the position factor) and cached rows, then the ring
int window_prep(const WindowArgs& a, bool dependent) {
    const int M = a.B * a.T;
    if (vectors(a) && a.taps >= 1 && a.taps <= 4 && a.B <= 65535 && ceil_div(a.T, kPrepTokens) <= 65535) {
        const dim3 grid(ceil_div(a.H * a.D + (a.own_kv ? a.row : 0), 1024), ceil_div(a.T, kPrepTokens), a.B), block(128);
        if (a.taps == 1) SPT_CUDA(launch_dependent(window_prep_vec_kernel<1>, grid, block, 0, dependent, 1, a));
        else if (a.taps == 2) SPT_CUDA(launch_dependent(window_prep_vec_kernel<2>, grid, block, 0, dependent, 1, a));
        else if (a.taps == 3) SPT_CUDA(launch_dependent(window_prep_vec_kernel<3>, grid, block, 0, dependent, 1, a));
        else SPT_CUDA(launch_dependent(window_prep_vec_kernel<4>, grid, block, 0, dependent, 1, a));
    } else if (a.dtype == BF16) SPT_CUDA(launch_dependent(window_prep_kernel<__nv_bfloat16>, dim3(M), dim3(128), 0, dependent, 1, a));
    else SPT_CUDA(launch_dependent(window_prep_kernel<float>, dim3(M), dim3(128), 0, dependent, 1, a));
    note_submit();
    const int keep = a.T < a.taps - 1 ? a.T : a.taps - 1;
    if (!a.ring || keep <= 0) return 0;
    if (a.dtype == BF16) SPT_CUDA(launch_dependent(window_tail_kernel<__nv_bfloat16>, dim3(a.B * keep), dim3(128), 0, dependent, 1, a, keep));
    else SPT_CUDA(launch_dependent(window_tail_kernel<float>, dim3(a.B * keep), dim3(128), 0, dependent, 1, a, keep));
    note_submit();
    return 0;
}

int window_plain(const WindowArgs& a, bool dependent) { return a.dtype == BF16 ? plain_t<__nv_bfloat16>(a, dependent) : plain_t<float>(a, dependent); }

bool window_decode_supported(const WindowArgs& a) { return vectors(a) && a.D <= 128 && a.V <= 128 && (a.taps == 0 || a.ring); }

int window_decode(const WindowArgs& a, bool fresh, bool dependent) {
    if (a.D <= 64) return a.V <= 64 ? choose_decode<2, 1>(a, fresh, dependent) : choose_decode<2, 2>(a, fresh, dependent);
    return a.V <= 64 ? choose_decode<4, 1>(a, fresh, dependent) : choose_decode<4, 2>(a, fresh, dependent);
}

}  // namespace spt
