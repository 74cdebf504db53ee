// layered.cu -- driver of the models built from a list of layers.  Each layer has its own mixer (gated linear attention, latent
// attention, window attention), sizes and optional feed-forward.  Two ways of joining the residual stream (sptorch_layered_options):
//   post-norm:  x <- x + rms(mixer(x)) w1;   x <- x + rms(mlp(x)) w2
//   parallel:   h = rms(x) w1;   x <- x + mixer(h) + mlp(h);   and, with a per-layer token input e,
//               x <- x + rms(proj (gelu(gate x) e)) ws
// and logits = head (rms(x) wf).  The residual stream x is f32; the sublayers read a copy of it in the model dtype (xb), which the kernel that updates x writes beside
// it.  Launches of a prompt (bf16), per layer:
//   gated linear attention: one GEMM for q, k, v, gate and decay latent | chunk kernels (gla.cu) | W_o | post-norm
//   latent attention: one GEMM for query latent, key/value latent and head gates | latent norms and rotation | W_uq | rotation of q |
//                     keys and values of every position from the latents (one GEMM) | fused attention | W_o | post-norm
//   feed-forward: W_up (+bias) | W_gate (+bias, SwiGLU product) | W_down (+bias) | post-norm
//   parallel block with window attention: one GEMM for q, k, v, gate of the heads and W_up | W_gate (activation, product with up in place) |
//                     convolutions, cached rows | ring | fused attention (gates in place) | one GEMM for W_o and W_down (+ f32 residual) |
//                     side: bf16 copy of x | gate (gelu, product with e in place) | proj | post-norm together with the next layer's norm
// A few tokens (a decode step, a short portion of a prompt) take the weight-streaming projections, the token-by-token recurrence and
// attention over the cached latents themselves; all of these are programmatic dependents of one another, and with one or two rows the
// projection behind a sublayer does the post-norm on the way.
// f32 models run every product as f32 multiply-adds (MM_F32), the recurrence token by token and the latent attention unexpanded.
#include "layered.h"
#include "pdl.cuh"
#include <cmath>
#include <cstdio>
#include <cstring>
#include <map>

namespace spt {

bool attention_latent_supported(int D, int rot, int V, int kv_off, long long ld_q, long long ld_kv, int row);
int attention_latent(const void* q, long long ld_q, const void* kn, const void* v, long long ld_kv, const void* kr, long long row, long long seq_stride,
                     void* out, long long ld_out, const void* gate, long long ld_gate, int B, int T, int n, int H, int D, int rot, int V, int first, float scale);
bool attention_window_supported(int D, int V, int row, long long ld_out);
int attention_window(const void* q, const void* rows, int row, long long seq_stride, void* out, long long ld_out, const void* gate, int B, int T, int n, int H, int G,
                     int D, int V, int first, int window, const float* slopes, float scale);

namespace {

// x = embed[id] * scale in f32 and in the model dtype, and the token's row of the side table (side_ld values, 0: none); an id outside the
// vocabulary gives zero rows and raises the status word
template <typename T>
__global__ void __launch_bounds__(128) embed_rows_kernel(const T* __restrict__ table, const int* __restrict__ ids, float* __restrict__ x, T* __restrict__ xb, int vocab,
                                                         int ld, float scale, const T* __restrict__ side_table, T* __restrict__ side, int side_ld, uint32_t* status) {
    pdl_release();
    pdl_acquire();
    const int m = blockIdx.x, id = ids[m];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0) atomicOr(status, 0x100u);
    const T* src = table + (size_t)(ok ? id : 0) * ld;
    for (int i = threadIdx.x; i < ld; i += 128) {
        const float v = ok ? (float)src[i] * scale : 0.0f;
        x[(size_t)m * ld + i] = v;
        xb[(size_t)m * ld + i] = (T)v;
    }
    const T* sr = side_table + (size_t)(ok ? id : 0) * side_ld;
    for (int i = threadIdx.x; i < side_ld; i += 128) side[(size_t)m * side_ld + i] = ok ? sr[i] : (T)0.0f;
}

__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; i++) { const float2 f = bf16x2_to_float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; i++) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
}

template <int THREADS>
__device__ __forceinline__ float row_sum(float v, float* sh) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if (THREADS == 32) return v;
    __syncthreads();
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.0f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; w++) s += sh[w];
    return s;
}

// One CTA per row, NV groups of eight elements per thread in registers.  HBM bytes per element: y + 4 (x in) + 4 (x out) + xb.
template <typename T, int THREADS, int NV>
__global__ void __launch_bounds__(THREADS) post_norm_kernel(const float* x, const T* __restrict__ y, const float* __restrict__ w, const float* __restrict__ w2,
                                                            float* x_out, T* __restrict__ xb, int dim, int ld, float eps) {
    __shared__ float sh[THREADS / 32];
    pdl_release();
    pdl_acquire();
    const size_t base = (size_t)blockIdx.x * ld;
    float xv[NV][8], yv[NV][8];
    float sq = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = (i * THREADS + (int)threadIdx.x) * 8;
        if (c < ld) {
            load8(x + base + c, xv[i]);
            if (y) {
                load8(y + base + c, yv[i]);
#pragma unroll
                for (int j = 0; j < 8; j++) sq = fmaf(yv[i][j], yv[i][j], sq);
            }
        }
    }
    if (y) {
        const float inv = 1.0f / sqrtf(row_sum<THREADS>(sq, sh) / (float)dim + eps);
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int c = (i * THREADS + (int)threadIdx.x) * 8;
            if (c < ld) {
                float g[8];
                load8(w + c, g);
#pragma unroll
                for (int j = 0; j < 8; j++) xv[i][j] += yv[i][j] * inv * g[j];
            }
        }
    }
    float inv2 = 1.0f;
    if (w2) {
        float s2 = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; i++)
            if ((i * THREADS + (int)threadIdx.x) * 8 < ld) {
#pragma unroll
                for (int j = 0; j < 8; j++) s2 = fmaf(xv[i][j], xv[i][j], s2);
            }
        inv2 = 1.0f / sqrtf(row_sum<THREADS>(s2, sh) / (float)dim + eps);
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = (i * THREADS + (int)threadIdx.x) * 8;
        if (c < ld) {
            if (x_out) store8(x_out + base + c, xv[i]);
            if (w2) {
                float g[8];
                load8(w2 + c, g);
#pragma unroll
                for (int j = 0; j < 8; j++) xv[i][j] = xv[i][j] * inv2 * g[j];
            }
            store8(xb + base + c, xv[i]);
        }
    }
}

template <typename T>
int post_norm_t(const float* x, const void* y, const float* w, const float* w2, float* x_out, void* xb, int rows, int dim, int ld, float eps, bool dependent) {
    const int vecs = ld / 8;
#define SPT_POST_NORM(TH_, NV_)                                                                                                                   \
    SPT_CUDA(launch_dependent(post_norm_kernel<T, TH_, NV_>, dim3(rows), dim3(TH_), 0, dependent, 1, x, static_cast<const T*>(y), w, w2, x_out,       \
                              static_cast<T*>(xb), dim, ld, eps))
    if (vecs <= 32) SPT_POST_NORM(32, 1);
    else if (vecs <= 128) SPT_POST_NORM(128, 1);
    else if (vecs <= 256) SPT_POST_NORM(128, 2);
    else if (vecs <= 512) SPT_POST_NORM(256, 2);
    else if (vecs <= 2048) SPT_POST_NORM(512, 4);
    else return fail("post_norm: width %d is larger than 16384", dim);
#undef SPT_POST_NORM
    note_submit();
    return 0;
}

}  // namespace

int post_norm_launch(const float* x, const void* y, const float* w, const float* w2, float* x_out, void* xb, int rows, int dim, int ld, float eps,
                     int dtype, bool dependent) {
    ProfScope ps(PROF_LAYERNORM);
    return dtype == BF16 ? post_norm_t<__nv_bfloat16>(x, y, w, w2, x_out, xb, rows, dim, ld, eps, dependent)
                         : post_norm_t<float>(x, y, w, w2, x_out, xb, rows, dim, ld, eps, dependent);
}

namespace {

int ensure(Gpt* g, LayeredScratch* s, size_t bytes) {
    if (bytes <= s->bytes) return 0;
    if (s->p) { if (stream_wait()) return 1; drop_graphs(g); gfree(g, s->p); }
    s->p = galloc(g, bytes);
    s->bytes = s->p ? bytes : 0;
    if (!s->p) return 1;
    return sptorch_ext_memset(s->p, 0, bytes);
}

// out[M, N] = act(a W^T + bias) (* r for the gated products); rows of a are lda apart and read for K elements, W is [N, ldw]
// pend (few rows only, may be null): a is the residual stream completed on the fly; *fused tells whether that was possible, otherwise
// nothing was launched
int product(Gpt* g, bool few, const void* a, long long lda, const void* w, long long ldw, int K, const float* bias, const void* r, void* out, long long ldo,
            int M, int N, int epi, const RowNorm* pend = nullptr, bool* fused = nullptr) {
    GemmDesc d;
    d.A = a; d.B = w; d.C = out; d.bias = bias; d.R = r;
    d.M = M; d.N = N; d.K = K; d.lda = lda; d.ldb = ldw; d.ldc = ldo;
    d.epilogue = epi; d.mode = g->c.dtype == BF16 ? MM_BF16 : MM_F32; d.out_dtype = g->c.dtype;
    if (pend) {
        *fused = few && linear_few_rows_norm_supported(d, *pend);
        if (!*fused) return 0;
        ProfScope ps(PROF_LINEAR);
        return linear_few_rows(d, pend, true);
    }
    if (few && linear_few_rows_supported(d)) { ProfScope ps(PROF_LINEAR); return linear_few_rows(d, nullptr, true); }
    return gemm_or_simt(d);
}

// x[M, d8] += a W^T, x f32; rows of a are lda apart, W is [d8, ldw].  Few rows: act_off as in GemmDesc, and xb gets a bf16 copy.
GemmDesc stream_product(Gpt* g, const void* a, long long lda, const void* w, long long ldw, int K, float* x, int M) {
    GemmDesc d;
    d.A = a; d.B = w; d.C = x; d.R = x;
    d.M = M; d.N = g->lay->d8; d.K = K; d.lda = lda; d.ldb = ldw; d.ldc = d.N;
    d.mode = g->c.dtype == BF16 ? MM_BF16 : MM_F32; d.out_dtype = F32;
    return d;
}

GlaArgs gla_args(Gpt* g, const LayeredLayer& w, int B, int T, bool cached) {
    GlaArgs a = {};
    a.in = g->lay->in.p; a.ld = w.n_in;
    a.c_q = w.c_q; a.c_k = w.c_k; a.c_v = w.c_v; a.c_g = w.c_g; a.c_a = w.c_a;
    a.B = B; a.T = T; a.H = w.c.heads; a.D = w.c.dim; a.V = w.c.vdim; a.R = w.c.decay_rank;
    a.a2 = w.a2; a.a2_b = w.a2_b; a.head_norm = w.head_norm;
    a.tau = w.c.tau; a.eps = g->c.eps;
    a.state = cached ? w.state : nullptr;
    a.out = g->lay->ao.p; a.ld_out = w.o_ld();
    a.dtype = g->c.dtype;
    return a;
}

LatentArgs latent_args(Gpt* g, const LayeredLayer& w, int B, int T, int first, const int* pos_dev, bool cached) {
    LatentArgs a = {};
    a.in = g->lay->in.p; a.ld_in = w.n_in; a.c_dq = w.c_dq; a.c_dkv = w.c_dkv; a.c_g = w.c_g;
    a.B = B; a.T = T; a.H = w.c.heads; a.D = w.c.dim; a.V = w.c.vdim; a.kv = w.c.kv_rank; a.rot = w.c.rot_dim; a.rope_dims = w.c.rope_dims; a.q_rank = w.c.q_rank;
    a.first = first; a.pos_dev = pos_dev; a.scale = w.c.scale; a.eps = g->c.eps;
    a.dq_norm = w.dq_norm; a.dkv_norm = w.dkv_norm; a.angles = w.angles;
    a.row = w.row(); a.kv8 = w.kv8();
    a.rows = cached ? w.rows : g->lay->rows.p;
    a.seq_stride = (long long)(cached ? g->cache_ctx : T) * a.row;
    a.cq = g->lay->cq.p; a.ld_cq = pad8(w.c.q_rank);
    a.q = g->lay->q.p; a.ld_q = w.q_ld();
    a.w_uk = w.w_ukv; a.w_uv = (const uint8_t*)w.w_ukv + (size_t)w.ukv_v() * a.kv8 * g->es; a.ld_w = a.kv8;
    a.qabs = g->lay->qabs.p; a.olat = g->lay->olat.p;
    a.capacity = cached ? g->cache_ctx : T;
    a.out = g->lay->ao.p; a.ld_out = w.o_ld();
    a.dtype = g->c.dtype;
    return a;
}

// prompts of bf16 models whose head sizes fit expand the keys and values and run the fused kernel
bool expands(const Gpt* g, const LayeredLayer& w) {
    return g->c.dtype == BF16 && attention_latent_supported(w.c.dim, w.c.rot_dim, w.c.vdim, w.ukv_v(), w.q_ld(), w.ukv_ld(), w.row());
}

int gla_layer(Gpt* g, const LayeredLayer& w, int B, int T, bool few, bool cached) {
    const GlaArgs a = gla_args(g, w, B, T, cached);
    ProfScope ps(PROF_RECURRENT);
    if (!few && gla_chunked_supported(a)) return gla_chunked(a, (float*)g->lay->gla_u.p, (float*)g->lay->gla_dec.p);
    return gla_recurrent(a, (float*)g->lay->gla_o.p, few);
}

int latent_layer(Gpt* g, const LayeredLayer& w, int B, int T, int first, const int* pos_dev, bool few, bool cached) {
    const LatentArgs a = latent_args(g, w, B, T, first, pos_dev, cached);
    const int M = B * T;
    { ProfScope ps(PROF_LATENT); if (latent_prep(a, few)) return 1; }
    if (product(g, few, a.cq, a.ld_cq, w.w_uq, a.ld_cq, (int)a.ld_cq, nullptr, nullptr, a.q, a.ld_q, M, (int)a.ld_q, EPI_NONE)) return 1;
    if (few && w.w_ukt && latent_decode_supported(a)) {
        // queries absorbed head by head, attention over the cached rows, values head by head with the gates
        GemmDesc d;
        d.mode = MM_BF16; d.out_dtype = BF16; d.M = M;
        d.A = a.q; d.lda = a.ld_q; d.B = w.w_ukt; d.K = a.D; d.ldb = a.D; d.N = a.H * a.kv8; d.C = a.qabs; d.ldc = d.N;
        d.group = a.kv8; d.group_a = a.D + a.rot; d.group_c = a.kv8;
        GemmDesc e = d;
        e.A = a.olat; e.lda = d.N; e.B = a.w_uv; e.K = a.kv8; e.ldb = a.ld_w; e.N = a.H * a.V; e.C = a.out; e.ldc = a.ld_out;
        e.group = a.V; e.group_a = a.kv8; e.group_c = a.V; e.gate = (const __nv_bfloat16*)a.in + a.c_g; e.ld_gate = a.ld_in;
        if (linear_few_rows_supported(d) && linear_few_rows_supported(e)) {
            ProfScope ps(PROF_ATTN_FUSED);
            return linear_few_rows(d, nullptr, true) || latent_decode(a, true) || linear_few_rows(e, nullptr, true);
        }
    }
    if (few || !expands(g, w)) { ProfScope ps(PROF_ATTN_FUSED); return latent_attention_absorbed(a, few); }
    { ProfScope ps(PROF_LATENT); if (latent_rope_q(a)) return 1; }
    // keys and values of positions 0 .. first + T - 1 of every sequence: [B][n][ukv_ld]
    const int n = first + T;
    GemmDesc d;
    d.A = a.rows; d.B = w.w_ukv; d.C = g->lay->kv.p;
    d.M = n; d.N = w.ukv_ld(); d.K = a.kv8; d.lda = a.row; d.ldb = a.kv8; d.ldc = d.N;
    if (B > 1 && a.seq_stride == (long long)n * a.row) d.M = B * n;               // one product over all sequences
    else if (B > 1) { d.nb1 = B; d.sA1 = a.seq_stride; d.sC1 = (long long)n * d.N; d.b_broadcast = 1; }
    d.mode = MM_BF16; d.out_dtype = BF16;
    if (gemm_or_simt(d)) return 1;
    const uint8_t* kv = (const uint8_t*)g->lay->kv.p;
    ProfScope ps(PROF_ATTN_FUSED);
    return attention_latent(a.q, a.ld_q, kv, kv + (size_t)w.ukv_v() * 2, w.ukv_ld(), (const uint8_t*)a.rows + (size_t)a.kv8 * 2, a.row, a.seq_stride,
                            a.out, a.ld_out, (const uint8_t*)a.in + (size_t)a.c_g * 2, a.ld_in, B, T, n, a.H, a.D, a.rot, a.V, first, a.scale);
}

const LayeredLayer& kv_layer(const Gpt* g, const LayeredLayer& w) { return w.own_kv() ? w : g->lay->L[w.c.kv_from]; }

WindowArgs window_args(Gpt* g, const LayeredLayer& w, int B, int T, int first, const int* pos_dev, bool cached) {
    const LayeredLayer& kv = kv_layer(g, w);
    uint8_t* in = (uint8_t*)g->lay->in.p;
    WindowArgs a = {};
    a.in = in; a.ld_in = w.n_in; a.c_q = w.c_q; a.c_k = w.c_k; a.c_v = w.c_v;
    a.B = B; a.T = T; a.H = w.c.heads; a.G = w.c.kv_heads; a.D = w.c.dim; a.V = w.c.vdim; a.D8 = pad8(a.D); a.V8 = pad8(a.V);
    a.taps = w.c.conv_taps; a.conv = w.conv; a.temp = w.temp; a.slopes = w.slopes;
    a.first = first; a.pos_dev = pos_dev; a.scale = w.c.scale; a.window = w.c.window;
    a.own_kv = w.own_kv();
    a.ring = cached ? w.ring : nullptr; a.ring_cols = w.c_g;
    a.rows = cached ? kv.rows : kv.kv_read ? kv.own.p : g->lay->rows.p;
    a.row = kv.row(); a.capacity = cached ? g->cache_ctx : T; a.seq_stride = (long long)a.capacity * a.row;
    a.q = g->lay->q.p;
    a.out = in + (size_t)w.c_g * g->es; a.ld_out = w.n_in; a.gate = w.c.out_gate ? a.out : nullptr;
    a.dtype = g->c.dtype;
    return a;
}

// The heads' outputs land in the gate's columns of the projections' output.
int window_layer(Gpt* g, const LayeredLayer& w, int B, int T, int first, const int* pos_dev, bool few, bool cached) {
    const WindowArgs a = window_args(g, w, B, T, first, pos_dev, cached);
    const bool decode = few && cached && window_decode_supported(a), fresh = decode && T == 1;
    if (!fresh) { ProfScope ps(PROF_CONV); if (window_prep(a, few)) return 1; }
    ProfScope ps(PROF_ATTN_FUSED);
    if (decode) return window_decode(a, fresh, true);
    if (!few && g->c.dtype == BF16 && attention_window_supported(a.D, a.V, a.row, a.ld_out))
        return attention_window(a.q, a.rows, a.row, a.seq_stride, a.out, a.ld_out, a.gate, B, T, first + T, a.H, a.G, a.D, a.V, first, a.window, a.slopes, a.scale);
    return window_plain(a, few);
}

// Every CTA of W_down's product applies the activation to all the rows it reads, which pays while the rows are few.
constexpr int kActOnReadRows = 16;
// Whether a few rows take the feed-forward's activation on the way into W_down: gate and up then come from one product.
bool act_on_read(const Gpt* g, const LayeredLayer& w, int M) {
    if (w.c.mlp != SPT_MLP_DENSE || w.c.mlp_act != SPT_ACT_RELU || w.c.mixer != SPT_MIXER_WINDOW || M > kActOnReadRows) return false;
    GemmDesc d = stream_product(const_cast<Gpt*>(g), g->lay->in.p, w.n_in, w.w_o, w.o_ld() + pad8(w.c.d_ff), w.o_ld() + pad8(w.c.d_ff), (float*)g->lay->x.p, M);
    d.act_off = pad8(w.c.d_ff); d.act_from = w.o_ld();
    return linear_few_rows_supported(d);
}

int mixer(Gpt* g, const LayeredLayer& w, int B, int T, int first, const int* pos_dev, bool few, bool cached) {
    if (w.c.mixer == SPT_MIXER_GLA) return gla_layer(g, w, B, T, few, cached);
    if (w.c.mixer == SPT_MIXER_LATENT) return latent_layer(g, w, B, T, first, pos_dev, few, cached);
    return window_layer(g, w, B, T, first, pos_dev, few, cached);
}
// where a mixer leaves the heads' outputs
const void* mixer_out(const Gpt* g, const LayeredLayer& w, long long* ld) {
    *ld = w.c.mixer == SPT_MIXER_WINDOW ? w.n_in : w.o_ld();
    return w.c.mixer == SPT_MIXER_WINDOW ? (const uint8_t*)g->lay->in.p + (size_t)w.c_g * g->es : (const uint8_t*)g->lay->ao.p;
}

int gated_epilogue(const LayeredLayer& w) { return w.c.mlp_act == SPT_ACT_RELU ? EPI_RELU_MUL : EPI_SWIGLU; }

// Whether the input projection of a parallel layer takes its rows as a stream to be completed (and the activation of its feed-forward is
// left to W_down, so that nothing else reads the normed rows).
bool parallel_takes_norm(Gpt* g, const LayeredLayer& w, const RowNorm& n, int M) {
    if (w.c.mlp == SPT_MLP_DENSE && !act_on_read(g, w, M)) return false;
    GemmDesc d;
    d.A = g->lay->xb.p; d.B = w.w_in; d.C = g->lay->in.p; d.M = M; d.N = w.n_in; d.K = g->lay->d8; d.lda = d.ldb = d.K; d.ldc = w.n_in;
    d.mode = g->c.dtype == BF16 ? MM_BF16 : MM_F32; d.out_dtype = g->c.dtype;
    return linear_few_rows_norm_supported(d, n);
}

// A layer of a parallel block.  lay.xb holds rms(x) * norm1, or (pend) the input projection makes it from the stream that lacks the layer
// before; afterwards x lacks only the normed lay.y (when there is a token input).
int parallel_layer(Gpt* g, const LayeredLayer& w, int l, const RowNorm* pend, float* x, int B, int T, int first, const int* pos_dev, bool few, bool cached) {
    Layered& lay = *g->lay;
    const int M = B * T, d8 = lay.d8, dense = w.c.mlp == SPT_MLP_DENSE, f8 = dense ? pad8(w.c.d_ff) : 0, o8 = w.o_ld();
    const bool act = few && act_on_read(g, w, M);
    uint8_t* in = (uint8_t*)lay.in.p;
    bool fused = false;
    if (product(g, few, lay.xb.p, d8, w.w_in, d8, d8, nullptr, nullptr, in, w.n_in, M, act ? w.n_in : w.n_in - f8, EPI_NONE, pend, &fused)) return 1;
    void* up = in + (size_t)w.c_up * g->es;
    if (dense && !act && product(g, few, lay.xb.p, d8, (uint8_t*)w.w_in + (size_t)w.c_gate * d8 * g->es, d8, d8, nullptr, up, up, w.n_in, M, f8, gated_epilogue(w))) return 1;
    if (mixer(g, w, B, T, first, pos_dev, few, cached)) return 1;
    const bool side = lay.opt.side_dim > 0;
    bool copied = false;
    auto to_stream = [&](const void* a, long long lda, int col, int K, bool last) -> int {
        GemmDesc d = stream_product(g, a, lda, (const uint8_t*)w.w_o + (size_t)col * g->es, o8 + f8, K, x, M);
        if (act) { d.act_off = f8; d.act_from = o8; }
        if (few) {
            d.C2 = last && side && g->c.dtype == BF16 ? lay.xb.p : nullptr;
            if (linear_few_rows_supported(d)) { copied = d.C2 != nullptr; ProfScope ps(PROF_LINEAR); return linear_few_rows(d, nullptr, true); }
            d.C2 = nullptr;
        }
        return gemm_or_simt(d);
    };
    long long ld_a;
    const void* a = mixer_out(g, w, &ld_a);
    if (w.c.mixer == SPT_MIXER_WINDOW) { if (to_stream(a, ld_a, 0, o8 + f8, true)) return 1; }
    else if (to_stream(a, ld_a, 0, o8, !dense) || (dense && to_stream(up, w.n_in, o8, f8, true))) return 1;
    if (!side) return 0;
    const int s8 = lay.side8;
    const void* xs = x;
    if (g->c.dtype == BF16) {
        if (!copied && post_norm_launch(x, nullptr, nullptr, nullptr, nullptr, lay.xb.p, M, g->c.d_model, d8, g->c.eps, BF16, few)) return 1;
        xs = lay.xb.p;
    }
    const long long ld_e = (long long)lay.L.size() * s8;
    void* e = (uint8_t*)lay.side.p + (size_t)l * s8 * g->es;
    return product(g, few, xs, d8, w.side_gate, d8, d8, nullptr, e, e, ld_e, M, s8, EPI_GELU_MUL) ||
           product(g, few, e, ld_e, w.side_proj, s8, s8, nullptr, nullptr, lay.y.p, d8, M, d8, EPI_NONE);
}

// The launches of one step over B sequences of T new tokens at positions first .. (or pos_dev[0] ..).
int run(Gpt* g, const void* ids, int B, int T, int first, const int* pos_dev, bool few, bool cached, void* logits, const HeadReduce* hr) {
    const sptorch_gpt_config& c = g->c;
    Layered& lay = *g->lay;
    const int M = B * T, d8 = lay.d8, dt = c.dtype, side_ld = (int)lay.L.size() * lay.side8;
    float* x = (float*)lay.x.p;
    {
        ProfScope ps(PROF_EMBED);
        // an ordinary launch: it starts when everything before this step is done, so the kernels behind it may read what earlier steps
        // left in the cache before they wait for their predecessor
        if (dt == BF16) SPT_CUDA(launch_dependent(embed_rows_kernel<__nv_bfloat16>, dim3(M), dim3(128), 0, false, 1, (const __nv_bfloat16*)lay.embed, (const int*)ids, x,
                                                  (__nv_bfloat16*)lay.xb.p, c.vocab, d8, lay.opt.embed_scale, (const __nv_bfloat16*)lay.side_embed, (__nv_bfloat16*)lay.side.p,
                                                  side_ld, rt().dev_status));
        else SPT_CUDA(launch_dependent(embed_rows_kernel<float>, dim3(M), dim3(128), 0, false, 1, (const float*)lay.embed, (const int*)ids, x, (float*)lay.xb.p, c.vocab, d8,
                                       lay.opt.embed_scale, (const float*)lay.side_embed, (float*)lay.side.p, side_ld, rt().dev_status));
        note_submit();
    }
    auto tap = [&](int i) -> int {
        if (!g->taps_on) return 0;
        SPT_CUDA(cudaMemcpy2DAsync(g->taps[i], (size_t)c.d_model * 4, x, (size_t)d8 * 4, (size_t)c.d_model * 4, (size_t)M, cudaMemcpyDeviceToDevice, rt().stream));
        return 0;
    };
    if (tap(0)) return 1;
    // y holds a sublayer's output that has not joined the stream yet: its norm weight.  With few rows the next projection completes the
    // stream while it reads it (x and x2 taken in turn: every CTA reads the old one); otherwise the post-norm kernel does.
    const float* pending = nullptr;
    float* x_other = (float*)lay.x2.p;
    auto settle = [&](const float* fin) -> int {
        if (!pending && !fin) return 0;
        if (post_norm_launch(x, pending ? lay.y.p : nullptr, pending, fin, x, lay.xb.p, M, c.d_model, d8, c.eps, dt, few)) return 1;
        pending = nullptr;
        return 0;
    };
    auto project = [&](const void* w, const float* bias, void* out, int N) -> int {              // a projection of the completed stream
        if (pending && few && !g->taps_on) {
            RowNorm n;
            n.kind = 3; n.gamma = pending; n.eps = c.eps; n.dim = c.d_model; n.x = x; n.y = (const __nv_bfloat16*)lay.y.p; n.x_out = x_other; n.xb = (__nv_bfloat16*)lay.xb.p;
            bool fused = false;
            if (product(g, few, lay.xb.p, d8, w, d8, d8, bias, nullptr, out, N, M, N, EPI_NONE, &n, &fused)) return 1;
            if (fused) { std::swap(x, x_other); pending = nullptr; return 0; }
        }
        return settle(nullptr) || product(g, few, lay.xb.p, d8, w, d8, d8, bias, nullptr, out, N, M, N, EPI_NONE);
    };
    const int nl = (int)lay.L.size();
    const bool parallel = lay.opt.block == SPT_BLOCK_PARALLEL;
    for (int l = 0; l < nl && parallel; l++) {
        const LayeredLayer& w = lay.L[l];
        // one or two rows: the input projection completes the stream and norms it
        RowNorm n;
        n.kind = 4; n.gamma = pending; n.gamma2 = w.norm1; n.eps = c.eps; n.dim = c.d_model; n.x = x; n.y = (const __nv_bfloat16*)lay.y.p; n.x_out = x_other;
        const bool on_the_way = pending && few && !g->taps_on && parallel_takes_norm(g, w, n, M);
        if (on_the_way) { std::swap(x, x_other); pending = nullptr; }
        else if (settle(w.norm1) || (l > 0 && tap(l))) return 1;
        if (parallel_layer(g, w, l, on_the_way ? &n : nullptr, x, B, T, first, pos_dev, few, cached)) return 1;
        if (lay.opt.side_dim > 0) pending = w.side_norm;
    }
    for (int l = 0; l < nl && !parallel; l++) {
        const LayeredLayer& w = lay.L[l];
        if (project(w.w_in, nullptr, lay.in.p, w.n_in)) return 1;
        if (mixer(g, w, B, T, first, pos_dev, few, cached)) return 1;
        long long ld_a;
        const void* a = mixer_out(g, w, &ld_a);
        if (product(g, few, a, ld_a, w.w_o, w.o_ld(), w.o_ld(), nullptr, nullptr, lay.y.p, d8, M, d8, EPI_NONE)) return 1;
        pending = w.norm1;
        if (w.c.mlp == SPT_MLP_DENSE) {
            const int f8 = pad8(w.c.d_ff);
            if (project(w.w_up, w.b_up, lay.f.p, f8)) return 1;
            if (product(g, few, lay.xb.p, d8, w.w_gate, d8, d8, w.b_gate, lay.f.p, lay.f.p, f8, M, f8, gated_epilogue(w))) return 1;
            if (product(g, few, lay.f.p, f8, w.w_down, f8, f8, w.b_down, nullptr, lay.y.p, d8, M, d8, EPI_NONE)) return 1;
            pending = w.norm2;
        }
        if (g->taps_on && l < nl - 1 && (settle(nullptr) || tap(l + 1))) return 1;
    }
    if (settle(lay.final_norm)) return 1;                              // the last update of x also makes the head's input
    if (nl > 0 && tap(nl)) return 1;
    if (few && !hr) return product(g, few, lay.xb.p, d8, g->head, d8, d8, nullptr, nullptr, logits, (long long)g->ldl, M, c.vocab, EPI_NONE);
    return lm_head(g, lay.xb.p, M, logits, hr);
}

constexpr int kFewRows = 64, kFewTokens = 16;

}  // namespace

bool layered_takes_few_rows(const Gpt*, int rows, int T) { return rows <= kFewRows && T <= kFewTokens; }

// scratch for B sequences of T tokens at positions first ..; outside any graph capture
int layered_prepare(Gpt* g, int B, int T, int first, bool cached) {
    Layered& lay = *g->lay;
    const size_t M = (size_t)B * T, es = g->es, n = (size_t)first + T;
    const bool few = cached && layered_takes_few_rows(g, (int)M, T);
    size_t in = 0, ao = 0, cq = 0, q = 0, kv = 0, f = 0, rows = 0, side = 0, qabs = 0, olat = 0, go = 0, gu = 0, gd = 0;
    auto up = [](size_t& a, size_t b) { if (b > a) a = b; };
    for (auto& w : lay.L) {
        up(in, w.n_in); up(ao, w.o_ld());
        if (w.c.mlp == SPT_MLP_DENSE && lay.opt.block != SPT_BLOCK_PARALLEL) up(f, pad8(w.c.d_ff));
        if (w.c.mixer == SPT_MIXER_GLA) {
            const GlaArgs a = gla_args(g, w, B, T, cached);
            if (!few && gla_chunked_supported(a)) { up(gu, gla_chunked_state_bytes(a)); up(gd, gla_chunked_decay_bytes(a)); }
            else up(go, M * w.c.heads * w.c.vdim * 4);
        } else if (w.c.mixer == SPT_MIXER_WINDOW) {
            up(q, (size_t)w.c.heads * pad8(w.c.dim));
            if (!cached && w.own_kv()) {
                if (!w.kv_read) up(rows, w.row());
                else if (ensure(g, &w.own, M * w.row() * es)) return 1;
            }
        } else {
            up(cq, pad8(w.c.q_rank)); up(q, w.q_ld());
            if (!cached) up(rows, w.row());
            if (!few && expands(g, w)) up(kv, w.ukv_ld());
            else { up(qabs, (size_t)w.c.heads * w.row()); up(olat, (size_t)w.c.heads * w.kv8()); }
        }
    }
    const size_t d8 = lay.d8;
    side = lay.L.size() * lay.side8;
    return ensure(g, &lay.side, M * side * es) || ensure(g, &lay.x, M * d8 * 4) || ensure(g, &lay.x2, M * d8 * 4) || ensure(g, &lay.xb, M * d8 * es) || ensure(g, &lay.y, M * d8 * es) || ensure(g, &lay.in, M * in * es) ||
           ensure(g, &lay.ao, M * ao * es) || ensure(g, &lay.cq, M * cq * es) || ensure(g, &lay.q, M * q * es) || ensure(g, &lay.kv, (size_t)B * n * kv * es) ||
           ensure(g, &lay.f, M * f * es) || ensure(g, &lay.rows, M * rows * es) || ensure(g, &lay.qabs, M * qabs * 4) || ensure(g, &lay.olat, M * olat * 4) ||
           ensure(g, &lay.gla_o, go) || ensure(g, &lay.gla_u, gu) || ensure(g, &lay.gla_dec, gd);
}

int layered_forward(Gpt* g, const void* ids, int B, int T, int first, bool cached, void* logits, const HeadReduce* hr) {
    return run(g, ids, B, T, first, nullptr, false, cached, logits, hr);
}
int layered_few_rows(Gpt* g, const void* ids, int B, int T, const int* state, int first, void* logits) {
    return run(g, ids, B, T, first, state, true, true, logits, nullptr);
}

int layered_enable_cache(Gpt* g, int max_context) {
    for (auto& w : g->lay->L) {
        if (w.c.mixer == SPT_MIXER_GLA) {
            w.state = (float*)galloc(g, (size_t)g->c.max_batch * w.c.heads * w.c.dim * w.c.vdim * 4);
            if (!w.state) return 1;
        }
        if (w.c.mixer == SPT_MIXER_WINDOW && w.c.conv_taps > 0) {
            const size_t bytes = (size_t)g->c.max_batch * w.c.conv_taps * w.c_g * g->es;
            w.ring = galloc(g, bytes);
            if (!w.ring || sptorch_ext_memset(w.ring, 0, bytes)) return 1;
        }
        if (w.c.mixer == SPT_MIXER_LATENT || (w.c.mixer == SPT_MIXER_WINDOW && w.own_kv())) {
            const size_t bytes = (size_t)g->c.max_batch * max_context * w.row() * g->es;
            w.rows = galloc(g, bytes);
            if (!w.rows || sptorch_ext_memset(w.rows, 0, bytes)) return 1;
        }
    }
    g->dstate = (int*)galloc(g, 256);
    if (!g->dstate) return 1;
    g->cache_ctx = max_context;
    return layered_reset_cache(g);
}

// Every sequence forgets what it has seen.  Cached rows and rings need no clearing: a position is written before it is read.
int layered_reset_cache(Gpt* g) {
    for (auto& w : g->lay->L)
        if (w.state && sptorch_ext_memset(w.state, 0, (size_t)g->c.max_batch * w.c.heads * w.c.dim * w.c.vdim * 4)) return 1;
    g->cached_len = 0; g->cache_batch = 0; g->window_start = 0;
    return 0;
}

int layered_launches(const Gpt* g, int B, int T) {
    (void)B; (void)T;
    const Layered& lay = *g->lay;
    const bool parallel = lay.opt.block == SPT_BLOCK_PARALLEL, side = lay.opt.side_dim > 0;
    int n = 2;                                                        // embedding, head
    if (lay.L.empty() || parallel) n++;                               // a norm of its own
    for (auto& w : lay.L) {
        const bool dense = w.c.mlp == SPT_MLP_DENSE;
        if (w.c.mixer == SPT_MIXER_GLA) n += g->c.dtype == BF16 && gla_chunked_supported(gla_args(const_cast<Gpt*>(g), w, B, T, false)) ? 3 : 2;
        else if (w.c.mixer == SPT_MIXER_LATENT) n += 5;
        else n += 2;                                                  // convolutions, attention
        if (!parallel) n += 3 + (dense ? 4 : 0);                      // input projection, W_o, post-norm
        else n += 2 + (dense ? w.c.mixer == SPT_MIXER_WINDOW ? 1 : 2 : 0) + (side ? g->c.dtype == BF16 ? 4 : 3 : 1);
    }
    return n;
}

void layered_release(Gpt* g) { delete g->lay; g->lay = nullptr; }

// ---------------- parameters ----------------
namespace {

// one entry per tensor: its name behind the layer's prefix, its shape, and where it goes
struct Slot { std::string name; size_t rows, cols; void* dst; bool f32; int ld; size_t dst_row; const LayeredLayer* ukt = nullptr; size_t part = 0, part_ld = 0; bool transposed = false; };
// cols 0: a vector of `rows` values; part: a row is cut into parts of so many values, part_ld apart on the device; transposed (f32):
// column i of the tensor is at dst + i * ld

// uk [heads*dim, kv] -> its transpose per head, [heads][kv8][dim]
int upload_ukt(Gpt* g, const Slot& s, const float* host) {
    const LayeredLayer& w = *s.ukt;
    const size_t H = w.c.heads, D = w.c.dim, kv = w.c.kv_rank, kv8 = w.kv8();
    std::vector<float> t(H * kv8 * D, 0.0f);
    for (size_t h = 0; h < H; h++)
        for (size_t d = 0; d < D; d++)
            for (size_t c = 0; c < kv; c++) t[(h * kv8 + c) * D + d] = host[(h * D + d) * kv + c];
    return upload_rows(g, w.w_ukt, t.data(), t.size());
}

std::vector<Slot> layer_slots(const Gpt* g, const LayeredLayer& w) {
    const size_t d = g->c.d_model;
    const int d8 = g->lay->d8;
    const sptorch_layer_config& c = w.c;
    std::vector<Slot> s;
    auto mat = [&](const char* n, size_t r, size_t k, void* dst, int ld, size_t row) { s.push_back({n, r, k, dst, false, ld, row}); };
    auto vec = [&](const char* n, size_t r, float* dst) { s.push_back({n, r, 0, dst, true, 0, 0}); };
    const bool mlp = c.mlp == SPT_MLP_DENSE;
    const bool parallel = g->lay->opt.block == SPT_BLOCK_PARALLEL;
    const int ld_wo = w.o_ld() + (parallel && mlp ? pad8(c.d_ff) : 0);
    vec("norm1", d, w.norm1);
    if (mlp && !parallel) vec("norm2", d, w.norm2);
    if (c.mixer == SPT_MIXER_GLA) {
        const size_t hd = (size_t)c.heads * c.dim, hv = (size_t)c.heads * c.vdim;
        mat("mix.q", hd, d, w.w_in, d8, w.c_q); mat("mix.k", hd, d, w.w_in, d8, w.c_k); mat("mix.v", hv, d, w.w_in, d8, w.c_v); mat("mix.g", hv, d, w.w_in, d8, w.c_g);
        mat("mix.o", d, hv, w.w_o, ld_wo, 0);
        vec("mix.norm", c.vdim, w.head_norm);
        mat("mix.a1", c.decay_rank, d, w.w_in, d8, w.c_a);
        s.push_back({"mix.a2", hd, (size_t)c.decay_rank, w.a2, true, c.decay_rank, 0});
        vec("mix.a2.b", hd, w.a2_b);
    } else if (c.mixer == SPT_MIXER_WINDOW) {
        const size_t hd = (size_t)c.heads * c.dim, gd = (size_t)c.kv_heads * c.dim, gv = (size_t)c.kv_heads * c.vdim, hv = (size_t)c.heads * c.vdim;
        const bool kv = w.own_kv();
        mat("mix.q", hd, d, w.w_in, d8, w.c_q);
        if (kv) { mat("mix.k", gd, d, w.w_in, d8, w.c_k); mat("mix.v", gv, d, w.w_in, d8, w.c_v); }
        if (c.conv_taps > 0) {
            auto taps = [&](const char* n, size_t rows, int col) { s.push_back({n, rows, (size_t)c.conv_taps, w.conv + col, true, w.c_g, 0}); s.back().transposed = true; };
            taps("mix.q.conv", hd, w.c_q);
            if (kv) { taps("mix.k.conv", gd, w.c_k); taps("mix.v.conv", gv, w.c_v); }
        }
        if (c.out_gate) mat("mix.g", hv, d, w.w_in, d8, w.c_g);
        mat("mix.o", d, hv, w.w_o, ld_wo, 0);
    } else {
        const int q8 = pad8(c.q_rank), kv8 = w.kv8();
        mat("mix.dq", c.q_rank, d, w.w_in, d8, w.c_dq); vec("mix.dq.norm", c.q_rank, w.dq_norm);
        mat("mix.uq", (size_t)c.heads * (c.dim + c.rot_dim), c.q_rank, w.w_uq, q8, 0);
        mat("mix.dkv", (size_t)c.kv_rank + c.rot_dim, d, w.w_in, d8, w.c_dkv); vec("mix.dkv.norm", c.kv_rank, w.dkv_norm);
        mat("mix.uk", (size_t)c.heads * c.dim, c.kv_rank, w.w_ukv, kv8, 0);
        if (w.w_ukt) s.back().ukt = &w;
        mat("mix.uv", (size_t)c.heads * c.vdim, c.kv_rank, w.w_ukv, kv8, w.ukv_v());
        mat("mix.g", c.heads, d, w.w_in, d8, w.c_g);
        mat("mix.o", d, (size_t)c.heads * c.vdim, w.w_o, ld_wo, 0);
    }
    if (mlp && parallel) {
        mat("mlp.gate", c.d_ff, d, w.w_in, d8, w.c_gate);
        mat("mlp.up", c.d_ff, d, w.w_in, d8, w.c_up);
        mat("mlp.down", d, c.d_ff, (uint8_t*)w.w_o + (size_t)w.o_ld() * g->es, ld_wo, 0);
    } else if (mlp) {
        const int f8 = pad8(c.d_ff);
        mat("mlp.gate", c.d_ff, d, w.w_gate, d8, 0); if (c.mlp_bias) vec("mlp.gate.b", c.d_ff, w.b_gate);
        mat("mlp.up", c.d_ff, d, w.w_up, d8, 0); if (c.mlp_bias) vec("mlp.up.b", c.d_ff, w.b_up);
        mat("mlp.down", d, c.d_ff, w.w_down, f8, 0); if (c.mlp_bias) vec("mlp.down.b", d, w.b_down);
    }
    if (g->lay->opt.side_dim > 0) {
        const size_t sd = g->lay->opt.side_dim;
        mat("side.gate", sd, d, w.side_gate, d8, 0); mat("side.proj", d, sd, w.side_proj, g->lay->side8, 0); vec("side.norm", d, w.side_norm);
    }
    return s;
}

std::vector<Slot> model_slots(const Gpt* g) {
    const size_t V = g->c.vocab, d = g->c.d_model;
    std::vector<Slot> s;
    s.push_back({"embed", V, d, g->lay->embed, false, g->lay->d8, 0});
    const size_t L = g->lay->L.size(), sd = g->lay->opt.side_dim, s8 = g->lay->side8;
    if (sd && L) {                                                       // a row holds sd values per layer, on the device s8
        s.push_back({"side.embed", V, L * sd, g->lay->side_embed, false, (int)(L * s8), 0});
        s.back().part = sd; s.back().part_ld = s8;
    }
    for (size_t l = 0; l < g->lay->L.size(); l++)
        for (auto& e : layer_slots(g, g->lay->L[l])) { s.push_back(e); s.back().name = "l" + std::to_string(l) + "." + e.name; }
    s.push_back({"final.norm", d, 0, g->lay->final_norm, true, 0, 0});
    if (!g->lay->opt.tied_head) s.push_back({"head", V, d, g->lay->head, false, g->lay->d8, 0});
    return s;
}

}  // namespace

std::vector<ParamInfo> layered_param_table(const Gpt* g) {
    std::vector<ParamInfo> t;
    for (auto& s : model_slots(g)) t.push_back({s.name, s.cols ? std::vector<size_t>{s.rows, s.cols} : std::vector<size_t>{s.rows}});
    return t;
}

int layered_set_param(Gpt* g, const char* name, const float* host, size_t n) {
    const std::string key(name);
    for (auto& s : model_slots(g)) {
        if (s.name != key) continue;
        const size_t want = s.rows * (s.cols ? s.cols : 1);
        if (n != want) return fail("gpt_set_param(%s): got %zu values, expected %zu", name, n, want);
        if (s.transposed) {
            std::vector<float> t(n);
            for (size_t r = 0; r < s.rows; r++)
                for (size_t i = 0; i < s.cols; i++) t[i * s.rows + r] = host[r * s.cols + i];
            SPT_CUDA(cudaMemcpy2DAsync(s.dst, (size_t)s.ld * 4, t.data(), s.rows * 4, s.rows * 4, s.cols, cudaMemcpyHostToDevice, rt().stream));
            return stream_wait();
        }
        if (s.f32) return sptorch_ext_copy_h2d_bytes(host, s.dst, n * 4) || stream_wait();
        void* dst = (uint8_t*)s.dst + s.dst_row * s.ld * g->es;
        if (s.ukt && upload_ukt(g, s, host)) return 1;
        if ((size_t)s.ld == s.cols) return upload_rows(g, dst, host, n) || stream_wait();
        const size_t parts = s.part ? s.cols / s.part : 1, part = s.part ? s.part : s.cols, part_ld = s.part ? s.part_ld : (size_t)pad8((int)s.cols), wide = parts * part_ld;
        std::vector<float> padded(s.rows * wide, 0.0f);
        for (size_t r = 0; r < s.rows; r++)
            for (size_t i = 0; i < parts; i++) memcpy(&padded[r * wide + i * part_ld], host + r * s.cols + i * part, part * 4);
        if (wide == (size_t)s.ld) return upload_rows(g, dst, padded.data(), padded.size()) || stream_wait();
        // columns of a wider matrix, whose other columns stay as they are
        void* tight = sptorch_ext_alloc_bytes(padded.size() * g->es);
        if (!tight) return 1;
        int rc = upload_rows(g, tight, padded.data(), padded.size());
        if (!rc && cudaMemcpy2DAsync(dst, (size_t)s.ld * g->es, tight, wide * g->es, wide * g->es, s.rows, cudaMemcpyDeviceToDevice, rt().stream) != cudaSuccess)
            rc = fail("gpt_set_param(%s): copy into the fused matrix failed", name);
        if (!rc) rc = stream_wait();
        sptorch_free(tight);
        return rc;
    }
    return fail("gpt_set_param: unknown parameter name '%s'", name);
}

static int check_layer(const sptorch_layer_config* layers, int i, const sptorch_layered_options& opt) {
    const sptorch_layer_config& c = layers[i];
    if (c.mixer != SPT_MIXER_GLA && c.mixer != SPT_MIXER_LATENT && c.mixer != SPT_MIXER_WINDOW) return fail_host("layered_create: layer %d: unknown mixer %d", i, c.mixer);
    if (c.heads <= 0 || c.dim <= 0 || c.vdim <= 0) return fail_host("layered_create: layer %d: non-positive head count or size", i);
    if (c.mixer == SPT_MIXER_GLA) {
        if (c.decay_rank <= 0 || !(c.tau > 0.0f)) return fail_host("layered_create: layer %d: decay_rank and tau must be positive", i);
        if (c.dim > 512) return fail_host("layered_create: layer %d: key size %d is larger than 512", i, c.dim);
    } else if (c.mixer == SPT_MIXER_LATENT) {
        if (c.kv_rank <= 0 || c.q_rank <= 0 || c.rot_dim < 0) return fail_host("layered_create: layer %d: latent sizes must be positive", i);
        if (c.rope_dims < 0 || c.rope_dims > c.rot_dim || c.rope_dims % 2) return fail_host("layered_create: layer %d: %d rotated dims of %d", i, c.rope_dims, c.rot_dim);
        if (c.rope_dims && !(c.rope_base > 0.0)) return fail_host("layered_create: layer %d: rope_base must be positive", i);
        if (pad8(c.kv_rank) + pad8(c.rot_dim) > 1280) return fail_host("layered_create: layer %d: cached rows of %d + %d values are larger than 1280", i, c.kv_rank, c.rot_dim);
    } else {
        if (c.dim > kWindowMaxHead || c.vdim > kWindowMaxHead) return fail_host("layered_create: layer %d: heads of %d and %d are larger than %d", i, c.dim, c.vdim, kWindowMaxHead);
        if (c.kv_heads <= 0 || c.heads % c.kv_heads) return fail_host("layered_create: layer %d: %d query heads on %d key/value heads", i, c.heads, c.kv_heads);
        if (c.window < 0 || c.conv_taps < 0) return fail_host("layered_create: layer %d: negative window or convolution", i);
        if (c.kv_shared) {
            if (c.kv_from < 0 || c.kv_from >= i) return fail_host("layered_create: layer %d: keys and values of layer %d, which does not come before it", i, c.kv_from);
            const sptorch_layer_config& s = layers[c.kv_from];
            if (s.mixer != SPT_MIXER_WINDOW || s.kv_shared || s.kv_heads != c.kv_heads || s.dim != c.dim || s.vdim != c.vdim)
                return fail_host("layered_create: layer %d: layer %d has no keys and values of %d heads of %d and %d", i, c.kv_from, c.kv_heads, c.dim, c.vdim);
        }
    }
    if (c.mlp_act != SPT_ACT_SILU && c.mlp_act != SPT_ACT_RELU) return fail_host("layered_create: layer %d: unknown activation %d", i, c.mlp_act);
    if (opt.block == SPT_BLOCK_PARALLEL && c.mlp == SPT_MLP_DENSE && c.mlp_bias) return fail_host("layered_create: layer %d: the feed-forward of a parallel block has no biases", i);
    if (c.mlp != SPT_MLP_NONE && c.mlp != SPT_MLP_DENSE) return fail_host("layered_create: layer %d: unknown feed-forward %d", i, c.mlp);
    if (c.mlp == SPT_MLP_DENSE && c.d_ff <= 0) return fail_host("layered_create: layer %d: non-positive d_ff", i);
    return 0;
}

}  // namespace spt

using namespace spt;

extern "C" void* sptorch_ext_layered_create(const sptorch_gpt_config* cfg, const sptorch_layer_config* layers, int n_layers,
                                             const sptorch_layered_options* options) {
    if (enter()) return nullptr;
    if (!cfg || (n_layers > 0 && !layers)) { fail("layered_create: null config"); return nullptr; }
    sptorch_gpt_config c = *cfg;
    c.arch = SPT_ARCH_LAYERED; c.n_layer = n_layers; c.n_head = 1; c.d_ff = 1; c.tp_size = 1; c.tp_rank = 0;
    if (cfg->tp_size > 1) { fail("layered_create: no tensor parallel shards"); return nullptr; }
    if (c.vocab <= 0 || c.d_model <= 0 || n_layers < 0 || c.seq_len <= 0 || c.max_batch <= 0) { fail("layered_create: non-positive dimension"); return nullptr; }
    if (c.dtype != SPT_F32 && c.dtype != SPT_BF16) { fail("layered_create: unknown dtype %d", c.dtype); return nullptr; }
    sptorch_layered_options opt = {};
    opt.embed_scale = 1.0f;
    if (options) opt = *options;
    if (opt.block != SPT_BLOCK_POST_NORM && opt.block != SPT_BLOCK_PARALLEL) { fail("layered_create: unknown block %d", opt.block); return nullptr; }
    if (opt.side_dim < 0 || (opt.side_dim > 0 && opt.block != SPT_BLOCK_PARALLEL)) { fail("layered_create: a per-layer token input needs a parallel block"); return nullptr; }
    for (int i = 0; i < n_layers; i++) if (check_layer(layers, i, opt)) return nullptr;
    const bool parallel = opt.block == SPT_BLOCK_PARALLEL;
    Gpt* g = new Gpt();
    g->c = c;
    g->es = c.dtype == SPT_BF16 ? 2 : 4;
    g->ldl = ((size_t)c.vocab + 63) / 64 * 64;
    g->lay = new Layered();
    Layered& lay = *g->lay;
    lay.d8 = pad8(c.d_model);
    const size_t d8 = lay.d8, es = g->es, V = c.vocab;
    bool ok = true;
    auto Z = [&](size_t bytes) { void* p = galloc(g, bytes); if (!p || sptorch_ext_memset(p, 0, bytes)) ok = false; return p; };
    auto F = [&](size_t n) { return (float*)Z((size_t)pad8((int)n) * 4); };
    lay.opt = opt;
    lay.side8 = pad8(opt.side_dim);
    lay.embed = Z(V * d8 * es); lay.head = opt.tied_head ? lay.embed : Z(V * d8 * es); lay.final_norm = F(d8);
    if (opt.side_dim && n_layers) lay.side_embed = Z(V * n_layers * lay.side8 * es);
    g->head = lay.head; g->tok = lay.embed;
    std::map<std::pair<int, double>, float2*> angles;
    std::map<std::pair<double, double>, float*> temps;
    auto table = [&](const std::vector<float>& host) -> float* {
        float* p = (float*)galloc(g, host.size() * 4);
        if (!p || sptorch_ext_copy_h2d_bytes(host.data(), p, host.size() * 4) || stream_wait()) { ok = false; return nullptr; }
        return p;
    };
    for (int i = 0; i < n_layers && ok; i++) {
        LayeredLayer w;
        w.c = layers[i];
        const sptorch_layer_config& lc = w.c;
        auto at = [&](int& col, int width) { col = w.n_in; w.n_in += pad8(width); };
        w.norm1 = F(d8);
        if (!parallel) w.norm2 = F(d8);
        if (lc.mixer == SPT_MIXER_GLA) {
            at(w.c_q, lc.heads * lc.dim); at(w.c_k, lc.heads * lc.dim); at(w.c_v, lc.heads * lc.vdim); at(w.c_g, lc.heads * lc.vdim); at(w.c_a, lc.decay_rank);
            w.a2 = F((size_t)lc.heads * lc.dim * lc.decay_rank); w.a2_b = F((size_t)lc.heads * lc.dim); w.head_norm = F(lc.vdim);
        } else if (lc.mixer == SPT_MIXER_WINDOW) {
            at(w.c_q, lc.heads * lc.dim);
            if (w.own_kv()) { at(w.c_k, lc.kv_heads * lc.dim); at(w.c_v, lc.kv_heads * lc.vdim); }
            at(w.c_g, lc.heads * lc.vdim);
            if (lc.conv_taps > 0) w.conv = F((size_t)w.c_g * lc.conv_taps);
            if (lc.q_temp_every > 0.0) {
                float*& tab = temps[{lc.q_temp_coef, lc.q_temp_every}];
                if (!tab) {
                    std::vector<float> host(c.seq_len);
                    for (int p = 0; p < c.seq_len; p++) host[p] = (float)(1.0 + lc.q_temp_coef * std::log(std::floor((p + 1.0) / lc.q_temp_every) + 1.0));
                    tab = table(host);
                }
                w.temp = tab;
            }
            if (lc.distance_bias) {
                std::vector<float> host(lc.heads);
                for (int h = 0; h < lc.heads; h++) host[h] = (float)std::pow(2.0, -8.0 * (h + 1) / lc.heads);
                w.slopes = table(host);
            }
            if (lc.kv_shared) lay.L[lc.kv_from].kv_read = true;
        } else {
            at(w.c_dq, lc.q_rank); at(w.c_dkv, lc.kv_rank + lc.rot_dim); at(w.c_g, lc.heads);
            w.dq_norm = F(lc.q_rank); w.dkv_norm = F(lc.kv_rank);
            w.w_uq = Z((size_t)w.q_ld() * pad8(lc.q_rank) * es); w.w_ukv = Z((size_t)w.ukv_ld() * w.kv8() * es);
            if (c.dtype == SPT_BF16 && lc.dim % 8 == 0) w.w_ukt = Z((size_t)lc.heads * w.kv8() * lc.dim * es);
            if (lc.rope_dims) {
                float2*& tab = angles[{lc.rope_dims, lc.rope_base}];
                if (!tab) {
                    const int half = lc.rope_dims / 2;
                    std::vector<float2> host((size_t)c.seq_len * half);
                    for (int k = 0; k < half; k++) {
                        const double f = std::pow(lc.rope_base, -2.0 * k / lc.rope_dims);
                        for (int p = 0; p < c.seq_len; p++) host[(size_t)p * half + k] = make_float2((float)std::cos(p * f), (float)std::sin(p * f));
                    }
                    tab = (float2*)galloc(g, host.size() * sizeof(float2));
                    if (!tab || sptorch_ext_copy_h2d_bytes(host.data(), tab, host.size() * sizeof(float2)) || stream_wait()) { ok = false; break; }
                }
                w.angles = tab;
            }
        }
        const size_t f8 = lc.mlp == SPT_MLP_DENSE ? pad8(lc.d_ff) : 0;
        if (parallel && f8) { at(w.c_up, lc.d_ff); at(w.c_gate, lc.d_ff); }
        w.w_in = Z((size_t)w.n_in * d8 * es);
        w.w_o = Z(d8 * (w.o_ld() + (parallel ? f8 : 0)) * es);
        if (lay.side8) { w.side_gate = Z((size_t)lay.side8 * d8 * es); w.side_proj = Z(d8 * lay.side8 * es); w.side_norm = F(d8); }
        if (f8 && !parallel) {
            w.w_gate = Z(f8 * d8 * es); w.w_up = Z(f8 * d8 * es); w.w_down = Z(d8 * f8 * es);
            w.b_gate = F(f8); w.b_up = F(f8); w.b_down = F(d8);
        }
        lay.L.push_back(w);
    }
    if (!ok) { sptorch_ext_gpt_destroy(g); return nullptr; }
    return g;
}
