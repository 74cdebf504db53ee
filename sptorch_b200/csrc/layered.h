// layered.h -- models built from a list of layers, each with its own mixer, sizes and feed-forward: the structures of the driver
// (layered.cu) and the launch functions of the mixers' kernels (gla.cu, latent_attention.cu, window_attention.cu).
//
// Every row buffer and weight matrix is padded to a multiple of eight elements per row with zeros (pad8): a row then starts on a
// 16-byte boundary in both dtypes, whatever the model's sizes, and a padded K adds zeros to a sum.
#pragma once
#include "common.h"
#include "gpt_model.h"

namespace spt {

inline int pad8(int n) { return (n + 7) / 8 * 8; }

// scratch grown on demand (outside any graph capture); new memory starts as zeros
struct LayeredScratch { void* p = nullptr; size_t bytes = 0; };

// One layer's weights (device), where its projections lie in the columns of its input projection's output, and what it keeps of
// every sequence.  Gated linear attention keeps a [dim, vdim] f32 matrix per (sequence, head); latent attention keeps a row
// [latent | rotated key part] per position; window attention keeps a row [keys | values] per position, unless it reads another layer's,
// and a ring of its last projected rows.  Layers of a parallel block have the feed-forward's projections in w_in too, and W_o and W_down
// side by side in w_o: the columns [gate of the heads | up] of the projections' output become [heads | feed-forward] in place, and
// one product takes both back to the stream.
struct LayeredLayer {
    sptorch_layer_config c;
    void* w_in = nullptr;                        // every projection that reads the layer's input, one matrix [n_in, pad8(width)]
    int n_in = 0;                                // its rows; each projection starts at a multiple of eight
    int c_q = 0, c_k = 0, c_v = 0, c_g = 0, c_a = 0;         // gated linear attention: columns of q, k, v, output gate, decay latent
    float *a2 = nullptr, *a2_b = nullptr;        // decay: [heads*dim, decay_rank] and its bias
    float* head_norm = nullptr;                  // [vdim]
    int c_dq = 0, c_dkv = 0;                     // latent attention: columns of the query latent and of [latent | rotated part]; c_g: the head gates
    float *dq_norm = nullptr, *dkv_norm = nullptr;
    void* w_ukt = nullptr;                       // bf16, dim a multiple of 8: uk transposed per head, [heads][pad8(kv_rank)][dim] (few tokens)
    void *w_uq = nullptr, *w_ukv = nullptr;      // [heads*(dim+rot_dim), pad8(q_rank)]; [uk rows, then at row pad8(heads*dim) uv rows][pad8(kv_rank)]
    void* w_o = nullptr;                         // [pad8(width), pad8(heads*vdim)]
    float *norm1 = nullptr, *norm2 = nullptr;
    void *w_gate = nullptr, *w_up = nullptr, *w_down = nullptr;
    float *b_gate = nullptr, *b_up = nullptr, *b_down = nullptr;
    float* state = nullptr;                      // gated linear attention: [max_batch][heads][dim][vdim]
    void* rows = nullptr;                        // latent and window attention: [max_batch][cache positions][row()]
    int c_up = 0, c_gate = 0;                    // parallel block: columns of the feed-forward's two projections
    float* conv = nullptr;                       // window attention: [taps][c_g], the columns of q, k and v as they lie in w_in
    const float *temp = nullptr, *slopes = nullptr;          // ... position factors of the queries [seq_len], distance slopes [heads]
    void* ring = nullptr;                        // ... [max_batch][taps][c_g]: projected rows of the last positions, slot = position % taps
    LayeredScratch own;                          // ... rows of a forward without a cache
    bool kv_read = false;                        // ... a later layer reads these keys and values
    void *side_gate = nullptr, *side_proj = nullptr;         // per-layer token input: [pad8(side_dim), d8], [d8, pad8(side_dim)]
    float* side_norm = nullptr;
    const float2* angles = nullptr;              // (cos, sin) of position p and pair i at [p * rope_dims / 2 + i]

    int q_ld() const { return pad8(c.heads * (c.dim + c.rot_dim)); }
    int kv8() const { return pad8(c.kv_rank); }
    bool own_kv() const { return !c.kv_shared; }
    int row() const { return c.mixer == SPT_MIXER_WINDOW ? c.kv_heads * (pad8(c.dim) + pad8(c.vdim)) : pad8(c.kv_rank) + pad8(c.rot_dim); }      // elements of a cached row
    int ukv_v() const { return pad8(c.heads * c.dim); }                // first row of the value part of w_ukv
    int ukv_ld() const { return ukv_v() + pad8(c.heads * c.vdim); }
    int o_ld() const { return pad8(c.heads * c.vdim); }
};

struct Layered {
    std::vector<LayeredLayer> L;
    sptorch_layered_options opt = {};
    int d8 = 0, side8 = 0;                       // pad8(width), pad8(side_dim)
    void* side_embed = nullptr;                  // [vocab, layers * side8]
    void *embed = nullptr, *head = nullptr;      // [vocab, d8]
    float* final_norm = nullptr;
    LayeredScratch x, x2, xb, y, in, ao, cq, q, kv, f, rows, qabs, olat, gla_o, gla_u, gla_dec, side;
};

// ---- entry points of gpt.cu's handle for such a model ----
int layered_forward(Gpt* g, const void* ids, int B, int T, int first, bool cached, void* logits, const HeadReduce* hr);
int layered_few_rows(Gpt* g, const void* ids, int B, int T, const int* state, int first, void* logits);
bool layered_takes_few_rows(const Gpt* g, int rows, int T);
int layered_prepare(Gpt* g, int B, int T, int first, bool cached);
int layered_enable_cache(Gpt* g, int max_context);
int layered_reset_cache(Gpt* g);
int layered_set_param(Gpt* g, const char* name, const float* host, size_t n);
std::vector<ParamInfo> layered_param_table(const Gpt* g);
int layered_launches(const Gpt* g, int B, int T);
void layered_release(Gpt* g);

// ---- row kernels of layered.cu ----
// x <- x + y / sqrt(mean(y^2) + eps) * w per row (y null: x as it is), all in f32; xb <- x in dtype, or, with w2, x / sqrt(mean(x^2)
// + eps) * w2.  The means run over dim elements; rows are ld elements apart.  x_out may be x.
int post_norm_launch(const float* x, const void* y, const float* w, const float* w2, float* x_out, void* xb, int rows, int dim, int ld, float eps,
                     int dtype, bool dependent);

// ---- gla.cu ----
// One call's view of a gated linear attention layer: `in` holds the projections of B*T tokens (rows of ld elements).
struct GlaArgs {
    const void* in; long long ld;
    int c_q, c_k, c_v, c_g, c_a;
    int B, T, H, D, V, R;                        // R: rank of the decay projection
    const float *a2, *a2_b, *head_norm;
    float tau, eps;
    float* state;                                // [B][H][D][V], read and written (null: starts at zero and is not kept)
    void* out; long long ld_out;                 // [B*T, ld_out]: normed, gated heads
    int dtype;
};
// token after token; any sizes; o_scratch: B*T*H*V floats
int gla_recurrent(const GlaArgs& a, float* o_scratch, bool dependent);
// chunks of tokens on the tensor cores (bf16)
bool gla_chunked_supported(const GlaArgs& a);
size_t gla_chunked_state_bytes(const GlaArgs& a);
size_t gla_chunked_decay_bytes(const GlaArgs& a);
int gla_chunked(const GlaArgs& a, float* u_scratch, float* dec_scratch);

// ---- latent_attention.cu ----
struct LatentArgs {
    const void* in; long long ld_in;             // projections of B*T tokens: query latent at c_dq, [latent | rotated part] at c_dkv, head gates at c_g
    int c_dq, c_dkv, c_g;
    int B, T, H, D, V, kv, rot, rope_dims, q_rank;
    int first;                                   // position of token 0 of every sequence ...
    const int* pos_dev;                          // ... or, when given, pos_dev[0] (decode graphs)
    float scale, eps;
    const float *dq_norm, *dkv_norm;
    const float2* angles;
    void* rows; long long seq_stride;            // cached rows of sequence b at rows + b * seq_stride; position p at p * row
    int row, kv8;
    void* cq; long long ld_cq;                   // out of prep: normed query latent
    void* q; long long ld_q;                     // queries, head by head [D | rot]
    const void *w_uk, *w_uv; long long ld_w;
    void *qabs, *olat;                           // per (token, head): absorbed query and attended latent.  Plain kernels: f32, [row] and
                                                 // [kv8]; the tensor-core kernel: bf16, [kv8] (rotation applied as it loads) and [kv8]
    int capacity;                                // positions the cache holds: what the split over CTAs is chosen for
    void* out; long long ld_out;
    int dtype;
};
// query latent normed into cq; latent normed and key part rotated into the cached row of the token's position
int latent_prep(const LatentArgs& a, bool dependent);
// rotates the rot part of every head of q in place (prompts; the few-token path rotates while it absorbs)
int latent_rope_q(const LatentArgs& a);
// few tokens, or any tokens of a shape the fused kernel does not take: attention over the cached rows themselves, W_uk folded into
// the query and W_uv applied to the attended latent
int latent_attention_absorbed(const LatentArgs& a, bool dependent);
// the attention of that path for bf16 on the tensor cores: qabs [M][H * kv8] without the rotated part -> olat [M][H * kv8]
bool latent_decode_supported(const LatentArgs& a);
int latent_decode(const LatentArgs& a, bool dependent);

// ---- window_attention.cu ----
constexpr int kWindowMaxHead = 1024;             // largest query/key and value size of a head
struct WindowArgs {
    const void* in; long long ld_in;             // projections of B*T tokens: q, k, v of every head at c_q, c_k, c_v
    int c_q, c_k, c_v;
    int B, T, H, G, D, V, D8, V8, taps;
    const float* conv;                           // [taps][ring_cols] (taps 0: none)
    const float *temp, *slopes;                  // may be null
    int first; const int* pos_dev;               // as in LatentArgs
    float scale; int window;                     // window 0: every earlier position
    bool own_kv;                                 // false: the rows are another layer's, complete for this call's tokens
    void* ring; int ring_cols;                   // null: nothing is kept, and the call starts its sequences
    void* rows; long long seq_stride; int row, capacity;
    void* q;                                     // out of prep: [B*T, H * D8]
    const void* gate; void* out; long long ld_out;           // [B*T, ld_out], head h at columns h*V; gate may be out, or null
    int dtype;
};
// projections -> convolved queries and cached rows; the ring's new slots
int window_prep(const WindowArgs& a, bool dependent);
// any sizes, from q and the rows
int window_plain(const WindowArgs& a, bool dependent);
// few tokens, bf16.  fresh (T = 1): window_prep has not run, the kernel does its work for the one token
bool window_decode_supported(const WindowArgs& a);
int window_decode(const WindowArgs& a, bool fresh, bool dependent);

}  // namespace spt
