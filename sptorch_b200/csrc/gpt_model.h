// gpt_model.h -- the model behind a sptorch_ext_gpt_* handle, shared by the two drivers that run one: gpt.cu (GPT and Qwen-like models,
// whose layers are all alike) and layered.cu (models built from a list of layers).
#pragma once
#include "gemm.h"
#include "../../include/sptorch_b200_hal.h"
#include "../../include/sptorch_b200_ext.h"
#include <string>
#include <vector>

namespace spt {

struct Layered;      // layered.h: the layers of a model built from a list (nullptr for GPT and Qwen-like models)

struct Layer {
    float *ln1g, *ln1b, *ln2g, *ln2b, *b1, *b2;     // Qwen-like: ln1g / ln2g hold the RMSNorm weights, the betas are unused
    void *wqkv;                                      // [Wq; Wk; Wv] of this rank, one [3*d_loc, d] matrix
    void *wqk, *wv, *wo, *w1, *w2;                   // wqk = rows 0..2*d_loc of wqkv, wv = rows 2*d_loc..
    void* wg = nullptr; float* bg = nullptr;         // Qwen-like: gate projection of the SwiGLU MLP
    // LayerNorm folded into the GEMMs that consume it (bf16 GPT): weights times gamma, their row sums s, and c = W beta (+ bias)
    void *wqkv_f = nullptr, *w1_f = nullptr;
    float *s_qkv = nullptr, *c_qkv = nullptr, *s_1 = nullptr, *c_1 = nullptr;
};

struct Gpt {
    sptorch_gpt_config c;
    Layered* lay = nullptr; // set for SPT_ARCH_LAYERED: the layers, their cache and scratch (layered.cu)
    int es;                 // bytes per activation/weight element
    int d_loc, H_loc, F_loc;
    size_t ldl;             // logits row stride
    void *tok, *pos, *head;
    float *lnfg, *lnfb;
    std::vector<Layer> L;
    // activations for max_batch * seq_len tokens
    void *x, *y, *h, *qkv, *ao, *f;                // qkv: [tokens, 3*d_loc] = [q | k | v] of every token
    void *vt = nullptr, *scores = nullptr;          // materialised attention only (ensure_scores): V^T [d_loc, tokens], scores [batch, heads, T, T]
    size_t scores_elems = 0, vt_elems = 0;
    std::vector<void*> taps; bool taps_on = false;
    sptorch_allreduce_fn ar = nullptr; void* ar_user = nullptr;
    std::vector<void*> owned;
    // pipelined host call
    void* logits_dev[2] = {nullptr, nullptr}; int* ids_dev = nullptr; int ids_cap = 0; size_t logits_cap = 0;
    cudaEvent_t ev_compute[2] = {nullptr, nullptr}, ev_copy[2] = {nullptr, nullptr};
    cudaEvent_t ev_partial[2] = {nullptr, nullptr}, ev_reduced[2] = {nullptr, nullptr};     // tensor-parallel pipeline
    // key/value cache for incremental decode: [layer][sequence][position][d_loc], allocated by gpt_enable_kv_cache
    void *kcache = nullptr, *vcache = nullptr;
    int cache_ctx = 0, cached_len = 0, cache_batch = 0;
    long long window_start = 0;   // absolute position of the oldest cached token (grows once the cache is full and slides)
    int* dstate = nullptr;        // device words of the current decode step: position, valid positions, ring slot, position-table row
    struct DecodeKey {
        const void* ids; void* logits; int batch, append; cudaStream_t stream; uint64_t epoch;
        bool operator==(const DecodeKey& o) const { return ids == o.ids && logits == o.logits && batch == o.batch && append == o.append && stream == o.stream && epoch == o.epoch; }
    };
    DecodeKey dkey = {nullptr, nullptr, 0, 0, nullptr, 0};
    cudaGraphExec_t dexec = nullptr; int d_eager = 0;
    bool fill_cache = false;      // set while a prefill runs
    void *dq = nullptr;                  // decode scratch: [max_batch, 3*d_loc] = [q | k | v] of the new tokens
    // CUDA graph of one forward, keyed by everything that is baked into its kernel arguments
    // (the config epoch covers the process-wide setters that change which kernels or grids a forward launches)
    struct GraphKey {
        const void* ids; void* logits; int batch, T; bool taps; cudaStream_t stream; uint64_t epoch;
        const void *targets, *argmax, *row_loss; int has_ignore; long long ignore_index; bool reduce;      // fused LM head (HeadReduce)
        bool operator==(const GraphKey& o) const {
            return ids == o.ids && logits == o.logits && batch == o.batch && T == o.T && taps == o.taps && stream == o.stream && epoch == o.epoch &&
                   targets == o.targets && argmax == o.argmax && row_loss == o.row_loss && has_ignore == o.has_ignore &&
                   ignore_index == o.ignore_index && reduce == o.reduce;
        }
    };
    // a few keys are kept so that callers alternating between buffers (double buffering) replay instead of re-capturing
    struct GraphSlot { GraphKey key; cudaGraphExec_t exec = nullptr; int eager_runs = 0; uint64_t last_use = 0; };
    static constexpr int kGraphSlots = 4;
    GraphSlot gslots[kGraphSlots];
    uint64_t guse = 0;
    bool graphs = true;
    // folded LayerNorm (see forward): per-token statistics, the head's folded copy, and whether the copies are stale
    float2* ln_stats = nullptr; void* head_f = nullptr; float *s_h = nullptr, *c_h = nullptr;
    bool ln_fold = false, fold_ready = false, fold_dirty = true;     // opt-in: measured neutral (see sptorch_ext_gpt_enable_ln_fold)
    int tp_overlap = 2;        // tensor parallel: reduce one half of the batch while the other half computes: 0 never, 1 always, 2 from 4 ranks up
    // LM head fused with the loss / greedy choice: per-row partial reductions of the head GEMM's tiles
    float2* red_part = nullptr; int* red_arg = nullptr; float* red_tgt = nullptr; size_t red_rows = 0;
    // host-buffer loss call: targets, greedy tokens and row losses of the whole batch on the device
    long long* loss_targets = nullptr; int* loss_argmax = nullptr; float* loss_rows = nullptr; size_t loss_cap = 0;
};

// What replaces the logits when the LM head is fused with the step after it (cross_entropy_loss(_ignore_index), core-ops/src/lib.rs:1079-1194;
// the greedy token = first candidate of sampling_candidates, nn/src/lib.rs:2381-2418): per-row loss and / or the column of the row maximum.
struct HeadReduce { const long long* targets; int has_ignore; long long ignore_index; int* argmax; float* row_loss; };

struct ParamInfo { std::string name; std::vector<size_t> shape; };

// ---- gpt.cu, used by both drivers ----
void drop_graphs(Gpt* g);                       // captured launches hold addresses and grids that are about to change
void gfree(Gpt* g, void* p);
void* galloc(Gpt* g, size_t bytes);             // owned by the model
// host f32 -> device in the model dtype (bf16: round to nearest even on the device); returns with the host buffer free again
int upload_rows(Gpt* g, void* dst_model_dtype, const float* host, size_t n);
int gemm_or_simt(const GemmDesc& d);
int lm_head(Gpt* g, const void* h, int M, void* logits, const HeadReduce* hr);

}  // namespace spt
