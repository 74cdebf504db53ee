// attention_fused.cu -- fused causal attention for bf16, head_dim 64 or 128 (sm_100a, tcgen05 + TMEM + TMA).
//
// Same function as crates/nn/src/lib.rs:600-637 (scores = Q K^T * 1/sqrt(hd); entries j > i set to -inf; row
// softmax; P V; heads merged back) but the [T,T] score and probability matrices never reach HBM, and the head
// split / merge and the K transpose (nn/src/lib.rs:763-793, 822-850, 879-903) are strides of the tensor maps.
//
// One CTA owns TWO 128-row query tiles of one (sequence, head) at a time and walks the 128-key tiles up to the
// diagonal with a running row maximum and row sum (the softmax is exact; only the order of the sums differs):
//
//   warp 0      TMA: both Q tiles once per work item, then per key tile K [128 keys, hd] and V [128 keys, hd]
//               (V in its natural token-major layout: it is the MN-major B operand of P V, no transposed copy)
//   warp 1      tcgen05.mma, one lane: S_g = Q_g K_j^T (M128 N128) into the TMEM buffer of tile g, and
//               O_g += P_g V_j with P read straight from TMEM; the two query tiles alternate, so the tensor
//               core works on one tile while the softmax warps work on the other
//   warps 2..5  softmax of query tile 0, warps 6..9 of query tile 1: ONE THREAD PER QUERY ROW.  A thread reads
//               its 128 scores from TMEM in four chunks of 32 (the next chunk's load in flight while one is worked on;
//               the running row maximum is the thread's own business, no other thread has a part in it), evaluates
//               2^(s*c - m*c) on the special-function unit, and writes P as bf16 back into the TMEM columns the scores
//               came from
// O accumulates in TMEM over the key tiles of an item and is rescaled in place only when a row maximum grows by
// more than 2^8 (lazy rescaling).  TMEM, head size 128: S/P of tile 0 at columns 0..127, of tile 1 at 128..255, O_0 at 256,
// O_1 at 384 (512 columns, one CTA per SM).  Head size 64 (accumulators of 64 columns): THREE score buffers at 0 / 128 / 256
// that the Q K^T products take in turn, O_0 at 384, O_1 at 448 -- a tile's next scores are ready before its softmax warps
// have finished the current ones.
// The same kernel serves latent attention (latent_attention.cu) once a prompt's keys and values are expanded: a score is then the sum of
// two products over separately stored parts -- the head's own D columns and a rotated part all heads share -- queries may start at a
// position `first` > 0 behind cached keys, values may be narrower or wider than the keys, and head h's output carries the factor
// sigmoid(gate_h).  There the softmax weights enter P V as the sum of two bf16 numbers (PSPLIT: 16 mantissa bits instead of 8; the
// second half sits in the score columns the first leaves free), so that the weights keep close to f32 precision.
// And window attention (WIN; window_attention.cu): several query heads read one key/value head, row i sees the last `window` keys up to
// its own, a score carries the distance bias - slope_h (i - j), and the output is multiplied element by element with a sigmoid.  A work
// item then walks the visible key tiles, and every tile's chunks, from the diagonal BACKWARDS: the bias makes near keys large and far
// ones small, so the maxima a row starts with stay, where a forward walk would rescale at nearly every chunk.  Query tile 0 joins one
// step late when its diagonal is one tile before query tile 1's; tile 1 leaves one step early when its window begins one tile later.
// Algorithmic work per (sequence, head): 2 * T(T+1) * hd FLOP; HBM traffic: Q, K, V read once per query tile
// (K/V re-reads hit L2 thanks to the work schedule below), O written once.
#include "gemm.h"
#include "sm100.cuh"
#include "../../include/sptorch_b200_ext.h"
#include <algorithm>
#include <array>
#include <type_traits>
#include <cstdlib>
#include <map>
#include <mutex>
#include <queue>
#include <vector>

namespace spt {

using namespace sm100;

constexpr int kAttnThreads = 320;           // TMA warp + MMA warp + 2 x 4 softmax warps
constexpr int kQTile = 128, kKvTile = 128;
constexpr int kQPair = 2 * kQTile;          // query rows per work item

struct AttnParams {
    __nv_bfloat16* out;
    long long ld_out;       // row stride of out in elements
    int T, H, B;            // T query rows per sequence, at positions first .. first + T - 1
    int n, first;           // keys 0 .. n - 1 per sequence
    int V;                  // width of a head's output in memory (at most the template's VD)
    int n_ptiles;           // 256-row query tile pairs per sequence
    float scale_log2;       // factor of the scores * log2(e)
    const __nv_bfloat16* gate;      // when given: head h of token m is multiplied by sigmoid(gate[m * ld_gate + h]); WIN: element by
    long long ld_gate;              // element, laid out like out (and may be out)
    int group, window;              // WIN: query heads per key/value head; keys a row sees
    const float* slopes;            // WIN: [H] or null
    uint32_t* status;
    const int* sched;       // work schedule [sched_len][gridDim.x]: item of CTA c at step k, -1 past the end of its list; null: items c, c + grid, ..
    int sched_len;
};

// 2^x on the special-function unit: one instruction, relative error 2^-22 (P is rounded to bf16 right after)
__device__ __forceinline__ float ex2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ float max3(float a, float b, float c) {
    float d;
    asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
    return d;
}

// two f32 as the sums of two bf16 each: hi and what hi misses (together 16 mantissa bits)
__device__ __forceinline__ void split2(float2 e, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h2 = __floats2bfloat162_rn(e.x, e.y);
    hi = *reinterpret_cast<const uint32_t*>(&h2);
    const float2 f = bf16x2_to_float2(h2);
    const __nv_bfloat162 l2 = __floats2bfloat162_rn(e.x - f.x, e.y - f.y);
    lo = *reinterpret_cast<const uint32_t*>(&l2);
}

// 32 lanes x 16 consecutive 32-bit columns: thread i of the warp owns lane (base_lane + i)
__device__ __forceinline__ void tmem_ld_32x32b_x16(uint32_t taddr, uint32_t (&r)[16]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
          "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(taddr)
        : "memory");
}
__device__ __forceinline__ void tmem_st_32x32b_x16(uint32_t taddr, const uint32_t (&r)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
          "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
        : "memory");
}

// tcgen05.mma with the A operand in TMEM (rows = lanes, two bf16 per 32-bit column) and B in shared memory
__device__ __forceinline__ void mma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}\n"
        ::"r"(d_tmem), "r"(a_tmem), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}

// Shared-memory descriptor of an MN-major operand tile stored as k-rows of exactly 128 bytes (64 bf16 along the MN
// dimension) with the 128-byte swizzle: what a TMA box of {64 elements, rows} writes for a row-major [k, n] matrix.
//   leading byte offset = distance between 64-element chunks along MN (for N = 128: the second TMA box)
//   stride byte offset  = distance between groups of 8 k-rows = 1024 B
// Advancing along K by one MMA (16 rows) adds 2048 B to the start address.
__device__ __forceinline__ uint64_t make_mnmajor_sw128_desc(uint32_t smem_addr, uint32_t chunk_bytes) {
    uint64_t d = 0;
    d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
    d |= (uint64_t)(chunk_bytes >> 4) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}

// KBN / KBR: 64-column blocks of the heads' own query/key part and of the shared part; VD: value columns
template <int KBN, int KBR, int VD>
struct AttnSmem {
    static constexpr int KB = KBN + KBR;
    static constexpr int kKStages = KB == 1 ? 4 : KB == 2 && VD == 64 && KBR == 1 ? 3 : 2;
    static constexpr int kVStages = KB == 3 && VD == 128 ? 1 : kKStages;
    static constexpr int kQTileBytes = KB * kQTile * 128;     // k-blocks of [128 rows x 128 B]
    static constexpr int kKBytes = KB * kKvTile * 128;        // k-blocks of [128 keys x 128 B]
    static constexpr int kVBytes = kKvTile * VD * 2;          // VD/64 chunks of [128 keys x 128 B] (64 head columns each)
    static constexpr int kQ = 0;
    static constexpr int kK = kQ + 2 * kQTileBytes;
    static constexpr int kV = kK + kKStages * kKBytes;
    static constexpr int kBars = kV + kVStages * kVBytes;     // mbarriers + TMEM slot + abort flag
    static constexpr int kBarBytes = 320;
    static constexpr int kTotal = kBars + kBarBytes;
    static_assert(kTotal <= 227 * 1024, "shared memory");
};

// Persistent kernel: CTA c works through column c of a schedule built on the host (attention_schedule below), and all
// roles run straight through item boundaries (barrier phases are driven by running counters), so the loads and the
// first Q K^T of the next item are in flight while the current one drains.
template <int KBN, int KBR, int VD, bool ROTP, bool PSPLIT, bool WIN = false>
__global__ void __launch_bounds__(kAttnThreads, 1)
attn_fused_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                  const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmQr, const __grid_constant__ CUtensorMap tmKr,
                  const AttnParams p) {
    using L = AttnSmem<KBN, KBR, VD>;
    constexpr uint32_t TMEM_COLS = 512;
    constexpr uint32_t IDESC_S = make_idesc(false, 128, kKvTile);
    constexpr uint32_t IDESC_O = make_idesc(false, 128, VD) | (1u << 16);      // B operand (V) is MN-major
    constexpr int KB = L::KB;                                 // 128-byte blocks along the query/key width
    constexpr int NSK = L::kKStages, NSV = L::kVStages;       // rings of key and of value tiles

    extern __shared__ __align__(1024) uint8_t smem[];
    const uint32_t base = smem_u32(smem);
    const uint32_t bar = base + L::kBars;
    const uint32_t q_full = bar;                    // 1
    const uint32_t q_free = q_full + 8;             // 1
    const uint32_t k_full = q_free + 8;             // NSK
    const uint32_t k_empty = k_full + 8 * NSK;      // NSK
    const uint32_t v_full = k_empty + 8 * NSK;      // NSV
    const uint32_t v_empty = v_full + 8 * NSV;      // NSV
    // Head size 64 leaves 128 TMEM columns free beside two score tiles and two 64-column accumulators: a THIRD score buffer.  The
    // three buffers go round robin to the Q K^T products in issue order (tile 0 / tile 1 alternating), so a query tile's next
    // scores are computed while its softmax warps are still on the current ones, and the softmax never waits for the tensor core
    // (ROT).  Head size 128 fills the 512 columns with two score tiles and two accumulators: buffer = query tile, as before.
    constexpr bool ROT = VD == 64 && ROTP;
    constexpr int NSB = ROT ? 3 : 2;                // score buffers
    constexpr uint32_t O_COL = ROT ? 384 : 256;     // first accumulator column
    constexpr uint32_t O_STRIDE = ROT ? 64 : 128;
    // Scores ready.  With rotating buffers: four barriers per query tile, taken in turn by the tile's own steps (index step & 3, phase
    // step >> 2): up to three of a tile's scores may be complete before its softmax takes the first, and a barrier that only this
    // tile's steps advance cannot be passed, or missed, because of what the other tile did meanwhile (an item may have no second tile).
    // One barrier per tile otherwise.
    const uint32_t s_full = v_empty + 8 * NSV;      // 8: [query tile][step & 3]
    const uint32_t p_full = s_full + 8 * 8;         // NSB
    // P V products done: two barriers per query tile, taken in turn by the tile's steps (index step & 1, phase step >> 1).  With
    // rotating score buffers a tile's softmax can finish step j before P V of step j - 1 has completed, so its wait for the
    // product of step j on a single barrier would be two phases ahead -- which a parity wait cannot tell from none; on the
    // barrier of its own parity class it is never more than one phase ahead (the product of step j + 2 needs this thread's P).  With one
    // query tile in the item the softmax can be a step further ahead; its end has a wait of its own for that (below).
    const uint32_t pv_done = p_full + 8 * 3;        // 4: [query tile][step & 1]
    const uint32_t o_free = pv_done + 32;           // 2
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + L::kBars + L::kBarBytes - 16);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + L::kBars + L::kBarBytes - 12);
    static_assert(8 * (2 + 2 * NSK + 2 * NSV + 17) <= L::kBarBytes - 16, "barrier block overflows");

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int BH = p.B * p.H;
    const int n_kv_seq = (p.n + kKvTile - 1) / kKvTile;

    if ((base & 1023u) != 0) {                                // swizzled tiles need 1024-byte alignment
        if (threadIdx.x == 0) atomicOr(p.status, 0x200u);
        return;
    }
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1); mbar_init(q_free, 1);
        for (int s = 0; s < NSK; s++) { mbar_init(k_full + 8 * s, 1); mbar_init(k_empty + 8 * s, 1); }
        for (int s = 0; s < NSV; s++) { mbar_init(v_full + 8 * s, 1); mbar_init(v_empty + 8 * s, 1); }
        for (int g = 0; g < 8; g++) mbar_init(s_full + 8 * g, 1);
        for (int g = 0; g < 3; g++) mbar_init(p_full + 8 * g, 4);           // one arrival per softmax warp of the tile
        for (int g = 0; g < 4; g++) mbar_init(pv_done + 8 * g, 1);
        for (int g = 0; g < 2; g++) mbar_init(o_free + 8 * g, 4);
        *abort_flag = 0;
        fence_barrier_init();
    }
    if (warp == 1) { tmem_alloc(smem_u32(tmem_slot), TMEM_COLS); tmem_relinquish(); }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;

    // step k of this CTA's list; the entry of the next step is fetched while the current item runs
    auto fetch = [&](int k) -> int {
        if (k >= p.sched_len) return -1;
        const int at = k * (int)gridDim.x + (int)blockIdx.x;
        return p.sched ? __ldg(p.sched + at) : at < p.n_ptiles * BH ? at : -1;
    };
    // work item -> (first query row, sequence, head); steps 0 .. N - 1 go over the key tiles (WIN: from k_last down, otherwise from 0 up);
    // query tile 0 takes part in steps b0 .. e0 - 1 (b0 = 0 without WIN), tile 1 in steps 0 .. e1 - 1
    struct Item {
        int q0, bb, hh, N, k_last, b0, e0, e1;
        __device__ __forceinline__ int key_tile(int step) const { return WIN ? k_last - step : step; }
        __device__ __forceinline__ int begin(int t) const { return WIN && t == 0 ? b0 : 0; }
        __device__ __forceinline__ int end(int t) const { return t == 0 ? e0 : e1; }
    };
    auto decode = [&](int item) -> Item {
        Item w;
        const int pt = p.n_ptiles - 1 - item / BH;
        const int bh = item % BH;
        w.bb = bh / p.H; w.hh = bh % p.H;
        w.q0 = pt * kQPair;
        const int last0 = min((p.first + w.q0 + kQTile - 1) / kKvTile, n_kv_seq - 1);               // causal: keys 0 .. first+q0+127
        const int last1 = (w.q0 + kQTile < p.T) ? min((p.first + w.q0 + 2 * kQTile - 1) / kKvTile, n_kv_seq - 1) : -1;      // second tile exists only inside the sequence
        const int last = max(last0, last1);
        if constexpr (WIN) {
            const int from0 = max(0, p.first + w.q0 - p.window + 1) / kKvTile, from1 = max(0, p.first + w.q0 + kQTile - p.window + 1) / kKvTile;
            w.N = w.e0 = last - from0 + 1; w.k_last = last; w.b0 = last - last0;
            w.e1 = last1 < 0 ? 0 : last - from1 + 1;
        } else {
            w.N = last + 1; w.k_last = 0; w.b0 = 0;
            w.e0 = last0 + 1; w.e1 = last1 + 1;
        }
        return w;
    };
    // the products of an item in issue order: step by step, query tile 0 before query tile 1 where both take part
    auto entries = [&](const Item& w) -> int { return w.e0 - w.begin(0) + w.e1; };
    auto entries_before = [&](const Item& w, int t, int j) -> int {
        if constexpr (WIN) return max(0, (t == 1 ? j + 1 : j) - w.b0) + min(j, w.e1);       // tile 0 stays to the last step
        else return min(j, w.e0) + min(j, w.e1) + ((t == 1 && j < w.e0) ? 1 : 0);
    };

    if (warp == 0) {
        // ---------------- TMA producer ----------------
        if (lane == 0) { tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV); }
        if (KBR > 0 && lane == 0) { tma_prefetch_desc(&tmQr); tma_prefetch_desc(&tmKr); }
        bool ok = true;
        uint32_t g = 0, it = 0;
        for (int k = 0, item = fetch(0); item >= 0 && ok; k++, it++) {
            const int item_next = fetch(k + 1);
            const Item w = decode(item);
            item = item_next;
            const int q0 = w.q0, bb = w.bb, hh = w.hh, nmax = w.N, kh = WIN ? hh / p.group : hh;
            ok = mbar_wait(q_free, (it & 1) ^ 1, abort_flag, p.status, kErrProducerWait);
            if (!ok) break;
            if (lane == 0) {
                mbar_expect_tx(q_full, 2 * L::kQTileBytes);
                for (int t = 0; t < 2; t++) {
                    const uint32_t dst = base + L::kQ + t * L::kQTileBytes;
                    for (int kb = 0; kb < KBN; kb++) tma_load_4d(dst + kb * (kQTile * 128), &tmQ, q_full, kb * 64, q0 + t * kQTile, hh, bb);
                    for (int kb = 0; kb < KBR; kb++) tma_load_4d(dst + (KBN + kb) * (kQTile * 128), &tmQr, q_full, kb * 64, q0 + t * kQTile, hh, bb);
                }
            }
            // keys run one tile ahead of the values: K_0, K_1, V_0, K_2, V_1, ... (the next scores are what the tensor core asks for first)
            for (int j = 0; j <= nmax && ok; j++) {
                if (j < nmax) {
                    const uint32_t gk = g + j, s = gk % NSK;
                    ok = mbar_wait(k_empty + 8 * s, ((gk / NSK) & 1) ^ 1, abort_flag, p.status, kErrProducerWait);
                    if (!ok) break;
                    if (lane == 0) {
                        const uint32_t dst = base + L::kK + s * L::kKBytes;
                        mbar_expect_tx(k_full + 8 * s, L::kKBytes);
                        for (int kb = 0; kb < KBN; kb++) tma_load_4d(dst + kb * (kKvTile * 128), &tmK, k_full + 8 * s, kb * 64, w.key_tile(j) * kKvTile, kh, bb);
                        for (int kb = 0; kb < KBR; kb++) tma_load_4d(dst + (KBN + kb) * (kKvTile * 128), &tmKr, k_full + 8 * s, kb * 64, w.key_tile(j) * kKvTile, 0, bb);
                    }
                    __syncwarp();
                }
                if (j > 0) {
                    const uint32_t gv = g + j - 1, s = gv % NSV;
                    ok = mbar_wait(v_empty + 8 * s, ((gv / NSV) & 1) ^ 1, abort_flag, p.status, kErrProducerWait);
                    if (!ok) break;
                    if (lane == 0) {
                        const uint32_t dst = base + L::kV + s * L::kVBytes;
                        mbar_expect_tx(v_full + 8 * s, L::kVBytes);
                        for (int kb = 0; kb < VD / 64; kb++) tma_load_4d(dst + kb * (kKvTile * 128), &tmV, v_full + 8 * s, kb * 64, w.key_tile(j - 1) * kKvTile, kh, bb);
                    }
                    __syncwarp();
                }
            }
            g += nmax;
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        bool ok = true;
        uint32_t g = 0, it = 0;                 // key tiles loaded so far (stage ring position); items so far
        uint32_t outs[2] = {0, 0};              // items so far that each query tile had a part in (phases of o_free)
        uint32_t steps[2] = {0, 0};             // softmax steps of each query tile so far (phases of p_full)
        // 16 keys per product: 8 columns of P, or with PSPLIT 8 columns of each half (a chunk of 32 keys is 16 + 16 columns)
        auto mma_pv = [&](int t, uint32_t p_addr, uint64_t bdesc, bool accumulate) {
#pragma unroll
            for (int k = 0; k < kKvTile / 16; k++) {
                const uint32_t o = tmem_base + O_COL + t * O_STRIDE, a = PSPLIT ? p_addr + 32 * (k / 2) + 8 * (k % 2) : p_addr + 8 * k;
                mma_ts(o, a, bdesc + (uint64_t)(128 * k), IDESC_O, (accumulate || k != 0) ? 1u : 0u);
                if (PSPLIT) mma_ts(o, a + 16, bdesc + (uint64_t)(128 * k), IDESC_O, 1u);
            }
        };
        // S_t = Q_t K^T with the key tile of ring position gg
        auto issue_s = [&](int t, uint32_t gg) {
            const uint32_t kaddr = base + L::kK + (gg % NSK) * L::kKBytes;
#pragma unroll
            for (int kb = 0; kb < KB; kb++) {
                const uint64_t adesc = make_kmajor_sw128_desc(base + L::kQ + t * L::kQTileBytes + kb * (kQTile * 128));
                const uint64_t bdesc = make_kmajor_sw128_desc(kaddr + kb * (kKvTile * 128));
#pragma unroll
                for (int k = 0; k < 4; k++) mma_ss<false>(tmem_base + t * 128, adesc + 2 * k, bdesc + 2 * k, IDESC_S, (kb | k) != 0 ? 1u : 0u);
            }
            mma_commit(s_full + 32 * t);
        };
        // O_t (+)= P_t V with the value tile of ring position gg; P is read from the TMEM columns of S_t
        auto issue_pv = [&](int t, uint32_t gg, bool accumulate, uint32_t pvidx) {      // pvidx: which product of this tile (over the whole kernel)
            const uint64_t bdesc = make_mnmajor_sw128_desc(base + L::kV + (gg % NSV) * L::kVBytes, kKvTile * 128);
            mma_pv(t, tmem_base + t * 128, bdesc, accumulate);
            mma_commit(pv_done + 8 * (2 * t + (pvidx & 1)));
        };
        auto k_ready = [&](uint32_t gg) -> bool { return mbar_wait(k_full + 8 * (gg % NSK), (gg / NSK) & 1, abort_flag, p.status, kErrMmaWait); };
        auto v_ready = [&](uint32_t gg) -> bool { return mbar_wait(v_full + 8 * (gg % NSV), (gg / NSV) & 1, abort_flag, p.status, kErrMmaWait); };
        if constexpr (ROT) {
            // The products of an item in issue order ("entries"): key tile by key tile, query tile 0 before query tile 1 where both
            // still have that key tile.  Scores run up to two entries ahead of the P V product that is issued next; score number n
            // (counted over the whole kernel) lives in buffer n % 3, which P V number n - 3 -- issued earlier by this thread, and
            // the tensor pipe runs one thread's MMAs in order -- has finished reading.
            uint32_t G = 0;                     // scores issued in earlier items
            uint32_t scored[2] = {0, 0};        // scores issued so far of each query tile
            auto issue_s3 = [&](int t, uint32_t gg, uint32_t n, uint32_t own) {
                const uint32_t buf = n % 3;
                const uint32_t kaddr = base + L::kK + (gg % NSK) * L::kKBytes;
#pragma unroll
                for (int kb = 0; kb < KB; kb++) {
                    const uint64_t adesc = make_kmajor_sw128_desc(base + L::kQ + t * L::kQTileBytes + kb * (kQTile * 128));
                    const uint64_t bdesc = make_kmajor_sw128_desc(kaddr + kb * (kKvTile * 128));
#pragma unroll
                    for (int k = 0; k < 4; k++) mma_ss<false>(tmem_base + buf * 128, adesc + 2 * k, bdesc + 2 * k, IDESC_S, (kb | k) != 0 ? 1u : 0u);
                }
                mma_commit(s_full + 8 * (4 * t + (own & 3)));
            };
            auto issue_pv3 = [&](int t, uint32_t gg, uint32_t n, bool accumulate, uint32_t pvidx) {
                const uint32_t buf = n % 3;
                const uint64_t bdesc = make_mnmajor_sw128_desc(base + L::kV + (gg % NSV) * L::kVBytes, kKvTile * 128);
                mma_pv(t, tmem_base + buf * 128, bdesc, accumulate);
                mma_commit(pv_done + 8 * (2 * t + (pvidx & 1)));
            };
            for (int k = 0, item = fetch(0); item >= 0 && ok; k++, it++) {
                const int item_next = fetch(k + 1);
                const Item w = decode(item);
                item = item_next;
                // before joined_0 tile 1 is alone, from joined_1 on the tile that has more
                const int E = entries(w), joined_0 = w.begin(0), joined_1 = max(joined_0, min(w.e0, w.e1)), two = 2 * joined_1 - joined_0, t_long = w.e1 > w.e0 ? 1 : 0;
                auto entry = [&](int e, int& t, int& j) {
                    if (WIN && e < joined_0) { j = e; t = 1; }
                    else if (e < two) { j = (e + joined_0) >> 1; t = (e + joined_0) & 1; }
                    else { j = joined_1 + (e - two); t = t_long; }
                };
                ok = mbar_wait(q_full, it & 1, abort_flag, p.status, kErrMmaWait);
                if (!ok) break;
                int issued = 0, k_seen = -1, v_seen = -1;
                for (int e = 0; e < E && ok; e++) {
                    while (issued < min(E, e + 3)) {
                        int ts, js;
                        entry(issued, ts, js);
                        if (js > k_seen) { ok = k_ready(g + js); k_seen = js; if (!ok) break; }
                        tc_fence_after();
                        int tn = 0, jn = -1;
                        if (issued + 1 < E) entry(issued + 1, tn, jn);
                        if (elect_one_sync()) {
                            issue_s3(ts, g + js, G + issued, ts ? scored[1] : scored[0]);
                            if (jn != js) mma_commit(k_empty + 8 * ((g + js) % NSK));            // every product that reads these keys has been issued
                            if (issued == E - 1) mma_commit(q_free);            // the item's last read of Q
                        }
                        __syncwarp();
                        if (ts) scored[1]++; else scored[0]++;
                        issued++;
                    }
                    if (!ok) break;
                    int t, j;
                    entry(e, t, j);
                    const uint32_t n = G + e, buf = n % 3;
                    ok = mbar_wait(p_full + 8 * buf, (n / 3) & 1, abort_flag, p.status, kErrMmaWait);
                    // the item's first product overwrites the accumulator: the previous item's output must have been read
                    if (ok && j == w.begin(t)) { ok = mbar_wait(o_free + 8 * t, ((t ? outs[1] : outs[0]) & 1) ^ 1, abort_flag, p.status, kErrMmaWait); if (t) outs[1]++; else outs[0]++; }
                    if (ok && j > v_seen) { ok = v_ready(g + j); v_seen = j; }
                    if (!ok) break;
                    tc_fence_after();
                    int tn = 0, jn = -1;
                    if (e + 1 < E) entry(e + 1, tn, jn);
                    if (elect_one_sync()) {
                        issue_pv3(t, g + j, n, j > w.begin(t), steps[t]);
                        if (jn != j) mma_commit(v_empty + 8 * ((g + j) % NSV));     // every MMA that reads these values has been issued
                    }
                    __syncwarp();
                    steps[t]++;
                }
                g += w.N;
                G += E;
            }
        } else
        for (int k = 0, item = fetch(0); item >= 0 && ok; k++, it++) {
            const int item_next = fetch(k + 1);
            const Item w = decode(item);
            item = item_next;
            const int nmax = w.N;
            ok = mbar_wait(q_full, it & 1, abort_flag, p.status, kErrMmaWait) && k_ready(g);
            if (!ok) break;
            tc_fence_after();
            if (elect_one_sync()) {
                for (int t = 0; t < 2; t++) if (w.begin(t) == 0 && w.end(t) > 0) issue_s(t, g);
                if (nmax == 1) mma_commit(q_free);          // the item's last read of Q
                mma_commit(k_empty + 8 * (g % NSK));
            }
            __syncwarp();
            for (int j = 0; j < nmax && ok; j++, g++) {
                ok = (j + 1 >= nmax || k_ready(g + 1)) && v_ready(g);
                if (!ok) break;
                for (int t = 0; t < 2 && ok; t++) {
                    if (j >= w.end(t)) continue;
                    if (j < w.begin(t)) {                          // joins at the next step: only its first scores
                        tc_fence_after();
                        if (elect_one_sync()) issue_s(t, g + 1);
                        __syncwarp();
                        continue;
                    }
                    ok = mbar_wait(p_full + 8 * t, steps[t] & 1, abort_flag, p.status, kErrMmaWait);
                    // the item's first product overwrites the accumulator: the previous item's output must have been read
                    if (ok && j == w.begin(t)) { ok = mbar_wait(o_free + 8 * t, ((t ? outs[1] : outs[0]) & 1) ^ 1, abort_flag, p.status, kErrMmaWait); if (t) outs[1]++; else outs[0]++; }
                    if (!ok) break;
                    steps[t]++;
                    tc_fence_after();
                    if (elect_one_sync()) {
                        issue_pv(t, g, j > w.begin(t), steps[t] - 1);
                        // the next scores of this tile go into the columns P was just read from: the tensor pipe runs the
                        // MMAs of one thread in order, so the product above has consumed P before these overwrite it
                        if (j + 1 < w.end(t)) issue_s(t, g + 1);
                    }
                    __syncwarp();
                }
                if (ok && elect_one_sync()) {                   // every MMA that reads V_j, and K_(j+1), has been issued
                    mma_commit(v_empty + 8 * (g % NSV));
                    if (j + 1 < nmax) mma_commit(k_empty + 8 * ((g + 1) % NSK));
                    if (j + 2 == nmax) mma_commit(q_free);
                }
                __syncwarp();
            }
        }
    } else {
        // ---------------- softmax + output: one thread per query row ----------------
        const int t = (warp - 2) >> 2;                           // query tile of this warp
        const int quarter = warp & 3;                            // TMEM lane quarter a warp may access = warp index % 4
        const int r = quarter * 32 + lane;                       // row inside the tile = TMEM lane
        const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
        const uint32_t o_addr = tmem_base + lane_off + O_COL + t * O_STRIDE;
        bool ok = true;
        uint32_t step = 0;                                       // softmax steps of this tile so far
        uint32_t G = 0;                                          // ROT: scores of earlier items (both tiles), as the MMA warp counts them
        for (int k = 0, item = fetch(0); item >= 0 && ok; k++) {
            const int item_next = fetch(k + 1);
            const Item w = decode(item);
            item = item_next;
            const int q0 = w.q0, bb = w.bb, hh = w.hh, j_first = w.begin(t), n_kv = w.end(t);
            const int qrow = q0 + t * kQTile + r;
            // WIN: kUnseen until the row's first visible key (masked scores are -inf: their weights and sums are then zeros)
            constexpr float kUnseen = -1e30f;
            float m = WIN ? kUnseen : -INFINITY, l = 0.0f;
            const float slope = WIN && p.slopes ? __ldg(p.slopes + hh) * 1.4426950408889634f : 0.0f;
            for (int j = j_first; j < n_kv && ok; j++, step++) {
                // ROT: this step's scores are number G + (entries of the item before (t, j)) of the kernel, in buffer number % 3
                const uint32_t sn = ROT ? G + (uint32_t)entries_before(w, t, j) : step;
                const uint32_t sbuf = ROT ? sn % 3 : (uint32_t)t;
                const uint32_t s_addr = tmem_base + lane_off + sbuf * 128;          // scores, and P over their first 64 columns
                ok = mbar_wait(s_full + 8 * (4 * t + (ROT ? step & 3 : 0)), (ROT ? step >> 2 : step) & 1, abort_flag, p.status, kErrEpilogueWait);
                if (!ok) break;
                tc_fence_after();
                // row r of the tile sees the keys of this tile up to column r + delta
                const int delta = p.first + q0 + t * kQTile - w.key_tile(j) * kKvTile;
                // ... and (WIN) from column r + delta - window + 1 on
                const bool diag = delta < kKvTile - 1 || (WIN && delta > p.window - kQTile);
                // The 128 scores of the row are taken in four chunks of 32: the load of chunk c + 1 is in flight while chunk c is
                // worked on, and a chunk needs only 32 registers.  The reference maximum m of the row is allowed to lag the true
                // maximum by up to 2^8 (lazy rescaling): a chunk whose maximum exceeds m by more moves m, and everything already
                // accumulated under the old m -- the row sum, the output in TMEM, and the chunks of P of this tile that are already
                // written -- is multiplied by 2^(old - new) at that moment.  tcgen05.ld / st are warp-wide, so a warp rescales when any
                // of its rows does (the others multiply by one).
                float2 sum_a = make_float2(0.0f, 0.0f), sum_b = make_float2(0.0f, 0.0f);
                // WIN: m is in units of the exponent, and the maximum of a chunk is estimated as that of the unbiased scores plus the bias of the
                // chunk's nearest key: too high by at most the bias of 31 keys (2^45), which a row sum in f32 does not notice
                const float mul = WIN ? 1.0f : p.scale_log2;
                const float2 c2 = make_float2(p.scale_log2, p.scale_log2);
                uint32_t va[32], vb[32];
                tmem_ld_32x32(s_addr + (WIN ? 96 : 0), va);
                auto chunk = [&](auto c_tag, uint32_t (&v)[32], uint32_t (&vnext)[32], auto diag_tag) -> bool {
                    const int n = c_tag;                               // chunks before this one
                    auto column_chunk = [](int i) { return WIN ? 3 - i : i; };
                    const int c = column_chunk(n);
                    constexpr bool DIAG = decltype(diag_tag)::value;
                    tmem_ld_wait();
                    if (n < 3) tmem_ld_32x32(s_addr + column_chunk(n + 1) * 32, vnext);
                    if (DIAG) {
#pragma unroll
                        for (int i = 0; i < 32; i++)
                            if (i > r + delta - c * 32 || (WIN && i <= r + delta - c * 32 - p.window)) v[i] = 0xff800000u;       // -inf right of the diagonal
                    }
                    float m0 = -INFINITY, m1 = -INFINITY, m2 = -INFINITY, m3 = -INFINITY;
#pragma unroll
                    for (int i = 0; i < 32; i += 8) {
                        m0 = max3(m0, __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
                        m1 = max3(m1, __uint_as_float(v[i + 2]), __uint_as_float(v[i + 3]));
                        m2 = max3(m2, __uint_as_float(v[i + 4]), __uint_as_float(v[i + 5]));
                        m3 = max3(m3, __uint_as_float(v[i + 6]), __uint_as_float(v[i + 7]));
                    }
                    float mx = fmaxf(max3(m0, m1, m2), m3);
                    const float bias0 = WIN ? slope * (float)(c * 32 - r - delta) : 0.0f;          // of the chunk's first key
                    if constexpr (WIN) mx = fmaf(mx, p.scale_log2, fminf(fmaf(31.0f, slope, bias0), 0.0f));
                    if constexpr (WIN) { if (m == kUnseen) m = fmaxf(mx, kUnseen); }     // everything accumulated so far is zero: nothing to rescale
                    else if (j == 0 && n == 0) m = mx;               // the first chunk of a row always holds key 0: finite
                    const bool grow = (mx - m) * mul > 8.0f;
                    if (__any_sync(0xffffffffu, grow)) {
                        tmem_ld_wait();                          // the next chunk's registers may be moved below: they must have arrived
                        float alpha = 1.0f;
                        if (grow) { alpha = ex2_approx((m - mx) * mul); m = mx; }
                        l *= alpha;
                        sum_a.x *= alpha; sum_a.y *= alpha; sum_b.x *= alpha; sum_b.y *= alpha;
                        if (j > j_first) {
                            // every product accumulated so far is in place (the commit of step - 1; the next one needs this thread's P)
                            if (!mbar_wait(pv_done + 8 * (2 * t + ((step - 1) & 1)), ((step - 1) >> 1) & 1, abort_flag, p.status, kErrEpilogueWait)) return false;
                            __syncwarp();                        // the wait's lanes leave it one by one, the loads below are warp-wide
                            tc_fence_after();
#pragma unroll 1
                            for (int cc = 0; cc < VD / 32; cc++) {       // the rare path: small code counts for more than unrolled loops
                                uint32_t o[32];
                                tmem_ld_32x32(o_addr + cc * 32, o);
                                tmem_ld_wait();
#pragma unroll
                                for (int i = 0; i < 32; i++) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                                tmem_st_32x32(o_addr + cc * 32, o);
                            }
                        }
                        if (n > 0) tmem_st_wait();               // P's chunks have landed before they are read back
                        if (n > 0 && PSPLIT) {
                            uint32_t u[32];
#pragma unroll 1
                            for (int cc = 0; cc < n; cc++) {
                                tmem_ld_32x32(s_addr + column_chunk(cc) * 32, u);
                                tmem_ld_wait();
#pragma unroll
                                for (int i = 0; i < 16; i++) {
                                    const float lo = (__uint_as_float(u[i] << 16) + __uint_as_float(u[i + 16] << 16)) * alpha;
                                    const float hi = (__uint_as_float(u[i] & 0xffff0000u) + __uint_as_float(u[i + 16] & 0xffff0000u)) * alpha;
                                    split2(make_float2(lo, hi), u[i], u[i + 16]);
                                }
                                tmem_st_32x32(s_addr + column_chunk(cc) * 32, u);
                            }
                        } else if (n > 0) {
                            // the chunks of P of this tile written so far: 16 columns (32 bf16) each
                            uint32_t u[16];
#pragma unroll 1
                            for (int cc = 0; cc < n; cc++) {
                                tmem_ld_32x32b_x16(s_addr + cc * 16, u);
                                tmem_ld_wait();
#pragma unroll
                                for (int i = 0; i < 16; i++) {
                                    const float lo = __uint_as_float(u[i] << 16) * alpha, hi = __uint_as_float(u[i] & 0xffff0000u) * alpha;
                                    __nv_bfloat162 h2 = __floats2bfloat162_rn(lo, hi);
                                    u[i] = *reinterpret_cast<uint32_t*>(&h2);
                                }
                                tmem_st_32x32b_x16(s_addr + cc * 16, u);
                            }
                        }
                        tmem_st_wait();
                        // the load of the next chunk was issued before this branch: the wait of the next chunk() call still covers it
                    }
                    const float mb = m * mul;
                    const float2 nmb2 = make_float2(-mb, -mb);
                    const float2 two_slopes = make_float2(2.0f * slope, 2.0f * slope);
                    float2 add = nmb2;                           // what the scaled scores of keys 2i, 2i + 1 lack to the exponent
                    uint32_t packed[PSPLIT ? 32 : 16];
#pragma unroll
                    for (int i = 0; i < 16; i++) {
                        if constexpr (WIN) {
                            if (i % 4 == 0) { add.x = fmaf(2.0f * i, slope, bias0 - mb); add.y = add.x + slope; }
                            else add = __fadd2_rn(add, two_slopes);
                        }
                        const float2 x = __ffma2_rn(make_float2(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1])), c2, add);
                        const float2 e = make_float2(ex2_approx(x.x), ex2_approx(x.y));
                        if (i & 1) sum_b = __fadd2_rn(sum_b, e); else sum_a = __fadd2_rn(sum_a, e);
                        if constexpr (PSPLIT) split2(e, packed[i], packed[i + 16]);
                        else {
                            __nv_bfloat162 h2 = __floats2bfloat162_rn(e.x, e.y);
                            packed[i] = *reinterpret_cast<uint32_t*>(&h2);
                        }
                    }
                    // keys 32c .. 32c+31 of this row, two per column: columns 16c .. 16c+15, whose scores have been read (c' <= c);
                    // the two halves of PSPLIT take the chunk's own 32 columns
                    if constexpr (PSPLIT) tmem_st_32x32(s_addr + c * 32, packed);
                    else tmem_st_32x32b_x16(s_addr + c * 16, packed);
                    return true;
                };
                auto tile = [&](auto diag_tag) -> bool {
                    if constexpr (WIN) {                             // a loop of two chunks: the whole tile unrolled outgrows the instruction cache
#pragma unroll 1
                        for (int h = 0; h < 4; h += 2)
                            if (!chunk(h, va, vb, diag_tag) || !chunk(h + 1, vb, va, diag_tag)) return false;
                        return true;
                    } else
                    return chunk(std::integral_constant<int, 0>(), va, vb, diag_tag) &&
                           chunk(std::integral_constant<int, 1>(), vb, va, diag_tag) &&
                           chunk(std::integral_constant<int, 2>(), va, vb, diag_tag) &&
                           chunk(std::integral_constant<int, 3>(), vb, va, diag_tag);
                };
                ok = diag ? tile(std::true_type()) : tile(std::false_type());
                if (!ok) break;
                tmem_st_wait();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(p_full + 8 * sbuf);
                l += (sum_a.x + sum_a.y) + (sum_b.x + sum_b.y);
            }
            G += (uint32_t)entries(w);
            if (!ok) break;
            if (n_kv > 0) {
                float inv = 1.0f / l;
                if (!WIN && p.gate && qrow < p.T) inv *= 1.0f / (1.0f + __expf(-__bfloat162float(p.gate[((long long)bb * p.T + qrow) * p.ld_gate + hh])));
                // (rows past the sequence read its last row's, so that the warp stays together: the TMEM loads below are warp-wide)
                const __nv_bfloat16* grow = WIN && p.gate ? p.gate + ((long long)bb * p.T + min(qrow, p.T - 1)) * p.ld_gate + (long long)hh * p.V : nullptr;
                uint4 graw[4];                                   // the next 32 columns' gates, requested ahead of the output they meet
                auto fetch_gates = [&](int c) {
#pragma unroll
                    for (int i = 0; i < 4; i++)
                        if (c * 32 + i * 8 < p.V) graw[i] = *reinterpret_cast<const uint4*>(grow + c * 32 + i * 8);
                };
                if (WIN && grow) fetch_gates(0);
                // The item's last product -- after the one before it: scores run up to two ahead, so with a single query tile only the product of
                // step - 4 is sure to be done here, and a parity wait for step - 1 could not tell step - 3 (same barrier, the phase before)
                // from step - 1.  The product of step - 2 waits on the other barrier, one phase ahead of step - 4, and brings step - 3 with it.
                ok = (n_kv - j_first < 2 || mbar_wait(pv_done + 8 * (2 * t + (step & 1)), ((step - 2) >> 1) & 1, abort_flag, p.status, kErrEpilogueWait)) &&
                     mbar_wait(pv_done + 8 * (2 * t + ((step - 1) & 1)), ((step - 1) >> 1) & 1, abort_flag, p.status, kErrEpilogueWait);
                if (!ok) break;
                __syncwarp();
                tc_fence_after();
                __nv_bfloat16* orow = p.out + ((long long)bb * p.T + qrow) * p.ld_out + (long long)hh * p.V;
#pragma unroll
                for (int c = 0; c < VD / 32; c++) {
                    uint32_t o[32];
                    __syncwarp();                                // lanes that stored and lanes that did not
                    tmem_ld_32x32(o_addr + c * 32, o);
                    tmem_ld_wait();
                    if constexpr (WIN) {
                        if (grow) {
#pragma unroll
                            for (int i = 0; i < 4; i++) {
                                const __nv_bfloat162* gh = reinterpret_cast<const __nv_bfloat162*>(&graw[i]);
#pragma unroll
                                for (int q = 0; q < 4; q++) {
                                    const float2 gv = bf16x2_to_float2(gh[q]);
                                    o[8 * i + 2 * q] = __float_as_uint(__fdividef(__uint_as_float(o[8 * i + 2 * q]), 1.0f + __expf(-gv.x)));
                                    o[8 * i + 2 * q + 1] = __float_as_uint(__fdividef(__uint_as_float(o[8 * i + 2 * q + 1]), 1.0f + __expf(-gv.y)));
                                }
                            }
                            if (c + 1 < VD / 32) fetch_gates(c + 1);
                        }
                    }
                    if (qrow < p.T) {
#pragma unroll
                        for (int i = 0; i < 32; i += 8) {
                            if ((KBR > 0 || WIN) && c * 32 + i >= p.V) break;
                            uint4 w;
                            __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&w);
#pragma unroll
                            for (int q = 0; q < 4; q++) oh[q] = __floats2bfloat162_rn(__uint_as_float(o[i + 2 * q]) * inv, __uint_as_float(o[i + 2 * q + 1]) * inv);
                            *reinterpret_cast<uint4*>(orow + c * 32 + i) = w;
                        }
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0 && n_kv > 0) mbar_arrive(o_free + 8 * t);      // the accumulator may be overwritten by the next item
        }
    }

    tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        // give loads that may still be in flight time to land before shared memory is released
        unsigned long long t0 = globaltimer();
        while (globaltimer() - t0 < 200000ull) { }
        __syncthreads();
    }
    if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, TMEM_COLS); }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static EncodeTiledFn attn_encode() {
    static EncodeTiledFn fn = nullptr;
    static std::once_flag once;
    std::call_once(once, [] {
        void* q = nullptr;
        cudaDriverEntryPointQueryResult r;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &q, cudaEnableDefault, &r) == cudaSuccess && r == cudaDriverEntryPointSuccess)
            fn = (EncodeTiledFn)q;
    });
    return fn;
}

// bf16 rank-4 map over a token-major [B*T, ld] matrix seen as (head_dim, T, H, B): box (64, 128, 1, 1), 128-byte swizzle.
// Rows past T read as zero (they belong to the next sequence in memory, but the T dimension of the map ends there).
static int encode_heads(CUtensorMap* map, const void* ptr, int hd, int T, int H, int B, long long ld, long long head_stride, long long seq_stride) {
    EncodeTiledFn enc = attn_encode();
    if (!enc) return fail("cuTensorMapEncodeTiled is not available from this driver");
    cuuint64_t dims[4] = {(cuuint64_t)hd, (cuuint64_t)T, (cuuint64_t)H, (cuuint64_t)B};
    cuuint64_t st[3] = {(cuuint64_t)ld * 2, (cuuint64_t)(H > 1 ? head_stride : ld) * 2, (cuuint64_t)(B > 1 ? seq_stride : ld) * 2};
    cuuint32_t box[4] = {64, 128, 1, 1};
    cuuint32_t es[4] = {1, 1, 1, 1};
    CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(ptr), dims, st, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                     CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail("attention: cuTensorMapEncodeTiled failed with CUresult %d", (int)r);
    return 0;
}

// Work schedule of the persistent kernel.  Items are (query tile pair, sequence*head); pair q reads the keys and values
// 0 .. 256 q + 255 of its (sequence, head), so the tiles of one (sequence, head) re-read the same K/V.  The list is cut into
// groups of (sequence, head)s whose K/V fit in L2 together, each group ordered longest item first, and the items are dealt out
// in that order to the CTA that has the least work so far (list scheduling, cost = key tiles of both query tiles + 1): the
// items of one (sequence, head) then run close together in time and their K/V come from L2 instead of DRAM, while the CTAs
// still finish together.  Schedules are cached per shape and released when the backend shuts down.
struct AttnSchedule { std::vector<int> host; int* dev = nullptr; int len = 0; };
static std::mutex g_sched_mu;
static std::map<std::array<int, 6>, AttnSchedule> g_sched;

static void attention_schedules_release() {
    std::lock_guard<std::mutex> lk(g_sched_mu);
    for (auto& kv : g_sched) if (kv.second.dev) cudaFree(kv.second.dev);
    g_sched.clear();
}

static int attention_schedule(int B, int H, int T, int hd, int npt, int grid, const int** dev, int* len) {
    static const int l2_mb = getenv("SPTORCH_B200_ATTN_L2_MB") ? atoi(getenv("SPTORCH_B200_ATTN_L2_MB")) : 32;
    const int BH = B * H;
    const long long pair_bytes = 2LL * T * hd * 2;                       // K and V of one (sequence, head)
    long long group = l2_mb > 0 ? ((long long)l2_mb << 20) / pair_bytes : BH;
    group = group < 1 ? 1 : (group > BH ? BH : group);
    std::lock_guard<std::mutex> lk(g_sched_mu);
    if (g_sched.size() > 64) {                                           // a bound on the cache: drop everything not in flight
        if (stream_wait()) return 1;
        for (auto& kv : g_sched) if (kv.second.dev) cudaFree(kv.second.dev);
        g_sched.clear();
    }
    AttnSchedule& s = g_sched[{B, H, T, hd, grid, (int)group}];
    if (!s.dev) {
        at_shutdown(attention_schedules_release);
        const int n_kv_seq = ceil_div(T, kKvTile);
        std::vector<std::vector<int>> lists(grid);
        using Slot = std::pair<long long, int>;                          // (work so far, CTA)
        std::priority_queue<Slot, std::vector<Slot>, std::greater<Slot>> heap;
        for (int c = 0; c < grid; c++) heap.push({0, c});
        for (int g0 = 0; g0 < BH; g0 += (int)group) {
            const int g1 = std::min<long long>(BH, g0 + group);
            for (int pt = npt - 1; pt >= 0; pt--) {
                const int q0 = pt * kQPair;
                const int n0 = std::min(q0 / kKvTile + 1, n_kv_seq);
                const int n1 = q0 + kQTile < T ? std::min(q0 / kKvTile + 2, n_kv_seq) : 0;
                for (int bh = g0; bh < g1; bh++) {
                    Slot t = heap.top(); heap.pop();
                    lists[t.second].push_back((npt - 1 - pt) * BH + bh);
                    heap.push({t.first + n0 + n1 + 1, t.second});
                }
            }
        }
        size_t len_max = 0;
        for (auto& l : lists) len_max = std::max(len_max, l.size());
        s.len = (int)len_max;
        s.host.assign(len_max * grid, -1);
        for (int c = 0; c < grid; c++)
            for (size_t k = 0; k < lists[c].size(); k++) s.host[k * grid + c] = lists[c][k];
        SPT_CUDA(cudaMalloc(&s.dev, s.host.size() * sizeof(int)));
        // the host copy lives as long as the cache entry, so the copy may stay asynchronous
        SPT_CUDA(cudaMemcpyAsync(s.dev, s.host.data(), s.host.size() * sizeof(int), cudaMemcpyHostToDevice, rt().stream));
    }
    *dev = s.dev; *len = s.len;
    return 0;
}

bool attention_fused_supported(int T, int hd, long long ld_q, long long ld_kv) {
    return (hd == 64 || hd == 128) && T > 0 && ld_q % 8 == 0 && ld_kv % 8 == 0;
}

// q, k, v: [B*T, ld] bf16, head h at columns h*hd (token-major: the layout the QKV projection writes);
// out: [B*T, ld_out] bf16, head h at columns h*hd.
int attention_fused(const void* q, const void* k, const void* v, void* out, int B, int T, int H, int hd, long long ld_q, long long ld_k,
                    long long ld_v, long long ld_out) {
    if (!attention_fused_supported(T, hd, ld_q, ld_k) || ld_v % 8) return fail("attention_fused: unsupported shape or stride");
    if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(out)) & 15)
        return fail("attention_fused: buffers must be 16-byte aligned");
    if (ld_out % 8) return fail("attention_fused: ld_out must be a multiple of 8");
    CUtensorMap tq, tk, tv;
    if (encode_heads(&tq, q, hd, T, H, B, ld_q, hd, (long long)T * ld_q)) return 1;
    if (encode_heads(&tk, k, hd, T, H, B, ld_k, hd, (long long)T * ld_k)) return 1;
    if (encode_heads(&tv, v, hd, T, H, B, ld_v, hd, (long long)T * ld_v)) return 1;
    AttnParams prm;
    prm.out = (__nv_bfloat16*)out; prm.ld_out = ld_out; prm.T = T; prm.H = H; prm.B = B; prm.n = T; prm.first = 0; prm.V = hd; prm.gate = nullptr; prm.ld_gate = 0; prm.group = 1; prm.window = 0; prm.slopes = nullptr;
    prm.n_ptiles = ceil_div(T, kQPair);
    prm.scale_log2 = (1.0f / sqrtf((float)hd)) * 1.4426950408889634f;
    prm.status = rt().dev_status;
    long long items = (long long)B * H * prm.n_ptiles;
    if (items > INT32_MAX) return fail("attention_fused: too many work items");
    const long long slots = compute_sms();                                      // one resident CTA per SM
    long long grid = items < slots ? items : slots;
    if (attention_schedule(B, H, T, hd, prm.n_ptiles, (int)grid, &prm.sched, &prm.sched_len)) return 1;
    ProfScope ps(PROF_ATTN_FUSED);
    auto launch = [&](auto kern, int smem_bytes) -> int {
        SPT_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_bytes));
        kern<<<(unsigned)grid, kAttnThreads, smem_bytes, rt().stream>>>(tq, tk, tv, tq, tk, prm);
        return 0;
    };
    int lrc;
    if (hd == 64) {
        static const bool rot_off = getenv("SPTORCH_B200_ATTN_ROT") && atoi(getenv("SPTORCH_B200_ATTN_ROT")) == 0;
        lrc = rot_off ? launch(attn_fused_kernel<1, 0, 64, false, false>, AttnSmem<1, 0, 64>::kTotal) : launch(attn_fused_kernel<1, 0, 64, true, false>, AttnSmem<1, 0, 64>::kTotal);
    } else lrc = launch(attn_fused_kernel<2, 0, 128, true, false>, AttnSmem<2, 0, 128>::kTotal);
    if (lrc) return lrc;
    SPT_LAUNCH_CHECK("attn_fused");
    return 0;
}

// ---- latent attention over expanded keys and values ----
// q: [B*T, ld_q], head h at columns h*(D+rot): [D | rot]; kn, v: [B*n, ld_kv], head h at columns h*D / h*V; kr: the shared key part, rows
// `row` elements apart, sequences seq_stride apart; gate: one logit per (token, head); out: [B*T, ld_out], head h at columns h*V.
// Queries are at positions first .. first + T - 1, keys at 0 .. n - 1.
bool attention_latent_supported(int D, int rot, int V, int kv_off, long long ld_q, long long ld_kv, int row) {
    return D >= 8 && D <= 128 && D % 8 == 0 && rot >= 8 && rot <= 64 && rot % 8 == 0 && V >= 8 && V <= 128 && V % 8 == 0 && kv_off % 8 == 0 && ld_q % 8 == 0 &&
           ld_kv % 8 == 0 && row % 8 == 0;
}

int attention_latent(const void* q, long long ld_q, const void* kn, const void* v, long long ld_kv, const void* kr, long long row, long long seq_stride,
                     void* out, long long ld_out, const void* gate, long long ld_gate, int B, int T, int n, int H, int D, int rot, int V, int first, float scale) {
    CUtensorMap tq, tqr, tk, tkr, tv;
    if (encode_heads(&tq, q, D, T, H, B, ld_q, D + rot, (long long)T * ld_q)) return 1;
    if (encode_heads(&tqr, (const __nv_bfloat16*)q + D, rot, T, H, B, ld_q, D + rot, (long long)T * ld_q)) return 1;
    if (encode_heads(&tk, kn, D, n, H, B, ld_kv, D, (long long)n * ld_kv)) return 1;
    if (encode_heads(&tv, v, V, n, H, B, ld_kv, V, (long long)n * ld_kv)) return 1;
    if (encode_heads(&tkr, kr, rot, n, 1, B, row, row, seq_stride)) return 1;
    AttnParams prm;
    prm.out = (__nv_bfloat16*)out; prm.ld_out = ld_out; prm.T = T; prm.H = H; prm.B = B; prm.n = n; prm.first = first; prm.V = V;
    prm.gate = (const __nv_bfloat16*)gate; prm.ld_gate = ld_gate; prm.group = 1; prm.window = 0; prm.slopes = nullptr;
    prm.n_ptiles = ceil_div(T, kQPair);
    prm.scale_log2 = scale * 1.4426950408889634f;
    prm.status = rt().dev_status;
    const long long items = (long long)B * H * prm.n_ptiles;
    if (items > INT32_MAX) return fail("attention_latent: too many work items");
    const long long slots = compute_sms(), grid = items < slots ? items : slots;
    prm.sched = nullptr; prm.sched_len = ceil_div(items, grid);
    // a prompt from position 0 uses a cached balanced schedule; a later portion, whose shape changes from call to call, the plain order
    if (first == 0 && attention_schedule(B, H, T, (D + rot + V) / 2, prm.n_ptiles, (int)grid, &prm.sched, &prm.sched_len)) return 1;
    auto launch = [&](auto kern, int smem_bytes) -> int {
        SPT_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_bytes));
        kern<<<(unsigned)grid, kAttnThreads, smem_bytes, rt().stream>>>(tq, tk, tv, tqr, tkr, prm);
        return 0;
    };
    int rc;
    if (D <= 64) rc = V <= 64 ? launch(attn_fused_kernel<1, 1, 64, true, true>, AttnSmem<1, 1, 64>::kTotal) : launch(attn_fused_kernel<1, 1, 128, true, true>, AttnSmem<1, 1, 128>::kTotal);
    else rc = V <= 64 ? launch(attn_fused_kernel<2, 1, 64, true, true>, AttnSmem<2, 1, 64>::kTotal) : launch(attn_fused_kernel<2, 1, 128, true, true>, AttnSmem<2, 1, 128>::kTotal);
    if (rc) return rc;
    SPT_LAUNCH_CHECK("attention_latent");
    return 0;
}

// ---- window attention over cached keys and values ----
// q: [B*T, H*D]; rows: [B][positions][row] with key head g at columns g*D and value head g at columns G*D + g*V, sequences seq_stride
// apart, of which positions 0 .. n - 1 are there; gate (null: none) and out: [B*T, ld_out], head h at columns h*V, may be the same.
bool attention_window_supported(int D, int V, int row, long long ld_out) {
    return D >= 8 && D <= 128 && D % 8 == 0 && V >= 8 && V <= 128 && V % 8 == 0 && row % 8 == 0 && ld_out % 8 == 0;
}

int attention_window(const void* q, const void* rows, int row, long long seq_stride, void* out, long long ld_out, const void* gate, int B, int T, int n, int H, int G,
                     int D, int V, int first, int window, const float* slopes, float scale) {
    CUtensorMap tq, tk, tv;
    if (encode_heads(&tq, q, D, T, H, B, (long long)H * D, D, (long long)T * H * D)) return 1;
    if (encode_heads(&tk, rows, D, n, G, B, row, D, seq_stride)) return 1;
    if (encode_heads(&tv, (const __nv_bfloat16*)rows + (size_t)G * D, V, n, G, B, row, V, seq_stride)) return 1;
    AttnParams prm;
    prm.out = (__nv_bfloat16*)out; prm.ld_out = ld_out; prm.T = T; prm.H = H; prm.B = B; prm.n = n; prm.first = first; prm.V = V;
    prm.gate = (const __nv_bfloat16*)gate; prm.ld_gate = ld_out; prm.group = H / G; prm.slopes = slopes;
    const bool all = window <= 0 || window >= n;
    prm.window = all ? n : window;
    prm.n_ptiles = ceil_div(T, kQPair);
    prm.scale_log2 = scale * 1.4426950408889634f;
    prm.status = rt().dev_status;
    const long long items = (long long)B * H * prm.n_ptiles;
    if (items > INT32_MAX) return fail("attention_window: too many work items");
    const long long slots = compute_sms(), grid = items < slots ? items : slots;
    prm.sched = nullptr; prm.sched_len = ceil_div(items, grid);
    // with a window that cuts, the items are nearly alike and the plain order does; otherwise as for latent attention
    if (all && first == 0 && attention_schedule(B, H, T, (D + V) / 2, prm.n_ptiles, (int)grid, &prm.sched, &prm.sched_len)) return 1;
    auto launch = [&](auto kern, int smem_bytes) -> int {
        SPT_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_bytes));
        kern<<<(unsigned)grid, kAttnThreads, smem_bytes, rt().stream>>>(tq, tk, tv, tq, tk, prm);
        return 0;
    };
    int rc;
    if (D <= 64) rc = V <= 64 ? launch(attn_fused_kernel<1, 0, 64, true, true, true>, AttnSmem<1, 0, 64>::kTotal) : launch(attn_fused_kernel<1, 0, 128, true, true, true>, AttnSmem<1, 0, 128>::kTotal);
    else rc = V <= 64 ? launch(attn_fused_kernel<2, 0, 64, true, true, true>, AttnSmem<2, 0, 64>::kTotal) : launch(attn_fused_kernel<2, 0, 128, true, true, true>, AttnSmem<2, 0, 128>::kTotal);
    if (rc) return rc;
    SPT_LAUNCH_CHECK("attention_window");
    return 0;
}

}  // namespace spt
