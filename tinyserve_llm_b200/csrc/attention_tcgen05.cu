// Prefill attention on the fifth-generation tensor cores, head sizes 64 and 128, bfloat16, pages of a
// multiple of 64 tokens, no window.  A CTA takes 128 consecutive tokens of one request for one query head
// (head size 128: rows lie in shared memory as two sub-tiles of 64 dims, key tiles hold 64 keys, so that
// two CTAs still fit an SM's shared and tensor memory):
//
//   * S = Q K^T for a tile of 128 keys is one tcgen05.mma chain (A = the query tile, B = the key
//     tile, both brought into 128-byte-swizzled shared memory by TMA straight from the qkv matrix
//     and from the paged pool) into tensor memory;
//   * two threads of the eight softmax warps own query row r, which is lane r of tensor memory: each reads
//     its half of the row of S with tcgen05.ld into registers, they exchange their maxima, keep the
//     reference of the exponentials and the sum in float32, write P = exp2(S - m) as bfloat16 pairs into
//     tensor-memory columns of P's own (tcgen05.st) and rescale their halves of the row of O, which is
//     needed only when the maximum has grown by more than 2^8 since the reference was taken;
//   * O += P V is a second tcgen05.mma chain with A = P read from tensor memory and B = the value
//     tile as it lies in shared memory (dims contiguous: the MN-major operand form).
//
// Warp 8 is the TMA producer over a two-stage ring of key/value tiles, warp 9 allocates tensor memory
// and issues the MMAs, warps 0..7 are the softmax.  Hand-offs are mbarriers: kv_full (TMA bytes),
// s_done / stage_free / all_done (tcgen05.commit) and p_ready (256 thread arrivals).  When the softmax
// hands over P of a tile, the scores of the next tile are issued before this tile's O += P V, so that
// the next softmax begins under that product.  Two CTAs share an SM, so one's softmax runs under the
// other's MMAs.  A query at position p sees keys 0..p
// (attention/torch_paged.py:36-45 of the reference, by positions); value rows beyond the request's
// length are zeroed in shared memory before they are multiplied.
//
// A form for keys of which every head has its own part and all heads share a second, rotated one (ROT): queries and keys
// have a further sub-tile of 64 channels, the keys' read from a matrix of its own, once for all heads.
//
// Every mbarrier wait gives up after about two seconds and records where in an error word.
#include <cuda.h>

#include "common.cuh"

namespace {

constexpr int QROWS = 128;                   // queries per CTA
// Sizes that follow from the head size.  A tile row of more than 64 dims lies in shared memory as
// sub-tiles of 64 dims (128 bytes, the widest row the 128-byte swizzle takes), one after the other.
// ROT (0 or 64): channels of the shared part of queries and keys, a sub-tile behind the others.
template <int HD, int ROT = 0>
struct Shape {
    static constexpr int KEYS = (HD == 64) == (ROT == 0) ? 128 : 64;     // keys per tile: two CTAs must fit an SM (HD 128 with ROT: one)
    static constexpr int SUBS = HD / 64, QK_SUBS = (HD + ROT) / 64;      // sub-tiles of 64 dims: of values, of queries and keys
    static constexpr int SUB_Q = QROWS * 128, SUB_KV = KEYS * 128; // bytes of a sub-tile
    static constexpr int Q_BYTES = QK_SUBS * SUB_Q, K_BYTES = QK_SUBS * SUB_KV, STAGE_BYTES = K_BYTES + SUBS * SUB_KV;
    static constexpr int O_COL = KEYS;       // S at columns 0..KEYS-1, O after it, P (bfloat16 pairs) after O
    static constexpr int P_COL = KEYS + HD;
    static constexpr int TMEM_COLS = P_COL + KEYS / 2 <= 256 ? 256 : 512;
    static constexpr int CTAS = TMEM_COLS == 256 ? 2 : 1;                // on an SM
    static_assert(HD == 64 || HD == 128, "head sizes 64 and 128");
    static_assert(ROT == 0 || ROT == 64, "one shared sub-tile or none");
    static_assert(P_COL + KEYS / 2 <= TMEM_COLS, "S, O and P must fit the allocation");
};
constexpr int SOFTMAX_WARPS = 8;             // two threads a query row: each takes half of the tile's keys and half of O's dims
constexpr int PRODUCER_WARP = SOFTMAX_WARPS, MMA_WARP = SOFTMAX_WARPS + 1, THREADS = (SOFTMAX_WARPS + 2) * 32;
constexpr long long WAIT_CYCLES = 4000000000ll;
constexpr uint32_t SUSPEND_NS = 1000000;      // a waiting thread may sleep this long in one try before it looks at the clock
constexpr float LOG2E = 1.4426950408889634f;
constexpr float RESCALE_STEP = 8.f;          // in powers of two

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mbar_init(uint64_t* bar, int count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t* bar, uint32_t bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity, int* error, int code) {
    const long long start = clock64();
    uint32_t done = 0;
    while (true) {
        asm volatile(
            "{\n\t.reg .pred p;\n\t"
            "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2, %3;\n\t"
            "selp.u32 %0, 1, 0, p;\n\t}"
            : "=r"(done) : "r"(smem_u32(bar)), "r"(parity), "r"(SUSPEND_NS) : "memory");
        if (done) return true;
        if (clock64() - start > WAIT_CYCLES) {
            atomicExch(error, code);
            return false;
        }
    }
}
__device__ __forceinline__ void tma_load_2d(void* smem, const CUtensorMap* map, uint64_t* bar, int x, int y) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
        ::"r"(smem_u32(smem)), "l"(map), "r"(smem_u32(bar)), "r"(x), "r"(y) : "memory");
}
// 128-byte-swizzled tile of rows of 128 bytes; groups of 8 rows are 1024 bytes apart.
__device__ __forceinline__ uint64_t smem_desc(const void* tile) {
    uint64_t d = 0;
    d |= (uint64_t)((smem_u32(tile) & 0x3FFFF) >> 4);
    d |= (uint64_t)1 << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// bfloat16 x bfloat16 -> float32; A K-major (or in tensor memory); B K-major, or MN-major if b_mn.
__device__ __forceinline__ uint32_t instr_desc(int m, int n, bool b_mn) {
    uint32_t d = 0;
    d |= 1u << 4;
    d |= 1u << 7;
    d |= 1u << 10;
    if (b_mn) d |= 1u << 16;
    d |= (uint32_t)(n >> 3) << 17;
    d |= (uint32_t)(m >> 4) << 24;
    return d;
}
__device__ __forceinline__ void umma_ss(uint32_t tmem_d, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t acc) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(tmem_d), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(acc) : "memory");
}
__device__ __forceinline__ void umma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t b_desc, uint32_t idesc, uint32_t acc) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
        ::"r"(tmem_d), "r"(tmem_a), "l"(b_desc), "r"(idesc), "r"(acc) : "memory");
}
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
        "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
          "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
          "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
          "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(taddr) : "memory");
}
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
        "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
          "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]),
          "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]),
          "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31]) : "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
          "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
// 2^x for any x (+inf above the float range) and 1 / x (0 for +inf): one instruction each.
__device__ __forceinline__ float fast_exp2_any(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float fast_rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
// tanh(x) = 1 - 2 / (e^(2x) + 1) from the exponential and the reciprocal (the hardware's approximate tanh keeps 11
// bits); beyond +-15 the result is +-1 in float32 anyway.
__device__ __forceinline__ float exp_tanh(float x) {
    x = fminf(fmaxf(x, -15.f), 15.f);
    return fmaf(-2.f, fast_rcp(1.f + fast_exp2_any(x * (2.f * LOG2E))), 1.f);
}
// The first key a query at position `pos` sees: inside its window and inside its chunk (0: no such bound).
__device__ __forceinline__ int first_visible(int pos, int window, int chunk) {
    int lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (chunk > 0 && pos > 0) lo = max(lo, pos / chunk * chunk);
    return lo;
}
// The forms of the kernel: softmax over every earlier key; sigmoid weights (with a window); softmax behind a mask with
// a lower bound (window, chunks), of scores that may be capped, over a value pool that may hold fewer heads.
enum { PLAIN = 0, SIGMOID = 1, BOUNDED = 2 };

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}

// The two softmax warps of a quadrant meet at a named barrier of their own (ids 1..4; 0 is __syncthreads).
__device__ __forceinline__ void pair_barrier(int quadrant) {
    switch (quadrant) {
        case 0: asm volatile("bar.sync 1, 64;" ::: "memory"); break;
        case 1: asm volatile("bar.sync 2, 64;" ::: "memory"); break;
        case 2: asm volatile("bar.sync 3, 64;" ::: "memory"); break;
        default: asm volatile("bar.sync 4, 64;" ::: "memory"); break;
    }
}

struct FlashParams {
    __nv_bfloat16* out;               // [T, nh * HD]
    const int* block_table;
    int table_width;
    const int* cu_q;
    const int* ctx_lens;
    const int* prefill_seqs;          // requests that feed more than one token (-1: none); null: every request has CTAs
    int nh, nkv;
    int page_tokens, num_pages;
    int entries, entry;               // cache entries of the layer group; this layer's index among them
    float scale_log2;
    int* error;
    // sigmoid weights (the SIG kernel): a window, terms of the score and the output gate; a null pointer: the term is absent
    int window;                       // a query at position p sees keys p - window + 1 .. p (0: all up to p)
    const float* slopes;              // [nh]: slopes[h] * (position - key) is taken off the score
    const float* head_bias;           // [nh]: added to every score of the head
    const __nv_bfloat16* gate;        // [T, nh] logits, gate_stride elements a row: the head's output times their sigmoid
    long long gate_stride;
    // the BOUNDED kernel
    int chunk;                        // n > 0: a query sees no key before floor(p / n) * n
    float cap_pre;                    // scores are capped: tanh(product * cap_pre), and scale_log2 is cap * log2(e); 0: not capped
    int value_heads;                  // heads of the value pool (a divisor of nkv)
    float sink2;                      // a score (times log2(e)) that joins the softmax's sum without a key or a value; -inf: none
    // keys and values in matrices of their own instead of pages: [rows, nkv * HD], request s's key j in row kv_start[s] + j
    const int* kv_start;              // null: keys and values come from the paged pools
    int q_head_cols;                  // columns of a head in q's rows (HD, and more where q holds other parts between the heads)
    const float* sinks;               // [nh], not null: a sink a head, in place of sink2
};

// SIG: a visible key's weight is sigmoid(score * scale - slope (position - key) + bias): no maximum, no sum, no
// rescaling, nothing exchanged between the two threads of a row; the epilogue multiplies by the head's gate.
// This form and BOUNDED take a window: the first key tile is the one that holds the first key the tile's first query sees.
// BOUNDED: softmax as in the plain form; a row's keys begin at first_visible(position); capped scores go through
// tanh in registers before the maximum is taken.
// ROT: map_q_rot [T, nh * 64] and map_k_rot [keys, <= 64] are the shared part of queries and keys (dense keys only).
template <int HD, int FORM, int ROT>
__global__ void __launch_bounds__(THREADS, (Shape<HD, ROT>::CTAS)) prefill_attention_tcgen05_kernel(
        const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
        const __grid_constant__ CUtensorMap map_q_rot, const __grid_constant__ CUtensorMap map_k_rot, FlashParams p) {
    using S_ = Shape<HD, ROT>;
    constexpr int TMEM_COLS = S_::TMEM_COLS;
    constexpr bool SIG = FORM == SIGMOID, LOW = FORM == BOUNDED;
    constexpr int KEYS = S_::KEYS, SUBS = S_::SUBS, SUB_Q = S_::SUB_Q, SUB_KV = S_::SUB_KV, Q_BYTES = S_::Q_BYTES,
                  K_BYTES = S_::K_BYTES, STAGE_BYTES = S_::STAGE_BYTES, O_COL = S_::O_COL, P_COL = S_::P_COL;
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t q_full, kv_full[2], stage_free[2], s_done, p_ready, all_done;
    __shared__ uint32_t tmem_base_slot;
    __shared__ int failed;
    __shared__ float half_max[2][2][QROWS];          // [tile parity][half][row]: the two threads of a row exchange their maxima
    __shared__ float half_sum[2][QROWS];             // ... and, at the end, their sums

    // blockIdx.x (which varies fastest in the order CTAs are handed out) is the head, blockIdx.y counts the
    // request's tiles from its last: the tile with the most keys of every head starts first, and
    // the short ones fill the SMs as the long ones finish.
    const int seq = p.prefill_seqs ? p.prefill_seqs[blockIdx.z] : (int)blockIdx.z, head = blockIdx.x;
    chain_wait();                                    // q, k and v of the step come from kernels ahead on the stream
    if (seq < 0) return;                             // a padding entry of the list (a step replayed from a graph)
    const int q_begin = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q_begin;
    if (q_len <= 1) return;                          // decode rows go to the split-key kernels
    const int tiles = (q_len + QROWS - 1) / QROWS;
    const int tile_index = tiles - 1 - (int)blockIdx.y;
    if (tile_index < 0) return;
    const int ctx = p.ctx_lens[seq];
    const int row0 = tile_index * QROWS;
    const int rows = min(QROWS, q_len - row0);
    const int pos0 = ctx - q_len + row0;             // position of the tile's first query
    const int last_pos = pos0 + rows - 1;
    const int num_kv = last_pos / KEYS + 1;
    // the first key any row of the tile sees
    const int first_seen = LOW ? first_visible(pos0, p.window, p.chunk) : (SIG && p.window > 0 ? max(0, pos0 - p.window + 1) : 0);
    const int low_last = LOW ? first_visible(last_pos, p.window, p.chunk) : 0;         // ... and the first key its last row sees
    const int kv_begin = first_seen / KEYS;          // tiles kv_begin .. num_kv - 1; `it` counts them from 0 for stages and parities
    const int kvh = head / (p.nh / p.nkv);
    const int nv = LOW ? p.value_heads : p.nkv, vh = LOW ? kvh / (p.nkv / p.value_heads) : kvh;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int* table = p.block_table + (long long)seq * p.table_width;
    const int dense_row0 = p.kv_start ? p.kv_start[seq] : -1;

    unsigned char* base = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char* q_tile = base;
    unsigned char* kv_tiles = base + Q_BYTES;        // stage s: K tile at s * STAGE_BYTES, V tile after it

    if (threadIdx.x == 0) {
        mbar_init(&q_full, 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init(&kv_full[s], 1);
            mbar_init(&stage_free[s], 1);
        }
        mbar_init(&s_done, 1);
        mbar_init(&p_ready, SOFTMAX_WARPS * 32);
        mbar_init(&all_done, 1);
        failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == MMA_WARP) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_slot)),
                     "r"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_base_slot;
    // Dependents are let in only now that this CTA holds its tensor memory: a kernel behind this one that
    // allocates tensor memory before it waits for this grid could otherwise starve a CTA of this grid.
    chain_release();

    if (warp == PRODUCER_WARP && lane == 0) {
        // ---------------------------------------------------------------- TMA producer
        mbar_expect_tx(&q_full, Q_BYTES);
#pragma unroll
        for (int h = 0; h < SUBS; ++h) tma_load_2d(q_tile + h * SUB_Q, &map_q, &q_full, head * p.q_head_cols + h * 64, q_begin + row0);
        if (ROT) tma_load_2d(q_tile + SUBS * SUB_Q, &map_q_rot, &q_full, head * 64, q_begin + row0);
        for (int j = kv_begin; j < num_kv; ++j) {
            const int it = j - kv_begin, s = it & 1;
            if (!mbar_wait(&stage_free[s], ((it >> 1) & 1) ^ 1, p.error, 11)) { failed = 1; break; }
            unsigned char* k_tile = kv_tiles + s * STAGE_BYTES;
            unsigned char* v_tile = k_tile + K_BYTES;
            mbar_expect_tx(&kv_full[s], STAGE_BYTES);
#pragma unroll
            for (int b = 0; b < KEYS / 64; ++b) {    // boxes of 64 keys x 64 dims: a box never crosses a page
                const int key = j * KEYS + b * 64;
                int row, v_row, col = 0, v_col = 0;
                if (dense_row0 >= 0) {               // rows past the request's last key belong to the next request, or to nobody
                    row = v_row = dense_row0 + key;  // (the copy fills those with zeros): masked anyway
                    col = kvh * HD;
                    v_col = vh * HD;
                } else {
                    int page = table[min(key / p.page_tokens, p.table_width - 1)];
                    if (page < 0 || page >= p.num_pages) page = 0;     // given back or beyond the request: masked anyway
                    row = ((page * p.entries + p.entry) * p.nkv + kvh) * p.page_tokens + key % p.page_tokens;
                    v_row = ((page * p.entries + p.entry) * nv + vh) * p.page_tokens + key % p.page_tokens;
                }
#pragma unroll
                for (int h = 0; h < SUBS; ++h) {
                    tma_load_2d(k_tile + h * SUB_KV + b * (64 * 128), &map_k, &kv_full[s], col + h * 64, row);
                    tma_load_2d(v_tile + h * SUB_KV + b * (64 * 128), &map_v, &kv_full[s], v_col + h * 64, v_row);
                }
                if (ROT) tma_load_2d(k_tile + SUBS * SUB_KV + b * (64 * 128), &map_k_rot, &kv_full[s], 0, row);
            }
        }
    } else if (warp == MMA_WARP && lane == 0) {
        // ---------------------------------------------------------------- MMA issuer
        const uint32_t idesc_s = instr_desc(QROWS, KEYS, false);
        const uint32_t idesc_o = instr_desc(QROWS, 64, true);        // O in column blocks of 64 dims, one per sub-tile of V
        bool ok = mbar_wait(&q_full, 0, p.error, 12);
        // S = Q K^T of tile j, once its keys have landed
        auto issue_scores = [&](int it) -> bool {
            const int s = it & 1;
            if (!mbar_wait(&kv_full[s], (it >> 1) & 1, p.error, 13)) return false;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
            for (int h = 0; h < S_::QK_SUBS; ++h) {
                const uint64_t q_desc = smem_desc(q_tile + h * SUB_Q);
                const uint64_t k_desc = smem_desc(kv_tiles + s * STAGE_BYTES + h * SUB_KV);
#pragma unroll
                for (int k = 0; k < 4; ++k) umma_ss(tmem, q_desc + 2 * k, k_desc + 2 * k, idesc_s, (h | k) != 0);
            }
            umma_commit(&s_done);
            return true;
        };
        ok = ok && issue_scores(0);
        const int num_it = num_kv - kv_begin;
        for (int j = 0; j < num_it && ok; ++j) {       // j counts the tiles from the first one here
            const int s = j & 1;
            if (!mbar_wait(&p_ready, j & 1, p.error, 14)) { ok = false; break; }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            // The softmax has read S of tile j (P lies in columns of its own), so the next tile's scores go first:
            // its softmax can begin while O += P V of this tile is still running.  The softmax waits for that
            // product (stage_free) before it writes P again or rescales O.
            if (j + 1 < num_it && !issue_scores(j + 1)) { ok = false; break; }
#pragma unroll
            for (int h = 0; h < SUBS; ++h) {         // O += P V: 16 keys are 8 columns of packed P and 16 rows (2048 bytes) of a V sub-tile
                const uint64_t v_desc = smem_desc(kv_tiles + s * STAGE_BYTES + K_BYTES + h * SUB_KV);
#pragma unroll
                for (int k = 0; k < KEYS / 16; ++k)
                    umma_ts(tmem + O_COL + 64 * h, tmem + P_COL + 8 * k, v_desc + 128 * k, idesc_o, (j | k) != 0);
            }
            umma_commit(&stage_free[s]);
        }
        if (!ok) failed = 1;
        umma_commit(&all_done);
    } else if (warp < SOFTMAX_WARPS) {
        // ---------------------------------------------------------------- softmax: two threads own query row r
        // Warp w reads the tensor-memory lanes of quadrant w % 4 (a warp can reach no others); the two
        // warps of a quadrant split the tile's keys, and O's dims, in halves.  They exchange their
        // halves' maxima through shared memory once a tile, behind a barrier of their 64 threads.
        const int quadrant = warp & 3, half = warp >> 2;
        const int r = quadrant * 32 + lane;
        const int pos = r < rows ? pos0 + r : -1;    // -1: a padding row sees nothing
        const uint32_t lane_addr = tmem + ((uint32_t)(quadrant * 32) << 16);
        constexpr int HK = KEYS / 2, HO = HD / 2;    // this thread's keys of a tile, and its dims of O
        const int col0 = half * HK;
        float m_run = -INFINITY, l_run = 0.f;
        // SIG: the row's first visible key, and the score's terms that do not depend on the key, in powers of two
        const int lo = LOW ? first_visible(pos, p.window, p.chunk) : (SIG && p.window > 0 ? max(0, pos - p.window + 1) : 0);
        const float slope2 = SIG && p.slopes ? p.slopes[head] * LOG2E : 0.f;
        const float bias2 = (SIG && p.head_bias ? p.head_bias[head] * LOG2E : 0.f) - slope2 * (float)pos;
        bool ok = true;
        for (int j = kv_begin; j < num_kv; ++j) {
            const int it = j - kv_begin, s = it & 1;
            const int key0 = j * KEYS;
            // a wait that ran out: the warp (as one) skips the work of this and the later tiles but still meets its
            // partner at the barrier below and still arrives at p_ready, so that nobody is left waiting for it
            if (ok && !mbar_wait(&s_done, it & 1, p.error, 15)) ok = false;
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) {
                if (!SIG) pair_barrier(quadrant);
                mbar_arrive(&p_ready);
                continue;
            }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            // some row of the tile does not see all of these keys (beyond its own position, or before its window)
            const bool masked = key0 + KEYS - 1 > pos0 || (SIG && p.window > 0 && key0 < last_pos - p.window + 1) ||
                                (LOW && key0 < low_last);
            // this thread's keys of S come into registers once, all loads under way together
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            uint32_t sv[HK / 32][32];
#pragma unroll
            for (int ch = 0; ch < HK / 32; ++ch) tmem_ld32(lane_addr + col0 + ch * 32, sv[ch]);
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
            if constexpr (SIG) {
                // O += P V of the tile before must have retired before P is written again
                if (it > 0 && !mbar_wait(&stage_free[(it - 1) & 1], ((it - 1) >> 1) & 1, p.error, 17)) ok = false;
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) {
                    mbar_arrive(&p_ready);
                    continue;
                }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
                for (int ch = 0; ch < HK / 32; ++ch) {
                    const int c = col0 + ch * 32;
                    const float term = fmaf(slope2, (float)(key0 + c), bias2);      // slope (key - position) + bias at the chunk's first key
                    uint32_t packed[16];
                    const uint32_t (&v)[32] = sv[ch];
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        // weight = 1 / (1 + 2^-x): 2^-x is +inf for a hopeless key, and the weight 0
                        const float x0 = fmaf(__uint_as_float(v[i]), p.scale_log2, fmaf(slope2, (float)i, term));
                        const float x1 = fmaf(__uint_as_float(v[i + 1]), p.scale_log2, fmaf(slope2, (float)(i + 1), term));
                        float w0 = fast_rcp(1.f + fast_exp2_any(-x0)), w1 = fast_rcp(1.f + fast_exp2_any(-x1));
                        if (masked) {
                            const int key = key0 + c + i;
                            if (key > pos || key < lo) w0 = 0.f;
                            if (key + 1 > pos || key + 1 < lo) w1 = 0.f;
                        }
                        packed[i >> 1] = pack_bf16(w0, w1);
                    }
                    tmem_st16(lane_addr + P_COL + (c >> 1), packed);
                }
                // value rows beyond the request's length, or before the first key the tile sees (their page may have been
                // given back), hold whatever the page held: zero them before they are multiplied
                if (half == 0 && r < KEYS && ((key0 + KEYS > ctx && key0 + r >= ctx) || key0 + r < first_seen)) {
#pragma unroll
                    for (int h = 0; h < SUBS; ++h) {
                        unsigned char* v_row = kv_tiles + s * STAGE_BYTES + K_BYTES + h * SUB_KV + r * 128;
#pragma unroll
                        for (int i = 0; i < 128; i += 16) *reinterpret_cast<uint4*>(v_row + i) = make_uint4(0, 0, 0, 0);
                    }
                    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
                }
                asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
                asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                mbar_arrive(&p_ready);
            } else {
            if constexpr (LOW) {
                if (p.cap_pre != 0.f) {              // capped scores: tanh(product * scale / cap); the cap joins the exponent's scale
#pragma unroll
                    for (int ch = 0; ch < HK / 32; ++ch)
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            sv[ch][i] = __float_as_uint(exp_tanh(__uint_as_float(sv[ch][i]) * p.cap_pre));
                }
            }
            // pass 1: the maximum over them (four running maxima: no long dependent chain)
#pragma unroll
            for (int ch = 0; ch < HK / 32; ++ch) {
                const int c = col0 + ch * 32;
                if (masked) {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (key0 + c + i <= pos && (!LOW || key0 + c + i >= lo)) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sv[ch][i]));
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sv[ch][i]));
                }
            }
            float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
            half_max[it & 1][half][r] = mx;
            pair_barrier(quadrant);
            mx = fmaxf(mx, half_max[it & 1][half ^ 1][r]);
            // O += P V of the tile before must have retired before P is written again and O is rescaled
            if (it > 0 && !mbar_wait(&stage_free[(it - 1) & 1], ((it - 1) >> 1) & 1, p.error, 17)) ok = false;
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) {
                mbar_arrive(&p_ready);
                continue;
            }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            // The reference the exponentials are taken against follows the maximum only when that has grown by
            // more than RESCALE_STEP: until then P holds values up to 2^RESCALE_STEP, which float32 sums and
            // bfloat16 products take without loss, and O needs no rescaling (softmax does not depend on the
            // reference it is computed against).
            const float m_tile = mx * p.scale_log2;
            const bool moved = m_tile > m_run + RESCALE_STEP;          // also the first tile that shows the row a key
            const float m_new = moved ? m_tile : m_run;
            const float m_use = m_new == -INFINITY ? 0.f : m_new;
            const float corr = moved ? fast_exp2(m_run - m_use) : 1.f;
            m_run = m_new;
            // pass 2: P = exp2(S * scale - m) as bfloat16 pairs into P's own columns (pair i covers keys 2i, 2i+1).
            // The tile on the diagonal has a loop of its own: inside one loop the compiler keeps the compare
            // and select of every element in the instruction stream of the tiles that need none.
            float l4[4] = {0.f, 0.f, 0.f, 0.f};
            if (masked) {
#pragma unroll
                for (int ch = 0; ch < HK / 32; ++ch) {
                    const int c = col0 + ch * 32;
                    uint32_t packed[16];
                    const uint32_t (&v)[32] = sv[ch];
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        float p0 = fast_exp2(fmaf(__uint_as_float(v[i]), p.scale_log2, -m_use));
                        float p1 = fast_exp2(fmaf(__uint_as_float(v[i + 1]), p.scale_log2, -m_use));
                        if (key0 + c + i > pos || (LOW && key0 + c + i < lo)) p0 = 0.f;
                        if (key0 + c + i + 1 > pos || (LOW && key0 + c + i + 1 < lo)) p1 = 0.f;
                        l4[(i >> 1) & 3] += p0 + p1;
                        packed[i >> 1] = pack_bf16(p0, p1);
                    }
                    tmem_st16(lane_addr + P_COL + (c >> 1), packed);
                }
            } else {
#pragma unroll
                for (int ch = 0; ch < HK / 32; ++ch) {
                    const int c = col0 + ch * 32;
                    uint32_t packed[16];
                    const uint32_t (&v)[32] = sv[ch];
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        const float p0 = fast_exp2(fmaf(__uint_as_float(v[i]), p.scale_log2, -m_use));
                        const float p1 = fast_exp2(fmaf(__uint_as_float(v[i + 1]), p.scale_log2, -m_use));
                        l4[(i >> 1) & 3] += p0 + p1;
                        packed[i >> 1] = pack_bf16(p0, p1);
                    }
                    tmem_st16(lane_addr + P_COL + (c >> 1), packed);
                }
            }
            l_run = l_run * corr + ((l4[0] + l4[1]) + (l4[2] + l4[3]));
            // this thread's dims of O follow the new reference; skipped when no row of the warp moved it
            if (it > 0 && !__all_sync(0xffffffffu, corr == 1.f)) {
#pragma unroll 1
                for (int c = half * HO; c < half * HO + HO; c += 32) {
                    uint32_t v[32];
                    tmem_ld32(lane_addr + O_COL + c, v);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * corr);
                    tmem_st32(lane_addr + O_COL + c, v);
                }
            }
            // value rows beyond the request's length (BOUNDED: or before the first key the tile sees, whose page may have
            // been given back) hold whatever the page held: zero them before they are multiplied
            if (half == 0 && r < KEYS && ((key0 + KEYS > ctx && key0 + r >= ctx) || (LOW && key0 + r < first_seen))) {
#pragma unroll
                for (int h = 0; h < SUBS; ++h) {
                    unsigned char* v_row = kv_tiles + s * STAGE_BYTES + K_BYTES + h * SUB_KV + r * 128;
#pragma unroll
                    for (int i = 0; i < 128; i += 16) *reinterpret_cast<uint4*>(v_row + i) = make_uint4(0, 0, 0, 0);
                }
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(&p_ready);
            }
        }
        if (ok) ok = mbar_wait(&all_done, 0, p.error, 16);
        ok = __all_sync(0xffffffffu, ok);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        // the row's sum is the two halves' sums (both were kept against the same maxima)
        if (!SIG) {
            half_sum[half][r] = l_run;
            pair_barrier(quadrant);
            l_run += half_sum[half ^ 1][r];
            const float sink2 = p.sinks ? p.sinks[head] * LOG2E : p.sink2;
            if (sink2 > -INFINITY) l_run += fast_exp2_any(sink2 - m_run);    // +inf where every score is far below it
        }
        if (ok && !failed) {                         // every thread of the warp takes part in the loads; only real rows store
            float inv = l_run > 0.f ? 1.f / l_run : 0.f;
            if (SIG) inv = (p.gate && r < rows) ? 1.f / (1.f + __expf(-__bfloat162float(p.gate[(long long)(q_begin + row0 + r) * p.gate_stride + head]))) : 1.f;
            __nv_bfloat16* o = p.out + ((long long)(q_begin + row0 + r) * p.nh + head) * HD;
#pragma unroll 1
            for (int c = half * HO; c < half * HO + HO; c += 32) {
                uint32_t v[32];
                tmem_ld32(lane_addr + O_COL + c, v);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (r < rows) {
#pragma unroll
                    for (int i = 0; i < 32; i += 8) {
                        uint4 packed;
                        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
                        for (int e = 0; e < 4; ++e)
                            h[e] = __floats2bfloat162_rn(__uint_as_float(v[i + 2 * e]) * inv, __uint_as_float(v[i + 2 * e + 1]) * inv);
                        *reinterpret_cast<uint4*>(o + c + i) = packed;
                    }
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == MMA_WARP) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(TMEM_COLS) : "memory");
    }
}

typedef CUresult (*EncodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiled encode_tiled() {
    static EncodeTiled fn = nullptr;
    if (!fn) {
        void* sym = nullptr;
        cudaDriverEntryPointQueryResult result;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &result) == cudaSuccess &&
            result == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiled>(sym);
    }
    return fn;
}

// [rows, 64] bfloat16 view with a row stride of ld elements; boxes of box_rows x 64, 128-byte swizzle.
int make_map(CUtensorMap* map, const void* base, long long rows, long long cols, long long ld, int box_rows) {
    EncodeTiled encode = encode_tiled();
    if (!encode) return ts_fail("attention_tcgen05: the driver does not export cuTensorMapEncodeTiled");
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {64u, (cuuint32_t)box_rows};
    const cuuint32_t elem[2] = {1, 1};
    const CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem,
                              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return ts_fail("attention_tcgen05: cuTensorMapEncodeTiled failed with %d", (int)r);
    return 0;
}

}  // namespace

TS_API int ts_attention_tcgen05_supported(int hd, int page_tokens, int nh, int nkv, int window) {
    return (hd == 64 || hd == 128) && page_tokens % 64 == 0 && nkv > 0 && nh % nkv == 0 && window == 0;
}

namespace {

// The part of queries and keys beside the heads' own: q_rot [T, nh * 64] (zeros past `rot` channels of a head), k_rot rows of
// `rot` channels, k_rot_stride elements apart; sinks [nh] or null.
struct SharedPart {
    const void* q_rot;
    const void* k_rot;
    long long k_rot_stride;
    int rot;                          // 0: no such part
    int q_head_cols;
    const float* sinks;
};

int run_prefill(const void* q, long long q_cols, long long q_stride, void* out, const void* k_pool, const void* v_pool,
                int num_pages, int entries, int entry, int page_tokens, const int* block_table, int table_width,
                const int* cu_q, const int* ctx_lens, int num_seqs, int num_tokens, int max_q_len, int nh, int nkv, int hd,
                float scale, const int* prefill_seqs, int num_prefill_seqs, int* error, bool sigmoid, int window,
                const float* slopes, const float* head_bias, const void* gate, long long gate_stride, cudaStream_t stream,
                bool bounded = false, int chunk = 0, float softcap = 0.f, int value_heads = 0, const int* kv_start = nullptr,
                long long dense_rows = 0, float sink = -INFINITY, const SharedPart* shared = nullptr) {
    TS_REQUIRE(ts_attention_tcgen05_supported(hd, page_tokens, nh, nkv, 0), "attention_tcgen05: sizes not taken (head_dim %d, page %d)", hd, page_tokens);
    TS_REQUIRE(sigmoid || bounded || window == 0, "attention_tcgen05: the plain form takes no window");
    TS_REQUIRE(window >= 0 && chunk >= 0 && softcap >= 0.f, "attention_tcgen05: a negative window, chunk or cap");
    if (value_heads <= 0) value_heads = nkv;
    TS_REQUIRE(nkv % value_heads == 0, "attention_tcgen05: %d value heads do not divide %d key heads", value_heads, nkv);
    TS_REQUIRE(error != nullptr, "attention_tcgen05: an error word is needed");
    TS_REQUIRE(num_seqs <= 65535 && (max_q_len + QROWS - 1) / QROWS <= 65535,
               "attention_tcgen05: more than 65535 requests, or tiles of a request, in a step");
    TS_REQUIRE(((uintptr_t)q % 16 == 0) && ((uintptr_t)k_pool % 16 == 0) && ((uintptr_t)v_pool % 16 == 0) && q_stride % 8 == 0,
               "attention_tcgen05: operands must be 16-byte aligned");
    if (num_seqs == 0 || max_q_len <= 1) return 0;
    TS_REQUIRE(prefill_seqs == nullptr || (num_prefill_seqs >= 0 && num_prefill_seqs <= num_seqs),
               "attention_tcgen05: %d prefill requests of %d", num_prefill_seqs, num_seqs);
    if (prefill_seqs != nullptr && num_prefill_seqs == 0) return 0;
    const long long pool_rows = (long long)num_pages * entries * nkv * page_tokens;
    TS_REQUIRE(pool_rows < 0x7fffffffll, "attention_tcgen05: the pool has too many rows for 32-bit TMA coordinates");
    CUtensorMap map_q, map_k, map_v, map_q_rot, map_k_rot;
    if (make_map(&map_q, q, num_tokens, q_cols, q_stride, QROWS)) return 1;
    if (kv_start != nullptr) {                           // matrices [dense_rows, heads * hd]
        TS_REQUIRE(dense_rows > 0 && dense_rows < 0x7fffffffll, "attention_tcgen05: %lld rows of keys", dense_rows);
        if (make_map(&map_k, k_pool, dense_rows, (long long)nkv * hd, (long long)nkv * hd, 64)) return 1;
        if (make_map(&map_v, v_pool, dense_rows, (long long)value_heads * hd, (long long)value_heads * hd, 64)) return 1;
    } else {
        if (make_map(&map_k, k_pool, pool_rows, hd, hd, 64)) return 1;
        if (make_map(&map_v, v_pool, pool_rows / nkv * value_heads, hd, hd, 64)) return 1;
    }
    const int rot = shared ? shared->rot : 0;
    if (rot > 0) {
        TS_REQUIRE(kv_start != nullptr && !sigmoid && !bounded, "attention_tcgen05: a shared key part comes with dense keys in the plain form");
        TS_REQUIRE(rot <= 64 && rot % 8 == 0 && shared->q_head_cols % 8 == 0 && shared->k_rot_stride % 8 == 0 &&
                   (uintptr_t)shared->q_rot % 16 == 0 && (uintptr_t)shared->k_rot % 16 == 0,
                   "attention_tcgen05: a shared key part of %d channels, or its alignment", rot);
        if (make_map(&map_q_rot, shared->q_rot, num_tokens, (long long)nh * 64, (long long)nh * 64, QROWS)) return 1;
        if (make_map(&map_k_rot, shared->k_rot, dense_rows, rot, shared->k_rot_stride, 64)) return 1;
    } else {
        map_q_rot = map_q;                               // not read
        map_k_rot = map_k;
    }
    FlashParams p;
    p.q_head_cols = shared ? shared->q_head_cols : hd;
    p.sinks = shared ? shared->sinks : nullptr;
    p.out = (__nv_bfloat16*)out;
    p.block_table = block_table;
    p.table_width = table_width;
    p.cu_q = cu_q;
    p.ctx_lens = ctx_lens;
    p.prefill_seqs = prefill_seqs;
    p.nh = nh;
    p.nkv = nkv;
    p.page_tokens = page_tokens;
    p.num_pages = num_pages;
    p.entries = entries;
    p.entry = entry;
    p.scale_log2 = softcap > 0.f ? softcap * LOG2E : scale * LOG2E;
    p.cap_pre = softcap > 0.f ? scale / softcap : 0.f;
    p.chunk = chunk;
    p.value_heads = value_heads;
    p.sink2 = sink > -INFINITY ? sink * LOG2E : -INFINITY;
    p.kv_start = kv_start;
    p.error = error;
    p.window = window;
    p.slopes = slopes;
    p.head_bias = head_bias;
    p.gate = (const __nv_bfloat16*)gate;
    p.gate_stride = gate_stride;
    dim3 grid(nh, (max_q_len + QROWS - 1) / QROWS, prefill_seqs ? num_prefill_seqs : num_seqs);
#define TS_FLASH_LAUNCH(HD, FORM, ROT)                                                                                    \
    do {                                                                                                                  \
        const size_t smem = (size_t)Shape<HD, ROT>::Q_BYTES + 2 * Shape<HD, ROT>::STAGE_BYTES + 1024;                     \
        auto kernel = prefill_attention_tcgen05_kernel<HD, FORM, ROT>;                                                    \
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                             \
        TS_CHAINED_CHECK("attention_tcgen05", launch_chained(kernel, grid, dim3(THREADS), smem, stream, map_q, map_k, map_v, \
                                                             map_q_rot, map_k_rot, p));                                   \
    } while (0)
    if (hd == 64 && rot > 0) TS_FLASH_LAUNCH(64, PLAIN, 64);
    else if (rot > 0) TS_FLASH_LAUNCH(128, PLAIN, 64);
    else if (hd == 64 && sigmoid) TS_FLASH_LAUNCH(64, SIGMOID, 0);
    else if (hd == 64 && bounded) TS_FLASH_LAUNCH(64, BOUNDED, 0);
    else if (hd == 64) TS_FLASH_LAUNCH(64, PLAIN, 0);
    else if (sigmoid) TS_FLASH_LAUNCH(128, SIGMOID, 0);
    else if (bounded) TS_FLASH_LAUNCH(128, BOUNDED, 0);
    else TS_FLASH_LAUNCH(128, PLAIN, 0);
#undef TS_FLASH_LAUNCH
    return 0;
}

}  // namespace

// Prompt portions (requests that feed more than one token) of a step; requests that feed one token
// are left to the decode kernels.  prefill_seqs (optional, device) lists the former, so that the grid
// has no CTAs for the latter.  The pools are [pages][entries][kv heads][page_tokens][64].
TS_API int ts_prefill_attention_tcgen05(const void* qkv, void* out, const void* k_pool, const void* v_pool, int num_pages,
                                        int entries, int entry, int page_tokens, const int* block_table, int table_width,
                                        const int* cu_q, const int* ctx_lens, int num_seqs, int num_tokens, int max_q_len,
                                        int nh, int nkv, int hd, float scale, const int* prefill_seqs, int num_prefill_seqs,
                                        int* error, cudaStream_t stream) {
    const long long row_width = (long long)(nh + 2 * nkv) * hd;
    return run_prefill(qkv, row_width, row_width, out, k_pool, v_pool, num_pages, entries, entry, page_tokens, block_table,
                       table_width, cu_q, ctx_lens, num_seqs, num_tokens, max_q_len, nh, nkv, hd, scale, prefill_seqs,
                       num_prefill_seqs, error, false, 0, nullptr, nullptr, nullptr, 0, stream);
}

// The same with sigmoid weights: a visible key's weight is sigmoid(score * scale - slopes[h] (i - j) + head_bias[h]),
// nothing is normalised over the keys, query i sees keys i - window + 1 .. i (window 0: all up to i), and head h's
// output is multiplied by sigmoid(gate[t, h]) (null pointers: the term is absent).  Queries [T, nh * hd] in a matrix
// of their own, q_stride elements a row.
TS_API int ts_prefill_attention_tcgen05_sigmoid(const void* q, long long q_stride, void* out, const void* k_pool,
                                                const void* v_pool, int num_pages, int entries, int entry, int page_tokens,
                                                const int* block_table, int table_width, const int* cu_q,
                                                const int* ctx_lens, int num_seqs, int num_tokens, int max_q_len, int nh,
                                                int nkv, int hd, float scale, int window, const float* slopes,
                                                const float* head_bias, const void* gate, long long gate_stride,
                                                const int* prefill_seqs, int num_prefill_seqs, int* error,
                                                cudaStream_t stream) {
    return run_prefill(q, (long long)nh * hd, q_stride, out, k_pool, v_pool, num_pages, entries, entry, page_tokens,
                       block_table, table_width, cu_q, ctx_lens, num_seqs, num_tokens, max_q_len, nh, nkv, hd, scale,
                       prefill_seqs, num_prefill_seqs, error, true, window, slopes, head_bias, gate, gate_stride, stream);
}

// Softmax attention behind a mask with a lower bound: query i sees keys max(i - window + 1, floor(i / chunk) chunk) .. i
// (0: no such bound); `softcap` c > 0 turns the scaled product into c tanh(. / c); the value pool holds `value_heads`
// heads (0: as many as key heads; key head j reads value head j / (nkv / value_heads)) in the same pages and entries;
// `sink` is a score that joins the softmax's sum without a key or a value (-inf: none).  With a sink and no bound, cap or
// shared values, the plain form of the kernel runs.  Queries [T, nh * hd] in a matrix of their own, q_stride elements a row.
TS_API int ts_prefill_attention_tcgen05_masked(const void* q, long long q_stride, void* out, const void* k_pool,
                                               const void* v_pool, int num_pages, int entries, int entry, int page_tokens,
                                               const int* block_table, int table_width, const int* cu_q,
                                               const int* ctx_lens, int num_seqs, int num_tokens, int max_q_len, int nh,
                                               int nkv, int hd, float scale, int window, int chunk, float softcap,
                                               int value_heads, const int* prefill_seqs, int num_prefill_seqs, int* error,
                                               float sink, cudaStream_t stream) {
    const bool bounded = window > 0 || chunk > 0 || softcap > 0.f || (value_heads > 0 && value_heads != nkv);
    return run_prefill(q, (long long)nh * hd, q_stride, out, k_pool, v_pool, num_pages, entries, entry, page_tokens,
                       block_table, table_width, cu_q, ctx_lens, num_seqs, num_tokens, max_q_len, nh, nkv, hd, scale,
                       prefill_seqs, num_prefill_seqs, error, false, window, nullptr, nullptr, nullptr, 0, stream, bounded,
                       chunk, softcap, value_heads, nullptr, 0, sink);
}

// Causal softmax attention of prompt portions over keys and values that lie in matrices of their own,
// k [kv_rows, nkv * hd] and v [kv_rows, nkv * hd] (bfloat16, rows back to back), request s's key j in row kv_start[s] + j
// (kv_start: int32 [num_seqs] on the device; ctx_lens[s] keys a request).  For keys and values that are worked out
// for the step instead of read from pages.  Queries [T, q_stride] in a matrix of their own, head h's hd columns from
// h * q_head_cols on.  With `rot` > 0 a score also has q_rot . k_rot, q_rot [T, nh * 64] (a head's channels past `rot` zero)
// and k_rot one row of `rot` channels a key for all heads, k_rot_stride elements apart, in the same row order as k.
// `sinks` [nh] (null: none): a score a head that joins every softmax's sum without a key or a value.
TS_API int ts_prefill_attention_tcgen05_dense(const void* q, long long q_stride, void* out, const void* k, const void* v,
                                              long long kv_rows, const int* kv_start, const int* cu_q, const int* ctx_lens,
                                              int num_seqs, int num_tokens, int max_q_len, int nh, int nkv, int hd,
                                              float scale, const int* prefill_seqs, int num_prefill_seqs, int* error,
                                              int q_head_cols, const void* q_rot, const void* k_rot, long long k_rot_stride, int rot,
                                              const float* sinks, cudaStream_t stream) {
    TS_REQUIRE(kv_start != nullptr, "attention_tcgen05: the first rows of the requests' keys are needed");
    TS_REQUIRE(q_head_cols >= hd && (rot == 0 || (q_rot && k_rot)), "attention_tcgen05: the queries' columns, or the shared key part");
    const SharedPart shared{q_rot, k_rot, k_rot_stride, rot, q_head_cols, sinks};
    return run_prefill(q, (long long)nh * q_head_cols, q_stride, out, k, v, 1, 1, 0, 64, nullptr, 1, cu_q, ctx_lens, num_seqs, num_tokens,
                       max_q_len, nh, nkv, hd, scale, prefill_seqs, num_prefill_seqs, error, false, 0, nullptr, nullptr,
                       nullptr, 0, stream, false, 0, 0.f, 0, kv_start, kv_rows, -INFINITY, &shared);
}
