// The recurrences of linear_recurrence.cu over prompt portions, sixteen tokens at a time.
//
// What one token writes into the state the next one reads, so a scan token by token is a chain.  Inside a tile
// of B = 16 tokens the chain can be written out (S_0 the state before the tile, columns of S independent):
//
// Delta rule with one decay a head (a_t), step size b_t.  With c_t = a_1 ... a_t and G[t][j] = a_(j+1) ... a_t,
//   u_t = b_t (v_t - c_t S_0^T k_t - sum_{j<t} G[t][j] (k_j . k_t) u_j)
//   o_t = c_t S_0^T q_t + sum_{j<=t} G[t][j] (k_j . q_t) u_j,     S_B = c_B S_0 + sum_j G[B][j] k_j u_j^T
// The first line is a unit lower triangular system, U = M diag(b) (V - diag(c) R), R = S_0^T K, with
// M = (I + A)^-1, A[t][j] = b_t G[t][j] (k_j . k_t) for j < t (the entries of M stay below one in size: each is
// a product of the contractions a (I - b k k^T) between two unit vectors).
//
// Time mixing with decays per channel (a_(t,i)) and a bonus.  With d_(t,i) = a_(1,i) ... a_(t,i),
//   o_t = sum_i r_(t,i) d_(t-1,i) S_0[i] + sum_{j<t} P[t][j] v_j + bonus_t v_t,
//   P[t][j] = sum_i r_(t,i) k_(j,i) a_(j+1,i) ... a_(t-1,i),   S_B = d_B S_0 + sum_j (k_j a_(j+1) ... a_B) v_j^T
//
// No decay is ever divided by another: products of decays are taken as they are needed.
//
// A first kernel works out, per tile and q/k head (time mixing: head), what all columns of the state share: the
// "pack" (16 rows for the q side, 16 for the k side, one with the channels' decays over the tile) and the coefficients
// (W = M diag(b); P W, so that O = diag(c) S_0^T Q + (P W) (V - diag(c) R) does not wait for U; c; G[B]).  The second
// kernel walks the tiles: a CTA owns one request, one head and 16 columns of the state and does three small
// products a tile on tensor cores,
//   [q side | k side] S_0   (each warp its own rows of S, the partial sums meet in shared memory in warp order)
//   U (two warps) and O (two warps) from the 16 x 16 coefficients
//   K^T U, by which the state moves on
// with the next tile's pack and coefficients on their way by cp.async.  The products are float32 to rounding: every
// factor is split into two TF32 numbers, x = hi + lo, and hi hi + hi lo + lo hi is summed in float32 (what is
// left out is 2^-22 of a term).  The state stays in registers, in the layout in which the third product
// leaves it (its transpose) and the first one takes it; the update is added to it by an ordinary fused
// multiply-add, so that what the tensor cores round is the update and not the state.
//
// A tile cut short by the portion's end is filled up with tokens that change nothing (k = 0, decay 1).  Requests that
// feed one token are left to the other scan.  Tiles count from the portion's first token, so where a prompt was cut
// moves sums inside rounding only.
#include "common.cuh"

namespace {

constexpr int B = 16;              // tokens a tile
constexpr int COLS = 16;           // value channels a CTA
constexpr int WARPS = 4, THREADS = WARPS * 32;   // of the scan
constexpr int CP = 20;             // pitch of a coefficient matrix: a warp's fragment loads fall into different banks
constexpr int COEF = 2 * B * CP + 2 * B;   // W [16][20], P W (time mixing: P) [16][20], c [16], g [16]
constexpr int RP = 24;             // pitch of the partial sums and of U: likewise
// A pack: 33 rows (16 q-side, 16 k-side, the channels' decays) of `rows` floats and a pad that does the same for it.
__host__ __device__ constexpr int pack_pitch(int rows) { return rows + 8; }
__host__ __device__ constexpr int pack_floats(int rows) { return (2 * B + 1) * pack_pitch(rows); }
enum { DELTA = 0, MIX = 1 };

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// Where a request's tiles lie among all tiles: request s's first at cu_q[s] / 16 + s.  Every request has room for its own
// (a portion of n tokens takes ceil(n / 16), and the next request's first lies at least that much further on).
__device__ __forceinline__ long long tile_slot(int seq, int begin, int tile) { return begin / B + seq + tile; }

struct PrepareArgs {
    const void* q; const void* k; long long qk_stride;   // delta: float32 after the convolution; mixing: r, k as projected
    const float* gates;                                  // delta: [tokens, 2 heads], logits of b, then of the decay; mixing: z [tokens, heads * dim]
    const float* bias;                                   // delta: dt_bias [heads]; mixing: w0 [heads * dim]
    const float* rate;                                   // delta: A_log [heads]; mixing: u [heads * dim]
    const int* cu_q; const int* prefill_seqs;
    float* pack; float* coef;
    int heads, kv_heads, dim, rows;                      // rows: dim rounded up to what the scan's threads hold
    float unit_eps, q_scale;
};

// grid (tiles, q/k heads, portions), 128 threads
__global__ void __launch_bounds__(128) delta_tile_prepare_kernel(PrepareArgs p) {
    extern __shared__ float smem[];
    const int seq = p.prefill_seqs[blockIdx.z], tile = blockIdx.x, g = blockIdx.y;
    if (seq < 0) return;                                 // a padding entry of the list
    const int begin = p.cu_q[seq], n = p.cu_q[seq + 1] - begin;
    if (n <= 1 || tile * B >= n) return;
    const int t0 = begin + tile * B, m = min(B, n - tile * B);
    const int pitch = p.rows + 1;
    float* qs = smem;                                    // [16][pitch]
    float* ks = qs + B * pitch;
    float* kk = ks + B * pitch;                          // [16][17]: k_t . k_j
    float* qk = kk + B * (B + 1);                        // q_t . k_j
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int t = warp; t < B; t += 4) {
        const float* qr = (const float*)p.q + (long long)(t0 + t) * p.qk_stride + (long long)g * p.dim;
        const float* kr = (const float*)p.k + (long long)(t0 + t) * p.qk_stride + (long long)g * p.dim;
        float sq = 0.f, sk = 0.f;
        for (int i = lane; i < p.rows; i += 32) {
            const bool ok = t < m && i < p.dim;
            const float qv = ok ? qr[i] : 0.f, kv = ok ? kr[i] : 0.f;
            qs[t * pitch + i] = qv;
            ks[t * pitch + i] = kv;
            sq += qv * qv;
            sk += kv * kv;
        }
        const float iq = p.q_scale / sqrtf(warp_sum(sq) + p.unit_eps), ik = 1.f / sqrtf(warp_sum(sk) + p.unit_eps);
        for (int i = lane; i < p.rows; i += 32) { qs[t * pitch + i] *= iq; ks[t * pitch + i] *= ik; }   // the lane's own elements
    }
    __syncthreads();
    const long long slot = tile_slot(seq, begin, tile);
    float* pack = p.pack + (slot * p.kv_heads + g) * pack_floats(p.rows);
    for (int e = threadIdx.x; e < B * p.rows; e += 128) {
        const int t = e / p.rows, i = e % p.rows;
        pack[t * pack_pitch(p.rows) + i] = qs[t * pitch + i];
        pack[(B + t) * pack_pitch(p.rows) + i] = ks[t * pitch + i];
    }
    {   // the dot products: thread (t, pair of j)
        const int t = threadIdx.x >> 3, j = (threadIdx.x & 7) * 2;
        float k0 = 0.f, k1 = 0.f, q0 = 0.f, q1 = 0.f;
        for (int i = 0; i < p.dim; ++i) {
            const float kt = ks[t * pitch + i], qt = qs[t * pitch + i], a = ks[j * pitch + i], b = ks[(j + 1) * pitch + i];
            k0 = fmaf(kt, a, k0); k1 = fmaf(kt, b, k1);
            q0 = fmaf(qt, a, q0); q1 = fmaf(qt, b, q1);
        }
        kk[t * (B + 1) + j] = k0; kk[t * (B + 1) + j + 1] = k1;
        qk[t * (B + 1) + j] = q0; qk[t * (B + 1) + j + 1] = q1;
    }
    __syncthreads();
    // a warp a value head of the group; lane j holds column j (lanes 16..31 mirror lanes 0..15 and store nothing)
    const int group = p.heads / p.kv_heads, j = lane & (B - 1);
    for (int hh = warp; hh < group; hh += 4) {
        const int h = g * group + hh;
        float b = 0.f, a = 1.f;                          // a token past the portion's end changes nothing
        if (j < m) {
            const float* gr = p.gates + (long long)(t0 + j) * 2 * p.heads;
            b = 1.f / (1.f + expf(-gr[h]));
            a = expf(-expf(p.rate[h]) * softplus(gr[p.heads + h] + p.bias[h]));
        }
        float* out = p.coef + (slot * p.heads + h) * COEF;
        float M[B], P[B];
        float decay = 1.f, c = 1.f, c_own = 1.f;         // G[t][j] as t runs; c_t; c_j
#pragma unroll
        for (int t = 0; t < B; ++t) {
            const float at = __shfl_sync(0xffffffffu, a, t), bt = __shfl_sync(0xffffffffu, b, t);
            c *= at;
            if (t == j) c_own = c;
            if (t > j) decay *= at;
            const float A = t > j ? bt * decay * kk[t * (B + 1) + j] : 0.f;
            P[t] = t >= j ? decay * qk[t * (B + 1) + j] : 0.f;
            float row = t == j ? 1.f : 0.f;              // M[t][j] = delta - sum_s A[t][s] M[s][j]
#pragma unroll
            for (int s = 0; s < t; ++s) row = fmaf(-__shfl_sync(0xffffffffu, A, s), M[s], row);
            M[t] = row;
        }
#pragma unroll
        for (int t = 0; t < B; ++t) {
            float pw = 0.f;
#pragma unroll
            for (int s = 0; s <= t; ++s) pw = fmaf(__shfl_sync(0xffffffffu, P[t], s), M[s] * b, pw);
            if (lane < B) {
                out[t * CP + j] = M[t] * b;
                out[B * CP + t * CP + j] = pw;
            }
        }
        if (lane < B) {
            out[2 * B * CP + j] = c_own;
            out[2 * B * CP + B + j] = decay;
        }
    }
}

// grid (tiles, heads, portions), 128 threads: thread (j, channel group of 8) for the coefficients
template <typename T>
__global__ void __launch_bounds__(128) mix_tile_prepare_kernel(PrepareArgs p) {
    extern __shared__ float smem[];
    const int seq = p.prefill_seqs[blockIdx.z], tile = blockIdx.x, h = blockIdx.y;
    if (seq < 0) return;
    const int begin = p.cu_q[seq], n = p.cu_q[seq + 1] - begin;
    if (n <= 1 || tile * B >= n) return;
    const int t0 = begin + tile * B, m = min(B, n - tile * B);
    const int pitch = p.rows + 1;
    float* rs = smem;                                    // [16][pitch]
    float* ks = rs + B * pitch;
    float* as = ks + B * pitch;
    const long long slot = tile_slot(seq, begin, tile);
    float* pack = p.pack + (slot * p.heads + h) * pack_floats(p.rows);
    const long long width = (long long)p.heads * p.dim, hc = (long long)h * p.dim;
    for (int e = threadIdx.x; e < B * p.rows; e += 128) {
        const int t = e / p.rows, i = e % p.rows;
        const bool ok = t < m && i < p.dim;
        float rv = 0.f, kv = 0.f, av = 1.f;
        if (ok) {
            rv = to_float<T>(((const T*)p.q)[(long long)(t0 + t) * p.qk_stride + hc + i]);
            kv = to_float<T>(((const T*)p.k)[(long long)(t0 + t) * p.qk_stride + hc + i]);
            av = expf(-expf(p.gates[(long long)(t0 + t) * width + hc + i] + p.bias[hc + i]));
        }
        rs[t * pitch + i] = rv;
        ks[t * pitch + i] = kv;
        as[t * pitch + i] = av;
    }
    __syncthreads();
    {   // P[t][j], t >= j: thread j = tid / 8 walks t with the running product of its channels
        const int j = threadIdx.x >> 3, part = threadIdx.x & 7;
        float sum[B];
#pragma unroll
        for (int t = 0; t < B; ++t) sum[t] = 0.f;
        for (int i = part; i < p.dim; i += 8) {
            float run = ks[j * pitch + i];
            const float own = run * rs[j * pitch + i] * p.rate[hc + i];                 // the bonus's share
#pragma unroll
            for (int t = 0; t < B; ++t) {
                if (t == j) sum[t] += own;
                if (t > j) {
                    sum[t] = fmaf(rs[t * pitch + i], run, sum[t]);
                    run *= as[t * pitch + i];
                }
            }
        }
        float* out = p.coef + (slot * p.heads + h) * COEF + B * CP;
#pragma unroll
        for (int t = 0; t < B; ++t) {
            float s = sum[t];
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
            if (part == 0) out[t * CP + j] = s;                                         // 0 where t < j
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.rows; i += 128) {    // a thread a channel: products from the left and from the right
        const int pp = pack_pitch(p.rows);
        float left = 1.f, right = 1.f;
        for (int t = 0; t < B; ++t) {
            pack[t * pp + i] = rs[t * pitch + i] * left;
            left *= as[t * pitch + i];
        }
        for (int t = B - 1; t >= 0; --t) {
            pack[(B + t) * pp + i] = ks[t * pitch + i] * right;
            right *= as[t * pitch + i];
        }
        pack[2 * B * pp + i] = left;
    }
}

struct ScanArgs {
    const float* pack; const float* coef;
    const void* v; long long v_stride;                   // elements between tokens; a head's values start at h * vdim
    const int* cu_q; const int* slots; const int* prefill_seqs;
    float* state; long long slot_stride;                 // floats between slots; a slot holds [heads, dim, vdim]
    float* out;                                          // [tokens, heads * vdim] float32
    int heads, qk_group, dim, vdim;
};

__device__ __forceinline__ void cp16(void* smem, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}

// A float32 number as the sum of two TF32 numbers (11 significant bits each): hi is x to the nearest (half of its last
// place added before the low 13 bits go), lo what is left, of which the tensor cores read the leading bits: 2^-23 of x is lost.
struct Split { uint32_t hi, lo; };
__device__ __forceinline__ Split split_tf32(float x) {
    Split s;
    s.hi = (__float_as_uint(x) + 0x1000u) & 0xffffe000u;
    s.lo = __float_as_uint(x - __uint_as_float(s.hi));
    return s;
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct SplitA { uint32_t hi[4], lo[4]; };
__device__ __forceinline__ SplitA split_a(float a0, float a1, float a2, float a3) {
    const Split s0 = split_tf32(a0), s1 = split_tf32(a1), s2 = split_tf32(a2), s3 = split_tf32(a3);
    return SplitA{{s0.hi, s1.hi, s2.hi, s3.hi}, {s0.lo, s1.lo, s2.lo, s3.lo}};
}
// The two large and the small parts of a product of split factors, each in an accumulator of its own (no long chain).
__device__ __forceinline__ void mma_split(float (&big)[4], float (&small)[4], const SplitA& a, Split b0, Split b1) {
    mma_tf32(big, a.hi, b0.hi, b1.hi);
    mma_tf32(small, a.hi, b0.lo, b1.lo);
    mma_tf32(small, a.lo, b0.hi, b1.hi);
}

// NT: eights of rows of the state a warp holds.  Fragments of mma.m16n8k8, lane = 4 r + c (r 0..7, c 0..3):
//   A (16 x 8): (r, c), (r + 8, c), (r, c + 4), (r + 8, c + 4);   B (8 x 8): (c, r), (c + 4, r);
//   C (16 x 8): (r, 2c), (r, 2c + 1), (r + 8, 2c), (r + 8, 2c + 1).
// The state is held as C fragments of S^T (16 columns x 8 rows of S).  Read as B fragments of S they hold rows 2c and
// 2c + 1 where the product counts k = c and c + 4: the A side takes its k in the same order.
template <typename T, int NT, int MODE>
__global__ void __launch_bounds__(THREADS) recurrence_tiles_kernel(ScanArgs p) {
    constexpr int WROWS = 8 * NT, ROWS = WARPS * WROWS;  // rows of a warp; rows of the state
    constexpr int PP = pack_pitch(ROWS);
    constexpr int PACK = pack_floats(ROWS), STAGE = PACK + COEF;
    constexpr int TQ = MODE == DELTA ? 2 * B : B;        // rows of the pack that meet S_0
    extern __shared__ __align__(16) float smem[];
    float* red = smem + 2 * STAGE;                       // [WARPS][TQ][RP]
    float* G_s = red + WARPS * TQ * RP;                  // [B][RP]: what the state's update takes, G[B] U or V
    const int seq = p.prefill_seqs[blockIdx.z], h = blockIdx.y, j0 = blockIdx.x * COLS;
    if (seq < 0) return;
    const int begin = p.cu_q[seq], n = p.cu_q[seq + 1] - begin, slot = p.slots[seq];
    if (n <= 1 || slot < 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane >> 2, c = lane & 3;
    const int qk_heads = p.heads / p.qk_group, qh = h / p.qk_group;
    float* st = p.state + (long long)slot * p.slot_stride + (long long)h * p.dim * p.vdim;

    auto element = [&](int nt, int e, int& i, int& j) {  // row and column of S of register e of tile nt
        i = warp * WROWS + 8 * nt + 2 * c + (e & 1);
        j = j0 + r + 8 * (e >> 1);
        return i < p.dim && j < p.vdim;
    };
    float S[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            int i, j;
            S[nt][e] = element(nt, e, i, j) ? st[(long long)i * p.vdim + j] : 0.f;
        }
    const int tiles = (n + B - 1) / B;
    const long long first = tile_slot(seq, begin, 0);
    auto issue = [&](int tile) {
        float* stage = smem + (tile & 1) * STAGE;
        const float* pack = p.pack + ((first + tile) * qk_heads + qh) * (long long)PACK;
        const float* coef = p.coef + ((first + tile) * p.heads + h) * (long long)COEF;
#pragma unroll
        for (int e = 0; e < PACK / 4; e += THREADS)
            if (e + tid < PACK / 4) cp16(stage + 4 * (e + tid), pack + 4 * (e + tid));
#pragma unroll
        for (int e = 0; e < COEF / 4; e += THREADS)
            if (e + tid < COEF / 4) cp16(stage + PACK + 4 * (e + tid), coef + 4 * (e + tid));
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    // Warps 0 and 1 make U (time mixing: hand the values on), warps 2 and 3 O, for columns 8 (warp & 1) .. + 7 each.
    // Their values, as B fragments: tokens c, c + 4, c + 8, c + 12 of column r.
    const int nt_uo = warp & 1, col = 8 * nt_uo + r;
    const bool makes_o = warp >= 2;
    static_assert(WARPS == 4, "two warps make U, two make O");
    const T* v = (const T*)p.v + (long long)(begin + c) * p.v_stride + (long long)h * p.vdim + j0 + col;
    T vnow[4], vnext[4];
    auto fetch_v = [&](int tile, T (&x)[4]) {            // as loaded: converting would wait for the load
#pragma unroll
        for (int k = 0; k < 4; ++k)
            x[k] = tile * B + c + 4 * k < n && j0 + col < p.vdim ? v[(long long)(tile * B + 4 * k) * p.v_stride] : from_float<T>(0.f);
    };
    issue(0);
    fetch_v(0, vnow);
#pragma unroll
    for (int k = 0; k < 4; ++k) vnext[k] = vnow[k];
    for (int tile = 0; tile < tiles; ++tile) {
        asm volatile("cp.async.wait_all;\n" ::: "memory");
        __syncthreads();                                 // the tile's inputs are in; the other stage, U and the sums have been read
        if (tile + 1 < tiles) {
            issue(tile + 1);
            fetch_v(tile + 1, vnext);
        }
        const float* pack = smem + (tile & 1) * STAGE;
        const float* coef = pack + PACK;
        // product 1: the pack's rows against this warp's rows of S
        {
            float big[TQ / B][2][4] = {}, small[TQ / B][2][4] = {};
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
                Split b[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) b[e] = split_tf32(S[nt][e]);
#pragma unroll
                for (int mt = 0; mt < TQ / B; ++mt) {
                    const float* row = pack + (mt * B + r) * PP + warp * WROWS + 8 * nt + 2 * c;
                    const float2 lo = *reinterpret_cast<const float2*>(row), hi = *reinterpret_cast<const float2*>(row + 8 * PP);
                    const SplitA a = split_a(lo.x, hi.x, lo.y, hi.y);
                    mma_split(big[mt][0], small[mt][0], a, b[0], b[1]);
                    mma_split(big[mt][1], small[mt][1], a, b[2], b[3]);
                }
            }
#pragma unroll
            for (int mt = 0; mt < TQ / B; ++mt)
#pragma unroll
                for (int nj = 0; nj < 2; ++nj)
#pragma unroll
                    for (int half = 0; half < 2; ++half)
                        *reinterpret_cast<float2*>(red + (warp * TQ + mt * B + r + 8 * half) * RP + 8 * nj + 2 * c) =
                            make_float2(big[mt][nj][2 * half] + small[mt][nj][2 * half],
                                        big[mt][nj][2 * half + 1] + small[mt][nj][2 * half + 1]);
        }
        __syncthreads();                                 // the partial sums are in
        {
            float x[4];                                  // V - c R (time mixing: V) at tokens c + 4 k of column `col`
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                x[k] = to_float<T>(vnow[k]);
                if (MODE == DELTA) {
                    float sum = 0.f;
#pragma unroll
                    for (int w = 0; w < WARPS; ++w) sum += red[(w * TQ + B + c + 4 * k) * RP + col];
                    x[k] = fmaf(-coef[2 * B * CP + c + 4 * k], sum, x[k]);
                }
            }
            if (MODE == MIX && !makes_o) {
#pragma unroll
                for (int k = 0; k < 4; ++k) G_s[(c + 4 * k) * RP + col] = x[k];
            }
            if (MODE == DELTA || makes_o) {
                const float* m = coef + (makes_o ? B * CP : 0);
                float big[4] = {}, small[4] = {};
#pragma unroll
                for (int ks = 0; ks < 2; ++ks) {
                    const float* a = m + r * CP + 8 * ks + c;
                    mma_split(big, small, split_a(a[0], a[8 * CP], a[4], a[8 * CP + 4]), split_tf32(x[2 * ks]), split_tf32(x[2 * ks + 1]));
                }
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int t = r + 8 * half;
                    float y0 = big[2 * half] + small[2 * half], y1 = big[2 * half + 1] + small[2 * half + 1];
                    if (!makes_o) {
                        const float g = coef[2 * B * CP + B + t];
                        *reinterpret_cast<float2*>(G_s + t * RP + 8 * nt_uo + 2 * c) = make_float2(g * y0, g * y1);
                    } else {
                        float q0 = 0.f, q1 = 0.f;
#pragma unroll
                        for (int w = 0; w < WARPS; ++w) {
                            const float2 q = *reinterpret_cast<const float2*>(red + (w * TQ + t) * RP + 8 * nt_uo + 2 * c);
                            q0 += q.x;
                            q1 += q.y;
                        }
                        const float ct = MODE == DELTA ? coef[2 * B * CP + t] : 1.f;
                        y0 = fmaf(ct, q0, y0);
                        y1 = fmaf(ct, q1, y1);
                        const int j = j0 + 8 * nt_uo + 2 * c;
                        if (tile * B + t < n) {
                            float* dst = p.out + ((long long)(begin + tile * B + t) * p.heads + h) * p.vdim + j;
                            if (j < p.vdim) dst[0] = y0;
                            if (j + 1 < p.vdim) dst[1] = y1;
                        }
                    }
                }
            }
        }
        __syncthreads();                                 // what the update takes is in
        // product 3, S^T <- decay S^T + G^T K, and the state after the tile
        {
            SplitA a[2];
#pragma unroll
            for (int ks = 0; ks < 2; ++ks) {
                const float* g = G_s + (8 * ks + c) * RP + r;
                a[ks] = split_a(g[0], g[8], g[4 * RP], g[4 * RP + 8]);
            }
            const float cB = MODE == DELTA ? coef[2 * B * CP + B - 1] : 1.f;
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
                float big[4] = {}, small[4] = {};
                const float* k = pack + (B + c) * PP + warp * WROWS + 8 * nt + r;
#pragma unroll
                for (int ks = 0; ks < 2; ++ks)
                    mma_split(big, small, a[ks], split_tf32(k[8 * ks * PP]), split_tf32(k[(8 * ks + 4) * PP]));
                float2 d = make_float2(cB, cB);
                if (MODE == MIX) d = *reinterpret_cast<const float2*>(pack + 2 * B * PP + warp * WROWS + 8 * nt + 2 * c);
                S[nt][0] = fmaf(d.x, S[nt][0], big[0] + small[0]);
                S[nt][1] = fmaf(d.y, S[nt][1], big[1] + small[1]);
                S[nt][2] = fmaf(d.x, S[nt][2], big[2] + small[2]);
                S[nt][3] = fmaf(d.y, S[nt][3], big[3] + small[3]);
            }
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) vnow[k] = vnext[k];
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            int i, j;
            if (element(nt, e, i, j)) st[(long long)i * p.vdim + j] = S[nt][e];
        }
}

int padded_rows(int dim) { return dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

template <typename T, int MODE>
int launch_scan(const ScanArgs& p, int portions, cudaStream_t stream) {
    const dim3 grid((p.vdim + COLS - 1) / COLS, p.heads, portions);
#define TS_TILES(NT)                                                                                                 \
    do {                                                                                                             \
        constexpr int TQ = MODE == DELTA ? 2 * B : B;                                                                \
        const size_t smem = sizeof(float) * (2 * (pack_floats(WARPS * 8 * NT) + COEF) + (WARPS * TQ + B) * RP);      \
        auto kernel = recurrence_tiles_kernel<T, NT, MODE>;                                                          \
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                        \
        kernel<<<grid, THREADS, smem, stream>>>(p);                                                                  \
    } while (0)
    const int rows = padded_rows(p.dim);
    if (rows == 64) TS_TILES(2);
    else if (rows == 128) TS_TILES(4);
    else TS_TILES(8);
#undef TS_TILES
    TS_LAUNCH_CHECK("recurrence_tiles");
    return 0;
}

}  // namespace

// Floats of the two buffers the tile kernels need: packs (`heads`: the q/k heads) and coefficients (`heads`: the value heads).
TS_API long long ts_recurrence_tiles_pack_floats(int num_tokens, int num_seqs, int heads, int dim) {
    return ((long long)num_tokens / B + num_seqs + 1) * heads * pack_floats(padded_rows(dim));
}
TS_API long long ts_recurrence_tiles_coef_floats(int num_tokens, int num_seqs, int heads) {
    return ((long long)num_tokens / B + num_seqs + 1) * heads * COEF;
}

// The delta rule with one decay a head over a step's prompt portions (`prefill_seqs`: the requests that feed more than
// one token, -1: none; `max_q_len` bounds their lengths).  q, k: float32 [tokens, kv_heads * dim] stretches after the
// convolution; gates [tokens, 2 heads]; v [tokens, heads * vdim] float32 stretch.  Rows of other requests are left alone.
TS_API int ts_delta_tiles(const float* q, const float* k, long long qk_stride, const float* gates, const float* dt_bias,
                          const float* a_log, const float* v, long long v_stride, const int* cu_q, const int* slots,
                          const int* prefill_seqs, int portions, int max_q_len, float* state, long long slot_stride,
                          float* pack, float* coef, float* out, int heads, int kv_heads, int dim, int vdim,
                          float unit_eps, float q_scale, cudaStream_t stream) {
    TS_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && dim <= 256 && vdim > 0,
               "delta_tiles: %d heads over %d q/k heads of %d channels", heads, kv_heads, dim);
    TS_REQUIRE(slot_stride >= (long long)heads * dim * vdim, "delta_tiles: a state slot is too small");
    TS_REQUIRE(portions >= 0 && portions <= 65535 && heads <= 65535, "delta_tiles: grid too large");
    if (portions == 0 || max_q_len <= 1) return 0;
    PrepareArgs a{q, k, qk_stride, gates, dt_bias, a_log, cu_q, prefill_seqs, pack, coef, heads, kv_heads, dim, padded_rows(dim),
                  unit_eps, q_scale};
    const size_t smem = sizeof(float) * (2 * B * (a.rows + 1) + 2 * B * (B + 1));
    delta_tile_prepare_kernel<<<dim3((max_q_len + B - 1) / B, kv_heads, portions), 128, smem, stream>>>(a);
    TS_LAUNCH_CHECK("delta_tiles (prepare)");
    ScanArgs s{pack, coef, v, v_stride, cu_q, slots, prefill_seqs, state, slot_stride, out, heads, heads / kv_heads, dim, vdim};
    return launch_scan<float, DELTA>(s, portions, stream);
}

// Time mixing over a step's prompt portions: r, k, v [tokens, heads * dim] of one dtype (r and k with one row stride),
// z float32 [tokens, heads * dim], w0 and u [heads * dim].
TS_API int ts_mix_tiles(const void* r, const void* k, long long rk_stride, const float* z, const float* w0, const float* u,
                        const void* v, long long v_stride, const int* cu_q, const int* slots, const int* prefill_seqs,
                        int portions, int max_q_len, float* state, long long slot_stride, float* pack, float* coef,
                        float* out, int heads, int dim, int dtype, cudaStream_t stream) {
    TS_REQUIRE(heads > 0 && dim > 0 && dim <= 256, "mix_tiles: %d heads of %d channels", heads, dim);
    TS_REQUIRE(slot_stride >= (long long)heads * dim * dim, "mix_tiles: a state slot is too small");
    TS_REQUIRE(portions >= 0 && portions <= 65535 && heads <= 65535, "mix_tiles: grid too large");
    if (portions == 0 || max_q_len <= 1) return 0;
    PrepareArgs a{r, k, rk_stride, z, w0, u, cu_q, prefill_seqs, pack, coef, heads, heads, dim, padded_rows(dim), 0.f, 1.f};
    const size_t smem = sizeof(float) * (3 * B * (a.rows + 1));
    const dim3 grid((max_q_len + B - 1) / B, heads, portions);
    ScanArgs s{pack, coef, v, v_stride, cu_q, slots, prefill_seqs, state, slot_stride, out, heads, 1, dim, dim};
    if (dtype == TS_F32) {
        cudaFuncSetAttribute(mix_tile_prepare_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        mix_tile_prepare_kernel<float><<<grid, 128, smem, stream>>>(a);
        TS_LAUNCH_CHECK("mix_tiles (prepare)");
        return launch_scan<float, MIX>(s, portions, stream);
    }
    if (dtype == TS_BF16) {
        cudaFuncSetAttribute(mix_tile_prepare_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        mix_tile_prepare_kernel<__nv_bfloat16><<<grid, 128, smem, stream>>>(a);
        TS_LAUNCH_CHECK("mix_tiles (prepare)");
        return launch_scan<__nv_bfloat16, MIX>(s, portions, stream);
    }
    return ts_fail("mix_tiles: unknown dtype code %d", dtype);
}
