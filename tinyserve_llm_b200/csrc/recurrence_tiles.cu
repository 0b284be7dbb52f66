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
// No decay is ever divided by another: products of decays are taken as they are needed.  Everything is float32.
// A first kernel works out, per tile and q/k head (time mixing: head), what all columns of the state share:
// the "pack", a row per key channel [16 q-side entries | 16 k-side entries | the row's decay over the tile], and
// the coefficients (W = M diag(b), P, c, G[B]).  The second kernel walks the tiles: a CTA owns one request, one
// head and 16 columns of the state and does three small products a tile,
//   S_0^T [q-side | k-side]  (rows of S split over the warps, 4 x 4 outputs a thread, partial sums added up in order)
//   U and O from the 16 x 16 coefficients,  S_B  (the state's own 4 columns x R rows a thread in registers)
// with the next tile's pack and coefficients on their way by cp.async.  A tile cut short by the portion's end is
// filled up with tokens that change nothing (k = 0, decay 1).  Requests that feed one token are left to the
// other scan.  Tiles count from the portion's first token, so where a prompt was cut moves sums inside
// rounding only.
#include "common.cuh"

namespace {

constexpr int B = 16;              // tokens a tile
constexpr int COLS = 16;           // value channels a CTA
constexpr int ROW = 36;            // floats a pack row: 16 + 16 entries, the row's decay, 3 unused (rows start 16-byte aligned)
constexpr int COEF = 2 * B * B + 2 * B;   // W [16][16], P [16][16], c [16], g [16]
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
    float* pack = p.pack + (slot * p.kv_heads + g) * p.rows * ROW;
    for (int e = threadIdx.x; e < p.rows * 32; e += 128) {
        const int i = e >> 5, t = e & 31;
        pack[i * ROW + t] = t < B ? qs[t * pitch + i] : ks[(t - B) * pitch + i];
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
        float M[B];
        float decay = 1.f, c = 1.f, c_own = 1.f;         // G[t][j] as t runs; c_t; c_j
#pragma unroll
        for (int t = 0; t < B; ++t) {
            const float at = __shfl_sync(0xffffffffu, a, t), bt = __shfl_sync(0xffffffffu, b, t);
            c *= at;
            if (t == j) c_own = c;
            if (t > j) decay *= at;
            const float A = t > j ? bt * decay * kk[t * (B + 1) + j] : 0.f;
            const float P = t >= j ? decay * qk[t * (B + 1) + j] : 0.f;
            float row = t == j ? 1.f : 0.f;              // M[t][j] = delta - sum_s A[t][s] M[s][j]
#pragma unroll
            for (int s = 0; s < t; ++s) row = fmaf(-__shfl_sync(0xffffffffu, A, s), M[s], row);
            M[t] = row;
            if (lane < B) {
                out[t * B + j] = row * b;
                out[B * B + t * B + j] = P;
            }
        }
        if (lane < B) {
            out[2 * B * B + j] = c_own;
            out[2 * B * B + B + j] = decay;
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
    float* pack = p.pack + (slot * p.heads + h) * p.rows * ROW;
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
        float* out = p.coef + (slot * p.heads + h) * COEF + B * B;
#pragma unroll
        for (int t = 0; t < B; ++t) {
            float s = sum[t];
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
            if (part == 0) out[t * B + j] = s;                                          // 0 where t < j
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.rows; i += 128) {    // a thread a channel: products from the left and from the right
        float left = 1.f, right = 1.f;
        for (int t = 0; t < B; ++t) {
            rs[t * pitch + i] *= left;
            left *= as[t * pitch + i];
        }
        for (int t = B - 1; t >= 0; --t) {
            ks[t * pitch + i] *= right;
            right *= as[t * pitch + i];
        }
        pack[i * ROW + 2 * B] = left;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < p.rows * 32; e += 128) {
        const int i = e >> 5, t = e & 31;
        pack[i * ROW + t] = t < B ? rs[t * pitch + i] : ks[(t - B) * pitch + i];
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

// R: rows of the state a thread holds (32 R rows in all)
template <typename T, int R, int MODE>
__global__ void __launch_bounds__(128) recurrence_tiles_kernel(ScanArgs p) {
    constexpr int ROWS = 32 * R, WROWS = 8 * R;          // rows of the state; rows of a warp
    constexpr int STAGE = ROWS * ROW + COEF;             // floats a stage
    constexpr int RP = COLS + 4;                         // pitch of the partial sums
    constexpr int TQ = MODE == DELTA ? 32 : 16;          // entries of a pack row that meet S_0
    extern __shared__ __align__(16) float smem[];
    float* S_s = smem + 2 * STAGE;                       // [ROWS][COLS]
    float* red = S_s + ROWS * COLS;                      // [4][TQ][RP]
    float* X_s = red + 4 * TQ * RP;                      // [B][COLS]: V - c R; mixing: V
    float* U_s = X_s + B * COLS;                         // [B][COLS]: U (delta)
    float* G_s = U_s + B * COLS;                         // [B][COLS]: G[B] U (delta)
    const int seq = p.prefill_seqs[blockIdx.z], h = blockIdx.y, j0 = blockIdx.x * COLS;
    if (seq < 0) return;
    const int begin = p.cu_q[seq], n = p.cu_q[seq + 1] - begin, slot = p.slots[seq];
    if (n <= 1 || slot < 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int tg = lane >> 2, cg = lane & 3;             // product 1: entries of group tg, columns 4 cg ..; product 3: rows tg + 8 e
    const int qk_heads = p.heads / p.qk_group, qh = h / p.qk_group;
    float* st = p.state + (long long)slot * p.slot_stride + (long long)h * p.dim * p.vdim;

    float S[R][4];
#pragma unroll
    for (int e = 0; e < R; ++e) {
        const int i = warp * WROWS + tg + 8 * e;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int j = j0 + 4 * cg + c;
            S[e][c] = i < p.dim && j < p.vdim ? st[(long long)i * p.vdim + j] : 0.f;
        }
        *reinterpret_cast<float4*>(S_s + i * COLS + 4 * cg) = make_float4(S[e][0], S[e][1], S[e][2], S[e][3]);
    }
    const int tiles = (n + B - 1) / B;
    const long long first = tile_slot(seq, begin, 0);
    auto issue = [&](int tile) {
        float* stage = smem + (tile & 1) * STAGE;
        const float* pack = p.pack + ((first + tile) * qk_heads + qh) * (long long)(ROWS * ROW);
        const float* coef = p.coef + ((first + tile) * p.heads + h) * (long long)COEF;
        for (int e = tid; e < ROWS * ROW / 4; e += 128) cp16(stage + 4 * e, pack + 4 * e);
        for (int e = tid; e < COEF / 4; e += 128) cp16(stage + ROWS * ROW + 4 * e, coef + 4 * e);
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    // thread (t, two columns) for the values, U and O
    const int vt = tid >> 3, vj = (tid & 7) * 2;
    const T* v = (const T*)p.v;
    auto fetch_v = [&](int tile, float (&x)[2]) {
        const int t = tile * B + vt;
#pragma unroll
        for (int c = 0; c < 2; ++c)
            x[c] = t < n && j0 + vj + c < p.vdim ? to_float<T>(v[(long long)(begin + t) * p.v_stride + (long long)h * p.vdim + j0 + vj + c]) : 0.f;
    };
    issue(0);
    float vnow[2], vnext[2] = {0.f, 0.f};
    fetch_v(0, vnow);
    for (int tile = 0; tile < tiles; ++tile) {
        asm volatile("cp.async.wait_all;\n" ::: "memory");
        __syncthreads();                                 // the tile's inputs and the state are in; the other stage has been read
        if (tile + 1 < tiles) {
            issue(tile + 1);
            fetch_v(tile + 1, vnext);
        }
        const float* pack = smem + (tile & 1) * STAGE;
        const float* coef = pack + ROWS * ROW;
        // product 1: this warp's rows of S against the pack's entries
        {
            constexpr int TT = TQ / 8;                   // entries a thread: 4 (delta) or 2
            float acc[TT][4];
#pragma unroll
            for (int x = 0; x < TT; ++x)
#pragma unroll
                for (int c = 0; c < 4; ++c) acc[x][c] = 0.f;
            const float* pk = pack + warp * WROWS * ROW + TT * tg;
            const float* sr = S_s + warp * WROWS * COLS + 4 * cg;
#pragma unroll
            for (int i = 0; i < WROWS; ++i) {
                __align__(16) float kq[TT];
                if constexpr (TT == 4) *reinterpret_cast<float4*>(kq) = *reinterpret_cast<const float4*>(pk + i * ROW);
                else *reinterpret_cast<float2*>(kq) = *reinterpret_cast<const float2*>(pk + i * ROW);
                const float4 s = *reinterpret_cast<const float4*>(sr + i * COLS);
#pragma unroll
                for (int x = 0; x < TT; ++x) {
                    acc[x][0] = fmaf(kq[x], s.x, acc[x][0]);
                    acc[x][1] = fmaf(kq[x], s.y, acc[x][1]);
                    acc[x][2] = fmaf(kq[x], s.z, acc[x][2]);
                    acc[x][3] = fmaf(kq[x], s.w, acc[x][3]);
                }
            }
#pragma unroll
            for (int x = 0; x < TT; ++x)
                *reinterpret_cast<float4*>(red + (warp * TQ + TT * tg + x) * RP + 4 * cg) = make_float4(acc[x][0], acc[x][1], acc[x][2], acc[x][3]);
        }
        if (MODE == MIX) *reinterpret_cast<float2*>(X_s + vt * COLS + vj) = make_float2(vnow[0], vnow[1]);
        __syncthreads();                                 // partial sums (and, mixing, the values) are in
        float o[2] = {0.f, 0.f}, rd[2] = {0.f, 0.f};
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float2 x = *reinterpret_cast<const float2*>(red + (w * TQ + vt) * RP + vj);
            o[0] += x.x; o[1] += x.y;
            if (MODE == DELTA) {
                const float2 y = *reinterpret_cast<const float2*>(red + (w * TQ + B + vt) * RP + vj);
                rd[0] += y.x; rd[1] += y.y;
            }
        }
        const float* in_s = X_s;                         // what O and the state's update take: U, or the values
        const float* up_s = X_s;
        if constexpr (MODE == DELTA) {
            const float c = coef[2 * B * B + vt];
            o[0] *= c; o[1] *= c;
            *reinterpret_cast<float2*>(X_s + vt * COLS + vj) = make_float2(fmaf(-c, rd[0], vnow[0]), fmaf(-c, rd[1], vnow[1]));
            __syncthreads();
            float u[2] = {0.f, 0.f};
#pragma unroll
            for (int s4 = 0; s4 < B; s4 += 4) {
                const float4 w = *reinterpret_cast<const float4*>(coef + vt * B + s4);
                const float ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int s = 0; s < 4; ++s) {
                    const float2 x = *reinterpret_cast<const float2*>(X_s + (s4 + s) * COLS + vj);
                    u[0] = fmaf(ww[s], x.x, u[0]);
                    u[1] = fmaf(ww[s], x.y, u[1]);
                }
            }
            const float gt = coef[2 * B * B + B + vt];
            *reinterpret_cast<float2*>(U_s + vt * COLS + vj) = make_float2(u[0], u[1]);
            *reinterpret_cast<float2*>(G_s + vt * COLS + vj) = make_float2(gt * u[0], gt * u[1]);
            __syncthreads();
            in_s = U_s;
            up_s = G_s;
        }
        // O
#pragma unroll
        for (int s4 = 0; s4 < B; s4 += 4) {
            const float4 w = *reinterpret_cast<const float4*>(coef + B * B + vt * B + s4);
            const float ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
            for (int s = 0; s < 4; ++s) {
                const float2 x = *reinterpret_cast<const float2*>(in_s + (s4 + s) * COLS + vj);
                o[0] = fmaf(ww[s], x.x, o[0]);
                o[1] = fmaf(ww[s], x.y, o[1]);
            }
        }
        if (tile * B + vt < n) {
            float* dst = p.out + ((long long)(begin + tile * B + vt) * p.heads + h) * p.vdim + j0 + vj;
            if (j0 + vj < p.vdim) dst[0] = o[0];
            if (j0 + vj + 1 < p.vdim) dst[1] = o[1];
        }
        // the state after the tile
        const float cB = coef[2 * B * B + B - 1];
#pragma unroll
        for (int e = 0; e < R; ++e) {
            const float d = MODE == DELTA ? cB : pack[(warp * WROWS + tg + 8 * e) * ROW + 2 * B];
#pragma unroll
            for (int c = 0; c < 4; ++c) S[e][c] *= d;
        }
#pragma unroll
        for (int t4 = 0; t4 < B; t4 += 4) {
            float4 u4[4];
#pragma unroll
            for (int t = 0; t < 4; ++t) u4[t] = *reinterpret_cast<const float4*>(up_s + (t4 + t) * COLS + 4 * cg);
#pragma unroll
            for (int e = 0; e < R; ++e) {
                const float4 k4 = *reinterpret_cast<const float4*>(pack + (warp * WROWS + tg + 8 * e) * ROW + B + t4);
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    S[e][0] = fmaf(kk[t], u4[t].x, S[e][0]);
                    S[e][1] = fmaf(kk[t], u4[t].y, S[e][1]);
                    S[e][2] = fmaf(kk[t], u4[t].z, S[e][2]);
                    S[e][3] = fmaf(kk[t], u4[t].w, S[e][3]);
                }
            }
        }
        // a warp's rows of S_s are read by that warp alone, and it has read them: no barrier before they change
#pragma unroll
        for (int e = 0; e < R; ++e)
            *reinterpret_cast<float4*>(S_s + (warp * WROWS + tg + 8 * e) * COLS + 4 * cg) = make_float4(S[e][0], S[e][1], S[e][2], S[e][3]);
        vnow[0] = vnext[0];
        vnow[1] = vnext[1];
    }
#pragma unroll
    for (int e = 0; e < R; ++e) {
        const int i = warp * WROWS + tg + 8 * e;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int j = j0 + 4 * cg + c;
            if (i < p.dim && j < p.vdim) st[(long long)i * p.vdim + j] = S[e][c];
        }
    }
}

int padded_rows(int dim) { return dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

template <typename T, int MODE>
int launch_scan(const ScanArgs& p, int portions, cudaStream_t stream) {
    const dim3 grid((p.vdim + COLS - 1) / COLS, p.heads, portions);
#define TS_TILES(R)                                                                                                  \
    do {                                                                                                             \
        constexpr int TQ = MODE == DELTA ? 32 : 16;                                                                  \
        const size_t smem = sizeof(float) * (2 * (32 * R * ROW + COEF) + 32 * R * COLS + 4 * TQ * (COLS + 4) + 3 * B * COLS); \
        auto kernel = recurrence_tiles_kernel<T, R, MODE>;                                                           \
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                        \
        kernel<<<grid, 128, smem, stream>>>(p);                                                                      \
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
    return ((long long)num_tokens / B + num_seqs + 1) * heads * padded_rows(dim) * ROW;
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
