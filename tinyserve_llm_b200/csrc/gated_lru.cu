// The inside of Griffin's recurrent block: a short causal convolution, block-diagonal gates and a real-gated
// linear recurrent unit, one number of state a channel.
//
//   v_t = x_t + x_bias                                   x, y: columns of a row of the projection's output
//   u_t[c] = conv_bias[c] + sum_{j < taps} w[c, j] v_(t - (taps - 1 - j))[c]            zeros before the start
//   r_t = sigmoid(R_b u_b + r_bias), i_t = sigmoid(I_b u_b + i_bias)    part b of u times part b's square matrices
//   log a = rate[c] * r_t       (rate = -c softplus(lam), worked out by the host; never positive)
//   S_t = a S_(t-1) + sqrt(1 - a^2) i_t u_t,   out_t = S_t * gelu_tanh(y_t + y_bias)
//
// Gates, decays and state are float32; u has the activation dtype, `out` too.  A request's state slot holds the last
// `taps` values v as a ring (the value of position p in entry p mod taps; no ring for one tap), then S, [channels]
// floats each.  The ring has an entry more than the convolution looks back, so the entry that a decoded token
// writes is one that no thread of that launch reads.
//
// lru_conv_kernel            u of every row of the step (a thread eight channels and a few tokens, a rolling window).
// lru_scan_kernel            requests of up to LRU_STRETCH tokens: a thread a (request, channel), tokens in order.
// lru_stretch_kernel,        longer portions: stretches of LRU_STRETCH tokens side by side; the first kernel turns the
// lru_finish_kernel          gates' logits into (a, sqrt(1 - a^2) i u) in place and each stretch into one step
//                            S_end = A S_begin + B; the second chains the stretches ahead of its own and walks.
// lru_decode_kernel          a step in which every request feeds one token, bfloat16: everything above in one kernel,
//                            the gates' products on mma.sync with the weights streamed once.
// Results of the forms, and of different cuts, differ by rounding only.
#include "common.cuh"

constexpr int LRU_STRETCH = 64;

struct LRUArgs {
    const void* xy; long long xy_stride; int y_off, x_off;              // columns of y and x inside a row
    const float* y_bias; const float* x_bias;
    const float* taps_w;                                                 // [taps][channels], last row the current token's
    const float* conv_bias;
    const float* gate_bias;                                              // [2][channels]: r's, then i's
    const float* rate;                                                   // [channels]
    const int* positions; const int* seq_of_token; const int* cu_q; const int* state_slots;
    float* state; long long state_stride;                                // floats between slots
    void* u; void* out;
    float* z; long long z_token, z_block;                                // gates' logits: r in [0, part), i in [part, 2 part) of a block's row
    int channels, part, taps, num_tokens, num_seqs;
};

__device__ __forceinline__ float lru_gelu(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z)));
}

// FAST (outputs of 16 bits): the exponential and the division by their one-instruction forms, whose error of a few units
// in the last place of a float is far below the output's rounding.
template <bool FAST>
__device__ __forceinline__ float lru_sigmoid(float x) {
    return FAST ? __fdividef(1.f, 1.f + __expf(-x)) : 1.f / (1.f + expf(-x));
}

// (a, sqrt(1 - a^2) i u): one expm1 gives both without cancellation, 1 - a^2 = -m (2 + m) with m = a - 1
template <bool FAST>
__device__ __forceinline__ void lru_gates(float zr, float zi, float rate, float u, float& a, float& in) {
    const float m = expm1f(rate * lru_sigmoid<FAST>(zr));
    a = 1.f + m;
    in = sqrtf(-m * (2.f + m)) * lru_sigmoid<FAST>(zi) * u;
}

template <typename T>
__device__ __forceinline__ float lru_value(const LRUArgs& p, int row, int c) {
    return to_float<T>(((const T*)p.xy)[(long long)row * p.xy_stride + p.x_off + c]) + p.x_bias[c];
}

// v of the token `back` positions before batch row `row` (request `seq`), from the batch or from the ring
template <typename T>
__device__ __forceinline__ float lru_earlier(const LRUArgs& p, int row, int begin, int pos, const float* ring, int back, int c) {
    if (row - back >= begin) return lru_value<T>(p, row - back, c);
    if (pos - back < 0 || !ring) return 0.f;
    return ring[(long long)((pos - back) % p.taps) * p.channels + c];
}

// the request's last values into the ring; called when nobody reads it any more in this step
template <typename T>
__device__ __forceinline__ void lru_advance_ring(const LRUArgs& p, float* ring, int t0, int t1, int c) {
    if (p.taps <= 1) return;
    for (int t = max(t0, t1 - p.taps); t < t1; ++t)
        ring[(long long)(p.positions[t] % p.taps) * p.channels + c] = lru_value<T>(p, t, c);
}

template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128) lru_conv_kernel(LRUArgs p, int group) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (c >= p.channels) return;
    const int taps = TAPS > 0 ? TAPS : p.taps;
    const int t_begin = blockIdx.y * group, t_end = min(p.num_tokens, t_begin + group);
    T* u = (T*)p.u;
    if (TAPS > 0) {
        constexpr int K = TAPS > 0 ? TAPS : 1;
        float w[K][VEC], bias[VEC], xb[VEC], win[K][VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            bias[i] = p.conv_bias[c + i];
            xb[i] = p.x_bias[c + i];
#pragma unroll
            for (int j = 0; j < K; ++j) w[j][i] = p.taps_w[(long long)j * p.channels + c + i];
        }
        int current = -2;
        for (int t = t_begin; t < t_end; ++t) {
            const int seq = p.seq_of_token[t];
            T* dst = u + (long long)t * p.channels + c;
            alignas(16) T o[VEC];
            if (seq < 0) {                                       // a padding row
#pragma unroll
                for (int i = 0; i < VEC; ++i) o[i] = from_float<T>(0.f);
            } else {
                if (seq != current) {                            // the values before this row
                    const int begin = p.cu_q[seq], slot = p.state_slots[seq], pos = p.positions[t];
                    const float* ring = slot >= 0 ? p.state + (long long)slot * p.state_stride : nullptr;
#pragma unroll
                    for (int j = 0; j < K - 1; ++j)
#pragma unroll
                        for (int i = 0; i < VEC; ++i) win[j + 1][i] = lru_earlier<T>(p, t, begin, pos, ring, K - 1 - j, c + i);
                    current = seq;
                }
                alignas(16) T x[VEC];
                const T* src = (const T*)p.xy + (long long)t * p.xy_stride + p.x_off + c;
                if (VEC * sizeof(T) == 16) *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(src);
                else
#pragma unroll
                    for (int i = 0; i < VEC; ++i) x[i] = src[i];
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
#pragma unroll
                    for (int j = 0; j < K - 1; ++j) win[j][i] = win[j + 1][i];
                    win[K - 1][i] = to_float<T>(x[i]) + xb[i];
                    float acc = bias[i];
#pragma unroll
                    for (int j = 0; j < K; ++j) acc = fmaf(w[j][i], win[j][i], acc);
                    o[i] = from_float<T>(acc);
                }
            }
            if (VEC * sizeof(T) == 16) *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(o);
            else
#pragma unroll
                for (int i = 0; i < VEC; ++i) dst[i] = o[i];
        }
    } else {                                                     // any number of taps, a channel a thread
        for (int t = t_begin; t < t_end; ++t) {
            const int seq = p.seq_of_token[t];
            float acc = 0.f;
            if (seq >= 0) {
                const int begin = p.cu_q[seq], slot = p.state_slots[seq], pos = p.positions[t];
                const float* ring = slot >= 0 ? p.state + (long long)slot * p.state_stride : nullptr;
                acc = p.conv_bias[c];
                for (int j = 0; j < taps; ++j)
                    acc = fmaf(p.taps_w[(long long)j * p.channels + c], lru_earlier<T>(p, t, begin, pos, ring, taps - 1 - j, c), acc);
            }
            u[(long long)t * p.channels + c] = from_float<T>(acc);
        }
    }
}

constexpr int LRU_AHEAD = 4;

// grid: (channels, requests); requests of more than `longest` tokens are left to the kernels of stretches
template <typename T>
__global__ void __launch_bounds__(128) lru_scan_kernel(LRUArgs p, int longest) {
    constexpr bool FAST = sizeof(T) == 2;
    const int c = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y;
    if (c >= p.channels) return;
    const int slot = p.state_slots[s], t0 = p.cu_q[s], t1 = p.cu_q[s + 1];
    if (slot < 0 || t1 <= t0 || t1 - t0 > longest) return;
    float* ring = p.state + (long long)slot * p.state_stride;
    float* sp = ring + (p.taps > 1 ? (long long)p.taps * p.channels : 0) + c;
    const float rb = p.gate_bias[c], ib = p.gate_bias[p.channels + c], rate = p.rate[c], yb = p.y_bias[c];
    const float* z = p.z + (long long)(c / p.part) * p.z_block + c % p.part;
    const T* y = (const T*)p.xy + p.y_off + c;
    const T* u = (const T*)p.u + c;
    T* out = (T*)p.out + c;
    float S = *sp;
    for (int t = t0; t < t1; t += LRU_AHEAD) {
        float zr[LRU_AHEAD], zi[LRU_AHEAD], uu[LRU_AHEAD], yy[LRU_AHEAD];
#pragma unroll
        for (int i = 0; i < LRU_AHEAD; ++i) {                    // rows beyond the request: its last row again, not used
            const long long row = min(t + i, t1 - 1);
            zr[i] = z[row * p.z_token];
            zi[i] = z[row * p.z_token + p.part];
            uu[i] = to_float<T>(u[row * p.channels]);
            yy[i] = to_float<T>(y[row * p.xy_stride]);
        }
#pragma unroll
        for (int i = 0; i < LRU_AHEAD; ++i) {
            if (t + i < t1) {
                float a, in;
                lru_gates<FAST>(zr[i] + rb, zi[i] + ib, rate, uu[i], a, in);
                S = fmaf(a, S, in);
                out[(long long)(t + i) * p.channels] = from_float<T>(S * lru_gelu(yy[i] + yb));
            }
        }
    }
    *sp = S;
    lru_advance_ring<T>(p, ring, t0, t1, c);
}

// grid: (channels, portions, stretches).  `chain` [portions][stretches + 1][2][channels]: (A, B) of what lies before a
// stretch, entry 0 being the state the portion starts from as (0, S).
template <typename T>
__global__ void __launch_bounds__(128) lru_stretch_kernel(LRUArgs p, const int* __restrict__ portions, float* __restrict__ chain) {
    constexpr bool FAST = sizeof(T) == 2;
    const int c = blockIdx.x * blockDim.x + threadIdx.x, s = portions[blockIdx.y], k = blockIdx.z;
    if (c >= p.channels || s < 0) return;
    const int slot = p.state_slots[s], t0 = p.cu_q[s], t1 = p.cu_q[s + 1];
    if (slot < 0 || t1 - t0 <= LRU_STRETCH) return;
    const int w0 = t0 + k * LRU_STRETCH, w1 = min(w0 + LRU_STRETCH, t1);
    float* mine = chain + ((long long)blockIdx.y * (gridDim.z + 1) + k) * 2 * p.channels + c;
    if (k == 0) {
        mine[0] = 0.f;
        mine[p.channels] = p.state[(long long)slot * p.state_stride + (p.taps > 1 ? (long long)p.taps * p.channels : 0) + c];
    }
    if (w0 >= w1) return;
    mine += 2 * p.channels;
    const float rb = p.gate_bias[c], ib = p.gate_bias[p.channels + c], rate = p.rate[c];
    float* z = p.z + (long long)(c / p.part) * p.z_block + c % p.part;
    const T* u = (const T*)p.u + c;
    float A = 1.f, B = 0.f;
    for (int t = w0; t < w1; t += LRU_AHEAD) {
        float zr[LRU_AHEAD], zi[LRU_AHEAD], uu[LRU_AHEAD];
#pragma unroll
        for (int i = 0; i < LRU_AHEAD; ++i) {
            const long long row = min(t + i, w1 - 1);
            zr[i] = z[row * p.z_token];
            zi[i] = z[row * p.z_token + p.part];
            uu[i] = to_float<T>(u[row * p.channels]);
        }
#pragma unroll
        for (int i = 0; i < LRU_AHEAD; ++i) {
            if (t + i < w1) {
                float a, in;
                lru_gates<FAST>(zr[i] + rb, zi[i] + ib, rate, uu[i], a, in);
                const long long row = (long long)(t + i) * p.z_token;
                z[row] = a;
                z[row + p.part] = in;
                A *= a;
                B = fmaf(a, B, in);
            }
        }
    }
    mine[0] = A;
    mine[p.channels] = B;
}

template <typename T>
__global__ void __launch_bounds__(128) lru_finish_kernel(LRUArgs p, const int* __restrict__ portions, const float* __restrict__ chain) {
    const int c = blockIdx.x * blockDim.x + threadIdx.x, s = portions[blockIdx.y], k = blockIdx.z;
    if (c >= p.channels || s < 0) return;
    const int slot = p.state_slots[s], t0 = p.cu_q[s], t1 = p.cu_q[s + 1];
    if (slot < 0 || t1 - t0 <= LRU_STRETCH) return;
    const int w0 = t0 + k * LRU_STRETCH, w1 = min(w0 + LRU_STRETCH, t1);
    if (w0 >= w1) return;
    const float* before = chain + (long long)blockIdx.y * (gridDim.z + 1) * 2 * p.channels + c;
    float S = 0.f;
    for (int j = 0; j <= k; j += 4) {                            // the stretches before this one, in order
        float A[4], B[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const long long e = (long long)min(j + i, k) * 2 * p.channels;
            A[i] = before[e];
            B[i] = before[e + p.channels];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (j + i <= k) S = fmaf(A[i], S, B[i]);
    }
    const float yb = p.y_bias[c];
    const float* z = p.z + (long long)(c / p.part) * p.z_block + c % p.part;
    const T* y = (const T*)p.xy + p.y_off + c;
    T* out = (T*)p.out + c;
    constexpr int AHEAD = 8;
    for (int t = w0; t < w1; t += AHEAD) {
        float a[AHEAD], in[AHEAD], yy[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const long long row = min(t + i, w1 - 1);
            a[i] = z[row * p.z_token];
            in[i] = z[row * p.z_token + p.part];
            yy[i] = to_float<T>(y[row * p.xy_stride]);
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (t + i < w1) {
                S = fmaf(a[i], S, in[i]);
                out[(long long)(t + i) * p.channels] = from_float<T>(S * lru_gelu(yy[i] + yb));
            }
        }
    }
    if (w1 == t1) {                                              // nobody reads the slot any more: the kernel ahead copied its state
        float* ring = p.state + (long long)slot * p.state_stride;
        ring[(p.taps > 1 ? (long long)p.taps * p.channels : 0) + c] = S;
        lru_advance_ring<T>(p, ring, t0, t1, c);
    }
}

// ------------------------------------------------------------------ one token a request, everything in one kernel
// A CTA takes 16 channels of one part: it works out u of the whole part for all tokens into shared memory (the gates
// read all of it), eight warps as 2 channel groups of 8 x 4 stretches of k form the gates' logits with m16n8k16 (rows of a
// product: 8 rows of R, then the same 8 of I; columns: 8 tokens), and the CTA's threads finish its 16 channels.  A lane's
// weights are two 16-byte stretches of a row for every 32 k's: the k's of a product may come in any order as long as
// both operands agree, so lane q takes k's 8q .. 8q + 7 of the 32.  They are asked for before the kernel ahead has ended.
constexpr int LD_THREADS = 256, LD_CHANNELS = 16, LD_SPLITS = 4, LD_MAX_TOKENS = 64;

__device__ __forceinline__ void lru_mma(float (&c)[4], unsigned a0, unsigned a1, unsigned a2, unsigned a3, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int CHUNKS>        // stretches of 32 k's a warp holds: part <= 128 CHUNKS
__global__ void __launch_bounds__(LD_THREADS) lru_decode_kernel(LRUArgs p, const __nv_bfloat16* __restrict__ gates_w) {
    extern __shared__ __align__(16) unsigned char lru_smem[];
    const int part = p.part, pitch = part + 8;
    const int padded = (p.num_tokens + 7) & ~7;
    __nv_bfloat16* us = reinterpret_cast<__nv_bfloat16*>(lru_smem);                         // [padded tokens][pitch]
    float2* zs = reinterpret_cast<float2*>(lru_smem + (((size_t)padded * pitch * 2 + 15) & ~(size_t)15));   // [splits][padded][16]: (r, i)
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int per_part = (part + LD_CHANNELS - 1) / LD_CHANNELS;
    const int b = blockIdx.x / per_part, n0 = (blockIdx.x % per_part) * LD_CHANNELS;
    const int group = warp & 1, split = warp >> 1, q = lane & 3;
    const int n = n0 + group * 8 + (lane >> 2);
    const __nv_bfloat16* wr = gates_w + ((long long)b * 2 * part + n) * part;
    uint4 fr[CHUNKS], fi[CHUNKS];
#pragma unroll
    for (int j = 0; j < CHUNKS; ++j) {
        const int k = (split + LD_SPLITS * j) * 32 + q * 8;
        fr[j] = fi[j] = make_uint4(0, 0, 0, 0);
        if (n < part && k < part) {
            fr[j] = *reinterpret_cast<const uint4*>(wr + k);
            fi[j] = *reinterpret_cast<const uint4*>(wr + (long long)part * part + k);
        }
    }
    chain_wait();
    // ---- u of the part, eight channels of a token an item
    const int vecs = part / 8;
    for (int e = tid; e < padded * vecs; e += LD_THREADS) {
        const int t = e / vecs, c0 = (e % vecs) * 8, c = b * part + c0;
        const int seq = t < p.num_tokens ? p.seq_of_token[t] : -1;
        const int slot = seq >= 0 ? p.state_slots[seq] : -1;
        alignas(16) __nv_bfloat16 o[8];
        if (slot < 0) {
#pragma unroll
            for (int i = 0; i < 8; ++i) o[i] = __float2bfloat16_rn(0.f);
        } else {
            const int pos = p.positions[t];
            const float* ring = p.state + (long long)slot * p.state_stride;
            alignas(16) __nv_bfloat16 x[8];
            *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)p.xy + (long long)t * p.xy_stride + p.x_off + c);
            float acc[8];
            const float* w = p.taps_w + (long long)(p.taps - 1) * p.channels + c;
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[i] = fmaf(w[i], __bfloat162float(x[i]) + p.x_bias[c + i], p.conv_bias[c + i]);
            for (int back = 1; back < p.taps && back <= pos; ++back) {
                const float* v = ring + (long long)((pos - back) % p.taps) * p.channels + c;
                w = p.taps_w + (long long)(p.taps - 1 - back) * p.channels + c;
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[i] = fmaf(w[i], v[i], acc[i]);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) o[i] = __float2bfloat16_rn(acc[i]);
        }
        *reinterpret_cast<uint4*>(us + t * pitch + c0) = *reinterpret_cast<const uint4*>(o);
    }
    __syncthreads();
    // ---- this warp's share of the gates' logits, eight tokens at a time
    for (int t0 = 0; t0 < padded; t0 += 8) {
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < CHUNKS; ++j) {
            const int k = (split + LD_SPLITS * j) * 32 + q * 8;
            uint4 ub = make_uint4(0, 0, 0, 0);
            if (k < part) ub = *reinterpret_cast<const uint4*>(us + (t0 + (lane >> 2)) * pitch + k);
            lru_mma(acc, fr[j].x, fi[j].x, fr[j].y, fi[j].y, ub.x, ub.y);
            lru_mma(acc, fr[j].z, fi[j].z, fr[j].w, fi[j].w, ub.z, ub.w);
        }
        // rows lane / 4 (r) and lane / 4 + 8 (i) are one channel's; columns 2q, 2q + 1 are tokens
        float2* dst = zs + ((long long)split * padded + t0 + 2 * q) * LD_CHANNELS + group * 8 + (lane >> 2);
        dst[0] = make_float2(acc[0], acc[2]);
        dst[LD_CHANNELS] = make_float2(acc[1], acc[3]);
    }
    __syncthreads();
    chain_release();
    for (int e = tid; e < p.num_tokens * LD_CHANNELS; e += LD_THREADS) {
        const int t = e / LD_CHANNELS, ch = e % LD_CHANNELS;
        const int seq = p.seq_of_token[t];
        if (seq < 0 || n0 + ch >= part) continue;
        const int slot = p.state_slots[seq];
        if (slot < 0) continue;
        float zr = 0.f, zi = 0.f;
#pragma unroll
        for (int s = 0; s < LD_SPLITS; ++s) {
            const float2 v = zs[((long long)s * padded + t) * LD_CHANNELS + ch];
            zr += v.x;
            zi += v.y;
        }
        const int c = b * part + n0 + ch;
        const __nv_bfloat16* row = (const __nv_bfloat16*)p.xy + (long long)t * p.xy_stride;
        float* ring = p.state + (long long)slot * p.state_stride;
        float* sp = ring + (p.taps > 1 ? (long long)p.taps * p.channels : 0) + c;
        float a, in;
        lru_gates<true>(zr + p.gate_bias[c], zi + p.gate_bias[p.channels + c], p.rate[c],
                        __bfloat162float(us[t * pitch + n0 + ch]), a, in);
        const float S = fmaf(a, *sp, in);
        *sp = S;
        if (p.taps > 1) ring[(long long)(p.positions[t] % p.taps) * p.channels + c] = __bfloat162float(row[p.x_off + c]) + p.x_bias[c];
        ((__nv_bfloat16*)p.out)[(long long)t * p.channels + c] =
            __float2bfloat16_rn(S * lru_gelu(__bfloat162float(row[p.y_off + c]) + p.y_bias[c]));
    }
}

static size_t lru_decode_smem(int num_tokens, int part) {
    const size_t padded = (size_t)((num_tokens + 7) & ~7);
    return ((padded * (part + 8) * 2 + 15) & ~(size_t)15) + LD_SPLITS * padded * LD_CHANNELS * sizeof(float2);
}

static int lru_check(const LRUArgs& p) {
    TS_REQUIRE(p.channels > 0 && p.part > 0 && p.channels % p.part == 0 && p.taps > 0 && p.num_tokens >= 0 && p.num_seqs >= 0,
               "gated_lru: bad sizes");
    TS_REQUIRE(p.state != nullptr && p.state_stride >= (long long)p.channels * (1 + (p.taps > 1 ? p.taps : 0)),
               "gated_lru: the state slot is too small for %d channels and %d taps", p.channels, p.taps);
    return 0;
}

#define TS_LRU_PARAMS                                                                                                     \
    const void *xy, long long xy_stride, int y_off, int x_off, const float *y_bias, const float *x_bias,                 \
        const float *taps_w, const float *conv_bias, const float *gate_bias, const float *rate, const int *positions,    \
        const int *seq_of_token, const int *cu_q, const int *state_slots, int num_seqs, float *state,                    \
        long long state_stride, void *out, int channels, int part, int taps, int num_tokens

// Whether ts_lru_decode takes a step of these sizes (bfloat16, every request feeds one token).
TS_API int ts_lru_decode_supported(int num_tokens, int channels, int part, long long xy_stride, int x_off) {
    return num_tokens > 0 && num_tokens <= LD_MAX_TOKENS && part % 8 == 0 && part <= 512 && channels % 8 == 0 && xy_stride % 8 == 0 &&
           x_off % 8 == 0 && lru_decode_smem(num_tokens, part) <= 200 * 1024;
}

TS_API int ts_lru_decode(TS_LRU_PARAMS, const void* gates_w, cudaStream_t stream) {
    LRUArgs p{xy, xy_stride, y_off, x_off, y_bias, x_bias, taps_w, conv_bias, gate_bias, rate, positions, seq_of_token, cu_q,
              state_slots, state, state_stride, nullptr, out, nullptr, 0, 0, channels, part, taps, num_tokens, num_seqs};
    if (lru_check(p)) return 1;
    if (num_tokens == 0 || num_seqs == 0) return 0;
    TS_REQUIRE(ts_lru_decode_supported(num_tokens, channels, part, xy_stride, x_off) && (uintptr_t)xy % 16 == 0 &&
               (uintptr_t)gates_w % 16 == 0, "lru_decode: sizes not taken");
    const size_t smem = lru_decode_smem(num_tokens, part);
    const dim3 grid((channels / part) * ((part + LD_CHANNELS - 1) / LD_CHANNELS));
    const __nv_bfloat16* w = (const __nv_bfloat16*)gates_w;
#define TS_LRU_DECODE(CHUNKS)                                                                                             \
    do {                                                                                                                  \
        if (smem > 48 * 1024)                                                                                             \
            cudaFuncSetAttribute(lru_decode_kernel<CHUNKS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);      \
        TS_CHAINED_CHECK("lru_decode", launch_chained(lru_decode_kernel<CHUNKS>, grid, dim3(LD_THREADS), smem, stream, p, w)); \
    } while (0)
    if (part <= 128) TS_LRU_DECODE(1);
    else if (part <= 256) TS_LRU_DECODE(2);
    else TS_LRU_DECODE(4);
#undef TS_LRU_DECODE
    return 0;
}

template <typename T>
static int lru_conv_launch(const LRUArgs& p, cudaStream_t stream) {
    constexpr int VEC = 16 / sizeof(T);
    const bool vector = p.channels % VEC == 0 && p.xy_stride % VEC == 0 && p.x_off % VEC == 0 && (uintptr_t)p.xy % 16 == 0 &&
                        (uintptr_t)p.u % 16 == 0;
    const int group = p.num_tokens >= 256 ? 8 : 1;
    TS_REQUIRE(p.num_tokens <= 65535 * group, "gated_lru: %d tokens a step are not supported", p.num_tokens);
    const int per_thread = vector && p.taps <= 8 ? VEC : 1;
    const int threads = (p.channels + per_thread - 1) / per_thread;
    const dim3 grid((threads + 127) / 128, (p.num_tokens + group - 1) / group);
#define TS_LRU_CONV(K) lru_conv_kernel<T, VEC, K><<<grid, 128, 0, stream>>>(p, group)
    if (per_thread == 1) lru_conv_kernel<T, 1, 0><<<grid, 128, 0, stream>>>(p, group);
    else switch (p.taps) {
        case 1: TS_LRU_CONV(1); break;
        case 2: TS_LRU_CONV(2); break;
        case 3: TS_LRU_CONV(3); break;
        case 4: TS_LRU_CONV(4); break;
        case 5: TS_LRU_CONV(5); break;
        case 6: TS_LRU_CONV(6); break;
        case 7: TS_LRU_CONV(7); break;
        default: TS_LRU_CONV(8); break;
    }
#undef TS_LRU_CONV
    TS_LAUNCH_CHECK("lru_conv");
    return 0;
}

// u [num_tokens, channels] of every row.
TS_API int ts_lru_conv(TS_LRU_PARAMS, int dtype, cudaStream_t stream) {
    LRUArgs p{xy, xy_stride, y_off, x_off, y_bias, x_bias, taps_w, conv_bias, gate_bias, rate, positions, seq_of_token, cu_q,
              state_slots, state, state_stride, out, nullptr, nullptr, 0, 0, channels, part, taps, num_tokens, num_seqs};
    if (lru_check(p)) return 1;
    if (num_tokens == 0 || num_seqs == 0) return 0;
    if (dtype == TS_F32) return lru_conv_launch<float>(p, stream);
    if (dtype == TS_BF16) return lru_conv_launch<__nv_bfloat16>(p, stream);
    return ts_fail("lru_conv: unknown dtype code %d", dtype);
}

// Floats of scratch that ts_lru_scan needs for these portions.
TS_API long long ts_lru_scan_scratch_floats(int portions, int max_q_len, int channels) {
    if (portions <= 0 || max_q_len <= LRU_STRETCH) return 0;
    return (long long)portions * ((max_q_len + LRU_STRETCH - 1) / LRU_STRETCH + 1) * 2 * channels;
}

// From u and the gates' logits z (strides in floats; overwritten for portions of more than LRU_STRETCH tokens) to `out`.
// `portions`: requests that feed more than one token, -1 padding; without a list every request is walked in order.
// `max_q_len` bounds a request's tokens.
TS_API int ts_lru_scan(TS_LRU_PARAMS, const void* u, float* z, long long z_token, long long z_block, const int* portions,
                       int num_portions, int max_q_len, float* scratch, long long scratch_floats, int dtype, cudaStream_t stream) {
    LRUArgs p{xy, xy_stride, y_off, x_off, y_bias, x_bias, taps_w, conv_bias, gate_bias, rate, positions, seq_of_token, cu_q,
              state_slots, state, state_stride, const_cast<void*>(u), out, z, z_token, z_block, channels, part, taps, num_tokens, num_seqs};
    if (lru_check(p)) return 1;
    TS_REQUIRE(num_seqs <= 65535 && num_portions <= 65535, "lru_scan: too many requests in a step");
    if (num_tokens == 0 || num_seqs == 0) return 0;
    const long long need = portions ? ts_lru_scan_scratch_floats(num_portions, max_q_len, channels) : 0;
    TS_REQUIRE(need == 0 || (scratch && scratch_floats >= need), "lru_scan: %lld floats of scratch needed, %lld given", need, scratch_floats);
    const int stretches = (max_q_len + LRU_STRETCH - 1) / LRU_STRETCH;
    TS_REQUIRE(need == 0 || stretches <= 65535, "lru_scan: portions of %d tokens are not supported", max_q_len);
    const unsigned cols = (unsigned)((channels + 127) / 128);
    const int longest = need ? LRU_STRETCH : 0x7fffffff;
#define TS_LRU_SCAN(T)                                                                                          \
    do {                                                                                                        \
        lru_scan_kernel<T><<<dim3(cols, num_seqs), 128, 0, stream>>>(p, longest);                               \
        if (need) {                                                                                             \
            const dim3 grid(cols, num_portions, stretches);                                                     \
            lru_stretch_kernel<T><<<grid, 128, 0, stream>>>(p, portions, scratch);                              \
            lru_finish_kernel<T><<<grid, 128, 0, stream>>>(p, portions, scratch);                               \
        }                                                                                                       \
    } while (0)
    if (dtype == TS_F32) TS_LRU_SCAN(float);
    else if (dtype == TS_BF16) TS_LRU_SCAN(__nv_bfloat16);
    else return ts_fail("lru_scan: unknown dtype code %d", dtype);
#undef TS_LRU_SCAN
    TS_LAUNCH_CHECK("lru_scan");
    return 0;
}
