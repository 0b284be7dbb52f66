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
// lru_conv_kernel            u of every row of the step.
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

template <int N>
__device__ __forceinline__ void load_floats(const float* src, float (&dst)[N]) {     // 16-byte aligned where N is a multiple of 4
    if (N % 4 == 0)
#pragma unroll
        for (int i = 0; i < N; i += 4) {
            const float4 v = *reinterpret_cast<const float4*>(src + i);
            dst[i] = v.x; dst[(i + 1) % N] = v.y; dst[(i + 2) % N] = v.z; dst[(i + 3) % N] = v.w;
        }
    else
#pragma unroll
        for (int i = 0; i < N; ++i) dst[i] = src[i];
}

constexpr int LRU_GROUP = 8;             // tokens a thread of the convolution takes in a step of many tokens

// A thread: 16 bytes of neighbouring channels, GROUP tokens whose rows are asked for together, a window that rolls over them.
template <typename T, int TAPS, int GROUP>
__global__ void __launch_bounds__(128) lru_conv_kernel(LRUArgs p) {
    constexpr int VEC = 16 / sizeof(T);
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (c >= p.channels) return;
    const int t_begin = blockIdx.y * GROUP, count = min(GROUP, p.num_tokens - t_begin);
    const T* x = (const T*)p.xy + p.x_off + c;
    uint4 rows[GROUP];
    int seqs[GROUP];
#pragma unroll
    for (int g = 0; g < GROUP; ++g) {
        rows[g] = make_uint4(0, 0, 0, 0);
        seqs[g] = -1;
        if (g < count) {
            rows[g] = *reinterpret_cast<const uint4*>(x + (long long)(t_begin + g) * p.xy_stride);
            seqs[g] = p.seq_of_token[t_begin + g];
        }
    }
    float w[TAPS][VEC], bias[VEC], xb[VEC], win[TAPS][VEC];
    load_floats(p.conv_bias + c, bias);
    load_floats(p.x_bias + c, xb);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_floats(p.taps_w + (long long)j * p.channels + c, w[j]);
    auto values = [&](const uint4& raw, float (&v)[VEC]) {
        const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = to_float<T>(e[i]) + xb[i];
    };
    int current = -2;
#pragma unroll
    for (int g = 0; g < GROUP; ++g) {
        if (g >= count) break;
        const int t = t_begin + g, seq = seqs[g];
        alignas(16) T o[VEC];
        if (seq < 0) {                                           // a padding row
#pragma unroll
            for (int i = 0; i < VEC; ++i) o[i] = from_float<T>(0.f);
        } else {
            if (seq != current) {                                // the values before this row: of the batch, of the ring, or zeros
                const int begin = p.cu_q[seq], slot = p.state_slots[seq], pos = p.positions[t];
                const float* ring = p.state + (long long)max(slot, 0) * p.state_stride + c;
#pragma unroll
                for (int back = TAPS - 1; back > 0; --back) {
                    float (&v)[VEC] = win[TAPS - back];          // moves one place down before it is used
                    if (t - back >= begin) values(*reinterpret_cast<const uint4*>(x + (long long)(t - back) * p.xy_stride), v);
                    else if (slot >= 0 && pos - back >= 0) load_floats(ring + (long long)((pos - back) % TAPS) * p.channels, v);
                    else
#pragma unroll
                        for (int i = 0; i < VEC; ++i) v[i] = 0.f;
                }
                current = seq;
            }
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
                for (int i = 0; i < VEC; ++i) win[j][i] = win[j + 1][i];
            values(rows[g], win[TAPS - 1]);
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                float acc = bias[i];
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j][i], win[j][i], acc);
                o[i] = from_float<T>(acc);
            }
        }
        *reinterpret_cast<uint4*>((T*)p.u + (long long)t * p.channels + c) = *reinterpret_cast<const uint4*>(o);
    }
}

// Any sizes: a thread a channel and token.
template <typename T>
__global__ void __launch_bounds__(128) lru_conv_any_kernel(LRUArgs p) {
    const int c = blockIdx.x * blockDim.x + threadIdx.x, t = blockIdx.y;
    if (c >= p.channels) return;
    const int seq = p.seq_of_token[t];
    float acc = 0.f;
    if (seq >= 0) {
        const int begin = p.cu_q[seq], slot = p.state_slots[seq], pos = p.positions[t];
        const float* ring = slot >= 0 ? p.state + (long long)slot * p.state_stride : nullptr;
        acc = p.conv_bias[c];
        for (int j = 0; j < p.taps; ++j)
            acc = fmaf(p.taps_w[(long long)j * p.channels + c], lru_earlier<T>(p, t, begin, pos, ring, p.taps - 1 - j, c), acc);
    }
    ((T*)p.u)[(long long)t * p.channels + c] = from_float<T>(acc);
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

// What the kernel does not get from the projection just ahead (weights, index data, the slot's ring and state, which earlier
// steps left) is asked for before it waits for that kernel.
// CHUNKS: stretches of 32 k's a warp holds, part <= 128 CHUNKS; TAPS 0: any number of them, loaded as they are used.
template <int CHUNKS, int TAPS>
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
    const int state_at = p.taps > 1 ? p.taps * p.channels : 0;
    // this thread's eight channels of u, and the tokens it takes them of
    const int vecs = part / 8, per_pass = LD_THREADS / vecs;
    const int c0 = (tid % vecs) * 8, c = b * part + c0, first = tid / vecs < per_pass ? tid / vecs : padded;
    constexpr int K = TAPS > 0 ? TAPS : 1;
    float w[K][8], bias[8], xb[8], past[K][8];
    load_floats(p.conv_bias + c, bias);
    load_floats(p.x_bias + c, xb);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_floats(p.taps_w + (long long)j * p.channels + c, w[j]);
    auto slot_of = [&](int t) {
        const int seq = t < p.num_tokens ? p.seq_of_token[t] : -1;
        return seq >= 0 ? p.state_slots[seq] : -1;
    };
    auto load_past = [&](int pos, const float* ring) {           // the token `back` before: entry TAPS - 1 - back
#pragma unroll
        for (int back = 1; back < TAPS; ++back) {
            if (back <= pos) load_floats(ring + (long long)((pos - back) % K) * p.channels + c, past[K - 1 - back < 0 ? 0 : K - 1 - back]);
            else
#pragma unroll
                for (int i = 0; i < 8; ++i) past[K - 1 - back < 0 ? 0 : K - 1 - back][i] = 0.f;
        }
    };
    int slot = slot_of(first), pos = slot >= 0 ? p.positions[first] : 0;
    if (slot >= 0) load_past(pos, p.state + (long long)slot * p.state_stride);
    // this thread's first (token, channel) of the last part
    const int mine_t = tid / LD_CHANNELS, mine_n = n0 + tid % LD_CHANNELS;
    const bool channel = mine_n < part;
    const int mc = b * part + (channel ? mine_n : n0);
    const int mine_slot = slot_of(mine_t);
    const float rb = p.gate_bias[mc], ib = p.gate_bias[p.channels + mc], rate = p.rate[mc], yb = p.y_bias[mc], mxb = p.x_bias[mc];
    float mine_S = mine_slot >= 0 ? p.state[(long long)mine_slot * p.state_stride + state_at + mc] : 0.f;
    chain_wait();
    const __nv_bfloat16* xy = (const __nv_bfloat16*)p.xy;
    float mine_y = 0.f, mine_x = 0.f;
    if (mine_slot >= 0) {
        mine_y = __bfloat162float(xy[(long long)mine_t * p.xy_stride + p.y_off + mc]);
        mine_x = __bfloat162float(xy[(long long)mine_t * p.xy_stride + p.x_off + mc]);
    }
    // ---- u of the part
    for (int t = first; t < padded; t += per_pass) {
        alignas(16) __nv_bfloat16 o[8];
        if (t != first) {
            slot = slot_of(t);
            if (slot >= 0) {
                pos = p.positions[t];
                load_past(pos, p.state + (long long)slot * p.state_stride);
            }
        }
        if (slot < 0) {
#pragma unroll
            for (int i = 0; i < 8; ++i) o[i] = __float2bfloat16_rn(0.f);
        } else {
            alignas(16) __nv_bfloat16 x[8];
            *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(xy + (long long)t * p.xy_stride + p.x_off + c);
            float acc[8];
            if (TAPS > 0) {
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    acc[i] = bias[i];
#pragma unroll
                    for (int j = 0; j < K - 1; ++j) acc[i] = fmaf(w[j][i], past[j][i], acc[i]);
                    acc[i] = fmaf(w[K - 1][i], __bfloat162float(x[i]) + xb[i], acc[i]);
                }
            } else {
                const float* ring = p.state + (long long)slot * p.state_stride;
                float wt[8], v[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[i] = bias[i];
                for (int back = min(p.taps - 1, pos); back > 0; --back) {
                    load_floats(p.taps_w + (long long)(p.taps - 1 - back) * p.channels + c, wt);
                    load_floats(ring + (long long)((pos - back) % p.taps) * p.channels + c, v);
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[i] = fmaf(wt[i], v[i], acc[i]);
                }
                load_floats(p.taps_w + (long long)(p.taps - 1) * p.channels + c, wt);
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[i] = fmaf(wt[i], __bfloat162float(x[i]) + xb[i], acc[i]);
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
    if (!channel) return;
    for (int t = mine_t; t < p.num_tokens; t += LD_THREADS / LD_CHANNELS) {
        if (t != mine_t) {
            slot = slot_of(t);
            if (slot >= 0) {
                mine_S = p.state[(long long)slot * p.state_stride + state_at + mc];
                mine_y = __bfloat162float(xy[(long long)t * p.xy_stride + p.y_off + mc]);
                mine_x = __bfloat162float(xy[(long long)t * p.xy_stride + p.x_off + mc]);
            }
        } else {
            slot = mine_slot;
        }
        if (slot < 0) continue;
        float zr = rb, zi = ib;
#pragma unroll
        for (int s = 0; s < LD_SPLITS; ++s) {
            const float2 v = zs[((long long)s * padded + t) * LD_CHANNELS + tid % LD_CHANNELS];
            zr += v.x;
            zi += v.y;
        }
        float* ring = p.state + (long long)slot * p.state_stride;
        float a, in;
        lru_gates<true>(zr, zi, rate, __bfloat162float(us[t * pitch + mine_n]), a, in);
        const float S = fmaf(a, mine_S, in);
        ring[state_at + mc] = S;
        if (p.taps > 1) ring[(long long)(p.positions[t] % p.taps) * p.channels + mc] = mine_x + mxb;
        ((__nv_bfloat16*)p.out)[(long long)t * p.channels + mc] = __float2bfloat16_rn(S * lru_gelu(mine_y + yb));
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
               (uintptr_t)gates_w % 16 == 0 && (uintptr_t)state % 16 == 0 && state_stride % 4 == 0,
               "lru_decode: sizes or alignment not taken");
    const size_t smem = lru_decode_smem(num_tokens, part);
    const dim3 grid((channels / part) * ((part + LD_CHANNELS - 1) / LD_CHANNELS));
    const __nv_bfloat16* w = (const __nv_bfloat16*)gates_w;
#define TS_LRU_DECODE(CHUNKS, TAPS)                                                                                       \
    do {                                                                                                                  \
        if (smem > 48 * 1024)                                                                                             \
            cudaFuncSetAttribute(lru_decode_kernel<CHUNKS, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        TS_CHAINED_CHECK("lru_decode", launch_chained(lru_decode_kernel<CHUNKS, TAPS>, grid, dim3(LD_THREADS), smem, stream, p, w)); \
    } while (0)
#define TS_LRU_DECODE_PART(TAPS)                    \
    do {                                            \
        if (part <= 128) TS_LRU_DECODE(1, TAPS);      \
        else if (part <= 256) TS_LRU_DECODE(2, TAPS); \
        else TS_LRU_DECODE(4, TAPS);                  \
    } while (0)
    if (taps == 4) TS_LRU_DECODE_PART(4);
    else if (taps == 3) TS_LRU_DECODE_PART(3);
    else if (taps == 2) TS_LRU_DECODE_PART(2);
    else TS_LRU_DECODE_PART(0);
#undef TS_LRU_DECODE_PART
#undef TS_LRU_DECODE
    return 0;
}

template <typename T>
static int lru_conv_launch(const LRUArgs& p, cudaStream_t stream) {
    constexpr int VEC = 16 / sizeof(T);
    const bool vector = p.channels % 8 == 0 && p.xy_stride % VEC == 0 && p.x_off % VEC == 0 && (uintptr_t)p.xy % 16 == 0 &&
                        (uintptr_t)p.u % 16 == 0 && (uintptr_t)p.state % 16 == 0 && p.state_stride % 4 == 0 && p.taps <= 8;
    const bool many = p.num_tokens >= 256;
    const int rows = vector && many ? (p.num_tokens + LRU_GROUP - 1) / LRU_GROUP : p.num_tokens;
    TS_REQUIRE(rows <= 65535, "gated_lru: %d tokens a step are not supported", p.num_tokens);
    const int threads = vector ? p.channels / VEC : p.channels;
    const dim3 grid((threads + 127) / 128, rows);
#define TS_LRU_CONV(K)                                                                     \
    do {                                                                                   \
        if (many) lru_conv_kernel<T, K, LRU_GROUP><<<grid, 128, 0, stream>>>(p);           \
        else lru_conv_kernel<T, K, 1><<<grid, 128, 0, stream>>>(p);                        \
    } while (0)
    if (!vector) lru_conv_any_kernel<T><<<grid, 128, 0, stream>>>(p);
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
