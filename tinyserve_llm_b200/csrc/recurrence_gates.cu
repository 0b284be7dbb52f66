// What enters the scan of linear_recurrence.cu for recurrences whose gates are computed from the input:
// the gated delta rule, the matrix memory with exponential gates (mLSTM), and time mixing with
// decays per channel and a bonus for the current token (RWKV).  Everything here is float32; the
// inputs are projections' outputs in the activation dtype (or float32).
//
// Gated delta rule.  q and k ([tokens, kv_heads * dim], float32, after their short convolution) become
// unit vectors per head, x / sqrt(sum(x^2) + unit_eps), q also times q_scale; value head h uses q/k
// head h / (heads / kv_heads).  The decay of head h, key channel i is
//   a = exp(-exp(A_log[h]) * softplus(z[t, h, i] + dt_bias[h, i])),   beta[t, h] = sigmoid(b[t, h]);
// or, with one decay a head, z and dt_bias have no channel index and neither has a; q and k are then written once a
// q/k head.
//
// Time mixing.  a[t, h, i] = exp(-exp(z[t, h, i] + w0[h, i])), r and k pass as they are, and what the current
// token's write adds to the read-out under the bonus u is v times sum_i u[h, i] k[t, h, i] r[t, h, i].
// The mixer's inputs are blends of the token's row and the one before it, h + (h' - h) mu, one for every mu;
// the row before a step's first token comes from the request's state slot (zeros at the start).
//
// Matrix memory.  Per head (x_i, x_f: float32 projections), log input gate i = cap tanh((x_i + b_i) / cap), log forget gate
// f = log_sigmoid(cap tanh((x_f + b_f) / cap)), running maximum m_t = max(f + m_(t-1), i) carried in the
// request's state (it starts at 0); the scan then runs with decay exp(f + m_(t-1) - m_t) for all of a
// head's key channels, k times exp(i - m_t), and q times q_scale.  m_t goes out per token for the read-out.
#include "common.cuh"

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

// one warp a (token, head)
template <typename T>
__global__ void delta_prepare_kernel(const float* __restrict__ q, const float* __restrict__ k, long long qk_stride,
                                     const float* __restrict__ z, const float* __restrict__ dt_bias,
                                     const float* __restrict__ a_log, const T* __restrict__ b, long long b_stride,
                                     float* __restrict__ prepared, float* __restrict__ beta, long long items, long long total,
                                     int heads, int kv_heads, int dim, float unit_eps, float q_scale) {
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= items) return;
    const int lane = threadIdx.x & 31;
    const long long t = item / heads;
    const int h = (int)(item % heads), g = h / (heads / kv_heads);
    const float* qr = q + t * qk_stride + (long long)g * dim;
    const float* kr = k + t * qk_stride + (long long)g * dim;
    float sq = 0.f, sk = 0.f;
    for (int i = lane; i < dim; i += 32) { sq += qr[i] * qr[i]; sk += kr[i] * kr[i]; }
    const float inv_q = q_scale / sqrtf(warp_sum(sq) + unit_eps), inv_k = 1.f / sqrtf(warp_sum(sk) + unit_eps);
    const float rate = expf(a_log[h]);
    const long long at = item * dim;
    for (int i = lane; i < dim; i += 32) {
        prepared[at + i] = qr[i] * inv_q;
        prepared[total + at + i] = kr[i] * inv_k;
        prepared[2 * total + at + i] = expf(-rate * softplus(z[at + i] + dt_bias[(long long)h * dim + i]));
    }
    if (lane == 0) beta[item] = 1.f / (1.f + expf(-to_float<T>(b[t * b_stride + h])));
}

TS_API int ts_delta_prepare(const float* q, const float* k, long long qk_stride, const float* z, const float* dt_bias,
                            const float* a_log, const void* b, long long b_stride, float* prepared, float* beta,
                            int num_tokens, int heads, int kv_heads, int dim, float unit_eps, float q_scale, int dtype,
                            cudaStream_t stream) {
    TS_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0, "delta_prepare: %d heads over %d q/k heads",
               heads, kv_heads);
    if (num_tokens <= 0) return 0;
    const long long items = (long long)num_tokens * heads, total = items * dim;
    const unsigned blocks = (unsigned)((items + 3) / 4);
    if (dtype == TS_F32)
        delta_prepare_kernel<float><<<blocks, 128, 0, stream>>>(q, k, qk_stride, z, dt_bias, a_log, (const float*)b, b_stride,
            prepared, beta, items, total, heads, kv_heads, dim, unit_eps, q_scale);
    else if (dtype == TS_BF16)
        delta_prepare_kernel<__nv_bfloat16><<<blocks, 128, 0, stream>>>(q, k, qk_stride, z, dt_bias, a_log,
            (const __nv_bfloat16*)b, b_stride, prepared, beta, items, total, heads, kv_heads, dim, unit_eps, q_scale);
    else
        return ts_fail("delta_prepare: unknown dtype code %d", dtype);
    TS_LAUNCH_CHECK("delta_prepare");
    return 0;
}

// With `single_of` (the request of every token): whether the token's request feeds it alone (a padding row does not).
__device__ __forceinline__ bool feeds_one(const int* single_of, const int* cu_q, long long t) {
    if (!single_of) return true;
    const int seq = single_of[t];
    return seq >= 0 && cu_q[seq + 1] - cu_q[seq] == 1;
}

// The same with one decay a head: one warp a (token, q/k head), which also takes its value heads' gates.  gates
// [tokens, 2 heads] float32 holds the step sizes' logits, then the decays'; prepared is [2][tokens, kv_heads * dim],
// beta and decay [tokens, heads].  `single_of` (optional): only tokens of requests that feed one are prepared.
__global__ void delta_prepare_head_kernel(const float* __restrict__ q, const float* __restrict__ k, long long qk_stride,
                                          const float* __restrict__ gates, const float* __restrict__ dt_bias,
                                          const float* __restrict__ a_log, float* __restrict__ prepared,
                                          float* __restrict__ beta, float* __restrict__ decay, long long items, int heads,
                                          int kv_heads, int dim, float unit_eps, float q_scale,
                                          const int* __restrict__ single_of, const int* __restrict__ cu_q) {
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= items) return;
    const int lane = threadIdx.x & 31;
    const long long t = item / kv_heads;
    if (!feeds_one(single_of, cu_q, t)) return;
    const int g = (int)(item % kv_heads), group = heads / kv_heads;
    const float* qr = q + t * qk_stride + (long long)g * dim;
    const float* kr = k + t * qk_stride + (long long)g * dim;
    for (int i = lane; i < group; i += 32) {
        const int h = g * group + i;
        const float b = gates[t * 2 * heads + h], z = gates[t * 2 * heads + heads + h];
        beta[t * heads + h] = 1.f / (1.f + expf(-b));
        decay[t * heads + h] = expf(-expf(a_log[h]) * softplus(z + dt_bias[h]));
    }
    float sq = 0.f, sk = 0.f;
    for (int i = lane; i < dim; i += 32) { sq += qr[i] * qr[i]; sk += kr[i] * kr[i]; }
    const float inv_q = q_scale / sqrtf(warp_sum(sq) + unit_eps), inv_k = 1.f / sqrtf(warp_sum(sk) + unit_eps);
    const long long at = item * dim, total = items * dim;
    for (int i = lane; i < dim; i += 32) {
        prepared[at + i] = qr[i] * inv_q;
        prepared[total + at + i] = kr[i] * inv_k;
    }
}

TS_API int ts_delta_prepare_head(const float* q, const float* k, long long qk_stride, const float* gates,
                                 const float* dt_bias, const float* a_log, float* prepared, float* beta, float* decay,
                                 int num_tokens, int heads, int kv_heads, int dim, float unit_eps, float q_scale,
                                 const int* single_of, const int* cu_q, cudaStream_t stream) {
    TS_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0, "delta_prepare: %d heads over %d q/k heads",
               heads, kv_heads);
    if (num_tokens <= 0) return 0;
    const long long items = (long long)num_tokens * kv_heads;
    delta_prepare_head_kernel<<<(unsigned)((items + 3) / 4), 128, 0, stream>>>(q, k, qk_stride, gates, dt_bias, a_log, prepared,
        beta, decay, items, heads, kv_heads, dim, unit_eps, q_scale, single_of, cu_q);
    TS_LAUNCH_CHECK("delta_prepare_head");
    return 0;
}

// mixes[s][t] = x[t] + (x'[t] - x[t]) * mu[s], x' the request's row before t: of this step, or from its slot.
// A thread takes a channel of a token and writes it for every s.
template <typename T>
__global__ void token_shift_kernel(const T* __restrict__ x, const float* __restrict__ mu, const int* __restrict__ seq_of_token,
                                   const int* __restrict__ cu_q, const int* __restrict__ slots, const float* __restrict__ state,
                                   long long slot_stride, T* __restrict__ mixes, int num_tokens, int width, int count) {
    const long long total = (long long)num_tokens * width;
    for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
        const int t = (int)(e / width), c = (int)(e % width);
        const int seq = seq_of_token[t];
        float now = 0.f, before = 0.f;                         // a padding row
        if (seq >= 0) {
            now = to_float<T>(x[e]);
            const int slot = slots[seq];
            if (t > cu_q[seq]) before = to_float<T>(x[e - width]);
            else if (slot >= 0) before = state[(long long)slot * slot_stride + c];
        }
        for (int s = 0; s < count; ++s)
            mixes[s * total + e] = from_float<T>(fmaf(before - now, mu[(long long)s * width + c], now));
    }
}

// `state` points at the request slots' previous rows ([width] floats a slot, `slot_stride` floats apart); it is read
// here and moved on by the kernel that prepares the scan's inputs.
TS_API int ts_token_shift(const void* x, const float* mu, const int* seq_of_token, const int* cu_q, const int* slots,
                          const float* state, long long slot_stride, void* mixes, int num_tokens, int width, int count,
                          int dtype, cudaStream_t stream) {
    TS_REQUIRE(width > 0 && count > 0 && slot_stride >= width, "token_shift: bad sizes");
    if (num_tokens <= 0) return 0;
    const long long total = (long long)num_tokens * width;
    const unsigned blocks = (unsigned)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    if (dtype == TS_F32)
        token_shift_kernel<float><<<blocks, 256, 0, stream>>>((const float*)x, mu, seq_of_token, cu_q, slots, state, slot_stride,
                                                              (float*)mixes, num_tokens, width, count);
    else if (dtype == TS_BF16)
        token_shift_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)x, mu, seq_of_token, cu_q, slots, state,
                                                                      slot_stride, (__nv_bfloat16*)mixes, num_tokens, width, count);
    else
        return ts_fail("token_shift: unknown dtype code %d", dtype);
    TS_LAUNCH_CHECK("token_shift");
    return 0;
}

// One warp a (token, head); the blocks past `item_blocks` move the requests' previous rows on (a warp takes 32 x 4
// channels of one request).
template <typename T>
__global__ void time_mix_prepare_kernel(const T* __restrict__ r, const T* __restrict__ k, long long rk_stride,
                                        const float* __restrict__ z, const float* __restrict__ w0, const float* __restrict__ u,
                                        float* __restrict__ prepared, float* __restrict__ bonus, long long items, int heads,
                                        int dim, unsigned item_blocks, const T* __restrict__ x, int width,
                                        const int* __restrict__ cu_q, const int* __restrict__ slots, int num_seqs,
                                        float* __restrict__ state, long long slot_stride, const int* __restrict__ single_of) {
    const int lane = threadIdx.x & 31;
    if (blockIdx.x >= item_blocks) {
        const int stretches = (width + 127) / 128;
        const long long w = (long long)(blockIdx.x - item_blocks) * (blockDim.x >> 5) + (threadIdx.x >> 5);
        const int seq = (int)(w / stretches), c0 = (int)(w % stretches) * 128;
        if (seq >= num_seqs) return;
        const int slot = slots[seq], last = cu_q[seq + 1] - 1;
        if (slot < 0 || last < cu_q[seq]) return;              // a padding request, or one that feeds nothing
        for (int c = c0 + lane; c < min(c0 + 128, width); c += 32)
            state[(long long)slot * slot_stride + c] = to_float<T>(x[(long long)last * width + c]);
        return;
    }
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= items) return;
    const long long t = item / heads;
    if (!feeds_one(single_of, cu_q, t)) return;
    const int h = (int)(item % heads);
    const T* rr = r + t * rk_stride + (long long)h * dim;
    const T* kr = k + t * rk_stride + (long long)h * dim;
    const long long at = item * dim, total = items * dim, hc = (long long)h * dim;
    float acc = 0.f;
    for (int i = lane; i < dim; i += 32) {
        const float rv = to_float<T>(rr[i]), kv = to_float<T>(kr[i]);
        prepared[at + i] = rv;
        prepared[total + at + i] = kv;
        prepared[2 * total + at + i] = expf(-expf(z[at + i] + w0[hc + i]));
        acc = fmaf(u[hc + i] * kv, rv, acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) bonus[item] = acc;
}

// r, k: [tokens, heads * dim] with one row stride; z float32 [tokens, heads * dim]; prepared [3][tokens, heads * dim],
// bonus [tokens, heads].  `x` [tokens, width] is the mixer's input, whose last row of every request goes to its slot.
// `portions_only` 1: no token is prepared, the rows move on all the same; `single_of` (optional): only tokens of
// requests that feed one are prepared.
TS_API int ts_time_mix_prepare(const void* r, const void* k, long long rk_stride, const float* z, const float* w0,
                               const float* u, float* prepared, float* bonus, int num_tokens, int heads, int dim,
                               const void* x, int width, const int* cu_q, const int* slots, int num_seqs, float* state,
                               long long slot_stride, int portions_only, const int* single_of, int dtype,
                               cudaStream_t stream) {
    TS_REQUIRE(heads > 0 && dim > 0 && width > 0 && slot_stride >= width, "time_mix_prepare: bad sizes");
    if (num_tokens <= 0 || num_seqs <= 0) return 0;
    const long long items = portions_only ? 0 : (long long)num_tokens * heads;
    const unsigned item_blocks = (unsigned)((items + 3) / 4);
    const unsigned more = (unsigned)(((long long)num_seqs * ((width + 127) / 128) + 3) / 4);
    if (dtype == TS_F32)
        time_mix_prepare_kernel<float><<<item_blocks + more, 128, 0, stream>>>((const float*)r, (const float*)k, rk_stride, z, w0, u,
            prepared, bonus, items, heads, dim, item_blocks, (const float*)x, width, cu_q, slots, num_seqs, state, slot_stride,
            single_of);
    else if (dtype == TS_BF16)
        time_mix_prepare_kernel<__nv_bfloat16><<<item_blocks + more, 128, 0, stream>>>((const __nv_bfloat16*)r, (const __nv_bfloat16*)k,
            rk_stride, z, w0, u, prepared, bonus, items, heads, dim, item_blocks, (const __nv_bfloat16*)x, width, cu_q, slots,
            num_seqs, state, slot_stride, single_of);
    else
        return ts_fail("time_mix_prepare: unknown dtype code %d", dtype);
    TS_LAUNCH_CHECK("time_mix_prepare");
    return 0;
}

// One warp a (request, head): 32 tokens at a time, each lane its token's gates; the running maximum is carried
// through the lanes by a scan.  factors[0] = decay, factors[1] = the key's factor, each [tokens, heads].
__global__ void mlstm_gates_kernel(const float* __restrict__ gi, const float* __restrict__ gf, long long gate_stride,
                                   const float* __restrict__ bias_i, const float* __restrict__ bias_f, float cap,
                                   const int* __restrict__ cu_q, const int* __restrict__ slots, float* __restrict__ state,
                                   long long slot_stride, float* __restrict__ log_max, float* __restrict__ factors,
                                   long long num_items, int num_seqs, int heads) {
    const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= num_seqs * heads) return;
    const int lane = threadIdx.x & 31;
    const int seq = item / heads, h = item % heads;
    const int slot = slots[seq];
    const int begin = cu_q[seq], end = cu_q[seq + 1];
    if (slot < 0 || end <= begin) return;
    float* m_state = state + (long long)slot * slot_stride + h;
    float m = *m_state;
    const float bi = bias_i[h], bf = bias_f[h];
    // a round's projections are loaded one round ahead of their use
    float next_i = begin + lane < end ? gi[(long long)(begin + lane) * gate_stride + h] : 0.f;
    float next_f = begin + lane < end ? gf[(long long)(begin + lane) * gate_stride + h] : 0.f;
    for (int t0 = begin; t0 < end; t0 += 32) {
        const int t = t0 + lane;
        const float raw_i = next_i, raw_f = next_f;
        if (t + 32 < end) {
            next_i = gi[(long long)(t + 32) * gate_stride + h];
            next_f = gf[(long long)(t + 32) * gate_stride + h];
        }
        float i_gate = 0.f, f_gate = 0.f;
        if (t < end) {
            i_gate = cap * tanhf((raw_i + bi) / cap);
            f_gate = log_sigmoid_f(cap * tanhf((raw_f + bf) / cap));
        }
        // m_t = max(f_t + m_(t-1), i_t) is the composition of the maps x -> max(x + a, b); an inclusive scan over the
        // lanes composes them: (a, b) after (a', b') = (a' + a, max(b' + a, b)).  Lanes past the end hold the identity.
        float a = t < end ? f_gate : 0.f, b = t < end ? i_gate : -INFINITY;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pa = __shfl_up_sync(0xffffffffu, a, o), pb = __shfl_up_sync(0xffffffffu, b, o);
            if (lane >= o) { b = fmaxf(pb + a, b); a = pa + a; }
        }
        const float after = fmaxf(m + a, b);
        float before = __shfl_up_sync(0xffffffffu, after, 1);
        if (lane == 0) before = m;
        m = __shfl_sync(0xffffffffu, after, 31);          // lanes past the end carry the last token's value on
        if (t < end) {
            const long long at = (long long)t * heads + h;
            log_max[at] = after;
            factors[at] = expf(f_gate + before - after);
            factors[num_items + at] = expf(i_gate - after);
        }
    }
    if (lane == 0) *m_state = m;
}

template <typename T>
__global__ void mlstm_prepare_kernel(const T* __restrict__ q, const T* __restrict__ k, long long q_stride, long long k_stride,
                                     const float* __restrict__ factors, long long num_items, float q_scale,
                                     float* __restrict__ prepared, long long total, int heads, int dim) {
    const int width = heads * dim;
    for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
        const long long t = e / width;
        const int c = (int)(e % width), h = c / dim;
        const long long item = t * heads + h;
        prepared[e] = to_float<T>(q[t * q_stride + c]) * q_scale;
        prepared[total + e] = to_float<T>(k[t * k_stride + c]) * factors[num_items + item];
        prepared[2 * total + e] = factors[item];
    }
}

// `state` points at the request slots' running maxima ([heads] floats a slot, `slot_stride` floats apart).
TS_API int ts_mlstm_prepare(const void* q, const void* k, long long q_stride, long long k_stride, const float* gi,
                            const float* gf, long long gate_stride, const float* bias_i, const float* bias_f, float cap,
                            float q_scale, const int* cu_q, const int* slots, int num_seqs, float* state,
                            long long slot_stride, float* log_max, float* factors, float* prepared, int num_tokens,
                            int heads, int dim, int dtype, cudaStream_t stream) {
    TS_REQUIRE(heads > 0 && dim > 0 && cap > 0.f, "mlstm_prepare: bad sizes or gate cap");
    if (num_tokens <= 0 || num_seqs <= 0) return 0;
    const long long items = (long long)num_tokens * heads, total = items * dim;
    const unsigned blocks_a = (unsigned)(((long long)num_seqs * heads + 3) / 4);
    const unsigned blocks_b = (unsigned)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
#define TS_MLSTM(TYPE)                                                                                                 \
    do {                                                                                                               \
        mlstm_gates_kernel<<<blocks_a, 128, 0, stream>>>(gi, gf, gate_stride, bias_i,                                  \
            bias_f, cap, cu_q, slots, state, slot_stride, log_max, factors, items, num_seqs, heads);                   \
        mlstm_prepare_kernel<TYPE><<<blocks_b, 256, 0, stream>>>((const TYPE*)q, (const TYPE*)k, q_stride, k_stride,   \
            factors, items, q_scale, prepared, total, heads, dim);                                                     \
    } while (0)
    if (dtype == TS_F32) TS_MLSTM(float);
    else if (dtype == TS_BF16) TS_MLSTM(__nv_bfloat16);
    else return ts_fail("mlstm_prepare: unknown dtype code %d", dtype);
#undef TS_MLSTM
    TS_LAUNCH_CHECK("mlstm_prepare");
    return 0;
}
