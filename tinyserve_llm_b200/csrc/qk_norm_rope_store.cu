// What lies between the q/k/v projection and the attention of a mixer whose queries and keys are
// normed over the whole projection:
//
//   q = y_q + b_q,  k = y_k + b_k,  v = y_v + b_v                      (biases optional)
//   q = q / sqrt(mean(q^2) + eps) * w_q     over all heads' channels at once, likewise k   (optional);
//       with `norm_per_head` every head is normed by itself and w_q, w_k hold one head's channels; `unweighted`
//       norms every head of q and of k without a weight
//   q = q * (1 + temp_coef * ln(floor((position + 1) / temp_every) + 1))             (temp_every > 0)
//   rotate-half rotation of the first `rot` channels of every head of q and k: channel i pairs with
//   i + rot/2, angle = position * freq[i], cos and sin both multiplied by `magnitude`; `interleaved` pairs channel
//   2i with 2i + 1 instead.  (A rotation by pairs keeps a head's sum of squares, so a norm of a head without a
//   weight is the same before the rotation and after it.)
//   k and v go to the token's slot of the paged cache, q to a compact [tokens, heads * dim] tensor.
//
// Keys and values may differ in their head size and in their number of heads (`v_heads`: several key heads over
// one value head), so the value pool has a geometry of its own.  Values may also be the keys as projected: their
// columns are then k's own (`v_off` = `k_off`), stored without norm and rotation.
// With `v_mix` (a stretch of rows like v's own, of another layer) the stored value is (1 - v_lambda) v + v_lambda v_mix.
// One CTA a token; sums, angles and the rotation are float32, the stores round to the activation dtype.
#include "common.cuh"

struct QKPrepareArgs {
    const void* y; long long y_stride; int q_off, k_off, v_off;     // columns of q, k and v inside a row of y
    const float* q_bias; const float* k_bias; const float* v_bias;
    const float* q_weight; const float* k_weight; float eps;        // null weights: no norm
    const float* freq; int rot; float magnitude;
    const int* positions; const int* seq_of_token;
    void* q_out;
    void* k_pool; void* v_pool; KVGeometry k_geo; KVGeometry v_geo;
    const int* block_table; int table_width; int writes;
    int heads, kv_heads, dim, vdim, v_heads;
    int norm_per_head; float temp_coef; int temp_every;
    int unweighted, interleaved;
    const void* v_mix; long long v_mix_stride; float v_lambda;
};

// VEC (1 or 2) neighbouring channels a lane: 2 where head sizes, half the rotation and all offsets are even.
template <typename T, int VEC>
struct alignas(sizeof(T) * VEC) Pack {
    T v[VEC];
};

template <typename T, int VEC>
__global__ void qk_norm_rope_store_kernel(QKPrepareArgs p) {
    __shared__ float scratch[32];
    extern __shared__ float turn[];                   // cos, then sin, of the token's rot / 2 angles, times the magnitude
    const int t = blockIdx.x;
    const int seq = p.seq_of_token[t];
    const int nq = p.heads * p.dim, nk = p.kv_heads * p.dim;
    T* q_out = (T*)p.q_out + (long long)t * nq;
    if (seq < 0) {                                    // a padding row
        for (int e = threadIdx.x; e < nq; e += blockDim.x) q_out[e] = from_float<T>(0.f);
        return;
    }
    const T* row = (const T*)p.y + (long long)t * p.y_stride;
    const T* yq = row + p.q_off;
    const T* yk = row + p.k_off;
    const T* yv = row + p.v_off;
    // what does not depend on the sums is asked for first: the position and the page
    const int pos = p.positions[t];
    const int half = p.freq ? p.rot / 2 : 0, rot = 2 * half;
    const int page = p.writes ? p.block_table[(long long)seq * p.table_width + pos / p.k_geo.page_tokens] : -1;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {        // one sine and cosine an angle, for all heads
        float sn, cs;
        sincosf((float)pos * p.freq[i], &sn, &cs);
        turn[i] = cs * p.magnitude;
        turn[half + i] = sn * p.magnitude;
    }
    float inv_q = 1.f, inv_k = 1.f;
    if (!p.norm_per_head && (p.q_weight || p.k_weight)) {         // both sums in one pass over the row, then two reductions
        float acc_q = 0.f, acc_k = 0.f;
        if (p.q_weight)
            for (int e = threadIdx.x; e < nq; e += blockDim.x) {
                const float x = to_float<T>(yq[e]) + (p.q_bias ? p.q_bias[e] : 0.f);
                acc_q += x * x;
            }
        if (p.k_weight)
            for (int e = threadIdx.x; e < nk; e += blockDim.x) {
                const float x = to_float<T>(yk[e]) + (p.k_bias ? p.k_bias[e] : 0.f);
                acc_k += x * x;
            }
        if (p.q_weight) {
            inv_q = 1.f / sqrtf(block_sum(acc_q, scratch) / (float)nq + p.eps);
            __syncthreads();
        }
        if (p.k_weight) inv_k = 1.f / sqrtf(block_sum(acc_k, scratch) / (float)nk + p.eps);
    }
    __syncthreads();                                  // turn
    const float temperature = p.temp_every > 0
        ? 1.f + p.temp_coef * logf((float)((pos + 1) / p.temp_every) + 1.f) : 1.f;
    const bool stores = p.writes && page >= 0 && page < p.k_geo.num_pages;
    const int slot = pos % p.k_geo.page_tokens;
    T* kp = stores ? (T*)p.k_pool + (long long)page * p.k_geo.page_stride + p.k_geo.entry_offset : nullptr;
    T* vp = stores ? (T*)p.v_pool + (long long)page * p.v_geo.page_stride + p.v_geo.entry_offset : nullptr;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    for (int hh = warp; hh < p.heads + (stores ? p.kv_heads : 0); hh += nwarps) {     // a warp a head of q or k
        const bool is_q = hh < p.heads;
        const int h = is_q ? hh : hh - p.heads, e0 = h * p.dim;
        const T* y = (is_q ? yq : yk) + e0;
        const float* bias = is_q ? p.q_bias : p.k_bias;
        if (bias) bias += e0;
        const float* weight = is_q ? p.q_weight : p.k_weight;
        if (weight && !p.norm_per_head) weight += e0;
        T* dst = is_q ? q_out + e0 : kp + ((long long)h * p.k_geo.page_tokens + slot) * p.dim;
        auto load = [&](int i, float (&x)[VEC]) {
            const Pack<T, VEC> raw = *reinterpret_cast<const Pack<T, VEC>*>(y + i);
#pragma unroll
            for (int j = 0; j < VEC; ++j) x[j] = to_float<T>(raw.v[j]) + (bias ? bias[i + j] : 0.f);
        };
        float gain = is_q ? temperature : 1.f;
        if (p.norm_per_head) {
            if (weight || p.unweighted) {
                float acc = 0.f, x[VEC];
                for (int i = lane * VEC; i < p.dim; i += 32 * VEC) {
                    load(i, x);
#pragma unroll
                    for (int j = 0; j < VEC; ++j) acc += x[j] * x[j];
                }
                gain *= 1.f / sqrtf(warp_sum(acc) / (float)p.dim + p.eps);
            }
        } else if (weight) {
            gain *= is_q ? inv_q : inv_k;
        }
        auto element = [&](int i, float (&x)[VEC]) {
            load(i, x);
#pragma unroll
            for (int j = 0; j < VEC; ++j) x[j] *= weight ? gain * weight[i + j] : gain;
        };
        auto store = [&](int i, const float (&x)[VEC]) {
            Pack<T, VEC> raw;
#pragma unroll
            for (int j = 0; j < VEC; ++j) raw.v[j] = from_float<T>(x[j]);
            *reinterpret_cast<Pack<T, VEC>*>(dst + i) = raw;
        };
        if (p.interleaved) {                          // channels 2i and 2i + 1
            for (int i = lane; i < half; i += 32) {
                float u[2];
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    u[j] = (to_float<T>(y[2 * i + j]) + (bias ? bias[2 * i + j] : 0.f)) * (weight ? gain * weight[2 * i + j] : gain);
                dst[2 * i] = from_float<T>(u[0] * turn[i] - u[1] * turn[half + i]);
                dst[2 * i + 1] = from_float<T>(u[1] * turn[i] + u[0] * turn[half + i]);
            }
        } else {
            for (int i = lane * VEC; i < half; i += 32 * VEC) {
                float u[VEC], v[VEC], a[VEC], b[VEC];
                element(i, u);
                element(i + half, v);
#pragma unroll
                for (int j = 0; j < VEC; ++j) {
                    a[j] = u[j] * turn[i + j] - v[j] * turn[half + i + j];
                    b[j] = v[j] * turn[i + j] + u[j] * turn[half + i + j];
                }
                store(i, a);
                store(i + half, b);
            }
        }
        for (int i = rot + lane * VEC; i < p.dim; i += 32 * VEC) {       // channels past the rotation
            float x[VEC];
            element(i, x);
            store(i, x);
        }
    }
    if (!stores) return;
    const T* mix = p.v_mix ? (const T*)p.v_mix + (long long)t * p.v_mix_stride : nullptr;
    for (int h = warp; h < p.v_heads; h += nwarps) {
        T* dst = vp + ((long long)h * p.v_geo.page_tokens + slot) * p.vdim;
        const int e0 = h * p.vdim;
        for (int i = lane * VEC; i < p.vdim; i += 32 * VEC) {
            const Pack<T, VEC> raw = *reinterpret_cast<const Pack<T, VEC>*>(yv + e0 + i);
            Pack<T, VEC> other{}, o;
            if (mix) other = *reinterpret_cast<const Pack<T, VEC>*>(mix + e0 + i);
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                float v = to_float<T>(raw.v[j]) + (p.v_bias ? p.v_bias[e0 + i + j] : 0.f);
                if (mix) v = (1.f - p.v_lambda) * v + p.v_lambda * to_float<T>(other.v[j]);
                o.v[j] = from_float<T>(v);
            }
            *reinterpret_cast<Pack<T, VEC>*>(dst + i) = o;
        }
    }
}

TS_API int ts_qk_norm_rope_store(const void* y, long long y_stride, int q_off, int k_off, int v_off, const float* q_bias,
                                 const float* k_bias, const float* v_bias, const float* q_weight, const float* k_weight,
                                 float eps, const float* freq, int rot, float magnitude, const int* positions,
                                 const int* seq_of_token, void* q_out, void* k_pool, void* v_pool, long long k_page_stride,
                                 long long k_entry_offset, long long v_page_stride, long long v_entry_offset,
                                 int page_tokens, int num_pages, const int* block_table, int table_width, int writes,
                                 int num_tokens, int heads, int kv_heads, int dim, int vdim, int dtype,
                                 int norm_per_head, float temp_coef, int temp_every, int value_heads, int unweighted,
                                 int interleaved, const void* v_mix, long long v_mix_stride, float v_lambda,
                                 cudaStream_t stream) {
    TS_REQUIRE(!unweighted || (norm_per_head && !q_weight && !k_weight), "qk_norm_rope_store: an unweighted norm is one a head");
    TS_REQUIRE(value_heads >= 0, "qk_norm_rope_store: bad number of value heads");
    TS_REQUIRE(heads > 0 && kv_heads > 0 && dim > 0 && vdim > 0 && num_tokens >= 0, "qk_norm_rope_store: bad sizes");
    TS_REQUIRE(rot >= 0 && rot <= dim && rot % 2 == 0, "qk_norm_rope_store: rotation over %d of %d channels", rot, dim);
    TS_REQUIRE(page_tokens > 0 && table_width > 0, "qk_norm_rope_store: bad page geometry");
    if (num_tokens == 0) return 0;
    QKPrepareArgs p{y, y_stride, q_off, k_off, v_off, q_bias, k_bias, v_bias, q_weight, k_weight, eps,
                    rot > 0 ? freq : nullptr, rot, magnitude, positions, seq_of_token, q_out, k_pool, v_pool,
                    KVGeometry{k_page_stride, k_entry_offset, page_tokens, num_pages},
                    KVGeometry{v_page_stride, v_entry_offset, page_tokens, num_pages}, block_table, table_width, writes,
                    heads, kv_heads, dim, vdim, value_heads > 0 ? value_heads : kv_heads, norm_per_head, temp_coef, temp_every,
                    unweighted, interleaved, v_mix, v_mix_stride, v_lambda};
    const size_t smem = (size_t)(p.freq ? rot : 0) * sizeof(float);
    TS_REQUIRE(smem <= 32 * 1024, "qk_norm_rope_store: rotation over %d channels is not supported", rot);
    const bool even = dim % 2 == 0 && vdim % 2 == 0 && (interleaved || (rot / 2) % 2 == 0) && y_stride % 2 == 0 && q_off % 2 == 0 &&
                      k_off % 2 == 0 && v_off % 2 == 0 && v_mix_stride % 2 == 0 && k_page_stride % 2 == 0 && k_entry_offset % 2 == 0 &&
                      v_page_stride % 2 == 0 && v_entry_offset % 2 == 0 &&
                      ((uintptr_t)y | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)v_mix) % 8 == 0;
    // many tokens: small CTAs, many of them on an SM (a CTA's life is a chain of loads and two sums); few tokens: wide ones
    const int threads = num_tokens >= 512 ? 128 : (heads * dim >= 2048 ? 512 : 256);
#define TS_QK_PREPARE(T)                                                                          \
    do {                                                                                          \
        if (even) qk_norm_rope_store_kernel<T, 2><<<num_tokens, threads, smem, stream>>>(p);      \
        else qk_norm_rope_store_kernel<T, 1><<<num_tokens, threads, smem, stream>>>(p);           \
    } while (0)
    if (dtype == TS_F32) TS_QK_PREPARE(float);
    else if (dtype == TS_BF16) TS_QK_PREPARE(__nv_bfloat16);
    else return ts_fail("qk_norm_rope_store: unknown dtype code %d", dtype);
#undef TS_QK_PREPARE
    TS_LAUNCH_CHECK("qk_norm_rope_store");
    return 0;
}

// out[t, c] = a[t, c] * sigmoid(gate[t, c]) * scale, each operand with a row stride of its own (the
// result may be a column stretch of a wider tensor).  An output gate on concatenated heads.
template <typename T>
__global__ void sigmoid_gate_kernel(const T* __restrict__ a, long long a_stride, const T* __restrict__ gate,
                                    long long gate_stride, T* __restrict__ out, long long out_stride, long long total,
                                    int cols, float scale) {
    for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (long long)gridDim.x * blockDim.x) {
        const long long t = idx / cols;
        const int c = (int)(idx % cols);
        const float g = to_float<T>(gate[t * gate_stride + c]);
        out[t * out_stride + c] = from_float<T>(to_float<T>(a[t * a_stride + c]) / (1.f + expf(-g)) * scale);
    }
}

TS_API int ts_sigmoid_gate(const void* a, long long a_stride, const void* gate, long long gate_stride, void* out,
                           long long out_stride, int num_tokens, int cols, float scale, int dtype, cudaStream_t stream) {
    TS_REQUIRE(num_tokens >= 0 && cols > 0, "sigmoid_gate: bad sizes");
    if (num_tokens == 0) return 0;
    const long long total = (long long)num_tokens * cols;
    const unsigned blocks = (unsigned)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    if (dtype == TS_F32)
        sigmoid_gate_kernel<float><<<blocks, 256, 0, stream>>>((const float*)a, a_stride, (const float*)gate, gate_stride,
                                                               (float*)out, out_stride, total, cols, scale);
    else if (dtype == TS_BF16)
        sigmoid_gate_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)a, a_stride,
            (const __nv_bfloat16*)gate, gate_stride, (__nv_bfloat16*)out, out_stride, total, cols, scale);
    else
        return ts_fail("sigmoid_gate: unknown dtype code %d", dtype);
    TS_LAUNCH_CHECK("sigmoid_gate");
    return 0;
}
