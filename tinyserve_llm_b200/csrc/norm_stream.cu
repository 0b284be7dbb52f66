// RMS norms around a residual stream that is kept in float32 whatever the activation dtype.
//
// One kernel does what lies between two sublayers of a block that norms each sublayer's input and
// output:  s = stream + closing(branch),  stream' = s,  out = opening(s)  with
//   closing(b) = b / sqrt(mean(b^2) + eps) * w_close      (the norm after the sublayer that made b)
//   opening(s) = s / sqrt(mean(s^2) + eps) * w_open       (the norm before the next sublayer)
// Every part is optional: no branch (the stream is only normed: a block's first norm after a block
// that closed its own branch), no opening weight (the branch is only added), `rows` (only these
// rows are normed into a compact output and the stream is not written: the final norm of the
// wanted places), `ids` (the row is table[ids[r]] * scale and starts the stream: the embedding; with
// `pos_freq` a sinusoidal position vector is added to it: entry 2i gets sin(position * pos_freq[i]),
// entry 2i + 1 the cosine of the same angle, the angle a float32 product; with `w_start` the gathered row is
// itself normed with that weight, in the way the opening norm is, before it starts the stream: a norm on the embedding).
// Statistics, weights, the sum and the stream are float32; the branch and `out` have the activation
// dtype.  The weights are given as they multiply (an offset of the stored weight is added by the host).
//
// With a second branch (`branch2`) the sublayer is two mixers side by side whose outputs are normed one by one:
//   b = branch_scale * branch / sqrt(mean(branch^2) + eps) * w_branch + branch_scale2 * (the same of branch2 with w_branch2)
// takes the place of the branch; with a closing weight of null and no plain add, b itself goes to `out` (no stream).
// Branches without norms of their own (null `w_branch`, TS_NORM_PLAIN_ADD) are added as they are, each times its scale.
//
// With `pairs.table` the gathered embedding row (times `scale`) gets a second row added, of a table of buckets + 1 rows
// picked by (previous token, token): (previous * mul_prev + token * mul_cur) mod buckets, the last row where there is no
// previous token.  The previous token is the one before in the batch, or prev_tokens[request] for a request's first row.
//
// `flags`: TS_NORM_CENTERED makes the opening norm a layer norm without bias,
//   opening(s) = (s - mean(s)) / sqrt(mean((s - mean(s))^2) + eps) * w_open;
// TS_NORM_PLAIN_ADD adds the branch as it is (a block that norms only the inputs of its sublayers);
// TS_NORM_COPY_OUT writes the new row of the stream to `out` without an opening norm (a block that norms only the
// outputs of its sublayers: the next sublayer reads the stream itself, rounded to the activation dtype).
#include "common.cuh"

enum { TS_NORM_CENTERED = 1, TS_NORM_PLAIN_ADD = 2, TS_NORM_COPY_OUT = 4 };

// Two branches of one sublayer, each under a norm of its own (null `branch2`: a single branch).
struct BranchPair {
    const void* branch2;
    const float* w_branch;
    const float* w_branch2;
    float scale, scale2;
};

// A second embedding by (previous token, token); null `table`: none.
struct PairTable {
    const void* table;
    const int* prev_tokens; const int* cu_q; const int* seq_of_token;
    int buckets;
    long long mul_prev, mul_cur;
};

// The row of the pair table for batch row `r` (a padding row: -1).
__device__ __forceinline__ long long pair_row(const PairTable& p, const int* ids, int r) {
    const int seq = p.seq_of_token[r];
    if (seq < 0) return -1;
    const int prev = r > p.cu_q[seq] ? ids[r - 1] : p.prev_tokens[seq];
    if (prev < 0) return p.buckets;
    return (prev * p.mul_prev + ids[r] * p.mul_cur) % p.buckets;
}

template <typename T>
__global__ void stream_norm_kernel(const T* __restrict__ branch, const float* __restrict__ w_close, float* stream,
                                   const float* __restrict__ w_open, T* __restrict__ out,
                                   const int* __restrict__ rows, int width, float eps, const T* __restrict__ table,
                                   const int* __restrict__ ids, int table_rows, float scale, int write_stream,
                                   int flags, const int* __restrict__ positions, const float* __restrict__ pos_freq,
                                   const float* __restrict__ w_start, BranchPair pair, PairTable pairs) {
    extern __shared__ float row[];                // width floats, then 64 of scratch
    float* scratch = row + width;
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    if (src < 0) return;                          // a padding row
    float* sr = stream + (long long)src * width;
    T* o = out + (long long)r * width;
    if (pair.branch2 && pair.w_branch) {          // the two branches' norms; their sum stands in for the branch from here on
        const T* b1 = branch + (long long)src * width;
        const T* b2 = (const T*)pair.branch2 + (long long)src * width;
        float acc1 = 0.f, acc2 = 0.f;
        for (int i = threadIdx.x; i < width; i += blockDim.x) {
            const float x1 = to_float<T>(b1[i]), x2 = to_float<T>(b2[i]);
            acc1 += x1 * x1;
            acc2 += x2 * x2;
        }
        const float inv1 = pair.scale / sqrtf(block_sum(acc1, scratch) / (float)width + eps);
        const float inv2 = pair.scale2 / sqrtf(block_sum(acc2, scratch + 32) / (float)width + eps);
        float acc = 0.f;
        for (int i = threadIdx.x; i < width; i += blockDim.x) {      // each thread reads back only the elements it wrote
            const float b = to_float<T>(b1[i]) * inv1 * pair.w_branch[i] + to_float<T>(b2[i]) * inv2 * pair.w_branch2[i];
            row[i] = b;
            acc += b * b;
        }
        if (!stream) {
            for (int i = threadIdx.x; i < width; i += blockDim.x) o[i] = from_float<T>(row[i]);
            return;
        }
        __syncthreads();                          // scratch is used again below
        if (flags & TS_NORM_PLAIN_ADD) {
            for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] += sr[i];
        } else {
            const float inv = 1.f / sqrtf(block_sum(acc, scratch) / (float)width + eps);
            __syncthreads();
            for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = sr[i] + row[i] * inv * w_close[i];
        }
    } else
    if (ids) {
        const int id = ids[src];
        const bool zeros = id < 0 || id >= table_rows;
        const T* tr = table + (long long)(zeros ? 0 : id) * width;
        if (pos_freq) {
            const float pos = (float)positions[src];
            for (int i = threadIdx.x; i < width; i += blockDim.x) {
                const float angle = pos * pos_freq[i >> 1];
                row[i] = (zeros ? 0.f : to_float<T>(tr[i]) * scale) + ((i & 1) ? cosf(angle) : sinf(angle));
            }
        } else if (pairs.table && !zeros) {
            const long long pr = pair_row(pairs, ids, src);
            const T* second = (const T*)pairs.table + (pr < 0 ? 0 : pr) * width;
            for (int i = threadIdx.x; i < width; i += blockDim.x)
                row[i] = to_float<T>(tr[i]) * scale + (pr < 0 ? 0.f : to_float<T>(second[i]));
        } else {
            for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = zeros ? 0.f : to_float<T>(tr[i]) * scale;
        }
        if (w_start) {                            // each thread reads back only the elements it wrote
            float mean = 0.f;
            if (flags & TS_NORM_CENTERED) {
                float sum = 0.f;
                for (int i = threadIdx.x; i < width; i += blockDim.x) sum += row[i];
                mean = block_sum(sum, scratch) / (float)width;
                __syncthreads();
            }
            float acc = 0.f;
            for (int i = threadIdx.x; i < width; i += blockDim.x) acc += (row[i] - mean) * (row[i] - mean);
            const float inv = 1.f / sqrtf(block_sum(acc, scratch) / (float)width + eps);
            __syncthreads();                      // scratch is used again below
            for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = (row[i] - mean) * inv * w_start[i];
        }
    } else if (branch && (flags & TS_NORM_PLAIN_ADD)) {
        const T* br = branch + (long long)src * width;
        if (pair.branch2) {
            const T* b2 = (const T*)pair.branch2 + (long long)src * width;
            for (int i = threadIdx.x; i < width; i += blockDim.x)
                row[i] = sr[i] + (pair.scale * to_float<T>(br[i]) + pair.scale2 * to_float<T>(b2[i]));
        } else {
            for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = sr[i] + pair.scale * to_float<T>(br[i]);
        }
    } else if (branch) {
        const T* br = branch + (long long)src * width;
        float acc = 0.f;
        for (int i = threadIdx.x; i < width; i += blockDim.x) {
            const float b = to_float<T>(br[i]);
            row[i] = b;
            acc += b * b;
        }
        const float inv = 1.f / sqrtf(block_sum(acc, scratch) / (float)width + eps);
        __syncthreads();                          // scratch is used again below
        for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = sr[i] + row[i] * inv * w_close[i];
    } else {
        for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = sr[i];
    }
    if (write_stream && (ids || branch))
        for (int i = threadIdx.x; i < width; i += blockDim.x) sr[i] = row[i];
    if (!w_open) {
        if (flags & TS_NORM_COPY_OUT)
            for (int i = threadIdx.x; i < width; i += blockDim.x) o[i] = from_float<T>(row[i]);
        return;
    }
    float mean = 0.f;
    if (flags & TS_NORM_CENTERED) {
        float sum = 0.f;
        for (int i = threadIdx.x; i < width; i += blockDim.x) sum += row[i];
        mean = block_sum(sum, scratch) / (float)width;
        __syncthreads();                          // scratch is used again below
    }
    float acc = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) acc += (row[i] - mean) * (row[i] - mean);
    const float inv = 1.f / sqrtf(block_sum(acc, scratch) / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) o[i] = from_float<T>((row[i] - mean) * inv * w_open[i]);
}

// The commonest case, a branch (or two, each times its scale) added as it is and the sum normed, for rows of a multiple of 16
// bytes of the branch's type: a thread VEC neighbouring columns, up to STREAM_ITEMS times, the row in registers.
constexpr int STREAM_ITEMS = 4;

template <typename T>
__global__ void __launch_bounds__(256)
stream_add_norm_kernel(const T* __restrict__ branch, const T* __restrict__ branch2, float scale, float scale2, float* stream,
                       const float* __restrict__ w_open, T* __restrict__ out, const int* __restrict__ rows, int width, float eps,
                       int write_stream, int centered) {
    constexpr int VEC = 16 / sizeof(T);
    __shared__ float scratch[64];
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    if (src < 0) return;                          // a padding row
    float* sr = stream + (long long)src * width;
    float x[STREAM_ITEMS][VEC];
    float sum = 0.f, sq = 0.f;
#pragma unroll
    for (int m = 0; m < STREAM_ITEMS; ++m) {
        const int c = (m * blockDim.x + threadIdx.x) * VEC;
        if (c >= width) break;
        const uint4 raw = *reinterpret_cast<const uint4*>(branch + (long long)src * width + c);
        uint4 raw2 = make_uint4(0, 0, 0, 0);
        if (branch2) raw2 = *reinterpret_cast<const uint4*>(branch2 + (long long)src * width + c);
        const T* e = reinterpret_cast<const T*>(&raw);
        const T* e2 = reinterpret_cast<const T*>(&raw2);
#pragma unroll
        for (int i = 0; i < VEC; i += 4) {
            const float4 s = *reinterpret_cast<const float4*>(sr + c + i);
            x[m][i] = s.x; x[m][i + 1] = s.y; x[m][i + 2] = s.z; x[m][i + 3] = s.w;
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const float b = branch2 ? scale * to_float<T>(e[i]) + scale2 * to_float<T>(e2[i]) : scale * to_float<T>(e[i]);
            x[m][i] += b;
            sum += x[m][i];
            sq += x[m][i] * x[m][i];
        }
        if (write_stream)
#pragma unroll
            for (int i = 0; i < VEC; i += 4)
                *reinterpret_cast<float4*>(sr + c + i) = make_float4(x[m][i], x[m][i + 1], x[m][i + 2], x[m][i + 3]);
    }
    float mean = 0.f;
    if (centered) {
        mean = block_sum(sum, scratch) / (float)width;
        sq = 0.f;
#pragma unroll
        for (int m = 0; m < STREAM_ITEMS; ++m) {
            if ((m * blockDim.x + threadIdx.x) * VEC >= width) break;
#pragma unroll
            for (int i = 0; i < VEC; ++i) sq += (x[m][i] - mean) * (x[m][i] - mean);
        }
    }
    const float inv = 1.f / sqrtf(block_sum(sq, scratch + 32) / (float)width + eps);
#pragma unroll
    for (int m = 0; m < STREAM_ITEMS; ++m) {
        const int c = (m * blockDim.x + threadIdx.x) * VEC;
        if (c >= width) break;
        alignas(16) T o[VEC];
#pragma unroll
        for (int i = 0; i < VEC; i += 4) {
            const float4 w = *reinterpret_cast<const float4*>(w_open + c + i);
            o[i] = from_float<T>((x[m][i] - mean) * inv * w.x);
            o[i + 1] = from_float<T>((x[m][i + 1] - mean) * inv * w.y);
            o[i + 2] = from_float<T>((x[m][i + 2] - mean) * inv * w.z);
            o[i + 3] = from_float<T>((x[m][i + 3] - mean) * inv * w.w);
        }
        *reinterpret_cast<uint4*>(out + (long long)r * width + c) = *reinterpret_cast<const uint4*>(o);
    }
}

template <typename T>
static void launch_stream_add_norm(const void* branch, const void* branch2, float scale, float scale2, float* stream, const float* w_open,
                                   void* out, const int* rows, int count, int width, float eps, int write, int centered, cudaStream_t s) {
    constexpr int VEC = 16 / sizeof(T);
    const int items = width / VEC;                // spread evenly: as many threads as take the row in the fewest rounds
    const int rounds = count <= 512 ? (items + 255) / 256 : (items + 127) / 128 <= STREAM_ITEMS ? (items + 127) / 128 : (items + 255) / 256;
    const int threads = ((items + rounds - 1) / rounds + 31) / 32 * 32;
    stream_add_norm_kernel<T><<<count, threads, 0, s>>>((const T*)branch, (const T*)branch2, scale, scale2, stream, w_open, (T*)out,
                                                        rows, width, eps, write, centered);
}

TS_API int ts_stream_norm(const void* branch, const float* w_close, float* stream, const float* w_open, void* out,
                          const int* rows, int count, int width, float eps, const void* table, const int* ids,
                          int table_rows, float scale, int flags, int dtype, const int* positions, const float* pos_freq,
                          const float* w_start, const void* branch2, const float* w_branch, const float* w_branch2,
                          float branch_scale, float branch_scale2, const void* pair_table, const int* prev_tokens,
                          const int* cu_q, const int* seq_of_token, int buckets, long long mul_prev, long long mul_cur,
                          cudaStream_t stream_handle) {
    TS_REQUIRE(count >= 0 && width > 0, "stream_norm: bad sizes rows=%d width=%d", count, width);
    TS_REQUIRE(!branch2 || (branch && (w_branch != nullptr) == (w_branch2 != nullptr)),
               "stream_norm: two branches need both their norms' weights, or neither");
    TS_REQUIRE(!branch2 || w_branch || (flags & TS_NORM_PLAIN_ADD), "stream_norm: branches without norms are added as they are");
    TS_REQUIRE(!pair_table || (ids && !pos_freq && prev_tokens && cu_q && seq_of_token && buckets > 0 && mul_prev >= 0 && mul_cur >= 0),
               "stream_norm: a pair table needs token ids, the previous tokens and the requests' rows, and no position vector");
    TS_REQUIRE(stream != nullptr || (branch2 && out && !w_open), "stream_norm: no residual stream");
    TS_REQUIRE(!(stream && branch && !w_close && !(flags & TS_NORM_PLAIN_ADD)),
               "stream_norm: a branch needs the weight of its closing norm");
    TS_REQUIRE(!((w_open || (flags & TS_NORM_COPY_OUT)) && !out), "stream_norm: an opening norm, or a copy of the stream, needs an output");
    TS_REQUIRE(!(ids && (!table || branch)), "stream_norm: token ids need the table and exclude a branch");
    TS_REQUIRE(!(pos_freq && (!ids || !positions)), "stream_norm: a position vector needs token ids and positions");
    TS_REQUIRE(!(w_start && !ids), "stream_norm: a norm on the embedding needs token ids");
    TS_REQUIRE(width <= 48 * 1024, "stream_norm: rows of %d elements are not supported", width);
    if (count == 0) return 0;
    // few rows (decoding) are bound by the chain of loads, not by their number: about four elements a thread and pass;
    // many rows keep more CTAs on an SM instead
    const int wide = width >= 4096 ? 1024 : width >= 2048 ? 512 : width >= 1024 ? 256 : 128;
    const int threads = count <= 512 ? wide : (width >= 1024 ? 256 : 128);
    const size_t smem = (size_t)(width + 64) * sizeof(float);
    const BranchPair pair{branch2, w_branch, w_branch2, branch_scale, branch_scale2};
    const PairTable pairs{pair_table, prev_tokens, cu_q, seq_of_token, buckets, mul_prev, mul_cur};
    const int write = rows ? 0 : 1;
    const int vec = dtype == TS_F32 ? 4 : 8;
    const uintptr_t all = (uintptr_t)branch | (uintptr_t)branch2 | (uintptr_t)stream | (uintptr_t)w_open | (uintptr_t)out;
    if (branch && (flags & TS_NORM_PLAIN_ADD) && !w_branch && w_open && width % vec == 0 && width / vec <= 256 * STREAM_ITEMS &&
        all % 16 == 0 && (dtype == TS_F32 || dtype == TS_BF16)) {
        const int centered = flags & TS_NORM_CENTERED;
        if (dtype == TS_F32) launch_stream_add_norm<float>(branch, branch2, branch_scale, branch_scale2, stream, w_open, out, rows, count, width, eps, write, centered, stream_handle);
        else launch_stream_add_norm<__nv_bfloat16>(branch, branch2, branch_scale, branch_scale2, stream, w_open, out, rows, count, width, eps, write, centered, stream_handle);
        TS_LAUNCH_CHECK("stream_norm (add)");
        return 0;
    }
#define TS_STREAM_NORM(TYPE)                                                                                      \
    do {                                                                                                          \
        if (smem > 48 * 1024)                                                                                     \
            cudaFuncSetAttribute(stream_norm_kernel<TYPE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        stream_norm_kernel<TYPE><<<count, threads, smem, stream_handle>>>(                                        \
            (const TYPE*)branch, w_close, stream, w_open, (TYPE*)out, rows, width, eps, (const TYPE*)table, ids,  \
            table_rows, scale, write, flags, positions, pos_freq, w_start, pair, pairs);                                       \
    } while (0)
    if (dtype == TS_F32) TS_STREAM_NORM(float);
    else if (dtype == TS_BF16) TS_STREAM_NORM(__nv_bfloat16);
    else return ts_fail("stream_norm: unknown dtype code %d", dtype);
#undef TS_STREAM_NORM
    TS_LAUNCH_CHECK("stream_norm");
    return 0;
}
