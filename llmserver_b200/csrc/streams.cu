// Several residual streams per token (the scheme of Zhu et al., "Hyper-Connections"): what a sub-layer's boundary does, in one
// pass over the streams.  The streams are 32-bit [N, S, width].
//
//   pending sub-layer   y      = sum over parts p of scale_p * norm_p(part_p + bias_p)      norm_p: RMS norm with a weight, or nothing
//                       x_t   <- sum_s mix[s][t] x_s + out[t] * y                            all streams at once from the old ones
//   next sub-layer      u      = sum_t read[t] x_t
//                       result = norm(u) * weight                                            layer norm (the mean taken off) or RMS norm
//
// Either half may be absent: without parts the streams are only read, without a result they are only brought up to date.
// Absent coefficients mean 1 on every stream (`out`, `read`) and the identity (`mix`).  With `rows` output row o comes from
// token rows[o] and the streams are left as they were (a final norm on the rows that are wanted).  S = 1 with absent
// coefficients is the ordinary residual add followed by a norm.
//
// Everything is 32-bit, the result is rounded once.  One block per row; the order of every sum depends on the width and on
// S alone.  Two forms: up to four streams and widths in eights hold a row in registers; any other sizes stage the old
// streams in shared memory.
#include "common.cuh"

namespace {

constexpr int kVec = 8;
constexpr int kMaxParts = 2;
constexpr int kMaxStreams = 32;

struct StreamsArgs {
    float* x;
    int streams, width;
    const void* part[kMaxParts];        // [N, width] in the activation type, or null
    const float* part_bias[kMaxParts];  // [width] or null
    const void* part_weight[kMaxParts]; // [width]: the part passes an RMS norm with this weight; or null
    float part_eps[kMaxParts], part_scale[kMaxParts];
    const float* mix;                   // [S, S], indexed [from, to], or null
    const float* out_w;                 // [S] or null
    const float* read_w;                // [S] or null
    const void* weight;                 // [width]
    float eps;
    int centre;                         // the mean is taken off (layer norm)
    void* result;                       // [rows, width] or null
    const int* rows;
    int write_streams;
};

// Sums of two values over the block; every thread gets both.  Every call has a scratch of its own (32 pairs), so that one
// barrier is enough.
__device__ __forceinline__ float2 block_sum2(float2 v, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
    v.x = warp_sum(v.x);
    v.y = warp_sum(v.y);
    if (warps == 1) return v;
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float2 mine = lane < warps ? scratch[lane] : make_float2(0.0f, 0.0f);
    mine.x = warp_sum(mine.x);
    mine.y = warp_sum(mine.y);
    return mine;
}

template <typename T, typename W, int S, int CHUNKS>
__global__ void __launch_bounds__(512) streams_vec_kernel(StreamsArgs a) {
    pdl_trigger();
    pdl_wait();
    __shared__ float2 scratch[3][32];
    const int o = blockIdx.x;
    const size_t row = a.rows ? (size_t)a.rows[o] : (size_t)o;
    const int width = a.width, chunks = width / kVec;
    float* x = a.x + row * S * width;
    const bool pending = a.part[0] != nullptr;

    float value[kMaxParts][CHUNKS][kVec];      // the parts, then (in [0]) what is normalised
    float old[CHUNKS][S][kVec];
    float2 squares = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < CHUNKS; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < chunks) {
#pragma unroll
            for (int s = 0; s < S; ++s) load8<float>(x + (size_t)s * width + c * kVec, old[i][s]);
#pragma unroll
            for (int p = 0; p < kMaxParts; ++p) {
                if (!a.part[p]) continue;
                load8<T>((const T*)a.part[p] + row * width + c * kVec, value[p][i]);
                if (a.part_bias[p]) {
                    float bias[kVec];
                    load8<float>(a.part_bias[p] + c * kVec, bias);
#pragma unroll
                    for (int j = 0; j < kVec; ++j) value[p][i][j] += bias[j];
                }
                float& sum = p == 0 ? squares.x : squares.y;
#pragma unroll
                for (int j = 0; j < kVec; ++j) sum = fmaf(value[p][i][j], value[p][i][j], sum);
            }
        }
    }
    if (a.part_weight[0] || a.part_weight[1]) squares = block_sum2(squares, scratch[0]);
    float factor[kMaxParts];
#pragma unroll
    for (int p = 0; p < kMaxParts; ++p)
        factor[p] = a.part_scale[p] * (a.part_weight[p] ? rsqrtf((p == 0 ? squares.x : squares.y) / (float)width + a.part_eps[p]) : 1.0f);

    float2 total = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < CHUNKS; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < chunks) {
            float y[kVec] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int p = 0; p < kMaxParts; ++p) {
                if (!a.part[p]) continue;
                if (a.part_weight[p]) {
                    float weight[kVec];
                    load8<W>((const W*)a.part_weight[p] + c * kVec, weight);
#pragma unroll
                    for (int j = 0; j < kVec; ++j) y[j] = fmaf(value[p][i][j] * factor[p], weight[j], y[j]);
                } else {
#pragma unroll
                    for (int j = 0; j < kVec; ++j) y[j] = fmaf(value[p][i][j], factor[p], y[j]);
                }
            }
            float u[kVec] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int t = 0; t < S; ++t) {
                float now[kVec];
                if (pending) {
                    const float out_w = a.out_w ? a.out_w[t] : 1.0f;
#pragma unroll
                    for (int j = 0; j < kVec; ++j) now[j] = out_w * y[j];
#pragma unroll
                    for (int s = 0; s < S; ++s) {
                        const float mix = a.mix ? a.mix[s * S + t] : (s == t ? 1.0f : 0.0f);
#pragma unroll
                        for (int j = 0; j < kVec; ++j) now[j] = fmaf(mix, old[i][s][j], now[j]);
                    }
                    if (a.write_streams) store8<float>(x + (size_t)t * width + c * kVec, now);
                } else {
#pragma unroll
                    for (int j = 0; j < kVec; ++j) now[j] = old[i][t][j];
                }
                const float read = a.read_w ? a.read_w[t] : 1.0f;
#pragma unroll
                for (int j = 0; j < kVec; ++j) u[j] = fmaf(read, now[j], u[j]);
            }
#pragma unroll
            for (int j = 0; j < kVec; ++j) {
                value[0][i][j] = u[j];
                total.x += u[j];
                total.y = fmaf(u[j], u[j], total.y);
            }
        }
    }
    if (!a.result) return;
    total = block_sum2(total, scratch[1]);
    float mean = 0.0f, square_sum = total.y;
    if (a.centre) {      // the squared deviations are summed around the mean itself
        mean = total.x / (float)width;
        float2 deviations = make_float2(0.0f, 0.0f);
#pragma unroll
        for (int i = 0; i < CHUNKS; ++i) {
            const int c = threadIdx.x + i * blockDim.x;
            if (c < chunks) {
#pragma unroll
                for (int j = 0; j < kVec; ++j) {
                    value[0][i][j] -= mean;
                    deviations.x = fmaf(value[0][i][j], value[0][i][j], deviations.x);
                }
            }
        }
        square_sum = block_sum2(deviations, scratch[2]).x;
    }
    const float inverse = rsqrtf(square_sum / (float)width + a.eps);
    T* dst = (T*)a.result + (size_t)o * width;
#pragma unroll
    for (int i = 0; i < CHUNKS; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < chunks) {
            float weight[kVec];
            load8<W>((const W*)a.weight + c * kVec, weight);
#pragma unroll
            for (int j = 0; j < kVec; ++j) weight[j] = value[0][i][j] * inverse * weight[j];
            store8<T>(dst + c * kVec, weight);
        }
    }
}

// Any number of streams and any width: a thread's elements of the old streams wait in shared memory ([S][width]) and their
// new reading behind them ([width]).
template <typename T, typename W>
__global__ void streams_kernel(StreamsArgs a) {
    pdl_trigger();
    pdl_wait();
    __shared__ float2 scratch[3][32];
    extern __shared__ float staged[];
    const int o = blockIdx.x, S = a.streams, width = a.width;
    const size_t row = a.rows ? (size_t)a.rows[o] : (size_t)o;
    float* x = a.x + row * S * width;
    float* u_row = staged + (size_t)S * width;
    const bool pending = a.part[0] != nullptr;
    float2 squares = make_float2(0.0f, 0.0f);
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        for (int s = 0; s < S; ++s) staged[(size_t)s * width + c] = x[(size_t)s * width + c];
        for (int p = 0; p < kMaxParts; ++p) {
            if (!a.part[p]) continue;
            const float v = Num<T>::load((const T*)a.part[p] + row * width + c) + (a.part_bias[p] ? a.part_bias[p][c] : 0.0f);
            float& sum = p == 0 ? squares.x : squares.y;
            sum = fmaf(v, v, sum);
        }
    }
    if (a.part_weight[0] || a.part_weight[1]) squares = block_sum2(squares, scratch[0]);
    float factor[kMaxParts];
    for (int p = 0; p < kMaxParts; ++p)
        factor[p] = a.part_scale[p] * (a.part_weight[p] ? rsqrtf((p == 0 ? squares.x : squares.y) / (float)width + a.part_eps[p]) : 1.0f);
    float2 total = make_float2(0.0f, 0.0f);
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        float y = 0.0f;
        for (int p = 0; p < kMaxParts; ++p) {
            if (!a.part[p]) continue;
            const float v = Num<T>::load((const T*)a.part[p] + row * width + c) + (a.part_bias[p] ? a.part_bias[p][c] : 0.0f);
            y = fmaf(v * factor[p], a.part_weight[p] ? Num<W>::load((const W*)a.part_weight[p] + c) : 1.0f, y);
        }
        float u = 0.0f;
        for (int t = 0; t < S; ++t) {
            float now = staged[(size_t)t * width + c];
            if (pending) {
                now = (a.out_w ? a.out_w[t] : 1.0f) * y;
                for (int s = 0; s < S; ++s) now = fmaf(a.mix ? a.mix[s * S + t] : (s == t ? 1.0f : 0.0f), staged[(size_t)s * width + c], now);
                if (a.write_streams) x[(size_t)t * width + c] = now;
            }
            u = fmaf(a.read_w ? a.read_w[t] : 1.0f, now, u);
        }
        u_row[c] = u;
        total.x += u;
        total.y = fmaf(u, u, total.y);
    }
    if (!a.result) return;
    total = block_sum2(total, scratch[1]);
    float mean = 0.0f, square_sum = total.y;
    if (a.centre) {
        mean = total.x / (float)width;
        float2 deviations = make_float2(0.0f, 0.0f);
        for (int c = threadIdx.x; c < width; c += blockDim.x) {
            const float d = u_row[c] - mean;
            deviations.x = fmaf(d, d, deviations.x);
        }
        square_sum = block_sum2(deviations, scratch[2]).x;
    }
    const float inverse = rsqrtf(square_sum / (float)width + a.eps);
    T* dst = (T*)a.result + (size_t)o * width;
    for (int c = threadIdx.x; c < width; c += blockDim.x)
        Num<T>::store(dst + c, (u_row[c] - mean) * inverse * Num<W>::load((const W*)a.weight + c));
}

}  // namespace

// part_a / part_b: [N, width] in the activation type (b may be null; both null: nothing is pending); their biases (32-bit) and
// RMS norm weights may each be null.  mix [S, S], out_w [S], read_w [S]: 32-bit, may be null.  result null: the streams are
// only brought up to date.  `dtype`: the activation type; `weight_dtype`: of all norm weights.
LLM_EXPORT int llm_streams_norm(float* x, int streams, int width, const void* part_a, const float* bias_a, const void* weight_a, float eps_a,
                                float scale_a, const void* part_b, const float* bias_b, const void* weight_b, float eps_b, float scale_b,
                                const float* mix, const float* out_w, const float* read_w, const void* weight, float eps, int centre,
                                void* result, const int* rows, int n_rows, int dtype, int weight_dtype, cudaStream_t stream) {
    if (n_rows == 0) return LLM_OK;
    if (streams < 1 || streams > kMaxStreams || width <= 0) {
        llm_set_error("streams_norm: %d streams (1 to %d) of %d elements are not supported", streams, kMaxStreams, width);
        return LLM_REFUSED;
    }
    if ((part_b && !part_a) || (result && !weight) || (!part_a && !result)) {
        llm_set_error("streams_norm: a second part needs a first, a result the norm's weight, and there must be something to do");
        return LLM_REFUSED;
    }
    StreamsArgs a;
    a.x = x; a.streams = streams; a.width = width;
    a.part[0] = part_a; a.part_bias[0] = bias_a; a.part_weight[0] = part_a ? weight_a : nullptr; a.part_eps[0] = eps_a; a.part_scale[0] = scale_a;
    a.part[1] = part_b; a.part_bias[1] = bias_b; a.part_weight[1] = part_b ? weight_b : nullptr; a.part_eps[1] = eps_b; a.part_scale[1] = scale_b;
    a.mix = mix; a.out_w = out_w; a.read_w = read_w;
    a.weight = weight; a.eps = eps; a.centre = centre; a.result = result; a.rows = rows;
    a.write_streams = rows == nullptr;
    const int chunks = width / kVec;
    const bool vector_form = streams <= 4 && width % kVec == 0 && chunks <= 512 * 4 && aligned16(x) && aligned16(part_a) && aligned16(bias_a) &&
                             aligned16(weight_a) && aligned16(part_b) && aligned16(bias_b) && aligned16(weight_b) && aligned16(weight) && aligned16(result);
    if (vector_form) {
        int threads = (chunks + 31) / 32 * 32;      // depends on the width only
        const bool one = threads <= 512;
        if (!one) threads = 512;
#define LLM_STREAMS(S)                                                                                               \
    do {                                                                                                             \
        if (one) llm_launch(streams_vec_kernel<T, W, S, 1>, n_rows, threads, 0, stream, a);                           \
        else llm_launch(streams_vec_kernel<T, W, S, 4>, n_rows, threads, 0, stream, a);                               \
    } while (0)
        LLM_DISPATCH_DTYPE_WEIGHT(dtype, weight_dtype, {
            if (streams == 1) LLM_STREAMS(1);
            else if (streams == 2) LLM_STREAMS(2);
            else if (streams == 3) LLM_STREAMS(3);
            else LLM_STREAMS(4);
        });
#undef LLM_STREAMS
        return llm_check_launch("streams_norm");
    }
    const size_t shared = (size_t)(streams + 1) * width * sizeof(float);
    if (shared > 200 * 1024) {
        llm_set_error("streams_norm: %d streams of %d elements need %zu bytes of shared memory", streams, width, shared);
        return LLM_REFUSED;
    }
    const int threads = width >= 1024 ? 512 : (width >= 256 ? 256 : 64);
    LLM_DISPATCH_DTYPE_WEIGHT(dtype, weight_dtype, {
        if (shared > 40 * 1024) {
            const int status = llm_raise_shared_limit((const void*)streams_kernel<T, W>, shared + 1024, "streams_norm");
            if (status != LLM_OK) return status;
        }
        llm_launch(streams_kernel<T, W>, n_rows, threads, shared, stream, a);
    });
    return llm_check_launch("streams_norm");
}
