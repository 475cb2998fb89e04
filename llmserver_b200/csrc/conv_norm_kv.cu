// From a packed q | k | v projection to attention's inputs, for layers that convolve over time and normalise whole
// projections:
//
//   1. y_t[c] = sum_j w[c][j] * x_(t - taps + 1 + j)[c]     a causal convolution per channel of q, k and v, zeros before the
//                                                           sequence's start, the last taps - 1 projected rows of every
//                                                           sequence carried in its state slot (absent: y = x)
//   2. q <- y_q / sqrt(mean(y_q^2) + eps) * q_weight        one root mean square over all of a token's query channels, one
//      k <- y_k / sqrt(mean(y_k^2) + eps) * k_weight        over all of its key channels (absent: as convolved)
//   3. q to `q_out` [N, Hq * D]; k and v to the token's slot of the pages [page, Hkv, slot, D | Dv].
//
// Sums, statistics and products are 32-bit and every element is rounded once, when it is stored.  A block takes `chunk`
// tokens of one sequence, one after the other: all of a token's channels, in vectors of eight where the sizes allow.
// Only a sequence's first block (whose chunk is no shorter than the history) reads the stored rows; it renews them
// behind its tokens.  The order of every sum depends on the sizes alone.  Convolutions of two to four taps over vectors
// of eight run a form that keeps the inputs of a vector in registers from token to token.
#include "common.cuh"

struct ConvNormArgs {
    const void* x;           // [N, row_width]: q | k | v
    int row_width;
    const float* taps_w;     // [taps, channels]
    int taps;
    float* state;            // [slots, max(taps - 1, 1), channels], oldest first (null with one tap)
    const int* state_slots;
    const int* q_start;
    const int* positions;
    const int* block_tables;
    int max_blocks;
    const void* q_weight;    // [q_channels] or null
    const void* k_weight;    // [k_channels] or null
    float eps;
    void* q_out;
    void* k_pages;
    void* v_pages;
    int q_channels, k_channels, v_channels, n_kv_heads, key_dim, value_dim, page_size, num_pages, write_cache, chunk;
    int* error_flag;
};

template <typename T, typename W, int VEC>
__global__ void __launch_bounds__(512) conv_norm_kv_kernel(ConvNormArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float4 conv_shared_raw[];
    float* values = reinterpret_cast<float*>(conv_shared_raw);      // [channels], the token's convolved row
    __shared__ float scratch[2][17];
    const int seq = blockIdx.y;
    const int begin = a.q_start[seq], end = a.q_start[seq + 1];
    const int first = begin + blockIdx.x * a.chunk, last = min(end, first + a.chunk);
    if (first >= end) return;
    const int channels = a.q_channels + a.k_channels + a.v_channels;
    const int history = a.taps - 1;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const T* x = (const T*)a.x;
    float* state = a.state ? a.state + (size_t)a.state_slots[seq] * max(history, 1) * channels : nullptr;
    for (int t = first; t < last; ++t) {
        float squares_q = 0.0f, squares_k = 0.0f;
        for (int c = threadIdx.x * VEC; c < channels; c += blockDim.x * VEC) {
            float y[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] = 0.0f;
            for (int j = 0; j < a.taps; ++j) {
                const int source = t - history + j;      // on the step's token axis; before `begin`: the stored rows
                float v[VEC], w[VEC];
                if constexpr (VEC == 8) {
                    if (source >= begin) load8<T>(x + (size_t)source * a.row_width + c, v);
                    else load8<float>(state + (size_t)(history + source - begin) * channels + c, v);
                    if (a.taps_w) load8<float>(a.taps_w + (size_t)j * channels + c, w);
                } else {
                    v[0] = source >= begin ? Num<T>::load(x + (size_t)source * a.row_width + c)
                                           : state[(size_t)(history + source - begin) * channels + c];
                    if (a.taps_w) w[0] = a.taps_w[(size_t)j * channels + c];
                }
#pragma unroll
                for (int i = 0; i < VEC; ++i) y[i] = a.taps_w ? fmaf(w[i], v[i], y[i]) : v[i];
            }
            float sum = 0.0f;
#pragma unroll
            for (int i = 0; i < VEC; ++i) sum = fmaf(y[i], y[i], sum);
            if (c < a.q_channels) squares_q += sum;      // a vector lies in one of the three ranges
            else if (c < a.q_channels + a.k_channels) squares_k += sum;
            if constexpr (VEC == 8) store8<float>(values + c, y);
            else values[c] = y[0];
        }
        // both sums over the block
        squares_q = warp_sum(squares_q);
        squares_k = warp_sum(squares_k);
        if (lane == 0) {
            scratch[0][warp] = squares_q;
            scratch[1][warp] = squares_k;
        }
        __syncthreads();
        squares_q = lane < warps ? scratch[0][lane] : 0.0f;
        squares_k = lane < warps ? scratch[1][lane] : 0.0f;
        squares_q = warp_sum(squares_q);
        squares_k = warp_sum(squares_k);
        const float inverse_q = a.q_weight ? rsqrtf(squares_q / (float)a.q_channels + a.eps) : 1.0f;
        const float inverse_k = a.k_weight ? rsqrtf(squares_k / (float)a.k_channels + a.eps) : 1.0f;
        const int position = a.positions[t];
        bool write = a.write_cache != 0;
        int page = 0;
        if (write) {
            page = a.block_tables[(size_t)seq * a.max_blocks + position / a.page_size];
            if (page < 0 || page >= a.num_pages) {
                if (threadIdx.x == 0) atomicExch(a.error_flag, 1 + t);   // the host turns this into an exception
                write = false;
            }
        }
        const size_t slot0 = (size_t)page * a.n_kv_heads * a.page_size + position % a.page_size;      // head 0's slot; heads lie page_size apart
        for (int c = threadIdx.x * VEC; c < channels; c += blockDim.x * VEC) {
            float y[VEC], w[VEC];
            if constexpr (VEC == 8) load8<float>(values + c, y);
            else y[0] = values[c];
            T* dst;
            if (c < a.q_channels) {
                dst = (T*)a.q_out + (size_t)t * a.q_channels + c;
                if (a.q_weight) {
                    if constexpr (VEC == 8) load8<W>((const W*)a.q_weight + c, w);
                    else w[0] = Num<W>::load((const W*)a.q_weight + c);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) y[i] = y[i] * inverse_q * w[i];
                }
            } else if (c < a.q_channels + a.k_channels) {
                if (!write) continue;
                const int k = c - a.q_channels;
                dst = (T*)a.k_pages + (slot0 + (size_t)(k / a.key_dim) * a.page_size) * a.key_dim + k % a.key_dim;
                if (a.k_weight) {
                    if constexpr (VEC == 8) load8<W>((const W*)a.k_weight + k, w);
                    else w[0] = Num<W>::load((const W*)a.k_weight + k);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) y[i] = y[i] * inverse_k * w[i];
                }
            } else {
                if (!write) continue;
                const int v = c - a.q_channels - a.k_channels;
                dst = (T*)a.v_pages + (slot0 + (size_t)(v / a.value_dim) * a.page_size) * a.value_dim + v % a.value_dim;
            }
            if constexpr (VEC == 8) store8<T>(dst, y);
            else Num<T>::store(dst, y[0]);
        }
        __syncthreads();      // the next token overwrites the scratch sums
    }
    if (blockIdx.x != 0 || history == 0) return;
    // the new stored rows: the last `history` of (old stored rows, this step's rows); a channel is one thread's, which walks
    // its rows oldest first, so a row is read before it is overwritten.  Every read above is done.
    const int length = end - begin;
    for (int c = threadIdx.x; c < channels; c += blockDim.x)
        for (int r = 0; r < history; ++r) {
            const int source = length - history + r;      // relative to `begin`
            state[(size_t)r * channels + c] = source >= 0 ? Num<T>::load(x + (size_t)(begin + source) * a.row_width + c)
                                                          : state[(size_t)(history + source) * channels + c];
        }
}

// The same for vectors of eight and a number of taps known at compile time: a thread walks a vector's tokens with the
// inputs in its registers, so each row is read once (and `TAPS` - 1 rows in front of the block's tokens); the convolved
// rows of all the block's tokens wait in shared memory for their root mean squares.
constexpr int kRollTokens = 8;
template <typename T, typename W, int TAPS>
__global__ void __launch_bounds__(512) conv_norm_kv_roll_kernel(ConvNormArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float4 conv_shared_raw[];
    float* values = reinterpret_cast<float*>(conv_shared_raw);      // [chunk][channels]
    __shared__ float scratch[2][kRollTokens][16];
    const int seq = blockIdx.y;
    const int begin = a.q_start[seq], end = a.q_start[seq + 1];
    const int first = begin + blockIdx.x * a.chunk, count = min(end - first, a.chunk);
    if (count <= 0) return;
    const int channels = a.q_channels + a.k_channels + a.v_channels;
    constexpr int history = TAPS - 1;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const T* x = (const T*)a.x;
    float* state = a.state + (size_t)a.state_slots[seq] * history * channels;
    float squares_q[kRollTokens], squares_k[kRollTokens];
#pragma unroll
    for (int t = 0; t < kRollTokens; ++t) squares_q[t] = squares_k[t] = 0.0f;
    for (int c = threadIdx.x * 8; c < channels; c += blockDim.x * 8) {
        float w[TAPS][8], v[TAPS][8];      // v[j]: the input that tap j meets; the newest is v[TAPS - 1]
#pragma unroll
        for (int j = 0; j < TAPS; ++j) load8<float>(a.taps_w + (size_t)j * channels + c, w[j]);
#pragma unroll
        for (int j = 0; j < history; ++j) {
            const int source = first - history + j;
            if (source >= begin) load8<T>(x + (size_t)source * a.row_width + c, v[j + 1]);
            else load8<float>(state + (size_t)(history + source - begin) * channels + c, v[j + 1]);
        }
        const bool is_q = c < a.q_channels, is_k = !is_q && c < a.q_channels + a.k_channels;
        constexpr int FETCH = 4;
        Raw8<T> raw[FETCH];
#pragma unroll
        for (int t = 0; t < kRollTokens; ++t) {
            if (t % FETCH == 0 && t < count) {
#pragma unroll
                for (int u = 0; u < FETCH; ++u) raw[u].fetch(x + (size_t)(first + min(t + u, count - 1)) * a.row_width + c);
            }
            if (t < count) {
#pragma unroll
                for (int j = 0; j < history; ++j)
#pragma unroll
                    for (int i = 0; i < 8; ++i) v[j][i] = v[j + 1][i];
                raw[t % FETCH].widen(v[TAPS - 1]);
                float y[8], sum = 0.0f;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    y[i] = 0.0f;
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) y[i] = fmaf(w[j][i], v[j][i], y[i]);
                    sum = fmaf(y[i], y[i], sum);
                }
                if (is_q) squares_q[t] += sum;
                if (is_k) squares_k[t] += sum;
                store8<float>(values + (size_t)t * channels + c, y);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < kRollTokens; ++t) {
        if (t < count) {
            const float q = warp_sum(squares_q[t]), k = warp_sum(squares_k[t]);
            if (lane == 0) {
                scratch[0][t][warp] = q;
                scratch[1][t][warp] = k;
            }
        }
    }
    __syncthreads();      // also: every read of the stored rows is done
    for (int t = 0; t < count; ++t) {
        const float squares_q = warp_sum(lane < warps ? scratch[0][t][lane] : 0.0f);
        const float squares_k = warp_sum(lane < warps ? scratch[1][t][lane] : 0.0f);
        const float inverse_q = a.q_weight ? rsqrtf(squares_q / (float)a.q_channels + a.eps) : 1.0f;
        const float inverse_k = a.k_weight ? rsqrtf(squares_k / (float)a.k_channels + a.eps) : 1.0f;
        const int token = first + t, position = a.positions[token];
        bool write = a.write_cache != 0;
        int page = 0;
        if (write) {
            page = a.block_tables[(size_t)seq * a.max_blocks + position / a.page_size];
            if (page < 0 || page >= a.num_pages) {
                if (threadIdx.x == 0) atomicExch(a.error_flag, 1 + token);   // the host turns this into an exception
                write = false;
            }
        }
        const size_t slot0 = (size_t)page * a.n_kv_heads * a.page_size + position % a.page_size;
        for (int c = threadIdx.x * 8; c < channels; c += blockDim.x * 8) {
            float y[8], w[8];
            load8<float>(values + (size_t)t * channels + c, y);
            if (c < a.q_channels) {
                if (a.q_weight) {
                    load8<W>((const W*)a.q_weight + c, w);
#pragma unroll
                    for (int i = 0; i < 8; ++i) y[i] = y[i] * inverse_q * w[i];
                }
                store8<T>((T*)a.q_out + (size_t)token * a.q_channels + c, y);
            } else if (c < a.q_channels + a.k_channels) {
                const int k = c - a.q_channels;
                if (a.k_weight) {
                    load8<W>((const W*)a.k_weight + k, w);
#pragma unroll
                    for (int i = 0; i < 8; ++i) y[i] = y[i] * inverse_k * w[i];
                }
                if (write) store8<T>((T*)a.k_pages + (slot0 + (size_t)(k / a.key_dim) * a.page_size) * a.key_dim + k % a.key_dim, y);
            } else if (write) {
                const int v = c - a.q_channels - a.k_channels;
                store8<T>((T*)a.v_pages + (slot0 + (size_t)(v / a.value_dim) * a.page_size) * a.value_dim + v % a.value_dim, y);
            }
        }
    }
    if (blockIdx.x != 0) return;
    // the new stored rows, as in the kernel above
    const int length = end - begin;
    for (int c = threadIdx.x; c < channels; c += blockDim.x)
        for (int r = 0; r < history; ++r) {
            const int source = length - history + r;      // relative to `begin`
            state[(size_t)r * channels + c] = source >= 0 ? Num<T>::load(x + (size_t)(begin + source) * a.row_width + c)
                                                          : state[(size_t)(history + source) * channels + c];
        }
}

LLM_EXPORT int llm_conv_norm_kv(const void* x, int row_width, const float* taps_w, int taps, float* state, const int* state_slots,
                                const int* q_start, const int* positions, const int* block_tables, int max_blocks,
                                const void* q_weight, const void* k_weight, float eps, void* q_out, void* k_pages, void* v_pages,
                                int n_seqs, int longest, int n_q_heads, int n_kv_heads, int key_dim, int value_dim, int page_size,
                                int num_pages, int write_cache, int* error_flag, int dtype, int weight_dtype, cudaStream_t stream) {
    if (n_seqs == 0 || longest <= 0) return LLM_OK;
    if (n_q_heads <= 0 || n_kv_heads <= 0 || key_dim <= 0 || value_dim <= 0 || page_size <= 0 || num_pages <= 0 || taps < 1 ||
        (taps > 1 && (!taps_w || !state)) || n_seqs > 65535) {
        llm_set_error("conv_norm_kv: sizes must be positive and a convolution of %d taps needs its weights and stored rows", taps);
        return LLM_REFUSED;
    }
    ConvNormArgs a;
    a.x = x; a.row_width = row_width; a.taps_w = taps_w; a.taps = taps; a.state = taps > 1 ? state : nullptr; a.state_slots = state_slots;
    a.q_start = q_start; a.positions = positions; a.block_tables = block_tables; a.max_blocks = max_blocks; a.q_weight = q_weight;
    a.k_weight = k_weight; a.eps = eps; a.q_out = q_out; a.k_pages = k_pages; a.v_pages = v_pages;
    a.q_channels = n_q_heads * key_dim; a.k_channels = n_kv_heads * key_dim; a.v_channels = n_kv_heads * value_dim;
    a.n_kv_heads = n_kv_heads; a.key_dim = key_dim; a.value_dim = value_dim; a.page_size = page_size; a.num_pages = num_pages;
    a.write_cache = write_cache; a.error_flag = error_flag;
    a.chunk = taps - 1 > 8 ? taps - 1 : 8;
    const int channels = a.q_channels + a.k_channels + a.v_channels;
    if (row_width < channels) {
        llm_set_error("conv_norm_kv: rows of %d columns cannot hold %d", row_width, channels);
        return LLM_REFUSED;
    }
    const size_t shared = (size_t)channels * sizeof(float);
    if (shared > 200 * 1024) {
        llm_set_error("conv_norm_kv: %d channels need %zu bytes of shared memory", channels, shared);
        return LLM_REFUSED;
    }
    const bool vec = key_dim % 8 == 0 && value_dim % 8 == 0 && row_width % 8 == 0 && aligned16(x) && aligned16(taps_w) && aligned16(state) &&
                     aligned16(q_weight) && aligned16(k_weight) && aligned16(q_out) && aligned16(k_pages) && aligned16(v_pages);
    int threads = ((vec ? channels / 8 : channels) + 31) / 32 * 32;
    if (threads > 512) threads = 512;
    if (vec && taps >= 2 && taps <= 4) {
        // as many tokens per block as leave room for two blocks on an SM; a sequence's first block must cover the history
        // (the choice depends on the sizes alone, and a token's result does not depend on it)
        int tokens = (int)((size_t)100 * 1024 / ((size_t)channels * sizeof(float)));
        if (tokens > kRollTokens) tokens = kRollTokens;
        if (tokens < taps - 1) tokens = taps - 1;
        const size_t rolled = (size_t)tokens * channels * sizeof(float);
        if (rolled <= 200 * 1024) {
            a.chunk = tokens;
            const dim3 grid((longest + tokens - 1) / tokens, n_seqs);
#define LLM_CONV_ROLL(TAPS)                                                                                                    \
    do {                                                                                                                       \
        if (rolled > 40 * 1024) {                                                                                              \
            const int status = llm_raise_shared_limit((const void*)conv_norm_kv_roll_kernel<T, W, TAPS>, rolled, "conv_norm_kv"); \
            if (status != LLM_OK) return status;                                                                               \
        }                                                                                                                      \
        llm_launch(conv_norm_kv_roll_kernel<T, W, TAPS>, grid, threads, rolled, stream, a);                                    \
    } while (0)
            LLM_DISPATCH_DTYPE_WEIGHT(dtype, weight_dtype, {
                if (taps == 2) LLM_CONV_ROLL(2);
                else if (taps == 3) LLM_CONV_ROLL(3);
                else LLM_CONV_ROLL(4);
            });
#undef LLM_CONV_ROLL
            return llm_check_launch("conv_norm_kv");
        }
    }
    const dim3 grid((longest + a.chunk - 1) / a.chunk, n_seqs);
#define LLM_CONV_NORM(VEC)                                                                                                     \
    do {                                                                                                                       \
        if (shared > 40 * 1024) {                                                                                              \
            const int status = llm_raise_shared_limit((const void*)conv_norm_kv_kernel<T, W, VEC>, shared, "conv_norm_kv");    \
            if (status != LLM_OK) return status;                                                                               \
        }                                                                                                                      \
        llm_launch(conv_norm_kv_kernel<T, W, VEC>, grid, threads, shared, stream, a);                                          \
    } while (0)
    LLM_DISPATCH_DTYPE_WEIGHT(dtype, weight_dtype, {
        if (vec) LLM_CONV_NORM(8);
        else LLM_CONV_NORM(1);
    });
#undef LLM_CONV_NORM
    return llm_check_launch("conv_norm_kv");
}
