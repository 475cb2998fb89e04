// The real-gated linear recurrent unit: a recurrence with one 32-bit number of state per channel, whose decay and input are
// gated by each token, and the gate on its output.  Per channel c (channels lie in equal units of `unit`, and a unit's
// pre-activations in z as [recurrence gates | input gates]):
//
//   r = sigmoid(z_r + b_r),  i = sigmoid(z_i + b_i)
//   log a = rate * r                                         rate = -8 softplus(lam), made once when the model is built
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u_t                    from and into the sequence's slot of `state`
//   out_t = S_t * gelu_tanh(y_t + y_bias)
//
// z is 32-bit, u and y are in the activation type, everything in between is 32-bit; 1 - a^2 is formed from log a without
// cancellation (a close to 1 is where the state is long).  A thread owns one or four neighbouring channels of a sequence and
// fetches several tokens ahead of the walk.
//
// Long portions can be walked segment by segment (a segment length given to the launcher): the local pass forms every
// token's decay and input once, leaves them where the pre-activations were, and notes per segment the product of its decays
// and the state it leaves from zero (the sequence's first segment: from the stored state, which is also put aside); the
// output pass combines the segments in front of its own, walks from there and writes the outputs, the last segment the state.
#include "common.cuh"

namespace {

constexpr int kScanThreads = 64;
constexpr int kAhead = 4;      // tokens fetched at a time

struct ScanArgs {
    float* z;                  // unit u of token t: 2 * unit numbers from t * z_token + u * z_unit on; the local pass overwrites it
    long long z_token, z_unit;
    const void* u;             // [N, width]
    const float* gate_bias;    // [2 * width]: per unit the biases of its recurrence gates, then of its input gates
    const float* rate;         // [width]
    const void* y;             // rows of y_row elements, the width channels from y_column on
    int y_row, y_column;
    const float* y_bias;       // [width]
    float* state;              // [slots, width]
    const int* state_slots;
    const int* q_start;
    void* out;                 // [N, width]
    int width, unit;
    int segment, max_segments;
    float2* summary;           // [S, max_segments, width]: (product of decays, state left)
    float* start;              // [S, width]: the stored state, put aside
};

enum : int { SCAN_ONE_PASS = 0, SCAN_LOCAL = 1, SCAN_OUTPUT = 2 };

template <typename T, int V>
__device__ __forceinline__ void load_values(const T* p, float (&v)[V]) {
    if constexpr (V == 4) {
        if constexpr (sizeof(T) == 2) {
            const uint2 raw = *reinterpret_cast<const uint2*>(p);
            const float2 low = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
            const float2 high = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
            v[0] = low.x; v[1] = low.y; v[2] = high.x; v[3] = high.y;
        } else {
            const float4 raw = *reinterpret_cast<const float4*>(p);
            v[0] = raw.x; v[1] = raw.y; v[2] = raw.z; v[3] = raw.w;
        }
    } else {
        v[0] = Num<T>::load(p);
    }
}

template <typename T, int V>
__device__ __forceinline__ void store_values(T* p, const float (&v)[V]) {
    if constexpr (V == 4) {
        if constexpr (sizeof(T) == 2) {
            const __nv_bfloat162 low = __floats2bfloat162_rn(v[0], v[1]), high = __floats2bfloat162_rn(v[2], v[3]);
            *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&low), *reinterpret_cast<const uint32_t*>(&high));
        } else {
            *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        }
    } else {
        Num<T>::store(p, v[0]);
    }
}

// Beside 16-bit activations the exponentials and divisions are the hardware's 32-bit approximations.
template <bool FAST>
__device__ __forceinline__ float sigmoid(float z) {
    return FAST ? __fdividef(1.0f, 1.0f + __expf(-z)) : 1.0f / (1.0f + expf(-z));
}

// 1 - exp(-v) for v >= 0: for small v the series v (1 - v/2 (1 - v/3 (1 - ...))), whose terms of alternating sign shrink.
template <bool FAST>
__device__ __forceinline__ float one_minus_exp(float v) {
    if (!FAST) return -expm1f(-v);
    float series = 1.0f;
#pragma unroll
    for (int k = 8; k >= 2; --k) series = fmaf(-v * (1.0f / (float)k), series, 1.0f);
    return v < 0.5f ? v * series : 1.0f - __expf(-v);
}

template <bool FAST>
__device__ __forceinline__ float gelu_tanh(float x) {
    const float twice = 1.5957691216057308f * fmaf(0.044715f * x * x, x, x);      // 2 sqrt(2 / pi) (x + 0.044715 x^3)
    return x * sigmoid<FAST>(twice);
}

template <typename T, int V, int MODE>
__global__ void __launch_bounds__(kScanThreads) gated_scan_kernel(ScanArgs a) {
    pdl_trigger();
    pdl_wait();
    constexpr bool FAST = sizeof(T) == 2;
    const int seq = blockIdx.z;
    const int c = (blockIdx.x * kScanThreads + threadIdx.x) * V;
    if (c >= a.width) return;
    int begin = a.q_start[seq], end = a.q_start[seq + 1];
    if (begin >= end) return;
    bool last = true;
    int segment = 0;
    if (MODE != SCAN_ONE_PASS) {
        segment = blockIdx.y;
        const int segments = (end - begin + a.segment - 1) / a.segment;
        if (segment >= segments) return;
        last = segment == segments - 1;
        begin += segment * a.segment;
        end = min(end, begin + a.segment);
    }
    // the channel's recurrence gate; its input gate lies `unit` further
    const int bias_column = c / a.unit * 2 * a.unit + c % a.unit;
    float* z = a.z + c / a.unit * a.z_unit + c % a.unit;
    const T* u = (const T*)a.u + c;
    const T* y = (const T*)a.y + a.y_column + c;
    T* out = (T*)a.out + c;
    float* state = a.state + (size_t)a.state_slots[seq] * a.width + c;
    float2* summary = a.summary + ((size_t)seq * a.max_segments) * a.width + c;

    float S[V], product[V], rate[V], bias_r[V], bias_i[V], y_bias[V];
    if (MODE != SCAN_OUTPUT) {
        load_values<float, V>(a.rate + c, rate);
        load_values<float, V>(a.gate_bias + bias_column, bias_r);
        load_values<float, V>(a.gate_bias + bias_column + a.unit, bias_i);
    }
    if (MODE != SCAN_LOCAL) load_values<float, V>(a.y_bias + c, y_bias);
#pragma unroll
    for (int v = 0; v < V; ++v) {
        S[v] = 0.0f;
        product[v] = 1.0f;
    }
    if (MODE == SCAN_ONE_PASS) load_values<float, V>(state, S);
    if (MODE == SCAN_LOCAL && segment == 0) {
        load_values<float, V>(state, S);
        store_values<float, V>(a.start + (size_t)seq * a.width + c, S);
    }
    if (MODE == SCAN_OUTPUT) {
        if (segment == 0) {
            load_values<float, V>(a.start + (size_t)seq * a.width + c, S);
        } else {
            constexpr int kBehind = 8;      // summaries fetched at a time; the first one already holds the stored state
            for (int k0 = 0; k0 < segment; k0 += kBehind) {
                float2 seen[kBehind][V];
#pragma unroll
                for (int k = 0; k < kBehind; ++k)
#pragma unroll
                    for (int v = 0; v < V; ++v) seen[k][v] = k0 + k < segment ? summary[(size_t)(k0 + k) * a.width + v] : make_float2(1.0f, 0.0f);
#pragma unroll
                for (int k = 0; k < kBehind; ++k)
#pragma unroll
                    for (int v = 0; v < V; ++v) S[v] = fmaf(seen[k][v].x, S[v], seen[k][v].y);
            }
        }
    }

    for (int t0 = begin; t0 < end; t0 += kAhead) {
        float zr[kAhead][V], zi[kAhead][V], us[kAhead][V], ys[kAhead][V];
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
            const size_t t = (size_t)min(t0 + k, end - 1);
            load_values<float, V>(z + t * a.z_token, zr[k]);
            load_values<float, V>(z + t * a.z_token + a.unit, zi[k]);
            if (MODE != SCAN_OUTPUT) load_values<T, V>(u + t * a.width, us[k]);
            if (MODE != SCAN_LOCAL) load_values<T, V>(y + t * a.y_row, ys[k]);
        }
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
            if (t0 + k >= end) break;
            const size_t t = (size_t)(t0 + k);
            float result[V];
#pragma unroll
            for (int v = 0; v < V; ++v) {
                float decay = zr[k][v], input = zi[k][v];
                if (MODE != SCAN_OUTPUT) {
                    const float log_a = rate[v] * sigmoid<FAST>(decay + bias_r[v]);
                    decay = FAST ? __expf(log_a) : expf(log_a);
                    input = sqrtf(one_minus_exp<FAST>(-2.0f * log_a)) * sigmoid<FAST>(input + bias_i[v]) * us[k][v];
                    zr[k][v] = decay;
                    zi[k][v] = input;
                }
                S[v] = fmaf(decay, S[v], input);
                if (MODE == SCAN_LOCAL) product[v] *= decay;
                else result[v] = S[v] * gelu_tanh<FAST>(ys[k][v] + y_bias[v]);
            }
            if (MODE == SCAN_LOCAL) {
                store_values<float, V>(z + t * a.z_token, zr[k]);
                store_values<float, V>(z + t * a.z_token + a.unit, zi[k]);
            } else {
                store_values<T, V>(out + t * a.width, result);
            }
        }
    }
    if (MODE == SCAN_LOCAL) {
#pragma unroll
        for (int v = 0; v < V; ++v) summary[(size_t)segment * a.width + v] = make_float2(product[v], S[v]);
    } else if (last) {
        store_values<float, V>(state, S);
    }
}

}  // namespace

// segment 0: one pass.  Otherwise `segments` = ceil(longest / segment), summary: float [n_seqs, segments, width, 2], start: float
// [n_seqs, width], and z is overwritten.
LLM_EXPORT int llm_gated_scan(float* z, long long z_token, long long z_unit, const void* u, const float* gate_bias, const float* rate, const void* y, int y_row, int y_column,
                              const float* y_bias, float* state, const int* state_slots, const int* q_start, void* out, int n_seqs, int width,
                              int unit, int longest, int segment, int segments, void* summary, float* start, int dtype, cudaStream_t stream) {
    if (n_seqs == 0 || longest <= 0) return LLM_OK;
    if (width <= 0 || unit <= 0 || width % unit || y_column < 0 || y_column + width > y_row) {
        llm_set_error("gated_scan: %d channels in units of %d, %d columns from column %d of rows of %d", width, unit, width, y_column, y_row);
        return LLM_REFUSED;
    }
    if (n_seqs > 65535 || segments > 65535 || (segment > 0 && (!summary || !start || (long long)segment * segments < longest))) {
        llm_set_error("gated_scan: %d sequences, %d segments of %d tokens for portions of up to %d, with scratch", n_seqs, segments, segment, longest);
        return LLM_REFUSED;
    }
    ScanArgs a;
    a.z = z; a.z_token = z_token; a.z_unit = z_unit; a.u = u; a.gate_bias = gate_bias; a.rate = rate; a.y = y; a.y_row = y_row; a.y_column = y_column; a.y_bias = y_bias;
    a.state = state; a.state_slots = state_slots; a.q_start = q_start; a.out = out; a.width = width; a.unit = unit;
    a.segment = segment; a.max_segments = segments; a.summary = (float2*)summary; a.start = start;
    const bool by_four = unit % 4 == 0 && z_token % 4 == 0 && z_unit % 4 == 0 && y_row % 4 == 0 && y_column % 4 == 0 && aligned16(z) && aligned16(u) && aligned16(gate_bias) &&
                         aligned16(rate) && aligned16(y) && aligned16(y_bias) && aligned16(state) && aligned16(out) && aligned16(start);
    const int per_block = kScanThreads * (by_four ? 4 : 1);
    const dim3 grid((width + per_block - 1) / per_block, segment > 0 ? segments : 1, n_seqs);
#define LLM_SCAN(MODE)                                                                                   \
    do {                                                                                                 \
        if (by_four) llm_launch(gated_scan_kernel<T, 4, MODE>, grid, kScanThreads, 0, stream, a);         \
        else llm_launch(gated_scan_kernel<T, 1, MODE>, grid, kScanThreads, 0, stream, a);                 \
    } while (0)
    LLM_DISPATCH_DTYPE(dtype, {
        if (segment > 0) {
            LLM_SCAN(SCAN_LOCAL);
            if (const int status = llm_check_launch("gated_scan")) return status;
            LLM_SCAN(SCAN_OUTPUT);
        } else {
            LLM_SCAN(SCAN_ONE_PASS);
        }
    });
#undef LLM_SCAN
    return llm_check_launch("gated_scan");
}
