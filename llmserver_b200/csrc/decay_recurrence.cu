// Linear attention with ONE decay per head and token and a matrix-valued state per head, kept in 32-bit per request.
// Per head, S in R^(dim x vdim):
//
//     S <- g_t S + k_t v_t^T;   o_t = S^T q_t
//
//   retention  g a constant of the head; q and k rotated by the token's position, k then scaled; followed by
//              out = o / sqrt(mean(o^2) + eps) * silu(gate)
//   ssd        g_t = exp(-exp(A) dt_t), dt_t = softplus(z_t + bias); q = C_t and k = B_t shared by a group of heads,
//              v = dt_t x_t; followed by out = (o + D x_t) * silu(gate), left in 32-bit (what is normalised next spans heads)
//
// One block per (sequence, head).  A thread owns R rows of two neighbouring columns of S in registers, as pairs of rows
// that the two-wide 32-bit instructions work on; P row partitions lie side by side in a warp's lanes, so a sum over the
// rows is R / 2 two-wide multiply-adds per column and log2(P) shuffles, with no block barrier inside the walk over tokens.
// Tokens are taken sixteen at a time: copied into shared memory while the sixteen before are worked on (two stages),
// rotated there where the layer does that, walked on the registers, then finished and stored.  The order of every sum depends on the sizes alone, so a
// token's result does not depend on how its prompt was cut or on what else is in the batch.
//
// Long portions can also be walked segment by segment in parallel (a segment length given to the launchers): pass A runs
// every segment but the last from zero and leaves L, its end state, and m, the product of its decays; a scan gives every
// segment the state it starts from, S_in(k + 1) = m_k S_in(k) + L_k; pass C runs the segments again from those states and
// writes the outputs.  All of it 32-bit; sums are then grouped by segment, so results agree with the one-pass form to
// rounding, not bit for bit (the 32-bit path keeps the one-pass form).
#include "common.cuh"
#include <type_traits>

namespace {

constexpr int kTokens = 16;       // tokens staged at a time
constexpr int kMaxThreads = 512;

struct DecayArgs {
    const void* proj;       // [N, row_width], the activation type
    int row_width, q_offset, k_offset, v_offset, g_offset;      // ssd: the gate only
    const float* pre;       // ssd: [N, pre_width]: x, B and C
    int pre_width, q_col, k_col, v_col, groups;
    const float* wide;      // ssd: [N, heads], dt before its bias
    const float* a_log;     // ssd: [heads]
    const float* dt_bias;   // ssd: [heads]
    const float* skip;      // ssd: D [heads]
    const float* head_decay;    // retention: [heads]
    const int* positions;       // retention: [N]
    const float* inv_freq;      // retention: [rotary_dim / 2]; null: nothing rotates
    int rotary_dim;
    float k_scale, eps;
    float* state;           // [slots, heads, dim, vdim]
    const int* state_slots;
    const int* q_start;
    void* out;              // [N, heads * vdim]: the activation type; ssd: float32
    int heads, dim, vdim, partitions;
    int vec4;               // ssd: rows and columns of `pre` allow 16-byte copies
    int vec_proj;           // rows and columns of `proj` do
    int segment, max_segments;
    float* segment_state;   // [S, max_segments, heads, dim, vdim]: pass A leaves L there, the scan S_in
    float* segment_move;    // [S, max_segments, heads]: m
};

enum : int { RETENTION = 0, SSD = 1 };
enum : int { ONE_PASS = 0, LOCAL = 1, OUTPUT = 3 };

// Two 32-bit values that one instruction works on.
using Pair = unsigned long long;
__device__ __forceinline__ Pair pair_of(float low, float high) {
    Pair p;
    asm("mov.b64 %0, {%1, %2};" : "=l"(p) : "f"(low), "f"(high));
    return p;
}
__device__ __forceinline__ float2 halves(Pair p) {
    float2 f;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(p));
    return f;
}
__device__ __forceinline__ Pair mul2(Pair a, Pair b) {
    Pair d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ Pair fma2(Pair a, Pair b, Pair c) {
    Pair d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}

__device__ __forceinline__ float2 load_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load_pair(const __nv_bfloat16* p) {
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void store_pair(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float2 v) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
}

// silu; for 16-bit activations with the hardware exponential and a fast division, whose errors are far below their rounding
template <typename T>
__device__ __forceinline__ float silu(float g) {
    if (sizeof(T) == 2) return __fdividef(g, 1.0f + __expf(-g));
    return g / (1.0f + expf(-g));
}

// A token's row of `dim` values lies in P partitions of R values, four floats between them: the partitions' 16-byte reads
// fall into different banks.
template <int R>
__device__ __forceinline__ int staged(int i) {
    return i / R * (R + 4) + i % R;
}

// Copies `count` rows of `size` elements, `stride` elements apart in `src` and placed by `place(row, element)` in shared
// memory: asynchronously in 16-byte pieces where `pieces` says that rows and columns allow it, else element by element.  A
// warp takes whole rows.
template <typename E, typename Place>
__device__ __forceinline__ void copy_rows(const E* __restrict__ src, size_t stride, int count, int size, bool pieces, E* shared, Place place) {
    constexpr int per = 16 / sizeof(E);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    if (pieces) {
        for (int t = warp; t < count; t += warps)
            for (int i = lane * per; i < size; i += 32 * per) {
                const unsigned target = (unsigned)__cvta_generic_to_shared(shared + place(t, i));
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(target), "l"(src + t * stride + i) : "memory");
            }
    } else {
        for (int t = warp; t < count; t += warps)
            for (int i = lane; i < size; i += 32) shared[place(t, i)] = src[t * stride + i];
    }
}

// Shared memory (bytes), in order: two stages, the working copies of q and k (retention), the outputs, the scalars.
struct Layout {
    int padded;          // floats of a staged q or k row
    int dim_stride;      // retention: elements of a raw q or k row
    int v_stride;        // elements of a v or gate row
    int stage;           // bytes of one stage
    int work;            // where the working copies start
    int outputs;
    int scalars;
    int total;
};
template <int R>
__host__ __device__ inline Layout layout_of(int mode, int dim, int vdim, int partitions, int element) {
    Layout l;
    const int per = 16 / element;      // rows start on 16-byte boundaries in either type
    l.padded = partitions * (R + 4);
    l.dim_stride = (dim + per - 1) / per * per;
    l.v_stride = (vdim + 7) / 8 * 8;
    if (mode == SSD) l.stage = kTokens * (2 * l.padded * 4 + l.v_stride * (4 + element));
    else l.stage = kTokens * (2 * l.dim_stride + 2 * l.v_stride) * element;
    l.work = 2 * l.stage;
    l.outputs = l.work + (mode == SSD ? 0 : 2 * kTokens * l.padded * 4);
    l.scalars = l.outputs + kTokens * l.v_stride * 4;
    l.total = l.scalars + 2 * kTokens * 2 * 4;
    return l;
}

template <typename T, int R, int MODE, int PASS>
__global__ void __launch_bounds__(kMaxThreads) decay_recurrence_kernel(DecayArgs a) {
    using V = typename std::conditional<MODE == SSD, float, T>::type;      // how values are staged
    pdl_trigger();
    pdl_wait();
    extern __shared__ float4 decay_shared_raw[];
    unsigned char* shared = reinterpret_cast<unsigned char*>(decay_shared_raw);
    const int seq = blockIdx.x, head = blockIdx.y;
    int begin = a.q_start[seq], end = a.q_start[seq + 1];
    if (begin >= end) return;
    bool last_segment = true;
    size_t segment_index = 0;
    if (PASS != ONE_PASS) {
        const int segments = (end - begin + a.segment - 1) / a.segment;
        const int segment = blockIdx.z;
        if (segment >= segments) return;
        last_segment = segment == segments - 1;
        if (PASS == LOCAL && last_segment) return;      // nobody needs what a zero start leaves behind the last one
        begin += segment * a.segment;
        end = min(end, begin + a.segment);
        segment_index = ((size_t)seq * a.max_segments + segment) * a.heads + head;
    }
    const int dim = a.dim, vdim = a.vdim, P = a.partitions;
    const Layout l = layout_of<R>(MODE, dim, vdim, P, sizeof(T));
    const int padded = l.padded, v_stride = l.v_stride;
    float* work = reinterpret_cast<float*>(shared + l.work);             // retention: q, then k, [kTokens][padded] each
    float* o_s = reinterpret_cast<float*>(shared + l.outputs);           // [kTokens][v_stride]
    float* scalar_s = reinterpret_cast<float*>(shared + l.scalars);      // ssd: [2][kTokens][2]: g, dt
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int per_warp = 32 / P;                       // column pairs per warp
    const int part = lane / per_warp, column = 2 * (warp * per_warp + lane % per_warp);
    const int row0 = part * R;
    const bool owner = column < vdim, second = column + 1 < vdim;
    const T* proj = (const T*)a.proj;
    const int group = MODE == SSD ? head / (a.heads / a.groups) : 0;

    // a stage: ssd: q, k (staged rows), v, gate; retention: q, k, v, gate as projected
    auto stage_q = [&](int buffer) { return shared + buffer * l.stage; };
    auto stage_v = [&](int buffer) {
        return reinterpret_cast<V*>(stage_q(buffer) + (MODE == SSD ? 2 * kTokens * padded * 4 : 2 * kTokens * l.dim_stride * (int)sizeof(T)));
    };
    auto stage_gate = [&](int buffer) { return reinterpret_cast<T*>(stage_v(buffer) + kTokens * v_stride); };
    float z_next = 0.0f;      // ssd: this thread's token's dt before bias and softplus
    auto issue = [&](int buffer, int first) {
        const int count = min(kTokens, end - first);
        if (MODE == SSD) {
            const float* row = a.pre + (size_t)first * a.pre_width;
            float* q = reinterpret_cast<float*>(stage_q(buffer));
            auto at = [&](int t, int i) { return t * padded + staged<R>(i); };
            copy_rows<float>(row + a.k_col + group * dim, a.pre_width, count, dim, a.vec4, q + kTokens * padded, at);
            if (PASS != LOCAL) copy_rows<float>(row + a.q_col + group * dim, a.pre_width, count, dim, a.vec4, q, at);
            copy_rows<float>(row + a.v_col + head * vdim, a.pre_width, count, vdim, a.vec4, reinterpret_cast<float*>(stage_v(buffer)),
                             [&](int t, int i) { return t * v_stride + i; });
            if (threadIdx.x < count) z_next = a.wide[(size_t)(first + threadIdx.x) * a.heads + head];
        } else {
            const T* row = proj + (size_t)first * a.row_width;
            T* q = reinterpret_cast<T*>(stage_q(buffer));
            auto at = [&](int t, int i) { return t * l.dim_stride + i; };
            copy_rows<T>(row + a.k_offset + head * dim, a.row_width, count, dim, a.vec_proj, q + kTokens * l.dim_stride, at);
            if (PASS != LOCAL) copy_rows<T>(row + a.q_offset + head * dim, a.row_width, count, dim, a.vec_proj, q, at);
            copy_rows<T>(row + a.v_offset + head * vdim, a.row_width, count, vdim, a.vec_proj, reinterpret_cast<T*>(stage_v(buffer)),
                         [&](int t, int i) { return t * v_stride + i; });
        }
        if (PASS != LOCAL)
            copy_rows<T>(proj + (size_t)first * a.row_width + a.g_offset + head * vdim, a.row_width, count, vdim, a.vec_proj,
                         stage_gate(buffer), [&](int t, int i) { return t * v_stride + i; });
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    issue(0, begin);

    // what lies behind dim in a staged row stays zero
    for (int e = threadIdx.x; e < kTokens * (P * R - dim); e += blockDim.x) {
        const int at = e / (P * R - dim) * padded + staged<R>(dim + e % (P * R - dim));
        for (int buffer = 0; buffer < (MODE == SSD ? 2 : 1); ++buffer) {
            float* q = MODE == SSD ? reinterpret_cast<float*>(stage_q(buffer)) : work;
            q[at] = 0.0f;
            q[kTokens * padded + at] = 0.0f;
        }
    }
    Pair S[2][R / 2];      // [column][pair of rows]; rows behind dim hold copies of the last one, which nothing reads
    float* state = a.state + ((size_t)a.state_slots[seq] * a.heads + head) * dim * vdim;
    float* segment_state = a.segment_state + segment_index * dim * vdim;
    const bool paired = (vdim & 1) == 0;      // both columns of a thread lie 8-byte aligned
    if (PASS == LOCAL) {
#pragma unroll
        for (int i = 0; i < R / 2; ++i) S[0][i] = S[1][i] = 0ull;
    } else {
        const float* source = (PASS == OUTPUT ? segment_state : state) + (owner ? column : 0);
        if (paired) {
#pragma unroll
            for (int i = 0; i < R; i += 2) {
                const float2 upper = load_pair(source + (size_t)min(row0 + i, dim - 1) * vdim);
                const float2 lower = load_pair(source + (size_t)min(row0 + i + 1, dim - 1) * vdim);
                S[0][i / 2] = pair_of(upper.x, lower.x);
                S[1][i / 2] = pair_of(upper.y, lower.y);
            }
        } else {
            const int next = second ? 1 : 0;
#pragma unroll
            for (int i = 0; i < R; i += 2) {
                const float* upper = source + (size_t)min(row0 + i, dim - 1) * vdim;
                const float* lower = source + (size_t)min(row0 + i + 1, dim - 1) * vdim;
                S[0][i / 2] = pair_of(upper[0], lower[0]);
                S[1][i / 2] = pair_of(upper[next], lower[next]);
            }
        }
    }
    float move = 1.0f;      // pass A: the product of the segment's decays
    const float head_decay = MODE == RETENTION ? a.head_decay[head] : 0.0f;
    const float decay_rate = MODE == SSD ? expf(a.a_log[head]) : 0.0f, dt_bias = MODE == SSD ? a.dt_bias[head] : 0.0f;
    const float skip = MODE == SSD ? a.skip[head] : 0.0f;

    const int position0 = MODE == RETENTION ? a.positions[begin] : 0;      // a sequence's tokens of a step lie one behind the other
    int buffer = 0;
    for (int first = begin; first < end; first += kTokens, buffer ^= 1) {
        const int count = min(kTokens, end - first);
        if (MODE == SSD && threadIdx.x < count) {
            const float z = z_next + dt_bias;
            const float dt = z > 20.0f ? z : log1pf(expf(z));
            scalar_s[(buffer * kTokens + threadIdx.x) * 2] = expf(-decay_rate * dt);
            scalar_s[(buffer * kTokens + threadIdx.x) * 2 + 1] = dt;
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();      // this stage is here; the other one, the outputs and the working copies have been read
        if (first + kTokens < end) issue(buffer ^ 1, first + kTokens);
        const V* v_s = stage_v(buffer);
        const float* q_s = MODE == SSD ? reinterpret_cast<const float*>(stage_q(buffer)) : work;
        const float* k_s = q_s + kTokens * padded;
        if (MODE == RETENTION) {      // q and k into 32-bit, rotated (element i turns with element i + half), k scaled
            const T* q_raw = reinterpret_cast<const T*>(stage_q(buffer));
            const T* k_raw = q_raw + kTokens * l.dim_stride;
            const int half = a.inv_freq ? a.rotary_dim >> 1 : 0;
            for (int t = warp; t < count; t += warps) {
                const T *q_row = q_raw + t * l.dim_stride, *k_row = k_raw + t * l.dim_stride;
                float *q_to = work + t * padded, *k_to = q_to + kTokens * padded;
                const float position = (float)(position0 + first + t - begin);
                for (int i = lane; i < half; i += 32) {
                    float s, c;
                    sincosf(position * a.inv_freq[i], &s, &c);
                    const int at = staged<R>(i), at2 = staged<R>(i + half);
                    const float ku = Num<T>::load(k_row + i), kv = Num<T>::load(k_row + i + half);
                    k_to[at] = (ku * c - kv * s) * a.k_scale;
                    k_to[at2] = (kv * c + ku * s) * a.k_scale;
                    if (PASS != LOCAL) {
                        const float qu = Num<T>::load(q_row + i), qv = Num<T>::load(q_row + i + half);
                        q_to[at] = qu * c - qv * s;
                        q_to[at2] = qv * c + qu * s;
                    }
                }
                for (int i = 2 * half + lane; i < dim; i += 32) {
                    k_to[staged<R>(i)] = Num<T>::load(k_row + i) * a.k_scale;
                    if (PASS != LOCAL) q_to[staged<R>(i)] = Num<T>::load(q_row + i);
                }
            }
            __syncthreads();
        }
        // ---- walk the tokens on the registers
        for (int t = 0; t < count; ++t) {
            float g = head_decay;
            float2 v = make_float2(0.0f, 0.0f);
            if (owner) v = load_pair(v_s + t * v_stride + column);      // an odd size's last pair reads into the row's padding
            if (!second) v.y = 0.0f;
            if (MODE == SSD) {
                const float2 scalars = load_pair(scalar_s + (buffer * kTokens + t) * 2);
                g = scalars.x;
                v.x *= scalars.y;
                v.y *= scalars.y;
            }
            const Pair gg = pair_of(g, g), v0 = pair_of(v.x, v.x), v1 = pair_of(v.y, v.y);
            const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(k_s + t * padded + part * (R + 4));
            const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(q_s + t * padded + part * (R + 4));
            if (PASS == LOCAL) {
#pragma unroll
                for (int i = 0; i < R / 4; ++i) {
                    const ulonglong2 kk = k4[i];
                    S[0][2 * i] = fma2(gg, S[0][2 * i], mul2(kk.x, v0));
                    S[1][2 * i] = fma2(gg, S[1][2 * i], mul2(kk.x, v1));
                    S[0][2 * i + 1] = fma2(gg, S[0][2 * i + 1], mul2(kk.y, v0));
                    S[1][2 * i + 1] = fma2(gg, S[1][2 * i + 1], mul2(kk.y, v1));
                }
                move *= g;
                continue;
            }
            Pair sums[4] = {0ull, 0ull, 0ull, 0ull};      // two zeros each
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const ulonglong2 kk = k4[i], qq = q4[i];
                S[0][2 * i] = fma2(gg, S[0][2 * i], mul2(kk.x, v0));
                S[1][2 * i] = fma2(gg, S[1][2 * i], mul2(kk.x, v1));
                sums[0] = fma2(S[0][2 * i], qq.x, sums[0]);
                sums[1] = fma2(S[1][2 * i], qq.x, sums[1]);
                S[0][2 * i + 1] = fma2(gg, S[0][2 * i + 1], mul2(kk.y, v0));
                S[1][2 * i + 1] = fma2(gg, S[1][2 * i + 1], mul2(kk.y, v1));
                sums[2] = fma2(S[0][2 * i + 1], qq.y, sums[2]);
                sums[3] = fma2(S[1][2 * i + 1], qq.y, sums[3]);
            }
            const float2 a0 = halves(sums[0]), a1 = halves(sums[1]), a2 = halves(sums[2]), a3 = halves(sums[3]);
            const float o0 = (a0.x + a0.y) + (a2.x + a2.y), o1 = (a1.x + a1.y) + (a3.x + a3.y);
            if (P == 1) {
                if (owner) store_pair(o_s + t * v_stride + column, make_float2(o0, o1));
            } else {
                // the partitions' parts: the first exchange leaves even partitions with column 0 and odd ones with column 1
                const bool odd = part & 1;
                float mine = odd ? o1 : o0;
                mine += __shfl_xor_sync(0xffffffffu, odd ? o0 : o1, per_warp);
                for (int offset = 2 * per_warp; offset < 32; offset <<= 1) mine += __shfl_xor_sync(0xffffffffu, mine, offset);
                if (owner && part < 2) o_s[t * v_stride + column + part] = mine;
            }
        }
        if (PASS == LOCAL) continue;
        __syncthreads();
        // ---- finish and store: a warp per token, a lane two neighbouring elements
        const T* gate_s = stage_gate(buffer);
        for (int t = warp; t < count; t += warps) {
            const size_t base = ((size_t)(first + t) * a.heads + head) * vdim;
            float inverse = 1.0f;
            if (MODE == RETENTION) {
                float squares = 0.0f;
                for (int j = lane; j < vdim; j += 32) squares = fmaf(o_s[t * v_stride + j], o_s[t * v_stride + j], squares);
                inverse = rsqrtf(warp_sum(squares) / (float)vdim + a.eps);
            }
            for (int j = 2 * lane; j < vdim; j += 64) {
                const float2 o = load_pair(o_s + t * v_stride + j), gate = load_pair(gate_s + t * v_stride + j);
                float2 y;
                if (MODE == SSD) {
                    const float2 x = load_pair(v_s + t * v_stride + j);
                    y = make_float2(fmaf(skip, x.x, o.x) * silu<T>(gate.x), fmaf(skip, x.y, o.y) * silu<T>(gate.y));
                    float* dst = (float*)a.out + base + j;
                    if (paired) store_pair(dst, y);
                    else {
                        dst[0] = y.x;
                        if (j + 1 < vdim) dst[1] = y.y;
                    }
                } else {
                    y = make_float2(o.x * inverse * silu<T>(gate.x), o.y * inverse * silu<T>(gate.y));
                    T* dst = (T*)a.out + base + j;
                    if (paired) store_pair(dst, y);
                    else {
                        Num<T>::store(dst, y.x);
                        if (j + 1 < vdim) Num<T>::store(dst + 1, y.y);
                    }
                }
            }
        }
    }
    if (PASS != LOCAL && !last_segment) return;
    if (owner) {
        float* target = (PASS == LOCAL ? segment_state : state) + column;
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const float2 c0 = halves(S[0][i / 2]), c1 = halves(S[1][i / 2]);
            const float2 value = i & 1 ? make_float2(c0.y, c1.y) : make_float2(c0.x, c1.x);
            if (row0 + i < dim) {
                float* dst = target + (size_t)(row0 + i) * vdim;
                if (paired) store_pair(dst, value);
                else {
                    dst[0] = value.x;
                    if (second) dst[1] = value.y;
                }
            }
        }
    }
    if (PASS == LOCAL && threadIdx.x == 0) a.segment_move[segment_index] = move;
}

// The scan between the passes, per (sequence, head): S_in(0) is the slot's state and S_in(k + 1) = m_k S_in(k) + L_k;
// S_in(k) takes L_k's place in the scratch.  The cells are independent: a thread takes VEC of them and loads the segments'
// values some ahead of the chain of multiply-adds that needs them.
template <int VEC>
__global__ void __launch_bounds__(128) decay_scan_kernel(DecayArgs a) {
    pdl_trigger();
    pdl_wait();
    const int seq = blockIdx.x, head = blockIdx.y;
    const int tokens = a.q_start[seq + 1] - a.q_start[seq];
    if (tokens <= 0) return;
    const int segments = (tokens + a.segment - 1) / a.segment;
    const int cells = a.dim * a.vdim;
    const int cell = (blockIdx.z * blockDim.x + threadIdx.x) * VEC;
    if (cell >= cells) return;
    const float* state = a.state + ((size_t)a.state_slots[seq] * a.heads + head) * cells + cell;
    const size_t first = ((size_t)seq * a.max_segments) * a.heads + head;
    constexpr int AHEAD = 8;
    float S[VEC];
    if constexpr (VEC == 4) Vec16<float>::load(state, S);
    else S[0] = state[0];
    for (int k0 = 0; k0 < segments; k0 += AHEAD) {
        float local[AHEAD][VEC], move[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int k = min(k0 + u, segments - 1);      // behind the last one nothing is used
            const size_t index = first + (size_t)k * a.heads;
            if constexpr (VEC == 4) Vec16<float>::load(a.segment_state + index * cells + cell, local[u]);
            else local[u][0] = a.segment_state[index * cells + cell];
            move[u] = a.segment_move[index];
        }
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int k = k0 + u;
            if (k < segments) {
                float* target = a.segment_state + (first + (size_t)k * a.heads) * cells + cell;
                if constexpr (VEC == 4) Vec16<float>::store(target, S);
                else target[0] = S[0];
                if (k + 1 < segments) {
#pragma unroll
                    for (int j = 0; j < VEC; ++j) S[j] = fmaf(move[u], S[j], local[u][j]);
                }
            }
        }
    }
}

// Rows per thread, partitions and threads for heads of `dim` x `vdim`; 0: no arrangement.
int arrangement(int dim, int vdim, int* partitions, int* threads) {
    const int rows = dim <= 16 ? 16 : 32;
    int parts = 1;
    while (parts * rows < dim) parts *= 2;
    if (parts > 32) return 0;
    const int per_warp = 32 / parts, pairs = (vdim + 1) / 2;
    *partitions = parts;
    *threads = (pairs + per_warp - 1) / per_warp * 32;
    return *threads <= kMaxThreads ? rows : 0;
}

constexpr int kSharedLimit = 200 * 1024;
int shared_bytes(int rows, int mode, int dim, int vdim, int partitions, int element) {
    return rows == 16 ? layout_of<16>(mode, dim, vdim, partitions, element).total : layout_of<32>(mode, dim, vdim, partitions, element).total;
}

int launch(DecayArgs& a, int mode, int n_seqs, int dtype, cudaStream_t stream) {
    if (n_seqs == 0) return LLM_OK;
    const bool segmented = a.segment > 0;
    if (segmented && (a.max_segments <= 0 || !a.segment_state || !a.segment_move)) {
        llm_set_error("decay recurrence: the segmented form needs its scratch");
        return LLM_REFUSED;
    }
    int threads = 0;
    const int rows = a.heads > 0 && a.dim > 0 && a.vdim > 0 ? arrangement(a.dim, a.vdim, &a.partitions, &threads) : 0;
    const int element = dtype == LLM_BF16 ? 2 : 4;
    const size_t shared = rows == 0 ? 0 : (size_t)shared_bytes(rows, mode, a.dim, a.vdim, a.partitions, element);
    const int per = 16 / element;
    a.vec_proj = a.row_width % per == 0 && a.g_offset % per == 0 && a.vdim % per == 0 && aligned16(a.proj) &&
                 (mode == SSD || (a.q_offset % per == 0 && a.k_offset % per == 0 && a.v_offset % per == 0 && a.dim % per == 0));
    if (!rows || shared > kSharedLimit) {
        llm_set_error("decay recurrence: %d heads of %d key and %d value channels are not supported", a.heads, a.dim, a.vdim);
        return LLM_REFUSED;
    }
#define DECAY_PASS(R, MODE, PASS, GRID)                                                                                       \
    do {                                                                                                                      \
        if (shared > 40 * 1024) {                                                                                             \
            const int status = llm_raise_shared_limit((const void*)decay_recurrence_kernel<T, R, MODE, PASS>, shared, "decay recurrence"); \
            if (status != LLM_OK) return status;                                                                              \
        }                                                                                                                     \
        llm_launch(decay_recurrence_kernel<T, R, MODE, PASS>, GRID, threads, shared, stream, a);                              \
    } while (0)
#define DECAY_MODE(R, MODE)                                                                                                   \
    do {                                                                                                                      \
        if (!segmented) {                                                                                                     \
            DECAY_PASS(R, MODE, ONE_PASS, dim3(n_seqs, a.heads));                                                             \
        } else {                                                                                                              \
            DECAY_PASS(R, MODE, LOCAL, dim3(n_seqs, a.heads, a.max_segments));                                                \
            const int cells = a.dim * a.vdim;                                                                                 \
            if (cells % 4 == 0) llm_launch(decay_scan_kernel<4>, dim3(n_seqs, a.heads, (cells / 4 + 127) / 128), 128, 0, stream, a); \
            else llm_launch(decay_scan_kernel<1>, dim3(n_seqs, a.heads, (cells + 127) / 128), 128, 0, stream, a);             \
            DECAY_PASS(R, MODE, OUTPUT, dim3(n_seqs, a.heads, a.max_segments));                                               \
        }                                                                                                                     \
    } while (0)
    LLM_DISPATCH_DTYPE(dtype, {
        if (mode == RETENTION) {
            if (rows == 16) DECAY_MODE(16, RETENTION);
            else DECAY_MODE(32, RETENTION);
        } else {
            if (rows == 16) DECAY_MODE(16, SSD);
            else DECAY_MODE(32, SSD);
        }
    });
#undef DECAY_MODE
#undef DECAY_PASS
    return llm_check_launch("decay recurrence");
}

}  // namespace

// Threads per block for heads of `dim` x `vdim` (0: not supported, in either type or form); the caller sizes its segments
// by it.
LLM_EXPORT int llm_decay_recurrence_threads(int dim, int vdim) {
    int partitions, threads;
    const int rows = dim > 0 && vdim > 0 ? arrangement(dim, vdim, &partitions, &threads) : 0;
    if (!rows) return 0;
    for (int mode = RETENTION; mode <= SSD; ++mode)
        if (shared_bytes(rows, mode, dim, vdim, partitions, 4) > kSharedLimit) return 0;
    return threads;
}

LLM_EXPORT int llm_retention_recurrent(const void* proj, int row_width, int q_offset, int k_offset, int v_offset, int g_offset,
                                       const float* head_decay, const int* positions, const float* inv_freq, int rotary_dim,
                                       float k_scale, float* state, const int* state_slots, const int* q_start, void* out, int n_seqs,
                                       int heads, int dim, int vdim, float eps, int dtype, int segment, int max_segments,
                                       float* segment_state, float* segment_move, cudaStream_t stream) {
    if (inv_freq && (rotary_dim < 0 || rotary_dim % 2 || rotary_dim > dim)) {
        llm_set_error("retention_recurrent: %d rotating elements must be an even number of at most %d", rotary_dim, dim);
        return LLM_REFUSED;
    }
    DecayArgs a = {};
    a.segment = segment; a.max_segments = max_segments; a.segment_state = segment_state; a.segment_move = segment_move;
    a.proj = proj; a.row_width = row_width; a.q_offset = q_offset; a.k_offset = k_offset; a.v_offset = v_offset; a.g_offset = g_offset;
    a.head_decay = head_decay; a.positions = positions; a.inv_freq = inv_freq; a.rotary_dim = rotary_dim; a.k_scale = k_scale;
    a.state = state; a.state_slots = state_slots; a.q_start = q_start; a.out = out; a.heads = heads; a.dim = dim; a.vdim = vdim;
    a.eps = eps; a.groups = 1;
    return launch(a, RETENTION, n_seqs, dtype, stream);
}

LLM_EXPORT int llm_ssd_recurrent(const void* proj, int row_width, int g_offset, const float* pre, int pre_width, int v_col, int k_col,
                                 int q_col, const float* wide, const float* a_log, const float* dt_bias, const float* skip,
                                 float* state, const int* state_slots, const int* q_start, float* out, int n_seqs, int heads,
                                 int groups, int dim, int vdim, int dtype, int segment, int max_segments, float* segment_state,
                                 float* segment_move, cudaStream_t stream) {
    if (groups <= 0 || heads % groups) {
        llm_set_error("ssd_recurrent: %d heads are no multiple of %d groups", heads, groups);
        return LLM_REFUSED;
    }
    DecayArgs a = {};
    a.segment = segment; a.max_segments = max_segments; a.segment_state = segment_state; a.segment_move = segment_move;
    a.proj = proj; a.row_width = row_width; a.g_offset = g_offset; a.pre = pre; a.pre_width = pre_width; a.v_col = v_col;
    a.k_col = k_col; a.q_col = q_col; a.groups = groups; a.wide = wide; a.a_log = a_log; a.dt_bias = dt_bias; a.skip = skip;
    a.state = state; a.state_slots = state_slots; a.q_start = q_start; a.out = out; a.heads = heads; a.dim = dim; a.vdim = vdim;
    a.vec4 = dim % 4 == 0 && vdim % 4 == 0 && pre_width % 4 == 0 && v_col % 4 == 0 && k_col % 4 == 0 && q_col % 4 == 0 && aligned16(pre);
    return launch(a, SSD, n_seqs, dtype, stream);
}
