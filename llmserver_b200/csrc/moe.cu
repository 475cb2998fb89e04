// A routed feed-forward: router, expert products taken through an index, and the weighted sum.
//
//   route      z = W_r x (32-bit), s = sigmoid(z); the `top` experts with the largest s + correction are chosen
//              (ties: the lower index), each with the weight s * scale (the correction only chooses; nothing is
//              renormalised).  One block per token.  `select` is the same choice from logits that a matrix product
//              has already made (one warp per token).  Options of the choice (RouteRule): s = softmax(z) over all
//              experts; the weights divided by their sum (+ 1e-20); only the `keep` best of `groups` equal groups of
//              neighbouring experts can be chosen, a group's score being the largest in it.  A router may have one
//              more row behind its experts': the pre-activation of a gate on the shared expert, whose sigmoid is
//              left in `gate_out`.
//   indexed    out[p] = W[index[p]] in[p / in_div]: every (token, chosen expert) pair p multiplies its own expert's
//   linear     matrix.  One warp per output element, its sum taken over k in an order that depends on the inner size
//              alone, so a pair's result does not depend on what else the step holds.  As a gated form the matrix
//              holds gate rows then up rows and the output is the expert's activation
//                  g = min(gate, limit), u = clamp(up, -limit, limit), y = g * sigmoid(alpha * g) * (u + up_shift)
//              computed in 32-bit and rounded once (an infinite limit, alpha 1 and up_shift 0 give silu(gate) * up).
//              With `in_scale` pair p's input row is multiplied by in_scale[p] as it is read (32-bit): a routing
//              weight that acts on what goes into an expert.  An expert without a gate has the output max(sum, 0)^2 instead
//              (squared_relu).  A pair whose index names no matrix (an identity output of the router) is left out.  Read-once for steps of few tokens; prompts take the tiled
//              kernels of moe_grouped.cu.
//   combine    out[t] = sum_j weight[t, j] * down[t * top + j] (+ gate[t] * shared[t]) in 32-bit, slots in order.  A router may
//              have identity outputs behind its experts: a pair that chose one contributes the token's own row x[t].
#include "common.cuh"

#define MOE_MAX_TOP 1024

struct RouteRule {
    int experts, top;
    int softmax;          // scores: 0 sigmoid, 1 softmax over all experts
    int groups, keep;     // groups > 0: only experts of the `keep` best groups can be chosen
    int renormalise;      // the chosen weights are divided by their sum
    float scale;
};

// The choice by one warp.  On entry `score` holds the router's logits z (32-bit); `choice` is scratch of the same size.
__device__ __forceinline__ void choose_experts(float* score, float* choice, const RouteRule& rule, const float* __restrict__ correction,
                                               int* __restrict__ chosen, float* __restrict__ weights, int* __restrict__ counts) {
    const int lane = threadIdx.x & 31, experts = rule.experts;
    if (rule.softmax) {
        float best = -INFINITY;
        for (int e = lane; e < experts; e += 32) best = fmaxf(best, score[e]);
        best = warp_max(best);
        float sum = 0.0f;
        for (int e = lane; e < experts; e += 32) {
            const float s = expf(score[e] - best);
            score[e] = s;
            sum += s;
        }
        sum = warp_sum(sum);
        for (int e = lane; e < experts; e += 32) score[e] /= sum;
    } else {
        for (int e = lane; e < experts; e += 32) score[e] = 1.0f / (1.0f + expf(-score[e]));
    }
    __syncwarp();
    for (int e = lane; e < experts; e += 32) choice[e] = score[e] + (correction ? correction[e] : 0.0f);
    __syncwarp();
    if (rule.groups > 0) {
        // a lane looks after whole groups: it ranks each of them among all (ties: the lower index) and, when `keep` groups
        // are better, takes its experts out of the choice; every rank is formed before anything is taken out
        const int size = experts / rule.groups;
        if (rule.groups <= 32) {      // a lane per group: the ranks from one another's best by shuffles
            float own = -INFINITY;
            if (lane < rule.groups)
                for (int e = 0; e < size; ++e) own = fmaxf(own, choice[lane * size + e]);
            int better = 0;
            for (int other = 0; other < rule.groups; ++other) {
                const float theirs = __shfl_sync(0xffffffffu, own, other);
                better += theirs > own || (theirs == own && other < lane);
            }
            if (lane < rule.groups && better >= rule.keep)
                for (int e = 0; e < size; ++e) choice[lane * size + e] = -INFINITY;
        } else for (int first = 0; first < rule.groups; first += 32) {
            const int g = first + lane;
            bool out = false;
            if (g < rule.groups) {
                float own = -INFINITY;
                for (int e = 0; e < size; ++e) own = fmaxf(own, choice[g * size + e]);
                int better = 0;
                for (int other = 0; other < rule.groups; ++other) {
                    float theirs = -INFINITY;
                    for (int e = 0; e < size; ++e) theirs = fmaxf(theirs, score[other * size + e] + (correction ? correction[other * size + e] : 0.0f));
                    better += theirs > own || (theirs == own && other < g);
                }
                out = better >= rule.keep;
            }
            if (out)
                for (int e = 0; e < size; ++e) choice[g * size + e] = -INFINITY;
        }
        __syncwarp();
    }
    float total = 0.0f;
    for (int j = 0; j < rule.top; ++j) {
        float best = -INFINITY;
        int best_index = 0x7fffffff;
        for (int e = lane; e < experts; e += 32) {
            const float c = choice[e];
            if (c > best) {      // within a lane indices ascend, so the first of equals stays
                best = c;
                best_index = e;
            }
        }
#pragma unroll
        for (int offset = 16; offset > 0; offset >>= 1) {
            const float other = __shfl_xor_sync(0xffffffffu, best, offset);
            const int other_index = __shfl_xor_sync(0xffffffffu, best_index, offset);
            if (other > best || (other == best && other_index < best_index)) {
                best = other;
                best_index = other_index;
            }
        }
        if (best_index == 0x7fffffff) best_index = 0;      // every score was NaN or -inf: never expected
        const float s = score[best_index];
        total += s;
        if (lane == 0) {
            chosen[j] = best_index;
            if (!rule.renormalise) weights[j] = s * rule.scale;
            if (counts) atomicAdd(counts + best_index, 1);
            choice[best_index] = -INFINITY;
        }
        __syncwarp();
    }
    if (rule.renormalise) {      // lane j looks after choice j
        const float factor = rule.scale / (total + 1e-20f);
        for (int j = lane; j < rule.top; j += 32) weights[j] = score[chosen[j]] * factor;
    }
}

template <typename T>
__global__ void moe_route_kernel(const T* __restrict__ x, const float* __restrict__ router, const float* __restrict__ correction,
                                 int* __restrict__ chosen, float* __restrict__ weights, int* __restrict__ counts,
                                 int width, RouteRule rule, float* __restrict__ gate_out) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float route_shared[];      // [width] the token's row, [experts] scores, [experts] choice scores
    float* row = route_shared;
    float* score = route_shared + width;
    float* choice = score + rule.experts;
    const int token = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const T* src = x + (size_t)token * width;
    for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = Num<T>::load(src + i);
    __syncthreads();
    const int rows = rule.experts + (gate_out ? 1 : 0);
    for (int e = warp; e < rows; e += warps) {
        const float* w = router + (size_t)e * width;
        float sum = 0.0f;
        for (int i = lane; i < width; i += 32) sum = fmaf(row[i], w[i], sum);
        sum = warp_sum(sum);
        if (lane == 0) {
            if (e < rule.experts) score[e] = sum;
            else gate_out[token] = 1.0f / (1.0f + expf(-sum));
        }
    }
    __syncthreads();
    if (warp != 0) return;
    choose_experts(score, choice, rule, correction, chosen + (size_t)token * rule.top, weights + (size_t)token * rule.top, counts);
}

// The choice alone, from router logits that a matrix product has made: z float32, `stride` numbers per token, the experts'
// first and then the gate's.  One warp per token.
__global__ void moe_select_kernel(const float* __restrict__ logits, const float* __restrict__ correction, int* __restrict__ chosen,
                                  float* __restrict__ weights, int n_tokens, RouteRule rule, int stride, float* __restrict__ gate_out) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float select_shared[];      // per warp: [experts] scores, [experts] choice scores
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int token = blockIdx.x * warps + warp;
    if (token >= n_tokens) return;
    float* score = select_shared + (size_t)warp * 2 * rule.experts;
    const float* z = logits + (size_t)token * stride;
    for (int e = lane; e < rule.experts; e += 32) score[e] = z[e];
    if (gate_out && lane == 0) gate_out[token] = 1.0f / (1.0f + expf(-z[rule.experts]));
    __syncwarp();
    choose_experts(score, score + rule.experts, rule, correction, chosen + (size_t)token * rule.top, weights + (size_t)token * rule.top, nullptr);
}

__device__ __forceinline__ float gated_activation(float gate, float up, float limit, float alpha, float up_shift = 1.0f) {
    const float g = fminf(gate, limit);
    const float u = fminf(fmaxf(up, -limit), limit);
    return g / (1.0f + expf(-alpha * g)) * (u + up_shift);
}

// One warp per (pair, output element).  `rows` output elements per pair; the gated form reads row r and row rows + r.
template <typename T, typename O, bool GATED>
__global__ void indexed_linear_kernel(const T* __restrict__ in, const T* __restrict__ weight, const int* __restrict__ index,
                                      O* __restrict__ out, int rows, int inner, int in_div, float limit, float alpha, int index_mod,
                                      const float* __restrict__ in_scale, float up_shift, int squared_relu, int n_matrices) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float in_row[];       // [inner]
    if (index && (unsigned)index[blockIdx.x] >= (unsigned)n_matrices) return;
    const int pair = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const T* src = in + (size_t)(pair / in_div) * inner;
    const float row_scale = in_scale ? in_scale[pair] : 1.0f;
    for (int i = threadIdx.x; i < inner; i += blockDim.x) in_row[i] = Num<T>::load(src + i) * row_scale;
    __syncthreads();
    const int expert = index ? index[pair] : (index_mod > 0 ? pair % index_mod : 0);     // no index: pair p uses matrix p mod index_mod
    const T* matrix = weight + (size_t)expert * (GATED ? 2 : 1) * rows * inner;
    // four consecutive output elements per warp, worked on together so that their loads are in flight at the same time;
    // each element's sum runs over k in an order that depends on the inner size alone
    const int r0 = (blockIdx.y * warps + warp) * 4;
    if (r0 >= rows) return;
    float sum[4] = {0.0f, 0.0f, 0.0f, 0.0f}, sum_up[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    if (inner % 8 == 0 && aligned16(weight)) {      // 16- or 32-byte runs per lane
        for (int i = lane * 8; i < inner; i += 256) {
            float values[4][8], up_values[GATED ? 4 : 1][8];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const int r = min(r0 + q, rows - 1);      // a warp at the edge reads the last row again and drops it below
                load8<T>(matrix + (size_t)r * inner + i, values[q]);
                if (GATED) load8<T>(matrix + ((size_t)rows + r) * inner + i, up_values[q]);
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float x = in_row[i + j];
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    sum[q] = fmaf(x, values[q][j], sum[q]);
                    if (GATED) sum_up[q] = fmaf(x, up_values[q][j], sum_up[q]);
                }
            }
        }
    } else {
        for (int i = lane; i < inner; i += 32) {
            const float x = in_row[i];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const int r = min(r0 + q, rows - 1);
                sum[q] = fmaf(x, Num<T>::load(matrix + (size_t)r * inner + i), sum[q]);
                if (GATED) sum_up[q] = fmaf(x, Num<T>::load(matrix + ((size_t)rows + r) * inner + i), sum_up[q]);
            }
        }
    }
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        const float total = warp_sum(sum[q]);
        const float total_up = GATED ? warp_sum(sum_up[q]) : 0.0f;
        if (lane == 0 && r0 + q < rows) {
            float value = GATED ? gated_activation(total, total_up, limit, alpha, up_shift) : total;
            if (!GATED && squared_relu) value = fmaxf(value, 0.0f) * fmaxf(value, 0.0f);
            Num<O>::store(out + (size_t)pair * rows + r0 + q, value);
        }
    }
}

template <typename T>
__global__ void moe_combine_kernel(const float* __restrict__ down, const float* __restrict__ weights, const T* __restrict__ shared_out,
                                   const float* __restrict__ shared_gate, T* __restrict__ out, int width, int top, size_t total,
                                   const int* __restrict__ chosen, int experts, const T* __restrict__ x) {
    pdl_trigger();
    pdl_wait();
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
        const size_t token = e / width;
        const int column = (int)(e % width);
        float sum = 0.0f;
        for (int j = 0; j < top; ++j)
            sum = fmaf(weights[token * top + j], x && chosen[token * top + j] >= experts ? Num<T>::load(x + e) : down[(token * top + j) * width + column], sum);
        if (shared_out) sum = fmaf(shared_gate ? shared_gate[token] : 1.0f, Num<T>::load(shared_out + e), sum);
        Num<T>::store(out + e, sum);
    }
}

// out[n, i] = act(gate_up[n, i], gate_up[n, I + i]) for a dense gated feed-forward with the same activation.
template <typename T>
__global__ void clamped_glu_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int intermediate, size_t total,
                                   float limit, float alpha) {
    pdl_trigger();
    pdl_wait();
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
        const size_t row = e / intermediate;
        const int column = (int)(e % intermediate);
        const T* src = gate_up + row * 2 * (size_t)intermediate + column;
        Num<T>::store(out + e, gated_activation(Num<T>::load(src), Num<T>::load(src + intermediate), limit, alpha));
    }
}

// The same, eight outputs per thread with 16-byte accesses (intermediate sizes that are a multiple of 8; the hardware
// exponential and a fast division for 16-bit activations, whose rounding is far coarser than theirs).
template <typename T>
__global__ void clamped_glu_vec_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int intermediate, size_t chunks,
                                       float limit, float alpha) {
    pdl_trigger();
    pdl_wait();
    const int per_row = intermediate / 8;
    for (size_t c = (size_t)blockIdx.x * blockDim.x + threadIdx.x; c < chunks; c += (size_t)gridDim.x * blockDim.x) {
        const size_t row = c / per_row;
        const int column = (int)(c % per_row) * 8;
        const T* src = gate_up + row * 2 * (size_t)intermediate + column;
        float gate[8], up[8], result[8];
        load8<T>(src, gate);
        load8<T>(src + intermediate, up);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (sizeof(T) == 2) {
                const float g = fminf(gate[j], limit);
                const float u = fminf(fmaxf(up[j], -limit), limit);
                result[j] = __fdividef(g, 1.0f + __expf(-alpha * g)) * (u + 1.0f);
            } else {
                result[j] = gated_activation(gate[j], up[j], limit, alpha);
            }
        }
        store8<T>(out + row * (size_t)intermediate + column, result);
    }
}

static int check_rule(const char* what, const RouteRule& rule) {
    if (rule.top <= 0 || rule.top > rule.experts || rule.top > MOE_MAX_TOP) {
        llm_set_error("%s: top %d must lie in 1..min(%d experts, %d)", what, rule.top, rule.experts, MOE_MAX_TOP);
        return LLM_REFUSED;
    }
    if (rule.groups < 0 || (rule.groups > 0 && (rule.experts % rule.groups || rule.keep <= 0 || rule.keep > rule.groups ||
                                                rule.top > rule.keep * (rule.experts / rule.groups)))) {
        llm_set_error("%s: %d experts in %d groups of which %d are kept cannot give %d choices", what, rule.experts, rule.groups, rule.keep, rule.top);
        return LLM_REFUSED;
    }
    return LLM_OK;
}

LLM_EXPORT int llm_moe_route(const void* x, const float* router, const float* correction, int* chosen, float* weights,
                             int* counts, int n_tokens, int width, int experts, int top, float scale, int softmax, int groups, int keep,
                             int renormalise, float* gate_out, int dtype, cudaStream_t stream) {
    if (n_tokens == 0) return LLM_OK;
    const RouteRule rule = {experts, top, softmax, groups, keep, renormalise, scale};
    if (const int refused = check_rule("moe_route", rule)) return refused;
    const size_t shared = ((size_t)width + 2 * (size_t)experts) * sizeof(float);
    if (shared > 200 * 1024) {
        llm_set_error("moe_route: width %d and %d experts need %zu bytes of shared memory", width, experts, shared);
        return LLM_REFUSED;
    }
    LLM_DISPATCH_DTYPE(dtype, {
        if (shared > 48 * 1024) {
            const int status = llm_raise_shared_limit((const void*)moe_route_kernel<T>, shared, "moe_route");
            if (status != LLM_OK) return status;
        }
        llm_launch(moe_route_kernel<T>, n_tokens, 256, shared, stream, (const T*)x, router, correction, chosen, weights,
                   counts, width, rule, gate_out);
    });
    return llm_check_launch("moe_route");
}

LLM_EXPORT int llm_moe_select(const float* logits, const float* correction, int* chosen, float* weights, int n_tokens,
                              int experts, int top, float scale, int softmax, int groups, int keep, int renormalise, int stride,
                              float* gate_out, cudaStream_t stream) {
    if (n_tokens == 0) return LLM_OK;
    const RouteRule rule = {experts, top, softmax, groups, keep, renormalise, scale};
    if (const int refused = check_rule("moe_select", rule)) return refused;
    if (stride < experts + (gate_out ? 1 : 0)) {
        llm_set_error("moe_select: %d numbers per token for %d experts", stride, experts);
        return LLM_REFUSED;
    }
    const int warps = 4;
    const size_t shared = (size_t)warps * 2 * experts * sizeof(float);
    if (shared > 40 * 1024) {
        llm_set_error("moe_select: %d experts are too many", experts);
        return LLM_REFUSED;
    }
    llm_launch(moe_select_kernel, (n_tokens + warps - 1) / warps, warps * 32, shared, stream, logits, correction, chosen, weights,
               n_tokens, rule, stride, gate_out);
    return llm_check_launch("moe_select");
}

LLM_EXPORT int llm_indexed_linear(const void* in, const void* weight, const int* index, void* out, int n_pairs, int rows,
                                  int inner, int in_div, int gated, float limit, float alpha, int dtype, int out_f32,
                                  int index_mod, const float* in_scale, float up_shift, int squared_relu, int n_matrices,
                                  cudaStream_t stream) {
    if (n_pairs == 0 || rows == 0) return LLM_OK;
    if (index && n_matrices <= 0) {
        llm_set_error("indexed_linear: an index over %d matrices", n_matrices);
        return LLM_REFUSED;
    }
    if (in_div <= 0 || inner <= 0) {
        llm_set_error("indexed_linear: in_div %d and inner %d must be positive", in_div, inner);
        return LLM_REFUSED;
    }
    const size_t shared = (size_t)inner * sizeof(float);
    if (shared > 200 * 1024) {
        llm_set_error("indexed_linear: an inner size of %d needs %zu bytes of shared memory", inner, shared);
        return LLM_REFUSED;
    }
    const int warps = 8;
    dim3 grid(n_pairs, (rows + warps * 4 - 1) / (warps * 4));
    if (grid.y > 65535) {
        llm_set_error("indexed_linear: %d output elements per pair are too many for one launch", rows);
        return LLM_REFUSED;
    }
#define LLM_INDEXED(O, GATED)                                                                                           \
    do {                                                                                                                \
        if (shared > 48 * 1024) {                                                                                       \
            const int status = llm_raise_shared_limit((const void*)indexed_linear_kernel<T, O, GATED>, shared, "indexed_linear"); \
            if (status != LLM_OK) return status;                                                                        \
        }                                                                                                               \
        llm_launch(indexed_linear_kernel<T, O, GATED>, grid, warps * 32, shared, stream, (const T*)in, (const T*)weight, index, \
                   (O*)out, rows, inner, in_div, limit, alpha, index_mod, in_scale, up_shift, squared_relu, n_matrices);        \
    } while (0)
    LLM_DISPATCH_DTYPE(dtype, {
        if (gated && out_f32) {
            llm_set_error("indexed_linear: the gated form writes the activation type");
            return LLM_REFUSED;
        }
        if (gated) LLM_INDEXED(T, true);
        else if (out_f32) LLM_INDEXED(float, false);
        else LLM_INDEXED(T, false);
    });
#undef LLM_INDEXED
    return llm_check_launch("indexed_linear");
}

LLM_EXPORT int llm_moe_combine(const float* down, const float* weights, const void* shared_out, const float* shared_gate, void* out, int n_tokens,
                               int width, int top, const int* chosen, int experts, const void* x, int dtype, cudaStream_t stream) {
    if (n_tokens == 0) return LLM_OK;
    if (x && !chosen) {
        llm_set_error("moe_combine: identity outputs need the choices");
        return LLM_REFUSED;
    }
    const size_t total = (size_t)n_tokens * width;
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    LLM_DISPATCH_DTYPE(dtype, (llm_launch(moe_combine_kernel<T>, (unsigned)blocks, 256, 0, stream, down, weights,
                                  (const T*)shared_out, shared_gate, (T*)out, width, top, total, chosen, experts, (const T*)x)));
    return llm_check_launch("moe_combine");
}

LLM_EXPORT int llm_clamped_glu(const void* gate_up, void* out, int n_rows, int intermediate, float limit, float alpha,
                               int dtype, cudaStream_t stream) {
    if (n_rows == 0 || intermediate == 0) return LLM_OK;
    const size_t total = (size_t)n_rows * intermediate;
    if (intermediate % 8 == 0 && aligned16(gate_up) && aligned16(out)) {
        const size_t chunks = total / 8;
        size_t vec_blocks = (chunks + 255) / 256;
        if (vec_blocks > 148 * 16) vec_blocks = 148 * 16;
        LLM_DISPATCH_DTYPE(dtype, (llm_launch(clamped_glu_vec_kernel<T>, (unsigned)vec_blocks, 256, 0, stream, (const T*)gate_up,
                                      (T*)out, intermediate, chunks, limit, alpha)));
        return llm_check_launch("clamped_glu");
    }
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    LLM_DISPATCH_DTYPE(dtype, (llm_launch(clamped_glu_kernel<T>, (unsigned)blocks, 256, 0, stream, (const T*)gate_up, (T*)out,
                                  intermediate, total, limit, alpha)));
    return llm_check_launch("clamped_glu");
}
