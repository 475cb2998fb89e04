// Token embedding: residual[n, :] = table[ids[n], :], widened to the 32-bit residual stream.
// The reference does a plain row lookup with no scaling (utils/model.py:56-59,110); `scale` multiplies the row for
// models that scale their embedding (1 elsewhere).
//
// With `frequencies` ([(hidden + 1) / 2] pairs of floats whose sum is the frequency) a sinusoidal position vector joins the
// row: element 2i gets sin(p f_i), element 2i + 1 cos(p f_i) at position p.  Far positions turn many times, so the angle is
// kept as two floats: a = fl(p * high), what that product's rounding left over (one fused multiply-add) and p * low are
// the small rest e, and sin(a + e) = sin a cos e + cos a sin e.
//
// `copies` > 1: the row is written that many times, one behind the other (models that carry several streams per token).
#include "common.cuh"

__device__ __forceinline__ void position_wave(float position, float2 frequency, float& sine, float& cosine) {
    const float angle = position * frequency.x;
    const float rest = fmaf(position, frequency.x, -angle) + position * frequency.y;
    float s, c;
    sincosf(angle, &s, &c);
    const float square = rest * rest;      // the first terms of the rest's own sine and cosine
    const float turn = fmaf(-rest * square, 1.0f / 6.0f, rest), shrink = square * fmaf(square, 1.0f / 24.0f, -0.5f);
    sine = s + fmaf(turn, c, shrink * s);
    cosine = c + fmaf(-turn, s, shrink * c);
}

template <typename T>
__global__ void embedding_gather_kernel(float* __restrict__ out, const T* __restrict__ table,
                                        const int* __restrict__ ids, int hidden, int vocab, int vector_form, float scale,
                                        int copies, const int* __restrict__ positions, const float2* __restrict__ frequencies) {
    pdl_trigger();   // let the next kernel start launching
    pdl_wait();      // everything before this kernel in the stream is complete and visible
    const int token = blockIdx.x;
    int id = ids[token];
    // ids are validated on the host; clamp so that a bad id can never read outside the table
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    const T* row = table + (size_t)id * hidden;
    float* dst = out + (size_t)token * copies * hidden;
    const float position = frequencies ? (float)positions[token] : 0.0f;
    if (vector_form) {
        for (int i = threadIdx.x * 8; i < hidden; i += blockDim.x * 8) {
            float values[8];
            load8<T>(row + i, values);
#pragma unroll
            for (int j = 0; j < 8; ++j) values[j] *= scale;
            if (frequencies) {
#pragma unroll
                for (int j = 0; j < 8; j += 2) {
                    float sine, cosine;
                    position_wave(position, frequencies[(i + j) / 2], sine, cosine);
                    values[j] += sine;
                    values[j + 1] += cosine;
                }
            }
            for (int copy = 0; copy < copies; ++copy) store8<float>(dst + (size_t)copy * hidden + i, values);
        }
    } else {
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            float value = Num<T>::load(row + i) * scale;
            if (frequencies) {
                float sine, cosine;
                position_wave(position, frequencies[i / 2], sine, cosine);
                value += i % 2 ? cosine : sine;
            }
            for (int copy = 0; copy < copies; ++copy) dst[(size_t)copy * hidden + i] = value;
        }
    }
}

LLM_EXPORT int llm_embedding_gather(float* out, const void* table, const int* ids, int n_tokens, int hidden,
                                    int vocab, int dtype, float scale, int copies, const int* positions, const void* frequencies,
                                    cudaStream_t stream) {
    if (n_tokens == 0) return LLM_OK;
    if (copies < 1 || (frequencies && !positions)) {
        llm_set_error("embedding_gather: %d copies of a row, and frequencies come with positions", copies);
        return LLM_REFUSED;
    }
    const int vector_form = hidden % 8 == 0 && aligned16(out) && aligned16(table);
    int threads = vector_form ? (hidden / 8 + 31) / 32 * 32 : (hidden >= 1024 ? 256 : 128);
    if (threads > 512) threads = 512;
    LLM_DISPATCH_DTYPE(dtype, (llm_launch(embedding_gather_kernel<T>, n_tokens, threads, 0, stream, 
                                  out, (const T*)table, ids, hidden, vocab, vector_form, scale, copies, positions, (const float2*)frequencies)));
    return llm_check_launch("embedding_gather");
}
