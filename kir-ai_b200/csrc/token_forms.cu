// What a model takes from a token's id beside its plain embedding row:
//
//   * embedding_norm: the row gathered and divided by its root mean square, times a weight: the 32-bit stream and, where asked
//     for, its bfloat16 copy in one pass;
//   * token_gate: gelu_tanh(z) times the token's own row of a second table, the part of the row that belongs to one layer.
#include "common.cuh"
#include "state_math.cuh"

// One block per token, four values a thread at a time where width and alignment allow (VEC 4), else one.
template <typename T, int VEC>
__global__ void embedding_norm_kernel(const T* __restrict__ table, const int* __restrict__ ids, const float* __restrict__ weight,
                                      float* __restrict__ out, bf16* __restrict__ copy, int hidden, int vocab, float eps,
                                      int* __restrict__ error_flag) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int token = blockIdx.x;
    const int id = ids[token];
    if (id < 0 || id >= vocab) {
        if (threadIdx.x == 0) atomicExch(error_flag, KIRAI_FLAG_BAD_TOKEN);
        return;
    }
    const T* row = table + (size_t)id * hidden;
    float acc = 0.0f;
    for (int i = threadIdx.x * VEC; i < hidden; i += blockDim.x * VEC) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const float v = to_f32<T>(row[i + e]);
            acc = fmaf(v, v, acc);
        }
    }
    const float variance = block_sum(acc, scratch) / (float)hidden + eps;
    const float scale = variance == 0.0f ? 0.0f : 1.0f / sqrtf(variance);
    float* dst = out + (size_t)token * hidden;
    bf16* dst_copy = copy ? copy + (size_t)token * hidden : nullptr;
    for (int i = threadIdx.x * VEC; i < hidden; i += blockDim.x * VEC) {
        float v[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = to_f32<T>(row[i + e]) * scale * weight[i + e];
        if (VEC == 4) {
            *reinterpret_cast<float4*>(dst + i) = make_float4(v[0], v[1 % VEC], v[2 % VEC], v[3 % VEC]);
            if (dst_copy) {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1 % VEC]), hi = __floats2bfloat162_rn(v[2 % VEC], v[3 % VEC]);
                uint2 packed;
                packed.x = *reinterpret_cast<const uint32_t*>(&lo);
                packed.y = *reinterpret_cast<const uint32_t*>(&hi);
                *reinterpret_cast<uint2*>(dst_copy + i) = packed;
            }
        } else {
            dst[i] = v[0];
            if (dst_copy) dst_copy[i] = __float2bfloat16_rn(v[0]);
        }
    }
}

template <typename T>
static int embedding_norm_launch(const void* table, const int* ids, const float* weight, float* out, void* copy, int tokens, int hidden,
                                 int vocab, float eps, int* error_flag, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (hidden <= 0 || vocab <= 0) return KIRAI_ERR_BAD_SIZE;
    const int threads = hidden >= 1024 ? 256 : 128;
    if (hidden % 4 == 0 && (((uintptr_t)out | (uintptr_t)copy) & 15) == 0)
        return launch_pdl(embedding_norm_kernel<T, 4>, dim3(tokens), dim3(threads), 0, stream, 1u, (const T*)table, ids, weight, out, (bf16*)copy,
                          hidden, vocab, eps, error_flag);
    return launch_pdl(embedding_norm_kernel<T, 1>, dim3(tokens), dim3(threads), 0, stream, 1u, (const T*)table, ids, weight, out, (bf16*)copy,
                      hidden, vocab, eps, error_flag);
}

KIRAI_EXPORT int kirai_embedding_norm_f32(const void* table, const int* ids, const float* weight, float* out, void* copy, int tokens, int hidden,
                                          int vocab, float eps, int* error_flag, cudaStream_t stream) {
    return embedding_norm_launch<float>(table, ids, weight, out, copy, tokens, hidden, vocab, eps, error_flag, stream);
}
KIRAI_EXPORT int kirai_embedding_norm_bf16(const void* table, const int* ids, const float* weight, float* out, void* copy, int tokens, int hidden,
                                           int vocab, float eps, int* error_flag, cudaStream_t stream) {
    return embedding_norm_launch<bf16>(table, ids, weight, out, copy, tokens, hidden, vocab, eps, error_flag, stream);
}

// out [T, dim] = gelu_tanh(z [T, dim]) * table[id, first .. first + dim); table rows have `row` numbers.
template <typename T, int VEC>
__global__ void token_gate_kernel(const float* __restrict__ z, const T* __restrict__ table, const int* __restrict__ ids, T* __restrict__ out,
                                  long tokens, int dim, long row, long first, int vocab, int* __restrict__ error_flag) {
    pdl_launch_dependents();
    pdl_wait();
    const long total = tokens * dim / VEC;
    for (long item = blockIdx.x * (long)blockDim.x + threadIdx.x; item < total; item += (long)gridDim.x * blockDim.x) {
        const long at = item * VEC;
        const long token = at / dim;
        const int c = (int)(at - token * dim);
        const int id = ids[token];
        const bool known = id >= 0 && id < vocab;
        if (!known) atomicExch(error_flag, KIRAI_FLAG_BAD_TOKEN);
        const T* e = table + (size_t)(known ? id : 0) * row + first + c;
        T values[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) values[j] = from_f32<T>(known ? sf_gelu_tanh(z[at + j]) * to_f32<T>(e[j]) : 0.0f);
#pragma unroll
        for (int j = 0; j < VEC; ++j) out[at + j] = values[j];
    }
}

template <typename T>
static int token_gate_launch(const float* z, const void* table, const int* ids, void* out, int tokens, int dim, long row, long first, int vocab,
                             int* error_flag, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (dim <= 0 || first < 0 || first + dim > row || vocab <= 0) return KIRAI_ERR_BAD_SIZE;
    // two columns a thread where a row has enough of them, so that a block has several rows' loads in flight
    const bool pairs = dim % 2 == 0 && tokens >= 64;
    const long total = (long)tokens * dim / (pairs ? 2 : 1);
    const unsigned blocks = (unsigned)min((total + 255) / 256, (long)148 * 16);
    if (pairs)
        return launch_pdl(token_gate_kernel<T, 2>, dim3(blocks), dim3(256), 0, stream, 1u, z, (const T*)table, ids, (T*)out, (long)tokens, dim, row,
                          first, vocab, error_flag);
    return launch_pdl(token_gate_kernel<T, 1>, dim3(blocks), dim3(256), 0, stream, 1u, z, (const T*)table, ids, (T*)out, (long)tokens, dim, row, first,
                      vocab, error_flag);
}

KIRAI_EXPORT int kirai_token_gate_f32(const float* z, const void* table, const int* ids, void* out, int tokens, int dim, long row, long first,
                                      int vocab, int* error_flag, cudaStream_t stream) {
    return token_gate_launch<float>(z, table, ids, out, tokens, dim, row, first, vocab, error_flag, stream);
}
KIRAI_EXPORT int kirai_token_gate_bf16(const float* z, const void* table, const int* ids, void* out, int tokens, int dim, long row, long first,
                                       int vocab, int* error_flag, cudaStream_t stream) {
    return token_gate_launch<bf16>(z, table, ids, out, tokens, dim, row, first, vocab, error_flag, stream);
}
