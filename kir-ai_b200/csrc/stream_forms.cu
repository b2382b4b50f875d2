// A residual stream kept as several copies, read and rewritten around every sub-layer.
//
// The stream of a token is `copies` rows x_1 .. x_s of `width` 32-bit values, laid out [T, s, width].  A sub-layer's norm
// reads u = sum_f in[f] x_f, and when the sub-layer has produced y every copy is made afresh from all the old ones:
// x_t <- sum_f mix[f, t] x_f + out[t] y.  Between two sub-layers both steps and the norm are one pass over the token's
// rows: the update of the sub-layer before, the reading of the one that follows, and its RMS norm.  At the start all
// copies equal the embedding's row: the source's stride between copies is then 0 and nothing has been written yet.  With
// row_index only those rows are produced and no copy is written (the rows ahead of the logits, in = ones: the copies'
// sum).  Everything is 32-bit but the normed rows, which leave in the runtime dtype.
#include "common.cuh"

namespace {

struct StreamArgs {
    const float* src;      // token t's copy f at src + t * src_token + f * src_copy (src_copy 0: all copies equal)
    long src_token, src_copy;
    float* dst;            // [T, copies, width], may be src; null: not written
    const float* y;        // [T, width], null: no update
    const float* mix;      // [copies (from), copies (to)]
    const float* add;      // [copies]: what y is multiplied by in each copy
    const float* read;     // [copies], null: ones
    const float* weight;   // [width], null: u leaves as it is
    const int* row_index;  // null: every row
    int copies, width;
    float eps;
};

template <typename T>
__device__ __forceinline__ void store_quad(T* dst, float4 v);
template <>
__device__ __forceinline__ void store_quad<float>(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
template <>
__device__ __forceinline__ void store_quad<bf16>(bf16* dst, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 packed;
    packed.x = *reinterpret_cast<const uint32_t*>(&lo);
    packed.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(dst) = packed;
}
__device__ __forceinline__ void fma_quad(float4& acc, float a, const float4& x) {
    acc.x = fmaf(a, x.x, acc.x), acc.y = fmaf(a, x.y, acc.y), acc.z = fmaf(a, x.z, acc.z), acc.w = fmaf(a, x.w, acc.w);
}

// One block per produced row, 16-byte accesses; a thread owns the same columns of every copy, so the update in place
// needs no barrier; u stays in registers between the statistics and the output.
template <typename T, int S, int VEC>
__global__ void __launch_bounds__(VEC == 4 ? 512 : 1024) streams_norm_vec_kernel(StreamArgs a, T* __restrict__ out) {
    pdl_launch_dependents();
    __shared__ float scratch[32];
    // the coefficients are weights: read before the wait
    float mix[S][S], add[S], read[S];
#pragma unroll
    for (int t = 0; t < S; ++t) {
        read[t] = a.read ? a.read[t] : 1.0f;
        add[t] = a.y ? a.add[t] : 0.0f;
#pragma unroll
        for (int f = 0; f < S; ++f) mix[f][t] = a.y ? a.mix[f * S + t] : 0.0f;
    }
    pdl_wait();
    const size_t row = a.row_index ? (size_t)a.row_index[blockIdx.x] : (size_t)blockIdx.x;
    const float* src = a.src + row * a.src_token;
    const float* y = a.y ? a.y + row * a.width : nullptr;
    float* dst = a.dst ? a.dst + row * S * (size_t)a.width : nullptr;
    float4 u[VEC];
    float acc = 0.0f;
    // (src and dst may be the same rows: every load of a pair of pieces stands ahead of its stores)
    constexpr int AHEAD = VEC >= 2 ? 2 : 1;
#pragma unroll
    for (int n0 = 0; n0 < VEC; n0 += AHEAD) {
    float4 old[AHEAD][S], new_y[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
        const int c = (threadIdx.x + (n0 + k) * blockDim.x) * 4;
        if (c >= a.width) continue;
#pragma unroll
        for (int f = 0; f < S; ++f) old[k][f] = *reinterpret_cast<const float4*>(src + f * a.src_copy + c);
        if (y) new_y[k] = *reinterpret_cast<const float4*>(y + c);
    }
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
        const int n = n0 + k;
        const int c = (threadIdx.x + n * blockDim.x) * 4;
        u[n] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (c >= a.width) continue;
        const float4 (&x)[S] = old[k];
        if (y) {
            const float4 v = new_y[k];
#pragma unroll
            for (int t = 0; t < S; ++t) {
                float4 now = make_float4(add[t] * v.x, add[t] * v.y, add[t] * v.z, add[t] * v.w);
#pragma unroll
                for (int f = 0; f < S; ++f) fma_quad(now, mix[f][t], x[f]);
                if (dst) *reinterpret_cast<float4*>(dst + (size_t)t * a.width + c) = now;
                fma_quad(u[n], read[t], now);
            }
        } else {
#pragma unroll
            for (int f = 0; f < S; ++f) fma_quad(u[n], read[f], x[f]);
        }
        acc += (u[n].x * u[n].x + u[n].y * u[n].y) + (u[n].z * u[n].z + u[n].w * u[n].w);
    }
    }
    float scale = 1.0f;
    if (a.weight) {
        const float variance = block_sum(acc, scratch) / (float)a.width + a.eps;
        scale = variance == 0.0f ? 0.0f : 1.0f / sqrtf(variance);
    }
    if (!out) return;
    T* o = out + (size_t)blockIdx.x * a.width;
#pragma unroll
    for (int n = 0; n < VEC; ++n) {
        const int c = (threadIdx.x + n * blockDim.x) * 4;
        if (c >= a.width) continue;
        float4 v = u[n];
        if (a.weight) {
            const float4 w = *reinterpret_cast<const float4*>(a.weight + c);
            v.x *= scale * w.x, v.y *= scale * w.y, v.z *= scale * w.z, v.w *= scale * w.w;
        }
        store_quad<T>(o + c, v);
    }
}

// Any number of copies, any width and alignment: u in shared memory, a column's old copies beside it.
template <typename T>
__global__ void streams_norm_kernel(StreamArgs a, T* __restrict__ out) {
    pdl_launch_dependents();
    extern __shared__ float smem[];
    __shared__ float scratch[32];
    float* u_s = smem;                                     // [width]
    float* old_s = smem + a.width + threadIdx.x;           // [copies][threads], this thread's column of it
    const int threads = blockDim.x, S = a.copies;
    pdl_wait();
    const size_t row = a.row_index ? (size_t)a.row_index[blockIdx.x] : (size_t)blockIdx.x;
    const float* src = a.src + row * a.src_token;
    const float* y = a.y ? a.y + row * a.width : nullptr;
    float* dst = a.dst ? a.dst + row * S * (size_t)a.width : nullptr;
    float acc = 0.0f;
    for (int c = threadIdx.x; c < a.width; c += threads) {
        float u = 0.0f;
        for (int f = 0; f < S; ++f) {
            const float x = src[f * a.src_copy + c];
            if (y) old_s[f * threads] = x;
            else u = fmaf(a.read ? a.read[f] : 1.0f, x, u);
        }
        if (y) {
            const float v = y[c];
            for (int t = 0; t < S; ++t) {
                float now = a.add[t] * v;
                for (int f = 0; f < S; ++f) now = fmaf(a.mix[f * S + t], old_s[f * threads], now);
                if (dst) dst[(size_t)t * a.width + c] = now;
                u = fmaf(a.read ? a.read[t] : 1.0f, now, u);
            }
        }
        u_s[c] = u;
        acc = fmaf(u, u, acc);
    }
    float scale = 1.0f;
    if (a.weight) {
        const float variance = block_sum(acc, scratch) / (float)a.width + a.eps;
        scale = variance == 0.0f ? 0.0f : 1.0f / sqrtf(variance);
    }
    if (!out) return;
    T* o = out + (size_t)blockIdx.x * a.width;
    for (int c = threadIdx.x; c < a.width; c += threads) o[c] = from_f32<T>(a.weight ? u_s[c] * scale * a.weight[c] : u_s[c]);
}

template <typename T>
int streams_norm_launch(const StreamArgs& a, void* out, int rows, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (a.copies < 1 || a.copies > 64 || a.width <= 0 || (a.y && (!a.mix || !a.add)) || (a.dst && (!a.y || a.row_index))) return KIRAI_ERR_BAD_SIZE;
    if (sizeof(T) != 4 && !a.weight && out) return KIRAI_ERR_UNSUPPORTED;  // unnormed rows leave in 32-bit
    const bool aligned = a.width % 4 == 0 && a.src_token % 4 == 0 && a.src_copy % 4 == 0 &&
                         (((uintptr_t)a.src | (uintptr_t)a.dst | (uintptr_t)a.y | (uintptr_t)a.weight | (uintptr_t)out) & 15) == 0;
    if (aligned && a.copies <= 4 && a.width <= 4 * 4 * 512) {
        // few rows: as many threads a row as it has pieces, so that all of it is asked for at once
        const int quads = a.width / 4;
        const bool few = rows <= 148;
        const int threads = few ? (quads <= 1024 ? (quads + 31) / 32 * 32 : 1024)
                                : (a.width <= 4 * 4 * 128 ? 128 : (a.width <= 4 * 4 * 256 ? 256 : 512));
        const int vec = few ? (quads + threads - 1) / threads : 4;
#define KIRAI_STREAMS(S)                                                                                                       \
    case S:                                                                                                                   \
        if (vec == 1)                                                                                                         \
            return launch_pdl(streams_norm_vec_kernel<T, S, 1>, dim3(rows), dim3(threads), 0, stream, 1u, a, (T*)out);        \
        if (vec == 2)                                                                                                         \
            return launch_pdl(streams_norm_vec_kernel<T, S, 2>, dim3(rows), dim3(threads), 0, stream, 1u, a, (T*)out);        \
        return launch_pdl(streams_norm_vec_kernel<T, S, 4>, dim3(rows), dim3(threads), 0, stream, 1u, a, (T*)out)
        switch (a.copies) {
            KIRAI_STREAMS(1);
            KIRAI_STREAMS(2);
            KIRAI_STREAMS(3);
            KIRAI_STREAMS(4);
            default: break;
        }
#undef KIRAI_STREAMS
    }
    const int threads = a.width >= 512 ? 256 : 128;
    const size_t smem = ((size_t)a.width + (size_t)a.copies * threads) * sizeof(float);
    if (smem > 200 * 1024) return KIRAI_ERR_BAD_SIZE;
    auto kernel = streams_norm_kernel<T>;
    if (smem > 48 * 1024) {
        const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (err != cudaSuccess) return (int)err;
    }
    return launch_pdl(kernel, dim3(rows), dim3(threads), smem, stream, 1u, a, (T*)out);
}

}  // namespace

KIRAI_EXPORT int kirai_streams_norm_f32(const float* src, long src_token, long src_copy, float* dst, const float* y, const float* mix,
                                        const float* add, const float* read, const float* weight, void* out, const int* row_index,
                                        int rows, int copies, int width, float eps, cudaStream_t stream) {
    return streams_norm_launch<float>(StreamArgs{src, src_token, src_copy, dst, y, mix, add, read, weight, row_index, copies, width, eps},
                                      out, rows, stream);
}
KIRAI_EXPORT int kirai_streams_norm_bf16(const float* src, long src_token, long src_copy, float* dst, const float* y, const float* mix,
                                         const float* add, const float* read, const float* weight, void* out, const int* row_index,
                                         int rows, int copies, int width, float eps, cudaStream_t stream) {
    return streams_norm_launch<bf16>(StreamArgs{src, src_token, src_copy, dst, y, mix, add, read, weight, row_index, copies, width, eps},
                                     out, rows, stream);
}
