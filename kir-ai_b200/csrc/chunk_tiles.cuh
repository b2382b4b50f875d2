// What the kernels that take a matrix state's tokens a chunk at a time share: the chunk's size, copies of rows into tiles
// of shared memory that nobody waits for, and where a step's chunks lie.
#pragma once
#include "common.cuh"

namespace {

constexpr int CHUNK = 64;         // tokens a chunk
constexpr int PITCH = CHUNK + 4;  // floats a row of the tiles that keep a chunk's tokens along a row
constexpr int THREADS = 256;      // 16 x 16 threads, 4 x 4 entries each

__host__ __device__ inline int cols_pitch(int cols) { return (cols + 15) / 16 * 16; }

// A 4-byte copy from global to shared memory that the thread does not wait for (any address, any stride).
__device__ __forceinline__ void copy_async(float* to, const float* from) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(to)), "l"(from) : "memory");
}
__device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// `len` rows of `d` columns from `from` (row stride `stride`) into a tile that keeps tokens along a row, [d][PITCH];
// the columns of tokens that the chunk does not have are zero.
__device__ __forceinline__ void fetch_across(float* tile, const float* from, long stride, int len, int d) {
    const int lane = threadIdx.x & 31;
    for (int t = threadIdx.x >> 5; t < CHUNK; t += THREADS / 32) {  // a warp takes a token's row
        const float* row = from + t * stride;
        if (t < len)
            for (int kd = lane; kd < d; kd += 32) copy_async(tile + kd * PITCH + t, row + kd);
        else
            for (int kd = lane; kd < d; kd += 32) tile[kd * PITCH + t] = 0.0f;
    }
}

// `len` rows of `cols` columns into a tile [CHUNK][cp]; zero elsewhere.
__device__ __forceinline__ void fetch_along(float* tile, const float* from, long stride, int len, int cols, int cp) {
    const int c = threadIdx.x & 15;
    for (int t = threadIdx.x >> 4; t < CHUNK; t += THREADS / 16) {
        const float* row = from + t * stride;
        for (int at = c; at < cp; at += 16) {
            if (t < len && at < cols) copy_async(tile + t * cp + at, row + at);
            else tile[t * cp + at] = 0.0f;
        }
    }
}

// The step's chunks are numbered request by request; a block finds its request by a walk over the row boundaries.
struct ChunkPlace {
    int request, chunk, chunks, len;
    long row0;
};

__device__ __forceinline__ bool find_chunk(const int* __restrict__ query_start, int requests, int at, ChunkPlace& place) {
    for (int r = 0; r < requests; ++r) {
        const int first = query_start[r], count = query_start[r + 1] - first;
        const int chunks = (count + CHUNK - 1) / CHUNK;
        if (at < chunks) {
            place.request = r, place.chunk = at, place.chunks = chunks;
            place.len = min(CHUNK, count - at * CHUNK);
            place.row0 = (long)first + (long)at * CHUNK;
            return true;
        }
        at -= chunks;
    }
    return false;
}

// The number of the first chunk of request `request`.
__device__ __forceinline__ int first_chunk(const int* __restrict__ query_start, int request) {
    int before = 0;
    for (int r = 0; r < request; ++r) before += (query_start[r + 1] - query_start[r] + CHUNK - 1) / CHUNK;
    return before;
}

template <typename Kernel>
int grant_shared(Kernel kernel, long bytes, long* granted) {
    if (bytes <= *granted) return 0;
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess) return launch_status();
    *granted = bytes;
    return 0;
}

#define KIRAI_BY_RUNS(runs, name) ((runs) == 1 ? name<1> : (runs) == 2 ? name<2> : (runs) == 3 ? name<3> : name<4>)

}  // namespace
