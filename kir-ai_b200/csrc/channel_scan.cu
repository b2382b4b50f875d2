// Gated linear attention: a matrix state per head whose rows decay each at a rate of their own,
//
//     S_t = diag(a_t) S_(t-1) + k_t v_t^T,     o_t = S_t^T q_t,     a_t = sigmoid(z_t)^(1 / tau),  z_t = W u_t + b,
//
// u_t a short row per token (the low-rank half of the decays' projection) and W [heads d, r].  Decays, their logarithms and
// sums, the state and all products with it are 32-bit.
//
// Short runs of tokens walk (channel_walk): a block has a request's head, its threads four value columns and every n-th
// state row each; the head's norm and the silu gate behind it are taken in the same kernel.
//
// Longer runs go a chunk of 64 tokens at a time.  With g = log a and G_t the sum of g inside the chunk up to t
//
//     o_t = S_0^T (q_t e^(G_t)) + sum_(s <= t) P_ts v_s,   P_ts = sum_c q_tc k_sc e^(G_tc - G_sc),
//     S_last = diag(e^(G_last)) S_0 + sum_s (k_s e^(G_last - G_s)) v_s^T.
//
//   1. channel_prepare: block (chunk, head) makes the decays, and from q and k the three things the rest needs: q_t e^(G_t),
//      k_s e^(G_last - G_s) and P, as tiles of tokens along a row, and e^(G_last).  e^(G_t - G_s) does not split into a factor
//      of t and one of s that both stay in range, so a chunk is cut into 4 pieces of 16 tokens: with q' decayed from its
//      piece's start, k' decayed to its piece's end and M_ij the decay over the pieces between j and i, P_ts = sum q' M_ij k'
//      has no positive exponent for j < i.  Inside one piece M_ii = e^(-L_i), L_i the piece's own sum; where some channel's L_i
//      is below -40 that piece's P is summed pair by pair with e^(G_t - G_s) instead.
//   2. channel_chain: block (request, head, run of columns) goes through the request's chunks with its columns of the state in
//      shared memory; or, for runs of many chunks, three launches as for the other matrix states: every chunk's own share of
//      the state, a carry over the chunks that leaves the state at each chunk's start, and the read-outs.
#include "chunk_tiles.cuh"
#include "common.cuh"
#include "state_math.cuh"

namespace {

constexpr int PIECE = 16;  // tokens a piece
constexpr int PIECES = CHUNK / PIECE;
constexpr float PAIRWISE_BELOW = -40.0f;

struct ChannelScan {
    const float* q;  // [*, heads d] (row stride `stride`, as for k, v, low)
    const float* k;
    const float* v;    // [*, heads dv]
    const float* low;  // [*, rank]
    long stride;
    const float* up;    // [rank, heads d]: the second half of the decays' projection, transposed
    const float* bias;  // [heads d]
    float tau_inverse, q_scale;
    float* state;  // [slots, state_len], S [heads, d, dv] from column 0
    long state_len;
    const int* query_start;
    const int* slots;
    float* tiles;  // [units, heads, 2 d + 64, 64]: decayed q, decayed k, P; tokens along a row
    float* kept;   // [units, heads, d]: e^(G_last)
    float* share;  // [units, heads, d, dv]: a chunk's own share of the state, then the state at its start
    float* out;    // [*, heads dv]
    int heads, d, dv, rank, cols, requests, num_slots;
};

__device__ __forceinline__ float log_decay(float z, float tau_inverse) { return sf_log_sigmoid(z) * tau_inverse; }

// Decay of channel `c` over the pieces after `from` and before `to`: e^(sum of their L).
__device__ __forceinline__ float between(const float* __restrict__ L, int d, int c, int from, int to) {
    float sum = 0.0f;
    for (int m = from + 1; m < to; ++m) sum += L[m * d + c];
    return sum == 0.0f ? 1.0f : expf(sum);
}

__host__ __device__ inline long prepare_floats(int d, int rank) {
    const long pairs = 10L * d, low = (long)rank * CHUNK;  // the table of M, and ahead of it the short rows
    return 3L * d * PITCH + (pairs > low ? pairs : low) + (long)PIECES * d;
}

__global__ void __launch_bounds__(THREADS) channel_prepare_kernel(const ChannelScan a) {
    extern __shared__ __align__(16) float smem[];
    __shared__ int pairwise[PIECES];
    pdl_launch_dependents();
    const int head = blockIdx.y, d = a.d, tid = threadIdx.x;
    float* Q = smem;
    float* K = Q + (long)d * PITCH;
    float* G = K + (long)d * PITCH;  // g summed from a piece's start, the token's own included
    float* L = G + (long)d * PITCH;  // [PIECES][d]
    float* M = L + PIECES * d;       // [10][d], pair (i, j <= i) at i (i + 1) / 2 + j
    float* low = M;                  // [rank][CHUNK], before M is made
    ChunkPlace at;
    const bool found = find_chunk(a.query_start, a.requests, blockIdx.x, at);
    pdl_wait();
    if (!found) return;
    const long c0 = (long)head * d;
    fetch_across(Q, a.q + at.row0 * a.stride + c0, a.stride, at.len, d);
    fetch_across(K, a.k + at.row0 * a.stride + c0, a.stride, at.len, d);
    for (int i = tid; i < CHUNK * a.rank; i += THREADS) {
        const int t = i / a.rank, r = i - t * a.rank;
        low[r * CHUNK + t] = t < at.len ? a.low[(at.row0 + t) * a.stride + r] : 0.0f;
    }
    if (tid < PIECES) pairwise[tid] = 0;
    __syncthreads();
    // a thread has (channel, piece): the decays of 16 tokens and their running sum
    for (int item = tid; item < PIECES * d; item += THREADS) {
        const int piece = item / d, c = item - piece * d;
        float z[PIECE];
        const float bias = a.bias[c0 + c];
#pragma unroll
        for (int t = 0; t < PIECE; ++t) z[t] = bias;
        for (int r = 0; r < a.rank; ++r) {
            const float w = a.up[(long)r * a.heads * d + c0 + c];
            const float4* lr = reinterpret_cast<const float4*>(low + r * CHUNK + piece * PIECE);
#pragma unroll
            for (int n = 0; n < PIECE / 4; ++n) {
                const float4 x = lr[n];
                z[4 * n] = fmaf(w, x.x, z[4 * n]), z[4 * n + 1] = fmaf(w, x.y, z[4 * n + 1]);
                z[4 * n + 2] = fmaf(w, x.z, z[4 * n + 2]), z[4 * n + 3] = fmaf(w, x.w, z[4 * n + 3]);
            }
        }
        float sum = 0.0f;
#pragma unroll
        for (int t = 0; t < PIECE; ++t) {
            if (piece * PIECE + t < at.len) sum += log_decay(z[t], a.tau_inverse);
            z[t] = sum;
        }
        float4* to = reinterpret_cast<float4*>(G + (long)c * PITCH + piece * PIECE);
#pragma unroll
        for (int n = 0; n < PIECE / 4; ++n) to[n] = make_float4(z[4 * n], z[4 * n + 1], z[4 * n + 2], z[4 * n + 3]);
        L[piece * d + c] = sum;
        if (sum < PAIRWISE_BELOW) pairwise[piece] = 1;
    }
    copies_wait();
    __syncthreads();

    const int tx = tid & 15, ty = tid >> 4;
    const int i_piece = ty >> 2, j_piece = tx >> 2;
    const bool lower = tx <= ty && 4 * tx < at.len;
    float acc[4][4] = {};
    const bool by_pairs = i_piece == j_piece && pairwise[i_piece];
    if (lower && by_pairs) {
        for (int c = 0; c < d; ++c) {
            const float4 qv = *reinterpret_cast<const float4*>(Q + c * PITCH + 4 * ty), kv = *reinterpret_cast<const float4*>(K + c * PITCH + 4 * tx);
            const float4 gt = *reinterpret_cast<const float4*>(G + c * PITCH + 4 * ty), gs = *reinterpret_cast<const float4*>(G + c * PITCH + 4 * tx);
            const float qs[4] = {qv.x, qv.y, qv.z, qv.w}, ks[4] = {kv.x, kv.y, kv.z, kv.w};
            const float gts[4] = {gt.x, gt.y, gt.z, gt.w}, gss[4] = {gs.x, gs.y, gs.z, gs.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j)  // (above the diagonal the difference is positive: those are set to zero below)
                    acc[i][j] = fmaf(qs[i] * ks[j], expf(fminf(gts[i] - gss[j], 0.0f)), acc[i][j]);
        }
    }
    __syncthreads();  // the tiles' own values have been read

    for (int item = tid; item < PIECES * d; item += THREADS) {
        const int piece = item / d, c = item - piece * d;
        const float total = L[piece * d + c];
        const long at4 = ((long)c * PITCH + piece * PIECE) / 4;
#pragma unroll
        for (int n = 0; n < PIECE / 4; ++n) {
            float4 q = reinterpret_cast<float4*>(Q)[at4 + n], k = reinterpret_cast<float4*>(K)[at4 + n];
            const float4 g = reinterpret_cast<const float4*>(G)[at4 + n];
            q.x *= a.q_scale * expf(g.x), q.y *= a.q_scale * expf(g.y), q.z *= a.q_scale * expf(g.z), q.w *= a.q_scale * expf(g.w);
            k.x *= expf(total - g.x), k.y *= expf(total - g.y), k.z *= expf(total - g.z), k.w *= expf(total - g.w);
            reinterpret_cast<float4*>(Q)[at4 + n] = q;
            reinterpret_cast<float4*>(K)[at4 + n] = k;
        }
        // this piece's rows of the table of decays between pieces
        for (int j = 0; j < piece; ++j) M[(piece * (piece + 1) / 2 + j) * d + c] = between(L, d, c, j, piece);
        M[(piece * (piece + 1) / 2 + piece) * d + c] = expf(fminf(-total, -PAIRWISE_BELOW));
    }
    __syncthreads();
    if (lower && !by_pairs) {
        const float* m = M + (i_piece * (i_piece + 1) / 2 + j_piece) * d;
#pragma unroll 4
        for (int c = 0; c < d; ++c) {
            const float4 qv = *reinterpret_cast<const float4*>(Q + c * PITCH + 4 * ty), kv = *reinterpret_cast<const float4*>(K + c * PITCH + 4 * tx);
            const float f = m[c];
            const float qs[4] = {qv.x * f, qv.y * f, qv.z * f, qv.w * f}, ks[4] = {kv.x, kv.y, kv.z, kv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(qs[i], ks[j], acc[i][j]);
        }
    }
    const long unit = (long)blockIdx.x * a.heads + head;
    float* tile = a.tiles + unit * (2L * d + CHUNK) * CHUNK;
    if (lower) {
        const float scale = by_pairs ? a.q_scale : 1.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int s = 4 * tx + j;
            float p[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) p[i] = s <= 4 * ty + i ? acc[i][j] * scale : 0.0f;
            *reinterpret_cast<float4*>(tile + (2L * d + s) * CHUNK + 4 * ty) = make_float4(p[0], p[1], p[2], p[3]);
        }
    }
    // decayed from the chunk's start, and to its end
    for (int item = tid; item < d * (CHUNK / 4); item += THREADS) {
        const int c = item / (CHUNK / 4), n = item - c * (CHUNK / 4), piece = n / (PIECE / 4);
        const float ahead = between(L, d, c, -1, piece), behind = between(L, d, c, piece, PIECES);
        float4 q = *reinterpret_cast<const float4*>(Q + (long)c * PITCH + 4 * n), k = *reinterpret_cast<const float4*>(K + (long)c * PITCH + 4 * n);
        q.x *= ahead, q.y *= ahead, q.z *= ahead, q.w *= ahead;
        k.x *= behind, k.y *= behind, k.z *= behind, k.w *= behind;
        *reinterpret_cast<float4*>(tile + (long)c * CHUNK + 4 * n) = q;
        *reinterpret_cast<float4*>(tile + (long)(d + c) * CHUNK + 4 * n) = k;
    }
    for (int c = tid; c < d; c += THREADS) a.kept[unit * d + c] = between(L, d, c, -1, PIECES);
}

// ------------------------------------------------------------------------------------------------ the chunks' products
// The tiles of a block, in this order as far as its kernel has them: q [d][64], k [d][64], P [64][64] as channel_prepare left
// them, v [64][cp], the state [d][cp], e^(G_last) [d].  A thread's columns are J tx .. J tx + J - 1 of cp = 16 J.
enum Kind { CHAIN, SHARE, READ };

struct Tiles {
    float *Q, *K, *P, *V, *S, *kept;
    __device__ Tiles(float* smem, int d, int cp, Kind kind) {
        Q = smem;
        K = Q + (kind == SHARE ? 0L : (long)d * CHUNK);
        P = K + (kind == READ ? 0L : (long)d * CHUNK);
        V = P + (kind == SHARE ? 0 : CHUNK * CHUNK);
        S = V + CHUNK * cp;
        kept = S + (long)d * cp;
    }
};

__host__ __device__ inline long product_floats(int d, int cols, Kind kind) {
    const int cp = cols_pitch(cols);
    const long tile = (long)d * CHUNK, square = (long)CHUNK * CHUNK, v = (long)CHUNK * cp, state = (long)d * cp;
    return kind == CHAIN ? 2 * tile + square + v + state + d : kind == SHARE ? tile + v : tile + square + v + state;
}

__device__ __forceinline__ void copy_async16(float* to, const float* from) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(to)), "l"(from) : "memory");
}
__device__ __forceinline__ void fetch_flat(float* to, const float* from, long floats) {
    for (long i = threadIdx.x * 4L; i < floats; i += THREADS * 4L) copy_async16(to + i, from + i);
}

// `live` of `rows` rows of `cols` columns (row stride `stride`) into a tile [rows][cp], zero elsewhere; 16 bytes a copy where
// the rows allow it.
__device__ __forceinline__ void fetch_rows(float* to, int cp, const float* from, long stride, int live, int rows, int cols) {
    if (cols == cp && stride % 4 == 0 && ((uintptr_t)from & 15) == 0) {
        const int quads = cp / 4;
        for (int i = threadIdx.x; i < rows * quads; i += THREADS) {
            const int r = i / quads, c = 4 * (i - r * quads);
            if (r < live) copy_async16(to + r * cp + c, from + r * stride + c);
            else *reinterpret_cast<float4*>(to + r * cp + c) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        return;
    }
    for (int i = threadIdx.x; i < rows * cp; i += THREADS) {
        const int r = i / cp, c = i - r * cp;
        if (r < live && c < cols) copy_async(to + i, from + r * stride + c);
        else to[i] = 0.0f;
    }
}

// A thread's J neighbouring columns of a tile's row.
template <int J>
__device__ __forceinline__ void columns(const float* row, int tx, float (&x)[J]) {
    if (J == 4) {
        const float4 v = *reinterpret_cast<const float4*>(row + 4 * tx);
        x[0] = v.x, x[1 % J] = v.y, x[2 % J] = v.z, x[3 % J] = v.w;
    } else if (J == 2) {
        const float2 v = *reinterpret_cast<const float2*>(row + 2 * tx);
        x[0] = v.x, x[1 % J] = v.y;
    } else {
#pragma unroll
        for (int j = 0; j < J; ++j) x[j] = row[J * tx + j];
    }
}

// The same columns to global memory, those below `cols` only.
template <int J>
__device__ __forceinline__ void store_columns(float* row, int tx, int cols, const float (&x)[J]) {
    if (J == 4 && 4 * tx + 4 <= cols && ((uintptr_t)(row + 4 * tx) & 15) == 0) {
        *reinterpret_cast<float4*>(row + 4 * tx) = make_float4(x[0], x[1 % J], x[2 % J], x[3 % J]);
        return;
    }
#pragma unroll
    for (int j = 0; j < J; ++j)
        if (J * tx + j < cols) row[J * tx + j] = x[j];
}

// o of tokens t = 4 ty + i at the thread's columns.
template <int J>
__device__ __forceinline__ void read_out(const ChannelScan& a, const Tiles& w, int head, int col0, int cols, long row0, int len) {
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4, d = a.d;
    constexpr int cp = 16 * J;
    float o[4][J] = {};
#pragma unroll 4
    for (int c = 0; c < d; ++c) {
        const float4 qv = *reinterpret_cast<const float4*>(w.Q + c * CHUNK + 4 * ty);
        const float qs[4] = {qv.x, qv.y, qv.z, qv.w};
        float sv[J];
        columns<J>(w.S + c * cp, tx, sv);
#pragma unroll
        for (int j = 0; j < J; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) o[i][j] = fmaf(qs[i], sv[j], o[i][j]);
    }
    const int s_end = min(4 * ty + 4, len);
#pragma unroll 4
    for (int s = 0; s < s_end; ++s) {
        const float4 pv = *reinterpret_cast<const float4*>(w.P + s * CHUNK + 4 * ty);
        const float ps[4] = {pv.x, pv.y, pv.z, pv.w};
        float vv[J];
        columns<J>(w.V + s * cp, tx, vv);
#pragma unroll
        for (int j = 0; j < J; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) o[i][j] = fmaf(ps[i], vv[j], o[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        if (t < len) store_columns<J>(a.out + (row0 + t) * ((long)a.heads * a.dv) + (long)head * a.dv + col0, tx, cols, o[i]);
    }
}

// sum_s k_s v_s^T over the chunk's tokens, R state rows a thread at a time, handed row by row to `take(row, sums)`.
template <int J, int R, typename Take>
__device__ __forceinline__ void outer_products(const Tiles& w, int d, int len, Take take) {
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    constexpr int cp = 16 * J;
    for (int r0 = 0; r0 < d; r0 += 16 * R) {
        float acc[R][J] = {};
        const int c0 = r0 + R * ty;
        const int quads = (len + 3) / 4;  // (tokens behind the last hold zeros)
        for (int s4 = 0; s4 < quads; ++s4) {
            float4 kv[R];
#pragma unroll
            for (int i = 0; i < R; ++i)
                kv[i] = c0 + i < d ? *reinterpret_cast<const float4*>(w.K + (c0 + i) * CHUNK + 4 * s4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float vv[J];
                columns<J>(w.V + (4 * s4 + e) * cp, tx, vv);
#pragma unroll
                for (int i = 0; i < R; ++i) {
                    const float k = e == 0 ? kv[i].x : e == 1 ? kv[i].y : e == 2 ? kv[i].z : kv[i].w;
#pragma unroll
                    for (int j = 0; j < J; ++j) acc[i][j] = fmaf(k, vv[j], acc[i][j]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < R; ++i)
            if (c0 + i < d) take(c0 + i, acc[i]);
    }
}

// S <- diag(kept) S + sum_s k_s v_s^T in shared memory.
template <int J>
__device__ __forceinline__ void update(const Tiles& w, int d, int len) {
    const int tx = threadIdx.x & 15;
    outer_products<J, 4>(w, d, len, [&](int c, const float(&sums)[J]) {
        float* at = w.S + c * 16 * J + J * tx;
#pragma unroll
        for (int j = 0; j < J; ++j) at[j] = fmaf(w.kept[c], at[j], sums[j]);
    });
}

template <int J>
__global__ void __launch_bounds__(THREADS) channel_chain_kernel(const ChannelScan a) {
    extern __shared__ __align__(16) float smem[];
    pdl_launch_dependents();
    const int request = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * a.cols, d = a.d, tid = threadIdx.x;
    const int cols = min(a.cols, a.dv - col0);
    constexpr int cp = 16 * J;
    const Tiles w(smem, d, cp, CHAIN);
    const long first = a.query_start[request];
    const int count = (int)(a.query_start[request + 1] - first);
    const int slot = a.slots[request];
    const int before = first_chunk(a.query_start, request);
    pdl_wait();
    if (slot < 0 || slot >= a.num_slots || count <= 0) return;
    float* Sg = a.state + slot * a.state_len + (long)head * d * a.dv + col0;
    for (int i = tid; i < d * cp; i += THREADS) {
        const int c = i / cp, j = i - c * cp;
        w.S[i] = j < cols ? Sg[(long)c * a.dv + j] : 0.0f;
    }
    const long tile_floats = (2L * d + CHUNK) * CHUNK;
    const float* v_from = a.v + (long)head * a.dv + col0;
    auto tile_of = [&](int chunk) { return a.tiles + ((long)(before + chunk) * a.heads + head) * tile_floats; };
    fetch_flat(w.Q, tile_of(0), tile_floats);
    fetch_rows(w.V, cp, v_from + first * a.stride, a.stride, min(CHUNK, count), CHUNK, cols);
    for (int c0 = 0; c0 < count; c0 += CHUNK) {
        const int len = min(CHUNK, count - c0), chunk = c0 / CHUNK;
        const int next_len = min(CHUNK, count - c0 - CHUNK);  // <= 0: this chunk is the last
        for (int c = tid; c < d; c += THREADS) w.kept[c] = a.kept[((long)(before + chunk) * a.heads + head) * d + c];
        copies_wait();
        __syncthreads();
        read_out<J>(a, w, head, col0, cols, first + c0, len);
        __syncthreads();  // q, P and the state of the chunk's start have been read
        if (next_len > 0) {
            fetch_flat(w.Q, tile_of(chunk + 1), (long)d * CHUNK);
            fetch_flat(w.P, tile_of(chunk + 1) + 2L * d * CHUNK, CHUNK * CHUNK);
        }
        update<J>(w, d, len);
        __syncthreads();
        if (next_len > 0) {
            fetch_flat(w.K, tile_of(chunk + 1) + (long)d * CHUNK, (long)d * CHUNK);
            fetch_rows(w.V, cp, v_from + (first + c0 + CHUNK) * a.stride, a.stride, next_len, CHUNK, cols);
        }
    }
    for (int i = tid; i < d * cp; i += THREADS) {
        const int c = i / cp, j = i - c * cp;
        if (j < cols) Sg[(long)c * a.dv + j] = w.S[i];
    }
}

template <int J>
__global__ void __launch_bounds__(THREADS) channel_share_kernel(const ChannelScan a) {
    extern __shared__ __align__(16) float smem[];
    pdl_launch_dependents();
    const int head = blockIdx.y, col0 = blockIdx.z * a.cols, d = a.d, tx = threadIdx.x & 15;
    const int cols = min(a.cols, a.dv - col0);
    constexpr int cp = 16 * J;
    const Tiles w(smem, d, cp, SHARE);
    ChunkPlace at;
    const bool found = find_chunk(a.query_start, a.requests, blockIdx.x, at);
    pdl_wait();
    if (!found) return;
    const long unit = (long)blockIdx.x * a.heads + head;
    fetch_flat(w.K, a.tiles + unit * (2L * d + CHUNK) * CHUNK + (long)d * CHUNK, (long)d * CHUNK);
    fetch_rows(w.V, cp, a.v + (long)head * a.dv + col0 + at.row0 * a.stride, a.stride, at.len, CHUNK, cols);
    copies_wait();
    __syncthreads();
    float* U = a.share + unit * d * a.dv + col0;
    const auto keep = [&](int c, const float(&sums)[J]) { store_columns<J>(U + (long)c * a.dv, tx, cols, sums); };
    if (d > 64) outer_products<J, 8>(w, d, at.len, keep);
    else outer_products<J, 4>(w, d, at.len, keep);
}

// Block (request, head, run of 256 entries of the state): the state at every chunk's start takes the place of the chunk's own share.
__global__ void __launch_bounds__(256) channel_carry_kernel(const ChannelScan a) {
    pdl_launch_dependents();
    const int request = blockIdx.x, head = blockIdx.y;
    const long entry = blockIdx.z * 256L + threadIdx.x, cells = (long)a.d * a.dv;
    const int before = first_chunk(a.query_start, request);
    const int chunks = (a.query_start[request + 1] - a.query_start[request] + CHUNK - 1) / CHUNK;
    const int slot = a.slots[request];
    pdl_wait();
    if (slot < 0 || slot >= a.num_slots || chunks <= 0 || entry >= cells) return;
    float* mine = a.state + slot * a.state_len + (long)head * cells + entry;
    float value = *mine;
    const float* kept = a.kept + ((long)before * a.heads + head) * a.d + entry / a.dv;
    float* share = a.share + ((long)before * a.heads + head) * cells + entry;
    float ahead = *share;
    for (int c = 0; c < chunks; ++c, share += a.heads * cells, kept += (long)a.heads * a.d) {
        const float own = ahead;
        if (c + 1 < chunks) ahead = share[a.heads * cells];
        *share = value;
        value = fmaf(*kept, value, own);
    }
    *mine = value;
}

template <int J>
__global__ void __launch_bounds__(THREADS) channel_out_kernel(const ChannelScan a) {
    extern __shared__ __align__(16) float smem[];
    pdl_launch_dependents();
    const int head = blockIdx.y, col0 = blockIdx.z * a.cols, d = a.d;
    const int cols = min(a.cols, a.dv - col0);
    constexpr int cp = 16 * J;
    const Tiles w(smem, d, cp, READ);
    ChunkPlace at;
    const bool found = find_chunk(a.query_start, a.requests, blockIdx.x, at);
    const int slot = found ? a.slots[at.request] : -1;
    pdl_wait();
    if (!found || slot < 0 || slot >= a.num_slots) return;
    const long unit = (long)blockIdx.x * a.heads + head;
    const float* tile = a.tiles + unit * (2L * d + CHUNK) * CHUNK;
    fetch_flat(w.Q, tile, (long)d * CHUNK);
    fetch_flat(w.P, tile + 2L * d * CHUNK, CHUNK * CHUNK);
    fetch_rows(w.V, cp, a.v + (long)head * a.dv + col0 + at.row0 * a.stride, a.stride, at.len, CHUNK, cols);
    fetch_rows(w.S, cp, a.share + unit * d * a.dv + col0, a.dv, d, d, cols);
    copies_wait();
    __syncthreads();
    read_out<J>(a, w, head, col0, cols, at.row0, at.len);
}

// How many value columns a block takes: as many as fit shared memory, fewer (16 at least) while the grid would leave most of
// the device idle.  0 when even 16 do not fit.
int choose_cols(long groups, int d, int dv, bool side_by_side) {
    int device = 0, limit = 0, sms = 0;
    if (cudaGetDevice(&device) != cudaSuccess ||
        cudaDeviceGetAttribute(&limit, cudaDevAttrMaxSharedMemoryPerBlockOptin, device) != cudaSuccess ||
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device) != cudaSuccess)
        return 0;
    const Kind kind = side_by_side ? READ : CHAIN;
    int cols = dv < 64 ? dv : 64;
    while (cols > 16 && (product_floats(d, cols, kind) * 4 > limit || groups * ((dv + cols - 1) / cols) < sms)) cols = cols > 32 ? cols - 16 : 16;
    return product_floats(d, cols, kind) * 4 <= limit ? cols : 0;
}

// ------------------------------------------------------------------------------------------------ short runs
// Thread (phase, group of V columns) has state rows phase, phase + phases, ...; a token's partial sums over the phases meet in
// shared memory.  A single token's state rows (at most HELD a thread) are asked for ahead of the decays.
constexpr int HELD = 16;

template <int V>
struct Cols {
    float x[V];
    __device__ __forceinline__ void load(const float* p) {
        if (V == 4) {
            const float4 v = *reinterpret_cast<const float4*>(p);
            x[0] = v.x, x[1 % V] = v.y, x[2 % V] = v.z, x[3 % V] = v.w;
        } else {
            x[0] = *p;
        }
    }
    __device__ __forceinline__ void store(float* p) const {
        if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1 % V], x[2 % V], x[3 % V]);
        else *p = x[0];
    }
};

template <typename T, int V, bool HOLD, int WALK_THREADS>
__global__ void __launch_bounds__(WALK_THREADS, 512 / WALK_THREADS) channel_walk_kernel(const ChannelScan a, const float* __restrict__ gate, const float* __restrict__ norm,
                                                                   float eps, T* __restrict__ out) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float scratch[32];
    pdl_launch_dependents();
    const int request = blockIdx.x, head = blockIdx.y, d = a.d, dv = a.dv, tid = threadIdx.x;
    float* decay = smem;               // [d]
    float* qs = decay + d;             // [d]
    float* ks = qs + d;                // [d]
    float* low = ks + d;               // [rank]
    float* os = low + a.rank;          // [dv]
    float* red = os + dv + (4 - (3 * d + a.rank + dv) % 4) % 4;  // [phases][groups V]
    const int groups_all = (dv + V - 1) / V;
    const int groups = groups_all < WALK_THREADS ? groups_all : WALK_THREADS;
    const int phases = WALK_THREADS / groups;
    const int phase = tid / groups, group = tid - phase * groups;
    const long first = a.query_start[request];
    const int count = (int)(a.query_start[request + 1] - first);
    const int slot = a.slots[request];
    pdl_wait();
    if (slot < 0 || slot >= a.num_slots || count <= 0) return;
    float* S = a.state + slot * a.state_len + (long)head * d * dv;
    Cols<V> held[HOLD ? HELD : 1];
    if (HOLD && phase < phases && group < groups_all) {
#pragma unroll
        for (int n = 0; n < HELD; ++n) {
            const int c = phase + n * phases;
            if (c < d) held[HOLD ? n : 0].load(S + (long)c * dv + group * V);
        }
    }
    const long c0 = (long)head * d;
    for (int t = 0; t < count; ++t) {
        const long row = first + t;
        for (int r = tid; r < a.rank; r += WALK_THREADS) low[r] = a.low[row * a.stride + r];
        __syncthreads();
        for (int c = tid; c < d; c += WALK_THREADS) {
            qs[c] = a.q[row * a.stride + c0 + c] * a.q_scale;
            ks[c] = a.k[row * a.stride + c0 + c];
            float z = a.bias[c0 + c];
#pragma unroll 8
            for (int r = 0; r < a.rank; ++r) z = fmaf(a.up[(long)r * a.heads * d + c0 + c], low[r], z);
            decay[c] = expf(log_decay(z, a.tau_inverse));
        }
        __syncthreads();
        for (int g0 = 0; g0 < groups_all; g0 += groups) {
            const int g = g0 + group;
            const bool live = phase < phases && g < groups_all;
            Cols<V> acc;
#pragma unroll
            for (int e = 0; e < V; ++e) acc.x[e] = 0.0f;
            if (live) {
                Cols<V> v;
                v.load(a.v + row * a.stride + (long)head * dv + g * V);
                if (HOLD) {
#pragma unroll
                    for (int n = 0; n < HELD; ++n) {
                        const int c = phase + n * phases;
                        if (c < d) {
                            const float kept = decay[c], k = ks[c], q = qs[c];
                            Cols<V>& s = held[HOLD ? n : 0];
#pragma unroll
                            for (int e = 0; e < V; ++e) {
                                s.x[e] = fmaf(kept, s.x[e], k * v.x[e]);
                                acc.x[e] = fmaf(q, s.x[e], acc.x[e]);
                            }
                            s.store(S + (long)c * dv + g * V);
                        }
                    }
                } else {
#pragma unroll 8
                    for (int c = phase; c < d; c += phases) {
                        Cols<V> s;
                        s.load(S + (long)c * dv + g * V);
                        const float kept = decay[c], k = ks[c], q = qs[c];
#pragma unroll
                        for (int e = 0; e < V; ++e) {
                            s.x[e] = fmaf(kept, s.x[e], k * v.x[e]);
                            acc.x[e] = fmaf(q, s.x[e], acc.x[e]);
                        }
                        s.store(S + (long)c * dv + g * V);
                    }
                }
            }
            if (phase < phases) acc.store(red + (phase * groups + group) * V);
            __syncthreads();
            for (int j = tid; j < groups * V; j += WALK_THREADS) {
                float sum = 0.0f;
                for (int p = 0; p < phases; ++p) sum += red[p * groups * V + j];
                if (g0 * V + j < dv) os[g0 * V + j] = sum;
            }
            __syncthreads();
        }
        float square = 0.0f;
        for (int j = tid; j < dv; j += WALK_THREADS) square = fmaf(os[j], os[j], square);
        const float variance = block_sum(square, scratch) / (float)dv + eps;
        const float r = variance == 0.0f ? 0.0f : 1.0f / sqrtf(variance);
        for (int j = tid; j < dv; j += WALK_THREADS)
            out[row * ((long)a.heads * dv) + (long)head * dv + j] =
                from_f32<T>(os[j] * r * norm[j] * sf_silu(gate[row * a.stride + (long)head * dv + j]));
        __syncthreads();  // os and the token's rows are free for the next token
    }
}

int fill(ChannelScan& a, const float* rows, long stride, const float* up, const float* bias, float tau_inverse, float q_scale, float* state,
         long state_len, const int* query_start, const int* slots, int requests, int heads, int d, int dv, int rank, int num_slots) {
    if (heads <= 0 || d <= 0 || dv <= 0 || rank <= 0 || heads > 65535 || (long)heads * d * dv > state_len || !(tau_inverse > 0.0f))
        return KIRAI_ERR_BAD_SIZE;
    a.q = rows, a.k = rows + (long)heads * d, a.v = rows + 2L * heads * d, a.low = a.v + 2L * heads * dv;
    a.stride = stride, a.up = up, a.bias = bias, a.tau_inverse = tau_inverse, a.q_scale = q_scale;
    a.state = state, a.state_len = state_len, a.query_start = query_start, a.slots = slots;
    a.heads = heads, a.d = d, a.dv = dv, a.rank = rank, a.requests = requests, a.num_slots = num_slots;
    return 0;
}

template <typename T>
int walk_launch(const ChannelScan& a, const float* norm, float eps, void* out, int longest, cudaStream_t stream) {
    const float* gate = a.v + (long)a.heads * a.dv;
    const bool vec = a.dv % 4 == 0 && a.state_len % 4 == 0 && a.stride % 4 == 0 && ((uintptr_t)a.v & 15) == 0 && ((uintptr_t)a.state & 15) == 0;
    const int V = vec ? 4 : 1, groups = (a.dv + V - 1) / V;
    // a single token's state in registers: with twice the threads where that is what it takes
    const auto holds = [&](int threads) { return vec && longest == 1 && groups <= threads && (a.d + threads / groups - 1) / (threads / groups) <= HELD; };
    const int threads = !holds(256) && holds(512) ? 512 : 256;
    const size_t bytes = (3L * a.d + a.rank + a.dv + 4 + (long)threads * V) * sizeof(float);
    if (bytes > 47 * 1024) return KIRAI_ERR_UNSUPPORTED;
    const dim3 grid(a.requests, a.heads), block(threads);
    if (threads == 512) return launch_pdl(channel_walk_kernel<T, 4, true, 512>, grid, block, bytes, stream, 1u, a, gate, norm, eps, (T*)out);
    if (holds(256)) return launch_pdl(channel_walk_kernel<T, 4, true, 256>, grid, block, bytes, stream, 1u, a, gate, norm, eps, (T*)out);
    if (vec) return launch_pdl(channel_walk_kernel<T, 4, false, 256>, grid, block, bytes, stream, 1u, a, gate, norm, eps, (T*)out);
    return launch_pdl(channel_walk_kernel<T, 1, false, 256>, grid, block, bytes, stream, 1u, a, gate, norm, eps, (T*)out);
}

}  // namespace

// 1 when a head of d state rows whose decays come through `rank` columns fits the chunked kernels' shared memory, else 0.
KIRAI_EXPORT int kirai_channel_chunks_fit(int d, int rank) {
    int device = 0, limit = 0;
    if (cudaGetDevice(&device) != cudaSuccess ||
        cudaDeviceGetAttribute(&limit, cudaDevAttrMaxSharedMemoryPerBlockOptin, device) != cudaSuccess)
        return 0;
    return d > 0 && rank > 0 && product_floats(d, 16, CHAIN) * 4 <= limit && prepare_floats(d, rank) * 4 + 64 <= limit ? 1 : 0;
}

// rows [T, 2 heads d + 2 heads dv + rank] (float32, row stride `stride`): q, k, v, the output gate's and the short decay rows.
// Single tokens and short runs: out [T, heads dv] = o / rms(o) * norm * silu(gate), rms per head with eps inside the root.
KIRAI_EXPORT int kirai_channel_walk_f32(const float* rows, long stride, const float* up, const float* bias, float tau_inverse, float q_scale,
                                        float* state, long state_len, const int* query_start, const int* slots, const float* norm, float eps,
                                        void* out, int requests, int heads, int d, int dv, int rank, int num_slots, int longest,
                                        cudaStream_t stream) {
    if (requests <= 0) return 0;
    ChannelScan a = {};
    const int status = fill(a, rows, stride, up, bias, tau_inverse, q_scale, state, state_len, query_start, slots, requests, heads, d, dv, rank, num_slots);
    return status != 0 ? status : walk_launch<float>(a, norm, eps, out, longest, stream);
}
KIRAI_EXPORT int kirai_channel_walk_bf16(const float* rows, long stride, const float* up, const float* bias, float tau_inverse, float q_scale,
                                         float* state, long state_len, const int* query_start, const int* slots, const float* norm, float eps,
                                         void* out, int requests, int heads, int d, int dv, int rank, int num_slots, int longest,
                                         cudaStream_t stream) {
    if (requests <= 0) return 0;
    ChannelScan a = {};
    const int status = fill(a, rows, stride, up, bias, tau_inverse, q_scale, state, state_len, query_start, slots, requests, heads, d, dv, rank, num_slots);
    return status != 0 ? status : walk_launch<bf16>(a, norm, eps, out, longest, stream);
}

// Runs of many tokens: o [T, heads dv] (float32) as it leaves the state.  `units` >= the step's chunks (tokens / 64 + requests):
// tiles [units, heads, 2 d + 64, 64], kept [units, heads, d]; with `share` [units, heads, d, dv] the chunks run side by side.
KIRAI_EXPORT int kirai_channel_chunks(const float* rows, long stride, const float* up, const float* bias, float tau_inverse, float q_scale,
                                      float* state, long state_len, const int* query_start, const int* slots, float* o, float* tiles,
                                      float* kept, float* share, int requests, int heads, int d, int dv, int rank, int num_slots, int units,
                                      cudaStream_t stream) {
    if (requests <= 0) return 0;
    ChannelScan a = {};
    int status = fill(a, rows, stride, up, bias, tau_inverse, q_scale, state, state_len, query_start, slots, requests, heads, d, dv, rank, num_slots);
    if (status != 0) return status;
    if (units <= 0 || !tiles || !kept) return KIRAI_ERR_BAD_SIZE;
    a.out = o, a.tiles = tiles, a.kept = kept, a.share = share;
    a.cols = choose_cols((long)(share ? units : requests) * heads, d, dv, share != nullptr);
    if (a.cols <= 0) return KIRAI_ERR_UNSUPPORTED;
    const int runs = cols_pitch(a.cols) / 16, pieces = (dv + a.cols - 1) / a.cols;
    static long granted_prepare = 0, granted[3][5] = {};  // (one device a process)
    const long prepare_bytes = prepare_floats(d, rank) * 4;
    status = grant_shared(channel_prepare_kernel, prepare_bytes, &granted_prepare);
    if (status == 0)
        status = launch_pdl(channel_prepare_kernel, dim3(units, heads), dim3(THREADS), (size_t)prepare_bytes, stream, 1u, a);
    if (status != 0) return status;
    if (!share) {
        auto chain = KIRAI_BY_RUNS(runs, channel_chain_kernel);
        const long bytes = product_floats(d, a.cols, CHAIN) * 4;
        status = grant_shared(chain, bytes, &granted[0][runs]);
        return status != 0 ? status : launch_pdl(chain, dim3(requests, heads, pieces), dim3(THREADS), (size_t)bytes, stream, 1u, a);
    }
    auto own = KIRAI_BY_RUNS(runs, channel_share_kernel);
    auto out = KIRAI_BY_RUNS(runs, channel_out_kernel);
    const long own_bytes = product_floats(d, a.cols, SHARE) * 4, bytes = product_floats(d, a.cols, READ) * 4;
    status = grant_shared(own, own_bytes, &granted[1][runs]);
    if (status == 0) status = grant_shared(out, bytes, &granted[2][runs]);
    if (status == 0) status = launch_pdl(own, dim3(units, heads, pieces), dim3(THREADS), (size_t)own_bytes, stream, 1u, a);
    if (status == 0)
        status = launch_pdl(channel_carry_kernel, dim3(requests, heads, (unsigned)(((long)d * dv + 255) / 256)), dim3(256), 0, stream, 1u, a);
    if (status == 0) status = launch_pdl(out, dim3(units, heads, pieces), dim3(THREADS), (size_t)bytes, stream, 1u, a);
    return status;
}
