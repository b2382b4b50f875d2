// Element-wise gated recurrences and the short convolution ahead of them.
//
//   * a causal convolution over a few taps per channel with a bias on what enters it, a bias on what leaves it and an
//     optional silu; a block walks a run of tokens with the taps' rows in registers, so that every row is read once (and
//     taps - 1 rows more a run); the last taps - 1 rows that entered are state of the request.  For a product on the
//     tensor cores that must not round its input to 16 bits the rows can leave a second time as two bfloat16 numbers
//     each, high + low (16 bits of the value's 24), block by block of channels;
//   * the whole of such a recurrence (convolution, gates, state, branch) for a step of single tokens as one kernel;
//   * S_t = a_t S_(t-1) + b_t per channel, both terms from the current token alone: a block owns a few channels of one
//     request and goes through the request's tokens in windows.  In a window every thread takes a run of TOKENS tokens of
//     one channel: its terms stay in registers while the runs' (product of a, end state from zero) meet in shared memory,
//     every thread folds the runs before its own, and walks its run again from the state that this gives.  One pass over
//     the rows, no scratch; what the terms are and what leaves is a form (`RealGatedForm` below).
//
// Everything is 32-bit but what a product reads next.
#include "common.cuh"
#include "state_math.cuh"

namespace {

template <typename T>
struct is_rounded { static constexpr bool value = false; };
template <>
struct is_rounded<bf16> { static constexpr bool value = true; };

// ------------------------------------------------------------------ convolution
#define CONV_RUN 8

struct ConvArgs {
    const float* in;  // [T, channels], row stride in_stride
    long in_stride;
    const float* taps_w;   // [channels, taps], the last column weighs the token itself
    const float* in_bias;  // [channels] or null: added to every row that enters (zeros lie before a sequence's start)
    const float* bias;     // [channels] or null
    float* state;          // [slots, state_len], kept rows [taps - 1, channels] from column conv_off, the newest last
    long state_len, conv_off;
    const int* request_of_token;
    const int* query_start;
    const int* slots;
    float* out;    // [T, channels]
    bf16* pair;    // null, or [channels / block, pair_tokens, 2 * block]: high parts, then low parts
    int block, pair_tokens;
    int tokens, channels, num_slots, silu;
    int run;     // tokens a block walks, at most CONV_RUN
    int single;  // every request brings one token: the thread that read a channel's kept rows moves them on itself
};

__device__ __forceinline__ void conv_store(const ConvArgs& a, long token, int c, float v) {
    if (a.silu) v = sf_silu(v);
    a.out[token * a.channels + c] = v;
    if (a.pair) {
        const bf16 high = __float2bfloat16_rn(v);
        const int b = c / a.block, j = c - b * a.block;
        bf16* p = a.pair + ((long)b * a.pair_tokens + token) * 2 * a.block + j;
        p[0] = high;
        p[a.block] = __float2bfloat16_rn(v - __bfloat162float(high));
    }
}

template <int TAPS>
__global__ void conv_run_kernel(ConvArgs a) {
    pdl_launch_dependents();
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= a.channels) return;
    const long t0 = (long)blockIdx.x * a.run;
    const int count = (int)min((long)a.run, a.tokens - t0);
    float w[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = a.taps_w[(long)c * TAPS + j];
    const float in_bias = a.in_bias ? a.in_bias[c] : 0.0f, bias = a.bias ? a.bias[c] : 0.0f;
    int request[CONV_RUN];
#pragma unroll
    for (int i = 0; i < CONV_RUN; ++i) request[i] = i < count ? a.request_of_token[t0 + i] : -1;
    pdl_wait();
    float x[CONV_RUN];
#pragma unroll
    for (int i = 0; i < CONV_RUN; ++i) x[i] = i < count ? a.in[(t0 + i) * a.in_stride + c] + in_bias : 0.0f;
    float past[TAPS > 1 ? TAPS - 1 : 1];  // the rows before the token at hand, the newest last
    int current = -1;
#pragma unroll
    for (int i = 0; i < CONV_RUN; ++i) {
        if (i >= count) break;
        if (TAPS > 1 && request[i] != current) {
            // the run's first token, or another request's first: its earlier rows of this step, or the kept rows
            current = request[i];
            const long first = a.query_start[current];
            const int local = (int)(t0 + i - first);
            const int slot = a.slots[current];
            float* kept = a.state + (long)slot * a.state_len + a.conv_off;
            const bool held = slot >= 0 && slot < a.num_slots;
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) {
                const int at = local - (TAPS - 1) + j;
                past[j] = at >= 0 ? a.in[(first + at) * a.in_stride + c] + in_bias : (held ? kept[(long)(TAPS - 1 + at) * a.channels + c] : 0.0f);
            }
            if (a.single && held) {
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) kept[(long)j * a.channels + c] = j + 1 < TAPS - 1 ? past[j + 1] : x[i];
            }
        }
        float acc = bias;
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) acc = fmaf(w[j], past[j], acc);
        conv_store(a, t0 + i, c, fmaf(w[TAPS - 1], x[i], acc));
#pragma unroll
        for (int j = 0; j + 1 < TAPS - 1; ++j) past[j] = past[j + 1];
        if (TAPS > 1) past[TAPS > 1 ? TAPS - 2 : 0] = x[i];
    }
}

// Any number of taps: every tap read from where it lies.
__global__ void conv_any_kernel(ConvArgs a, int taps) {
    pdl_launch_dependents();
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    const long token = blockIdx.x;
    if (c >= a.channels) return;
    const int request = a.request_of_token[token];
    const long first = a.query_start[request];
    const int slot = a.slots[request];
    pdl_wait();
    if (slot < 0 || slot >= a.num_slots) return;
    const float in_bias = a.in_bias ? a.in_bias[c] : 0.0f;
    const int local = (int)(token - first);
    const float* kept = a.state + (long)slot * a.state_len + a.conv_off;
    float acc = a.bias ? a.bias[c] : 0.0f;
    for (int j = 0; j < taps; ++j) {
        const int at = local - (taps - 1) + j;
        const float v = at >= 0 ? a.in[(first + at) * a.in_stride + c] + in_bias : kept[(long)(taps - 1 + at) * a.channels + c];
        acc = fmaf(a.taps_w[(long)c * taps + j], v, acc);
    }
    conv_store(a, token, c, acc);
}

// A thread per (request, channel): the kept rows become the last taps - 1 rows that entered.
__global__ void conv_keep_kernel(const float* __restrict__ in, long in_stride, const float* __restrict__ in_bias, float* __restrict__ state,
                                 long state_len, long conv_off, const int* __restrict__ query_start, const int* __restrict__ slots,
                                 int requests, int channels, int taps, int num_slots) {
    pdl_launch_dependents();
    pdl_wait();
    const long at = blockIdx.x * (long)blockDim.x + threadIdx.x;
    if (at >= (long)requests * channels) return;
    const int request = (int)(at / channels), c = (int)(at - (long)request * channels);
    const int slot = slots[request];
    if (slot < 0 || slot >= num_slots) return;
    const float add = in_bias ? in_bias[c] : 0.0f;
    const long first = query_start[request];
    const int count = (int)(query_start[request + 1] - first);
    float* kept = state + (long)slot * state_len + conv_off;
    // ascending: entry k takes row count - (taps - 1) + k, or the kept row count + k (> k, not yet overwritten)
    for (int k = 0; k < taps - 1; ++k) {
        const int src = count - (taps - 1) + k;
        kept[(long)k * channels + c] = src >= 0 ? in[(first + src) * in_stride + c] + add : kept[(long)(count + k) * channels + c];
    }
}

// ------------------------------------------------------------------ the scan
// The real-gated linear recurrence: with r = sigmoid(pre_r + r_bias), i = sigmoid(pre_i + i_bias) and rate <= 0 per channel,
// a = exp(rate r), b = sqrt(1 - a^2) i u; what leaves is factor * S * gelu_tanh(branch + branch_bias).
// The gates' pre-activations come from a product per block of channels: the token's pair of a channel lies at
// gates[token * gate_token + block * gate_block + j] (r) and `block` columns further (i).
template <typename O>
struct RealGatedForm {
    const float* u;  // [T, channels]
    const float* gates;
    long gate_token, gate_block;
    int block;
    const float* branch;  // [T, channels], row stride branch_stride
    long branch_stride;
    const float *r_bias, *i_bias, *branch_bias, *rate;
    float factor;
    O* out;
    long out_stride;
    int width;

    static constexpr bool FAST = is_rounded<O>::value;
    struct Channel { float rb, ib, bb, rate; long gate_at; int c; };
    struct Row { float r, i, u, branch; };
    using Kept = float;  // what the store of a token needs of its row

    __device__ __forceinline__ Channel channel(int c) const {
        const int b = c / block;
        return Channel{r_bias[c], i_bias[c], branch_bias[c], rate[c], b * gate_block + (c - b * block), c};
    }
    __device__ __forceinline__ Row load(const Channel& ch, long token) const {
        const float* g = gates + token * gate_token + ch.gate_at;
        return Row{g[0], g[block], u[token * width + ch.c], branch[token * branch_stride + ch.c]};
    }
    __device__ __forceinline__ void terms(const Channel& ch, const Row& row, float& a, float& b) const {
        float decay, left;  // a, and 1 - a^2
        if (FAST) {
            const float log_a = ch.rate * __fdividef(1.0f, 1.0f + __expf(-(row.r + ch.rb)));
            decay = __expf(log_a);
            // 1 - a where a is close to one from the series of the exponential, else directly
            const float gap = log_a > -0.06f ? -log_a * (1.0f + log_a * (0.5f + log_a * (0.16666667f + log_a * 0.041666667f))) : 1.0f - decay;
            left = gap * (1.0f + decay);
            a = decay;
            b = sqrtf(left) * __fdividef(row.u, 1.0f + __expf(-(row.i + ch.ib)));
        } else {
            const float log_a = ch.rate * sf_sigmoid(row.r + ch.rb);
            decay = expf(log_a);
            left = -expm1f(2.0f * log_a);
            a = decay;
            b = sqrtf(left) * (sf_sigmoid(row.i + ch.ib) * row.u);
        }
    }
    __device__ __forceinline__ Kept keep(const Row& row) const { return row.branch; }
    __device__ __forceinline__ void store(const Channel& ch, Kept branch, long token, float s) const {
        const float z = branch + ch.bb;
        // 0.5 z (1 + tanh(y)) = z sigmoid(2 y)
        const float gate = FAST ? __fdividef(z, 1.0f + __expf(-1.5957691216057308f * fmaf(0.044715f * z * z, z, z))) : sf_gelu_tanh(z);
        out[token * out_stride + ch.c] = from_f32<O>(factor * (s * gate));
    }
};

// Blocks (run of CH channels, request); threads: `runs` * CH.
template <class Form, int CH, int TOKENS>
__global__ void __launch_bounds__(256)
gated_scan_kernel(Form form, float* __restrict__ state, long state_len, long state_off, const int* __restrict__ query_start,
                  const int* __restrict__ slots, int channels, int num_slots) {
    pdl_launch_dependents();
    extern __shared__ float2 ends[];  // [2][runs][CH]: a run's (product of a, end state from zero); two windows take turns
    const int runs = blockDim.x / CH;
    const int lane = threadIdx.x % CH, run = threadIdx.x / CH;
    const int c = blockIdx.x * CH + lane;
    const int request = blockIdx.y;
    const bool live = c < channels;
    const long first = query_start[request];
    const int count = (int)(query_start[request + 1] - first);
    const int slot = slots[request];
    if (slot < 0 || slot >= num_slots) return;  // the whole block
    typename Form::Channel ch = form.channel(live ? c : 0);
    float* kept = state + (long)slot * state_len + state_off + c;
    pdl_wait();
    float carry = live ? *kept : 0.0f;
    int turn = 0;
    typename Form::Row row[TOKENS];
#pragma unroll
    for (int i = 0; i < TOKENS; ++i)
        if (live && run * TOKENS + i < count) row[i] = form.load(ch, first + run * TOKENS + i);
    for (int w0 = 0; w0 < count; w0 += runs * TOKENS, turn ^= 1) {
        const int t0 = w0 + run * TOKENS;
        float a[TOKENS], b[TOKENS];
        float prod = 1.0f, end = 0.0f;
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) {
            a[i] = 1.0f, b[i] = 0.0f;
            if (live && t0 + i < count) form.terms(ch, row[i], a[i], b[i]);
            prod *= a[i];
            end = fmaf(a[i], end, b[i]);
        }
        // the next window's rows are asked for here, ahead of the meeting and of this window's stores
        typename Form::Kept held[TOKENS];
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) held[i] = form.keep(row[i]);
        const int next = t0 + runs * TOKENS;
#pragma unroll
        for (int i = 0; i < TOKENS; ++i)
            if (live && next + i < count) row[i] = form.load(ch, first + next + i);
        float s = carry;
        if (runs > 1) {
            float2* here = ends + (size_t)turn * blockDim.x;
            here[threadIdx.x] = make_float2(prod, end);
            __syncthreads();
            for (int p = 0; p < runs; ++p) {
                if (p == run) s = carry;
                const float2 e = here[p * CH + lane];
                carry = fmaf(e.x, carry, e.y);
            }
        } else {
            carry = fmaf(prod, carry, end);
        }
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) {
            s = fmaf(a[i], s, b[i]);
            if (live && t0 + i < count) form.store(ch, held[i], first + t0 + i, s);
        }
    }
    // (every thread of the channel read the old state ahead of its first barrier, or is the only one)
    if (live && run == 0 && count > 0) *kept = carry;
}

template <class Form>
int gated_scan_launch(const Form& form, float* state, long state_len, long state_off, const int* query_start, const int* slots,
                      int requests, int max_query_len, int channels, int num_slots, cudaStream_t stream) {
    constexpr int TOKENS = 8;
    // a warp's rows are runs of 32 channels (one line), or of 16 or 8 (whole sectors) where that brings two blocks to an SM
    int ch = 32;
    while (ch > 8 && (long)((channels + ch - 1) / ch) * requests < 256) ch >>= 1;
    int runs = (max_query_len + TOKENS - 1) / TOKENS;
    const int most = 256 / ch, least = 32 / ch;
    if (runs > most) runs = most;
    if (runs < least) runs = least;
    const int threads = ((runs * ch + 31) / 32) * 32;
    const size_t smem = 2 * (size_t)threads * sizeof(float2);
    const dim3 grid((channels + ch - 1) / ch, requests);
    auto kernel = ch == 32 ? gated_scan_kernel<Form, 32, TOKENS> : ch == 16 ? gated_scan_kernel<Form, 16, TOKENS> : gated_scan_kernel<Form, 8, TOKENS>;
    return launch_pdl(kernel, grid, dim3(threads), smem, stream, 1u, form, state, state_len, state_off, query_start, slots, channels, num_slots);
}

template <typename O>
int real_gated_launch(const float* u, const float* gates, long gate_token, long gate_block, int block, const float* branch,
                      long branch_stride, const float* r_bias, const float* i_bias, const float* branch_bias, const float* rate,
                      float factor, float* state, long state_len, long state_off, const int* query_start, const int* slots, void* out,
                      long out_stride, int requests, int max_query_len, int channels, int num_slots, cudaStream_t stream) {
    if (requests <= 0 || max_query_len <= 0) return 0;
    if (channels <= 0 || block <= 0 || channels % block || requests > 65535 || state_off < 0 || state_off + channels > state_len ||
        out_stride < channels || branch_stride < channels)
        return KIRAI_ERR_BAD_SIZE;
    const RealGatedForm<O> form{u, gates, gate_token, gate_block, block, branch, branch_stride, r_bias, i_bias, branch_bias, rate, factor,
                                (O*)out, out_stride, channels};
    return gated_scan_launch(form, state, state_len, state_off, query_start, slots, requests, max_query_len, channels, num_slots, stream);
}

// ------------------------------------------------------------------ a step of single tokens
// Convolution, the gates' products, the recurrence and the gelu branch for a step in which every request brings one token
// (row r is request r's).  A cluster of CTAs takes a block of channels; every CTA makes the block's u for STEP_ROWS requests
// at a time in its own shared memory, multiplies it with the rows of its share of the block's two gate matrices (a warp
// per channel, 32-bit multiply-adds, the lanes' partial sums of all requests folded together), and finishes its channels.
// The kept rows of the convolution are read by the whole cluster: they move on after the cluster has met.
#define STEP_ROWS 8
#define STEP_REQUESTS 128

template <typename W>
__device__ __forceinline__ float4 weights4(const W* p);
template <>
__device__ __forceinline__ float4 weights4<float>(const float* p) { return __ldg(reinterpret_cast<const float4*>(p)); }
template <>
__device__ __forceinline__ float4 weights4<bf16>(const bf16* p) {
    const uint2 q = __ldg(reinterpret_cast<const uint2*>(p));
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}

struct StepArgs {
    const float* rows;  // [R, >= 2 width], row stride: the branch's columns, then the convolution's input
    long row_stride;
    const float *taps_w, *in_bias, *bias;
    const void* gates;  // [blocks, 2 block, block]
    const float *r_bias, *i_bias, *branch_bias, *rate;
    float factor;
    float* state;
    long state_len, conv_off, state_off;
    const int* slots;
    long out_stride;
    int requests, width, block, taps, num_slots;
};

// u of one channel for the STEP_ROWS requests from r0 on; every load of the channel is asked for ahead of the sums.
template <int TAPS>
__device__ __forceinline__ void step_convolution(const StepArgs& a, int r0, int count, int c, const int* slot_s, float (&u)[STEP_ROWS]) {
    const int taps = TAPS > 0 ? TAPS : a.taps;
    const float bias = __ldg(a.bias + c), in_bias = __ldg(a.in_bias + c);
    const float* w = a.taps_w + (long)c * taps;
    float x[STEP_ROWS];
#pragma unroll
    for (int r = 0; r < STEP_ROWS; ++r) x[r] = r < count ? a.rows[(r0 + r) * a.row_stride + a.width + c] + in_bias : 0.0f;
    if (TAPS > 0) {
        float past[STEP_ROWS][TAPS > 1 ? TAPS - 1 : 1];
#pragma unroll
        for (int r = 0; r < STEP_ROWS; ++r) {
            const int slot = r < count ? slot_s[r0 + r] : -1;
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j)
                past[r][j] = slot >= 0 ? a.state[(long)slot * a.state_len + a.conv_off + (long)j * a.width + c] : 0.0f;
        }
#pragma unroll
        for (int r = 0; r < STEP_ROWS; ++r) {
            float acc = bias;
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) acc = fmaf(__ldg(w + j), past[r][j], acc);
            u[r] = fmaf(__ldg(w + TAPS - 1), x[r], acc);
        }
    } else {
#pragma unroll
        for (int r = 0; r < STEP_ROWS; ++r) {
            const int slot = r < count ? slot_s[r0 + r] : -1;
            float acc = bias;
            for (int j = 0; slot >= 0 && j + 1 < taps; ++j)
                acc = fmaf(w[j], a.state[(long)slot * a.state_len + a.conv_off + (long)j * a.width + c], acc);
            u[r] = fmaf(w[taps - 1], x[r], acc);
        }
    }
}

// 2 * ROWS sums over 32 lanes: halves change hands until a lane holds one sum's share (lane bits from the highest say which
// sum), then the lanes that are left of it add up.
template <int SUMS>
__device__ __forceinline__ float fold_sums(float (&sum)[SUMS], int lane) {
    int lanes = 16;
#pragma unroll
    for (int half = SUMS / 2; half >= 1; half >>= 1) {
        const bool upper = (lane & lanes) != 0;
#pragma unroll
        for (int r = 0; r < half; ++r) {
            const float give = upper ? sum[r] : sum[half + r];
            const float got = __shfl_xor_sync(0xffffffffu, give, lanes);
            sum[r] = (upper ? sum[half + r] : sum[r]) + got;
        }
        lanes >>= 1;
    }
    float total = sum[0];
    for (; lanes >= 1; lanes >>= 1) total += __shfl_xor_sync(0xffffffffu, total, lanes);
    return total;
}

template <typename O, typename W, bool VEC, int TAPS>
__global__ void __launch_bounds__(256) real_gated_step_kernel(StepArgs a, O* __restrict__ out) {
    pdl_launch_dependents();
    extern __shared__ float step_smem[];
    __shared__ int slot_s[STEP_REQUESTS];
    const int d = a.block, cuts = gridDim.x, b = blockIdx.y;
    const int per = (d + cuts - 1) / cuts;
    const int lo = min(d, (int)blockIdx.x * per), hi = min(d, lo + per);
    float* u_s = step_smem;                    // [STEP_ROWS][d]
    float* gate_s = step_smem + STEP_ROWS * d;  // [2][STEP_ROWS][per]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const W* gates = reinterpret_cast<const W*>(a.gates) + (size_t)b * 2 * d * d;
    // this CTA's rows of the two matrices, asked into L2 while the kernel before still runs
    for (int gate = 0; gate < 2; ++gate) {
        const char* from = reinterpret_cast<const char*>(gates + ((size_t)gate * d + lo) * d);
        const size_t bytes = (size_t)(hi - lo) * d * sizeof(W);
        for (size_t at = threadIdx.x * 128u; at < bytes; at += blockDim.x * 128u) asm volatile("prefetch.global.L2 [%0];" ::"l"(from + at));
    }
    for (int r = threadIdx.x; r < a.requests; r += blockDim.x) {
        const int slot = a.slots[r];
        slot_s[r] = slot < a.num_slots ? slot : -1;
    }
    __syncthreads();
    pdl_wait();
    const int taps = TAPS > 0 ? TAPS : a.taps, width = a.width, own = hi - lo;
    const RealGatedForm<O> form{nullptr, nullptr, 0, 0, d, nullptr, 0, a.r_bias, a.i_bias, a.branch_bias, a.rate, a.factor, out, a.out_stride, width};
    for (int r0 = 0; r0 < a.requests; r0 += STEP_ROWS) {
        const int count = min(STEP_ROWS, a.requests - r0);
        if (r0) __syncthreads();
        for (int j = threadIdx.x; j < d; j += blockDim.x) {
            float u[STEP_ROWS];
            step_convolution<TAPS>(a, r0, count, b * d + j, slot_s, u);
#pragma unroll
            for (int r = 0; r < STEP_ROWS; ++r) u_s[r * d + j] = u[r];
        }
        // the first (request, channel) that this thread will finish: its state and branch are asked for here
        float first_s = 0.0f, first_branch = 0.0f;
        if (threadIdx.x < count * own) {
            const int r = threadIdx.x / own, c = b * d + lo + threadIdx.x - r * own, slot = slot_s[r0 + r];
            if (slot >= 0) first_s = a.state[(long)slot * a.state_len + a.state_off + c];
            first_branch = a.rows[(r0 + r) * a.row_stride + c];
        }
        __syncthreads();
        for (int j = lo + warp; j < hi; j += warps) {
            const W* row_r = gates + (size_t)j * d;
            const W* row_i = gates + (size_t)(d + j) * d;
            float sum[2 * STEP_ROWS];  // the requests' r sums, then their i sums
#pragma unroll
            for (int r = 0; r < 2 * STEP_ROWS; ++r) sum[r] = 0.0f;
            if (VEC) {
                for (int k0 = lane * 4; k0 < d; k0 += 256) {
                    // two pieces' weights at once
                    const int k1 = k0 + 128;
                    const float4 none = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                    const float4 wr0 = weights4<W>(row_r + k0), wi0 = weights4<W>(row_i + k0);
                    const float4 wr1 = k1 < d ? weights4<W>(row_r + k1) : none, wi1 = k1 < d ? weights4<W>(row_i + k1) : none;
#pragma unroll
                    for (int r = 0; r < STEP_ROWS; ++r) {
                        const float4 u = *reinterpret_cast<const float4*>(u_s + r * d + k0);
                        sum[r] = fmaf(wr0.x, u.x, fmaf(wr0.y, u.y, fmaf(wr0.z, u.z, fmaf(wr0.w, u.w, sum[r]))));
                        sum[STEP_ROWS + r] = fmaf(wi0.x, u.x, fmaf(wi0.y, u.y, fmaf(wi0.z, u.z, fmaf(wi0.w, u.w, sum[STEP_ROWS + r]))));
                    }
                    if (k1 < d) {
#pragma unroll
                        for (int r = 0; r < STEP_ROWS; ++r) {
                            const float4 u = *reinterpret_cast<const float4*>(u_s + r * d + k1);
                            sum[r] = fmaf(wr1.x, u.x, fmaf(wr1.y, u.y, fmaf(wr1.z, u.z, fmaf(wr1.w, u.w, sum[r]))));
                            sum[STEP_ROWS + r] = fmaf(wi1.x, u.x, fmaf(wi1.y, u.y, fmaf(wi1.z, u.z, fmaf(wi1.w, u.w, sum[STEP_ROWS + r]))));
                        }
                    }
                }
            } else {
                for (int k = lane; k < d; k += 32) {
                    const float wr = to_f32<W>(row_r[k]), wi = to_f32<W>(row_i[k]);
#pragma unroll
                    for (int r = 0; r < STEP_ROWS; ++r) {
                        sum[r] = fmaf(wr, u_s[r * d + k], sum[r]);
                        sum[STEP_ROWS + r] = fmaf(wi, u_s[r * d + k], sum[STEP_ROWS + r]);
                    }
                }
            }
            const float total = fold_sums<2 * STEP_ROWS>(sum, lane);
            if ((lane & 1) == 0) gate_s[(lane >> 1) * per + (j - lo)] = total;
        }
        __syncthreads();
        for (int at = threadIdx.x; at < count * own; at += blockDim.x) {
            const int r = at / own, j = at - r * own, slot = slot_s[r0 + r];
            if (slot < 0) continue;
            const int c = b * d + lo + j;
            float* S = a.state + (long)slot * a.state_len + a.state_off + c;
            const bool held = at == (int)threadIdx.x;
            const typename RealGatedForm<O>::Channel ch = form.channel(c);
            const typename RealGatedForm<O>::Row row{gate_s[r * per + j], gate_s[(STEP_ROWS + r) * per + j], u_s[r * d + lo + j],
                                                     held ? first_branch : a.rows[(r0 + r) * a.row_stride + c]};
            float keep, take;
            form.terms(ch, row, keep, take);
            const float s = fmaf(keep, held ? first_s : *S, take);
            *S = s;
            form.store(ch, form.keep(row), r0 + r, s);
        }
    }
    // every CTA of the cluster has read the block's kept rows
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (taps > 1) {
        for (int at = threadIdx.x; at < a.requests * own; at += blockDim.x) {
            const int r = at / own, c = b * d + lo + (at - r * own), slot = slot_s[r];
            if (slot < 0) continue;
            float* kept = a.state + (long)slot * a.state_len + a.conv_off + c;
            for (int k = 0; k + 2 < taps; ++k) kept[(long)k * width] = kept[(long)(k + 1) * width];
            kept[(long)(taps - 2) * width] = a.rows[r * a.row_stride + width + c] + a.in_bias[c];
        }
    }
}

template <typename O, typename W, bool VEC>
void (*step_kernel(int taps))(StepArgs, O*) {
    return taps == 2 ? real_gated_step_kernel<O, W, VEC, 2> : taps == 3 ? real_gated_step_kernel<O, W, VEC, 3>
         : taps == 4 ? real_gated_step_kernel<O, W, VEC, 4> : real_gated_step_kernel<O, W, VEC, 0>;
}

template <typename O>
int real_gated_step_launch(const StepArgs& a, int gates_bf16, void* out, cudaStream_t stream) {
    if (a.requests <= 0) return 0;
    if (a.requests > STEP_REQUESTS) return KIRAI_ERR_BAD_SIZE;
    if (a.width <= 0 || a.block <= 0 || a.width % a.block || a.taps < 1 || a.conv_off < 0 || a.state_off < 0 || a.out_stride < a.width ||
        a.conv_off + (long)(a.taps - 1) * a.width > a.state_len || a.state_off + a.width > a.state_len)
        return KIRAI_ERR_BAD_SIZE;
    const int blocks = a.width / a.block;
    if (blocks > 65535) return KIRAI_ERR_BAD_SIZE;
    int cuts = 1;
    while (cuts < 8 && blocks * cuts < 148 && a.block / (cuts * 2) >= 8) cuts *= 2;
    const int per = (a.block + cuts - 1) / cuts;
    const size_t smem = (size_t)STEP_ROWS * (a.block + 2 * per) * sizeof(float);
    if (smem > 200 * 1024) return KIRAI_ERR_BAD_SIZE;
    const bool vec = a.block % 4 == 0 && ((uintptr_t)a.gates & 15) == 0;
    auto kernel = gates_bf16 ? (vec ? step_kernel<O, bf16, true>(a.taps) : step_kernel<O, bf16, false>(a.taps))
                             : (vec ? step_kernel<O, float, true>(a.taps) : step_kernel<O, float, false>(a.taps));
    if (smem > 48 * 1024) {
        const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (err != cudaSuccess) return (int)err;
    }
    return launch_pdl_clusters(kernel, dim3(cuts, blocks), dim3(256), smem, stream, dim3(cuts, 1, 1), a, (O*)out);
}

}  // namespace

// A step of single tokens in one kernel (see real_gated_step_kernel): the kept rows at columns [conv_off, conv_off +
// (taps - 1) width) of the request's slot, S at [state_off, state_off + width).
#define KIRAI_REAL_GATED_STEP(NAME, O)                                                                                            \
    KIRAI_EXPORT int NAME(const float* rows, long row_stride, const float* taps_w, const float* in_bias, const float* bias,       \
                          const void* gates, int gates_bf16, const float* r_bias, const float* i_bias, const float* branch_bias, \
                          const float* rate, float factor, float* state, long state_len, long conv_off, long state_off,          \
                          const int* slots, void* out, long out_stride, int requests, int width, int block, int taps,            \
                          int num_slots, cudaStream_t stream) {                                                                  \
        const StepArgs a{rows, row_stride, taps_w, in_bias, bias, gates, r_bias, i_bias, branch_bias, rate, factor, state,       \
                         state_len, conv_off, state_off, slots, out_stride, requests, width, block, taps, num_slots};            \
        return real_gated_step_launch<O>(a, gates_bf16, out, stream);                                                            \
    }
KIRAI_REAL_GATED_STEP(kirai_real_gated_step_f32, float)
KIRAI_REAL_GATED_STEP(kirai_real_gated_step_bf16, bf16)
#undef KIRAI_REAL_GATED_STEP

// out [T, channels] (float32) = (silu of) bias + sum_j taps_w[c, j] * (in[t - (taps - 1) + j, c] + in_bias[c]) per request,
// kept rows before a request's first row of this step; then the kept rows move on.  pair (may be null): the same rows as
// high and low bfloat16 parts, [channels / block, pair_tokens, 2 block].  single: every request brings one token.
KIRAI_EXPORT int kirai_conv_rows(const float* in, long in_stride, const float* taps_w, const float* in_bias, const float* bias,
                                 float* state, long state_len, long conv_off, const int* request_of_token, const int* query_start,
                                 const int* slots, float* out, void* pair, int block, int pair_tokens, int silu, int single,
                                 int tokens, int requests, int channels, int taps, int num_slots, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (channels <= 0 || taps <= 0 || requests <= 0 || conv_off < 0 || conv_off + (long)(taps - 1) * channels > state_len)
        return KIRAI_ERR_BAD_SIZE;
    if (pair && (block <= 0 || channels % block || pair_tokens < tokens)) return KIRAI_ERR_BAD_SIZE;
    const int threads = channels >= 8192 || tokens >= 512 ? 256 : 128;
    const unsigned columns = (unsigned)((channels + threads - 1) / threads);
    // few tokens: shorter runs, so that more blocks ask for rows at the same time
    int run = CONV_RUN;
    while (run > 1 && (long)((tokens + run - 1) / run) * columns < 592) run >>= 1;
    if (single) run = 1;
    const ConvArgs a{in, in_stride, taps_w, in_bias, bias, state, state_len, conv_off, request_of_token, query_start, slots, out,
                     (bf16*)pair, block, pair_tokens, tokens, channels, num_slots, silu, run, single && taps <= 4};
    const unsigned walks = (unsigned)((tokens + run - 1) / run);
    int status;
    switch (taps) {
        case 1: status = launch_pdl(conv_run_kernel<1>, dim3(walks, columns), dim3(threads), 0, stream, 1u, a); break;
        case 2: status = launch_pdl(conv_run_kernel<2>, dim3(walks, columns), dim3(threads), 0, stream, 1u, a); break;
        case 3: status = launch_pdl(conv_run_kernel<3>, dim3(walks, columns), dim3(threads), 0, stream, 1u, a); break;
        case 4: status = launch_pdl(conv_run_kernel<4>, dim3(walks, columns), dim3(threads), 0, stream, 1u, a); break;
        default: status = launch_pdl(conv_any_kernel, dim3(tokens, columns), dim3(threads), 0, stream, 1u, a, taps); break;
    }
    if (status != 0 || taps == 1 || a.single) return status;
    const long units = (long)requests * channels;
    return launch_pdl(conv_keep_kernel, dim3((unsigned)((units + 255) / 256)), dim3(256), 0, stream, 1u, in, in_stride, in_bias, state,
                      state_len, conv_off, query_start, slots, requests, channels, taps, num_slots);
}

// S <- a S + b per channel over each request's tokens of this step (see RealGatedForm), S in the request's slot of `state`
// [slots, state_len] from column state_off.
KIRAI_EXPORT int kirai_real_gated_scan_f32(const float* u, const float* gates, long gate_token, long gate_block, int block,
                                           const float* branch, long branch_stride, const float* r_bias, const float* i_bias,
                                           const float* branch_bias, const float* rate, float factor, float* state, long state_len,
                                           long state_off, const int* query_start, const int* slots, void* out, long out_stride,
                                           int requests, int max_query_len, int channels, int num_slots, cudaStream_t stream) {
    return real_gated_launch<float>(u, gates, gate_token, gate_block, block, branch, branch_stride, r_bias, i_bias, branch_bias, rate,
                                    factor, state, state_len, state_off, query_start, slots, out, out_stride, requests, max_query_len,
                                    channels, num_slots, stream);
}
KIRAI_EXPORT int kirai_real_gated_scan_bf16(const float* u, const float* gates, long gate_token, long gate_block, int block,
                                            const float* branch, long branch_stride, const float* r_bias, const float* i_bias,
                                            const float* branch_bias, const float* rate, float factor, float* state, long state_len,
                                            long state_off, const int* query_start, const int* slots, void* out, long out_stride,
                                            int requests, int max_query_len, int channels, int num_slots, cudaStream_t stream) {
    return real_gated_launch<bf16>(u, gates, gate_token, gate_block, block, branch, branch_stride, r_bias, i_bias, branch_bias, rate,
                                   factor, state, state_len, state_off, query_start, slots, out, out_stride, requests, max_query_len,
                                   channels, num_slots, stream);
}
