// The residual stream's sum and a short causal convolution beside it, in one pass:
//
//   s[t]   = x[t] + bscale * br[t]                 br = branch, or branch * rsqrt(mean(branch^2) + beps) * (boffset + bw)
//   out[t] = s[t] + sum_j taps[:, j] * s[t - (K-1) + j]        s = 0 before a sequence's start
//
// x, s, the branch, the taps and every sum are float32; out leaves in the engine's type.  The K-1 sums before a
// step's first token of a request are the request's state, state[slot, K-1, C] (oldest first, zero when a request
// opens).  s goes to a buffer other than x, because a block forms the sums of the K-1 tokens before its own again and
// so reads rows of x that belong to another block.  Without a branch s is x and nothing is stored.
//
// A block takes `run` consecutive tokens.  First its warps reduce the branch's rows (every row in kSegments pieces of
// fixed bounds, so a row's norm does not depend on the run or the batch), then every thread walks over the tokens for V
// neighbouring channels with the K-1 sums before in registers.  Taps are added in the order j = 0 .. K-1 whatever the
// cut.  The state a step leaves behind is written in the same pass where every request brings one token (`single`);
// otherwise by conv_state_kernel afterwards, since other blocks still read the old state.
#include "common.cuh"

namespace {
constexpr int kThreads = 256;
constexpr int kSegments = 8;      // pieces of a row in the reduction
constexpr int kMaxRun = 8;        // tokens of a block
constexpr int kMaxTaps = 8;       // taps of the fused form
constexpr int kAhead = 4;         // tokens whose rows are asked for together

struct StreamConvArgs {
    float* s_out;                 // absent: no branch, s is x
    const float* x;
    const float* branch;
    const float* bw;              // absent: the branch is added as it is
    const float* taps;            // [C, K]
    float* state;                 // [slots, K-1, C]; absent where K is 1
    const int* req_of_token;
    const int* q_start;
    const int* slots;
    int tokens, C, run, single;
    float beps, boffset, bscale;
};

template <int V>
__device__ __forceinline__ void load_channels(const float* p, float (&v)[V]) {
    if (V == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        v[0] = q.x, v[1 % V] = q.y, v[2 % V] = q.z, v[3 % V] = q.w;
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = p[i];
    }
}
template <int V>
__device__ __forceinline__ void store_channels(float* p, const float (&v)[V]) {
    if (V == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) p[i] = v[i];
    }
}
template <int V>
__device__ __forceinline__ void store_channels(__nv_bfloat16* p, const float (&v)[V]) {
    if (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1 % V]), b = __floats2bfloat162_rn(v[2 % V], v[3 % V]);
        uint2 q;
        q.x = *reinterpret_cast<const unsigned*>(&a);
        q.y = *reinterpret_cast<const unsigned*>(&b);
        *reinterpret_cast<uint2*>(p) = q;
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) p[i] = __float2bfloat16_rn(v[i]);
    }
}

template <typename TO, int K, int V>
__global__ void __launch_bounds__(kThreads) stream_conv_kernel(TO* __restrict__ out, StreamConvArgs a) {
    __shared__ float part[(kMaxRun + kMaxTaps) * kSegments];
    __shared__ float inv_of[kMaxRun + kMaxTaps];
    const int C = a.C;
    const int first = blockIdx.x * a.run, last = min(first + a.run, a.tokens);
    // the rows whose sums this block forms: its own and the K-1 before them that belong to the same request
    const int b0 = a.req_of_token[first];
    const int low = b0 >= 0 ? max(a.q_start[b0], first - (K - 1)) : first;
    if (a.bw != nullptr) {
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
        const int rows = last - low;
        const int piece = ((C + kSegments - 1) / kSegments + V - 1) / V * V;
        for (int i = warp; i < rows * kSegments; i += kThreads / 32) {
            const int r = i / kSegments, g = i % kSegments;
            const float* row = a.branch + (size_t)(low + r) * C;
            const int hi = min(C, (g + 1) * piece);
            float ss = 0.f;
#pragma unroll 4
            for (int c = g * piece + lane * V; c < hi; c += 32 * V) {
                float v[V];
                load_channels<V>(row + c, v);
#pragma unroll
                for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
            }
            ss = warp_sum(ss);
            if (lane == 0) part[i] = ss;
        }
        __syncthreads();
        if (threadIdx.x < rows) {
            float ss = 0.f;
#pragma unroll
            for (int g = 0; g < kSegments; ++g) ss += part[threadIdx.x * kSegments + g];
            inv_of[threadIdx.x] = 1.f / sqrtf(ss / (float)C + a.beps);
        }
        __syncthreads();
    }
    for (int c = (blockIdx.y * kThreads + threadIdx.x) * V; c < C; c += gridDim.y * kThreads * V) {
        float tap[K][V], win[K > 1 ? K - 1 : 1][V], bwv[V];
#pragma unroll
        for (int v = 0; v < V; ++v) {
            bwv[v] = a.bw != nullptr ? (a.boffset + a.bw[c + v]) * a.bscale : a.bscale;
        }
        if (V == 4 && K % 4 == 0) {
#pragma unroll
            for (int i = 0; i < K; ++i) {       // V * K neighbouring floats, four at a time
                const float4 q = *reinterpret_cast<const float4*>(a.taps + (size_t)c * K + 4 * i);
                const float e[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                for (int u = 0; u < 4; ++u) tap[(4 * i + u) % K][(4 * i + u) / K % V] = e[u];
            }
        } else {
#pragma unroll
            for (int v = 0; v < V; ++v)
#pragma unroll
                for (int j = 0; j < K; ++j) tap[j][v] = a.taps[(size_t)(c + v) * K + j];
        }
        // a row's sum at this thread's channels, from its parts
        auto sum_of = [&](int t, const float (&xv)[V], const float (&bv)[V], float (&s)[V]) {
            const float inv = a.bw != nullptr ? inv_of[t - low] : 1.f;
#pragma unroll
            for (int v = 0; v < V; ++v) s[v] = fmaf(bv[v] * inv, bwv[v], xv[v]);
        };
        int held = -1;          // the request whose sums the registers hold
        for (int tu = first; tu < last; tu += kAhead) {
            float xv[kAhead][V], bv[kAhead][V];
            int bs[kAhead];
#pragma unroll
            for (int i = 0; i < kAhead; ++i) {
                const int t = min(tu + i, last - 1);
                bs[i] = a.req_of_token[t];
                load_channels<V>(a.x + (size_t)t * C + c, xv[i]);
                if (a.branch != nullptr) load_channels<V>(a.branch + (size_t)t * C + c, bv[i]);
            }
#pragma unroll
            for (int i = 0; i < kAhead; ++i) {
                const int t = tu + i;
                if (t >= last) break;
                float s[V];
                if (a.branch != nullptr) {
                    sum_of(t, xv[i], bv[i], s);
                    store_channels<V>(a.s_out + (size_t)t * C + c, s);
                } else {
#pragma unroll
                    for (int v = 0; v < V; ++v) s[v] = xv[i][v];
                }
                const int b = bs[i];
                float r[V];
                if (b < 0) {        // padding: nothing reads it, but it stays finite
                    held = -1;
#pragma unroll
                    for (int v = 0; v < V; ++v) r[v] = 0.f;
                    store_channels<V>(out + (size_t)t * C + c, r);
                    continue;
                }
                const int slot = a.slots[b];
                if (b != held) {    // the block's first token, or another request's first token of this step
                    held = b;
                    const int t0 = a.q_start[b];
#pragma unroll
                    for (int j = 0; j < K - 1; ++j) {
                        const int src = t - (K - 1) + j;
                        if (src >= t0) {
                            float px[V];
                            load_channels<V>(a.x + (size_t)src * C + c, px);
                            if (a.branch != nullptr) {
                                float pb[V];
                                load_channels<V>(a.branch + (size_t)src * C + c, pb);
                                sum_of(src, px, pb, win[j]);
                            } else {
#pragma unroll
                                for (int v = 0; v < V; ++v) win[j][v] = px[v];
                            }
                        } else if (slot >= 0) {
                            load_channels<V>(a.state + ((size_t)slot * (K - 1) + (K - 1 + src - t0)) * C + c, win[j]);
                        } else {
#pragma unroll
                            for (int v = 0; v < V; ++v) win[j][v] = 0.f;
                        }
                    }
                }
#pragma unroll
                for (int v = 0; v < V; ++v) {
                    float acc = 0.f;
#pragma unroll
                    for (int j = 0; j < K - 1; ++j) acc = fmaf(tap[j][v], win[j][v], acc);
                    acc = fmaf(tap[K - 1][v], s[v], acc);
                    r[v] = s[v] + acc;
#pragma unroll
                    for (int j = 0; j + 1 < K - 1; ++j) win[j][v] = win[j + 1][v];
                    if (K > 1) win[K - 2 < 0 ? 0 : K - 2][v] = s[v];
                }
                store_channels<V>(out + (size_t)t * C + c, r);
                if (K > 1 && a.single && slot >= 0) {
#pragma unroll
                    for (int j = 0; j < K - 1; ++j) store_channels<V>(a.state + ((size_t)slot * (K - 1) + j) * C + c, win[j]);
                }
            }
        }
    }
}

// Any number of taps, no branch: a thread per token and channel.
template <typename TO>
__global__ void stream_conv_plain_kernel(TO* __restrict__ out, const float* __restrict__ x, const float* __restrict__ taps,
                                         const float* __restrict__ state, const int* __restrict__ req_of_token,
                                         const int* __restrict__ q_start, const int* __restrict__ slots, int C, int K) {
    const int t = blockIdx.x;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int b = req_of_token[t];
    float r = 0.f;
    if (b >= 0) {
        const int t0 = q_start[b], slot = slots[b];
        float acc = 0.f;
        for (int j = 0; j < K; ++j) {
            const int src = t - (K - 1) + j;
            float v = 0.f;
            if (src >= t0)
                v = x[(size_t)src * C + c];
            else if (slot >= 0)
                v = state[((size_t)slot * (K - 1) + (K - 1 + src - t0)) * C + c];
            acc = fmaf(taps[(size_t)c * K + j], v, acc);
        }
        r = x[(size_t)t * C + c] + acc;
    }
    out[(size_t)t * C + c] = from_f32<TO>(r);
}

template <typename TO, int V>
int launch_taps(TO* out, const StreamConvArgs& a, int K, dim3 grid, cudaStream_t stream) {
#define XB_TAPS(KV)                                                        \
    case KV:                                                               \
        stream_conv_kernel<TO, KV, V><<<grid, kThreads, 0, stream>>>(out, a); \
        return xb_launch_status();
    switch (K) {
        XB_TAPS(1) XB_TAPS(2) XB_TAPS(3) XB_TAPS(4) XB_TAPS(5) XB_TAPS(6) XB_TAPS(7) XB_TAPS(8)
        default: return (int)cudaErrorInvalidValue;
    }
#undef XB_TAPS
}
}  // namespace

XB_EXPORT int xb_stream_conv(int out_dtype, void* out, float* s_out, const float* x, const float* branch, const float* bw,
                             const float* taps, float* state, const int* req_of_token, const int* q_start, const int* slots,
                             int tokens, int C, int K, float beps, float boffset, float bscale, int single,
                             cudaStream_t stream) {
    if (tokens <= 0 || C <= 0) return 0;
    if (K < 1 || (K > 1 && state == nullptr) || (branch != nullptr && s_out == nullptr) || (bw != nullptr && branch == nullptr) ||
        s_out == x)
        return (int)cudaErrorInvalidValue;
    if (K > kMaxTaps) {
        if (branch != nullptr || single) return (int)cudaErrorInvalidValue;
        const dim3 grid(tokens, (C + 127) / 128);
        if (out_dtype == XB_F32)
            stream_conv_plain_kernel<float><<<grid, 128, 0, stream>>>((float*)out, x, taps, state, req_of_token, q_start, slots, C, K);
        else
            stream_conv_plain_kernel<__nv_bfloat16><<<grid, 128, 0, stream>>>((__nv_bfloat16*)out, x, taps, state, req_of_token,
                                                                              q_start, slots, C, K);
        return xb_launch_status();
    }
    StreamConvArgs a;
    a.s_out = s_out; a.x = x; a.branch = branch; a.bw = bw; a.taps = taps; a.state = state;
    a.req_of_token = req_of_token; a.q_start = q_start; a.slots = slots;
    a.tokens = tokens; a.C = C; a.single = single;
    a.beps = beps; a.boffset = boffset; a.bscale = bscale;
    const size_t osz = out_dtype == XB_F32 ? 16 : 8;
    const bool vec = C % 4 == 0 && !(((uintptr_t)x | (uintptr_t)branch | (uintptr_t)s_out | (uintptr_t)state | (uintptr_t)taps) & 15) &&
                     ((uintptr_t)out & (osz - 1)) == 0;
    // long runs pay for the rows before them only once, short ones fill the machine
    int run = kMaxRun;
    while (run > 1 && (tokens + run - 1) / run < 2 * 148) run /= 2;
    a.run = run;
    const int V = vec ? 4 : 1;
    // with a norm every block of a row reduces it again: one block takes all channels then, but for steps of few tokens
    const int runs = (tokens + run - 1) / run;
    int cols = (C + kThreads * V - 1) / (kThreads * V);
    if (bw != nullptr && runs >= 148) cols = 1;
    if (cols > 65535) cols = 65535;
    const dim3 grid(runs, cols);
    typedef __nv_bfloat16 bf;
    if (out_dtype == XB_F32)
        return vec ? launch_taps<float, 4>((float*)out, a, K, grid, stream) : launch_taps<float, 1>((float*)out, a, K, grid, stream);
    return vec ? launch_taps<bf, 4>((bf*)out, a, K, grid, stream) : launch_taps<bf, 1>((bf*)out, a, K, grid, stream);
}
