// Several residual streams X[0..n-1] of float32 rows in place of one (hyper-connections).  One pass over a token's rows:
//
//   X'[t] = sum_s M[s, t] X[s] + w[t] * branch          all streams at once from the old ones   (branch absent: X' = X)
//   u     = sum_t r[t] X'[t]                            (r absent: ones)
//   out   = norm ? u * rsqrt(mean(u^2) + eps) * (offset + norm) : u          in TO; out absent: only X'
//
// x_out (nullable; may be x itself when no rows are gathered) receives X'.  The streams of a row lie x_stream apart and
// its rows x_row apart, so that n equal streams can be read from one copy (x_stream 0).  A thread owns its channels in
// every stream, so writing in place needs no order; u stays in shared memory between its two uses.  The rows of M and
// the vectors are small and read before the kernel waits for the one before it.
#include "common.cuh"

namespace {
constexpr int SM_MAX_STREAMS = 32;

template <int V>
__device__ __forceinline__ void sm_load(const float* p, float (&v)[V]) {
    if (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1 % V] = t.y; v[2 % V] = t.z; v[3 % V] = t.w;
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = p[i];
    }
}
template <int V>
__device__ __forceinline__ void sm_load(const __nv_bfloat16* p, float (&v)[V]) {
    if (V == 4) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
        v[0] = a.x; v[1 % V] = a.y; v[2 % V] = b.x; v[3 % V] = b.y;
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = to_f32<__nv_bfloat16>(p[i]);
    }
}
template <int V>
__device__ __forceinline__ void sm_store(float* p, const float (&v)[V]) {
    if (V == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) p[i] = v[i];
    }
}
template <int V>
__device__ __forceinline__ void sm_store(__nv_bfloat16* p, const float (&v)[V]) {
    if (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1 % V]), b = __floats2bfloat162_rn(v[2 % V], v[3 % V]);
        uint2 t;
        t.x = *reinterpret_cast<const unsigned*>(&a);
        t.y = *reinterpret_cast<const unsigned*>(&b);
        *reinterpret_cast<uint2*>(p) = t;
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) p[i] = from_f32<__nv_bfloat16>(v[i]);
    }
}

struct StreamMixArgs {
    void* out;
    float* x_out;
    const float* x;
    long long x_row, x_stream;
    const void* branch;
    const int* rows;
    const float *read, *mix, *write, *norm;
    int n, dim, src_rows;
    float eps, offset;
    int* err;
};

// S: the number of streams, or 0: any number up to SM_MAX_STREAMS (a.n)
template <typename TB, typename TO, int S, int V>
__global__ void __launch_bounds__(1024) stream_mix_kernel(const StreamMixArgs a) {
    constexpr int CAP = S ? S : SM_MAX_STREAMS, UNROLL = S ? S : 1;
    const int n = S ? S : a.n;
    __shared__ float scratch[33];
    __shared__ float sM[CAP * CAP], sr[CAP], sw[CAP];
    extern __shared__ __align__(16) float su[];
    pdl_launch_dependents();
    for (int i = threadIdx.x; i < n * n; i += blockDim.x) sM[i] = a.branch ? a.mix[i] : 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        sr[i] = a.read ? a.read[i] : 1.f;
        sw[i] = a.branch ? a.write[i] : 0.f;
    }
    const int r = blockIdx.x;
    int src = a.rows ? a.rows[r] : r;
    if (src < 0 || src >= a.src_rows) {
        if (threadIdx.x == 0) atomicOr(a.err, XB_ERR_BAD_ROW);
        src = 0;
    }
    __syncthreads();
    pdl_wait();
    const float* xr = a.x + (size_t)src * a.x_row;
    const TB* br = a.branch ? (const TB*)a.branch + (size_t)src * a.dim : nullptr;
    float* xo = a.x_out ? a.x_out + (size_t)r * n * a.dim : nullptr;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < a.dim; i += blockDim.x * V) {
        float old[CAP][V], u[V];
#pragma unroll UNROLL
        for (int s = 0; s < CAP; ++s)
            if (s < n) sm_load<V>(xr + (size_t)s * a.x_stream + i, old[s]);
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = 0.f;
        if (br) {
            float b[V];
            sm_load<V>(br + i, b);
#pragma unroll UNROLL
            for (int t = 0; t < CAP; ++t) {
                if (t >= n) break;
                float v[V];
#pragma unroll
                for (int e = 0; e < V; ++e) v[e] = sw[t] * b[e];
#pragma unroll UNROLL
                for (int s = 0; s < CAP; ++s) {
                    if (s >= n) break;
                    const float m = sM[s * n + t];
#pragma unroll
                    for (int e = 0; e < V; ++e) v[e] = fmaf(m, old[s][e], v[e]);
                }
                if (xo) sm_store<V>(xo + (size_t)t * a.dim + i, v);
                const float rt = sr[t];
#pragma unroll
                for (int e = 0; e < V; ++e) u[e] = fmaf(rt, v[e], u[e]);
            }
        } else {
#pragma unroll UNROLL
            for (int s = 0; s < CAP; ++s) {
                if (s >= n) break;
                const float rs = sr[s];
#pragma unroll
                for (int e = 0; e < V; ++e) u[e] = fmaf(rs, old[s][e], u[e]);
                if (xo) sm_store<V>(xo + (size_t)s * a.dim + i, old[s]);
            }
        }
        sm_store<V>(su + i, u);
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(u[e], u[e], ss);
    }
    if (!a.out) return;
    float inv = 1.f;
    if (a.norm) inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)a.dim + a.eps);
    TO* o = (TO*)a.out + (size_t)r * a.dim;
    for (int i = threadIdx.x * V; i < a.dim; i += blockDim.x * V) {     // (a thread's own channels: no barrier needed)
        float u[V];
        sm_load<V>(su + i, u);
        if (a.norm) {
            float w[V];
            sm_load<V>(a.norm + i, w);
#pragma unroll
            for (int e = 0; e < V; ++e) u[e] = u[e] * inv * (a.offset + w[e]);
        }
        sm_store<V>(o + i, u);
    }
}

template <typename TB, typename TO, int V>
int stream_mix_launch(const StreamMixArgs& a, int nrows, cudaStream_t stream) {
    const size_t smem = (size_t)a.dim * sizeof(float);
    const int vecs = (a.dim + V - 1) / V;
    // as many threads as a row has accesses, up to 512 where many rows fill the machine and 1,024 where few do
    int threads = 64;
    const int most = nrows >= 2 * 148 ? 512 : 1024;
    while (threads < most && threads < vecs) threads *= 2;
    if (a.n > 8 && threads > 256) threads = 256;
#define XB_SM(SV)                                                                                                      \
    {                                                                                                                  \
        if (smem > 40 * 1024) {                                                                                        \
            const int rc = (int)cudaFuncSetAttribute(stream_mix_kernel<TB, TO, SV, V>,                                 \
                                                     cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);          \
            if (rc) return rc;                                                                                         \
        }                                                                                                              \
        return xb_launch(stream_mix_kernel<TB, TO, SV, V>, dim3(nrows), dim3(threads), smem, stream, a);               \
    }
    switch (a.n) {
        case 1: XB_SM(1)
        case 2: XB_SM(2)
        case 3: XB_SM(3)
        case 4: XB_SM(4)
        case 6: XB_SM(6)
        case 8: XB_SM(8)
        default: XB_SM(0)
    }
#undef XB_SM
}

template <typename TB, typename TO>
int stream_mix_vec(const StreamMixArgs& a, int nrows, cudaStream_t stream) {
    auto al = [](const void* p, unsigned m) { return ((uintptr_t)p & m) == 0; };
    const bool v4 = a.dim % 4 == 0 && a.x_row % 4 == 0 && a.x_stream % 4 == 0 && al(a.x, 15) && al(a.x_out, 15) &&
                    al(a.norm, 15) && al(a.branch, 4 * sizeof(TB) - 1) && al(a.out, 4 * sizeof(TO) - 1);
    return v4 ? stream_mix_launch<TB, TO, 4>(a, nrows, stream) : stream_mix_launch<TB, TO, 1>(a, nrows, stream);
}
}  // namespace

XB_EXPORT int xb_stream_mix(int branch_dtype, int out_dtype, void* out, float* x_out, const float* x, long long x_row,
                            long long x_stream, const void* branch, const int* rows, const float* read, const float* mix,
                            const float* write, const float* norm, int nrows, int n, int dim, int src_rows, float eps,
                            float offset, int* err, cudaStream_t stream) {
    if (nrows <= 0 || dim <= 0) return 0;
    if (n < 1 || n > SM_MAX_STREAMS || (size_t)dim * 4 > 200 * 1024 || (branch && (!mix || !write)) || (rows && x_out))
        return (int)cudaErrorInvalidValue;
    const StreamMixArgs a{out, x_out, x, x_row, x_stream, branch, rows, read, mix, write, norm, n, dim, src_rows, eps, offset, err};
    typedef __nv_bfloat16 bf;
    if (branch_dtype == XB_F32)
        return out_dtype == XB_F32 ? stream_mix_vec<float, float>(a, nrows, stream) : stream_mix_vec<float, bf>(a, nrows, stream);
    return out_dtype == XB_F32 ? stream_mix_vec<bf, float>(a, nrows, stream) : stream_mix_vec<bf, bf>(a, nrows, stream);
}
