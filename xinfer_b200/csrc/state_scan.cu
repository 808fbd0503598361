// Recurrences whose state is a matrix per head, carried per request in float32:
//
//   selective_scan_kernel   (state-space duality)   S[N, P]:  S <- exp(-A dt) S + dt B x^T,   y = S^T C + D x
//   delta_rule_kernel       (gated delta rule)      S[d, dv]: S <- diag(g) S,  u = beta (v - S^T k),  S <- S + k u^T,
//                                                             o = S^T q      (read after the token's own update)    
//   linear_scan_kernel      (gated linear attention)  S[d, dv]: S <- diag(alpha) S + k v^T,  o = scale S^T q
//   matrix_memory_kernel    (xLSTM's mLSTM)         S[d, dv]: S <- e^(f+m-m') S + e^(i-m') k v^T, n[d] likewise with k alone,
//                                                             o = S^T q and the divisor max(|n . q|, e^(-m')) + eps
//   low_rank_decay_kernel   alpha = sigmoid(W_a2 low + b)^(1 / tau) for it, per token and key channel
//   gated_head_norm_kernel  the gate and the RMS norm over a head (or a group of channels) behind either
//
// Layout of the scans: a block takes one (request, head) and a tile of the state's columns (columns never mix).
// Its first warps compute: a lane keeps kRows rows of two neighbouring columns in registers; DS lanes of a warp
// share a column pair and fold their sums over rows with shuffles.  Its last warps feed them: tokens of a request
// are walked in order, a tile of TT tokens at a time, and while the computing warps work on one tile the feeding
// warps bring the next one into shared memory with asynchronous copies, work out what every column needs alike
// (step sizes, decays, unit vectors, beta) once per token, and write the tile before to memory.  The step loop
// reads broadcast vectors from shared memory only.  One block barrier per tile hands the buffers over.  The state
// is read from state[slot] at the step's first token and left there after its last, so a cut between steps changes
// nothing but when the state crosses memory.  Everything is float32: decays, softplus, exponentials, step sizes,
// unit norms, gates.
#include "common.cuh"

__device__ __forceinline__ float softplus_f32(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float sigmoid_exact(float v) { return 1.f / (1.f + expf(-v)); }

namespace {
constexpr int kRows = 16;            // state rows a lane keeps per column
constexpr int kRowsPad = kRows + 4;  // the same rows in shared memory, spaced so that row groups fall on different banks
constexpr int kScanTile = 16;        // tokens per tile, at most

__device__ __forceinline__ void scan_cp4(float* dst, const float* src) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(s), "l"(src) : "memory");
}
__device__ __forceinline__ void scan_cp16(float* dst, const float* src) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(src) : "memory");
}
__device__ __forceinline__ void scan_cp_land() {
    asm volatile("cp.async.commit_group;\n" ::: "memory");
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncwarp();
}

// lanes of a warp are laid out [DS row groups][32 / DS column pairs]; the sum runs over the row groups
template <int DS>
__device__ __forceinline__ float fold_rows(float v) {
#pragma unroll
    for (int o = 16; o >= 32 / DS; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_total(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ int padded_row(int j) { return (j / kRows) * kRowsPad + (j % kRows); }

// A row vector of `len` floats (rows up to `padded` are zero) into the padded layout; `vec` says that source and
// length allow 16-byte copies.
__device__ __forceinline__ void stage_rows(float* dst, const float* src, int len, int padded, int lane, bool vec) {
    if (vec) {
        for (int j = lane * 4; j < padded; j += 128) {
            if (j < len)
                scan_cp16(dst + padded_row(j), src + j);
            else
                *reinterpret_cast<float4*>(dst + padded_row(j)) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else {
        for (int j = lane; j < padded; j += 32) {
            if (j < len)
                scan_cp4(dst + padded_row(j), src + j);
            else
                dst[padded_row(j)] = 0.f;
        }
    }
}
// The block's columns [c_base, c_base + VT) of a row of `cols` columns; the ones past the end are zero.
__device__ __forceinline__ void stage_cols(float* dst, const float* src, int c_base, int cols, int VT, int lane, bool vec) {
    if (vec) {
        for (int c = lane * 4; c < VT; c += 128) {
            if (c_base + c < cols)
                scan_cp16(dst + c, src + c_base + c);
            else
                *reinterpret_cast<float4*>(dst + c) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else {
        for (int c = lane; c < VT; c += 32) {
            if (c_base + c < cols)
                scan_cp4(dst + c, src + c_base + c);
            else
                dst[c] = 0.f;
        }
    }
}
}  // namespace

// xbc[t] = [x: H*P | B: G*N | C: G*N] after the short convolution; dt is column dt_off + h of proj[t] (before
// the bias and the softplus).  state [slots, H, N, P].  y [T, H*P].  Shared memory: two stages of
// B[TT][NP] C[TT][NP] x[TT][VT] dt[TT] dec[TT], then two tiles y[TT][VT].  `cw` of the block's warps compute.
template <int DS>
__global__ void __launch_bounds__(384, 1) selective_scan_kernel(float* __restrict__ y, const float* __restrict__ xbc, int C,
                                                             const float* __restrict__ proj, long long ldp, int dt_off,
                                                             const float* __restrict__ dt_bias,
                                                             const float* __restrict__ A_log, const float* __restrict__ Dv,
                                                             float* __restrict__ state, const int* __restrict__ q_start,
                                                             const int* __restrict__ slots, int H, int P, int N, int G,
                                                             int TT, int stage, int cw, int vec) {
    extern __shared__ __align__(16) float scan_smem[];
    constexpr int CGW = 32 / DS, NP = DS * kRowsPad, NR = DS * kRows;
    const int b = blockIdx.x, h = blockIdx.y;
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    const int VT = cw * CGW * 2, c_base = blockIdx.z * VT;
    const int slot = slots[b];
    const int t0 = q_start[b], t1 = q_start[b + 1];
    if (slot < 0 || t1 <= t0) return;
    const int inner = H * P, g = h / (H / G);
    const int ntiles = (t1 - t0 + TT - 1) / TT;
    float* sy = scan_smem + 2 * stage;
    if (w >= cw) {
        // feeding warps: warp `pi` of `pw` takes tokens pi, pi + pw, ... of every tile
        const int pi = w - cw, pw = (blockDim.x >> 5) - cw;
        const float A = expf(A_log[h]), dtb = dt_bias[h];
        auto bring = [&](int tile) {
            float* sB = scan_smem + (tile & 1) * stage;
            float* sC = sB + TT * NP;
            float* sx = sC + TT * NP;
            float* sdt = sx + TT * VT;
            const int tb = t0 + tile * TT, nt = min(TT, t1 - tb);
            for (int tt = pi; tt < nt; tt += pw) {
                const float* row = xbc + (size_t)(tb + tt) * C;
                stage_rows(sB + tt * NP, row + inner + g * N, N, NR, lane, vec);
                stage_rows(sC + tt * NP, row + inner + (G + g) * N, N, NR, lane, vec);
                stage_cols(sx + tt * VT, row + h * P, c_base, P, VT, lane, vec);
            }
            const int mine = pi + lane * pw;
            if (mine < nt) scan_cp4(sdt + mine, proj + (size_t)(tb + mine) * ldp + dt_off + h);
            scan_cp_land();
            if (mine < nt) {
                const float dt = softplus_f32(sdt[mine] + dtb);
                sdt[mine] = dt;
                sdt[TT + mine] = expf(-A * dt);
            }
        };
        auto leave = [&](int tile) {
            const float* src = sy + (tile & 1) * TT * VT;
            const int tb = t0 + tile * TT, nt = min(TT, t1 - tb);
            for (int tt = pi; tt < nt; tt += pw)
                for (int c = lane; c < VT; c += 32)
                    if (c_base + c < P) y[(size_t)(tb + tt) * inner + h * P + c_base + c] = src[tt * VT + c];
        };
        bring(0);
        __syncthreads();
        for (int tile = 0; tile < ntiles; ++tile) {
            if (tile + 1 < ntiles) bring(tile + 1);
            if (tile > 0) leave(tile - 1);
            __syncthreads();
        }
        leave(ntiles - 1);
        return;
    }
    const int ds = lane / CGW, cl = (w * CGW + lane % CGW) * 2, p0 = c_base + cl;
    const float Dh = Dv[h];
    float S0[kRows], S1[kRows];
    float* st = state + ((size_t)slot * H + h) * N * P;
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const int n = ds * kRows + r;
        S0[r] = (n < N && p0 < P) ? st[(size_t)n * P + p0] : 0.f;
        S1[r] = (n < N && p0 + 1 < P) ? st[(size_t)n * P + p0 + 1] : 0.f;
    }
    __syncthreads();
    for (int tile = 0; tile < ntiles; ++tile) {
        const float* sB = scan_smem + (tile & 1) * stage + ds * kRowsPad;
        const float* sC = sB + TT * NP;
        const float* sx = scan_smem + (tile & 1) * stage + 2 * TT * NP;
        const float* sdt = sx + TT * VT;
        sx += cl;
        float* out = sy + (tile & 1) * TT * VT + cl;
        const int nt = min(TT, t1 - t0 - tile * TT);
        for (int tt = 0; tt < nt; ++tt, sB += NP, sC += NP, sx += VT, out += VT) {
            const float dt = sdt[tt], dec = sdt[TT + tt];
            const float2 xv = *reinterpret_cast<const float2*>(sx);
            const float dx0 = dt * xv.x, dx1 = dt * xv.y;
            const float4* Bp = reinterpret_cast<const float4*>(sB);
            const float4* Cp = reinterpret_cast<const float4*>(sC);
            float a0 = 0.f, a1 = 0.f;
#pragma unroll
            for (int i = 0; i < kRows / 4; ++i) {
                const float4 bv = Bp[i], cv = Cp[i];
                const float bq[4] = {bv.x, bv.y, bv.z, bv.w}, cq[4] = {cv.x, cv.y, cv.z, cv.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    S0[4 * i + e] = fmaf(dec, S0[4 * i + e], bq[e] * dx0);
                    S1[4 * i + e] = fmaf(dec, S1[4 * i + e], bq[e] * dx1);
                    a0 = fmaf(S0[4 * i + e], cq[e], a0);
                    a1 = fmaf(S1[4 * i + e], cq[e], a1);
                }
            }
            a0 = fold_rows<DS>(a0);
            a1 = fold_rows<DS>(a1);
            if (ds == 0) *reinterpret_cast<float2*>(out) = make_float2(fmaf(Dh, xv.x, a0), fmaf(Dh, xv.y, a1));
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const int n = ds * kRows + r;
        if (n < N && p0 < P) st[(size_t)n * P + p0] = S0[r];
        if (n < N && p0 + 1 < P) st[(size_t)n * P + p0 + 1] = S1[r];
    }
}

// qkv[t] = [q: G*d | k: G*d | v: H*dv] after the short convolution; beta is column beta_off + h of proj[t] before
// the sigmoid; ag[t] holds the decay's pre-activation for (head, key channel) at its front.  q and k become unit
// vectors over a head (q also times d^-1/2); g = exp(-exp(A_log_h) softplus(a + dt_bias)) per (head, key channel).
// state [slots, H, d, dv].  o [T, H*dv].  Shared memory: two stages of q[TT][DP] k[TT][DP] g[TT][DP] v[TT][VT]
// beta[TT] kq[TT], then two tiles o[TT][VT].  With gS the decayed state, o = (gS)^T q + u (k . q).
template <int DS>
__global__ void __launch_bounds__(384, 1) delta_rule_kernel(float* __restrict__ o, const float* __restrict__ qkv, int Cq,
                                                         const float* __restrict__ proj, long long ldp, int beta_off,
                                                         const float* __restrict__ ag, long long ldag,
                                                         const float* __restrict__ dt_bias, const float* __restrict__ A_log,
                                                         float* __restrict__ state, const int* __restrict__ q_start,
                                                         const int* __restrict__ slots, int H, int G, int d, int dv,
                                                         float unit_eps, int TT, int stage, int cw, int vec) {
    extern __shared__ __align__(16) float scan_smem[];
    constexpr int CGW = 32 / DS, DP = DS * kRowsPad, NR = DS * kRows;
    const int b = blockIdx.x, h = blockIdx.y;
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    const int VT = cw * CGW * 2, c_base = blockIdx.z * VT;
    const int slot = slots[b];
    const int t0 = q_start[b], t1 = q_start[b + 1];
    if (slot < 0 || t1 <= t0) return;
    const int kvh = h / (H / G);
    const int ntiles = (t1 - t0 + TT - 1) / TT;
    float* so = scan_smem + 2 * stage;
    if (w >= cw) {
        // feeding warps: warp `pi` of `pw` takes tokens pi, pi + pw, ... of every tile
        const int pi = w - cw, pw = (blockDim.x >> 5) - cw;
        const float A = expf(A_log[h]);
        const float qk_scale = 1.f / sqrtf((float)d);
        const float* bias = dt_bias + (size_t)h * d;
        auto bring = [&](int tile) {
            float* sq = scan_smem + (tile & 1) * stage;
            float* sk = sq + TT * DP;
            float* sg = sk + TT * DP;
            float* sv = sg + TT * DP;
            float* sbeta = sv + TT * VT;
            const int tb = t0 + tile * TT, nt = min(TT, t1 - tb);
            for (int tt = pi; tt < nt; tt += pw) {
                const float* row = qkv + (size_t)(tb + tt) * Cq;
                stage_rows(sq + tt * DP, row + kvh * d, d, NR, lane, vec);
                stage_rows(sk + tt * DP, row + (G + kvh) * d, d, NR, lane, vec);
                stage_rows(sg + tt * DP, ag + (size_t)(tb + tt) * ldag + h * d, d, NR, lane, vec);
                stage_cols(sv + tt * VT, row + 2 * G * d + h * dv, c_base, dv, VT, lane, vec);
                if (lane == 0) scan_cp4(sbeta + tt, proj + (size_t)(tb + tt) * ldp + beta_off + h);
            }
            scan_cp_land();
            for (int tt = pi; tt < nt; tt += pw) {
                float* q = sq + tt * DP;
                float* k = sk + tt * DP;
                float* gd = sg + tt * DP;
                float qq = 0.f, kk = 0.f;
                for (int j = lane; j < d; j += 32) {
                    const int at = padded_row(j);
                    qq = fmaf(q[at], q[at], qq);
                    kk = fmaf(k[at], k[at], kk);
                }
                qq = warp_total(qq);
                kk = warp_total(kk);
                const float qs = qk_scale / sqrtf(qq + unit_eps), ks = 1.f / sqrtf(kk + unit_eps);
                float kq = 0.f;
                for (int j = lane; j < d; j += 32) {
                    const int at = padded_row(j);
                    const float qn = q[at] * qs, kn = k[at] * ks;
                    q[at] = qn;
                    k[at] = kn;
                    kq = fmaf(kn, qn, kq);
                    gd[at] = expf(-A * softplus_f32(gd[at] + bias[j]));
                }
                kq = warp_total(kq);
                if (lane == 0) {
                    sbeta[TT + tt] = kq;
                    sbeta[tt] = sigmoid_exact(sbeta[tt]);
                }
            }
        };
        auto leave = [&](int tile) {
            const float* src = so + (tile & 1) * TT * VT;
            const int tb = t0 + tile * TT, nt = min(TT, t1 - tb);
            for (int tt = pi; tt < nt; tt += pw)
                for (int c = lane; c < VT; c += 32)
                    if (c_base + c < dv) o[((size_t)(tb + tt) * H + h) * dv + c_base + c] = src[tt * VT + c];
        };
        bring(0);
        __syncthreads();
        for (int tile = 0; tile < ntiles; ++tile) {
            if (tile + 1 < ntiles) bring(tile + 1);
            if (tile > 0) leave(tile - 1);
            __syncthreads();
        }
        leave(ntiles - 1);
        return;
    }
    const int ds = lane / CGW, cl = (w * CGW + lane % CGW) * 2, v0 = c_base + cl;
    float S0[kRows], S1[kRows];
    float* st = state + ((size_t)slot * H + h) * d * dv;
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const int j = ds * kRows + r;
        S0[r] = (j < d && v0 < dv) ? st[(size_t)j * dv + v0] : 0.f;
        S1[r] = (j < d && v0 + 1 < dv) ? st[(size_t)j * dv + v0 + 1] : 0.f;
    }
    __syncthreads();
    for (int tile = 0; tile < ntiles; ++tile) {
        const float* sq = scan_smem + (tile & 1) * stage + ds * kRowsPad;
        const float* sk = sq + TT * DP;
        const float* sg = sk + TT * DP;
        const float* sv = scan_smem + (tile & 1) * stage + 3 * TT * DP;
        const float* sbeta = sv + TT * VT;
        sv += cl;
        float* out = so + (tile & 1) * TT * VT + cl;
        const int nt = min(TT, t1 - t0 - tile * TT);
        for (int tt = 0; tt < nt; ++tt, sq += DP, sk += DP, sg += DP, sv += VT, out += VT) {
            const float beta = sbeta[tt], kq = sbeta[TT + tt];
            const float2 vv = *reinterpret_cast<const float2*>(sv);
            const float4* qp = reinterpret_cast<const float4*>(sq);
            const float4* kp = reinterpret_cast<const float4*>(sk);
            const float4* gp = reinterpret_cast<const float4*>(sg);
            float kr[kRows];
            float a10 = 0.f, a11 = 0.f, a20 = 0.f, a21 = 0.f;
#pragma unroll
            for (int i = 0; i < kRows / 4; ++i) {
                const float4 g4 = gp[i], k4 = kp[i], q4 = qp[i];
                const float gq[4] = {g4.x, g4.y, g4.z, g4.w}, kq4[4] = {k4.x, k4.y, k4.z, k4.w};
                const float qq4[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = 4 * i + e;
                    S0[r] *= gq[e];
                    S1[r] *= gq[e];
                    a10 = fmaf(S0[r], kq4[e], a10);
                    a11 = fmaf(S1[r], kq4[e], a11);
                    a20 = fmaf(S0[r], qq4[e], a20);
                    a21 = fmaf(S1[r], qq4[e], a21);
                    kr[r] = kq4[e];
                }
            }
            a10 = fold_rows<DS>(a10);
            a11 = fold_rows<DS>(a11);
            a20 = fold_rows<DS>(a20);
            a21 = fold_rows<DS>(a21);
            const float u0 = beta * (vv.x - a10), u1 = beta * (vv.y - a11);
#pragma unroll
            for (int r = 0; r < kRows; ++r) {
                S0[r] = fmaf(kr[r], u0, S0[r]);
                S1[r] = fmaf(kr[r], u1, S1[r]);
            }
            if (ds == 0) *reinterpret_cast<float2*>(out) = make_float2(fmaf(u0, kq, a20), fmaf(u1, kq, a21));
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const int j = ds * kRows + r;
        if (j < d && v0 < dv) st[(size_t)j * dv + v0] = S0[r];
        if (j < d && v0 + 1 < dv) st[(size_t)j * dv + v0 + 1] = S1[r];
    }
}

// proj[t] holds q (H*d from column 0), k (H*d behind it) and v (H*dv behind that) of a token; alpha[t] the decay of
// every (head, key channel).  state [slots, H, d, dv].  o [T, H*dv] = scale * S^T q after the token's own write.  Shared
// memory: two stages of q[TT][DP] k[TT][DP] alpha[TT][DP] v[TT][VT], then two tiles o[TT][VT].
template <int DS>
__global__ void __launch_bounds__(384, 1) linear_scan_kernel(float* __restrict__ o, const float* __restrict__ proj,
                                                             long long ldp, const float* __restrict__ alpha,
                                                             float* __restrict__ state, const int* __restrict__ q_start,
                                                             const int* __restrict__ slots, int H, int d, int dv, float scale,
                                                             int TT, int stage, int cw, int vec) {
    extern __shared__ __align__(16) float scan_smem[];
    constexpr int CGW = 32 / DS, DP = DS * kRowsPad, NR = DS * kRows;
    const int b = blockIdx.x, h = blockIdx.y;
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    const int VT = cw * CGW * 2, c_base = blockIdx.z * VT;
    const int slot = slots[b];
    const int t0 = q_start[b], t1 = q_start[b + 1];
    if (slot < 0 || t1 <= t0) return;
    const int ntiles = (t1 - t0 + TT - 1) / TT;
    float* so = scan_smem + 2 * stage;
    if (w >= cw) {
        // feeding warps: warp `pi` of `pw` takes tokens pi, pi + pw, ... of every tile
        const int pi = w - cw, pw = (blockDim.x >> 5) - cw;
        auto bring = [&](int tile) {
            float* sq = scan_smem + (tile & 1) * stage;
            float* sk = sq + TT * DP;
            float* sa = sk + TT * DP;
            float* sv = sa + TT * DP;
            const int tb = t0 + tile * TT, nt = min(TT, t1 - tb);
            for (int tt = pi; tt < nt; tt += pw) {
                const float* row = proj + (size_t)(tb + tt) * ldp;
                stage_rows(sq + tt * DP, row + h * d, d, NR, lane, vec);
                stage_rows(sk + tt * DP, row + (H + h) * d, d, NR, lane, vec);
                stage_rows(sa + tt * DP, alpha + ((size_t)(tb + tt) * H + h) * d, d, NR, lane, vec);
                stage_cols(sv + tt * VT, row + 2 * H * d + h * dv, c_base, dv, VT, lane, vec);
            }
            scan_cp_land();
        };
        auto leave = [&](int tile) {
            const float* src = so + (tile & 1) * TT * VT;
            const int tb = t0 + tile * TT, nt = min(TT, t1 - tb);
            for (int tt = pi; tt < nt; tt += pw)
                for (int c = lane; c < VT; c += 32)
                    if (c_base + c < dv) o[((size_t)(tb + tt) * H + h) * dv + c_base + c] = src[tt * VT + c];
        };
        bring(0);
        __syncthreads();
        for (int tile = 0; tile < ntiles; ++tile) {
            if (tile + 1 < ntiles) bring(tile + 1);
            if (tile > 0) leave(tile - 1);
            __syncthreads();
        }
        leave(ntiles - 1);
        return;
    }
    const int ds = lane / CGW, cl = (w * CGW + lane % CGW) * 2, v0 = c_base + cl;
    float S0[kRows], S1[kRows];
    float* st = state + ((size_t)slot * H + h) * d * dv;
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const int j = ds * kRows + r;
        S0[r] = (j < d && v0 < dv) ? st[(size_t)j * dv + v0] : 0.f;
        S1[r] = (j < d && v0 + 1 < dv) ? st[(size_t)j * dv + v0 + 1] : 0.f;
    }
    __syncthreads();
    for (int tile = 0; tile < ntiles; ++tile) {
        const float* sq = scan_smem + (tile & 1) * stage + ds * kRowsPad;
        const float* sk = sq + TT * DP;
        const float* sa = sk + TT * DP;
        const float* sv = scan_smem + (tile & 1) * stage + 3 * TT * DP + cl;
        float* out = so + (tile & 1) * TT * VT + cl;
        const int nt = min(TT, t1 - t0 - tile * TT);
        for (int tt = 0; tt < nt; ++tt, sq += DP, sk += DP, sa += DP, sv += VT, out += VT) {
            const float2 vv = *reinterpret_cast<const float2*>(sv);
            const float4* qp = reinterpret_cast<const float4*>(sq);
            const float4* kp = reinterpret_cast<const float4*>(sk);
            const float4* ap = reinterpret_cast<const float4*>(sa);
            float a0 = 0.f, a1 = 0.f;
#pragma unroll
            for (int i = 0; i < kRows / 4; ++i) {
                const float4 q4 = qp[i], k4 = kp[i], g4 = ap[i];
                const float qq[4] = {q4.x, q4.y, q4.z, q4.w}, kq[4] = {k4.x, k4.y, k4.z, k4.w};
                const float gq[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = 4 * i + e;
                    S0[r] = fmaf(gq[e], S0[r], kq[e] * vv.x);
                    S1[r] = fmaf(gq[e], S1[r], kq[e] * vv.y);
                    a0 = fmaf(S0[r], qq[e], a0);
                    a1 = fmaf(S1[r], qq[e], a1);
                }
            }
            a0 = fold_rows<DS>(a0);
            a1 = fold_rows<DS>(a1);
            if (ds == 0) *reinterpret_cast<float2*>(out) = make_float2(scale * a0, scale * a1);
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const int j = ds * kRows + r;
        if (j < d && v0 < dv) st[(size_t)j * dv + v0] = S0[r];
        if (j < d && v0 + 1 < dv) st[(size_t)j * dv + v0 + 1] = S1[r];
    }
}

// proj[t] holds q (H*d from column 0), k (H*d behind it), v (H*dv behind that) and at gate_off the input gates' and the
// forget gates' pre-activations (H each, without their biases).  With i = cap tanh((z_i + b_i) / cap) and
// f = -softplus(-cap tanh((z_f + b_f) / cap)):
//   m' = max(f + m, i);  a = e^(f + m - m');  b = e^(i - m');   S <- a S + b k v^T;   n <- a n + b k
//   o[t, h*dv ..] = scale S^T q,   div[t, h] = max(|scale n . q|, e^(-m')) + div_eps          after the token's own write
// state_s [slots, H, d, dv], state_n [slots, H, d].  The running maximum m is read by every block of a head but left by
// one of them, so it has two places: state_m [slots, H, 2, 2] holds (tokens it stands behind, m) twice; a step reads the
// place that stands behind its start and writes the other one.  Zeros are a request's start.
// Shared memory: two stages of q[TT][DP] k[TT][DP] v[TT][VT] a[TT] b[TT] e^(-m')[TT], then two tiles o[TT][VT].  Besides
// the computing and the feeding warps there is one (warp `cw`) that carries n where the block has the head's first
// columns; the first feeding warp works out the gates, a lane per token, and walks m over the tile.
template <int DS>
__global__ void __launch_bounds__(384, 1) matrix_memory_kernel(
    float* __restrict__ o, float* __restrict__ div, const float* __restrict__ proj, long long ldp, int gate_off,
    const float* __restrict__ bi, const float* __restrict__ bf, float cap, float* __restrict__ state_s,
    float* __restrict__ state_n, float* state_m, const int* __restrict__ q_start, const int* __restrict__ start_pos,
    const int* __restrict__ slots, int H, int d, int dv, float scale, float div_eps, int TT, int stage, int cw, int vec) {
    extern __shared__ __align__(16) float scan_smem[];
    constexpr int CGW = 32 / DS, DP = DS * kRowsPad, NR = DS * kRows;
    const int b = blockIdx.x, h = blockIdx.y;
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    const int VT = cw * CGW * 2, c_base = blockIdx.z * VT;
    const int slot = slots[b];
    const int t0 = q_start[b], t1 = q_start[b + 1];
    if (slot < 0 || t1 <= t0) return;
    const int ntiles = (t1 - t0 + TT - 1) / TT;
    float* so = scan_smem + 2 * stage;
    if (w > cw) {
        // feeding warps: warp `pi` of `pw` takes tokens pi, pi + pw, ... of every tile
        const int pi = w - cw - 1, pw = (blockDim.x >> 5) - cw - 1;
        float* place = state_m + ((size_t)slot * H + h) * 4;
        const float at_start = (float)start_pos[b];
        const int from = place[0] == at_start ? 0 : 1;
        float m = place[2 * from + 1];
        const float b_i = bi[h], b_f = bf[h];
        auto bring = [&](int tile) {
            float* sq = scan_smem + (tile & 1) * stage;
            float* sk = sq + TT * DP;
            float* sv = sk + TT * DP;
            float* sg = sv + TT * VT;
            const int tb = t0 + tile * TT, nt = min(TT, t1 - tb);
            float zi = 0.f, zf = 0.f;
            if (pi == 0 && lane < nt) {
                const float* g = proj + (size_t)(tb + lane) * ldp + gate_off + h;
                zi = g[0];
                zf = g[H];
            }
            for (int tt = pi; tt < nt; tt += pw) {
                const float* row = proj + (size_t)(tb + tt) * ldp;
                stage_rows(sq + tt * DP, row + h * d, d, NR, lane, vec);
                stage_rows(sk + tt * DP, row + (H + h) * d, d, NR, lane, vec);
                stage_cols(sv + tt * VT, row + 2 * H * d + h * dv, c_base, dv, VT, lane, vec);
            }
            if (pi == 0) {
                const float gi = cap * tanhf((zi + b_i) / cap), y = cap * tanhf((zf + b_f) / cap);
                const float gf = fminf(y, 0.f) - log1pf(expf(-fabsf(y)));      // log of the sigmoid
                float before = m, after = m;
                for (int tt = 0; tt < nt; ++tt) {
                    const float f_t = __shfl_sync(0xffffffffu, gf, tt), i_t = __shfl_sync(0xffffffffu, gi, tt);
                    const float next = fmaxf(f_t + m, i_t);
                    if (lane == tt) {
                        before = m;
                        after = next;
                    }
                    m = next;
                }
                if (lane < nt) {
                    sg[lane] = expf(gf + before - after);
                    sg[TT + lane] = expf(gi - after);
                    sg[2 * TT + lane] = expf(-after);
                }
            }
            scan_cp_land();
        };
        auto leave = [&](int tile) {
            const float* src = so + (tile & 1) * TT * VT;
            const int tb = t0 + tile * TT, nt = min(TT, t1 - tb);
            for (int tt = pi; tt < nt; tt += pw)
                for (int c = lane; c < VT; c += 32)
                    if (c_base + c < dv) o[((size_t)(tb + tt) * H + h) * dv + c_base + c] = src[tt * VT + c];
        };
        bring(0);
        __syncthreads();
        for (int tile = 0; tile < ntiles; ++tile) {
            if (tile + 1 < ntiles) bring(tile + 1);
            if (tile > 0) leave(tile - 1);
            __syncthreads();
        }
        leave(ntiles - 1);
        if (pi == 0 && lane == 0 && blockIdx.z == 0) {
            place[2 * (from ^ 1)] = at_start + (float)(t1 - t0);
            place[2 * (from ^ 1) + 1] = m;
        }
        return;
    }
    if (w == cw) {
        // n and the divisors; a lane keeps rows lane, lane + 32, ...
        constexpr int NN = (NR + 31) / 32;
        const bool mine = blockIdx.z == 0;
        float n[NN];
        float* sn = state_n + ((size_t)slot * H + h) * d;
#pragma unroll
        for (int r = 0; r < NN; ++r) n[r] = mine && lane + 32 * r < d ? sn[lane + 32 * r] : 0.f;
        __syncthreads();
        for (int tile = 0; tile < ntiles; ++tile) {
            if (mine) {
                const float* sq = scan_smem + (tile & 1) * stage;
                const float* sk = sq + TT * DP;
                const float* sg = scan_smem + (tile & 1) * stage + 2 * TT * DP + TT * VT;
                const int nt = min(TT, t1 - t0 - tile * TT);
                float* dst = div + (size_t)(t0 + tile * TT) * H + h;
#pragma unroll 4
                for (int tt = 0; tt < nt; ++tt) {
                    const float a = sg[tt], bb = sg[TT + tt];
                    float acc = 0.f;
#pragma unroll
                    for (int r = 0; r < NN; ++r) {
                        if (lane + 32 * r >= NR) break;
                        const int at = tt * DP + padded_row(lane + 32 * r);
                        n[r] = fmaf(a, n[r], bb * sk[at]);
                        acc = fmaf(n[r], sq[at], acc);
                    }
                    acc = warp_total(acc);
                    if (lane == 0) dst[(size_t)tt * H] = fmaxf(fabsf(scale * acc), sg[2 * TT + tt]) + div_eps;
                }
            }
            __syncthreads();
        }
#pragma unroll
        for (int r = 0; r < NN; ++r)
            if (mine && lane + 32 * r < d) sn[lane + 32 * r] = n[r];
        return;
    }
    const int ds = lane / CGW, cl = (w * CGW + lane % CGW) * 2, v0 = c_base + cl;
    float S0[kRows], S1[kRows];
    float* st = state_s + ((size_t)slot * H + h) * d * dv;
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const int j = ds * kRows + r;
        S0[r] = (j < d && v0 < dv) ? st[(size_t)j * dv + v0] : 0.f;
        S1[r] = (j < d && v0 + 1 < dv) ? st[(size_t)j * dv + v0 + 1] : 0.f;
    }
    __syncthreads();
    for (int tile = 0; tile < ntiles; ++tile) {
        const float* sq = scan_smem + (tile & 1) * stage + ds * kRowsPad;
        const float* sk = sq + TT * DP;
        const float* sv = scan_smem + (tile & 1) * stage + 2 * TT * DP;
        const float* sg = sv + TT * VT;
        sv += cl;
        float* out = so + (tile & 1) * TT * VT + cl;
        const int nt = min(TT, t1 - t0 - tile * TT);
        for (int tt = 0; tt < nt; ++tt, sq += DP, sk += DP, sv += VT, out += VT) {
            const float dec = sg[tt], in = sg[TT + tt];
            const float2 vv = *reinterpret_cast<const float2*>(sv);
            const float w0 = in * vv.x, w1 = in * vv.y;
            const float4* qp = reinterpret_cast<const float4*>(sq);
            const float4* kp = reinterpret_cast<const float4*>(sk);
            float a0 = 0.f, a1 = 0.f;
#pragma unroll
            for (int i = 0; i < kRows / 4; ++i) {
                const float4 q4 = qp[i], k4 = kp[i];
                const float qq[4] = {q4.x, q4.y, q4.z, q4.w}, kq[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = 4 * i + e;
                    S0[r] = fmaf(dec, S0[r], kq[e] * w0);
                    S1[r] = fmaf(dec, S1[r], kq[e] * w1);
                    a0 = fmaf(S0[r], qq[e], a0);
                    a1 = fmaf(S1[r], qq[e], a1);
                }
            }
            a0 = fold_rows<DS>(a0);
            a1 = fold_rows<DS>(a1);
            if (ds == 0) *reinterpret_cast<float2*>(out) = make_float2(scale * a0, scale * a1);
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
        const int j = ds * kRows + r;
        if (j < d && v0 < dv) st[(size_t)j * dv + v0] = S0[r];
        if (j < d && v0 + 1 < dv) st[(size_t)j * dv + v0 + 1] = S1[r];
    }
}

// alpha[t, c] = sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau),  z = bias[c] + sum_r w[c, r] low[t, r].  low is a
// column range of wider float32 rows.  A block takes a tile of tokens and 128 channels, a thread one channel of all its
// tokens; both operands pass through shared memory, so that memory is read in order; r in order for every output.
constexpr int kDecayTokens = 16, kDecayRanks = 16, kDecayChannels = 128;
__global__ void __launch_bounds__(kDecayChannels) low_rank_decay_kernel(float* __restrict__ alpha, const float* __restrict__ low,
                                                                        long long ldl, const float* __restrict__ w,
                                                                        const float* __restrict__ bias, int tokens, int C, int R,
                                                                        float inv_tau) {
    __shared__ __align__(16) float sl[kDecayRanks][kDecayTokens];
    __shared__ float sw[kDecayRanks][kDecayChannels + 1];
    const int tb = blockIdx.x * kDecayTokens, nt = min(kDecayTokens, tokens - tb);
    const int c0 = blockIdx.y * kDecayChannels, c = c0 + threadIdx.x;
    float z[kDecayTokens];
    const float b = c < C ? bias[c] : 0.f;
#pragma unroll
    for (int i = 0; i < kDecayTokens; ++i) z[i] = b;
    for (int r0 = 0; r0 < R; r0 += kDecayRanks) {
        if (r0 > 0) __syncthreads();
        for (int i = threadIdx.x; i < kDecayRanks * kDecayTokens; i += kDecayChannels) {
            const int tt = i / kDecayRanks, r = i % kDecayRanks;
            sl[r][tt] = (tt < nt && r0 + r < R) ? low[(size_t)(tb + tt) * ldl + r0 + r] : 0.f;
        }
        for (int i = threadIdx.x; i < kDecayRanks * kDecayChannels; i += kDecayChannels) {
            const int cc = i / kDecayRanks, r = i % kDecayRanks;
            sw[r][cc] = (c0 + cc < C && r0 + r < R) ? w[(size_t)(c0 + cc) * R + r0 + r] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < kDecayRanks; ++r) {
            const float wv = sw[r][threadIdx.x];
#pragma unroll
            for (int i = 0; i < kDecayTokens; i += 4) {
                const float4 l4 = *reinterpret_cast<const float4*>(&sl[r][i]);
                z[i] = fmaf(wv, l4.x, z[i]);
                z[i + 1] = fmaf(wv, l4.y, z[i + 1]);
                z[i + 2] = fmaf(wv, l4.z, z[i + 2]);
                z[i + 3] = fmaf(wv, l4.w, z[i + 3]);
            }
        }
    }
    if (c >= C) return;
#pragma unroll
    for (int i = 0; i < kDecayTokens; ++i)
        if (i < nt) {
            const float sp = fmaxf(-z[i], 0.f) + log1pf(expf(-fabsf(z[i])));      // softplus(-z), for any z without a branch
            alpha[(size_t)(tb + i) * C + c] = expf(-sp * inv_tau);
        }
}

// Row groups per column pair: the smallest power of two with DS * kRows >= rows.
static inline int scan_row_groups(int rows) {
    int ds = 1;
    while (ds * kRows < rows) ds *= 2;
    return ds;
}

// Computing warps per block: enough to cover the columns (at most 8), fewer (down to 2) while the grid would
// leave a third of the processors idle.  Every block of a head repeats the feeding warps' work, so column tiles
// are not cut finer than that.
static inline int scan_warps(int cols, int ds, long long heads_total) {
    const int per_warp = (32 / ds) * 2;
    int warps = 1;
    while (warps < 8 && warps * per_warp < cols) warps *= 2;
    while (warps > 2 && heads_total * ((cols + warps * per_warp - 1) / (warps * per_warp)) < 100) warps /= 2;
    return warps;
}

static inline bool scan_aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

// Floats of one stage (`vectors` row vectors and a few scalars per token beside the column tile), rounded so that
// the second stage stays 16-byte aligned; the tile shrinks until two stages and two output tiles fit.
static inline void scan_tile(int vectors, int ds, int vt, int& tt, int& stage, size_t& bytes, int scalars = 2) {
    for (tt = kScanTile;; tt /= 2) {
        stage = (tt * (vectors * ds * kRowsPad + vt + scalars) + 3) & ~3;
        bytes = ((size_t)2 * stage + (size_t)2 * tt * vt) * sizeof(float);
        if (bytes <= 200 * 1024 || tt == 1) return;
    }
}

template <typename K>
static inline int scan_smem_opt_in(K kernel, size_t bytes) {
    if (bytes <= 48 * 1024) return 0;
    return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

#define XB_SCAN_DISPATCH(KERNEL, DSV, ...)                                                       \
    switch (DSV) {                                                                              \
        case 1: XB_SCAN_LAUNCH(KERNEL<1>, __VA_ARGS__) break;                                   \
        case 2: XB_SCAN_LAUNCH(KERNEL<2>, __VA_ARGS__) break;                                   \
        case 4: XB_SCAN_LAUNCH(KERNEL<4>, __VA_ARGS__) break;                                   \
        case 8: XB_SCAN_LAUNCH(KERNEL<8>, __VA_ARGS__) break;                                   \
        case 16: XB_SCAN_LAUNCH(KERNEL<16>, __VA_ARGS__) break;                                 \
        default: XB_SCAN_LAUNCH(KERNEL<32>, __VA_ARGS__) break;                                 \
    }
#define XB_SCAN_LAUNCH(K, ...)                                  \
    {                                                           \
        const int rc = scan_smem_opt_in(K, bytes);              \
        if (rc) return rc;                                      \
        K<<<grid, threads, bytes, stream>>>(__VA_ARGS__);       \
    }

XB_EXPORT int xb_selective_scan(float* y, const float* xbc, int C, const float* proj, long long ldp, int dt_off,
                                const float* dt_bias, const float* A_log, const float* Dv, float* state, const int* q_start,
                                const int* slots, int entries, int H, int P, int N, int G, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (N < 1 || N > 32 * kRows || P < 1 || G < 1 || H % G || H > 65535) return (int)cudaErrorInvalidValue;
    const int ds = scan_row_groups(N);
    const int warps = scan_warps(P, ds, (long long)entries * H);
    const int vt = warps * (32 / ds) * 2;
    int tt, stage;
    size_t bytes;
    scan_tile(2, ds, vt, tt, stage, bytes);
    const dim3 grid(entries, H, (P + vt - 1) / vt);
    const int threads = (warps + 4) * 32;  // four feeding warps
    const int vec = scan_aligned16(xbc) && C % 4 == 0 && P % 4 == 0 && N % 4 == 0 && vt % 4 == 0;
    XB_SCAN_DISPATCH(selective_scan_kernel, ds, y, xbc, C, proj, ldp, dt_off, dt_bias, A_log, Dv, state, q_start, slots, H, P, N,
                     G, tt, stage, warps, vec)
    return xb_launch_status();
}

XB_EXPORT int xb_delta_rule(float* o, const float* qkv, int Cq, const float* proj, long long ldp, int beta_off, const float* ag,
                            long long ldag, const float* dt_bias, const float* A_log, float* state, const int* q_start,
                            const int* slots, int entries, int H, int G, int d, int dv, float unit_eps, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (d < 1 || d > 32 * kRows || dv < 1 || G < 1 || H % G || H > 65535) return (int)cudaErrorInvalidValue;
    const int ds = scan_row_groups(d);
    const int warps = scan_warps(dv, ds, (long long)entries * H);
    const int vt = warps * (32 / ds) * 2;
    int tt, stage;
    size_t bytes;
    scan_tile(3, ds, vt, tt, stage, bytes);
    const dim3 grid(entries, H, (dv + vt - 1) / vt);
    // the unit vectors and decays are the feeding warps' work: eight of them where the block has room, else four
    const int threads = (warps + (warps <= 4 ? 8 : 4)) * 32;
    const int vec = scan_aligned16(qkv) && scan_aligned16(ag) && Cq % 4 == 0 && ldag % 4 == 0 && d % 4 == 0 && dv % 4 == 0 &&
                    vt % 4 == 0;
    XB_SCAN_DISPATCH(delta_rule_kernel, ds, o, qkv, Cq, proj, ldp, beta_off, ag, ldag, dt_bias, A_log, state, q_start, slots, H,
                     G, d, dv, unit_eps, tt, stage, warps, vec)
    return xb_launch_status();
}

XB_EXPORT int xb_linear_scan(float* o, const float* proj, long long ldp, const float* alpha, float* state, const int* q_start,
                             const int* slots, int entries, int H, int d, int dv, float scale, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (d < 1 || d > 32 * kRows || dv < 1 || H < 1 || H > 65535) return (int)cudaErrorInvalidValue;
    const int ds = scan_row_groups(d);
    const int warps = scan_warps(dv, ds, (long long)entries * H);
    const int vt = warps * (32 / ds) * 2;
    int tt, stage;
    size_t bytes;
    scan_tile(3, ds, vt, tt, stage, bytes);
    const dim3 grid(entries, H, (dv + vt - 1) / vt);
    const int threads = (warps + 4) * 32;  // four feeding warps: they only copy
    const int vec = scan_aligned16(proj) && scan_aligned16(alpha) && ldp % 4 == 0 && d % 4 == 0 && dv % 4 == 0 && vt % 4 == 0;
    XB_SCAN_DISPATCH(linear_scan_kernel, ds, o, proj, ldp, alpha, state, q_start, slots, H, d, dv, scale, tt, stage, warps, vec)
    return xb_launch_status();
}

XB_EXPORT int xb_matrix_memory(float* o, float* div, const float* proj, long long ldp, int gate_off, const float* bi,
                               const float* bf, float cap, float* state_s, float* state_n, float* state_m, const int* q_start,
                               const int* start_pos, const int* slots, int entries, int H, int d, int dv, float scale,
                               float div_eps, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (d < 1 || d > 32 * kRows || dv < 1 || H < 1 || H > 65535 || !(cap > 0.f)) return (int)cudaErrorInvalidValue;
    const int ds = scan_row_groups(d);
    const int warps = scan_warps(dv, ds, (long long)entries * H);
    const int vt = warps * (32 / ds) * 2;
    int tt, stage;
    size_t bytes;
    scan_tile(2, ds, vt, tt, stage, bytes, 3);
    const dim3 grid(entries, H, (dv + vt - 1) / vt);
    const int threads = (warps + 1 + (warps == 8 ? 3 : 4)) * 32;   // the warp of n, then three or four feeding warps
    const int vec = scan_aligned16(proj) && ldp % 4 == 0 && d % 4 == 0 && dv % 4 == 0 && vt % 4 == 0;
    XB_SCAN_DISPATCH(matrix_memory_kernel, ds, o, div, proj, ldp, gate_off, bi, bf, cap, state_s, state_n, state_m, q_start,
                     start_pos, slots, H, d, dv, scale, div_eps, tt, stage, warps, vec)
    return xb_launch_status();
}

XB_EXPORT int xb_low_rank_decay(float* alpha, const float* low, long long ldl, const float* w, const float* bias, int tokens,
                                int C, int R, float tau, cudaStream_t stream) {
    if (tokens <= 0 || C <= 0) return 0;
    const int cols = (C + kDecayChannels - 1) / kDecayChannels;
    if (R < 1 || !(tau > 0.f) || cols > 65535) return (int)cudaErrorInvalidValue;
    const dim3 grid((tokens + kDecayTokens - 1) / kDecayTokens, cols);
    low_rank_decay_kernel<<<grid, kDecayChannels, 0, stream>>>(alpha, low, ldl, w, bias, tokens, C, R, 1.f / tau);
    return xb_launch_status();
}

// One block per (token, group of `part` consecutive channels of the W):
//   mode 0:  v = y * silu(gate);  out = v * rsqrt(mean(v^2) + eps) * w[c mod w_len]          (gate before the norm)
//   mode 1:  out = y * rsqrt(mean(y^2) + eps) * w[c mod w_len] * sigmoid(gate)               (gate behind it)
//   mode 2:  the same with silu(gate)
// gate is column g_off + c of a wider float32 row.  div (nullable): every y of a part is first divided by div[t, part].
// out's rows lie ldo apart and receive out_scale times the result.
template <typename TO>
__global__ void gated_head_norm_kernel(TO* __restrict__ out, const float* __restrict__ y, const float* __restrict__ gate,
                                       long long ldg, int g_off, const float* __restrict__ w, int w_len, int W, int part,
                                       float eps, int mode, const float* __restrict__ div, long long ldo, float out_scale) {
    __shared__ float scratch[33];
    const int t = blockIdx.x, c0 = blockIdx.y * part;
    const float* yr = y + (size_t)t * W + c0;
    const float* gr = gate + (size_t)t * ldg + g_off + c0;
    float dv = div ? div[(size_t)t * gridDim.y + blockIdx.y] : 1.f;
    if (dv == 0.f) dv = 1.f;        // (a padding token's, which nothing has written)
    float ss = 0.f;
    for (int i = threadIdx.x; i < part; i += blockDim.x) {
        float v = yr[i] / dv;
        if (mode == 0) {
            const float z = gr[i];
            v *= z / (1.f + expf(-z));
        }
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)part + eps);
    TO* o = out + (size_t)t * ldo + c0;
    for (int i = threadIdx.x; i < part; i += blockDim.x) {
        const float z = gr[i];
        float v = yr[i] / dv;
        if (mode == 0)
            v = v * (z / (1.f + expf(-z))) * inv * w[(c0 + i) % w_len];
        else
            v = v * inv * w[(c0 + i) % w_len] * (mode == 2 ? z * sigmoid_exact(z) : sigmoid_exact(z));
        o[i] = from_f32<TO>(out_scale * v);
    }
}

// The same for parts of at most 32 * NV channels: a warp per (token, part) keeps its channels in registers, one pass
// over memory, sums by shuffles; a block's warps take neighbouring parts of a token.
template <typename TO, int NV>
__global__ void __launch_bounds__(256) gated_head_norm_warp_kernel(TO* __restrict__ out, const float* __restrict__ y,
                                                                   const float* __restrict__ gate, long long ldg, int g_off,
                                                                   const float* __restrict__ w, int w_len, int W, int part,
                                                                   float eps, int mode, const float* __restrict__ div,
                                                                   long long ldo, float out_scale, long long units) {
    const int lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= units) return;
    const int parts = W / part;
    const long long t = unit / parts;
    const int c0 = (int)(unit % parts) * part;
    const float* yr = y + (size_t)t * W + c0;
    const float* gr = gate + (size_t)t * ldg + g_off + c0;
    float v[NV], z[NV];
    float dv = div ? div[unit] : 1.f;
    if (dv == 0.f) dv = 1.f;        // (a padding token's, which nothing has written)
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        v[k] = i < part ? yr[i] : 0.f;
        z[k] = i < part ? gr[i] : 0.f;
        if (div) v[k] /= dv;
        if (mode == 0) v[k] *= z[k] / (1.f + expf(-z[k]));
        ss = fmaf(v[k], v[k], ss);
    }
    const float inv = 1.f / sqrtf(warp_total(ss) / (float)part + eps);
    TO* o = out + (size_t)t * ldo + c0;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = lane + 32 * k;
        if (i >= part) continue;
        float r = v[k] * inv * w[(c0 + i) % w_len];
        if (mode != 0) r *= mode == 2 ? z[k] * sigmoid_exact(z[k]) : sigmoid_exact(z[k]);
        o[i] = from_f32<TO>(out_scale * r);
    }
}

template <typename TO>
static void gated_head_norm_launch(TO* out, const float* y, const float* gate, long long ldg, int g_off, const float* w,
                                   int w_len, int tokens, int W, int part, float eps, int mode, const float* div,
                                   long long ldo, float out_scale, cudaStream_t stream) {
    const long long units = (long long)tokens * (W / part);
    const int warps = 8;
    const unsigned blocks = (unsigned)((units + warps - 1) / warps);
#define XB_HEAD_NORM_NV(NVV)                                                                                              \
    gated_head_norm_warp_kernel<TO, NVV><<<blocks, warps * 32, 0, stream>>>(out, y, gate, ldg, g_off, w, w_len, W, part, \
                                                                            eps, mode, div, ldo, out_scale, units)
    if (part <= 32) XB_HEAD_NORM_NV(1);
    else if (part <= 64) XB_HEAD_NORM_NV(2);
    else if (part <= 128) XB_HEAD_NORM_NV(4);
    else if (part <= 256) XB_HEAD_NORM_NV(8);
    else if (part <= 512) XB_HEAD_NORM_NV(16);
    else {
        const dim3 grid(tokens, W / part);
        const int threads = part >= 1024 ? 256 : 128;
        gated_head_norm_kernel<TO><<<grid, threads, 0, stream>>>(out, y, gate, ldg, g_off, w, w_len, W, part, eps, mode, div, ldo,
                                                             out_scale);
    }
#undef XB_HEAD_NORM_NV
}

XB_EXPORT int xb_gated_head_norm(int out_dtype, void* out, const float* y, const float* gate, long long ldg, int g_off,
                                 const float* w, int w_len, int tokens, int W, int part, float eps, int mode,
                                 const float* div, long long ldo, float out_scale, cudaStream_t stream) {
    if (tokens <= 0 || W <= 0) return 0;
    if (part <= 0 || W % part || W / part > 65535) return (int)cudaErrorInvalidValue;
    if (out_dtype == XB_F32)
        gated_head_norm_launch<float>((float*)out, y, gate, ldg, g_off, w, w_len, tokens, W, part, eps, mode, div, ldo,
                                      out_scale, stream);
    else
        gated_head_norm_launch<__nv_bfloat16>((__nv_bfloat16*)out, y, gate, ldg, g_off, w, w_len, tokens, W, part, eps, mode,
                                              div, ldo, out_scale, stream);
    return xb_launch_status();
}
