// Gated linear attention: S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head, with a decay alpha_t in (0, 1) for every
// key channel that depends on the token: alpha = sigmoid(z)^(1 / tau), z = a2 (a1 h) + b.  The f32 state is [dim, vS] per head.
//   gated_decode_kernel    one token: decays, state, output, norm over the head, SiLU gate, in one launch
//   prompt portions in bf16, kGatedChunk tokens a chunk, all chunks side by side.  With beta_t the product of the decays of a
//   chunk's tokens up to t (kept as a sum of logarithms) and n its tokens:
//     gated_chunk_kernel   beta; what the chunk adds to the state, U = sum_j (beta_n / beta_j * k_j) v_j^T; the chunk's own part of the
//                          output, o_t = sum_{j <= t} (sum_d q_t k_j beta_t / beta_j) v_j
//     gated_scan_kernel    state before every chunk: S <- beta_n S + U, in place of U
//     gated_output_kernel  o_t += (beta_t * q_t)^T S, norm, gate
//   A ratio of betas is the exponential of a difference of logarithms that is never positive: blocks of 16 tokens are scored
//   against earlier blocks from the boundary between them, pairs inside a block one by one.
//   q, k, v are bf16 already; every f32 factor (state, decayed queries and keys, scores) enters a tensor-core product as three
//   bf16 terms, and a product of two such sums keeps the six pairs of terms that reach into 24 bits.
#include <algorithm>

#include "stack.cuh"

namespace im {

namespace {

constexpr float kLog2eGated = 1.4426950408889634f;

// ---- decode ---------------------------------------------------------------------------------------------------------------
// grid (heads, sequences); a thread owns 4 value columns and the key channels slice, slice + slices, ... (R of them).
constexpr int kGdThreads = 512, kGdGateMax = 8192;  // floats of a2 that are staged

template <typename T, int R>
__global__ void __launch_bounds__(kGdThreads) gated_decode_kernel(const LinearArgs a, int nv, int slices) {
    extern __shared__ __align__(16) unsigned char gated_smem[];
    __shared__ float sh[32];
    const LinearShape &s = a.s;
    const int tid = threadIdx.x, h = blockIdx.x, m = blockIdx.y;
    const int slice = tid / nv, vec = tid % nv, v4 = vec * 4, HD = s.heads * s.dim;
    float *red = reinterpret_cast<float *>(gated_smem);  // [slices][4 nv]
    float *qs = red + slices * nv * 4, *ks = qs + s.dim, *as = ks + s.dim, *gate = as + s.dim;
    const bool staged = s.rank * s.dim <= kGdGateMax;
    pdl_trigger();
    // Weights, the positions and the state come from before this step's first kernel (a one-token step is captured with the
    // position update as its last node, and a captured step starts when the one before it has ended): no need to wait for them.
    if (staged)
        for (int i = tid; i < s.rank * s.dim; i += kGdThreads) gate[i] = a.a2[(size_t)(i / s.dim) * HD + h * s.dim + i % s.dim];
    const int slot = a.slot_map ? a.slot_map[m] : m;
    float *state = a.state + ((size_t)slot * s.heads + h) * s.dim * s.vS + v4;
    const bool fresh = a.pos_dev[slot] == 0, mine = slice < slices && v4 < s.vS;
    float4 S[R];
#pragma unroll
    for (int i = 0; i < R; i++) {
        const int d = i * slices + slice;
        S[i] = (!fresh && mine && d < s.dim) ? *reinterpret_cast<const float4 *>(state + (size_t)d * s.vS) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    pdl_wait();
    const T *y = static_cast<const T *>(a.y) + (size_t)m * a.ldy;
    const int rank8 = (s.rank + 7) & ~7;
    if (staged) __syncthreads();
    for (int d = tid; d < s.dim; d += kGdThreads) {
        qs[d] = to_f<T>(y[s.q_off + h * s.dimP + d]) * s.q_scale;
        ks[d] = to_f<T>(y[s.k_off + h * s.dimP + d]);
        const float *a1 = a.a1 + (size_t)m * rank8;
        float z = a.a2b[h * s.dim + d];
        if (staged) {
            for (int r = 0; r < s.rank; r++) z = fmaf(gate[r * s.dim + d], a1[r], z);
        } else {
            for (int r = 0; r < s.rank; r++) z = fmaf(a.a2[(size_t)r * HD + h * s.dim + d], a1[r], z);
        }
        as[d] = expf(-softplus_f(-z) * s.inv_tau);
    }
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; j++) v[j] = mine && v4 + j < s.vdim ? to_f<T>(y[s.v_off + h * s.vP + v4 + j]) : 0.0f;
    __syncthreads();
    float4 o = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < R; i++) {
        const int d = i * slices + slice;
        if (mine && d < s.dim) {
            const float al = as[d], k = ks[d], q = qs[d];
            S[i].x = fmaf(al, S[i].x, k * v[0]);
            S[i].y = fmaf(al, S[i].y, k * v[1]);
            S[i].z = fmaf(al, S[i].z, k * v[2]);
            S[i].w = fmaf(al, S[i].w, k * v[3]);
            o.x = fmaf(q, S[i].x, o.x);
            o.y = fmaf(q, S[i].y, o.y);
            o.z = fmaf(q, S[i].z, o.z);
            o.w = fmaf(q, S[i].w, o.w);
            if (!a.keep_state) *reinterpret_cast<float4 *>(state + (size_t)d * s.vS) = S[i];
        }
    }
    if (slice < slices) *reinterpret_cast<float4 *>(red + (slice * nv + vec) * 4) = o;
    __syncthreads();
    float sum = 0.0f;
    const bool col = tid < s.vdim;
    if (col)
        for (int i = 0; i < slices; i++) sum += red[i * nv * 4 + tid];
    const float inv = 1.0f / sqrtf(block_sum_f(sum * sum, sh) / (float)s.vdim + s.eps);
    if (tid < s.vP) {
        const float z = to_f<T>(y[s.g_off + h * s.vP + tid]);
        static_cast<T *>(a.out)[(size_t)m * a.ldo + h * s.vP + tid] = from_f<T>(col ? sum * inv * a.norm[tid] * silu_f(z) : 0.0f);
    }
}

// ---- prompt chunks ----------------------------------------------------------------------------------------------------------
constexpr int kGc = kGatedChunk, kGcThreads = 256, kGcARow = (kGc + 8) * 2;  // bytes of a row of scores
struct GatedSizes {
    int dimK, vK, nchunks;  // key and value sizes padded to 16
};
inline size_t gated_chunk_smem(const LinearShape &s, const GatedSizes &z) {
    return (size_t)2 * kGc * (z.dimK + 8) * 2 + (size_t)kGc * (z.vK + 8) * 2 + (size_t)kGc * (z.dimK + 4) * 4 +
           std::max((size_t)3 * kGc * kGcARow, (size_t)kGc * round_up(s.rank, 8) * 4);
}

__device__ __forceinline__ float bf_lo(unsigned p) { return __uint_as_float(p << 16); }
__device__ __forceinline__ float bf_hi(unsigned p) { return __uint_as_float(p & 0xffff0000u); }
__device__ __forceinline__ float bf_at(const unsigned char *row, int i) { return __bfloat162float(*reinterpret_cast<const __nv_bfloat16 *>(row + i * 2)); }

// acc += (a0 + a1 + a2)(b0 + b1 + b2) without the pairs below 24 bits, smallest first
__device__ __forceinline__ void mma_six(float (&acc)[4], const unsigned (&a)[4][3], const unsigned (&b0)[3], const unsigned (&b1)[3]) {
#pragma unroll
    for (int sum = 2; sum >= 0; sum--)
#pragma unroll
        for (int i = 0; i <= sum; i++) mma_bf16(acc, a[0][i], a[1][i], a[2][i], a[3][i], b0[sum - i], b1[sum - i]);
}

// grid (chunks, heads), 8 warps
__global__ void __launch_bounds__(kGcThreads) gated_chunk_kernel(const LinearArgs a, const GatedSizes z) {
    typedef __nv_bfloat16 T;
    extern __shared__ __align__(16) unsigned char gated_smem[];
    const LinearShape &s = a.s;
    const int dimK = z.dimK, vK = z.vK, rs = (dimK + 8) * 2, vs = (vK + 8) * 2, bs = dimK + 4, rank8 = (s.rank + 7) & ~7;
    unsigned char *qb = gated_smem, *kb = qb + kGc * rs, *vb = kb + kGc * rs;
    float *bt = reinterpret_cast<float *>(vb + kGc * vs);             // log2 beta [token][channel]
    unsigned char *sc = reinterpret_cast<unsigned char *>(bt + kGc * bs);  // scores, three terms [3][64][72]
    float *a1 = reinterpret_cast<float *>(sc);  // in use before the scores are
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int chunk = blockIdx.x, h = blockIdx.y, c0 = chunk * kGc, n = min(kGc, a.T - c0), HD = s.heads * s.dim;
    pdl_trigger();
    pdl_wait();
    {
        const T *y = static_cast<const T *>(a.y) + (size_t)c0 * a.ldy;
        const int nq = dimK / 8, nvv = vK / 8, rq = s.dimP / 8, rv = s.vP / 8, per = 2 * nq + nvv;
        for (int i = tid; i < kGc * per; i += kGcThreads) {
            const int r = i / per, c = i % per;
            const bool q = c < nq, k = !q && c < 2 * nq;
            const int cc = q ? c : k ? c - nq : c - 2 * nq;
            unsigned char *dst = q ? qb + r * rs + cc * 16 : k ? kb + r * rs + cc * 16 : vb + r * vs + cc * 16;
            if (r < n && cc < (q || k ? rq : rv)) cp_async16(dst, y + (size_t)r * a.ldy + (q ? s.q_off + h * s.dimP : k ? s.k_off + h * s.dimP : s.v_off + h * s.vP) + cc * 8);
            else *reinterpret_cast<uint4 *>(dst) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
        for (int i = tid; i < kGc * rank8; i += kGcThreads) a1[i] = i / rank8 < n ? a.a1[(size_t)c0 * rank8 + i] : 0.0f;
    }
    __syncthreads();
    // logarithms of the decays: a thread takes one channel of 16 tokens
    for (int i = tid; i < dimK * (kGc / 16); i += kGcThreads) {
        const int d = i % dimK, j0 = i / dimK * 16;
        float acc[16];
        const float b0 = d < s.dim ? a.a2b[h * s.dim + d] : 0.0f;
#pragma unroll
        for (int j = 0; j < 16; j++) acc[j] = b0;
        if (d < s.dim)
            for (int r = 0; r < s.rank; r++) {
                const float w = a.a2[(size_t)r * HD + h * s.dim + d];
#pragma unroll
                for (int j = 0; j < 16; j++) acc[j] = fmaf(w, a1[(j0 + j) * rank8 + r], acc[j]);
            }
#pragma unroll
        for (int j = 0; j < 16; j++) bt[(j0 + j) * bs + d] = d < s.dim && j0 + j < n ? -softplus_f(-acc[j]) * s.inv_tau * kLog2eGated : 0.0f;
    }
    cp_async_wait<0>();
    __syncthreads();
    for (int d = tid; d < dimK; d += kGcThreads) {
        float sum = 0.0f;
#pragma unroll 8
        for (int j = 0; j < kGc; j++) {
            sum += bt[j * bs + d];
            bt[j * bs + d] = sum;
        }
    }
    __syncthreads();
    for (int i = tid; i < n * s.dimP; i += kGcThreads) {
        const int j = i / s.dimP, d = i % s.dimP;
        a.decays[((size_t)(c0 + j) * s.heads + h) * s.dimP + d] = bt[j * bs + d];
    }
    const unsigned vbase = (unsigned)__cvta_generic_to_shared(vb), sbase = (unsigned)__cvta_generic_to_shared(sc);
    // U: a warp per 16 key channels; rows of A are channels, columns tokens
    float *U = a.chunk_states + ((size_t)chunk * s.heads + h) * s.dim * s.vS;
    for (int mt = warp; mt * 16 < dimK; mt += kGcThreads / 32) {
        unsigned ka[kGc / 16][4][3];
        const float bn[2] = {bt[(kGc - 1) * bs + mt * 16 + g], bt[(kGc - 1) * bs + mt * 16 + g + 8]};
#pragma unroll
        for (int kk = 0; kk < kGc / 16; kk++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int d = mt * 16 + g + 8 * (e & 1), j = kk * 16 + 2 * t + 8 * (e >> 1);
                const float x0 = bf_at(kb + j * rs, d) * exp2f(bn[e & 1] - bt[j * bs + d]);
                const float x1 = bf_at(kb + (j + 1) * rs, d) * exp2f(bn[e & 1] - bt[(j + 1) * bs + d]);
                split_bf2<3>(x0, x1, ka[kk][e]);
            }
        for (int v0 = 0; v0 < vK; v0 += 32) {
            float acc[4][4] = {};
#pragma unroll
            for (int kk = 0; kk < kGc / 16; kk++)
#pragma unroll
                for (int nb = 0; nb < 4; nb += 2)
                    if (v0 + nb * 8 < vK) {
                        unsigned b[4];
                        ldsm_x4_t(b, vbase + (kk * 16 + (lane & 15)) * vs + (lane >> 4) * 16 + (v0 + nb * 8) * 2);
#pragma unroll
                        for (int i = 2; i >= 0; i--) {
                            mma_bf16(acc[nb], ka[kk][0][i], ka[kk][1][i], ka[kk][2][i], ka[kk][3][i], b[0], b[1]);
                            mma_bf16(acc[nb + 1], ka[kk][0][i], ka[kk][1][i], ka[kk][2][i], ka[kk][3][i], b[2], b[3]);
                        }
                    }
#pragma unroll
            for (int nb = 0; nb < 4; nb++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int d = mt * 16 + g + 8 * e, v = v0 + nb * 8 + 2 * t;
                    if (d < s.dim && v < s.vS) *reinterpret_cast<float2 *>(U + (size_t)d * s.vS + v) = make_float2(acc[nb][2 * e], acc[nb][2 * e + 1]);
                }
        }
    }
    // scores of 16 x 16 blocks: warps 0-3 the blocks on the diagonal, warps 4-7 the six below it
    auto put = [&](int ib, int jb, int nb, int r, float x0, float x1) {
        unsigned terms[3];
        split_bf2<3>(x0, x1, terms);
#pragma unroll
        for (int i = 0; i < 3; i++) *reinterpret_cast<unsigned *>(sc + (size_t)(i * kGc + ib * 16 + g + 8 * r) * kGcARow + (jb * 16 + nb * 8 + 2 * t) * 2) = terms[i];
    };
    if (warp < 4) {
        const int ib = warp;
        if (ib * 16 < n) {
            const int r0 = ib * 16 + g, cj = ib * 16 + 2 * t;  // rows r0, r0 + 8; columns cj, cj + 1 and 8 further on
            float acc[6] = {};
#pragma unroll 2
            for (int d = 0; d < dimK; d += 2) {  // two channels; padding channels hold zeros
                unsigned q[2], k[4];
                float2 e[2], f[4];
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    q[j] = *reinterpret_cast<const unsigned *>(qb + (r0 + 8 * j) * rs + d * 2);
                    e[j] = *reinterpret_cast<const float2 *>(bt + (r0 + 8 * j) * bs + d);
                }
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const int c = cj + (j & 1) + 8 * (j >> 1);
                    k[j] = *reinterpret_cast<const unsigned *>(kb + c * rs + d * 2);
                    f[j] = *reinterpret_cast<const float2 *>(bt + c * bs + d);
                }
                // the pairs above the diagonal, whose difference would be positive, are dropped below
                auto add = [&](float &x, int r, int c) {
                    x = fmaf(bf_lo(q[r]) * bf_lo(k[c]), exp2f(fminf(e[r].x - f[c].x, 0.0f)), x);
                    x = fmaf(bf_hi(q[r]) * bf_hi(k[c]), exp2f(fminf(e[r].y - f[c].y, 0.0f)), x);
                };
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    add(acc[j], 0, j);
                    add(acc[2 + j], 1, j);
                    add(acc[4 + j], 1, 2 + j);
                }
            }
            put(ib, ib, 0, 0, 2 * t <= g ? acc[0] : 0.0f, 2 * t + 1 <= g ? acc[1] : 0.0f);
            put(ib, ib, 0, 1, acc[2], acc[3]);
            put(ib, ib, 1, 0, 0.0f, 0.0f);
            put(ib, ib, 1, 1, 2 * t <= g ? acc[4] : 0.0f, 2 * t + 1 <= g ? acc[5] : 0.0f);
        }
    } else {
        for (int bi = warp - 4; bi < 6; bi += 4) {
            const int ib = bi < 1 ? 1 : bi < 3 ? 2 : 3, jb = bi < 1 ? 0 : bi < 3 ? bi - 1 : bi - 3;
            if (ib * 16 >= n) continue;
            const float *edge = bt + (ib * 16 - 1) * bs;  // beta at the end of the block before the rows
            float acc[2][4] = {};
            for (int kk = 0; kk < dimK / 16; kk++) {
                unsigned qa[4][3];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int r = ib * 16 + g + 8 * (e & 1), d = kk * 16 + 2 * t + 8 * (e >> 1);
                    const unsigned p = *reinterpret_cast<const unsigned *>(qb + r * rs + d * 2);
                    const float2 b = *reinterpret_cast<const float2 *>(bt + r * bs + d), b0 = *reinterpret_cast<const float2 *>(edge + d);
                    split_bf2<3>(bf_lo(p) * exp2f(b.x - b0.x), bf_hi(p) * exp2f(b.y - b0.y), qa[e]);
                }
#pragma unroll
                for (int nb = 0; nb < 2; nb++) {
                    unsigned kf[2][3];
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        const int r = jb * 16 + nb * 8 + g, d = kk * 16 + 2 * t + 8 * e;
                        const unsigned p = *reinterpret_cast<const unsigned *>(kb + r * rs + d * 2);
                        const float2 b = *reinterpret_cast<const float2 *>(bt + r * bs + d), b0 = *reinterpret_cast<const float2 *>(edge + d);
                        split_bf2<3>(bf_lo(p) * exp2f(b0.x - b.x), bf_hi(p) * exp2f(b0.y - b.y), kf[e]);
                    }
                    mma_six(acc[nb], qa, kf[0], kf[1]);
                }
            }
#pragma unroll
            for (int nb = 0; nb < 2; nb++)
#pragma unroll
                for (int r = 0; r < 2; r++) put(ib, jb, nb, r, acc[nb][2 * r], acc[nb][2 * r + 1]);
        }
    }
    __syncthreads();
    // the chunk's own part of the output: a warp takes 16 tokens and half of the value columns
    const int ib = warp >> 1, vh = (vK / 2 + 15) / 16 * 16, v_begin = (warp & 1) * vh, v_end = min(vK, v_begin + vh);
    if (ib * 16 < n) {
        for (int v0 = v_begin; v0 < v_end; v0 += 32) {
            float acc[4][4] = {};
            for (int jb = 0; jb <= ib; jb++) {
                unsigned p[3][4];
#pragma unroll
                for (int i = 0; i < 3; i++) ldsm_x4(p[i], sbase + (i * kGc + ib * 16 + (lane & 15)) * kGcARow + (lane >> 4) * 16 + jb * 32);
#pragma unroll
                for (int nb = 0; nb < 4; nb += 2)
                    if (v0 + nb * 8 < v_end) {
                        unsigned b[4];
                        ldsm_x4_t(b, vbase + (jb * 16 + (lane & 15)) * vs + (lane >> 4) * 16 + (v0 + nb * 8) * 2);
#pragma unroll
                        for (int i = 2; i >= 0; i--) {
                            mma_bf16(acc[nb], p[i][0], p[i][1], p[i][2], p[i][3], b[0], b[1]);
                            mma_bf16(acc[nb + 1], p[i][0], p[i][1], p[i][2], p[i][3], b[2], b[3]);
                        }
                    }
            }
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int j = ib * 16 + g + 8 * r;
                if (j < n)
#pragma unroll
                    for (int nb = 0; nb < 4; nb++) {
                        const int v = v0 + nb * 8 + 2 * t;
                        if (v < s.vP && v < v_end)
                            *reinterpret_cast<float2 *>(a.o + ((size_t)(c0 + j) * s.heads + h) * s.vP + v) = make_float2(acc[nb][2 * r], acc[nb][2 * r + 1]);
                    }
            }
        }
    }
}

// grid (blocks of 256 four-column vectors of a head's state, heads)
__global__ void __launch_bounds__(256) gated_scan_kernel(const LinearArgs a, int nchunks) {
    const LinearShape &s = a.s;
    const int i = blockIdx.x * 256 + threadIdx.x, h = blockIdx.y, per = s.vS / 4;
    pdl_trigger();
    pdl_wait();
    if (i >= s.dim * per) return;
    const int d = i / per, slot = a.slot_map ? a.slot_map[0] : 0;
    const size_t stride = (size_t)s.heads * s.dim * per;
    float4 *st = reinterpret_cast<float4 *>(a.state) + (size_t)slot * stride + (size_t)h * s.dim * per + i;
    float4 *u = reinterpret_cast<float4 *>(a.chunk_states) + (size_t)h * s.dim * per + i;
    float4 S = a.pos_dev[slot] == 0 ? make_float4(0.0f, 0.0f, 0.0f, 0.0f) : *st;
    constexpr int B = 8;  // chunks whose sums are requested together
    for (int c0 = 0; c0 < nchunks; c0 += B) {
        float4 x[B];
        float e[B];
#pragma unroll
        for (int j = 0; j < B; j++)
            if (c0 + j < nchunks) {
                x[j] = u[(size_t)(c0 + j) * stride];
                e[j] = a.decays[((size_t)(min(a.T, (c0 + j + 1) * kGc) - 1) * s.heads + h) * s.dimP + d];
            }
#pragma unroll
        for (int j = 0; j < B; j++)
            if (c0 + j < nchunks) {
                u[(size_t)(c0 + j) * stride] = S;
                const float f = exp2f(e[j]);
                S.x = fmaf(f, S.x, x[j].x);
                S.y = fmaf(f, S.y, x[j].y);
                S.z = fmaf(f, S.z, x[j].z);
                S.w = fmaf(f, S.w, x[j].w);
            }
    }
    if (!a.keep_state) *st = S;
}

// grid (chunks, heads), 8 warps: 16 tokens x half of the value columns each.  NV: 8-column tiles per warp, even.
constexpr int kGoSlab = 64, kGoQRow = (kGoSlab + 8) * 2;
inline size_t gated_output_smem(int vW) { return (size_t)3 * kGc * kGoQRow + (size_t)3 * kGoSlab * (vW + 8) * 2; }
template <int NV>
__global__ void __launch_bounds__(kGcThreads, NV <= 8 ? 2 : 1) gated_output_kernel(const LinearArgs a) {
    typedef __nv_bfloat16 T;
    constexpr int VW = NV * 16;  // value columns of the tile
    constexpr int ss = (VW + 8) * 2;
    extern __shared__ __align__(16) unsigned char gated_smem[];
    __shared__ float sums[2][kGc];
    const LinearShape &s = a.s;
    unsigned char *qt = gated_smem, *stt = qt + 3 * kGc * kGoQRow;  // decayed queries [3][64][72], state [3][64][VW + 8]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int chunk = blockIdx.x, h = blockIdx.y, c0 = chunk * kGc, n = min(kGc, a.T - c0);
    const int ib = warp >> 1, half = warp & 1;
    pdl_trigger();
    pdl_wait();
    const T *y = static_cast<const T *>(a.y) + (size_t)c0 * a.ldy + s.q_off + h * s.dimP;
    const float *beta = a.decays + ((size_t)c0 * s.heads + h) * s.dimP;
    const float *S = a.chunk_states + ((size_t)chunk * s.heads + h) * s.dim * s.vS;
    const unsigned qbase = (unsigned)__cvta_generic_to_shared(qt), sbase = (unsigned)__cvta_generic_to_shared(stt);
    float acc[NV][4];
#pragma unroll
    for (int i = 0; i < NV; i++) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    for (int d0 = 0; d0 < s.dim; d0 += kGoSlab) {
        const int kmax = min(kGoSlab, (s.dim - d0 + 15) & ~15);
        __syncthreads();
        for (int i = tid; i < kGc * kGoSlab / 2; i += kGcThreads) {
            const int r = i / (kGoSlab / 2), d = d0 + i % (kGoSlab / 2) * 2;
            float x0 = 0.0f, x1 = 0.0f;
            if (r < n && d < s.dimP) {  // the padding of q is zero
                const unsigned p = *reinterpret_cast<const unsigned *>(y + (size_t)r * a.ldy + d);
                const float2 b = *reinterpret_cast<const float2 *>(beta + (size_t)r * s.heads * s.dimP + d);
                x0 = bf_lo(p) * exp2f(b.x);
                x1 = bf_hi(p) * exp2f(b.y);
            }
            unsigned terms[3];
            split_bf2<3>(x0, x1, terms);
#pragma unroll
            for (int k = 0; k < 3; k++) *reinterpret_cast<unsigned *>(qt + (size_t)(k * kGc + r) * kGoQRow + (d - d0) * 2) = terms[k];
        }
        for (int i = tid; i < kmax * (VW / 4); i += kGcThreads) {
            const int r = i / (VW / 4), v = i % (VW / 4) * 4;
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (d0 + r < s.dim && v < s.vS) x = *reinterpret_cast<const float4 *>(S + (size_t)(d0 + r) * s.vS + v);
            unsigned lo[3], hi[3];
            split_bf2<3>(x.x, x.y, lo);
            split_bf2<3>(x.z, x.w, hi);
#pragma unroll
            for (int k = 0; k < 3; k++) *reinterpret_cast<uint2 *>(stt + (size_t)(k * kGoSlab + r) * ss + v * 2) = make_uint2(lo[k], hi[k]);
        }
        __syncthreads();
        if (ib * 16 < n)
            for (int kk = 0; kk < kmax / 16; kk++) {
                unsigned q[3][4];
#pragma unroll
                for (int i = 0; i < 3; i++) ldsm_x4(q[i], qbase + (i * kGc + ib * 16 + (lane & 15)) * kGoQRow + (lane >> 4) * 16 + kk * 32);
#pragma unroll
                for (int nb = 0; nb < NV; nb += 2) {
                    if (half * NV * 8 + nb * 8 >= s.vP) break;
#pragma unroll
                    for (int k = 2; k >= 0; k--) {
                        unsigned b[4];
                        ldsm_x4_t(b, sbase + (k * kGoSlab + kk * 16 + (lane & 15)) * ss + (lane >> 4) * 16 + (half * NV + nb) * 16);
#pragma unroll
                        for (int i = 2 - k; i >= 0; i--) {
                            mma_bf16(acc[nb], q[i][0], q[i][1], q[i][2], q[i][3], b[0], b[1]);
                            mma_bf16(acc[nb + 1], q[i][0], q[i][1], q[i][2], q[i][3], b[2], b[3]);
                        }
                    }
                }
            }
    }
    // own part, norm over the head, gate
    float sq[2] = {0.0f, 0.0f};
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int j = ib * 16 + g + 8 * r;
        if (j < n) {
            const float *own = a.o + ((size_t)(c0 + j) * s.heads + h) * s.vP;
#pragma unroll
            for (int nb = 0; nb < NV; nb++) {
                const int v = (half * NV + nb) * 8 + 2 * t;
                if (v < s.vP) {
                    const float2 x = *reinterpret_cast<const float2 *>(own + v);
                    acc[nb][2 * r] = (acc[nb][2 * r] + x.x) * s.q_scale;
                    acc[nb][2 * r + 1] = (acc[nb][2 * r + 1] + x.y) * s.q_scale;
                    sq[r] = fmaf(acc[nb][2 * r], acc[nb][2 * r], fmaf(acc[nb][2 * r + 1], acc[nb][2 * r + 1], sq[r]));  // padding columns hold zeros
                }
            }
        }
        sq[r] += __shfl_xor_sync(0xffffffffu, sq[r], 1);
        sq[r] += __shfl_xor_sync(0xffffffffu, sq[r], 2);
        if (t == 0) sums[half][ib * 16 + g + 8 * r] = sq[r];
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int j = ib * 16 + g + 8 * r;
        if (j < n) {
            const float inv = 1.0f / sqrtf((sums[0][j] + sums[1][j]) / (float)s.vdim + s.eps);
            const T *gate = static_cast<const T *>(a.y) + (size_t)(c0 + j) * a.ldy + s.g_off + h * s.vP;
            T *out = static_cast<T *>(a.out) + (size_t)(c0 + j) * a.ldo + h * s.vP;
#pragma unroll
            for (int nb = 0; nb < NV; nb++) {
                const int v = (half * NV + nb) * 8 + 2 * t;
                if (v < s.vP) {
                    const unsigned p = *reinterpret_cast<const unsigned *>(gate + v);
                    const float2 w = *reinterpret_cast<const float2 *>(a.norm + v);
                    *reinterpret_cast<unsigned *>(out + v) = pack_bf2(acc[nb][2 * r] * inv * w.x * silu_f(bf_lo(p)), acc[nb][2 * r + 1] * inv * w.y * silu_f(bf_hi(p)));
                }
            }
        }
    }
}

// ---- host ---------------------------------------------------------------------------------------------------------------
constexpr size_t kGatedSmemMax = 220 * 1024;
struct DecodePlan {
    int nv, slices, rows;
    size_t smem;
};
DecodePlan decode_plan(const LinearShape &s) {
    DecodePlan p;
    p.nv = s.vS / 4;
    p.slices = p.nv > kGdThreads ? 0 : std::min(kGdThreads / p.nv, 64);
    p.rows = p.slices ? (s.dim + p.slices - 1) / p.slices : 1 << 20;
    p.smem = ((size_t)p.slices * p.nv * 4 + 3 * (size_t)s.dim + (s.rank * s.dim <= kGdGateMax ? (size_t)s.rank * s.dim : 0)) * sizeof(float);
    return p;
}
GatedSizes chunk_sizes(const LinearShape &s, int T) {
    GatedSizes z;
    z.dimK = round_up(s.dim, 16);
    z.vK = round_up(s.vdim, 16);
    z.nchunks = (T + kGc - 1) / kGc;
    return z;
}
template <typename T, int R>
int decode_launch(const LinearArgs &a, const DecodePlan &p, cudaStream_t st) {
    IM_CUDA_CHECK(launch_k(gated_decode_kernel<T, R>, dim3(a.s.heads, a.nseq), dim3(kGdThreads), p.smem, st, a, p.nv, p.slices));
    return IM_OK;
}
template <typename T>
int decode_any(const LinearArgs &a, const DecodePlan &p, cudaStream_t st) {
    if (p.rows <= 2) return decode_launch<T, 2>(a, p, st);
    if (p.rows <= 4) return decode_launch<T, 4>(a, p, st);
    if (p.rows <= 8) return decode_launch<T, 8>(a, p, st);
    return decode_launch<T, 16>(a, p, st);
}

}  // namespace

// A thread per value column in the norm, at most 16 channels a thread
bool gated_decode_takes(const LinearShape &s) { return s.vP <= kGdThreads && decode_plan(s).rows <= 16 && decode_plan(s).smem <= kGatedSmemMax; }
bool gated_chunk_takes(const LinearShape &s) {
    return round_up(s.dim, 16) <= 256 && s.vP <= 256 && gated_chunk_smem(s, chunk_sizes(s, 1)) <= kGatedSmemMax;
}

int gated_prepare() {
#define IM_SMEM(k) IM_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGatedSmemMax))
    IM_SMEM((gated_decode_kernel<float, 2>)); IM_SMEM((gated_decode_kernel<float, 4>)); IM_SMEM((gated_decode_kernel<float, 8>));
    IM_SMEM((gated_decode_kernel<float, 16>));
    IM_SMEM((gated_decode_kernel<__nv_bfloat16, 2>)); IM_SMEM((gated_decode_kernel<__nv_bfloat16, 4>)); IM_SMEM((gated_decode_kernel<__nv_bfloat16, 8>));
    IM_SMEM((gated_decode_kernel<__nv_bfloat16, 16>));
    IM_SMEM(gated_chunk_kernel);
    IM_SMEM(gated_output_kernel<4>); IM_SMEM(gated_output_kernel<8>); IM_SMEM(gated_output_kernel<16>);
#undef IM_SMEM
    return IM_OK;
}

int gated_decode_run(const LinearArgs &a, cudaStream_t st) {
    const DecodePlan p = decode_plan(a.s);
    return a.f32 ? decode_any<float>(a, p, st) : decode_any<__nv_bfloat16>(a, p, st);
}

int gated_chunk_run(const LinearArgs &a, cudaStream_t st, int *launches) {
    const LinearShape &s = a.s;
    const GatedSizes z = chunk_sizes(s, a.T);
    if (!a.decays || !a.chunk_states || (size_t)z.nchunks * s.heads * s.dim * s.vS * 4 > a.chunk_bytes) return IM_ERR_BOUNDS;
    const dim3 grid(z.nchunks, s.heads), block(kGcThreads);
    IM_CUDA_CHECK(launch_k(gated_chunk_kernel, grid, block, gated_chunk_smem(s, z), st, a, z));
    IM_CUDA_CHECK(launch_k(gated_scan_kernel, dim3((s.dim * s.vS / 4 + 255) / 256, s.heads), dim3(256), 0, st, a, z.nchunks));
    if (s.vP <= 64) IM_CUDA_CHECK(launch_k(gated_output_kernel<4>, grid, block, gated_output_smem(64), st, a));
    else if (s.vP <= 128) IM_CUDA_CHECK(launch_k(gated_output_kernel<8>, grid, block, gated_output_smem(128), st, a));
    else IM_CUDA_CHECK(launch_k(gated_output_kernel<16>, grid, block, gated_output_smem(256), st, a));
    *launches += 3;
    return IM_OK;
}

}  // namespace im
