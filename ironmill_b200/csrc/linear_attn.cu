// Decayed linear attention: per head a state S [dim x vdim] in f32, S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.
//   linear_step_kernel    token by token from registers (decode, short chunks, and everything in f32)
//   linear_chunk_kernel   prompt chunks in bf16: C tokens at a time on the tensor cores.  With the tokens of a chunk
//                         numbered from 0: o_i = decay^(i+1) S^T q_i + sum_{j<=i} decay^(i-j) (q_i . k_j) v_j,
//                         S <- decay^n S + sum_j decay^(n-1-j) k_j v_j^T.  q, k, v are bf16 already; the f32 factors (state,
//                         decayed scores, decayed values) enter a product as three bf16 terms each, which carry all 24 bits
//   linear_finish_kernel  RMS norm over the heads together, sigmoid gate
// The gated form has a decay per token and key channel in place of a constant per head, a norm per head and a SiLU gate; here it
// runs token by token (everything in f32, short portions), linear_gated.cu has its decode step and its prompt chunks.
// A sequence at position 0 starts from a zero state, whatever its slot held before.
#include <algorithm>

#include "stack.cuh"

namespace im {

namespace {

constexpr int kLtCols = 32, kLtSlices = 8, kLtBlock = 8;  // value columns per CTA, shares of the key dimension, tokens staged at once

// grid (heads, column blocks, sequences); warp = share of the key dimension, lane = value column.
template <typename T, int DR, bool GATED>
__global__ void __launch_bounds__(256) linear_step_kernel(const LinearArgs a) {
    extern __shared__ __align__(16) unsigned char linear_smem[];
    const LinearShape &s = a.s;
    float *qs = reinterpret_cast<float *>(linear_smem), *ks = qs + kLtBlock * s.dim, *vs = ks + kLtBlock * s.dim, *red = vs + kLtBlock * kLtCols;
    float *as = red + kLtBlock * kLtSlices * kLtCols;  // gated: decays of the staged tokens
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.x, v0 = blockIdx.y * kLtCols, seq = blockIdx.z, col = v0 + lane;
    const bool live = col < s.vdim;
    const float decay = GATED ? 0.0f : a.pows[(size_t)h * (kLinearPow + 1) + 1];
    pdl_trigger();
    pdl_wait();
    const int slot = a.slot_map ? a.slot_map[seq] : seq;
    float *state = a.state + ((size_t)slot * s.heads + h) * s.dim * s.vS + col;
    const bool fresh = a.pos_dev[slot] == 0;
    float S[DR];
#pragma unroll
    for (int i = 0; i < DR; i++) {
        const int d = i * kLtSlices + warp;
        S[i] = (!fresh && live && d < s.dim) ? state[(size_t)d * s.vS] : 0.0f;
    }
    for (int t0 = 0; t0 < a.T; t0 += kLtBlock) {
        const int nt = min(kLtBlock, a.T - t0);
        const T *y = static_cast<const T *>(a.y) + (size_t)(seq * a.T + t0) * a.ldy;
        __syncthreads();
        for (int i = tid; i < nt * s.dim; i += 256) {
            const int b = i / s.dim, d = i % s.dim;
            qs[i] = to_f<T>(y[(size_t)b * a.ldy + s.q_off + h * s.dimP + d]) * (GATED ? s.q_scale : 1.0f);
            if (GATED) {
                const int rank8 = (s.rank + 7) & ~7, HD = s.heads * s.dim;
                const float *a1 = a.a1 + (size_t)(seq * a.T + t0 + b) * rank8, *a2 = a.a2 + h * s.dim + d;
                float z = a.a2b[h * s.dim + d];
                for (int r = 0; r < s.rank; r++) z = fmaf(a2[(size_t)r * HD], a1[r], z);
                as[i] = expf(-softplus_f(-z) * s.inv_tau);
            }
            ks[i] = to_f<T>(y[(size_t)b * a.ldy + s.k_off + h * s.dimP + d]);
        }
        for (int i = tid; i < nt * kLtCols; i += 256) {
            const int b = i / kLtCols, c = v0 + i % kLtCols;
            vs[i] = c < s.vdim ? to_f<T>(y[(size_t)b * a.ldy + s.v_off + h * s.vP + c]) : 0.0f;
        }
        __syncthreads();
        for (int b = 0; b < nt; b++) {
            const float v = vs[b * kLtCols + lane];
            float o = 0.0f;
#pragma unroll
            for (int i = 0; i < DR; i++) {
                const int d = i * kLtSlices + warp;
                if (d < s.dim) {
                    S[i] = fmaf(GATED ? as[b * s.dim + d] : decay, S[i], ks[b * s.dim + d] * v);
                    o = fmaf(S[i], qs[b * s.dim + d], o);
                }
            }
            red[(b * kLtSlices + warp) * kLtCols + lane] = o;
        }
        __syncthreads();
        for (int i = tid; i < nt * kLtCols; i += 256) {
            const int b = i / kLtCols, c = i % kLtCols;
            float o = 0.0f;
#pragma unroll
            for (int w = 0; w < kLtSlices; w++) o += red[(b * kLtSlices + w) * kLtCols + c];
            if (v0 + c < s.vdim) a.o[(size_t)(seq * a.T + t0 + b) * s.heads * s.vP + h * s.vP + v0 + c] = o;
        }
    }
    if (!a.keep_state && live)
#pragma unroll
        for (int i = 0; i < DR; i++) {
            const int d = i * kLtSlices + warp;
            if (d < s.dim) state[(size_t)d * s.vS] = S[i];
        }
}

constexpr int kLcRow = (kLtCols + 8) * 2;  // bytes of a row of 32 value columns in shared memory
inline size_t linear_chunk_smem(int C, int dimK, int bufs) {
    return (size_t)bufs * C * (2 * (dimK + 8) * 2 + kLcRow) + 3 * (size_t)C * kLcRow + 3 * (size_t)dimK * kLcRow + (size_t)(C + 1) * 4;
}

// A long prompt of one sequence is cut into segments that run side by side: a first pass (`local`) leaves what each segment
// but the last adds to a zero state, the second starts every segment from the state those sums make before it.
struct LinearSegments {
    int count = 1, tokens = 0;  // segments, tokens of each (a multiple of kLinearPow)
    int local = 0;
    float *sums = nullptr;      // [count - 1][heads][dim][vS]
};

// grid (column blocks of 32, heads, sequences or segments), C / 16 warps.  MW: 16-row tiles of the state per warp.
template <int C, int MW>
__global__ void __launch_bounds__(C * 2, 1) linear_chunk_kernel(const LinearArgs a, int dimK, int bufs, const LinearSegments sg) {
    typedef __nv_bfloat16 T;
    constexpr int NT = C * 2, W = C / 16;
    extern __shared__ __align__(16) unsigned char linear_smem[];
    const LinearShape &s = a.s;
    const int rs = (dimK + 8) * 2;
    unsigned char *qb = linear_smem, *kb = qb + (size_t)bufs * C * rs, *vb = kb + (size_t)bufs * C * rs, *vw = vb + (size_t)bufs * C * kLcRow,
                  *sb = vw + 3 * C * kLcRow;
    float *pw = reinterpret_cast<float *>(sb + 3 * (size_t)dimK * kLcRow);  // decay^0 .. decay^C
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int v0 = blockIdx.x * kLtCols, h = blockIdx.y, seg = sg.count > 1 ? blockIdx.z : 0, seq = sg.count > 1 ? 0 : blockIdx.z;
    const int t_begin = seg * sg.tokens, t_end = sg.count > 1 ? min(a.T, t_begin + sg.tokens) : a.T;
    for (int i = tid; i <= C; i += NT) pw[i] = a.pows[(size_t)h * (kLinearPow + 1) + i];
    const int nq = s.dimP / 8, nvc = min(kLtCols, s.vP - v0) / 8;
    for (int i = tid; i < 2 * bufs * C * (dimK / 8); i += NT)  // padding columns once
        if (i % (dimK / 8) >= nq) *reinterpret_cast<uint4 *>(qb + (size_t)(i / (dimK / 8)) * rs + (i % (dimK / 8)) * 16) = make_uint4(0, 0, 0, 0);
    for (int i = tid; i < bufs * C * 4; i += NT)
        if (i % 4 >= nvc) *reinterpret_cast<uint4 *>(vb + (i / 4) * kLcRow + (i % 4) * 16) = make_uint4(0, 0, 0, 0);
    pdl_trigger();
    pdl_wait();
    const T *y = static_cast<const T *>(a.y) + (size_t)seq * a.T * a.ldy;
    auto load = [&](int buf, int c0) {
        for (int i = tid; i < C * (2 * nq + nvc); i += NT) {
            const int r = i / (2 * nq + nvc), c = i % (2 * nq + nvc);
            const T *row = y + (size_t)min(c0 + r, a.T - 1) * a.ldy;
            if (c < nq && sg.local) continue;
            if (c < nq) cp_async16(qb + (size_t)(buf * C + r) * rs + c * 16, row + s.q_off + h * s.dimP + c * 8);
            else if (c < 2 * nq) cp_async16(kb + (size_t)(buf * C + r) * rs + (c - nq) * 16, row + s.k_off + h * s.dimP + (c - nq) * 8);
            else cp_async16(vb + (size_t)(buf * C + r) * kLcRow + (c - 2 * nq) * 16, row + s.v_off + h * s.vP + v0 + (c - 2 * nq) * 8);
        }
        cp_async_commit();
    };
    load(0, t_begin);
    const int slot = a.slot_map ? a.slot_map[seq] : seq;
    float *state = a.state + ((size_t)slot * s.heads + h) * s.dim * s.vS + v0;
    const bool fresh = a.pos_dev[slot] == 0 || sg.local;
    float S[MW][4][4];  // rows 16 mt + g (+ 8), columns 8 n + 2 t (+ 1); mt = warp + W * i
#pragma unroll
    for (int i = 0; i < MW; i++)
#pragma unroll
        for (int n = 0; n < 4; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int d = 16 * (warp + W * i) + g + 8 * (e >> 1), c = 8 * n + 2 * t + (e & 1);
                S[i][n][e] = (!fresh && d < s.dim && v0 + c < s.vdim) ? state[(size_t)d * s.vS + c] : 0.0f;
            }
    if (!sg.local && seg > 0) {
        const float d1 = a.pows[(size_t)h * (kLinearPow + 1) + kLinearPow];
        float dl = 1.0f;
        for (int i = 0; i < sg.tokens; i += kLinearPow) dl *= d1;
        for (int r = 0; r < seg; r++) {
            const float *sum = sg.sums + ((size_t)r * s.heads + h) * s.dim * s.vS + v0;
#pragma unroll
            for (int i = 0; i < MW; i++)
#pragma unroll
                for (int n = 0; n < 4; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int d = 16 * (warp + W * i) + g + 8 * (e >> 1), c = 8 * n + 2 * t + (e & 1);
                        if (d < s.dim && v0 + c < s.vdim) S[i][n][e] = fmaf(S[i][n][e], dl, sum[(size_t)d * s.vS + c]);
                    }
        }
    }
    const unsigned base = (unsigned)__cvta_generic_to_shared(linear_smem);
    const unsigned qa0 = base + (warp * 16 + (lane & 15)) * rs + (lane >> 4) * 16;
    const unsigned ka0 = base + (unsigned)(kb - linear_smem) + ((lane & 7) + 8 * (lane >> 4)) * rs + ((lane >> 3) & 1) * 16;
    const unsigned kt0 = base + (unsigned)(kb - linear_smem) + ((lane >> 4) * 8 + (lane & 7)) * rs + ((lane >> 3) & 1) * 16;
    const unsigned vrow = (lane & 15) * kLcRow + (lane >> 4) * 16;
    const unsigned va0 = base + (unsigned)(vb - linear_smem) + vrow, wa0 = base + (unsigned)(vw - linear_smem) + vrow, sa0 = base + (unsigned)(sb - linear_smem) + vrow;
    const int nchunks = (t_end - t_begin + C - 1) / C;
    for (int ci = 0; ci < nchunks; ci++) {
        const int buf = bufs == 2 ? ci & 1 : 0, c0 = t_begin + ci * C, n = min(C, t_end - c0);
        if (bufs == 2 && ci + 1 < nchunks) {
            load(buf ^ 1, c0 + C);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        // the state before this chunk, as three bf16 matrices
#pragma unroll
        for (int i = 0; i < MW; i++) {
            const int mt = warp + W * i;
            if (mt * 16 < dimK && !sg.local)
#pragma unroll
                for (int nb = 0; nb < 4; nb++)
#pragma unroll
                    for (int r = 0; r < 2; r++) {
                        unsigned terms[3];
                        split_bf2<3>(S[i][nb][2 * r], S[i][nb][2 * r + 1], terms);
#pragma unroll
                        for (int z = 0; z < 3; z++)
                            *reinterpret_cast<unsigned *>(sb + (size_t)(z * dimK + 16 * mt + g + 8 * r) * kLcRow + (8 * nb + 2 * t) * 2) = terms[z];
                    }
        }
        __syncthreads();
        for (int i = tid; i < C * (kLtCols / 2); i += NT) {  // decayed values
            const int j = i / (kLtCols / 2), c = i % (kLtCols / 2);
            const unsigned p = *reinterpret_cast<const unsigned *>(vb + (size_t)(buf * C + j) * kLcRow + c * 4);
            const float wgt = j < n ? pw[n - 1 - j] : 0.0f;
            unsigned terms[3];
            split_bf2<3>(wgt * __uint_as_float(p << 16), wgt * __uint_as_float(p & 0xffff0000u), terms);
#pragma unroll
            for (int z = 0; z < 3; z++) *reinterpret_cast<unsigned *>(vw + (size_t)(z * C + j) * kLcRow + c * 4) = terms[z];
        }
        __syncthreads();
        const unsigned qa = qa0 + buf * C * rs, ka = ka0 + buf * C * rs, kt = kt0 + buf * C * rs, va = va0 + buf * C * kLcRow;
        if (warp * 16 < n && !sg.local) {
            float o[4][4];
#pragma unroll
            for (int nb = 0; nb < 4; nb++) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.0f;
            for (int kk = 0; kk < dimK / 16; kk++) {
                unsigned q[4];
                ldsm_x4(q, qa + kk * 32);
#pragma unroll
                for (int z = 2; z >= 0; z--)
#pragma unroll
                    for (int nb = 0; nb < 4; nb += 2) {
                        unsigned b[4];
                        ldsm_x4_t(b, sa0 + (z * dimK + 16 * kk) * kLcRow + nb * 16);
                        mma_bf16(o[nb], q[0], q[1], q[2], q[3], b[0], b[1]);
                        mma_bf16(o[nb + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
                    }
            }
            const int i0 = warp * 16 + g;
#pragma unroll
            for (int nb = 0; nb < 4; nb++) {
                o[nb][0] *= pw[i0 + 1]; o[nb][1] *= pw[i0 + 1];
                o[nb][2] *= pw[i0 + 9]; o[nb][3] *= pw[i0 + 9];
            }
            for (int jb = 0; jb <= warp; jb++) {
                float sc[2][4] = {};
                for (int kk = 0; kk < dimK / 16; kk++) {
                    unsigned q[4], b[4];
                    ldsm_x4(q, qa + kk * 32);
                    ldsm_x4(b, ka + jb * 16 * rs + kk * 32);
                    mma_bf16(sc[0], q[0], q[1], q[2], q[3], b[0], b[1]);
                    mma_bf16(sc[1], q[0], q[1], q[2], q[3], b[2], b[3]);
                }
                unsigned p[4][3];
#pragma unroll
                for (int nb = 0; nb < 2; nb++)
#pragma unroll
                    for (int r = 0; r < 2; r++) {
                        float w[2];
#pragma unroll
                        for (int e = 0; e < 2; e++) {
                            const int diff = i0 + 8 * r - (jb * 16 + 8 * nb + 2 * t + e);
                            w[e] = diff >= 0 ? sc[nb][2 * r + e] * pw[diff] : 0.0f;
                        }
                        split_bf2<3>(w[0], w[1], p[2 * nb + r]);
                    }
#pragma unroll
                for (int nb = 0; nb < 4; nb += 2) {
                    unsigned b[4];
                    ldsm_x4_t(b, va + jb * 16 * kLcRow + nb * 16);
#pragma unroll
                    for (int z = 2; z >= 0; z--) {
                        mma_bf16(o[nb], p[0][z], p[1][z], p[2][z], p[3][z], b[0], b[1]);
                        mma_bf16(o[nb + 1], p[0][z], p[1][z], p[2][z], p[3][z], b[2], b[3]);
                    }
                }
            }
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int i = i0 + 8 * r;
                if (i < n) {
                    float *dst = a.o + (size_t)(seq * a.T + c0 + i) * s.heads * s.vP + h * s.vP + v0;
#pragma unroll
                    for (int nb = 0; nb < 4; nb++)
#pragma unroll
                        for (int e = 0; e < 2; e++)
                            if (v0 + 8 * nb + 2 * t + e < s.vdim) dst[8 * nb + 2 * t + e] = o[nb][2 * r + e];
                }
            }
        }
        const float dn = pw[n];
#pragma unroll
        for (int i = 0; i < MW; i++) {
            const int mt = warp + W * i;
            if (mt * 16 < dimK) {
#pragma unroll
                for (int nb = 0; nb < 4; nb++)
#pragma unroll
                    for (int e = 0; e < 4; e++) S[i][nb][e] *= dn;
                for (int jb = 0; jb * 16 < n; jb++) {
                    unsigned k[4];
                    ldsm_x4_t(k, kt + jb * 16 * rs + mt * 32);
#pragma unroll
                    for (int z = 2; z >= 0; z--)
#pragma unroll
                        for (int nb = 0; nb < 4; nb += 2) {
                            unsigned b[4];
                            ldsm_x4_t(b, wa0 + (z * C + 16 * jb) * kLcRow + nb * 16);
                            mma_bf16(S[i][nb], k[0], k[1], k[2], k[3], b[0], b[1]);
                            mma_bf16(S[i][nb + 1], k[0], k[1], k[2], k[3], b[2], b[3]);
                        }
                }
            }
        }
        __syncthreads();
        if (bufs == 1 && ci + 1 < nchunks) load(0, c0 + C);
    }
    float *out_state = sg.local ? sg.sums + ((size_t)seg * s.heads + h) * s.dim * s.vS + v0 : state;
    if (sg.local || (!a.keep_state && seg == sg.count - 1))
#pragma unroll
        for (int i = 0; i < MW; i++)
#pragma unroll
            for (int nb = 0; nb < 4; nb++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int d = 16 * (warp + W * i) + g + 8 * (e >> 1), c = 8 * nb + 2 * t + (e & 1);
                    if (d < s.dim && v0 + c < s.vdim) out_state[(size_t)d * s.vS + c] = S[i][nb][e];
                }
}

template <typename T>
__global__ void __launch_bounds__(256) linear_finish_kernel(const LinearArgs a) {
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    const LinearShape &s = a.s;
    const int m = blockIdx.x, n = s.heads * s.vP;
    const float *o = a.o + (size_t)m * n;
    const T *gate = static_cast<const T *>(a.y) + (size_t)m * a.ldy + s.g_off;
    if (s.gated) {  // a warp per head
        T *out = static_cast<T *>(a.out) + (size_t)m * a.ldo;
        for (int h = threadIdx.x >> 5; h < s.heads; h += 8) {
            const float *oh = o + h * s.vP;
            float ss = 0.0f;
            for (int v = threadIdx.x & 31; v < s.vdim; v += 32) ss = fmaf(oh[v], oh[v], ss);
            const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)s.vdim + s.eps);
            for (int v = threadIdx.x & 31; v < s.vP; v += 32)
                out[h * s.vP + v] = from_f<T>(v < s.vdim ? oh[v] * inv * a.norm[v] * silu_f(to_f<T>(gate[h * s.vP + v])) : 0.0f);
        }
        return;
    }
    float ss = 0.0f;
    for (int i = threadIdx.x; i < n; i += 256)
        if (i % s.vP < s.vdim) ss = fmaf(o[i], o[i], ss);
    const float inv = 1.0f / sqrtf(block_sum_f(ss, sh) / (float)(s.heads * s.vdim) + s.eps);
    T *out = static_cast<T *>(a.out) + (size_t)m * a.ldo;
    for (int i = threadIdx.x; i < n; i += 256) out[i] = from_f<T>(i % s.vP < s.vdim ? o[i] * inv * a.norm[i] * sigmoid_f(to_f<T>(gate[i])) : 0.0f);
}

constexpr size_t kLinearSmemMax = 226 * 1024;

template <typename T, int DR>
int step_launch(const LinearArgs &a, cudaStream_t st) {
    const size_t smem = ((size_t)(a.s.gated ? 3 : 2) * kLtBlock * a.s.dim + kLtBlock * kLtCols + (size_t)kLtBlock * kLtSlices * kLtCols) * sizeof(float);
    const dim3 grid(a.s.heads, (a.s.vdim + kLtCols - 1) / kLtCols, a.nseq);
    if (a.s.gated) IM_CUDA_CHECK(launch_k(linear_step_kernel<T, DR, true>, grid, dim3(256), smem, st, a));
    else IM_CUDA_CHECK(launch_k(linear_step_kernel<T, DR, false>, grid, dim3(256), smem, st, a));
    return IM_OK;
}
template <typename T>
int step_any(const LinearArgs &a, cudaStream_t st) {
    const int dr = (a.s.dim + kLtSlices - 1) / kLtSlices;
    if (dr <= 4) return step_launch<T, 4>(a, st);
    if (dr <= 8) return step_launch<T, 8>(a, st);
    if (dr <= 16) return step_launch<T, 16>(a, st);
    if (dr <= 32) return step_launch<T, 32>(a, st);
    if (dr <= 64) return step_launch<T, 64>(a, st);
    return fail(IM_ERR_INVALID, "linear attention is built for key dimensions up to 512 (got %d)", a.s.dim);
}
template <int C, int MW>
int chunk_launch(const LinearArgs &a, int dimK, int bufs, LinearSegments sg, cudaStream_t st) {
    const int vb = (a.s.vdim + kLtCols - 1) / kLtCols;
    if (sg.count > 1) {
        sg.local = 1;
        IM_CUDA_CHECK(launch_k(linear_chunk_kernel<C, MW>, dim3(vb, a.s.heads, sg.count - 1), dim3(C * 2), linear_chunk_smem(C, dimK, bufs), st, a, dimK, bufs, sg));
        sg.local = 0;
    }
    IM_CUDA_CHECK(launch_k(linear_chunk_kernel<C, MW>, dim3(vb, a.s.heads, sg.count > 1 ? sg.count : a.nseq), dim3(C * 2), linear_chunk_smem(C, dimK, bufs), st, a, dimK,
                           bufs, sg));
    return IM_OK;
}
int chunk_any(const LinearArgs &a, int dimK, int bufs, const LinearSegments &sg, cudaStream_t st) {
    return dimK <= 64 ? chunk_launch<64, 1>(a, dimK, bufs, sg, st) : dimK <= 128 ? chunk_launch<64, 2>(a, dimK, bufs, sg, st) : chunk_launch<64, 4>(a, dimK, bufs, sg, st);
}

}  // namespace

int linear_prepare(const Device *dev) {
    static DeviceOnce once;
    if (!once.first(dev->ordinal)) return IM_OK;
#define IM_SMEM(k) IM_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLinearSmemMax))
    IM_SMEM((linear_step_kernel<float, 64, false>)); IM_SMEM((linear_step_kernel<float, 32, false>));
    IM_SMEM((linear_step_kernel<__nv_bfloat16, 64, false>)); IM_SMEM((linear_step_kernel<__nv_bfloat16, 32, false>));
    IM_SMEM((linear_step_kernel<float, 64, true>)); IM_SMEM((linear_step_kernel<float, 32, true>));
    IM_SMEM((linear_step_kernel<__nv_bfloat16, 64, true>)); IM_SMEM((linear_step_kernel<__nv_bfloat16, 32, true>));
    IM_SMEM((linear_chunk_kernel<128, 1>)); IM_SMEM((linear_chunk_kernel<64, 1>)); IM_SMEM((linear_chunk_kernel<64, 2>));
    IM_SMEM((linear_chunk_kernel<64, 4>));
#undef IM_SMEM
    return gated_prepare();
}

int linear_attention_run(const Device *dev, const LinearArgs &a, cudaStream_t st, int *launches) {
    const int dimK = round_up(a.s.dimP, 16), M = a.nseq * a.T;
    int rc = IM_ERR_BOUNDS;
    if (a.s.gated) {
        if (a.T == 1 && gated_decode_takes(a.s)) {
            *launches += 1;
            return gated_decode_run(a, st);
        }
        if (!a.f32 && a.nseq == 1 && a.T >= kGatedChunkMin && gated_chunk_takes(a.s)) {
            rc = gated_chunk_run(a, st, launches);
            if (rc != IM_ERR_BOUNDS) return rc;
        }
    } else if (!a.f32 && a.T >= 16 && dimK <= 256 && linear_chunk_smem(64, dimK, 1) <= kLinearSmemMax) {
        LinearSegments sg;
        sg.sums = a.seg_sums;
        const int ctas = (a.s.vdim + kLtCols - 1) / kLtCols * a.s.heads, per_sm = 2 * linear_chunk_smem(64, dimK, 1) <= kLinearSmemMax ? 2 : 1;
        if (a.nseq == 1 && a.T >= 2 * kLinearPow && a.seg_sums) {  // enough segments to fill the GPU
            const int want = std::min(std::min(per_sm * dev->sm_count / ctas, a.T / kLinearPow), kLinearSegMax);
            if (want > 1) {
                sg.tokens = round_up((a.T + want - 1) / want, kLinearPow);
                sg.count = (a.T + sg.tokens - 1) / sg.tokens;
            }
        }
        if (sg.count > 1) {
            *launches += 1;
            rc = chunk_any(a, dimK, 1, sg, st);
        } else if (a.T > 64 && dimK <= 128 && linear_chunk_smem(128, dimK, 2) <= kLinearSmemMax) {
            rc = chunk_launch<128, 1>(a, dimK, 2, sg, st);
        } else {
            rc = chunk_any(a, dimK, linear_chunk_smem(64, dimK, 2) <= kLinearSmemMax ? 2 : 1, sg, st);
        }
    }
    if (rc == IM_ERR_BOUNDS) rc = a.f32 ? step_any<float>(a, st) : step_any<__nv_bfloat16>(a, st);
    if (rc != IM_OK) return rc;
    if (a.f32) IM_CUDA_CHECK(launch_k(linear_finish_kernel<float>, dim3(M), dim3(256), 0, st, a));
    else IM_CUDA_CHECK(launch_k(linear_finish_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, st, a));
    *launches += 2;
    return IM_OK;
}

}  // namespace im
