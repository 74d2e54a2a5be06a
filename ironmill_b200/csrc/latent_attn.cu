// Latent attention: one cached row per token, [normed latent c | rotated key part], shared by all heads; the keys of head h
// are W_uk[h] c next to the rotated part, its values W_uv[h] c; softmax with an optional keyless sink logit per head.
//
// Two equal forms:
//   absorbed   q' = W_uk^T q is a query against the latents themselves, the weighted sum of latents goes through W_uv at
//              the end: every head reads the same cached row.  Decode, batches and short chunks.
//                latent_absorb_kernel   q', the rotated query part, the token's cache row
//                latent_attn_kernel     16 (token, head) rows per CTA and row tile on the tensor cores, positions split over
//                                       the grid (bf16);  latent_attn_simt_kernel: the same in f32 FMA
//                latent_combine_kernel, latent_out_kernel   splits and sink, then W_uv
//   expanded   keys and values of a group of heads by one GEMM over the cached latents, then a causal tensor-core pass
//              (latent_prefill_kernel).  Prompt chunks in bf16, where it is 3-4 times fewer operations.
// Scores, softmax and sums are f32; on the tensor cores a softmax weight enters the second product as two bf16 terms.
#include <math.h>

#include <algorithm>

#include "stack.cuh"

namespace im {

void latent_layout(LatentShape *s) {
    s->dimP = round_up(s->dim, 8);
    s->rotP = round_up(s->rot_dim, 8);
    s->vP = round_up(s->vdim, 8);
    s->latP = round_up(s->kv_rank, 8);
    s->rowP = round_up(s->latP + s->rotP, 32);
    s->q_off = 0;
    s->c_off = s->heads * (s->dimP + s->rotP);
}

namespace {

struct TokenPlace {
    int slot, pos;
};
__device__ __forceinline__ TokenPlace place_of(const LatentArgs &a, int m) {
    const int s = m / a.T;
    TokenPlace p;
    p.slot = a.slot_map ? a.slot_map[s] : s;
    p.pos = a.pos_dev[p.slot] + m % a.T;
    return p;
}
// element i of the rotated vector src (pairs 2i, 2i + 1)
template <typename T>
__device__ __forceinline__ float rotated(const LatentArgs &a, const T *src, int pos, int i) {
    const int half = a.s.rot_dim / 2, j = i >> 1;
    const float c = a.cosc[(size_t)pos * half + j], s = a.sinc[(size_t)pos * half + j];
    const float u = to_f<T>(src[2 * j]), v = to_f<T>(src[2 * j + 1]);
    return (i & 1) ? v * c + u * s : u * c - v * s;
}

// Cache row of token m: normed latent, rotated key part.  Whole block.
template <typename T>
__device__ void write_row(const LatentArgs &a, int m, float *sh) {
    const TokenPlace p = place_of(a, m);
    if (p.pos >= a.max_seq) return;
    const T *src = static_cast<const T *>(a.y) + (size_t)m * a.ldy + a.s.c_off;
    T *row = static_cast<T *>(a.cache) + ((size_t)p.slot * a.max_seq + p.pos) * a.s.rowP;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.s.kv_rank; i += blockDim.x) {
        const float v = to_f<T>(src[i]);
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum_f(ss, sh) / (float)a.s.kv_rank + a.s.eps);
    for (int i = threadIdx.x; i < a.s.kv_rank; i += blockDim.x) row[i] = from_f<T>(to_f<T>(src[i]) * inv * a.c_norm[i]);
    for (int i = threadIdx.x; i < a.s.rot_dim; i += blockDim.x) row[a.s.latP + i] = from_f<T>(rotated<T>(a, src + a.s.latP, p.pos, i));
}

// Prefill form: cache rows, and the rotated part of every query in place.  One CTA per token.
template <typename T>
__global__ void __launch_bounds__(256) latent_rows_kernel(const LatentArgs a) {
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    const int m = blockIdx.x;
    write_row<T>(a, m, sh);
    const TokenPlace p = place_of(a, m);
    if (p.pos >= a.max_seq) return;
    const int half = a.s.rot_dim / 2, stride = a.s.dimP + a.s.rotP;
    T *q = static_cast<T *>(a.y) + (size_t)m * a.ldy + a.s.q_off + a.s.dimP;
    for (int i = threadIdx.x; i < a.s.heads * half; i += blockDim.x) {
        T *x = q + (size_t)(i / half) * stride + 2 * (i % half);
        const float c = a.cosc[(size_t)p.pos * half + i % half], s = a.sinc[(size_t)p.pos * half + i % half];
        const float u = to_f<T>(x[0]), v = to_f<T>(x[1]);
        x[0] = from_f<T>(u * c - v * s);
        x[1] = from_f<T>(v * c + u * s);
    }
}

// grid (heads + 1, column slices, token groups of MB).  CTA (h, c, g): columns of slice c of q' = W_uk[h]^T q for MB tokens:
// a thread owns one 16-byte column vector and a share of the rows of W_uk[h]; the shares are added in shared memory.
// Slice 0 also writes the rotated part and the zero tail of the query row; CTA (heads, 0, g) writes the cache rows.
template <typename T, int MB>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const LatentArgs a, int M, int cw) {
    constexpr int V = Vec16<T>::n;
    extern __shared__ __align__(16) unsigned char latent_smem[];
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x, m0 = blockIdx.z * MB, nm = min(MB, M - m0);
    const LatentShape &s = a.s;
    if (h == s.heads) {
        if (blockIdx.y == 0)
            for (int i = 0; i < nm; i++) write_row<T>(a, m0 + i, sh);
        return;
    }
    float *qs = reinterpret_cast<float *>(latent_smem);  // [MB][dim]
    float *red = qs + MB * s.dim;                         // [shares][MB][cw]
    const int stride = s.dimP + s.rotP;
    const T *q = static_cast<const T *>(a.y) + s.q_off + (size_t)h * stride;
    for (int i = threadIdx.x; i < MB * s.dim; i += blockDim.x) {
        const int b = i / s.dim, d = i % s.dim;
        qs[i] = b < nm ? to_f<T>(q[(size_t)(m0 + b) * a.ldy + d]) : 0.0f;
    }
    __syncthreads();
    const int nv = cw / V, shares = 256 / nv, sharei = threadIdx.x / nv, vec = threadIdx.x % nv;
    const int c0 = blockIdx.y * cw + vec * V;
    float acc[MB][V];
#pragma unroll
    for (int b = 0; b < MB; b++)
#pragma unroll
        for (int j = 0; j < V; j++) acc[b][j] = 0.0f;
    if (sharei < shares && c0 < s.latP) {
        const T *W = static_cast<const T *>(a.ukv) + (size_t)h * (s.dimP + s.vP) * a.uk_ld + c0;
#pragma unroll 4
        for (int d = sharei; d < s.dim; d += shares) {
            float w[V];
            Vec16<T>::unpack(*reinterpret_cast<const uint4 *>(W + (size_t)d * a.uk_ld), w);
#pragma unroll
            for (int b = 0; b < MB; b++) {
                const float x = qs[b * s.dim + d];
#pragma unroll
                for (int j = 0; j < V; j++) acc[b][j] = fmaf(w[j], x, acc[b][j]);
            }
        }
    }
    if (sharei < shares)
#pragma unroll
        for (int b = 0; b < MB; b++)
#pragma unroll
            for (int j = 0; j < V; j++) red[((size_t)sharei * MB + b) * cw + vec * V + j] = acc[b][j];
    __syncthreads();
    T *out = static_cast<T *>(a.qabs);
    for (int i = threadIdx.x; i < nm * cw; i += blockDim.x) {
        const int b = i / cw, c = i % cw;
        if (blockIdx.y * cw + c >= s.latP) continue;
        float v = 0.0f;
        for (int k = 0; k < shares; k++) v += red[((size_t)k * MB + b) * cw + c];
        out[((size_t)(m0 + b) * s.heads + h) * s.rowP + blockIdx.y * cw + c] = from_f<T>(v);
    }
    if (blockIdx.y == 0) {
        const int tail = s.rowP - s.latP;
        for (int i = threadIdx.x; i < nm * tail; i += blockDim.x) {
            const int b = i / tail, c = i % tail;
            float v = 0.0f;
            if (c < s.rot_dim) {
                const TokenPlace p = place_of(a, m0 + b);
                if (p.pos < a.max_seq) v = rotated<T>(a, q + (size_t)(m0 + b) * a.ldy + s.dimP, p.pos, c);
            }
            out[((size_t)(m0 + b) * s.heads + h) * s.rowP + s.latP + c] = from_f<T>(v);
        }
    }
}

struct LatentPart {
    float *po, *pm, *pl;  // [rows][splits][latP], [rows][splits] x 2
    int splits;
};
// positions [r0, r1) of a split that a tile of rows ending at token t_last reads
__device__ __forceinline__ void split_range(const LatentArgs &a, int seq, int t_last, int split, int splits, int tile, int *pos, int *r0, int *r1) {
    const int slot = a.slot_map ? a.slot_map[seq] : seq;
    *pos = a.pos_dev[slot];
    const int len = min(*pos + a.T, a.max_seq);
    const int chunk = ((len + splits - 1) / splits + tile - 1) / tile * tile;
    *r0 = split * chunk;
    *r1 = min(*r0 + chunk, min(*pos + t_last + 1, a.max_seq));
}

// ---- absorbed form on the tensor cores ---------------------------------------------------------------------------------
// grid (row tiles, splits, sequences), 8 warps.  Rows are (token, head) pairs of one sequence, 16 * MT per CTA.  Per tile of
// 64 positions: warp w scores positions 8w .. 8w + 7 for all rows, the row maxima meet in shared memory, the weights go to
// shared memory as two bf16 terms, and warp w adds up its NV * 8 columns of the weighted latents.
constexpr int kLaN = 64, kLaWarps = 8, kLaPRow = (kLaN + 8) * 2;
template <int MT>
constexpr size_t latent_attn_smem(int rowP) {
    return (size_t)(16 * MT + 2 * kLaN) * (rowP + 8) * 2 + 2 * (size_t)16 * MT * kLaPRow + (size_t)kLaWarps * 16 * MT * 4;
}
template <int NV, int MT>
__global__ void __launch_bounds__(kLaWarps * 32, 1) latent_attn_kernel(const LatentArgs a, const LatentPart part) {
    constexpr int R = 16 * MT, NT = kLaWarps * 32;
    extern __shared__ __align__(16) unsigned char latent_smem[];
    const LatentShape &s = a.s;
    const int rs = (s.rowP + 8) * 2;  // bytes of a row in shared memory
    unsigned char *qs = latent_smem, *kt = qs + R * rs, *ph = kt + 2 * kLaN * rs, *plo = ph + R * kLaPRow;
    float *wmax = reinterpret_cast<float *>(plo + R * kLaPRow);  // [warps][R]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int row0 = blockIdx.x * R, split = blockIdx.y, seq = blockIdx.z, nrows = a.T * s.heads;
    pdl_trigger();
    pdl_wait();
    const int t_last = min(a.T - 1, (row0 + R - 1) / s.heads);
    int pos, r0, r1;
    split_range(a, seq, t_last, split, part.splits, kLaN, &pos, &r0, &r1);
    const size_t grow0 = (size_t)seq * nrows + row0;
    if (r1 <= r0) {
        if (tid < R && row0 + tid < nrows) {
            part.pm[(grow0 + tid) * part.splits + split] = -INFINITY;
            part.pl[(grow0 + tid) * part.splits + split] = 0.0f;
        }
        return;
    }
    const int slot = a.slot_map ? a.slot_map[seq] : seq, nch = s.rowP / 8;
    const __nv_bfloat16 *cache = static_cast<const __nv_bfloat16 *>(a.cache) + (size_t)slot * a.max_seq * s.rowP;
    auto load_tile = [&](int buf, int p0) {
        unsigned char *dst = kt + (size_t)buf * kLaN * rs;
#pragma unroll
        for (int j = 0; j < kLaN / kLaWarps; j++) {  // a warp per cached row
            const int r = warp + j * kLaWarps;
            const __nv_bfloat16 *src = cache + (size_t)min(p0 + r, r1 - 1) * s.rowP;
            for (int c = lane; c < nch; c += 32) cp_async16(dst + r * rs + c * 16, src + c * 8);
        }
        cp_async_commit();
    };
    load_tile(0, r0);
    {
        const __nv_bfloat16 *q = static_cast<const __nv_bfloat16 *>(a.qabs) + grow0 * s.rowP;
        for (int i = tid; i < R * nch; i += NT) {
            const int r = i / nch, c = i % nch;
            *reinterpret_cast<uint4 *>(qs + r * rs + c * 16) =
                row0 + r < nrows ? *reinterpret_cast<const uint4 *>(q + (size_t)r * s.rowP + c * 8) : make_uint4(0, 0, 0, 0);
        }
    }
    int lim[MT][2];  // last position each of this thread's rows sees
    float m_run[MT][2], l_run[MT][2];
    float o[MT][NV][4];
#pragma unroll
    for (int mt = 0; mt < MT; mt++) {
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int r = row0 + mt * 16 + g + 8 * e;
            lim[mt][e] = r < nrows ? pos + r / s.heads : -1;
            m_run[mt][e] = -INFINITY;
            l_run[mt][e] = 0.0f;
        }
#pragma unroll
        for (int n = 0; n < NV; n++) o[mt][n][0] = o[mt][n][1] = o[mt][n][2] = o[mt][n][3] = 0.0f;
    }
    const unsigned qa = (unsigned)__cvta_generic_to_shared(qs) + (lane & 15) * rs + (lane >> 4) * 16;
    const unsigned ka = (unsigned)__cvta_generic_to_shared(kt) + (8 * warp + (lane & 7)) * rs + (lane >> 3) * 16;
    const unsigned va = (unsigned)__cvta_generic_to_shared(kt) + (lane & 15) * rs + (lane >> 4) * 16 + warp * NV * 16;
    const unsigned pa = (unsigned)__cvta_generic_to_shared(ph) + (lane & 15) * kLaPRow + (lane >> 4) * 16;
    const int ntiles = (r1 - r0 + kLaN - 1) / kLaN;
    for (int it = 0; it < ntiles; it++) {
        const int buf = it & 1, p0 = r0 + it * kLaN;
        if (it + 1 < ntiles) {
            load_tile(buf ^ 1, p0 + kLaN);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        float sc[MT][4];
#pragma unroll
        for (int mt = 0; mt < MT; mt++) sc[mt][0] = sc[mt][1] = sc[mt][2] = sc[mt][3] = 0.0f;
#pragma unroll 2
        for (int kk = 0; kk < s.rowP / 32; kk++) {
            unsigned b[4];
            ldsm_x4(b, ka + buf * kLaN * rs + kk * 64);
#pragma unroll
            for (int mt = 0; mt < MT; mt++) {
                unsigned a0[4], a1[4];
                ldsm_x4(a0, qa + mt * 16 * rs + kk * 64);
                ldsm_x4(a1, qa + mt * 16 * rs + kk * 64 + 32);
                mma_bf16(sc[mt], a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
                mma_bf16(sc[mt], a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
            }
        }
        const int pcol = p0 + 8 * warp + 2 * t;
#pragma unroll
        for (int mt = 0; mt < MT; mt++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                float mx = -INFINITY;
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    const int p = pcol + j;
                    float &v = sc[mt][2 * e + j];
                    v = (p <= lim[mt][e] && p < r1) ? v * s.scale : -INFINITY;
                    mx = fmaxf(mx, v);
                }
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                if (t == 0) wmax[warp * R + mt * 16 + g + 8 * e] = mx;
            }
        __syncthreads();
#pragma unroll
        for (int mt = 0; mt < MT; mt++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int row = mt * 16 + g + 8 * e;
                float m_new = m_run[mt][e];
#pragma unroll
                for (int w = 0; w < kLaWarps; w++) m_new = fmaxf(m_new, wmax[w * R + row]);
                const float corr = m_new == -INFINITY ? 1.0f : __expf(m_run[mt][e] - m_new);
                m_run[mt][e] = m_new;
                const float p0v = sc[mt][2 * e] == -INFINITY ? 0.0f : __expf(sc[mt][2 * e] - m_new);
                const float p1v = sc[mt][2 * e + 1] == -INFINITY ? 0.0f : __expf(sc[mt][2 * e + 1] - m_new);
                l_run[mt][e] = l_run[mt][e] * corr + p0v + p1v;
                unsigned terms[2];
                split_bf2<2>(p0v, p1v, terms);
                *reinterpret_cast<unsigned *>(ph + row * kLaPRow + (8 * warp + 2 * t) * 2) = terms[0];
                *reinterpret_cast<unsigned *>(plo + row * kLaPRow + (8 * warp + 2 * t) * 2) = terms[1];
#pragma unroll
                for (int n = 0; n < NV; n++) {
                    o[mt][n][2 * e] *= corr;
                    o[mt][n][2 * e + 1] *= corr;
                }
            }
        __syncthreads();
#pragma unroll
        for (int kb = 0; kb < kLaN / 16; kb++) {
            unsigned hi[MT][4], lo[MT][4];
#pragma unroll
            for (int mt = 0; mt < MT; mt++) {
                ldsm_x4(hi[mt], pa + mt * 16 * kLaPRow + kb * 32);
                ldsm_x4(lo[mt], pa + (R + mt * 16) * kLaPRow + kb * 32);
            }
#pragma unroll
            for (int n = 0; n < NV; n += 2) {
                if ((warp * NV + n) * 8 < s.latP) {
                    unsigned b[4];
                    ldsm_x4_t(b, va + (buf * kLaN + 16 * kb) * rs + n * 16);
#pragma unroll
                    for (int mt = 0; mt < MT; mt++) {
                        mma_bf16(o[mt][n], hi[mt][0], hi[mt][1], hi[mt][2], hi[mt][3], b[0], b[1]);
                        mma_bf16(o[mt][n + 1], hi[mt][0], hi[mt][1], hi[mt][2], hi[mt][3], b[2], b[3]);
                        mma_bf16(o[mt][n], lo[mt][0], lo[mt][1], lo[mt][2], lo[mt][3], b[0], b[1]);
                        mma_bf16(o[mt][n + 1], lo[mt][0], lo[mt][1], lo[mt][2], lo[mt][3], b[2], b[3]);
                    }
                }
            }
        }
        __syncthreads();  // before the next tile's copies land in the other buffer's successor and the weights are rewritten
    }
#pragma unroll
    for (int mt = 0; mt < MT; mt++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            float l = l_run[mt][e];
            l += __shfl_xor_sync(0xffffffffu, l, 1);
            l += __shfl_xor_sync(0xffffffffu, l, 2);
            const int row = mt * 16 + g + 8 * e;
            if (t == 0) wmax[warp * R + row] = l;
            if (warp == 0 && t == 0 && row0 + row < nrows) part.pm[(grow0 + row) * part.splits + split] = m_run[mt][e];
            if (row0 + row < nrows) {
                float *dst = part.po + ((grow0 + row) * part.splits + split) * s.latP;
#pragma unroll
                for (int n = 0; n < NV; n++) {
                    const int col = (warp * NV + n) * 8 + 2 * t;
                    if (col < s.latP) *reinterpret_cast<float2 *>(dst + col) = make_float2(o[mt][n][2 * e], o[mt][n][2 * e + 1]);
                }
            }
        }
    __syncthreads();
    if (tid < R && row0 + tid < nrows) {
        float l = 0.0f;
        for (int w = 0; w < kLaWarps; w++) l += wmax[w * R + tid];
        part.pl[(grow0 + tid) * part.splits + split] = l;
    }
}

// ---- absorbed form in f32 FMA (also shapes the tensor-core kernel does not take) ----------------------------------------
// grid (token * heads + head, splits, sequences), 4 warps; tiles of 128 positions: a warp per position for the scores, a
// thread per latent column (up to 8 of them) for the weighted sum.
constexpr int kLsThreads = 128, kLsTile = 128, kLsCols = 8;
template <typename T>
__global__ void __launch_bounds__(kLsThreads) latent_attn_simt_kernel(const LatentArgs a, const LatentPart part) {
    constexpr int V = Vec16<T>::n;
    extern __shared__ __align__(16) unsigned char latent_smem[];
    float *qs = reinterpret_cast<float *>(latent_smem), *w = qs + a.s.rowP;
    __shared__ float sh[32];
    const LatentShape &s = a.s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x, split = blockIdx.y, seq = blockIdx.z, nrows = a.T * s.heads;
    int pos, r0, r1;
    split_range(a, seq, row / s.heads, split, part.splits, kLsTile, &pos, &r0, &r1);
    const size_t grow = (size_t)seq * nrows + row;
    if (r1 <= r0) {
        if (tid == 0) {
            part.pm[grow * part.splits + split] = -INFINITY;
            part.pl[grow * part.splits + split] = 0.0f;
        }
        return;
    }
    const int slot = a.slot_map ? a.slot_map[seq] : seq;
    const T *cache = static_cast<const T *>(a.cache) + (size_t)slot * a.max_seq * s.rowP;
    const T *q = static_cast<const T *>(a.qabs) + grow * s.rowP;
    for (int i = tid; i < s.rowP; i += kLsThreads) qs[i] = to_f<T>(q[i]);
    float m = -INFINITY, l = 0.0f, acc[kLsCols];
#pragma unroll
    for (int c = 0; c < kLsCols; c++) acc[c] = 0.0f;
    for (int p0 = r0; p0 < r1; p0 += kLsTile) {
        __syncthreads();
        const int n = min(kLsTile, r1 - p0);
        for (int j = warp; j < n; j += kLsThreads / 32) {
            const uint4 *kr = reinterpret_cast<const uint4 *>(cache + (size_t)(p0 + j) * s.rowP);
            float dot = 0.0f;
            for (int i = lane; i < s.rowP / V; i += 32) {
                float k[V];
                Vec16<T>::unpack(kr[i], k);
#pragma unroll
                for (int e = 0; e < V; e++) dot = fmaf(qs[i * V + e], k[e], dot);
            }
            dot = warp_sum(dot);
            if (lane == 0) w[j] = dot * s.scale;
        }
        __syncthreads();
        const float sv = tid < n ? w[tid] : -INFINITY;
        float mx = warp_max(sv);
        if (lane == 0) sh[warp] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(sh[0], sh[1]), fmaxf(sh[2], sh[3]));
        const float m_new = fmaxf(m, mx), corr = expf(m - m_new);
        m = m_new;
        const float e = tid < n ? expf(sv - m) : 0.0f;
        w[tid] = e;
        l = l * corr + block_sum_f(e, sh);
#pragma unroll
        for (int c = 0; c < kLsCols; c++) acc[c] *= corr;
        for (int j = 0; j < n; j++) {
            const T *vr = cache + (size_t)(p0 + j) * s.rowP;
            const float wj = w[j];
#pragma unroll
            for (int c = 0; c < kLsCols; c++)
                if (tid + c * kLsThreads < s.latP) acc[c] = fmaf(wj, to_f<T>(vr[tid + c * kLsThreads]), acc[c]);
        }
    }
#pragma unroll
    for (int c = 0; c < kLsCols; c++)
        if (tid + c * kLsThreads < s.latP) part.po[(grow * part.splits + split) * s.latP + tid + c * kLsThreads] = acc[c];
    if (tid == 0) {
        part.pm[grow * part.splits + split] = m;
        part.pl[grow * part.splits + split] = l;
    }
}

// Weight of split k of a row in the normalised sum: exp(m_k - m) / (sum + sink)
__device__ __forceinline__ float row_norm(const LatentPart &p, size_t row, float sink, float *gm_out) {
    float gm = sink;
    for (int k = 0; k < p.splits; k++) gm = fmaxf(gm, p.pm[row * p.splits + k]);
    float l = sink == -INFINITY ? 0.0f : expf(sink - gm);
    for (int k = 0; k < p.splits; k++) {
        const float m = p.pm[row * p.splits + k];
        if (m != -INFINITY) l += p.pl[row * p.splits + k] * expf(m - gm);
    }
    *gm_out = gm;
    return 1.0f / l;
}

// grid (rows, column blocks of 128), GR groups of 128 threads: the splits of a row (at most 256, or 128 for one group) added
// up, a share of them per group, and normalised
template <int GR>
__global__ void __launch_bounds__(GR * 128) latent_combine_kernel(const LatentPart p, const float *__restrict__ sink, int heads, int latP, float *__restrict__ out) {
    constexpr int NW = GR == 1 ? 4 : 8;  // warps that hold a split's maximum
    __shared__ float wk[NW * 32], sm[NW], sl[NW], part[GR][128];
    const size_t row = blockIdx.x;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const float s = sink ? sink[row % heads] : -INFINITY;
    pdl_trigger();
    pdl_wait();
    float m = -INFINITY, l = 0.0f;
    if (tid < p.splits) {
        m = p.pm[row * p.splits + tid];
        l = p.pl[row * p.splits + tid];
    }
    const float wm = warp_max(m);
    if (lane == 0 && warp < NW) sm[warp] = wm;
    __syncthreads();
    float gm = s;
#pragma unroll
    for (int i = 0; i < NW; i++) gm = fmaxf(gm, sm[i]);
    const float w = m == -INFINITY ? 0.0f : expf(m - gm), ws = warp_sum(l * w);
    if (warp < NW) wk[tid] = w;
    if (lane == 0 && warp < NW) sl[warp] = ws;
    __syncthreads();
    float sum = s == -INFINITY ? 0.0f : expf(s - gm);
#pragma unroll
    for (int i = 0; i < NW; i++) sum += sl[i];
    const int grp = tid >> 7, c = blockIdx.y * 128 + (tid & 127);
    const int per = (p.splits + GR - 1) / GR, k0 = grp * per, k1 = min(p.splits, k0 + per);
    float acc = 0.0f;
    if (c < latP) {
        const float *src = p.po + row * p.splits * latP + c;
#pragma unroll 8
        for (int k = k0; k < k1; k++) {
            const float v = src[(size_t)k * latP], wt = wk[k];  // a split without positions left its sums unwritten
            acc += wt == 0.0f ? 0.0f : wt * v;
        }
    }
    if (GR > 1) {
        part[grp][tid & 127] = acc;
        __syncthreads();
#pragma unroll
        for (int i = 1; i < GR; i++) acc += part[i][tid & 127];
    }
    if (grp == 0 && c < latP) out[row * latP + c] = acc / sum;
}

// grid (heads, slices of the value rows, token groups of MB): out[m, h] = W_uv[h] o'.  src: the normalised sums, or (single
// split) the partials of the attention kernel, normalised here.
template <typename T, int MB>
__global__ void __launch_bounds__(256) latent_out_kernel(const LatentArgs a, const LatentPart p, const float *__restrict__ src, int normalised, int M, int rows_per) {
    constexpr int V = Vec16<T>::n;
    extern __shared__ __align__(16) unsigned char latent_smem[];
    float *os = reinterpret_cast<float *>(latent_smem);  // [MB][latP]
    pdl_trigger();
    pdl_wait();
    const LatentShape &s = a.s;
    const int h = blockIdx.x, m0 = blockIdx.z * MB, nm = min(MB, M - m0), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int b = 0; b < MB; b++) {
        const size_t row = (size_t)(m0 + min(b, nm - 1)) * s.heads + h;
        float inv = 1.0f;
        if (!normalised) {  // one split: exp(m - max(m, sink)) / (l exp(m - max) + exp(sink - max))
            float gm;
            inv = row_norm(p, row, a.sink ? a.sink[h] : -INFINITY, &gm);
            inv *= expf(p.pm[row] - gm);
        }
        for (int i = threadIdx.x; i < s.latP; i += 256) os[b * s.latP + i] = src[row * s.latP + i] * inv;
    }
    __syncthreads();
    const T *W = static_cast<const T *>(a.ukv) + ((size_t)h * (s.dimP + s.vP) + s.dimP) * a.uk_ld;
    const int v0 = blockIdx.y * rows_per, v1 = min(v0 + rows_per, s.vdim);
    for (int v = v0 + warp; v < v1; v += 8) {
        float acc[MB];
#pragma unroll
        for (int b = 0; b < MB; b++) acc[b] = 0.0f;
        for (int i = lane; i < s.latP / V; i += 32) {
            float w[V];
            Vec16<T>::unpack(*reinterpret_cast<const uint4 *>(W + (size_t)v * a.uk_ld + i * V), w);
#pragma unroll
            for (int b = 0; b < MB; b++)
#pragma unroll
                for (int j = 0; j < V; j++) acc[b] = fmaf(w[j], os[b * s.latP + i * V + j], acc[b]);
        }
#pragma unroll
        for (int b = 0; b < MB; b++) {
            acc[b] = warp_sum(acc[b]);
            if (lane == 0 && b < nm) static_cast<T *>(a.out)[(size_t)(m0 + b) * a.ldo + h * s.vP + v] = from_f<T>(acc[b]);
        }
    }
}

// ---- expanded form ------------------------------------------------------------------------------------------------------
// grid (ceil(T / 64), heads of the group), 4 warps of 16 tokens, three such CTAs per SM.  K tile: [expanded key | rotated part of the cache row].
constexpr int kLpM = 64, kLpN = 32, kLpThreads = kLpM * 2, kLpNB = kLpN / 8;
inline int prefill_qk(const LatentShape &s) { return round_up(s.dimP + s.rotP, 32); }
inline size_t latent_prefill_smem(const LatentShape &s, int dv) { return (size_t)(kLpM + 2 * kLpN) * (prefill_qk(s) + 8) * 2 + (size_t)2 * kLpN * (dv + 8) * 2; }

template <int DV>  // value columns, padded
__global__ void __launch_bounds__(kLpThreads, DV <= 128 ? 3 : 1) latent_prefill_kernel(const LatentArgs a, const __nv_bfloat16 *__restrict__ kv, int ldkv, int h0, int qk) {
    constexpr int NT = kLpThreads, ND = DV / 8;
    extern __shared__ __align__(16) unsigned char latent_smem[];
    const LatentShape &s = a.s;
    const int rs = (qk + 8) * 2, vs = (DV + 8) * 2;
    unsigned char *qs = latent_smem, *kt = qs + kLpM * rs, *vt = kt + 2 * kLpN * rs;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int tb = gridDim.x - 1 - blockIdx.x, hl = blockIdx.y, h = h0 + hl;  // latest (longest) blocks first
    pdl_trigger();
    pdl_wait();
    const int P = a.host_pos;
    const __nv_bfloat16 *cache = static_cast<const __nv_bfloat16 *>(a.cache) + (size_t)a.host_slot * a.max_seq * s.rowP;
    const __nv_bfloat16 *q = static_cast<const __nv_bfloat16 *>(a.y) + s.q_off + (size_t)h * (s.dimP + s.rotP);
    const int nq = (s.dimP + s.rotP) / 8, nk = s.dimP / 8, nr = s.rotP / 8, nvv = s.vP / 8;
    // padding columns once; everything else is overwritten by the copies
    for (int i = tid; i < (kLpM + 2 * kLpN) * (qk / 8); i += NT)
        if (i % (qk / 8) >= nq) *reinterpret_cast<uint4 *>(qs + (size_t)(i / (qk / 8)) * rs + (i % (qk / 8)) * 16) = make_uint4(0, 0, 0, 0);
    for (int i = tid; i < 2 * kLpN * (DV / 8); i += NT)
        if (i % (DV / 8) >= nvv) *reinterpret_cast<uint4 *>(vt + (size_t)(i / (DV / 8)) * vs + (i % (DV / 8)) * 16) = make_uint4(0, 0, 0, 0);
    for (int i = tid; i < kLpM * nq; i += NT) {
        const int r = i / nq, c = i % nq, tok = tb * kLpM + r;
        *reinterpret_cast<uint4 *>(qs + r * rs + c * 16) = tok < a.T ? *reinterpret_cast<const uint4 *>(q + (size_t)tok * a.ldy + c * 8) : make_uint4(0, 0, 0, 0);
    }
    const int n_end = P + min(tb * kLpM + kLpM, a.T);
    const int ntiles = (n_end + kLpN - 1) / kLpN;
    auto load_tile = [&](int buf, int p0) {
        const __nv_bfloat16 *kvh = kv + (size_t)hl * (s.dimP + s.vP);
        unsigned char *kd = kt + (size_t)buf * kLpN * rs, *vd = vt + (size_t)buf * kLpN * vs;
        // the chunks of a row: [key | value] as they lie in kv, then the rotated part from the cache
        for (int r = warp; r < kLpN; r += kLpThreads / 32) {
            const size_t p = (size_t)min(p0 + r, n_end - 1);
            const __nv_bfloat16 *krow = kvh + p * ldkv, *rrow = cache + p * s.rowP + s.latP;
            for (int c = lane; c < nk + nvv + nr; c += 32) {
                const bool key = c < nk, rot = c >= nk + nvv;
                unsigned char *dst = key ? kd + r * rs + c * 16 : rot ? kd + r * rs + (c - nvv) * 16 : vd + r * vs + (c - nk) * 16;
                cp_async16(dst, rot ? rrow + (c - nk - nvv) * 8 : krow + c * 8);
            }
        }
        cp_async_commit();
    };
    load_tile(0, 0);
    const int tok0 = tb * kLpM + warp * 16 + g, tok1 = tok0 + 8;
    const int lim[2] = {tok0 < a.T ? P + tok0 : -1, tok1 < a.T ? P + tok1 : -1};
    const int warp_end = P + min(tb * kLpM + warp * 16 + 16, a.T);  // tiles from here on are masked for the whole warp
    const int warp_full = tb * kLpM + warp * 16 + 16 <= a.T ? P + tb * kLpM + warp * 16 : -1;  // every row sees the positions up to here
    constexpr float kLog2e = 1.4426950408889634f;
    const float scale2 = s.scale * kLog2e;  // scores in units of log 2: one exponential instruction each
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
    float o[ND][4];
#pragma unroll
    for (int i = 0; i < ND; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const unsigned qa = (unsigned)__cvta_generic_to_shared(qs) + (warp * 16 + (lane & 15)) * rs + (lane >> 4) * 16;
    const unsigned ka = (unsigned)__cvta_generic_to_shared(kt) + (lane & 7) * rs + (lane >> 3) * 16;
    const unsigned va = (unsigned)__cvta_generic_to_shared(vt) + (lane & 15) * vs + (lane >> 4) * 16;
    for (int it = 0; it < ntiles; it++) {
        const int buf = it & 1, p0 = it * kLpN;
        if (it + 1 < ntiles) {
            load_tile(buf ^ 1, p0 + kLpN);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        if (p0 < warp_end) {
            float sc[kLpNB][4];
#pragma unroll
            for (int nb = 0; nb < kLpNB; nb++) sc[nb][0] = sc[nb][1] = sc[nb][2] = sc[nb][3] = 0.0f;
#pragma unroll 2
            for (int kk = 0; kk < qk / 32; kk++) {
                unsigned a0[4], a1[4];
                ldsm_x4(a0, qa + kk * 64);
                ldsm_x4(a1, qa + kk * 64 + 32);
#pragma unroll
                for (int nb = 0; nb < kLpNB; nb++) {
                    unsigned b[4];
                    ldsm_x4(b, ka + (buf * kLpN + 8 * nb) * rs + kk * 64);
                    mma_bf16(sc[nb], a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
                    mma_bf16(sc[nb], a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
                }
            }
            float corr[2], mx[2] = {-INFINITY, -INFINITY};
            if (p0 + kLpN - 1 <= warp_full) {
#pragma unroll
                for (int nb = 0; nb < kLpNB; nb++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        sc[nb][e] *= scale2;
                        mx[e >> 1] = fmaxf(mx[e >> 1], sc[nb][e]);
                    }
            } else {
#pragma unroll
                for (int nb = 0; nb < kLpNB; nb++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int p = p0 + 8 * nb + 2 * t + (e & 1);
                        sc[nb][e] = p <= lim[e >> 1] ? sc[nb][e] * scale2 : -INFINITY;
                        mx[e >> 1] = fmaxf(mx[e >> 1], sc[nb][e]);
                    }
            }
            bool moved = false;
#pragma unroll
            for (int r = 0; r < 2; r++) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                const float m_new = fmaxf(m_run[r], mx[r]);
                moved |= m_new > m_run[r];
                corr[r] = m_new == -INFINITY ? 1.0f : exp2f(m_run[r] - m_new);
                m_run[r] = m_new;
                l_run[r] *= corr[r];
            }
            if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
                for (int i = 0; i < ND; i++) {
                    o[i][0] *= corr[0]; o[i][1] *= corr[0];
                    o[i][2] *= corr[1]; o[i][3] *= corr[1];
                }
            }
            const float base[2] = {m_run[0] == -INFINITY ? 0.0f : m_run[0], m_run[1] == -INFINITY ? 0.0f : m_run[1]};
#pragma unroll
            for (int kb = 0; kb < kLpN / 16; kb++) {
                unsigned hi[4], lo[4];
#pragma unroll
                for (int hb = 0; hb < 2; hb++)
#pragma unroll
                    for (int r = 0; r < 2; r++) {
                        const float s0 = sc[2 * kb + hb][2 * r], s1 = sc[2 * kb + hb][2 * r + 1];
                        const float w0 = exp2f(s0 - base[r]), w1 = exp2f(s1 - base[r]);  // a masked score gives zero
                        l_run[r] += w0 + w1;
                        unsigned terms[2];
                        split_bf2<2>(w0, w1, terms);
                        hi[2 * hb + r] = terms[0];
                        lo[2 * hb + r] = terms[1];
                    }
#pragma unroll
                for (int nd = 0; nd < ND; nd += 2) {
                    unsigned b[4];
                    ldsm_x4_t(b, va + (buf * kLpN + 16 * kb) * vs + nd * 16);
                    mma_bf16(o[nd], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                    mma_bf16(o[nd + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                    mma_bf16(o[nd], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
                    mma_bf16(o[nd + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
    const float sink = a.sink ? a.sink[h] * kLog2e : -INFINITY;
#pragma unroll
    for (int r = 0; r < 2; r++) {
        float l = l_run[r];
        l += __shfl_xor_sync(0xffffffffu, l, 1);
        l += __shfl_xor_sync(0xffffffffu, l, 2);
        const int tok = r == 0 ? tok0 : tok1;
        if (tok < a.T) {
            const float gm = fmaxf(m_run[r], sink), c = exp2f(m_run[r] - gm);
            const float inv = c / (l * c + (sink == -INFINITY ? 0.0f : exp2f(sink - gm)));
            __nv_bfloat16 *dst = static_cast<__nv_bfloat16 *>(a.out) + (size_t)tok * a.ldo + h * s.vP;
#pragma unroll
            for (int nd = 0; nd < ND; nd++) {
                const int c2 = 8 * nd + 2 * t;
                if (c2 < s.vP) *reinterpret_cast<unsigned *>(dst + c2) = pack_bf2(o[nd][2 * r] * inv, o[nd][2 * r + 1] * inv);
            }
        }
    }
}

// ---- host ---------------------------------------------------------------------------------------------------------------
constexpr size_t kLatentSmemMax = 220 * 1024;
bool tc_takes(const LatentShape &s) { return s.latP <= kLaWarps * 16 * 8 && latent_attn_smem<1>(s.rowP) <= kLatentSmemMax; }
int rows_per_tile(const LatentShape &s, int T, bool tc) {
    if (!tc) return 1;
    return T * s.heads > 16 && s.latP <= kLaWarps * 8 * 8 && latent_attn_smem<2>(s.rowP) <= kLatentSmemMax ? 32 : 16;
}
int auto_splits(const Device *dev, const LatentShape &s, int f32, int T, int nseq, int ctx) {
    const bool tc = !f32 && tc_takes(s);
    const int per = rows_per_tile(s, T, tc), ctas = (T * s.heads + per - 1) / per * nseq, unit = tc ? kLaN : kLsTile;
    int n = dev->sm_count * (tc ? 1 : 4) / ctas;
    n = std::min(n, (ctx + unit - 1) / unit);
    return std::max(1, std::min(n, 256));
}
size_t part_bytes_for(const LatentShape &s, size_t rows, int splits) { return rows * ((size_t)splits * (s.latP + 2) + s.latP) * sizeof(float); }

template <int NV, int MT>
int attn_launch(const LatentArgs &a, const LatentPart &p, cudaStream_t st) {
    IM_CUDA_CHECK(launch_k(latent_attn_kernel<NV, MT>, dim3((a.T * a.s.heads + 16 * MT - 1) / (16 * MT), p.splits, a.nseq), dim3(kLaWarps * 32),
                           latent_attn_smem<MT>(a.s.rowP), st, a, p));
    return IM_OK;
}
template <int MT>
int attn_tc(const LatentArgs &a, const LatentPart &p, cudaStream_t st) {
    const int tiles = (a.s.latP + 63) / 64;  // value columns per warp / 8
    if (tiles <= 2) return attn_launch<2, MT>(a, p, st);
    if (tiles <= 4) return attn_launch<4, MT>(a, p, st);
    if (tiles <= 8 || MT == 2) return attn_launch<8, MT>(a, p, st);
    return attn_launch<16, 1>(a, p, st);
}

template <typename T, int MB>
int absorb_launch(const LatentArgs &a, int M, cudaStream_t st) {
    constexpr int V = Vec16<T>::n;
    int cs = std::max(1, std::min(8, a.s.latP / 128));  // column slices
    int cw = round_up((a.s.latP + cs - 1) / cs, V);
    while (cw / V > 256) {  // a thread per column vector
        cs *= 2;
        cw = round_up((a.s.latP + cs - 1) / cs, V);
    }
    const int shares = 256 / (cw / V);
    const size_t smem = ((size_t)MB * a.s.dim + (size_t)shares * MB * cw) * sizeof(float);
    IM_CUDA_CHECK(launch_k(latent_absorb_kernel<T, MB>, dim3(a.s.heads + 1, cs, (M + MB - 1) / MB), dim3(256), smem, st, a, M, cw));
    return IM_OK;
}
template <typename T, int MB>
int out_launch(const LatentArgs &a, const LatentPart &p, const float *src, int normalised, int M, cudaStream_t st) {
    const int vs = std::max(1, std::min(8, a.s.vdim / 32)), rows_per = (a.s.vdim + vs - 1) / vs;
    IM_CUDA_CHECK(launch_k(latent_out_kernel<T, MB>, dim3(a.s.heads, vs, (M + MB - 1) / MB), dim3(256), (size_t)MB * a.s.latP * sizeof(float), st, a, p, src, normalised,
                           M, rows_per));
    return IM_OK;
}

template <int DV>
int prefill_launch(const LatentArgs &a, const __nv_bfloat16 *kv, int ldkv, int h0, int nh, cudaStream_t st) {
    IM_CUDA_CHECK(launch_k(latent_prefill_kernel<DV>, dim3((a.T + kLpM - 1) / kLpM, nh), dim3(kLpThreads), latent_prefill_smem(a.s, DV), st, a, kv, ldkv, h0, prefill_qk(a.s)));
    return IM_OK;
}
int prefill_dv(const LatentShape &s) { return s.vP <= 32 ? 32 : s.vP <= 64 ? 64 : s.vP <= 128 ? 128 : s.vP <= 256 ? 256 : 0; }

}  // namespace

bool latent_expands(const LatentShape &s) { return prefill_dv(s) > 0 && latent_prefill_smem(s, prefill_dv(s)) <= kLatentSmemMax; }

int latent_prepare(const Device *dev) {
    static DeviceOnce once;
    if (!once.first(dev->ordinal)) return IM_OK;
    const int mx = (int)kLatentSmemMax;
#define IM_SMEM(k) IM_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, mx))
    IM_SMEM((latent_attn_kernel<2, 1>)); IM_SMEM((latent_attn_kernel<4, 1>)); IM_SMEM((latent_attn_kernel<8, 1>)); IM_SMEM((latent_attn_kernel<16, 1>));
    IM_SMEM((latent_attn_kernel<2, 2>)); IM_SMEM((latent_attn_kernel<4, 2>)); IM_SMEM((latent_attn_kernel<8, 2>));
    IM_SMEM(latent_prefill_kernel<32>); IM_SMEM(latent_prefill_kernel<64>); IM_SMEM(latent_prefill_kernel<128>); IM_SMEM(latent_prefill_kernel<256>);
    IM_SMEM((latent_absorb_kernel<float, 1>)); IM_SMEM((latent_absorb_kernel<float, 4>));
    IM_SMEM((latent_absorb_kernel<__nv_bfloat16, 1>)); IM_SMEM((latent_absorb_kernel<__nv_bfloat16, 4>));
    IM_SMEM((latent_out_kernel<float, 1>)); IM_SMEM((latent_out_kernel<float, 4>));
    IM_SMEM((latent_out_kernel<__nv_bfloat16, 1>)); IM_SMEM((latent_out_kernel<__nv_bfloat16, 4>));
#undef IM_SMEM
    return IM_OK;
}

// Scratch for the partials of `tokens` tokens in `nseq` sequences, whatever the context.
size_t latent_part_bytes(const Device *dev, const LatentShape &s, int tokens, int nseq) {
    const int T = (tokens + nseq - 1) / nseq;
    size_t b = 0;
    for (int f32 = 0; f32 < 2; f32++) b = std::max(b, part_bytes_for(s, (size_t)tokens * s.heads, auto_splits(dev, s, f32, T, nseq, 1 << 30)));
    return b;
}

int latent_attention_run(const Device *dev, const LatentArgs &a, cudaStream_t st, int *launches) {
    const LatentShape &s = a.s;
    const int M = a.nseq * a.T;
    const int dv = prefill_dv(s);
    const size_t per_head = (size_t)(s.dimP + s.vP) * 2;
    if (!a.f32 && a.nseq == 1 && a.host_slot >= 0 && a.T >= kLatentExpandMin && latent_expands(s) && a.kv) {
        const int ctx = a.host_pos + a.T;
        const int group = (int)std::min<size_t>(s.heads, a.kv_bytes / (per_head * ctx));
        if (group >= 1) {
            IM_CUDA_CHECK(launch_k(latent_rows_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, st, a));
            *launches += 1;
            const __nv_bfloat16 *lat = static_cast<const __nv_bfloat16 *>(a.cache) + (size_t)a.host_slot * a.max_seq * s.rowP;
            for (int h0 = 0; h0 < s.heads; h0 += group) {
                const int nh = std::min(group, s.heads - h0), ldkv = nh * (s.dimP + s.vP);
                DenseWeight w;
                w.N = ldkv; w.K = s.kv_rank; w.ld = a.uk_ld; w.f32 = 0;
                w.w = const_cast<__nv_bfloat16 *>(static_cast<const __nv_bfloat16 *>(a.ukv) + (size_t)h0 * (s.dimP + s.vP) * a.uk_ld);
                DenseSrc src;
                src.x = lat; src.ldx = s.rowP;
                DenseEpi e;
                e.y = a.kv; e.ldy = ldkv; e.pair0 = 1 << 30;
                int rc = dense_project(dev, w, src, e, ctx, nullptr, st);
                if (rc != IM_OK) return rc;
                const __nv_bfloat16 *kv = static_cast<const __nv_bfloat16 *>(a.kv);
                rc = dv == 32 ? prefill_launch<32>(a, kv, ldkv, h0, nh, st) : dv == 64 ? prefill_launch<64>(a, kv, ldkv, h0, nh, st)
                     : dv == 128 ? prefill_launch<128>(a, kv, ldkv, h0, nh, st) : prefill_launch<256>(a, kv, ldkv, h0, nh, st);
                if (rc != IM_OK) return rc;
                *launches += 2;
            }
            return IM_OK;
        }
    }
    int rc;
    if (a.f32) rc = M >= 4 ? absorb_launch<float, 4>(a, M, st) : absorb_launch<float, 1>(a, M, st);
    else rc = M >= 4 ? absorb_launch<__nv_bfloat16, 4>(a, M, st) : absorb_launch<__nv_bfloat16, 1>(a, M, st);
    if (rc != IM_OK) return rc;
    const bool tc = !a.f32 && tc_takes(s);
    int splits = auto_splits(dev, s, a.f32, a.T, a.nseq, a.splits_ctx);
    const size_t rows = (size_t)M * s.heads;
    while (splits > 1 && part_bytes_for(s, rows, splits) > a.part_bytes) splits--;
    if (part_bytes_for(s, rows, splits) > a.part_bytes) return fail(IM_ERR_BOUNDS, "latent attention scratch is too small for %d tokens", M);
    LatentPart p;
    p.splits = splits;
    p.po = a.part;
    p.pm = p.po + rows * splits * s.latP;
    p.pl = p.pm + rows * splits;
    float *comb = p.pl + rows * splits;
    if (tc) {
        rc = rows_per_tile(s, a.T, true) == 32 ? attn_tc<2>(a, p, st) : attn_tc<1>(a, p, st);
        if (rc != IM_OK) return rc;
    } else {
        if (s.latP > kLsThreads * kLsCols) return fail(IM_ERR_INVALID, "kv_rank %d is larger than %d", s.kv_rank, kLsThreads * kLsCols);
        const size_t smem = (size_t)(s.rowP + kLsTile) * sizeof(float);
        const dim3 grid(a.T * s.heads, splits, a.nseq);
        if (a.f32) IM_CUDA_CHECK(launch_k(latent_attn_simt_kernel<float>, grid, dim3(kLsThreads), smem, st, a, p));
        else IM_CUDA_CHECK(launch_k(latent_attn_simt_kernel<__nv_bfloat16>, grid, dim3(kLsThreads), smem, st, a, p));
    }
    const float *src = p.po;
    if (splits > 1) {
        const dim3 grid((unsigned)rows, (s.latP + 127) / 128);
        if (splits > 32) IM_CUDA_CHECK(launch_k(latent_combine_kernel<4>, grid, dim3(512), 0, st, p, a.sink, s.heads, s.latP, comb));
        else IM_CUDA_CHECK(launch_k(latent_combine_kernel<1>, grid, dim3(128), 0, st, p, a.sink, s.heads, s.latP, comb));
        src = comb;
        *launches += 1;
    }
    if (a.f32) rc = M >= 4 ? out_launch<float, 4>(a, p, src, splits > 1, M, st) : out_launch<float, 1>(a, p, src, splits > 1, M, st);
    else rc = M >= 4 ? out_launch<__nv_bfloat16, 4>(a, p, src, splits > 1, M, st) : out_launch<__nv_bfloat16, 1>(a, p, src, splits > 1, M, st);
    *launches += 3;
    return rc;
}

}  // namespace im
