// Building blocks of models described by a list of layers (stack.cu): dense bf16 / f32 projections with fused
// prologues and epilogues (dense.cu), latent attention over a cache of latents (latent_attn.cu), grouped-query attention
// over cached keys and values (grouped_attn.cu), decayed linear attention with a recurrent state (linear_attn.cu, and
// linear_gated.cu for decays that depend on the token).  Every block takes its sizes and constants as arguments.
//
// Element type: `f32 == 0` keeps activations, weights and latent caches in bf16 (products accumulate in f32), `f32 == 1`
// keeps all of them in f32 and never touches a reduced-precision unit.  The residual, norms, attention scores and
// weights, recurrent states and logits are f32 in both.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace im {

inline int round_up(int v, int m) { return (v + m - 1) / m * m; }
inline size_t elem_size(int f32) { return f32 ? 4 : 2; }

// ---- dense projections ---------------------------------------------------------------------------------------------
struct DenseWeight {
    int N = 0, K = 0, ld = 0;  // rows, columns, row stride in elements (a multiple of 8; columns K .. ld - 1 are zero)
    int f32 = 0;
    void *w = nullptr;
};

// What the projection reads: activations as they are; rms(xf) * gamma; the two f32 vectors [xf | xf2] side by side; or
// r = xf + rms(xf2) * gamma (the residual with a sublayer's output normed and added), then rms(r) * gamma2 if gamma2 is there.
// With xf2 == nullptr that is r = xf.  r goes to xout as well, if given (not the buffer xf).
enum { kSrcPlain = 0, kSrcNorm = 1, kSrcConcat = 2, kSrcAddNorm = 3 };
struct DenseSrc {
    int kind = kSrcPlain;
    const void *x = nullptr;      // kSrcPlain: elements [M, ldx]
    const float *xf = nullptr, *xf2 = nullptr;  // f32 [M, ldx]
    const float *gamma = nullptr, *gamma2 = nullptr;
    float *xout = nullptr;
    int ldx = 0;
    int width = 0;                // columns of xf (and of xf2)
    float eps = 0.0f;
};

// Where it goes.  kEpiProj: rows below `pair0` to y (rows below `silu_end` through SiLU), except that rows from `f0` on (a multiple
// of eight) go to xf as f32, columns from 0; rows from `pair0` on are (gate, up) pairs, act(gate) * up to act, with gelu_tanh or
// (pair_silu) SiLU.  kEpiResidual: xf[m, n] += sum.  kEpiF32: xf[m, n] = sum (+ bias[n]),
// then cap * tanh(. / cap) when cap > 0.
enum { kEpiProj = 0, kEpiResidual = 1, kEpiF32 = 2 };
struct DenseEpi {
    int kind = kEpiProj;
    int silu_end = 0, pair0 = 0, f0 = 1 << 30;
    int pair_silu = 0;
    void *y = nullptr, *act = nullptr;
    float *xf = nullptr;
    const float *bias = nullptr;
    int ldy = 0, ldact = 0, ldx = 0;
    float cap = 0.0f;
};

constexpr int kDenseGemmMin = 16;  // tokens from which a projection is a dense contraction
constexpr int kDenseMaxRows = 8;   // tokens per matvec launch

// y = W x for M tokens.  h_scratch: M x round_up(K, 8) elements, used when the source is not plain and M >= kDenseGemmMin.
int dense_project(const Device *dev, const DenseWeight &w, const DenseSrc &src, const DenseEpi &epi, int M, void *h_scratch, cudaStream_t st);
// Sets every launch attribute of this file's kernels on the current device (so that a capture can be their first use).
int dense_prepare(const Device *dev);
int dense_launches(int M, int K, int src_kind);

// x[m] = x0[m] = rms(table[token]) * gamma, or without gamma table[token] * scale (f32); tokens past the vocabulary read as zeros.
int stack_embed(const uint32_t *tokens, const void *table, int f32, int ld, const float *gamma, float scale, float *x, float *x0, int width, uint32_t vocab, float eps,
                int M, cudaStream_t st);

// ---- latent attention ------------------------------------------------------------------------------------------------
// Per head a query [dim | rot_dim], a cached latent c (kv_rank, normed) and one rotated key part (rot_dim) shared by the
// heads; keys W_uk c, values W_uv c; softmax with an optional sink logit per head.
struct LatentShape {
    int heads, dim, rot_dim, vdim, kv_rank;
    float scale, eps;
    // padded strides (elements)
    int dimP, rotP, vP;    // per-head parts of the projected row, multiples of 8
    int latP, rowP;        // cache row: [latent, latP | rotated key | zeros], rowP in all (multiple of 32)
    int q_off, c_off;      // where the queries and the latent | key part sit in a projected row
};
void latent_layout(LatentShape *s);

struct LatentArgs {
    LatentShape s;
    int f32;
    void *y;                 // projected rows [M, ldy] (queries are rotated in place by the prefill form)
    int ldy;
    const void *ukv;         // [heads][dimP rows of W_uk | vP rows of W_uv], row stride uk_ld
    int uk_ld;
    const float *c_norm;     // [kv_rank]
    const float *sink;       // [heads] or nullptr
    const float *cosc, *sinc;  // [max_seq, rot_dim / 2], amplitude included
    void *cache;             // [slots, max_seq, rowP]
    int max_seq, nseq, T;
    const int *pos_dev, *slot_map;
    void *out;               // [M, ldo]: column h * vP
    int ldo;
    void *qabs;              // [M, heads, rowP] scratch
    float *part;             // split partials scratch
    size_t part_bytes;
    void *kv;                // expanded keys | values of a head group (prefill form)
    size_t kv_bytes;
    int host_pos;            // one sequence whose slot and position the host knows: position before this call; -1 otherwise
    int host_slot;
    int splits_ctx;          // context length the split count is chosen for
};
constexpr int kLatentExpandMin = 64;  // tokens of one sequence from which keys and values are expanded per head
int latent_attention_run(const Device *dev, const LatentArgs &a, cudaStream_t st, int *launches);
size_t latent_part_bytes(const Device *dev, const LatentShape &s, int tokens, int nseq);
bool latent_expands(const LatentShape &s);  // prompt chunks of this shape can take the expanded form
int latent_prepare(const Device *dev);

// ---- grouped-query attention -------------------------------------------------------------------------------------------
// q and k per head RMS-normed over dim (weights q_norm, k_norm) and rotated in their first rot_dims dimensions (neighbours
// paired); a position sees its own chunk (chunk = 0: everything) up to itself; softmax with a keyless sink logit per head; heads
// times sigmoid(gate).
struct GroupedShape {
    int heads, kv_heads, dim, vdim, rot_dims, chunk;
    float scale, eps;
    int dimP, vP;                    // per-head parts of the projected row and of a cache row, multiples of 8
    int q_off, k_off, v_off, g_off;  // places in a projected row; k_off < 0: the cache belongs to another layer, which has filled it
};
void grouped_layout(GroupedShape *s, bool own_kv);

struct GroupedArgs {
    GroupedShape s;
    int f32;
    void *y;                 // projected rows [M, ldy]; queries may be normed and rotated in place
    int ldy;
    const float *q_norm, *k_norm;  // [dim]
    const float *sink;       // [heads]
    const float *cosc, *sinc;  // [max_seq, rot_dims / 2]
    void *kcache, *vcache;   // [slots, kv_heads, max_seq, dimP], [slots, kv_heads, max_seq, vP]; padding is zero
    int max_seq, nseq, T;
    const int *pos_dev, *slot_map;
    void *out;               // [M, ldo]: column h * vP
    int ldo;
    float *part;             // split partials scratch
    size_t part_bytes;
    unsigned *counters;      // [grouped_counters()], zero between launches
    int host_pos, host_slot; // as in LatentArgs
    int splits_ctx;
};
int grouped_attention_run(const Device *dev, const GroupedArgs &a, cudaStream_t st, int *launches);
size_t grouped_part_bytes(const Device *dev, const GroupedShape &s, int f32, int tokens);
int grouped_counters(const GroupedShape &s, int tokens);
constexpr int kGroupedPrefillMin = 16;  // tokens of one sequence from which the prompt kernel runs (bf16)
bool grouped_prefills(const GroupedShape &s);  // ... for shapes it takes
int grouped_prepare(const Device *dev);

// ---- decayed linear attention ----------------------------------------------------------------------------------------
struct LinearShape {
    int heads, dim, vdim;
    int dimP, vP;
    int vS;              // row stride of a state [dim, vS], a multiple of 4
    int q_off, k_off, v_off, g_off;
    float eps;
    // gated form: a decay per token and key channel, sigmoid(a2 a1 + b)^(1 / tau); q scaled; norm over each head; SiLU gate
    int gated, rank;
    float inv_tau, q_scale;
};
struct LinearArgs {
    LinearShape s;
    int f32;
    const void *y;      // projected rows [M, ldy]: q | k | v (already activated) | gate
    int ldy;
    const float *norm;  // [heads * vP] (gated: [vP], shared by the heads), zeros in the padding
    const float *pows;  // [heads][kLinearPow + 1]: decay^0 .. decay^kLinearPow
    const float *a1;    // gated: f32 [M, rank8], rank8 = rank rounded up to 8
    const float *a2, *a2b;  // gated: [rank, heads * dim] (transposed), [heads * dim]
    float *decays;      // gated: [M, heads * dimP] f32 scratch of prompt chunks
    float *chunk_states;  // gated: [chunks of kGatedChunk tokens][heads][dim][vS] f32 scratch (optional)
    size_t chunk_bytes;
    float *state;       // [slots, heads, dim, vS]
    int nseq, T;
    const int *pos_dev, *slot_map;
    int keep_state;     // 1: leave the state as it was (a pass that is not counted)
    float *o;           // [M, heads * vP] f32 scratch
    float *seg_sums;    // [kLinearSegMax - 1][heads][dim][vS] f32 scratch of a long prompt's segments (optional)
    void *out;          // [M, ldo]
    int ldo;
};
constexpr int kLinearPow = 128;
constexpr int kLinearSegMax = 8;
constexpr int kGatedChunk = 64, kGatedChunkMin = 16;  // tokens of a chunk; shortest portion that runs in chunks (bf16)
int linear_attention_run(const Device *dev, const LinearArgs &a, cudaStream_t st, int *launches);
int linear_prepare(const Device *dev);
// linear_gated.cu, called by linear_attention_run: IM_ERR_BOUNDS when the shape or the scratch does not allow it
bool gated_decode_takes(const LinearShape &s);
bool gated_chunk_takes(const LinearShape &s);
int gated_decode_run(const LinearArgs &a, cudaStream_t st);
int gated_chunk_run(const LinearArgs &a, cudaStream_t st, int *launches);
int gated_prepare();

#ifdef __CUDACC__
template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// 16 bytes of elements <-> floats
template <typename T>
struct Vec16;
template <>
struct Vec16<float> {
    static constexpr int n = 4;
    static __device__ __forceinline__ void unpack(const uint4 &v, float *f) {
        f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
    }
    static __device__ __forceinline__ uint4 pack(const float *f) {
        return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
    }
};
template <>
struct Vec16<__nv_bfloat16> {
    static constexpr int n = 8;
    static __device__ __forceinline__ void unpack(const uint4 &v, float *f) {
        const unsigned w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    static __device__ __forceinline__ uint4 pack(const float *f) {
        unsigned w[4];
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const __nv_bfloat162 h = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
            w[i] = *reinterpret_cast<const unsigned *>(&h);
        }
        return make_uint4(w[0], w[1], w[2], w[3]);
    }
};

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return 0.5f * z * (1.0f + tanhf(u));
}
// Sum over the block; every thread gets it.  sh: 32 floats.
__device__ __forceinline__ float block_sum_f(float v, float *sh) {
    v = warp_sum(v);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (lane == 0) sh[warp] = v;
    __syncthreads();
    float t = 0.0f;
    for (int w = 0; w < nw; w++) t += sh[w];
    return t;
}

// bf16 tensor-core product of one 16 x 8 x 16 block and its operand loads
__device__ __forceinline__ void mma_bf16(float (&c)[4], unsigned a0, unsigned a1, unsigned a2, unsigned a3, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(unsigned (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(unsigned (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ unsigned pack_bf2(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned *>(&h);
}
// x = sum of bf16 terms: the rounded value and what the rounding left (two terms carry 16 bits, three all 24)
template <int TERMS>
__device__ __forceinline__ void split_bf2(float lo, float hi, unsigned (&out)[TERMS]) {
#pragma unroll
    for (int i = 0; i < TERMS; i++) {
        const unsigned p = pack_bf2(lo, hi);
        out[i] = p;
        lo -= __uint_as_float(p << 16);
        hi -= __uint_as_float(p & 0xffff0000u);
    }
}
__device__ __forceinline__ void cp_async16(void *dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
#endif

}  // namespace im
