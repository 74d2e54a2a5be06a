// The session half of the model-level engine (session.cuh): the CUDA counterpart of the family-independent part of
// MetalInference (crates/ironmill-inference/src/metal/engine.rs:122-270, pipeline.rs:228-1313).
// A decode step is captured once per batch size into a CUDA graph; the sequence positions live in device memory so that
// the graph replays unchanged as the sequences grow.
#include <string.h>

#include <algorithm>

#include "session.cuh"
#if defined(__x86_64__)
#include <immintrin.h>
#endif

namespace im {


__global__ void advance_pos_kernel(int *pos, const int *slot_map, int n, int by) {
    pdl_trigger();
    pdl_wait();
    if ((int)threadIdx.x < n) pos[slot_map ? slot_map[threadIdx.x] : threadIdx.x] += by;
}
__global__ void set_pos_kernel(int *pos, int n, int v) {
    if ((int)threadIdx.x < n) pos[threadIdx.x] = v;
}

// Greedy pick per sequence: LAST maximal index (Iterator::max_by keeps the last of equal maxima,
// crates/ironmill-inference/src/sampling.rs:331-339).  logits are laid out [parts][nseq][vocab_part].
// grid (kArgmaxCtas, nseq): every CTA scans a slice of the vocabulary and leaves its candidate in `cand`; the last
// CTA of a sequence to arrive combines the candidates, writes the token and clears the counter for the next launch.
constexpr int kArgmaxThreads = 256;
__device__ __forceinline__ bool argmax_better(float ov, int oi, float best, int bi) {  // is (ov, oi) preferred over (best, bi)?
    return oi >= 0 && (bi < 0 || ov > best || (ov == best && oi > bi));
}
__device__ __forceinline__ float logit_f(__half v) { return __half2float(v); }
__device__ __forceinline__ float logit_f(float v) { return v; }
template <typename L>
__global__ void __launch_bounds__(kArgmaxThreads) argmax_kernel(const L *__restrict__ logits, int vocab_part, int parts, int nseq,
                                                                uint32_t *__restrict__ tokens, uint32_t *__restrict__ hist,
                                                                const int *__restrict__ step, int hist_stride, int hist_rows,
                                                                float2 *__restrict__ cand, unsigned *__restrict__ counters) {
    __shared__ float sv[kArgmaxThreads / 32];
    __shared__ int si[kArgmaxThreads / 32];
    __shared__ int s_last;
    pdl_trigger();
    pdl_wait();
    const int seq = blockIdx.y;
    const int vocab = vocab_part * parts;
    const int per = (vocab + gridDim.x - 1) / gridDim.x, i0 = blockIdx.x * per, i1 = min(vocab, i0 + per);
    float best = -INFINITY;
    int bi = -1;
    for (int i = i0 + threadIdx.x; i < i1; i += blockDim.x) {
        const int part = i / vocab_part, j = i % vocab_part;
        const float v = logit_f(logits[((size_t)part * nseq + seq) * vocab_part + j]);
        if (!(v < best) || bi < 0) {  // ascending i per thread: ties move to the later index
            best = v;
            bi = i;
        }
    }
    auto block_reduce = [&]() {
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (argmax_better(ov, oi, best, bi)) {
                best = ov;
                bi = oi;
            }
        }
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
        if (lane == 0) {
            sv[warp] = best;
            si[warp] = bi;
        }
        __syncthreads();
        if (threadIdx.x == 0)
            for (int w = 1; w < (int)(blockDim.x >> 5); w++)
                if (argmax_better(sv[w], si[w], best, bi)) {
                    best = sv[w];
                    bi = si[w];
                }
    };
    block_reduce();
    if (threadIdx.x == 0) {
        cand[(size_t)seq * gridDim.x + blockIdx.x] = make_float2(best, __int_as_float(bi));
        __threadfence();
        s_last = atomicAdd(&counters[seq], 1u) == gridDim.x - 1;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    best = -INFINITY;
    bi = -1;
    if (threadIdx.x < gridDim.x) {
        const float2 c = __ldcg(&cand[(size_t)seq * gridDim.x + threadIdx.x]);
        best = c.x;
        bi = __float_as_int(c.y);
    }
    __syncthreads();
    block_reduce();
    if (threadIdx.x == 0) {
        tokens[seq] = (uint32_t)bi;
        if (hist) hist[(size_t)(*step % hist_rows) * hist_stride + seq] = (uint32_t)bi;
        counters[seq] = 0;
    }
}
__global__ void bump_kernel(int *step) {
    pdl_trigger();
    pdl_wait();
    *step += 1;
}

// mapped: the sequences of the batch live in the slots listed in m->slot_map (continuous batching); otherwise in slots 0 .. batch - 1.
static int get_graph(im_model *m, int batch, cudaGraphExec_t *out, bool mapped = false) {
    const int key = batch + (mapped ? 1000 : 0);
    const int *slots = mapped ? m->slot_map : nullptr;
    auto it = m->graphs.find(key);
    if (it != m->graphs.end()) {
        *out = it->second;
        return IM_OK;
    }
    cudaStream_t st = m->stream;
    // one eager pass first: sets function attributes and warms NCCL outside the capture
    m->uncounted = true;
    int rc = m->forward(batch, 1, st, nullptr, nullptr, false, slots);
    m->uncounted = false;
    IM_TRY(rc);
    IM_CUDA_CHECK(cudaStreamSynchronize(st));
    cudaGraph_t g = nullptr;
    IM_CUDA_CHECK(cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal));
    int nl = 0;
    rc = m->forward(batch, 1, st, &nl, nullptr, false, slots);
    if (rc == IM_OK) {
        const int vp = m->cfg.vocab_size / m->logit_parts;
        const dim3 grid(kArgmaxCtas, batch);
        cudaError_t le =
            m->logits_f32
                ? launch_k(argmax_kernel<float>, grid, dim3(kArgmaxThreads), 0, st, static_cast<const float *>(m->logits_dev), vp, m->logit_parts, batch, m->tokens_dev,
                           m->tok_hist, (const int *)m->step_dev, m->cfg.max_batch, m->cfg.max_seq_len, m->argmax_cand, m->argmax_counters)
                : launch_k(argmax_kernel<__half>, grid, dim3(kArgmaxThreads), 0, st, static_cast<const __half *>(m->logits_dev), vp, m->logit_parts, batch, m->tokens_dev,
                           m->tok_hist, (const int *)m->step_dev, m->cfg.max_batch, m->cfg.max_seq_len, m->argmax_cand, m->argmax_counters);
        if (le == cudaSuccess) le = launch_k(bump_kernel, dim3(1), dim3(1), 0, st, m->step_dev);
        if (le == cudaSuccess) le = launch_k(advance_pos_kernel, dim3(1), dim3(64), 0, st, m->pos_dev, slots, batch, 1);
        if (le != cudaSuccess) rc = fail(IM_ERR_CUDA, "launch failed: %s", cudaGetErrorString(le));
        nl += 3;
    }
    cudaError_t e = cudaStreamEndCapture(st, &g);
    if (rc != IM_OK) {
        if (g) cudaGraphDestroy(g);
        return rc;
    }
    if (e != cudaSuccess) return fail(IM_ERR_CUDA, "graph capture failed: %s", cudaGetErrorString(e));
    cudaGraphExec_t ge = nullptr;
    e = cudaGraphInstantiate(&ge, g, 0);
    cudaGraphDestroy(g);
    if (e != cudaSuccess) return fail(IM_ERR_CUDA, "graph instantiate failed: %s", cudaGetErrorString(e));
    m->graphs[key] = ge;
    m->launches_per_step = nl;
    *out = ge;
    return IM_OK;
}

// fp16 -> f32 on the host: 128 K logits per step.  With F16C (every x86-64-v3 CPU) eight at a time.
#if defined(__x86_64__)
__attribute__((target("avx,f16c"))) static void widen_f16c(const __half *src, float *dst, int n) {
    int j = 0;
    for (; j + 8 <= n; j += 8) _mm256_storeu_ps(dst + j, _mm256_cvtph_ps(_mm_loadu_si128(reinterpret_cast<const __m128i *>(src + j))));
    for (; j < n; j++) dst[j] = __half2float(src[j]);
}
#endif
static void widen(const __half *src, float *dst, int n) {
#if defined(__x86_64__)
    static const bool have = __builtin_cpu_supports("f16c") && __builtin_cpu_supports("avx");
    if (have) return widen_f16c(src, dst, n);
#endif
    for (int j = 0; j < n; j++) dst[j] = __half2float(src[j]);
}
// `rows` rows of pinned logits [parts][rows][vocab / parts] as f32 [rows][vocab]
static void logits_to_host(const im_model *m, const void *pin, int rows, float *out) {
    const int parts = m->logit_parts, V = m->cfg.vocab_size, vl = V / parts;
    for (int p = 0; p < parts; p++)
        for (int s = 0; s < rows; s++) {
            const size_t src = ((size_t)p * rows + s) * vl;
            float *dst = out + (size_t)s * V + (size_t)p * vl;
            if (m->logits_f32) memcpy(dst, static_cast<const float *>(pin) + src, (size_t)vl * 4);
            else widen(static_cast<const __half *>(pin) + src, dst, vl);
        }
}

// A kernel whose bounded wait ran out leaves a non-zero word; the step's results are then invalid.  Clears the
// word and the grid-barrier counters so that the next step starts clean.
int session_error_check(im_model *m) {
    if (*m->err_pin == 0) return IM_OK;
    const int code = *m->err_pin;
    *m->err_pin = 0;
    cudaMemset(m->dev->err_flag, 0, sizeof(int));
    cudaMemset(m->dev->sk_counters, 0, (size_t)kSkMaxBlocks * sizeof(int));
    m->clear_step_error();
    return fail(IM_ERR_TIMEOUT, "a device-side bounded wait ran out (code %d); the results of this step are invalid", code);
}

// Positions of every slot (reset, truncate of the single-sequence / lockstep interface).
static int set_positions(im_model *m, int pos) {
    set_pos_kernel<<<1, 64, 0, m->stream>>>(m->pos_dev, m->cfg.max_batch, pos);
    IM_CUDA_CHECK(cudaGetLastError());
    for (int &p : m->slot_pos) p = pos;
    return IM_OK;
}
__global__ void set_one_pos_kernel(int *pos, int slot, int v) { pos[slot] = v; }

// n tokens into cache slot `slot`, continuing at that slot's position.  last_logits (optional): f32 [vocab] of the last
// token; all_logits (optional): f32 [n, vocab]; want (optional, ascending places among the tokens): rows of wanted_logits.
static int prefill_slot(im_model *m, int slot, const uint32_t *tokens_host, int n, float *last_logits, float *all_logits, const int *want = nullptr,
                        int n_want = 0, float *wanted_logits = nullptr) {
    if (m->slot_pos[slot] + n > m->cfg.max_seq_len)
        return fail(IM_ERR_BOUNDS, "sequence position %d + %d tokens exceeds max_seq_len %d", m->slot_pos[slot], n, m->cfg.max_seq_len);
    cudaStream_t st = m->stream;
    const bool rows = all_logits || n_want > 0;
    int chunk = m->prefill_chunk();
    if (rows && chunk > kAllLogitsChunk) chunk = kAllLogitsChunk;
    const size_t V = (size_t)m->cfg.vocab_size, es = m->logit_size();
    const int *slots = slot == 0 ? nullptr : m->slot_ident + slot;
    if (rows && !m->logits_rows) {  // first use: a chunk's worth of logits on the device and in pinned host memory
        IM_TRY(m->alloc_logits_rows());
        IM_CUDA_CHECK(cudaMallocHost(&m->logits_rows_pin, (size_t)kAllLogitsChunk * V * es));
    }
    std::vector<float> tmp;
    int w = 0;
    for (int done = 0; done < n; done += chunk) {
        const int T = n - done < chunk ? n - done : chunk;
        const bool rows_here = all_logits || (w < n_want && want[w] < done + T);
        memcpy(m->tokens_pin, tokens_host + done, (size_t)T * 4);
        IM_CUDA_CHECK(cudaMemcpyAsync(m->tokens_dev, m->tokens_pin, (size_t)T * 4, cudaMemcpyHostToDevice, st));
        m->prefill_slot_id = slot;
        m->prefill_ctx_begin = m->slot_pos[slot];
        m->prefill_ctx_end = m->slot_pos[slot] + T;
        const int frc = m->forward(1, T, st, nullptr, nullptr, rows_here, slots);
        m->prefill_slot_id = -1;
        IM_TRY(frc);
        advance_pos_kernel<<<1, 64, 0, st>>>(m->pos_dev, slots, 1, T);
        IM_CUDA_CHECK(cudaGetLastError());
        if (rows_here) IM_CUDA_CHECK(cudaMemcpyAsync(m->logits_rows_pin, m->logits_rows, (size_t)T * V * es, cudaMemcpyDeviceToHost, st));
        IM_CUDA_CHECK(cudaMemcpyAsync(m->err_pin, m->dev->err_flag, sizeof(int), cudaMemcpyDeviceToHost, st));
        IM_CUDA_CHECK(cudaStreamSynchronize(st));  // tokens_pin is reused by the next chunk
        IM_TRY(session_error_check(m));
        m->slot_pos[slot] += T;
        if (all_logits) {
            logits_to_host(m, m->logits_rows_pin, T, all_logits + (size_t)done * V);
        } else if (rows_here) {
            tmp.resize((size_t)T * V);
            logits_to_host(m, m->logits_rows_pin, T, tmp.data());
            for (; w < n_want && want[w] < done + T; w++) memcpy(wanted_logits + (size_t)w * V, tmp.data() + (size_t)(want[w] - done) * V, V * 4);
        }
    }
    if (last_logits) {
        IM_CUDA_CHECK(cudaMemcpyAsync(m->logits_pin, m->logits_dev, V * es, cudaMemcpyDeviceToHost, st));
        IM_CUDA_CHECK(cudaStreamSynchronize(st));
        logits_to_host(m, m->logits_pin, 1, last_logits);
    }
    return IM_OK;
}

int session_open(im_model *m) {
    IM_CUDA_CHECK(cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking));
    return IM_OK;
}

int session_alloc(im_model *m) {
    const im_model_config &c = m->cfg;
    IM_TRY(m->alloc((void **)&m->tokens_dev, (size_t)m->MT * 4));
    IM_TRY(m->alloc((void **)&m->tok_hist, (size_t)c.max_seq_len * c.max_batch * 4));
    IM_TRY(m->alloc((void **)&m->pos_dev, kMaxSlots * 4));
    IM_TRY(m->alloc((void **)&m->slot_ident, kMaxSlots * 4));
    IM_TRY(m->alloc((void **)&m->slot_map, kMaxSlots * 4));
    int ident[kMaxSlots];
    for (int i = 0; i < kMaxSlots; i++) ident[i] = i;
    IM_CUDA_CHECK(cudaMemcpy(m->slot_ident, ident, sizeof(ident), cudaMemcpyHostToDevice));
    IM_CUDA_CHECK(cudaMemcpy(m->slot_map, ident, sizeof(ident), cudaMemcpyHostToDevice));
    IM_CUDA_CHECK(cudaMallocHost((void **)&m->slot_pin, kMaxSlots * sizeof(int)));
    m->slot_pos.assign((size_t)c.max_batch, 0);
    m->slot_used.assign((size_t)c.max_batch, 0);
    IM_TRY(m->alloc((void **)&m->step_dev, 4));
    IM_CUDA_CHECK(cudaMemset(m->pos_dev, 0, kMaxSlots * 4));
    IM_CUDA_CHECK(cudaMemset(m->step_dev, 0, 4));
    IM_TRY(m->alloc((void **)&m->argmax_cand, (size_t)c.max_batch * kArgmaxCtas * sizeof(float2)));
    IM_TRY(m->alloc((void **)&m->argmax_counters, (size_t)c.max_batch * sizeof(unsigned)));
    IM_CUDA_CHECK(cudaMemset(m->argmax_counters, 0, (size_t)c.max_batch * sizeof(unsigned)));
    IM_CUDA_CHECK(cudaMallocHost((void **)&m->tokens_pin, (size_t)m->MT * 4));
    IM_CUDA_CHECK(cudaMallocHost(&m->logits_pin, (size_t)c.max_batch * c.vocab_size * m->logit_size()));
    IM_CUDA_CHECK(cudaMallocHost((void **)&m->err_pin, sizeof(int)));
    *m->err_pin = 0;
    return IM_OK;
}


}  // namespace im

using namespace im;

IM_EXPORT void im_cuda_model_free(im_model *m) {
    if (!m) return;
    cudaSetDevice(m->dev->ordinal);
    if (m->stream) cudaStreamSynchronize(m->stream);
    for (auto &g : m->graphs) cudaGraphExecDestroy(g.second);
    for (auto &a : m->allocs) dev_free(m->dev, a.first, a.second);
    m->allocs.clear();
    if (m->tokens_pin) cudaFreeHost(m->tokens_pin);
    if (m->logits_pin) cudaFreeHost(m->logits_pin);
    if (m->logits_rows_pin) cudaFreeHost(m->logits_rows_pin);
    if (m->slot_pin) cudaFreeHost(m->slot_pin);
    if (m->err_pin) cudaFreeHost(m->err_pin);
    cudaStream_t st = m->stream;
    delete m;
    if (st) cudaStreamDestroy(st);
}

IM_EXPORT int im_cuda_model_finalize(im_model *m) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m, "bad argument");
    if (m->finalized) return IM_OK;
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    IM_TRY(m->finalize());
    m->finalized = true;
    return IM_OK;
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_reset(im_model *m) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    for (char &u : m->slot_used) u = 0;
    return set_positions(m, 0);
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_truncate(im_model *m, int pos) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    if (pos < 0 || pos > m->slot_pos[0]) return fail(IM_ERR_BOUNDS, "truncate_to(%d) is outside the current sequence of %d tokens", pos, m->slot_pos[0]);
    if (m->recurrent() && pos != 0 && pos != m->slot_pos[0])
        return fail(IM_ERR_STATE, "truncate_to(%d): this model carries a recurrent state, which can only be kept or started over", pos);
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    return set_positions(m, pos);
    IM_GUARD_END
}

// The final RMSNorm output the lm_head consumed in the last step (norm_out of
// crates/ironmill-inference/src/metal/pipeline.rs:176-226, decode_step_with_hidden / last_hidden_state) widened
// to f32: `rows` rows of hidden_size, one per sequence of that step in its order (row 0 for the single-sequence calls;
// after prefill_all_logits: one row per token of the last chunk).
IM_EXPORT int im_cuda_model_last_hidden_state(im_model *m, int rows, float *out_host) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && out_host, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    const int cap = m->MT;
    if (rows < 1 || rows > cap) return fail(IM_ERR_BOUNDS, "rows must be in 1..%d, got %d", cap, rows);
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    return m->hidden_rows(rows, out_host);
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_seq_pos(const im_model *m) { return m && !m->slot_pos.empty() ? m->slot_pos[0] : 0; }
IM_EXPORT int im_cuda_model_max_seq_len(const im_model *m) { return m ? m->cfg.max_seq_len : 0; }
IM_EXPORT size_t im_cuda_model_memory_bytes(const im_model *m) { return m ? m->bytes : 0; }
IM_EXPORT int im_cuda_model_step_launches(const im_model *m) { return m ? m->launches_per_step : 0; }
IM_EXPORT size_t im_cuda_model_step_bytes(const im_model *m, int ctx, int batch) { return m && m->finalized ? m->step_bytes(ctx, batch) : 0; }

IM_EXPORT int im_cuda_model_prefill(im_model *m, const uint32_t *tokens_host, int n, float *logits_out_host) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && tokens_host && logits_out_host, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_REQUIRE(n > 0, "prefill needs at least one token");
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    return prefill_slot(m, 0, tokens_host, n, logits_out_host, nullptr);
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_prefill_all_logits(im_model *m, const uint32_t *tokens_host, int n, float *logits_out_host) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && tokens_host && logits_out_host, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_REQUIRE(n > 0, "prefill needs at least one token");
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    return prefill_slot(m, 0, tokens_host, n, nullptr, logits_out_host);
    IM_GUARD_END
}

// ---- continuous batching: BatchInferenceEngine (crates/ironmill-inference/src/engine.rs:121-131) -------------------
// A free cache slot at position 0 (not claimed yet)
static int fresh_slot(im_model *m, int *out) {
    int slot = -1;
    for (int s = 0; s < m->cfg.max_batch && slot < 0; s++)
        if (!m->slot_used[s]) slot = s;
    if (slot < 0) return fail(IM_ERR_BOUNDS, "all %d sequence slots are in use (max_batch)", m->cfg.max_batch);
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    set_one_pos_kernel<<<1, 1, 0, m->stream>>>(m->pos_dev, slot, 0);
    IM_CUDA_CHECK(cudaGetLastError());
    m->slot_pos[slot] = 0;
    *out = slot;
    return IM_OK;
}

IM_EXPORT int im_cuda_model_seq_add(im_model *m, const uint32_t *tokens_host, int n, int *seq_id_out, float *logits_out_host) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && tokens_host && seq_id_out, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_REQUIRE(n > 0, "a sequence needs at least one prompt token");
    int slot = -1;
    IM_TRY(fresh_slot(m, &slot));
    int rc = prefill_slot(m, slot, tokens_host, n, logits_out_host, nullptr);
    if (rc != IM_OK) return rc;
    m->slot_used[slot] = 1;
    *seq_id_out = slot;
    return IM_OK;
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_seq_open(im_model *m, int *seq_id_out) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && seq_id_out, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_TRY(fresh_slot(m, seq_id_out));
    m->slot_used[*seq_id_out] = 1;
    return IM_OK;
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_seq_extend(im_model *m, int seq_id, const uint32_t *tokens_host, int n, const int *want_host, int n_want, float *logits_out_host) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && tokens_host && n > 0 && n_want >= 0 && (n_want == 0 || (want_host && logits_out_host)), "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    if (seq_id < 0 || seq_id >= m->cfg.max_batch || !m->slot_used[seq_id]) return fail(IM_ERR_INVALID, "no sequence %d", seq_id);
    for (int i = 0; i < n_want; i++)
        IM_REQUIRE(want_host[i] >= (i ? want_host[i - 1] + 1 : 0) && want_host[i] < n, "wanted places must ascend within 0..%d", n - 1);
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    return prefill_slot(m, seq_id, tokens_host, n, nullptr, nullptr, want_host, n_want, logits_out_host);
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_seq_remove(im_model *m, int seq_id) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    if (seq_id < 0 || seq_id >= m->cfg.max_batch || !m->slot_used[seq_id]) return fail(IM_ERR_INVALID, "no sequence %d", seq_id);
    m->slot_used[seq_id] = 0;   // the slot's cache rows are simply overwritten by the next tenant
    m->slot_pos[seq_id] = 0;
    return IM_OK;
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_seq_position(const im_model *m, int seq_id) {
    if (!m || seq_id < 0 || seq_id >= (int)m->slot_pos.size() || !m->slot_used[seq_id]) return -1;
    return m->slot_pos[seq_id];
}

// One decode step for the listed sequences (any subset of the live ones, each at its own position): tokens_host[i] is
// appended to sequence seq_ids[i]; logits_out_host f32 [n, vocab] in the same order.
IM_EXPORT int im_cuda_model_batch_decode_step(im_model *m, const int *seq_ids, const uint32_t *tokens_host, int n, float *logits_out_host) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && seq_ids && tokens_host && logits_out_host, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_REQUIRE(n >= 1 && n <= m->cfg.max_batch, "batch %d outside 1..max_batch (%d)", n, m->cfg.max_batch);
    for (int i = 0; i < n; i++) {
        const int s = seq_ids[i];
        if (s < 0 || s >= m->cfg.max_batch || !m->slot_used[s]) return fail(IM_ERR_INVALID, "no sequence %d", s);
        for (int j = 0; j < i; j++)
            if (seq_ids[j] == s) return fail(IM_ERR_INVALID, "sequence %d listed twice", s);
        if (m->slot_pos[s] + 1 > m->cfg.max_seq_len)
            return fail(IM_ERR_BOUNDS, "sequence %d: position %d + 1 exceeds max_seq_len %d", s, m->slot_pos[s], m->cfg.max_seq_len);
    }
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    cudaStream_t st = m->stream;
    memcpy(m->slot_pin, seq_ids, (size_t)n * sizeof(int));
    IM_CUDA_CHECK(cudaMemcpyAsync(m->slot_map, m->slot_pin, (size_t)n * sizeof(int), cudaMemcpyHostToDevice, st));
    cudaGraphExec_t g = nullptr;
    IM_TRY(get_graph(m, n, &g, true));
    memcpy(m->tokens_pin, tokens_host, (size_t)n * 4);
    IM_CUDA_CHECK(cudaMemcpyAsync(m->tokens_dev, m->tokens_pin, (size_t)n * 4, cudaMemcpyHostToDevice, st));
    IM_CUDA_CHECK(cudaGraphLaunch(g, st));
        IM_CUDA_CHECK(cudaMemcpyAsync(m->logits_pin, m->logits_dev, (size_t)n * m->cfg.vocab_size * m->logit_size(), cudaMemcpyDeviceToHost, st));
    IM_CUDA_CHECK(cudaMemcpyAsync(m->err_pin, m->dev->err_flag, sizeof(int), cudaMemcpyDeviceToHost, st));
    IM_CUDA_CHECK(cudaStreamSynchronize(st));
    IM_TRY(session_error_check(m));
    for (int i = 0; i < n; i++) m->slot_pos[seq_ids[i]] += 1;
    logits_to_host(m, m->logits_pin, n, logits_out_host);
    return IM_OK;
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_decode_step(im_model *m, const uint32_t *tokens_host, int batch, float *logits_out_host) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && tokens_host && logits_out_host, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_REQUIRE(batch >= 1 && batch <= m->cfg.max_batch, "batch %d outside 1..max_batch (%d)", batch, m->cfg.max_batch);
    int far = 0;
    for (int b = 0; b < batch; b++) far = m->slot_pos[b] > far ? m->slot_pos[b] : far;
    if (far + 1 > m->cfg.max_seq_len)
        return fail(IM_ERR_BOUNDS, "sequence position %d + 1 exceeds max_seq_len %d", far, m->cfg.max_seq_len);
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    cudaStream_t st = m->stream;
    cudaGraphExec_t g = nullptr;
    IM_TRY(get_graph(m, batch, &g));
    memcpy(m->tokens_pin, tokens_host, (size_t)batch * 4);
    IM_CUDA_CHECK(cudaMemcpyAsync(m->tokens_dev, m->tokens_pin, (size_t)batch * 4, cudaMemcpyHostToDevice, st));
    IM_CUDA_CHECK(cudaGraphLaunch(g, st));
        IM_CUDA_CHECK(cudaMemcpyAsync(m->logits_pin, m->logits_dev, (size_t)batch * m->cfg.vocab_size * m->logit_size(), cudaMemcpyDeviceToHost, st));
    IM_CUDA_CHECK(cudaMemcpyAsync(m->err_pin, m->dev->err_flag, sizeof(int), cudaMemcpyDeviceToHost, st));
    IM_CUDA_CHECK(cudaStreamSynchronize(st));
    IM_TRY(session_error_check(m));
    for (int b = 0; b < batch; b++) m->slot_pos[b] += 1;
    logits_to_host(m, m->logits_pin, batch, logits_out_host);
    return IM_OK;
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_decode_greedy(im_model *m, const uint32_t *first_tokens_host, int batch, int n_steps,
                                          uint32_t *tokens_out_host, float *elapsed_ms_out) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && first_tokens_host, "bad argument");
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_REQUIRE(batch >= 1 && batch <= m->cfg.max_batch, "batch %d outside 1..max_batch (%d)", batch, m->cfg.max_batch);
    IM_REQUIRE(n_steps >= 0, "n_steps must be >= 0");
    int far = 0;
    for (int b = 0; b < batch; b++) far = m->slot_pos[b] > far ? m->slot_pos[b] : far;
    if (far + n_steps > m->cfg.max_seq_len)
        return fail(IM_ERR_BOUNDS, "sequence position %d + %d steps exceeds max_seq_len %d", far, n_steps, m->cfg.max_seq_len);
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    cudaStream_t st = m->stream;
    cudaGraphExec_t g = nullptr;
    IM_TRY(get_graph(m, batch, &g));
    memcpy(m->tokens_pin, first_tokens_host, (size_t)batch * 4);
    IM_CUDA_CHECK(cudaMemcpyAsync(m->tokens_dev, m->tokens_pin, (size_t)batch * 4, cudaMemcpyHostToDevice, st));
    IM_CUDA_CHECK(cudaMemsetAsync(m->step_dev, 0, 4, st));
    cudaEvent_t e0, e1;
    IM_CUDA_CHECK(cudaEventCreate(&e0));
    IM_CUDA_CHECK(cudaEventCreate(&e1));
    cudaEventRecord(e0, st);
    for (int i = 0; i < n_steps; i++) {
        cudaError_t e = cudaGraphLaunch(g, st);
        if (e != cudaSuccess) {
            cudaEventDestroy(e0);
            cudaEventDestroy(e1);
            return fail(IM_ERR_CUDA, "graph launch failed: %s", cudaGetErrorString(e));
        }
    }
    cudaEventRecord(e1, st);
    cudaMemcpyAsync(m->err_pin, m->dev->err_flag, sizeof(int), cudaMemcpyDeviceToHost, st);
    cudaError_t e = cudaStreamSynchronize(st);
    float ms = 0.0f;
    cudaEventElapsedTime(&ms, e0, e1);
    cudaEventDestroy(e0);
    cudaEventDestroy(e1);
    if (e != cudaSuccess) return fail(IM_ERR_CUDA, "decode loop failed: %s", cudaGetErrorString(e));
    IM_TRY(session_error_check(m));
    for (int b = 0; b < batch; b++) m->slot_pos[b] += n_steps;
    if (elapsed_ms_out) *elapsed_ms_out = ms;
    if (tokens_out_host && n_steps > 0)
        IM_CUDA_CHECK(cudaMemcpy2D(tokens_out_host, (size_t)batch * 4, m->tok_hist, (size_t)m->cfg.max_batch * 4, (size_t)batch * 4, n_steps,
                                   cudaMemcpyDeviceToHost));
    return IM_OK;
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_profile_step(im_model *m, int batch, float *ms_by_category, int n_categories) {
    IM_GUARD_BEGIN
    IM_REQUIRE(m && ms_by_category && n_categories >= kCatCount, "bad argument (need %d categories)", (int)kCatCount);
    if (!m->finalized) return fail(IM_ERR_STATE, "model not loaded");
    IM_REQUIRE(batch >= 1 && batch <= m->cfg.max_batch, "batch %d outside 1..max_batch (%d)", batch, m->cfg.max_batch);
    for (int b = 0; b < batch; b++)
        if (m->slot_pos[b] + 1 > m->cfg.max_seq_len) return fail(IM_ERR_BOUNDS, "no room for one more position");
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    cudaStream_t st = m->stream;
    m->uncounted = true;
    int rc = m->forward(batch, 1, st, nullptr, nullptr, false, nullptr);  // warm
    Prof prof;
    prof.st = st;
    prof.mark(-1);
    if (rc == IM_OK) rc = m->forward(batch, 1, st, nullptr, &prof, false, nullptr);
    m->uncounted = false;
    cudaError_t e = cudaStreamSynchronize(st);
    for (int i = 0; i < n_categories; i++) ms_by_category[i] = 0.0f;
    if (rc == IM_OK && e == cudaSuccess)
        for (size_t i = 1; i < prof.ev.size(); i++) {
            float ms = 0.0f;
            cudaEventElapsedTime(&ms, prof.ev[i - 1], prof.ev[i]);
            ms_by_category[prof.cat[i]] += ms;
        }
    for (cudaEvent_t ev : prof.ev) cudaEventDestroy(ev);
    if (rc != IM_OK) return rc;
    if (e != cudaSuccess) return fail(IM_ERR_CUDA, "profile step failed: %s", cudaGetErrorString(e));
    return IM_OK;
    IM_GUARD_END
}
