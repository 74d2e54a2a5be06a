// What every model family shares: cache slots and positions, the prompt-chunk loop, captured decode steps, greedy
// decoding, logits on their way to the host.  A family (model.cu: quantized Llama / Qwen3 blocks; stack.cu: models given as
// a list of layers) derives from im_model, owns weights and caches, and runs one forward pass when asked to.
#pragma once
#include <map>
#include <string>
#include <utility>
#include <vector>

#include "common.cuh"

namespace im {

// Per-category GPU timing of one eager step (the counterpart of MetalConfig.kernel_timing /
// the profile-metal feature, crates/ironmill-inference/src/metal/pipeline.rs:353-422,1215-1234):
// an event is recorded after each group of launches and the interval is charged to its category.
enum ProfCat { kCatEmbed = 0, kCatQkv, kCatRope, kCatKvWrite, kCatAttn, kCatOProj, kCatResNorm, kCatFfn, kCatDown, kCatComm, kCatHead, kCatCount };
struct Prof {
    cudaStream_t st;
    std::vector<cudaEvent_t> ev;
    std::vector<int> cat;
    void mark(int c) {
        cudaEvent_t e;
        cudaEventCreate(&e);
        cudaEventRecord(e, st);
        ev.push_back(e);
        cat.push_back(c);
    }
};
#define IM_MARK(c) do { if (prof) prof->mark(c); } while (0)

#define IM_TRY(expr)                  \
    do {                              \
        int _rc = (expr);             \
        if (_rc != IM_OK) return _rc; \
    } while (0)

constexpr int kAllLogitsChunk = 256;  // prefill_all_logits holds a chunk's logits for every token
constexpr int kMaxSlots = 64;
constexpr int kArgmaxCtas = 64;

}  // namespace im

struct im_model {
    im::Device *dev = nullptr;
    im_model_config cfg{};  // a family fills the fields that apply to it
    cudaStream_t stream = nullptr;
    bool finalized = false;
    size_t bytes = 0;
    int MT = 0;  // most tokens of one forward pass
    uint32_t *tokens_dev = nullptr, *tok_hist = nullptr;
    int *pos_dev = nullptr, *step_dev = nullptr;
    uint32_t *tokens_pin = nullptr;
    float2 *argmax_cand = nullptr;  // [max_batch][kArgmaxCtas] candidates of the greedy pick
    unsigned *argmax_counters = nullptr;
    int *err_pin = nullptr;  // the device's bounded-wait error word, copied back with every step
    std::map<int, cudaGraphExec_t> graphs;
    int launches_per_step = 0;
    // Cache slots (continuous batching): every sequence owns one of max_batch slots = its rows of every layer's caches
    // and its position.  The single-sequence calls work on slot 0, the lockstep batch calls on slots 0 .. batch - 1.
    std::vector<int> slot_pos;      // host copy of the positions
    std::vector<char> slot_used;    // claimed by im_cuda_model_seq_add / _seq_open
    int *slot_ident = nullptr;      // device: 0, 1, 2, ... (a one-sequence forward into slot s passes slot_ident + s)
    int *slot_map = nullptr;        // device: slots of the sequences of the batch being decoded
    int *slot_pin = nullptr;
    // Logits of a step, [parts][rows][vocab / parts] on the device (fp16, or f32 when logits_f32); logits_rows: the same
    // for every token of a prompt chunk, allocated on first use.
    int logits_f32 = 0, logit_parts = 1;
    void *logits_dev = nullptr, *logits_pin = nullptr, *logits_rows = nullptr, *logits_rows_pin = nullptr;
    // set around a prompt chunk's forward pass: the slot and its positions before and after the chunk
    int prefill_slot_id = -1, prefill_ctx_begin = 0, prefill_ctx_end = 0;
    // a pass that is run but not counted (warm-up before a capture, profiling): recurrent states must stay as they are
    bool uncounted = false;
    std::vector<std::pair<void *, size_t>> allocs;

    virtual ~im_model() {}
    // One forward pass over nseq sequences x T tokens each (decode: T = 1; prefill: nseq = 1), tokens in tokens_dev.
    // Logits of the last token of every sequence go to logits_dev, or of every token to logits_rows.
    // slots: device array naming the cache slot of each sequence (nullptr: slots 0 .. nseq - 1).
    virtual int forward(int nseq, int T, cudaStream_t st, int *launches, im::Prof *prof, bool all_logits, const int *slots) = 0;
    virtual int finalize() = 0;
    virtual int prefill_chunk() const { return cfg.prefill_chunk_size; }
    virtual int alloc_logits_rows() = 0;
    virtual void clear_step_error() {}
    virtual bool recurrent() const { return false; }  // a state that cannot go back to an earlier position
    virtual int hidden_rows(int rows, float *out_host) = 0;
    virtual size_t step_bytes(int ctx, int batch) const = 0;
    virtual const char *family() const = 0;

    int alloc(void **p, size_t n) {
        const int rc = im::dev_malloc(dev, p, n);
        if (rc == IM_OK && n) {
            allocs.push_back({*p, n});
            bytes += n;
        }
        return rc;
    }
    size_t logit_size() const { return logits_f32 ? 4 : 2; }
};

namespace im {
int session_open(im_model *m);   // the stream; m->dev and m->cfg are set
int session_error_check(im_model *m);  // IM_ERR_TIMEOUT when the step just copied back reported a bounded wait that ran out
int session_alloc(im_model *m);  // tokens, positions, slots, pinned buffers; m->MT is set
}  // namespace im
