// The layered decoder: a model assembled from layer descriptions (jgpt_layer_spec) instead of one fixed block.
// Internal interface used by the entry points of model.cu (forward step, generation) and sched.cu.
#pragma once

#include "common.cuh"

namespace jgpt {

struct Decoder;
Registry<Decoder> &decoder_registry();

// How the next token of a row is picked on the device.
struct SampleSpec {
    float temperature = 0.f;
    int top_k = 0;
};

// One step: entry i brings the tokens ids[starts[i], starts[i + 1]) of sequence seq_ids[i], which continue what the sequence
// already holds.  want: rows (indices into ids, ascending) whose logits are asked for; logits_host [n_want, vocab] and
// next_host [n_want] may be null.  u01: one draw per wanted row when spec.temperature > 0.
struct StepCall {
    int n = 0;
    const int *seq_ids = nullptr, *starts = nullptr, *ids = nullptr;
    int n_want = 0;
    const int *want = nullptr;
    float *logits_host = nullptr;
    int *next_host = nullptr;
    SampleSpec spec;
    const float *u01 = nullptr;
};
int32_t decoder_step(Decoder *d, Pool *p, jgpt_kvpool poolh, const StepCall &c);
int decoder_max_rows(const Decoder *d);
int decoder_max_positions(const Decoder *d);
const int *decoder_next_tokens_device(const Decoder *d);
Ctx *decoder_ctx(const Decoder *d);
int32_t decoder_destroy(Decoder *d);
int32_t decoder_check_pool(const Decoder *d, const Pool *p);

// The forms the fixed-block model offers, on top of decoder_step.
int32_t decoder_prefill_batch(Decoder *d, jgpt_kvpool poolh, const int *seq_ids, const int *starts, const int *ids, const int *rope_offsets,
                              int n, float *all_logits, float *last_logits, int *next);
int32_t decoder_decode(Decoder *d, jgpt_kvpool poolh, const int *seq_ids, const int *ids, const int *len_before, const int *rope_pos, int n,
                       float *logits, int *next, const SampleSpec &spec, const float *u01);
int32_t decoder_generate_greedy(Decoder *d, jgpt_kvpool poolh, const int *prompt, int S, int max_new, int *out, int *n_sampled);

// model.cu
int32_t launch_argmax(const float *logits, int rows, int vocab, int *next_dev, cudaStream_t st);
int32_t launch_sample(const float *logits, float *work, int rows, int vocab, const SampleSpec &spec, const float *u01_dev, int *next_dev,
                      cudaStream_t st);

// kvpool.cu: a pool whose layers have their own geometry and whose sequence slots carry recurrent state.
int32_t pool_create_layered(Ctx *c, const std::vector<KvLayerGeom> &layers, int elem_bytes, int n_blocks, int max_seqs, int max_blocks_per_seq,
                            uint64_t state_stride, jgpt_kvpool *out);

}  // namespace jgpt
