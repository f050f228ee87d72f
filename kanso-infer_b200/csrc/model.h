// What every model of the library offers to its step functions and to the engine, and the
// registry that picks a model by its architecture name.
#pragma once
#include <string>

#include "json.h"
#include "kv_pool.h"

namespace kanso {

// One ragged step, host arrays. Sequence s brings query_lens[s] tokens, the last ones of its
// context_lens[s]; its cache pages are tables[s * max_blocks ...] and its recurrent state, where the
// model has one, lies in slot state_slots[s] (nullptr: slot s). `want` names rows of the step
// (0 .. T-1, ascending or not) whose logits are asked for.
struct StepBatch {
  uint32_t S = 0, T = 0, max_blocks = 0;
  const uint32_t* tokens = nullptr;
  const uint32_t* query_lens = nullptr;
  const uint32_t* context_lens = nullptr;
  const uint32_t* tables = nullptr;
  const uint32_t* state_slots = nullptr;
  const uint32_t* want = nullptr;
  uint32_t n_want = 0;
};

}  // namespace kanso

struct kanso_cuda_model {
  kanso_cuda_ctx* ctx = nullptr;
  // device copies of a step's host inputs, and its logits
  uint32_t* d_in = nullptr;
  size_t d_in_cap = 0;
  float* logits = nullptr;
  size_t logits_cap = 0;

  virtual ~kanso_cuda_model();
  virtual const char* architecture() const = 0;
  virtual uint32_t vocab_size() const = 0;
  virtual uint32_t num_layers() const = 0;
  virtual uint32_t block_size() const = 0;
  // Positions the model can take; 0: no limit.
  virtual uint32_t max_positions() const = 0;
  // Tokens of one sequence that a step can bring; 0: any number.
  virtual uint32_t max_query_len() const = 0;
  // The widest window of its layers: keys further back are never read. 0: no window.
  virtual uint32_t max_window() const { return 0; }
  // A sequence has a state besides its pages: it needs a slot of the pool.
  virtual bool has_state() const { return false; }
  // A pool of the geometry and element type its step reads, with that many state slots.
  virtual int32_t create_pool(uint32_t num_blocks, uint32_t num_slots, kanso_cuda_kv** out) = 0;
  virtual int32_t check_pool(const kanso_cuda_kv* kv) = 0;
  // One token per sequence, device arrays, asynchronous (kanso_cuda_decode_step_device).
  // state_slots nullptr: sequence s has slot s.
  virtual int32_t decode_device(kanso_cuda_kv* kv, const uint32_t* tokens,
                                const uint32_t* positions, const uint32_t* slots,
                                const uint32_t* tables, const uint32_t* context_lens,
                                const uint32_t* state_slots, uint32_t B, uint32_t max_blocks,
                                uint32_t max_ctx, int32_t act_mode, float* logits_dev) = 0;
  // A ragged step on checked host arrays; asynchronous, logits [n_want, vocab] on the device.
  virtual int32_t forward(kanso_cuda_kv* kv, const kanso::StepBatch& b, float* logits_dev) = 0;
};

namespace kanso {

// Grow-on-demand buffers of a model; growing waits for the stream.
int32_t model_inputs(kanso_cuda_model* m, size_t words);
int32_t model_logits(kanso_cuda_model* m, size_t rows);
// Host-side checks of a ragged step that need the pool and the model.
int32_t check_step(kanso_cuda_model* m, const kanso_cuda_kv* kv, const StepBatch& b);
// check_step + forward into the model's own logits buffer.
int32_t run_step(kanso_cuda_model* m, kanso_cuda_kv* kv, const StepBatch& b);

// A model class that loads from a folder with config.json and model.safetensors.
struct ModelClass {
  const char* architecture;
  // Checks the configuration; on success `summary` is one JSON object of its main figures.
  int32_t (*describe)(kanso_cuda_ctx* ctx, const Json& config, std::string* summary);
  int32_t (*load)(kanso_cuda_ctx* ctx, const Json& config, const std::string& dir, int32_t dtype,
                  kanso_cuda_model** out);
};
// Registration is static: a library holds the classes whose translation units are linked in.
struct ModelRegistrar {
  explicit ModelRegistrar(const ModelClass& c);
};

}  // namespace kanso
