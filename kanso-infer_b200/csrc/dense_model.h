// What the classes of unquantised (bfloat16 or f32) models share: reading config.json, putting
// the tensors of model.safetensors on the device, the workspace, and turning a step's host
// arrays into the row lists that the kernels take. A class adds its layers: parse, load and run.
#pragma once
#include <functional>
#include <memory>

#include "dense.cuh"
#include "model.h"
#include "safetensors.h"

namespace kanso {

// ---- config.json: a value at a dotted path below `j` ----
int32_t need_num(kanso_cuda_ctx* ctx, const Json& j, const char* path, double* out);
int32_t need_size(kanso_cuda_ctx* ctx, const Json& j, const char* path, uint32_t* out);
int32_t need_float(kanso_cuda_ctx* ctx, const Json& j, const char* path, float* out);

// Tokens of one sequence from which a portion goes to the prompt kernels.
constexpr uint32_t PROMPT_MIN_ROWS = 16;

// Rows of the step on the device and what the host knows of them.
struct DenseStep {
  int64_t T = 0, S = 0;
  const uint32_t* tokens = nullptr;
  RowMap map;
  const uint32_t* want = nullptr;  // nullptr: every row
  int64_t n_want = 0;
  const AttnTile *tiles128 = nullptr, *tiles64 = nullptr;  // the rows in tiles of that many
  uint32_t n_tiles128 = 0, n_tiles64 = 0;
  bool one_each = false;  // one row per sequence
  bool use_tiles = false;
  uint32_t max_keys = 0;
  // The sequences' portions, those shorter than PROMPT_MIN_ROWS first. nullptr: row t is all of
  // sequence t.
  const AttnTile* portions = nullptr;
  uint32_t n_short = 0, n_long = 0, max_short_rows = 1, max_long_rows = 0;
  const uint32_t* short_rows = nullptr;  // the rows of short portions (nullptr: every row)
  int64_t n_short_rows = 0;
  // Long portions in tiles of 128 rows whose last word is where the sequence's keys begin when
  // the keys of all long portions lie one after the other, and per long portion the run
  // {first of those places, keys, sequence, 0}.
  const AttnTile* long_tiles = nullptr;
  uint32_t n_long_tiles = 0;
  const AttnTile* key_runs = nullptr;
  int64_t long_keys = 0;
  const uint32_t* slots = nullptr;  // state slot per sequence; nullptr: sequence s has slot s
};

struct DenseModel : kanso_cuda_model {
  int32_t compute = KANSO_COMPUTE_BF16;
  std::vector<void*> owned;
  int64_t ws_rows = 0;  // rows that the workspace holds
  void* ws = nullptr;
  std::vector<uint32_t> step_in;  // host image of a step's inputs

  ~DenseModel() override {
    for (void* p : owned) cudaFree(p);
    if (ws) cudaFree(ws);
  }
  uint32_t block_size() const override { return 16; }
  uint32_t max_positions() const override { return 0; }
  uint32_t max_query_len() const override { return 0; }
  size_t elem() const { return compute == KANSO_COMPUTE_BF16 ? 2 : 4; }
  int32_t kv_type() const {
    return compute == KANSO_COMPUTE_BF16 ? KANSO_KV_BF16 : KANSO_KV_F32;
  }
  // What a layer keeps per token and per sequence.
  virtual std::vector<kanso_kv_layer> cache_layers() const = 0;
  int32_t create_pool(uint32_t num_blocks, uint32_t num_slots, kanso_cuda_kv** out) override;
  int32_t check_pool(const kanso_cuda_kv* kv) override;
  int32_t decode_device(kanso_cuda_kv* kv, const uint32_t* tokens, const uint32_t* positions,
                        const uint32_t* slots, const uint32_t* tables,
                        const uint32_t* context_lens, const uint32_t* state_slots, uint32_t B,
                        uint32_t max_blocks, uint32_t max_ctx, int32_t act_mode,
                        float* logits_dev) override;
  int32_t forward(kanso_cuda_kv* kv, const StepBatch& b, float* logits_dev) override;

 protected:
  virtual int32_t run(kanso_cuda_kv* kv, const DenseStep& s, float* logits_dev) = 0;

  int32_t tensor(const SafeTensors& st, const std::string& name, std::vector<int64_t> shape,
                 const StTensor** out);
  int32_t upload(const void* host, size_t bytes, void** out);
  int32_t vec(const SafeTensors& st, const std::string& name, int64_t n, float** out,
              std::vector<float>* host = nullptr);
  // Row r of the matrix is row source(r) of the parts one under the other (negative: zeros);
  // `groups` equal groups of rows, columns padded to 8.
  int32_t mat_rows(const std::vector<const StTensor*>& parts, int64_t rows, int64_t groups,
                   int64_t cols, bool f32, const std::function<int64_t(int64_t)>& source,
                   DenseMat* out);
  // The parts' rows one under the other.
  int32_t mat(const std::vector<const StTensor*>& parts, int64_t groups, int64_t cols, bool f32,
              DenseMat* out);
  // Transposed blocks: group g is the transpose of rows [g * block, (g + 1) * block) of `t`.
  int32_t mat_transposed(const StTensor* t, int64_t block, int64_t cols, bool f32, DenseMat* out);

  struct Room {
    void** p;
    size_t bytes;
  };
  // One allocation for the parts, cleared (pad columns are multiplied by zero: they must be
  // finite).
  int32_t make_ws(int64_t rows, const std::vector<Room>& parts);
  // logits = head . rmsnorm(x) * norm of the step's wanted rows; xe: T rows of the products' element
  // type to work in
  int32_t logits_of_rows(const DenseMat& head, const float* norm, float eps, const float* x, void* xe,
                         const DenseStep& s, float* logits_dev);
};

}  // namespace kanso
