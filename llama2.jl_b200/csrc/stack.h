// Layer-stack models inside the library: what api.cu needs to build, run and free one.  The session's loop state, sampling,
// graphs and entry points are those of api.cu for every model; this part provides the weights, the cache and the kernels of a
// position (decode) or of many positions (prompts, batched decode).
#pragma once
#include <string>
#include <vector>

#include "host_common.h"
#include "stack_config.h"

struct StackModel;
struct StackSession;

// compute_f32: activations and cache in f32 and f32 arithmetic throughout; else bf16 operands, f32 accumulation, bf16 cache.
int32_t stack_model_create(const char* config_json, size_t n, bool compute_f32, StackModel** out);
const l2b::StackConfig& stack_model_config(const StackModel* m);
// Shape is the file's, `dtype` an l2b_ggml_type (bf16, or f32 for vectors); names the design does not have are refused.
int32_t stack_model_upload(StackModel* m, const char* name, int dtype, const void* host, const int64_t* shape, int ndim);
bool stack_model_has(const StackModel* m, const std::string& name);
int32_t stack_model_finalize(StackModel* m);
void stack_model_free(StackModel* m);
int64_t stack_model_bytes_per_token(const StackModel* m);

struct StackSessionInfo {
    int seq_len = 0;     // positions per sequence
    int n_seq = 1;       // sequences with a cache of their own (batched decode)
    int max_rows = 0;    // rows of a many-token pass
    bool decode = true;  // one-position passes are needed
};
int32_t stack_session_create(const StackModel* m, const StackSessionInfo& info, const DeviceInfo& di, cudaStream_t st, StackSession** out);
void stack_session_free(StackSession* s);
int32_t stack_session_reset(StackSession* s, cudaStream_t st);
int stack_session_max_rows(const StackSession* s);
const float* stack_session_residual(const StackSession* s);  // after the last layer of the most recent one-position pass

// One position (token and pos are device scalars): every kernel up to the logits and their per-block maxima (*nparts of them).
int32_t stack_enqueue_token(StackSession* s, const int* token, const int* pos, float* logits, float* amax_val, int* amax_idx, int* status, cudaStream_t st,
                            int* nlaunch, int* nparts);
// n rows through every layer: row r is token dev_tokens[r] at position pos0 + r of sequence 0, or at pos_list[r] of sequence r.
int32_t stack_enqueue_rows(StackSession* s, const int* dev_tokens, int n, int pos0, const int* pos_list, int* status, cudaStream_t st, long long* launches);
// Logits of some rows of the most recent stack_enqueue_rows (dev_index: row numbers, null: rows 0 .. n-1) -> logits [n][vocab].
int32_t stack_enqueue_logits(StackSession* s, const int* dev_index, int n, float* logits, int* status, cudaStream_t st, long long* launches);
