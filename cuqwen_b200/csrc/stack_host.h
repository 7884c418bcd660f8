// What engine.cu calls on a design read from a model directory (stack.cu).  Every function returns a CUQWEN_* code and
// leaves its message through report_error.
#pragma once
#include <functional>

#include "engine.h"
#include "model_dir.h"

namespace cq {

// Sizes, caches and recurrent states.  Fills e->p's model fields.
int stack_create(cuqwen_engine* e, const StackSpec& spec, int act, int max_seq_len);
int stack_load(cuqwen_engine* e, const char* dir);
void stack_destroy(cuqwen_engine* e);
const StackSpec& stack_spec(const Stack* s);
int stack_act(const Stack* s);
float* stack_logits(const Stack* s);              // [vocab] float32, the decode step's
size_t stack_cache_bytes(const Stack* s, void** ptr);
void stack_residual(const Stack* s, void** ptr, size_t* bytes);
// Algorithmic bytes of one decode step at context length ctx.
uint64_t stack_step_bytes(const Stack* s, int ctx);

// Around everything that runs tokens at positions pos0 .. pos - 1.  States of a recurrence cannot go back: a run begins at position 0 or
// where the last one ended; after a failed run only position 0 is left.
int stack_begin(Stack* s, int pos0);
void stack_end(Stack* s, int pos);
// The launches of one decode step from the embedding to the logits, for the token / position in e->ctl.  `after` is called
// after every launch (launch counting, profiling events).
int stack_record_step(cuqwen_engine* e, const LaunchCfg& cfg, const std::function<int()>& after);
// A portion of a sequence: T tokens (device ids at e->pf_tok) at cache positions pos0 ..; leaves their cache rows.  Logits of
// the rows want[0 .. n_want) (ascending row numbers of this portion) go to logits_host [n_want][vocab]; with none wanted the
// last layer stops after its cache rows.  At most stack_chunk() tokens.
int stack_chunk();
int stack_run_chunk(cuqwen_engine* e, int T, int pos0, const int* want, int n_want, float* logits_host);

}  // namespace cq
