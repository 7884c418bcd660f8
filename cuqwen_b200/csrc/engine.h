// The engine object behind the C ABI, shared by the translation units that implement it: engine.cu (create / load /
// step / prefill and the entry points) and stack.cu (designs described layer by layer by their config.json).
#pragma once
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <nccl.h>
#include <stdint.h>

#include <vector>

#include "../../include/cuqwen_b200.h"
#include "errors.h"
#include "launch.h"
#include "tp_plan.h"

namespace cq {

struct Stack;

struct Mat { uint8_t* w = nullptr; __half* s = nullptr; int rows = 0, cols = 0; };
struct Layer {
    __half *in_norm = nullptr, *post_norm = nullptr, *bq = nullptr, *bk = nullptr, *bv = nullptr;
    Mat q, k, v, o, gate, up, down;
};

}  // namespace cq

struct cuqwen_engine {
    cuqwen_params p{};
    int sms = 0;
    cudaStream_t stream = nullptr;
    cq::TpPlan plan{};
    int tp = 1, rank = 0;
    // local sizes
    int n_heads_l = 0, n_kv_l = 0, q_dim_l = 0, kv_dim_l = 0, inter_l = 0, vocab_l = 0, nsplit = 0;
    // weights
    uint8_t* warena = nullptr; size_t warena_bytes = 0;
    std::vector<cq::Layer> layers;
    __half *embed = nullptr, *norm = nullptr;
    cq::Mat lm; int lm_quant = 0; int lm_kind = 0;   // kind: 0 fp16 separate, 1 int8, 2 tied
    bool loaded = false;
    uint64_t weight_bytes = 0;                   // algorithmic bytes of all tensors a step reads (this rank)
    // state
    __half *x = nullptr, *xn = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *att = nullptr, *gate = nullptr, *logits = nullptr;
    __half *kc = nullptr, *vc = nullptr;                  // CUQWEN_FLAG_KV_INT8: int8 rows behind these pointers, scales below
    float *kscale = nullptr, *vscale = nullptr; bool kv8 = false;
    __half *spare_up = nullptr, *spare_out = nullptr;     // QwenState::up / mlp_out of the source-compatible layer (never read by the step)
    float *part_o = nullptr, *part_ml = nullptr; unsigned* counters = nullptr;
    cq::StepCtl* ctl = nullptr; cq::StepCtl* h_ctl = nullptr;
    cq::HostIo* hio = nullptr; cq::HostIo* hio_dev = nullptr; int io_seq = 0; bool ctl_dirty = true;   // mailbox of cuqwen_step (launch.h); ctl_dirty: the device block must be rewritten first
    int* d_hist = nullptr; unsigned* bitmap = nullptr; unsigned long long* best = nullptr; unsigned* ticket = nullptr;
    int* out_ring = nullptr; int ring_cap = 65536; int* h_out = nullptr;   // h_out holds ring_cap + 1 ints
    float* tp_partial = nullptr; unsigned long long* tp_keys = nullptr;
    // peer exchange (tensor parallel without collective calls): one receive block per rank, mapped into every peer
    unsigned char* tp_rx = nullptr; size_t tp_rx_bytes = 0; unsigned char* peer_rx[8] = {}; bool tp_peer = false;
    __half* x2 = nullptr; bool tp_sum_separate = false;
    unsigned char* gate_xd = nullptr; int* gate_corr = nullptr; float* gate_xscale = nullptr;    // SwiGLU output in staged form (see GemvArgs::xd_out)
    unsigned char* att_xd = nullptr; int* att_corr = nullptr; float* att_xscale = nullptr;       // attention output in staged form (see AttnArgs::xd_out)
    // batched prefill workspace (cuqwen_prefill), allocated at the first call for kPrefillChunk tokens
    __half *pf_x = nullptr, *pf_xn = nullptr, *pf_q = nullptr, *pf_att = nullptr, *pf_g = nullptr; float* pf_qkv = nullptr; int* pf_tok = nullptr;
    int steps_done = 0;                          // mirrors the device-side step counter (StepCtl::pad[1])
    std::vector<cudaEvent_t>* prof = nullptr;    // cuqwen_step_profile: an event is recorded after every launch of the step
    unsigned long long* step_trace = nullptr; size_t step_trace_bytes = 0;     // CUQWEN_FLAG_STEP_TRACE: eight timeline words per launch (tma.cuh)
    // graph
    cudaGraph_t graph = nullptr; cudaGraphExec_t gexec = nullptr; bool graph_ready = false;
    int launches = 0;
    cudaEvent_t ev0 = nullptr, ev1 = nullptr; float last_ms = 0.f;
    // a design read from a model directory (cuqwen_open): its layers, cache and kernels (stack.h); null for the models of the table
    cq::Stack* stack = nullptr;
    // nccl
    ncclComm_t comm = nullptr;
};
