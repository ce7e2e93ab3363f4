// Plain-C structures that cross the library boundary (decode engine descriptors, GEMM staging request).
// prometorch_b200/_native.py mirrors them with ctypes; keep the two in step.
#pragma once

#define PTB_MAX_PEERS 8

// One quantised matrix in the layout its kernel streams.
typedef struct PtbWeightDesc {
    const void* w;          // a GEMV streaming layout (see `layout`) or, for tables, row-major rows
    const void* bias;       // optional fp32 [rows]
    int qtype;              // 0 = Q4_K, 1 = Q6_K (structure of arrays), tables also: 2 = fp16, 3 = fp32
    int rows, cols;
    int rowbytes;           // > 0 only for row-major tables (the embedding)
    int layout;             // 0: [segment][row][segment bytes] (dp4a kernel); 1: tiles of 16 rows (tensor-pipe kernel)
    int pad;
} PtbWeightDesc;

typedef struct PtbLayerDesc {
    PtbWeightDesc q, k, v, o, gate, up, down;
    const float* attn_norm;
    const float* ffn_norm;
    const float* q_norm;
    const float* k_norm;
    const float* cos;       // per-layer RoPE tables [max_seq][head_dim / 2] (sliding-window layers may use another base)
    const float* sin;
    int window;             // sliding-window width, 0 = full attention
    int pad;
    const float* post_attn_norm;   // RMSNorm of the attention block's output before the residual add (or null)
    const float* post_ffn_norm;    // ... and of the FFN block's output
} PtbLayerDesc;

typedef struct PtbModelDesc {
    int n_layers, hidden, n_heads, n_kv_heads, head_dim, inter, vocab, max_seq;   // head counts are per rank
    float eps, emb_scale;
    int neox, act_gelu, norm_add_one, want_logits;
    PtbWeightDesc embed, lm_head;
    const float* out_norm;
    int tp_rank, tp_world, vocab_offset, pad;
    void* peer_inbox[3][PTB_MAX_PEERS];     // tensor parallelism: three receive buffers (attention out, FFN down, lm_head pair)
    int slot_elems, pad2;
} PtbModelDesc;

// Request to stage a row-sharded GEMM operand from the peers inside the launch.
typedef struct PtbStaging {
    void* peer[PTB_MAX_PEERS];   // peer r's full-size buffer as mapped on this GPU
    void* local;                 // this GPU's full-size buffer
    void* flags;                 // uint32 [ceil(stored_rows / 128)]: last sequence number staged per 128-row block
    int rank, world, shard_rows, stored_rows;
    long long row_bytes;
    unsigned seq;                // 0 disables staging
    int external;                // non-zero: someone else (copy engines on a side stream) copies the rows and raises the
                                 // flags; the launch adds no stager CTAs and only waits on the flags
} PtbStaging;

// One request of ptb_sample_logits_batch: a row of fp32 logits, the request's id history (the chosen id is appended at
// history[n_hist] when it fits), its scratch (ptb_sample_scratch_bytes, zeroed once) and where the result goes
// (out[0] = id, out[1] = float bits of its probability).  `u` is the uniform number of the draw.
typedef struct PtbSampleRequest {
    const float* logits;
    int* history;
    void* scratch;
    int* out;
    int n_hist, hist_cap, top_k, pad;
    float repeat_penalty, temperature, top_p, u;
} PtbSampleRequest;

// A recurrent layer over the rows of a batch (recurrence.cuh has the equations).
typedef struct PtbRecurrence {
    const void* x;          // [n] rows of pitch ld, bf16 or fp32: q [G D], k [G D], v [H Dv] at the three columns
    long long ld;
    int q_col, k_col, v_col;
    int silu;               // decay attention: q, k and v pass SiLU first
    int delta;              // 1: gated delta rule; 0: decay attention (G == H)
    int bf16;
    const void* beta;       // delta: [n][H] of pitch ld_beta in the type of x, before the sigmoid
    long long ld_beta;
    const float* a;         // delta: [n][H D] of pitch ld_a
    long long ld_a;
    const float* decay;     // [H]: the decay, or exp(A_log)
    const float* dt_bias;   // delta: [H D]
    float* state;           // [slots][H][D][Dv]
    int slots, n, H, G, D, Dv;
    const void* seqs;       // [n_seqs] int4 (first row, rows, position of the first, slot); null: one token per row
    int n_seqs, pos_stride, req_stride, pad;
    const int* pos;         // [n] of pos_stride
    const int* req;         // [n] of req_stride: slots
    float* out;             // [n][H Dv]
    int* status;
    const void* chunks;     // the matrix form: [n_chunks] int4 (first row, rows <= 64, sequence, 0), sequence by sequence
    const int* first_chunk; // [n_seqs]
    int n_chunks, rank;
    const void* low;        // the matrix form may take a as low low_w^T instead: [n][rank] of pitch ld_low, bf16
    long long ld_low;
    const void* low_w;      // [H D][rank], bf16
} PtbRecurrence;
