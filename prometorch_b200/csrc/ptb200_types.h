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
    int delta;              // 1: gated delta rule, decays per key channel; 2: one decay per head; 0: decay attention (G == H); 3: state-space step
    int bf16;
    const void* beta;       // delta: [n][H] of pitch ld_beta in the type of x, before the sigmoid
    long long ld_beta;
    const void* a;          // delta 1: fp32 [n][H D] of pitch ld_a; delta 2, 3: [n][H] of pitch ld_a in the type of x
    long long ld_a;
    const float* decay;     // [H]: the decay, or exp(A_log)
    const float* dt_bias;   // delta 1: [H D]; delta 2, 3: [H]
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
    const float* skip;      // delta 3: [H]
} PtbRecurrence;

// Softmax attention over the paged cache (window_attn.cuh has the meaning of the mask and of the two maps).
typedef struct PtbWindowAttn {
    const void* q;          // [n][H maps][Dp]
    void* out;              // [n][H Dv]
    const void* k_pages;    // [pages][G][64][maps Dp]
    const void* v_pages;    // [pages][G][64] rows of v_ld, of which Dvp are read (the latent cache: the same rows as the keys)
    const int* page_table;
    const int* pos;         // rows: [n] of pos_stride
    const int* req;         // rows: [n] of req_stride, rows of the page table
    const float* sink;      // [H] or null
    const void* gate;       // [n][H] of pitch gate_ld, in the type of q, or null
    long long gate_ld;
    float* work;            // rows: ptb_window_rows_work_floats(n, H maps, Dvp, nsplit) floats where nsplit or maps is above one
    int* status;
    const void* tiles;      // tiles: [n_tiles] int4 (first row, its position, rows <= 128, row of the page table or first row of the flat context)
    const float* rel;       // [H][rel_n]: added to a score by the key's distance, the last entry for all beyond; or null
    const void* k_rot;      // flat: the rotated key part that all heads share, rows of rot_ld
    long long k_ld, v_row, rot_ld;      // flat: pitches of the context's rows in k_pages ([rows][H][Dp]), v_pages ([rows][H][Dvp]) and k_rot
    int n, H, G, D, Dp, Dv, Dvp, v_ld, maps;
    int pos_stride, req_stride, pt_stride, n_pages;
    int window, keep, chunked;
    int max_keys, nsplit, bf16;
    int rel_n;
    int n_tiles, flat_rows, rot_dim;    // flat_rows > 0: keys and values lie flat, flat_rows of them; q is [n][H][Dq], see ptb_window_attn_tiles
    float scale, mix, mix_gain, mix_eps;
} PtbWindowAttn;

// What stands between two sublayers of a decoder with elementwise tanh norms: x += post(y); x += table[ids]; out = pre(x).
typedef struct PtbTanhResidual {
    float* x;               // [n][W]
    const void* y;          // bf16 (f32 = 0) or the sum of `splits` fp32 matrices `stride` apart; rows of pitch ld
    int f32, splits;
    long long stride, ld;
    const int* index;       // [n][top] rows of y, summed with `weight` [n][top]; null: row i is y's row i
    const float* weight;
    int top, y_rows;
    float post_alpha, pre_alpha;
    const float* post_w;
    const float* post_b;
    const float* pre_w;     // null: no out
    const float* pre_b;
    const int* ids;         // [n] of id_stride, or null
    int id_stride, V;
    const void* table;      // [V][W] in the type of out
    void* out;              // [n][W] bf16 or fp32
    int n, W, bf16, pad;
    int* status;
} PtbTanhResidual;

// Token, pair and position tables into the residual streams of every token.
typedef struct PtbPairEmbed {
    const int* ids;         // [n] of id_stride
    const int* pos;         // [n] of pos_stride
    const int* req;         // [n] of req_stride: slots
    int* last;              // [slots]: the id a sequence ended with; what it held counts for positions above zero
    const void* seqs;       // [n_seqs] int4 (first row, rows, position of the first, slot): a prompt pass; null: one token per row
    const void* table;      // [V][W]
    const void* pairs;      // [rows + 1][W]: row (id before * mul_before + id * mul_id) mod rows, the last one for a first token
    const void* at;         // [positions][W]
    float* x;               // [n][streams][W]
    int* status;
    long long mul_before, mul_id;
    int id_stride, pos_stride, req_stride, slots, n_seqs, n, V, rows, positions, W, streams, bf16;
} PtbPairEmbed;

// A matrix [n][W] in bf16 (f32 = 0), or the sum of `splits` fp32 matrices `stride` apart; rows of pitch ld.  y null: absent.
typedef struct PtbDense {
    const void* y;
    int f32, splits;
    long long stride, ld;
} PtbDense;

// Between two sublayers: with `mix`, stream t becomes sum_s mix[s][t] x_s + way_out[t] f sigmoid(gate + gate_bias), f the sum of y and of `top`
// weighed rows; then u = sum_s way_in[s] x_s (null: their sum), h = (u - mean) / sqrt(variance + eps) norm, and with `conv` conv_out = h + the
// causal convolution of h over the sequence's tokens, one token per sequence.
typedef struct PtbStreamStep {
    float* x;               // [n][streams][W]
    const float* mix;       // [streams][streams] from, to; null: the streams stay as they are
    const float* way_out;   // [streams]
    const float* way_in;    // [streams]
    PtbDense y, gate;
    const float* gate_bias; // [W]
    const int* index_of;    // [n][top] rows of `experts`, -1: the token's own row of `self`; null: none
    const float* weight;    // [n][top]
    const void* experts;    // [e_rows] of pitch e_ld, in the compute type
    const void* self;       // [n][W]
    long long e_ld;
    const float* norm;      // [W]; null: no h
    void* h;                // [m][W] bf16 or fp32
    const float* conv;      // [taps][W], the current token's tap last, or null
    void* conv_state;       // [slots][taps - 1][W] in the type of h
    void* conv_out;         // [m][W]
    const int* pos;
    const int* req;
    const long long* index; // [m] rows of x, or null (m = n)
    int* status;
    int top, e_rows, taps, slots, pos_stride, req_stride, n, m, W, streams, bf16;
    float eps;
} PtbStreamStep;
