/*
 * C-ABI of the layer operations for decoders that keep their weights in BF16 (or float): the residual stream in
 * float, linears with fused epilogues, layer / RMS norm, attention over a KV cache with separate key and value sizes
 * (rotary positions, windows, sinks), latent attention, the mLSTM recurrence, mixture-of-experts routing, greedy choice
 * over float logits.  Library: libcccc-b200-decoder.so.
 *
 * `dtype` says how weights, activations and caches are held: 3 (BF16, float accumulation) or 0 (float, everything in
 * true float).  Pointers are device pointers; `stream` is a cudaStream_t; every call is asynchronous.  flags bit 0:
 * programmatic dependent launch.  Returns 0, 1 (CUDA error, reported on stderr) or -1 (an argument the call does not
 * take).  Row strides (ld*) are in elements.  Inputs of linears are 32-byte aligned with
 * row strides that are multiples of 64 elements, and columns from K up to the next multiple of 64 hold zeros in the
 * weights and finite values in the activations.
 */
#pragma once

#ifndef C_EXPORT
#define C_EXPORT extern "C" __attribute__((visibility("default")))
#endif

enum { B200_ACT_NONE = 0, B200_ACT_RELU2 = 1, B200_ACT_SILU_GATE = 2, B200_ACT_GELU_GATE = 3, B200_ACT_SOFTCAP = 4 };
enum { B200_NORM_RMS = 0, B200_NORM_LAYER = 1 };

/* X[i][:] = scale * table[ids[i]][:] into the float residual stream; an id outside [0, vocab) gives zeros. */
C_EXPORT int cuda_b200_embed_f32(int dtype, const void* ids, const void* table, unsigned int ld_table, void* X, unsigned int ldx,
    unsigned int n, unsigned int width, unsigned int vocab, float scale, void* stream, unsigned int flags);

/* Adds pending branch outputs to the float residual stream, then normalises:
 *   X[r][:] += sum_s slot_weight[r * slots + s] * Y[slot_row[r * slots + s]][:]      (slots == 0: nothing)
 *   X[r][:] += norm(branch[r][:])       (kind's norm without bias, branch_weight; branch NULL: nothing; not with slots)
 *   out[i][:] = norm(X[rows ? rows[i] : i][:])                                       (out NULL: only the addition)
 * kind B200_NORM_LAYER: (x - mean) / sqrt(var + eps) * weight + bias; B200_NORM_RMS: x / sqrt(mean(x^2) + eps) *
 * weight (bias ignored).  weight and bias are float (NULL: 1 and 0).  All sums in float.  `rows` only without slots or branch. */
typedef struct cuda_b200_norm
{
    void* X;
    const void* weight;
    const void* bias;
    void* out;
    const void* Y;             /* dtype */
    const void* slot_row;      /* int32 */
    const void* slot_weight;   /* float */
    const void* rows;          /* int32 */
    const void* branch;        /* float */
    const void* branch_weight; /* float */
    unsigned int n, width, ldx, ldo, ldy, slots, ldb;
    int kind;
    float eps;
} cuda_b200_norm;
C_EXPORT int cuda_b200_norm_rows(int dtype, const cuda_b200_norm* a, void* stream, unsigned int flags);

/* One linear of a launch:  Y[r][n] = epilogue(alpha * sum_k W[n][k] * X[xr][k]).
 * Dense (group_offset NULL): rows r = 0..rows-1, xr = r.  Grouped: group g owns the Y rows group_offset[g] ..
 * group_offset[g+1]-1 and the weight rows starting at g * group_rows; xr = x_row ? x_row[r] : r; `rows` is the most rows
 * all groups hold together, group_max the most rows one of them holds.
 * activation B200_ACT_SILU_GATE / _GELU_GATE: feature n uses weight rows n (gate) and up_row + n, Y = act(gate) * up (GELU
 * in its tanh form); B200_ACT_SOFTCAP: Y = cap * tanh(z / cap).
 * Block-diagonal (blocks > 1, not grouped): block b is a linear of its own, weight rows from b * group_rows, X columns from
 * b * x_step, Y columns from b * y_step (X's columns behind K up to the next multiple of 64 hold finite values; x_step a
 * multiple of 8).  head_gate: block b of row r is multiplied by sigmoid(head_gate[r * ld_gate + b]) (dtype).
 * tail > 0 (dense, not gated, not accumulated): the features from `tail` on go to Y_tail[r][n - tail], as floats.
 * out_type 0: float (accumulate != 0: Y += row_scale[r] * result), 3: BF16 (float mode: always 0).  row_scale: float per
 * row, or NULL. */
typedef struct cuda_b200_linear
{
    const void* W;
    const void* X;
    void* Y;
    const void* row_scale;
    const void* group_offset;   /* int32, groups + 1 */
    const void* x_row;          /* int32 */
    const void* active;         /* int32: ids of the non-empty groups, -1 behind them; `active_cap` entries (NULL: all groups) */
    const void* head_gate;
    void* Y_tail;
    unsigned int rows, N, K, ldw, ldx, ldy;
    unsigned int groups, group_rows, group_max, up_row, active_cap;
    unsigned int blocks, x_step, y_step, ld_gate;
    unsigned int tail, ld_tail;
    int out_type, activation, accumulate;
    float alpha, cap;
} cuda_b200_linear;
/* Up to three independent members.  BF16: where no member has more than 32 rows (in one group), one launch of a weight-
 * streaming kernel runs all of them that hold about as many rows; else one tcgen05 launch per member (x_row not taken there).  kernel: 0 = by shape,
 * 1 = weight streaming, 2 = tcgen05 (tests and tuning). */
C_EXPORT int cuda_b200_linear_rows(int dtype, unsigned int count, const cuda_b200_linear* members, void* stream, unsigned int flags, int kernel);

/* A step's ragged batch: entry e brings n[e] tokens, rows start[e].. of the flat token arrays, which continue the
 * sequence in cache slot slot[e] at position pos[e].  token_entry[i] is the entry of token i.  Device int32 arrays.  A call
 * runs the entries first_entry .. first_entry + entries - 1, whose tokens are first_token .. first_token + tokens - 1. */
typedef struct cuda_b200_batch
{
    const void* slot;
    const void* pos;
    const void* start;
    const void* n;
    const void* token_entry;
    const void* floor;                      /* nullable: attention does not let entry e see keys below floor[e] */
    unsigned int entries, tokens, max_n;    /* max_n: the largest n[e]; launch bounds only */
    unsigned int max_len;                   /* no sequence is longer than this after the step; launch bounds only */
    unsigned int first_entry, first_token;
} cuda_b200_batch;

/* cos and sin of p * base^(-2i / dims) for p < rows, i < dims / 2: table[p][i] = (cos, sin), floats, computed in double. */
C_EXPORT int cuda_b200_rotary_table(void* table, unsigned int rows, unsigned int dims, double base, void* stream);

/* Attention of a layer from its projections on.  First (append), for every token of the batch: q and k are normalised (qk_norm:
 * every head to unit RMS; q_norm / k_norm: the whole projection to unit RMS, times these weights) and rotated (rotary: the first
 * rot_dims elements of each head; element i goes with i + rot_dims / 2, or, interleaved, 2i with 2i + 1), q in place, k
 * appended to its cache; v (mixed with v_first: v = (1 - mix) v + mix v_first) appended as projected, v_first stored.  v_off
 * may be k_off: the values are the keys as projected.  Caches hold rows of k_ld / v_ld elements (multiples of 8) whose padding
 * is zero; k_cache and v_cache may be one (vdim <= dim) with append off.  A batch entry's sequence must fit: pos + n <= T_max.
 * qkvg, the caches and work are 16-byte aligned. */
typedef struct cuda_b200_attention
{
    void* qkvg;                /* [tokens][ld] dtype: q at 0 (a head every q_ld), k at k_off, v at v_off, output gate at g_off */
    void* out;                 /* [tokens][ldo] dtype: H * vdim */
    void* k_cache;             /* [slots][Hkv][T_max][k_ld] dtype */
    void* v_cache;             /* [slots][Hkv][T_max][v_ld] dtype */
    void* v_first;             /* [tokens][v_first_ld] dtype: written (v_mix 1) or read (v_mix 2) */
    void* work;                /* float scratch of cuda_b200_attention_work_bytes, zeroed once */
    const void* q_norm;        /* float [H * dim] */
    const void* k_norm;        /* float [Hkv * dim] */
    const void* rotary;        /* cuda_b200_rotary_table of T_max rows */
    const void* sink;          /* float [H]: a score that takes part in the softmax denominator only */
    const void* head_gate;     /* [tokens][ld_gate] dtype: head h's output is multiplied by sigmoid(head_gate[h]) */
    unsigned int ld, ldo, k_off, v_off, g_off, v_first_ld;
    unsigned int H, Hkv, dim, vdim, k_ld, v_ld, T_max, slots;
    unsigned int q_ld;         /* 0: dim.  Others only with append off */
    unsigned int rot_dims;     /* even */
    unsigned int ld_gate;
    unsigned int window;       /* a token sees itself and the window - 1 before it; 0: all */
    int v_mix;                 /* 0: plain, 1: this layer's values are the ones later layers mix in, 2: mix */
    int qk_norm, gate;         /* 1: unit RMS of q and k heads; multiply the output by sigmoid(gate) */
    int rot_interleaved;
    int no_append;             /* 1: the queries are ready and the caches hold the batch's keys and values */
    float mix, eps, scale;
} cuda_b200_attention;
C_EXPORT unsigned long long cuda_b200_attention_work_bytes(unsigned int vdim);
/* Appends, then causal softmax attention over the caches (query head h reads kv head h / (H / Hkv)), then the output gate.
 * kernel: 0 = by shape, 1 = split-KV through shared memory (few query rows), 2 = tiled on mma.sync, 3 = the plain kernel
 * (always in float mode, and for key or value sizes above 256), 4 = split-KV straight into registers (sizes up to 128, k_ld
 * and v_ld multiples of 16, caches 32-byte aligned; with one token per entry the append is part of it), 5 = tiled on
 * tcgen05 (prompts; sizes up to 256, caches 16-byte aligned, `slots` given: the caches end after that many), 6 = split
 * over latent rows (k_cache is v_cache, Hkv 1; dim up to 576, vdim up to 512). */
C_EXPORT int cuda_b200_attention_rows(int dtype, const cuda_b200_attention* a, const cuda_b200_batch* b, void* stream, unsigned int flags,
    int kernel);

/* Latent attention keeps per token one row [latent | rotated key part] for all heads.
 * _down: for every token of the batch, query latent cq = rms_norm(down[0 .. q_rank)) * q_norm, and the cache row
 * [rms_norm(down[kv_off .. + kv_rank)) * kv_norm | rotated down[kv_off + kv_rank .. + rot_dim)]; pairs are 2i and 2i + 1.
 * _query: dst[t][h * dst_step + dst_off ..] = rotated src[t][h * src_step + src_off .. + rot_dim).  src may be dst.
 * _expand (prompts): the cache rows that entry e's tokens may read, the last n + pos2 - floor of its first pos + n, go one behind
 * the other to rows floor[e] .. pos2[e] + n[e] - 1: the latents into c, the rotated part beside every head's key, K[h][row][dim
 * .. dim + rot_dim). */
typedef struct cuda_b200_latent
{
    const void* down;          /* [tokens][ld] dtype */
    void* cq;                  /* [tokens][ld_cq] dtype */
    void* cache;               /* [slots][T_max][c_ld] dtype */
    const void* q_norm;        /* float */
    const void* kv_norm;       /* float */
    const void* rotary;        /* cuda_b200_rotary_table of T_max rows */
    unsigned int ld, ld_cq, kv_off, q_rank, kv_rank, rot_dim, c_ld, T_max;
    float eps;
} cuda_b200_latent;
C_EXPORT int cuda_b200_latent_down(int dtype, const cuda_b200_latent* a, const cuda_b200_batch* b, void* stream, unsigned int flags);
C_EXPORT int cuda_b200_latent_query(int dtype, const void* src, unsigned int ld_src, unsigned int src_step, unsigned int src_off, void* dst,
    unsigned int ld_dst, unsigned int dst_step, unsigned int dst_off, unsigned int heads, unsigned int rot_dim, const void* rotary, unsigned int T_max,
    const cuda_b200_batch* b, void* stream, unsigned int flags);
typedef struct cuda_b200_expand
{
    const void* cache;         /* [slots][T_max][c_ld] dtype */
    void* c;                   /* [rows][ld_c] dtype */
    void* K;                   /* [heads][T][k_ld] dtype */
    const void* floor;         /* int32 per entry */
    const void* pos2;          /* int32 per entry */
    unsigned int c_ld, T_max, kv_rank, rot_dim, ld_c, k_ld, T, dim, heads;
    unsigned int max_rows;     /* the most rows an entry has; launch bounds only */
} cuda_b200_expand;
C_EXPORT int cuda_b200_latent_expand(int dtype, const cuda_b200_expand* a, const cuda_b200_batch* b, void* stream, unsigned int flags);

/* The mLSTM recurrence (xLSTM's matrix memory) of a layer from its projections on, per head, in float:
 *   i = cap tanh((gate_i + i_bias) / cap), f = log sigmoid(cap tanh((gate_f + f_bias) / cap)), m' = max(f + m, i),
 *   S' = e^(f + m - m') S + e^(i - m') k v^T, n' = e^(f + m - m') n + e^(i - m') k, o = S'^T q / (max(|n' q|, e^-m') + 1e-6),
 * q times q_scale, then o to unit RMS over the head, times `norm`, times sigmoid(output gate).  A sequence at position 0 starts
 * from zeros (also m), whatever its slot holds. */
typedef struct cuda_b200_mlstm
{
    const void* qkvg;          /* [tokens][ld] dtype: q at 0 (heads * dim), k at k_off, v at v_off (heads * vdim), gate at g_off */
    const void* gates;         /* float [tokens][ld_gates]: heads input gates, and from f_off on heads forget gates */
    const void* bias;          /* float [2 * heads]: input gates, forget gates */
    const void* norm;          /* float [heads * vdim] */
    void* out;                 /* [tokens][ldo] dtype: heads * vdim */
    void* state;               /* float [slots][heads][cuda_b200_mlstm_state_floats] */
    void* work;                /* float scratch of cuda_b200_mlstm_work_floats, 16-byte aligned */
    unsigned int ld, ld_gates, ldo, k_off, v_off, g_off, f_off;
    unsigned int heads, dim, vdim;
    float cap, eps, q_scale;
} cuda_b200_mlstm;
C_EXPORT unsigned long long cuda_b200_mlstm_state_floats(unsigned int dim, unsigned int vdim);
C_EXPORT unsigned long long cuda_b200_mlstm_work_floats(unsigned int tokens, unsigned int entries, unsigned int heads, unsigned int dim,
    unsigned int vdim);
/* kernel: 0 = by shape, 1 = token by token, any size, 2 = state in registers (BF16; up to 8 tokens per entry, dim up to 512,
 * vdim up to 1024), 3 = in chunks of 128 tokens on tcgen05 (BF16, prompts; dim up to 256 and a multiple of 16, vdim up to 1024 and a
 * multiple of 8; qkvg's offsets and strides multiples of 8). */
C_EXPORT int cuda_b200_mlstm_rows(int dtype, const cuda_b200_mlstm* a, const cuda_b200_batch* b, void* stream, unsigned int flags, int kernel);

/* Router: the `top` largest of each row of float logits [n][ldl] (ties: the lower expert), softmax over them; the
 * pairs (token, choice) are dealt to groups: pair_row[t * slots + s] = its row in group order, pair_weight, row_token[row]
 * = its token, group_offset[experts + 1], active (see cuda_b200_linear).  slots >= top.  sg_col >= 0: also
 * shared_weight[t] = sigmoid(logits[t][sg_col]).  counters: experts * 2 + 2 int32 of scratch. */
typedef struct cuda_b200_route
{
    const void* logits;
    void* pair_row;
    void* pair_weight;
    void* row_token;
    void* group_offset;
    void* active;
    void* shared_weight;
    void* choice;              /* int32 scratch, n * top */
    void* counters;
    unsigned int n, ldl, experts, top, active_cap;
    int sg_col;
} cuda_b200_route;
C_EXPORT int cuda_b200_route_rows(const cuda_b200_route* a, void* stream, unsigned int flags);

/* out[r][:] = X[row_token[r]][:], r < n. */
C_EXPORT int cuda_b200_gather_rows(int dtype, const void* X, unsigned int ldx, const void* row_token, void* out, unsigned int ldo, unsigned int n,
    unsigned int width, void* stream, unsigned int flags);

/* idx[r] = first maximum of a row of float logits (NaN never wins; only NaN: -1), val[r] its value. */
C_EXPORT int cuda_b200_argmax_f32(const void* logits, unsigned int rows, unsigned int cols, unsigned int ld, void* idx, void* val, void* stream,
    unsigned int flags);

/* Device sync and report; the status word of this library's bounded waits is included.  0 = clean. */
C_EXPORT int cuda_b200_decoder_check(const char* label);
/* Kernels launched by this library in the calling process. */
C_EXPORT unsigned long long cuda_b200_decoder_launches(void);
