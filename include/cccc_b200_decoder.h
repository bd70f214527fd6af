/*
 * C-ABI of the layer operations for decoders that keep their weights in BF16 (or float): the residual stream in
 * float, linears with fused epilogues, layer / RMS norm, attention over a KV cache with separate key and value sizes,
 * mixture-of-experts routing, greedy choice over float logits.  Library: libcccc-b200-decoder.so.
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

enum { B200_ACT_NONE = 0, B200_ACT_RELU2 = 1, B200_ACT_SILU_GATE = 2 };
enum { B200_NORM_RMS = 0, B200_NORM_LAYER = 1 };

/* X[i][:] = scale * table[ids[i]][:] into the float residual stream; an id outside [0, vocab) gives zeros. */
C_EXPORT int cuda_b200_embed_f32(int dtype, const void* ids, const void* table, unsigned int ld_table, void* X, unsigned int ldx,
    unsigned int n, unsigned int width, unsigned int vocab, float scale, void* stream, unsigned int flags);

/* Adds pending branch outputs to the float residual stream, then normalises:
 *   X[r][:] += sum_s slot_weight[r * slots + s] * Y[slot_row[r * slots + s]][:]      (slots == 0: nothing)
 *   out[i][:] = norm(X[rows ? rows[i] : i][:])                                       (out NULL: only the addition)
 * kind B200_NORM_LAYER: (x - mean) / sqrt(var + eps) * weight + bias; B200_NORM_RMS: x / sqrt(mean(x^2) + eps) *
 * weight (bias ignored).  weight and bias are float (NULL: 1 and 0).  All sums in float.  `rows` only without slots. */
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
    unsigned int n, width, ldx, ldo, ldy, slots;
    int kind;
    float eps;
} cuda_b200_norm;
C_EXPORT int cuda_b200_norm_rows(int dtype, const cuda_b200_norm* a, void* stream, unsigned int flags);

/* One linear of a launch:  Y[r][n] = epilogue(alpha * sum_k W[n][k] * X[xr][k]).
 * Dense (group_offset NULL): rows r = 0..rows-1, xr = r.  Grouped: group g owns the Y rows group_offset[g] ..
 * group_offset[g+1]-1 and the weight rows starting at g * group_rows; xr = x_row ? x_row[r] : r; `rows` is the most rows
 * all groups hold together, group_max the most rows one of them holds.
 * activation B200_ACT_SILU_GATE: feature n uses weight rows n (gate) and up_row + n, Y = silu(gate) * up.
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
    unsigned int rows, N, K, ldw, ldx, ldy;
    unsigned int groups, group_rows, group_max, up_row, active_cap;
    int out_type, activation, accumulate;
    float alpha;
} cuda_b200_linear;
/* Up to three independent members.  BF16: where no member has more than 32 rows (in one group), one launch of a weight-
 * streaming kernel runs all of them that hold about as many rows; else one tcgen05 launch per member (x_row not taken there).  kernel: 0 = by shape,
 * 1 = weight streaming, 2 = tcgen05 (tests and tuning). */
C_EXPORT int cuda_b200_linear_rows(int dtype, unsigned int count, const cuda_b200_linear* members, void* stream, unsigned int flags, int kernel);

/* A step's ragged batch: entry e brings n[e] tokens, rows start[e].. of the flat token arrays, which continue the
 * sequence in cache slot slot[e] at position pos[e].  token_entry[i] is the entry of token i.  Device int32 arrays. */
typedef struct cuda_b200_batch
{
    const void* slot;
    const void* pos;
    const void* start;
    const void* n;
    const void* token_entry;
    unsigned int entries, tokens, max_n;    /* max_n: the largest n[e]; launch bounds only */
    unsigned int max_len;                   /* no sequence is longer than this after the step; launch bounds only */
} cuda_b200_batch;

/* Attention of a layer from its projections on.  First, for every token of the batch: q heads to unit RMS in place
 * (qk_norm), k heads to unit RMS and v (mixed with v_first: v = (1 - mix) v + mix v_first) appended to the caches,
 * v_first stored.  Caches hold rows of k_ld / v_ld elements (multiples of 8) whose padding is zero.  A batch entry's
 * sequence must fit: pos + n <= T_max.  qkvg, the caches and work are 16-byte aligned. */
typedef struct cuda_b200_attention
{
    void* qkvg;                /* [tokens][ld] dtype: q at 0, k at k_off, v at v_off, output gate at g_off */
    void* out;                 /* [tokens][ldo] dtype: H * vdim */
    void* k_cache;             /* [slots][Hkv][T_max][k_ld] dtype */
    void* v_cache;             /* [slots][Hkv][T_max][v_ld] dtype */
    void* v_first;             /* [tokens][v_first_ld] dtype: written (v_mix 1) or read (v_mix 2) */
    void* work;                /* float scratch of cuda_b200_attention_work_bytes, zeroed once */
    unsigned int ld, ldo, k_off, v_off, g_off, v_first_ld;
    unsigned int H, Hkv, dim, vdim, k_ld, v_ld, T_max, slots;
    int v_mix;                 /* 0: plain, 1: this layer's values are the ones later layers mix in, 2: mix */
    int qk_norm, gate;         /* 1: unit RMS of q and k; multiply the output by sigmoid(gate) */
    float mix, eps, scale;
} cuda_b200_attention;
C_EXPORT unsigned long long cuda_b200_attention_work_bytes(unsigned int vdim);
/* Appends, then causal softmax attention over the caches (query head h reads kv head h / (H / Hkv)), then the output gate.
 * kernel: 0 = by shape, 1 = split-KV through shared memory (few query rows), 2 = tiled on mma.sync, 3 = the plain kernel
 * (always in float mode, and for key or value sizes above 256), 4 = split-KV straight into registers (sizes up to 128, k_ld
 * and v_ld multiples of 16, caches 32-byte aligned; with one token per entry the append is part of it), 5 = tiled on
 * tcgen05 (prompts; sizes up to 128, caches 16-byte aligned, `slots` given: the caches end after that many). */
C_EXPORT int cuda_b200_attention_rows(int dtype, const cuda_b200_attention* a, const cuda_b200_batch* b, void* stream, unsigned int flags,
    int kernel);

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
