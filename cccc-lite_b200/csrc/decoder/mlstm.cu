// The mLSTM recurrence token by token, any size and both number formats, and its entry point.
#include "mlstm.cuh"

namespace b200
{

constexpr unsigned int MP_COLS = 32, MP_ROWS = 8;    // 32 value columns x 8 groups of key rows

// grid (column blocks, heads, entries).  The CTA's columns of S stay in shared memory for the whole entry.  Outputs go to
// work as floats, the new n and m behind them: other column blocks may still have to read the old ones.
template <class T>
__global__ void __launch_bounds__(MP_COLS* MP_ROWS) mlstm_plain_kernel(const MlstmParams p)
{
    extern __shared__ float mp_smem[];
    __shared__ float red[MP_ROWS][MP_COLS + 1], red_n[MP_ROWS];
    float* S = mp_smem;                        // [dim][33]
    float* nn = S + p.dim * (MP_COLS + 1);     // [dim]
    float* q = nn + p.dim;                     // [dim]
    float* k = q + p.dim;                      // [dim]
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int c0 = blockIdx.x * MP_COLS, h = blockIdx.y, e = p.e0 + blockIdx.z, tid = threadIdx.x, col = tid % MP_COLS, rg = tid / MP_COLS;
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e];
    const bool fresh = p.pos[e] == 0, live = c0 + col < p.vdim;
    float* st = mlstm_state_of(p, e, h);
    const unsigned int v_ld = mlstm_v_ld(p.vdim);
    float* st_n = st + (size_t)p.dim * v_ld;
    for (unsigned int d = rg; d < p.dim; d += MP_ROWS) { S[d * (MP_COLS + 1) + col] = fresh || !live ? 0.f : st[(size_t)d * v_ld + c0 + col]; }
    for (unsigned int d = tid; d < p.dim; d += MP_COLS * MP_ROWS) { nn[d] = fresh ? 0.f : st_n[d]; }
    float m = fresh ? 0.f : st_n[mlstm_n_ld(p.dim)];
    const size_t o_ld = (size_t)p.heads * p.vdim;
    for (unsigned int t = 0; t < n; t++)
    {
        const unsigned int i = start + t;
        const T* x = (const T*)p.qkvg + (size_t)i * p.ld;
        __syncthreads();
        for (unsigned int d = tid; d < p.dim; d += MP_COLS * MP_ROWS)
        {
            q[d] = Elem<T>::get(x[h * p.dim + d]) * p.q_scale;
            k[d] = Elem<T>::get(x[p.k_off + h * p.dim + d]);
        }
        const float v = live ? Elem<T>::get(x[p.v_off + h * p.vdim + c0 + col]) : 0.f;
        float in, forget;
        mlstm_gates(p, i, h, in, forget);
        const float m1 = fmaxf(forget + m, in), keep = expf(forget + m - m1), add = expf(in - m1);
        m = m1;
        __syncthreads();
        float o = 0.f, nq = 0.f;
        for (unsigned int d = rg; d < p.dim; d += MP_ROWS)
        {
            float& s = S[d * (MP_COLS + 1) + col];
            s = keep * s + add * k[d] * v;
            o = fmaf(s, q[d], o);
            if (col == 0)
            {
                nn[d] = keep * nn[d] + add * k[d];
                nq = fmaf(nn[d], q[d], nq);
            }
        }
        red[rg][col] = o;
        if (col == 0) { red_n[rg] = nq; }
        __syncthreads();
        if (rg == 0 && live)
        {
            o = nq = 0.f;
#pragma unroll
            for (unsigned int r = 0; r < MP_ROWS; r++)
            {
                o += red[r][col];
                nq += red_n[r];
            }
            p.work[(size_t)(i - p.t0) * o_ld + h * p.vdim + c0 + col] = o / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
        }
    }
    __syncthreads();
    if (live)
    {
        for (unsigned int d = rg; d < p.dim; d += MP_ROWS) { st[(size_t)d * v_ld + c0 + col] = S[d * (MP_COLS + 1) + col]; }
    }
    if (blockIdx.x == 0)
    {
        float* w = p.work + p.tokens * o_ld + ((size_t)blockIdx.z * p.heads + h) * (p.dim + 1);
        for (unsigned int d = tid; d < p.dim; d += MP_COLS * MP_ROWS) { w[d] = nn[d]; }
        if (tid == 0) { w[p.dim] = m; }
    }
}

// A warp per (token, head): unit RMS of the output, norm weights, output gate; the last token's warp stores n and m.
template <class T>
__global__ void __launch_bounds__(128) mlstm_finish_kernel(const MlstmParams p)
{
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int i = p.t0 + blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (h >= p.heads) { return; }
    const size_t o_ld = (size_t)p.heads * p.vdim;
    const float* o = p.work + (size_t)blockIdx.x * o_ld + (size_t)h * p.vdim;
    const T* gate = (const T*)p.qkvg + (size_t)i * p.ld + p.g_off + h * p.vdim;
    float sq = 0.f;
    for (unsigned int c = lane; c < p.vdim; c += 32) { sq += o[c] * o[c]; }
    const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)p.vdim + p.eps);
    T* out = (T*)p.out + (size_t)i * p.ldo + (size_t)h * p.vdim;
    for (unsigned int c = lane; c < p.vdim; c += 32) { out[c] = Elem<T>::put(o[c] * inv * p.norm[h * p.vdim + c] * sigmoid_f32(Elem<T>::get(gate[c]))); }
    const unsigned int e = (unsigned int)p.token_entry[i];
    if ((int)i == p.start[e] + p.n[e] - 1)
    {
        const float* w = p.work + p.tokens * o_ld + ((size_t)(e - p.e0) * p.heads + h) * (p.dim + 1);
        float* st_n = mlstm_state_of(p, e, h) + (size_t)p.dim * mlstm_v_ld(p.vdim);
        for (unsigned int d = lane; d < p.dim; d += 32) { st_n[d] = w[d]; }
        if (lane == 0) { st_n[mlstm_n_ld(p.dim)] = w[p.dim]; }
    }
}

template <class T>
static int mlstm_plain(const MlstmParams& p, unsigned int entries, void* stream, bool pdl)
{
    const DecoderDevice* dev = decoder_device();
    const size_t smem = (size_t)p.dim * (MP_COLS + 4) * 4;
    if (!dev || smem > (size_t)dev->max_smem - 2048) { return -1; }
    const int rc = launch_kernel("mlstm_plain", mlstm_plain_kernel<T>, dim3((p.vdim + MP_COLS - 1) / MP_COLS, p.heads, entries), dim3(MP_COLS * MP_ROWS), smem, stream,
        pdl, p);
    return rc ? rc : launch_kernel("mlstm_finish", mlstm_finish_kernel<T>, dim3(p.tokens, (p.heads + 3) / 4), dim3(128), 0, stream, pdl, p);
}

}    // namespace b200

using namespace b200;

C_EXPORT unsigned long long cuda_b200_mlstm_state_floats(unsigned int dim, unsigned int vdim) { return mlstm_state_floats(dim, vdim); }

C_EXPORT unsigned long long cuda_b200_mlstm_work_floats(unsigned int tokens, unsigned int entries, unsigned int heads, unsigned int dim,
    unsigned int vdim)
{
    const unsigned long long plain = (unsigned long long)tokens * heads * (vdim + dim + 1);
    const unsigned long long chunks = mlstm_chunk_takes(dim, vdim) ? mlstm_chunk_floats(tokens, entries, heads, dim, vdim) : 0;
    return plain > chunks ? plain : chunks;
}

C_EXPORT int cuda_b200_mlstm_rows(int dtype, const cuda_b200_mlstm* a, const cuda_b200_batch* b, void* stream, unsigned int flags, int kernel)
{
    if (!a || !b || (dtype != DT_BF16 && dtype != DT_FLOAT)) { return -1; }
    if (b->tokens == 0 || b->entries == 0) { return 0; }
    if (!a->qkvg || !a->gates || !a->bias || !a->norm || !a->out || !a->state || !a->work || !b->slot || !b->pos || !b->start || !b->n || !b->token_entry
        || a->heads == 0 || a->dim == 0 || a->vdim == 0 || !(a->cap > 0.f) || a->heads > 65535u || b->entries > 65535u)
    {
        return -1;
    }
    MlstmParams p;
    p.qkvg = a->qkvg;
    p.gates = (const float*)a->gates;
    p.bias = (const float*)a->bias;
    p.norm = (const float*)a->norm;
    p.out = a->out;
    p.state = (float*)a->state;
    p.work = (float*)a->work;
    p.slot = (const int*)b->slot;
    p.pos = (const int*)b->pos;
    p.start = (const int*)b->start;
    p.n = (const int*)b->n;
    p.token_entry = (const int*)b->token_entry;
    p.ld = a->ld;
    p.ld_gates = a->ld_gates;
    p.ldo = a->ldo;
    p.k_off = a->k_off;
    p.v_off = a->v_off;
    p.g_off = a->g_off;
    p.f_off = a->f_off;
    p.heads = a->heads;
    p.dim = a->dim;
    p.vdim = a->vdim;
    p.e0 = b->first_entry;
    p.t0 = b->first_token;
    p.entries = b->entries;
    p.tokens = b->tokens;
    p.max_n = b->max_n;
    p.cap = a->cap;
    p.eps = a->eps;
    p.q_scale = a->q_scale;
    const bool pdl = (flags & 1u) != 0;
    if (dtype == DT_FLOAT) { kernel = 1; }
    if (kernel == 3 || (kernel == 0 && b->max_n > 8))
    {
        const int rc = launch_mlstm_chunk(p, b->entries, (cudaStream_t)stream, pdl);
        if (rc != -1 || kernel == 3) { return rc; }
    }
    if (kernel == 0 || kernel == 2)
    {
        const int rc = launch_mlstm_step(p, b->entries, (cudaStream_t)stream, pdl);
        if (rc != -1 || kernel == 2) { return rc; }
    }
    return dtype == DT_BF16 ? mlstm_plain<__nv_bfloat16>(p, b->entries, stream, pdl) : mlstm_plain<float>(p, b->entries, stream, pdl);
}
