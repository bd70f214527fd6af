// The mLSTM recurrence for entries of a few tokens (decoding), HBM-bound: a head's matrix memory is read once, carried in
// registers over the entry's tokens and written once.
//
// A cluster holds one head of one entry, a CTA a slice of up to 64 value columns: a thread owns four columns of every RG-th key
// row.  Sums over key rows meet in shared memory once per entry, the head's sum of squares through the cluster's shared
// memory.  n is too small to share out: every CTA carries all of it, the first one stores it.
#include "mlstm.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace b200
{

constexpr unsigned int MS_THREADS = 256, MS_WARPS = MS_THREADS / 32, MS_TOKENS = 8, MS_COLS = 64, MS_MAX_DIM = 512, MS_MAX_CLUSTER = 16;

// ROWS: key rows per thread; QUADS: threads side by side (four columns each)
template <int ROWS, int QUADS>
__global__ void __launch_bounds__(MS_THREADS, ROWS <= 8 ? 3 : (ROWS <= 16 ? 2 : 1)) mlstm_step_kernel(const MlstmParams p, const unsigned int cols)
{
    constexpr unsigned int RG = MS_THREADS / QUADS;
    extern __shared__ __align__(16) float ms_smem[];
    __shared__ float red_n[MS_TOKENS][MS_WARPS], peers[MS_TOKENS][MS_MAX_CLUSTER], sq[MS_TOKENS][MS_COLS / 32], inv[MS_TOKENS];
    __shared__ float gate[MS_TOKENS][3];    // keep, add, floor of the denominator
    __shared__ float last_m;
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, quad = tid % QUADS, rg = tid / QUADS;
    const unsigned int rank = blockIdx.x, h = blockIdx.y, e = p.e0 + blockIdx.z, v_ld = mlstm_v_ld(p.vdim);
    const unsigned int c0 = rank * cols, col = c0 + 4 * quad;
    const bool live = 4 * quad < cols && col < v_ld;
    // (the batch's arrays are written before the step's first launch)
    float* st = mlstm_state_of(p, e, h);
    float* st_n = st + (size_t)p.dim * v_ld;
    const bool fresh = p.pos[e] == 0;
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e];
    if (!fresh && live && quad % 8 == 0)
    {
        for (unsigned int d = rg; d < p.dim; d += RG) { asm volatile("prefetch.global.L2 [%0];" ::"l"(st + (size_t)d * v_ld + col)); }
    }
    grid_dependency_launch();
    grid_dependency_wait();
    float4 S[ROWS];
#pragma unroll
    for (int i = 0; i < ROWS; i++)
    {
        const unsigned int d = rg + i * RG;
        S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && live && d < p.dim) { S[i] = *reinterpret_cast<const float4*>(st + (size_t)d * v_ld + col); }
    }
    float nn[MS_MAX_DIM / MS_THREADS];
#pragma unroll
    for (unsigned int j = 0; j < MS_MAX_DIM / MS_THREADS; j++)
    {
        const unsigned int d = tid + j * MS_THREADS;
        nn[j] = !fresh && d < p.dim ? st_n[d] : 0.f;
    }
    const __nv_bfloat16* base = (const __nv_bfloat16*)p.qkvg + (size_t)start * p.ld;
    float* part = ms_smem;                           // [n][warps][64]
    float* q = part + n * (MS_WARPS * MS_COLS);      // [n][dim]
    float* k = q + n * p.dim;                        // [n][dim]
    for (unsigned int j = tid; j < n * p.dim; j += MS_THREADS)
    {
        const __nv_bfloat16* x = base + (size_t)(j / p.dim) * p.ld + h * p.dim + j % p.dim;
        q[j] = __bfloat162float(x[0]) * p.q_scale;
        k[j] = __bfloat162float(x[p.k_off]);
    }
    if (warp == 0)
    {
        float in = 0.f, forget = 0.f;
        if (lane < n) { mlstm_gates(p, start + lane, h, in, forget); }
        float m = fresh ? 0.f : st_n[mlstm_n_ld(p.dim)];
        for (unsigned int t = 0; t < n; t++)
        {
            const float i = __shfl_sync(0xFFFFFFFFu, in, t), f = __shfl_sync(0xFFFFFFFFu, forget, t), m1 = fmaxf(f + m, i);
            if (lane == 0)
            {
                gate[t][0] = expf(f + m - m1);
                gate[t][1] = expf(i - m1);
                gate[t][2] = expf(-m1);
            }
            m = m1;
        }
        if (lane == 0) { last_m = m; }
    }
    __syncthreads();
    for (unsigned int t = 0; t < n; t++)
    {
        const float keep = gate[t][0], add = gate[t][1];
        const float *qt = q + t * p.dim, *kt = k + t * p.dim;
        float v[4] = { 0.f, 0.f, 0.f, 0.f };
        if (live)
        {
            const __nv_bfloat16* x = base + (size_t)t * p.ld + p.v_off + h * p.vdim + col;
#pragma unroll
            for (int j = 0; j < 4; j++) { v[j] = col + j < p.vdim ? add * __bfloat162float(x[j]) : 0.f; }
        }
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < ROWS; i++)
        {
            const unsigned int d = rg + i * RG;
            if (d < p.dim)
            {
                const float kd = kt[d], qd = qt[d];
                S[i].x = fmaf(kd, v[0], keep * S[i].x);
                S[i].y = fmaf(kd, v[1], keep * S[i].y);
                S[i].z = fmaf(kd, v[2], keep * S[i].z);
                S[i].w = fmaf(kd, v[3], keep * S[i].w);
                o.x = fmaf(S[i].x, qd, o.x);
                o.y = fmaf(S[i].y, qd, o.y);
                o.z = fmaf(S[i].z, qd, o.z);
                o.w = fmaf(S[i].w, qd, o.w);
            }
        }
#pragma unroll
        for (int s = QUADS; s < 32; s *= 2)
        {
            o.x += __shfl_xor_sync(0xFFFFFFFFu, o.x, s);
            o.y += __shfl_xor_sync(0xFFFFFFFFu, o.y, s);
            o.z += __shfl_xor_sync(0xFFFFFFFFu, o.z, s);
            o.w += __shfl_xor_sync(0xFFFFFFFFu, o.w, s);
        }
        if (lane < QUADS) { *reinterpret_cast<float4*>(part + (t * MS_WARPS + warp) * MS_COLS + 4 * lane) = o; }
        float nq = 0.f;
#pragma unroll
        for (unsigned int j = 0; j < MS_MAX_DIM / MS_THREADS; j++)
        {
            const unsigned int d = tid + j * MS_THREADS;
            if (d < p.dim)
            {
                nn[j] = fmaf(add, kt[d], keep * nn[j]);
                nq = fmaf(nn[j], qt[d], nq);
            }
        }
        nq = warp_sum(nq);
        if (lane == 0) { red_n[t][warp] = nq; }
    }
#pragma unroll
    for (int i = 0; i < ROWS; i++)
    {
        const unsigned int d = rg + i * RG;
        if (live && d < p.dim) { *reinterpret_cast<float4*>(st + (size_t)d * v_ld + col) = S[i]; }
    }
    __syncthreads();
    // outputs of the CTA's columns: a warp per 32 columns of a token
    for (unsigned int w = warp; w < n * (MS_COLS / 32); w += MS_WARPS)
    {
        const unsigned int t = w / (MS_COLS / 32), half = w % (MS_COLS / 32), c = half * 32 + lane;
        float o = 0.f, nq = 0.f;
        if (c < 4 * QUADS)
        {
#pragma unroll
            for (unsigned int r = 0; r < MS_WARPS; r++) { o += part[(t * MS_WARPS + r) * MS_COLS + c]; }
        }
#pragma unroll
        for (unsigned int r = 0; r < MS_WARPS; r++) { nq += red_n[t][r]; }
        o /= fmaxf(fabsf(nq), gate[t][2]) + 1e-6f;
        if (c >= cols || c0 + c >= p.vdim) { o = 0.f; }
        const float s = warp_sum(o * o);
        part[t * MS_WARPS * MS_COLS + c] = o;    // this lane alone reads and writes the column
        if (lane == 0) { sq[t][half] = s; }
    }
    __syncthreads();
    cg::cluster_group cluster = cg::this_cluster();
    const unsigned int ranks = cluster.num_blocks();
    if (tid < n * ranks)
    {
        const unsigned int t = tid / ranks, r = tid % ranks;
        float s = 0.f;
#pragma unroll
        for (unsigned int j = 0; j < MS_COLS / 32; j++) { s += sq[t][j]; }
        *cluster.map_shared_rank(&peers[t][rank], r) = s;
    }
    cluster.sync();    // also: every CTA has read n and m
    if (tid < n)
    {
        float s = 0.f;
        for (unsigned int r = 0; r < ranks; r++) { s += peers[tid][r]; }
        inv[tid] = 1.0f / sqrtf(s / (float)p.vdim + p.eps);
    }
    __syncthreads();
    for (unsigned int j = tid; j < n * cols; j += MS_THREADS)
    {
        const unsigned int t = j / cols, c = j % cols;
        if (c0 + c < p.vdim)
        {
            const unsigned int at = h * p.vdim + c0 + c;
            const float g = sigmoid_f32(__bfloat162float(base[(size_t)t * p.ld + p.g_off + at]));
            ((__nv_bfloat16*)p.out)[(size_t)(start + t) * p.ldo + at] = __float2bfloat16_rn(part[t * MS_WARPS * MS_COLS + c] * inv[t] * p.norm[at] * g);
        }
    }
    if (rank == 0)
    {
#pragma unroll
        for (unsigned int j = 0; j < MS_MAX_DIM / MS_THREADS; j++)
        {
            const unsigned int d = tid + j * MS_THREADS;
            if (d < p.dim) { st_n[d] = nn[j]; }
        }
        if (tid == 0) { st_n[mlstm_n_ld(p.dim)] = last_m; }
    }
}

template <int ROWS, int QUADS>
static int run_step(const MlstmParams& p, unsigned int entries, unsigned int ranks, unsigned int cols, void* stream, bool pdl)
{
    const size_t smem = (size_t)p.max_n * (2 * p.dim + MS_WARPS * MS_COLS) * 4;
    return launch_cluster("mlstm_step", mlstm_step_kernel<ROWS, QUADS>, dim3(ranks, p.heads, entries), dim3(MS_THREADS), smem, ranks, stream, pdl, p, cols);
}

template <int QUADS>
static int step_rows(const MlstmParams& p, unsigned int entries, unsigned int ranks, unsigned int cols, void* stream, bool pdl)
{
    const unsigned int rows = (p.dim + MS_THREADS / QUADS - 1) / (MS_THREADS / QUADS);
    if (rows <= 4) { return run_step<4, QUADS>(p, entries, ranks, cols, stream, pdl); }
    if (rows <= 8) { return run_step<8, QUADS>(p, entries, ranks, cols, stream, pdl); }
    if (rows <= 16) { return run_step<16, QUADS>(p, entries, ranks, cols, stream, pdl); }
    return run_step<32, QUADS>(p, entries, ranks, cols, stream, pdl);
}

int launch_mlstm_step(const MlstmParams& p, unsigned int entries, cudaStream_t stream, bool pdl)
{
    if (p.max_n > MS_TOKENS || p.dim > MS_MAX_DIM || p.vdim > MS_COLS * MS_MAX_CLUSTER) { return -1; }
    const DecoderDevice* dev = decoder_device();
    if (!dev) { return 1; }
    // slices of 16 columns, of more in clusters of eight; clusters of sixteen where they are needed, or all fit at once
    unsigned int ranks = (p.vdim + 15) / 16;
    const bool wide = p.vdim > 8 * MS_COLS || (p.vdim > 256 && entries * p.heads * 16 <= (unsigned int)dev->sm_count);
    if (ranks > 8) { ranks = wide ? 16 : 8; }
    const unsigned int cols = ((p.vdim + ranks - 1) / ranks + 3) / 4 * 4;
    ranks = (p.vdim + cols - 1) / cols;
    if (cols <= 16) { return step_rows<4>(p, entries, ranks, cols, stream, pdl); }
    if (cols <= 32) { return step_rows<8>(p, entries, ranks, cols, stream, pdl); }
    return step_rows<16>(p, entries, ranks, cols, stream, pdl);
}

}    // namespace b200
