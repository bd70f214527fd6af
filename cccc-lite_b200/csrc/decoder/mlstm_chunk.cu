// The mLSTM recurrence over prompts, in chunks of 128 tokens.
//
// Inside a chunk, with F the running sum of the log forget gates, a_s = i_s - F_s and M_t = max(m_0, a_s up to t), the running
// maximum is m_t = F_t + M_t, and unrolled from the chunk's first token
//   o_t ~ e^(m_0 - M_t) S_0^T q_t + sum_{s <= t} e^(a_s - M_t) (q_t . k_s) v_s,   S_L = e^(m_0 - M_L) S_0 + sum_s e^(a_s - M_L) k_s v_s^T,
// no exponent above zero.  Three kernels:
//   gates  : F and a of every chunk.
//   states : a CTA per 32 value columns of a head walks an entry's chunks, its columns of S as float accumulators in registers
//            (mma.sync); it leaves the state ahead of every chunk in scratch memory.
//   outputs: a cluster per (chunk, head), a CTA per 64 or 128 value columns, on tcgen05; the head's sum of squares meets in the
//            cluster.
// One operand of every product is exact (q, k or v); the other - S, weighted values, weighted scores - enters as the sum of two
// BF16 numbers.
#include "../gemm_stream.cuh"
#include "attention_mma.cuh"
#include "mlstm.cuh"
#include "tile_common.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace b200
{

constexpr unsigned int MC_L = 128, MC_WARPS = 16, MC_THREADS = 32 * MC_WARPS, MC_COLS = 32, MC_MAX_DIM = 256, MC_MAX_CLUSTER = 8;

__host__ __device__ __forceinline__ unsigned int mc_dp(unsigned int dim) { return dim <= 64 ? 64 : (dim <= 128 ? 128 : 256); }
__host__ __device__ __forceinline__ unsigned int mc_vp(unsigned int vdim) { return (vdim + MC_COLS - 1) / MC_COLS * MC_COLS; }
// Scratch: of every (chunk, head) S high [dp][vp] and S low; behind all of these, n and m ahead of the chunk, n and m behind the
// entry's last chunk, F, a, the largest a and the last F.
__host__ __device__ __forceinline__ size_t mc_matrix(unsigned int dim, unsigned int vdim) { return (size_t)mc_dp(dim) * mc_vp(vdim); }
__host__ __device__ __forceinline__ size_t mc_record(unsigned int dim) { return 2 * (mc_dp(dim) + 4) + 2 * MC_L + 4; }
__host__ __device__ __forceinline__ unsigned int mc_slots(unsigned int tokens, unsigned int entries) { return tokens / MC_L + entries; }
struct ChunkRecord
{
    unsigned int at;                  // (chunk, head)
    __nv_bfloat16* S;
    float *n, *last, *F, *a, *top;    // m behind n, the last m behind last
};
__device__ __forceinline__ ChunkRecord mc_record_of(const MlstmParams& p, unsigned int e, unsigned int chunk, unsigned int head)
{
    // entries' chunks one behind the other
    const unsigned int at = (((unsigned int)p.start[e] - p.t0) / MC_L + (e - p.e0) + chunk) * p.heads + head, dp = mc_dp(p.dim);
    const size_t matrix = mc_matrix(p.dim, p.vdim);
    ChunkRecord c;
    c.at = at;
    c.S = reinterpret_cast<__nv_bfloat16*>(p.work + at * matrix);
    c.n = p.work + (size_t)mc_slots(p.tokens, p.entries) * p.heads * matrix + at * mc_record(p.dim);
    c.last = c.n + dp + 4;
    c.F = c.last + dp + 4;
    c.a = c.F + MC_L;
    c.top = c.a + MC_L;
    return c;
}

// grid (chunks, heads, entries), a thread per token.  Tokens behind the last: F stays, a = -inf.
__global__ void __launch_bounds__(MC_L) mlstm_gates_kernel(const MlstmParams p)
{
    __shared__ float sums[MC_L / 32], tops[MC_L / 32];
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c = blockIdx.x, h = blockIdx.y, e = p.e0 + blockIdx.z;
    const unsigned int n = (unsigned int)p.n[e], t = c * MC_L + tid;
    if (c * MC_L >= n) { return; }
    float in = -INFINITY, f = 0.f;
    if (t < n) { mlstm_gates(p, (unsigned int)p.start[e] + t, h, in, f); }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1)
    {
        const float x = __shfl_up_sync(0xFFFFFFFFu, f, o);
        if (lane >= (unsigned int)o) { f += x; }
    }
    if (lane == 31) { sums[warp] = f; }
    __syncthreads();
    for (unsigned int w = 0; w < warp; w++) { f += sums[w]; }
    const float a = in - f;
    const ChunkRecord rec = mc_record_of(p, e, c, h);
    rec.F[tid] = f;
    rec.a[tid] = a;
    float top = a;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) { top = fmaxf(top, __shfl_xor_sync(0xFFFFFFFFu, top, o)); }
    if (lane == 0) { tops[warp] = top; }
    __syncthreads();
    if (tid == MC_L - 1)
    {
        rec.top[0] = fmaxf(fmaxf(tops[0], tops[1]), fmaxf(tops[2], tops[3]));
        rec.top[1] = f;
    }
}

// Rows [0, live) of a projection, `width` elements from `src` on, into padded shared rows of PADDED elements; rows behind and columns
// past `width` are zero.
template <unsigned int PADDED>
__device__ __forceinline__ void mc_fetch(uint32_t dst, const __nv_bfloat16* src, unsigned int ld, unsigned int live, unsigned int width)
{
    constexpr unsigned int PER = PADDED / 8, STRIDE = (PADDED + 8) * 2;
#pragma unroll
    for (unsigned int i = 0; i < (MC_L * PER + MC_THREADS - 1) / MC_THREADS; i++)
    {
        const unsigned int c = threadIdx.x + i * MC_THREADS, r = c / PER, d = c % PER;
        if (MC_L * PER % MC_THREADS == 0 || c < MC_L * PER)
        {
            const bool ok = r < live && d * 8 < width;
            cp_async16(dst + r * STRIDE + d * 16, src + (ok ? (size_t)r * ld + d * 8 : 0), ok);
        }
    }
}

// grid (column blocks of 32, heads, entries); a warp owns 16 rows of S
template <int DP>
__global__ void __launch_bounds__(MC_THREADS) mlstm_states_kernel(const MlstmParams p)
{
    extern __shared__ __align__(16) unsigned char mc_raw[];
    constexpr unsigned int VS = (MC_COLS + 8) * 2, KS = (DP + 8) * 2, KBYTES = MC_L * KS;
    __shared__ float w[MC_L];
    // weighted values; behind the columns the weights themselves, which make n
    __shared__ __align__(16) __nv_bfloat16 hi[MC_L * (MC_COLS + 8)], lo[MC_L * (MC_COLS + 8)];
    const unsigned int vp = mc_vp(p.vdim);
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, gt = lane & 3, gc = gt * 2, d0 = warp * 16;
    const unsigned int c0 = blockIdx.x * MC_COLS, h = blockIdx.y, e = p.e0 + blockIdx.z;
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], chunks = (n + MC_L - 1) / MC_L;
    const bool fresh = p.pos[e] == 0;
    float* st = mlstm_state_of(p, e, h);
    const unsigned int v_ld = mlstm_v_ld(p.vdim), vw = min(MC_COLS, p.vdim - c0);
    float* st_n = st + (size_t)p.dim * v_ld;
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg + (size_t)start * p.ld;
    const uint32_t ks = smem_u32(mc_raw), vs = ks + 2 * KBYTES, hs = smem_u32(hi), ls = smem_u32(lo);
    const __nv_bfloat16* v_raw = reinterpret_cast<const __nv_bfloat16*>(mc_raw + 2 * KBYTES);
    auto fetch = [&](unsigned int c) {
        if (c < chunks)
        {
            const unsigned int live = min(MC_L, n - c * MC_L);
            mc_fetch<DP>(ks + (c & 1u) * KBYTES, x + (size_t)c * MC_L * p.ld + p.k_off + h * p.dim, p.ld, live, p.dim);
            mc_fetch<MC_COLS>(vs + (c & 1u) * MC_L * VS, x + (size_t)c * MC_L * p.ld + p.v_off + h * p.vdim + c0, p.ld, live, vw);
        }
        cp_async_commit();
    };
    fetch(0);
    float S[MC_COLS / 8][4];
#pragma unroll
    for (int j = 0; j < (int)MC_COLS / 8; j++)
    {
#pragma unroll
        for (int half = 0; half < 2; half++)
        {
            const unsigned int d = d0 + gr + 8 * half, col = c0 + j * 8 + gc;
            float2 v = make_float2(0.f, 0.f);
            if (!fresh && d < p.dim && col < p.vdim) { v = *reinterpret_cast<const float2*>(st + (size_t)d * v_ld + col); }
            S[j][2 * half] = v.x;
            S[j][2 * half + 1] = v.y;
        }
    }
    float m = fresh ? 0.f : st_n[mlstm_n_ld(p.dim)];
    float nn[4] = { 0.f, 0.f, 0.f, 0.f };    // n of rows gr and gr + 8 in the first column's lanes, elements 0 and 2
    const bool carries = blockIdx.x == 0, holds = carries && gt == 0 && d0 < (unsigned int)DP;
#pragma unroll
    for (int half = 0; half < 2; half++)
    {
        const unsigned int d = d0 + gr + 8 * half;
        if (holds && !fresh && d < p.dim) { nn[2 * half] = st_n[d]; }
    }
    if (tid < MC_L)
    {
#pragma unroll
        for (int j = 0; j < 4; j++)
        {
            reinterpret_cast<uint32_t*>(hi + tid * (MC_COLS + 8) + MC_COLS)[j] = 0u;
            reinterpret_cast<uint32_t*>(lo + tid * (MC_COLS + 8) + MC_COLS)[j] = 0u;
        }
    }
    ChunkRecord rec = mc_record_of(p, e, 0, h);
    float a = tid < MC_L ? rec.a[tid] : 0.f;
    float2 end = *reinterpret_cast<const float2*>(rec.top);
    for (unsigned int c = 0; c < chunks; c++)
    {
        const unsigned int live = min(MC_L, n - c * MC_L);
        fetch(c + 1);
        const float top = fmaxf(m, end.x), keep = expf(m - top);    // M at the chunk's end
        if (tid < MC_L)
        {
            const float y = expf(a - top);
            const __nv_bfloat16 high = __float2bfloat16_rn(y);
            w[tid] = y;
            hi[tid * (MC_COLS + 8) + MC_COLS] = high;
            lo[tid * (MC_COLS + 8) + MC_COLS] = __float2bfloat16_rn(y - __bfloat162float(high));
        }
        if (d0 < (unsigned int)DP && (!fresh || c > 0))
        {
#pragma unroll
            for (int half = 0; half < 2; half++)
            {
                uint32_t part[2][4];    // high, low; of the eight columns of tile j
#pragma unroll
                for (int j = 0; j < 4; j++)
                {
                    const float s0 = S[j][2 * half], s1 = S[j][2 * half + 1];
                    part[0][j] = pack_bf16x2(s0, s1);
                    part[1][j] = pack_bf16x2(s0 - __uint_as_float(part[0][j] << 16), s1 - __uint_as_float(part[0][j] & 0xFFFF0000u));
                }
                // the four lanes of a row exchange, so that lane t has all of tile t
#pragma unroll
                for (int k = 0; k < 2; k++)
                {
                    uint32_t row[4];
#pragma unroll
                    for (int step = 0; step < 4; step++)
                    {
                        // to lane gt ^ step goes tile gt ^ step
                        const unsigned int j = gt ^ step;
                        const uint32_t give = j == 0 ? part[k][0] : (j == 1 ? part[k][1] : (j == 2 ? part[k][2] : part[k][3]));
                        const uint32_t got = __shfl_xor_sync(0xFFFFFFFFu, give, step);
#pragma unroll
                        for (unsigned int i = 0; i < 4; i++)
                        {
                            if (i == (gt ^ (unsigned int)step)) { row[i] = got; }
                        }
                    }
                    __nv_bfloat16* y = rec.S + (size_t)(k * DP + d0 + gr + 8 * half) * vp + c0 + gt * 8;
                    *reinterpret_cast<uint4*>(y) = make_uint4(row[0], row[1], row[2], row[3]);
                }
            }
        }
        if (holds)
        {
            rec.n[d0 + gr] = nn[0];
            rec.n[d0 + gr + 8] = nn[2];
        }
        if (carries && tid == 0) { rec.n[DP] = m; }
        m = end.y + top;
        const ChunkRecord now = rec;
        if (c + 1 < chunks)
        {
            rec = mc_record_of(p, e, c + 1, h);
            if (tid < MC_L) { a = rec.a[tid]; }
            end = *reinterpret_cast<const float2*>(rec.top);
        }
        cp_async_wait<1>();
        __syncthreads();
        const __nv_bfloat16* v = v_raw + (c & 1u) * MC_L * (MC_COLS + 8);
#pragma unroll
        for (unsigned int i = tid; i < MC_L * MC_COLS / 2; i += MC_THREADS)
        {
            const unsigned int s = i / (MC_COLS / 2), at = s * (MC_COLS + 8) + (i % (MC_COLS / 2)) * 2;
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v + at));
            const float y0 = w[s] * f.x, y1 = w[s] * f.y;
            const uint32_t u = pack_bf16x2(y0, y1);
            *reinterpret_cast<uint32_t*>(hi + at) = u;
            *reinterpret_cast<uint32_t*>(lo + at) = pack_bf16x2(y0 - __uint_as_float(u << 16), y1 - __uint_as_float(u & 0xFFFF0000u));
        }
        __syncthreads();
        if (d0 < (unsigned int)DP)
        {
            const uint32_t kb = ks + (c & 1u) * KBYTES + ((lane & 7) + ((lane >> 4) << 3)) * KS + ((lane >> 3) & 1) * 16 + d0 * 2;
            const uint32_t vb = (lane & 15) * VS + (lane >> 4) * 16;
#pragma unroll
            for (int j = 0; j < (int)MC_COLS / 8; j++)
            {
#pragma unroll
                for (int i = 0; i < 4; i++) { S[j][i] *= keep; }
            }
#pragma unroll
            for (int i = 0; i < 4; i++) { nn[i] *= keep; }
#pragma unroll 4
            for (unsigned int s0 = 0; s0 < live; s0 += 16)
            {
                uint32_t b[2][MC_COLS / 16][4], k[4];
                if (carries)
                {
                    uint32_t x[4];
                    ldmatrix_x4_trans(x, (lane < 16 ? hs : ls) + (s0 + (lane & 15)) * VS + MC_COLS * 2);
                    uint32_t k2[4];
                    ldmatrix_x4_trans(k2, kb + s0 * KS);
                    mma_bf16_16816(nn, k2[0], k2[1], k2[2], k2[3], x[0], x[1]);
                    mma_bf16_16816(nn, k2[0], k2[1], k2[2], k2[3], x[2], x[3]);
                }
                ldmatrix_x4_trans(k, kb + s0 * KS);
#pragma unroll
                for (int j = 0; j < (int)MC_COLS / 16; j++)
                {
                    ldmatrix_x4_trans(b[0][j], hs + vb + s0 * VS + j * 32);
                    ldmatrix_x4_trans(b[1][j], ls + vb + s0 * VS + j * 32);
                }
#pragma unroll
                for (int part = 0; part < 2; part++)
                {
#pragma unroll
                    for (int j = 0; j < (int)MC_COLS / 16; j++)
                    {
                        mma_bf16_16816(S[2 * j], k[0], k[1], k[2], k[3], b[part][j][0], b[part][j][1]);
                        mma_bf16_16816(S[2 * j + 1], k[0], k[1], k[2], k[3], b[part][j][2], b[part][j][3]);
                    }
                }
            }
        }
        // other column blocks may still have to read the old n and m: the last kernel puts the new ones in place
        if (c + 1 == chunks)
        {
            if (holds)
            {
                now.last[d0 + gr] = nn[0];
                now.last[d0 + gr + 8] = nn[2];
            }
            if (carries && tid == 0) { now.last[DP] = m; }
        }
        __syncthreads();    // the next chunk but one takes this one's place
    }
    cp_async_wait<0>();
#pragma unroll
    for (int j = 0; j < (int)MC_COLS / 8; j++)
    {
#pragma unroll
        for (int half = 0; half < 2; half++)
        {
            const unsigned int d = d0 + gr + 8 * half, col = c0 + j * 8 + gc;
            if (d < p.dim && col < p.vdim) { *reinterpret_cast<float2*>(st + (size_t)d * v_ld + col) = make_float2(S[j][2 * half], S[j][2 * half + 1]); }
        }
    }
}

__host__ __device__ constexpr unsigned int mc_states_smem(unsigned int dp) { return 2 * MC_L * ((dp + 8) * 2 + (MC_COLS + 8) * 2); }
// ---- outputs ---------------------------------------------------------------------------------------
constexpr int MO_THREADS = 32 * 10;
constexpr int MO_BLOCK = 64 * 128, MO_ROWS = 2 * MO_BLOCK;    // 64 rows x 64 elements; the 128 tokens' block of 64 elements
constexpr uint32_t MO_P = 128, MO_O = 256, MO_TMEM = 512;      // columns: scores, weighted scores (high, low), what the chunk gives, what S gives
__host__ __device__ constexpr int mo_slice(int vb) { return 2 * (vb / 64) * MO_BLOCK; }    // 64 rows of S: high, low
__host__ __device__ constexpr int mo_smem(int dp, int vb) { return 1024 + 2 * (dp / 64) * MO_ROWS + (vb / 64) * MO_ROWS + mo_slice(vb) + 1024; }

// grid (column blocks of VB = the cluster, heads, entries x chunks).  A TMA lane fetches q, k and v of the chunk and slices of 64 rows of
// S: the first beside them, the following ones where k was, once the scores are out.  The MMA lane issues q k^T, then q S, then
// (weighted scores) v.  Eight warps own a row of scores per thread, half of its columns each.
template <int VB>
__global__ void __launch_bounds__(MO_THREADS, 1) mlstm_outputs_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ CUtensorMap tmS,
    const __grid_constant__ MlstmParams p, const unsigned int max_chunks, unsigned int* status)
{
    extern __shared__ unsigned char mo_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(mo_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ float F[MC_L], a[MC_L], M[MC_L], maxima[MC_L / 32], sq[2][MC_L], nq[2][MC_L], peers[MC_MAX_CLUSTER][MC_L], n0[MC_MAX_DIM];
    constexpr int SLICE = mo_slice(VB), HB = VB / 2, MAX_PLACES = 8;
    const unsigned int dp = mc_dp(p.dim), blocks = dp / 64;
    uint64_t* qk_full = reinterpret_cast<uint64_t*>(smem);
    uint64_t *v_full = qk_full + 1, *s_full = qk_full + 2, *p_ready = qk_full + 3, *o_full = qk_full + 4, *slice_full = qk_full + 5,
             *slice_empty = slice_full + MAX_PLACES;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(slice_empty + MAX_PLACES);
    volatile unsigned int* abort_flag = reinterpret_cast<volatile unsigned int*>(tmem_slot + 1);
    unsigned char* qs = smem + 1024;
    unsigned char* ks = qs + blocks * MO_ROWS;
    unsigned char* vs = ks + blocks * MO_ROWS;
    unsigned char* ss = vs + (VB / 64) * MO_ROWS;
    const unsigned int places = min((unsigned int)MAX_PLACES, 1u + blocks * MO_ROWS / SLICE);    // of slices
    auto place = [&](unsigned int i) { return i % places == 0 ? ss : ks + (i % places - 1) * SLICE; };

    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const unsigned int rank = blockIdx.x, h = blockIdx.y, e = p.e0 + blockIdx.z / max_chunks, c = blockIdx.z % max_chunks, c0 = rank * VB;
    if (tid == 0)
    {
        for (int i = 0; i < 5 + 2 * MAX_PLACES; i++) { mbar_init(qk_full + i, i == 3 ? 8 : 1); }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e];
    if (c * MC_L >= n) { return; }    // the whole cluster
    if (warp == 1) { tmem_alloc(tmem_slot, MO_TMEM); }
    const unsigned int live = min(MC_L, n - c * MC_L), first = start + c * MC_L;
    const bool fresh = p.pos[e] == 0 && c == 0;
    const ChunkRecord rec = mc_record_of(p, e, c, h);
    const unsigned int slices = fresh ? 0 : blocks, steps = p.dim / 16;
    const float m0 = fresh ? 0.f : rec.n[dp];
    float t_max = -INFINITY;
    if (tid < MC_L)    // M: running maxima of a, with m0
    {
        F[tid] = rec.F[tid];
        t_max = rec.a[tid];
        a[tid] = t_max * 1.44269504088896341f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1)
        {
            const float y = __shfl_up_sync(0xFFFFFFFFu, t_max, o);
            if (lane >= (unsigned int)o) { t_max = fmaxf(t_max, y); }
        }
        if (lane == 31) { maxima[warp] = t_max; }
    }
    for (unsigned int d = tid; d < dp; d += MO_THREADS) { n0[d] = fresh || d >= p.dim ? 0.f : rec.n[d]; }
    __syncthreads();
    if (tid < MC_L)
    {
        t_max = fmaxf(m0, t_max);
        for (unsigned int j = 0; j < warp; j++) { t_max = fmaxf(t_max, maxima[j]); }
        M[tid] = t_max;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    auto give_up = [&](unsigned int role, unsigned int step) {
        note_timeout(status, WAIT_MLSTM_TILE, role, step);
        *abort_flag = 1;
    };
    auto wait = [&](uint64_t* bar, unsigned int parity) { return *abort_flag == 0 && mbar_wait_bounded(bar, parity & 1u); };
    const unsigned int quarter = warp & 3u, half = warp >= 2 ? (warp - 2u) >> 2 : 0u, t = quarter * 32 + lane;    // row of an epilogue thread
    float o[HB], inv = 0.f;
    bool good = false;

    if (warp == 0)
    {
        if (lane == 0)
        {
            const int y = (int)first, xq = (int)(h * p.dim), xk = (int)(p.k_off + h * p.dim), xv = (int)(p.v_off + h * p.vdim + c0);
            mbar_expect_tx(qk_full, 2 * blocks * MO_ROWS);
            for (unsigned int b = 0; b < blocks; b++)
            {
                for (int r = 0; r < 2; r++)
                {
                    tma_load_2d(qs + b * MO_ROWS + r * MO_BLOCK, &tmX, xq + (int)b * 64, y + r * 64, qk_full);
                    tma_load_2d(ks + b * MO_ROWS + r * MO_BLOCK, &tmX, xk + (int)b * 64, y + r * 64, qk_full);
                }
            }
            mbar_arrive(qk_full);
            mbar_expect_tx(v_full, (VB / 64) * MO_ROWS);
            for (int r = 0; r < 2; r++)    // 64 rows by 64 rows
            {
                for (int b = 0; b < VB / 64; b++) { tma_load_2d(vs + (r * (VB / 64) + b) * MO_BLOCK, &tmX, xv + b * 64, y + r * 64, v_full); }
            }
            mbar_arrive(v_full);
            bool ok = true;
            unsigned int issued = 0;
            for (unsigned int i = 0; i < slices && ok; i++)
            {
                const unsigned int at = i % places;
                if (i == 1) { ok = wait(s_full, 0); }    // k has been read
                if (ok && i >= places) { ok = wait(slice_empty + at, i / places - 1); }
                if (!ok) { break; }
                mbar_expect_tx(slice_full + at, SLICE);
                for (int part = 0; part < 2; part++)
                {
                    for (int b = 0; b < VB / 64; b++)
                    {
                        tma_load_2d(place(i) + (part * (VB / 64) + b) * MO_BLOCK, &tmS, (int)c0 + b * 64, (int)((rec.at * 2 + part) * dp + i * 64), slice_full + at);
                    }
                }
                mbar_arrive(slice_full + at);
                issued++;
            }
            if (!ok)
            {
                give_up(0, issued);
                // wait (bounded) for the copies in flight before the CTA may leave
                auto drain = [&](uint64_t* bar, unsigned int parity) {
                    const unsigned long long t0 = global_timer_ns();
                    while (!mbar_try_wait(bar, parity & 1u) && global_timer_ns() - t0 < 100000ull) {}
                };
                drain(qk_full, 0);
                drain(v_full, 0);
                for (unsigned int i = issued > places ? issued - places : 0; i < issued; i++) { drain(slice_full + i % places, i / places); }
            }
        }
    }
    else if (warp == 1)
    {
        const uint32_t q_addr = smem_u32(qs), k_addr = smem_u32(ks), v_addr = smem_u32(vs);
        const uint32_t idesc_s = umma_idesc_bf16(MC_L, MC_L), idesc_o = umma_idesc_bf16(MC_L, VB) | (1u << 16);    // B is MN-major
        unsigned int at = 0;
        bool ok = wait(qk_full, 0);
        if (ok)
        {
            tc_fence_after();
            if (elect_one())
            {
                for (unsigned int k = 0; k < steps; k++)
                {
                    const uint32_t off = (k / 4) * MO_ROWS + (k % 4) * 32;
                    umma_bf16(tmem, umma_desc_kmajor_sw128(q_addr + off), umma_desc_kmajor_sw128(k_addr + off), idesc_s, k != 0 ? 1u : 0u);
                }
                umma_commit(s_full);
            }
            __syncwarp();
        }
        for (unsigned int i = 0; i < slices && ok; i++)
        {
            at = i + 1;
            ok = wait(slice_full + i % places, i / places);
            if (!ok) { break; }
            tc_fence_after();
            if (elect_one())
            {
                const uint32_t s_addr = smem_u32(place(i));
                for (unsigned int part = 0; part < 2; part++)
                {
                    for (unsigned int k = 0; k < 4 && i * 4 + k < steps; k++)
                    {
                        umma_bf16(tmem + MO_O + VB, umma_desc_kmajor_sw128(q_addr + i * MO_ROWS + k * 32),
                            umma_desc_mnmajor_sw128(s_addr + part * (VB / 64) * MO_BLOCK + k * 2048), idesc_o, (i | part | k) != 0 ? 1u : 0u);
                    }
                }
                umma_commit(slice_empty + i % places);
            }
            __syncwarp();
        }
        if (ok)
        {
            at = slices + 1;
            ok = wait(v_full, 0) && wait(p_ready, 0);
        }
        if (ok)
        {
            tc_fence_after();
            if (elect_one())
            {
                for (unsigned int part = 0; part < 2; part++)
                {
                    for (unsigned int k = 0; k < MC_L / 16; k++)
                    {
                        umma_bf16_ts(tmem + MO_O, tmem + MO_P + part * 64 + k * 8, umma_desc_mnmajor_sw128(v_addr + (k / 4) * (VB / 64) * MO_BLOCK + (k % 4) * 2048),
                            idesc_o, (part | k) != 0 ? 1u : 0u);
                    }
                }
                umma_commit(o_full);
            }
            __syncwarp();
        }
        else
        {
            if (lane == 0) { give_up(1, at); }
            if (elect_one()) { umma_commit(o_full); }    // completes once the MMAs in flight have stopped reading shared memory
            __syncwarp();
        }
    }
    else
    {
        const uint32_t lanes = tmem + ((quarter * 32u) << 16);
        const float mt = M[t], mt2 = mt * 1.44269504088896341f, carry = p.q_scale * expf(m0 - mt);
        float sum = 0.f;
        good = __all_sync(0xFFFFFFFFu, wait(s_full, 0));
        if (good)
        {
            tc_fence_after();
            // this half's 64 keys; none of them where the rows of the warp end before
#pragma unroll
            for (int q = 0; q < 2; q++)
            {
                const unsigned int s0 = half * 64 + q * 32;
                uint32_t z[32], hi[16], lo[16];
#pragma unroll
                for (int j = 0; j < 16; j++) { hi[j] = lo[j] = 0u; }
                if (s0 <= quarter * 32 + 31)
                {
                    tmem_ld_32x32(lanes + s0, z);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 16; j++)
                    {
                        float w[2];
#pragma unroll
                        for (int k = 0; k < 2; k++)
                        {
                            const unsigned int s = s0 + 2 * j + k;
                            w[k] = s <= t ? __uint_as_float(z[2 * j + k]) * p.q_scale * exp2_f32(a[s] - mt2) : 0.f;
                            sum += w[k];
                        }
                        hi[j] = pack_bf16x2(w[0], w[1]);
                        lo[j] = pack_bf16x2(w[0] - __uint_as_float(hi[j] << 16), w[1] - __uint_as_float(hi[j] & 0xFFFF0000u));
                    }
                }
                tmem_st_32x16(lanes + MO_P + s0 / 2, hi);
                tmem_st_32x16(lanes + MO_P + 64 + s0 / 2, lo);
            }
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) { mbar_arrive(p_ready); }
            if (!fresh && wait(qk_full, 0))    // n0 . q over half of the elements
            {
                float dot = 0.f;
                for (unsigned int b = half; b < 2 * blocks; b += 2)    // 32 elements at a time
                {
                    const unsigned char* row = qs + (b / 2) * MO_ROWS + t * 128;
#pragma unroll
                    for (unsigned int q = 0; q < 4; q++)
                    {
                        const unsigned int chunk = (b & 1u) * 4 + q;
                        const uint4 u = *reinterpret_cast<const uint4*>(row + ((chunk ^ (t & 7u)) * 16));
                        const uint32_t w[4] = { u.x, u.y, u.z, u.w };
                        const float* g = n0 + (b / 2) * 64 + chunk * 8;
#pragma unroll
                        for (int j = 0; j < 4; j++)
                        {
                            dot = fmaf(__uint_as_float(w[j] << 16), g[2 * j], dot);
                            dot = fmaf(__uint_as_float(w[j] & 0xFFFF0000u), g[2 * j + 1], dot);
                        }
                    }
                }
                sum = fmaf(carry, dot, sum);
            }
            nq[half][t] = sum;
            bar_sync_named(1, 256);
            inv = 1.0f / (fmaxf(fabsf(nq[0][t] + nq[1][t]), expf(-(F[t] + mt))) + 1e-6f);
            good = __all_sync(0xFFFFFFFFu, wait(o_full, 0)) && *abort_flag == 0;
            good = __all_sync(0xFFFFFFFFu, good);
        }
        else { bar_sync_named(1, 256); }
        float s = 0.f;
        if (good)
        {
            tc_fence_after();
#pragma unroll
            for (int d = 0; d < HB; d += 32)
            {
                uint32_t x[32];
                tmem_ld_32x32(lanes + MO_O + half * HB + d, x);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; j++) { o[d + j] = __uint_as_float(x[j]); }
                if (!fresh)
                {
                    tmem_ld_32x32(lanes + MO_O + VB + half * HB + d, x);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 32; j++) { o[d + j] = fmaf(carry, __uint_as_float(x[j]), o[d + j]); }
                }
#pragma unroll
                for (int j = 0; j < 32; j++)
                {
                    o[d + j] *= inv;
                    if (c0 + half * HB + d + j < p.vdim) { s += o[d + j] * o[d + j]; }
                }
            }
        }
        else if (lane == 0) { give_up(2 + quarter, half); }
        sq[half][t] = s;
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) { tmem_dealloc(tmem, MO_TMEM); }
    cg::cluster_group cluster = cg::this_cluster();
    const unsigned int ranks = cluster.num_blocks();
    for (unsigned int j = tid; j < ranks * MC_L; j += MO_THREADS)
    {
        const unsigned int r = j % MC_L;
        cluster.map_shared_rank(&peers[0][0], j / MC_L)[rank * MC_L + r] = sq[0][r] + sq[1][r];
    }
    cluster.sync();
    if (good && t < live)
    {
        float s = 0.f;
        for (unsigned int r = 0; r < ranks; r++) { s += peers[r][t]; }
        const float unit = 1.0f / sqrtf(s / (float)p.vdim + p.eps);
        const unsigned int at = h * p.vdim + c0 + half * HB;
        const __nv_bfloat16* gate = (const __nv_bfloat16*)p.qkvg + (size_t)(first + t) * p.ld + p.g_off + at;
        __nv_bfloat16* out = (__nv_bfloat16*)p.out + (size_t)(first + t) * p.ldo + at;
        const float* w = p.norm + at;
#pragma unroll
        for (int d = 0; d < HB; d += 8)
        {
            if (c0 + half * HB + d >= p.vdim) { continue; }
            const uint4 u = *reinterpret_cast<const uint4*>(gate + d);
            const uint32_t g[4] = { u.x, u.y, u.z, u.w };
            uint32_t y[4];
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                y[j] = pack_bf16x2(o[d + 2 * j] * unit * w[d + 2 * j] * sigmoid_f32(__uint_as_float(g[j] << 16)),
                    o[d + 2 * j + 1] * unit * w[d + 2 * j + 1] * sigmoid_f32(__uint_as_float(g[j] & 0xFFFF0000u)));
            }
            *reinterpret_cast<uint4*>(out + d) = make_uint4(y[0], y[1], y[2], y[3]);
        }
    }
    if (rank == 0 && (c + 1) * MC_L >= n)
    {
        float* st_n = mlstm_state_of(p, e, h) + (size_t)p.dim * mlstm_v_ld(p.vdim);
        for (unsigned int d = tid; d < p.dim; d += MO_THREADS) { st_n[d] = rec.last[d]; }
        if (tid == 0) { st_n[mlstm_n_ld(p.dim)] = rec.last[dp]; }
    }
}

template <int VB>
static int run_outputs(const MlstmParams& p, cudaStream_t stream, bool pdl)
{
    unsigned int* status = decoder_status_word();
    if (!status) { return 1; }
    const unsigned int ranks = (p.vdim + VB - 1) / VB, chunks = (p.max_n + MC_L - 1) / MC_L, dp = mc_dp(p.dim), vp = mc_vp(p.vdim);
    CUtensorMap tx, ts;
    if (!make_map_2d(&tx, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.qkvg, p.ld, (unsigned long long)p.t0 + p.tokens, (unsigned long long)p.ld * 2, 64, 64, true)
        || !make_map_2d(&ts, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.work, vp, (unsigned long long)mc_slots(p.tokens, p.entries) * p.heads * 2 * dp,
            (unsigned long long)vp * 2, 64, 64, true))
    {
        return -1;
    }
    return launch_cluster("mlstm_outputs", mlstm_outputs_kernel<VB>, dim3(ranks, p.heads, p.entries * chunks), dim3(MO_THREADS), (size_t)mo_smem((int)dp, VB), ranks,
        stream, pdl, tx, ts, p, chunks, status);
}

template <int DP>
static int run_chunks(const MlstmParams& p, unsigned int entries, cudaStream_t stream, bool pdl)
{
    const unsigned int chunks = (p.max_n + MC_L - 1) / MC_L;
    int rc = launch_kernel("mlstm_gates", mlstm_gates_kernel, dim3(chunks, p.heads, entries), dim3(MC_L), 0, stream, pdl, p);
    if (rc) { return rc; }
    rc = launch_kernel("mlstm_states", mlstm_states_kernel<DP>, dim3(mc_vp(p.vdim) / MC_COLS, p.heads, entries), dim3(MC_THREADS), (size_t)mc_states_smem(DP),
        stream, pdl, p);
    if (rc) { return rc; }
    return p.vdim <= 64 ? run_outputs<64>(p, stream, pdl) : run_outputs<128>(p, stream, pdl);
}

unsigned long long mlstm_chunk_floats(unsigned int tokens, unsigned int entries, unsigned int heads, unsigned int dim, unsigned int vdim)
{
    return (unsigned long long)mc_slots(tokens, entries) * heads * (mc_matrix(dim, vdim) + mc_record(dim));
}

bool mlstm_chunk_takes(unsigned int dim, unsigned int vdim) { return (dim % 16) == 0 && (vdim % 8) == 0 && dim <= MC_MAX_DIM && vdim <= 128 * MC_MAX_CLUSTER; }

int launch_mlstm_chunk(const MlstmParams& p, unsigned int entries, cudaStream_t stream, bool pdl)
{
    const unsigned int chunks = (p.max_n + MC_L - 1) / MC_L;
    auto low = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) != 0; };
    if (!mlstm_chunk_takes(p.dim, p.vdim) || (p.ld % 8) || (p.k_off % 8) || (p.v_off % 8) || (p.g_off % 8) || (p.ldo % 8)
        || low(p.qkvg) || low(p.work) || low(p.out) || (unsigned long long)entries * chunks > 65535ull)
    {
        return -1;
    }
    if (p.dim <= 64) { return run_chunks<64>(p, entries, stream, pdl); }
    if (p.dim <= 128) { return run_chunks<128>(p, entries, stream, pdl); }
    return run_chunks<256>(p, entries, stream, pdl);
}

}    // namespace b200
