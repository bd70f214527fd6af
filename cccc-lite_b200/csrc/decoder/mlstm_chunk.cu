// The mLSTM recurrence over prompts, in chunks of 128 tokens.
//
// Inside a chunk, with F the running sum of the log forget gates, a_s = i_s - F_s and M_t = max(m_0, a_s up to t), the running
// maximum is m_t = F_t + M_t, and unrolled from the chunk's first token
//   o_t ~ e^(m_0 - M_t) S_0^T q_t + sum_{s <= t} e^(a_s - M_t) (q_t . k_s) v_s,   S_L = e^(m_0 - M_L) S_0 + sum_s e^(a_s - M_L) k_s v_s^T,
// no exponent above zero.  Three kernels:
//   gates  : F and a of every chunk.
//   states : a CTA per 64 value columns of a head (and one for n) walks an entry's chunks, its columns of S as the accumulator in
//            tensor memory; it leaves the state ahead of every chunk in scratch memory.
//   outputs: a cluster per (chunk, head), a CTA per 64 or 128 value columns; the head's sum of squares meets in the cluster.
// One operand of every product is exact (q, k or v); the other - S, weighted values, weighted scores - enters as the sum of two
// BF16 numbers.  The products of states and outputs are tcgen05's.  Every wait is bounded; on expiry the status word is raised, the
// roles drain, tensor memory is freed and the CTA returns.
#include "../gemm_stream.cuh"
#include "mlstm.cuh"
#include "tile_common.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace b200
{

constexpr unsigned int MC_L = 128, MC_COLS = 64, MC_MAX_DIM = 256, MC_MAX_CLUSTER = 8;
constexpr int MC_BLOCK = 64 * 128, MC_ROWS = 2 * MC_BLOCK;    // 64 rows x 64 elements; the 128 tokens' block of 64 elements

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

// ---- states ----------------------------------------------------------------------------------------
constexpr int MS_ROLES = 32 * 14;
constexpr uint32_t MS_TMEM = 128;    // 64 columns for each 128 rows of S
// header, k twice, v, weighted values (high, low), 32 rows of S per warp on their way out
__host__ __device__ constexpr int mc_states_smem(int dp) { return 1024 + 2 * (dp / 64) * MC_ROWS + MC_ROWS + 2 * MC_ROWS + 8 * 32 * 128 + 1024; }

// grid (column blocks of 64 and one for n, heads, entries).  A TMA lane fetches k and v of the chunks; four warps weight the values, a
// token per thread; eight warps own the rows of S, one per thread: between the chunks they take S out of tensor memory, store it
// for the second kernel and put it back scaled; the MMA lane adds k^T (weighted v) onto it.  The block of n has ones for its
// values' first column.
__global__ void __launch_bounds__(MS_ROLES, 1) mlstm_states_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ MlstmParams p,
    unsigned int* status)
{
    extern __shared__ unsigned char ms_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(ms_raw) + 1023) & ~(uintptr_t)1023);
    const unsigned int dp = mc_dp(p.dim), vp = mc_vp(p.vdim), blocks = dp / 64;
    uint64_t* k_full = reinterpret_cast<uint64_t*>(smem);
    uint64_t *k_empty = k_full + 2, *w_full = k_full + 4, *v_full = k_full + 5, *v_empty = k_full + 6, *s_ready = k_full + 7, *s_done = k_full + 8;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(k_full + 9);
    volatile unsigned int* abort_flag = reinterpret_cast<volatile unsigned int*>(tmem_slot + 1);
    unsigned char* ks = smem + 1024;
    unsigned char* vs = ks + 2 * blocks * MC_ROWS;
    unsigned char* ws = vs + MC_ROWS;    // high, low
    unsigned char* out_rows = ws + 2 * MC_ROWS;

    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool is_n = blockIdx.x == gridDim.x - 1;
    const unsigned int c0 = is_n ? 0u : blockIdx.x * MC_COLS, h = blockIdx.y, e = p.e0 + blockIdx.z;
    if (tid == 0)
    {
        for (int i = 0; i < 9; i++) { mbar_init(k_full + i, i == 4 || i == 6 ? 4 : (i == 7 ? 8 : 1)); }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) { tmem_alloc(tmem_slot, MS_TMEM); }
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], chunks = (n + MC_L - 1) / MC_L;
    const bool fresh = p.pos[e] == 0;
    const ChunkRecord first = mc_record_of(p, e, 0, h);
    // of chunk c: its largest a and its last F
    auto end_of = [&](unsigned int c) { return *reinterpret_cast<const float2*>(first.top + (size_t)c * p.heads * mc_record(p.dim)); };
    float* st = mlstm_state_of(p, e, h);
    const unsigned int v_ld = mlstm_v_ld(p.vdim);
    float* st_n = st + (size_t)p.dim * v_ld;
    const float m_start = fresh ? 0.f : st_n[mlstm_n_ld(p.dim)];
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    auto give_up = [&](unsigned int role, unsigned int step) {
        note_timeout(status, WAIT_MLSTM_STATES, role, step);
        *abort_flag = 1;
    };
    auto wait = [&](uint64_t* bar, unsigned int parity) { return *abort_flag == 0 && mbar_wait_bounded(bar, parity & 1u); };

    if (warp == 0)
    {
        if (lane == 0)
        {
            const int xk = (int)(p.k_off + h * p.dim), xv = (int)(p.v_off + h * p.vdim + c0);
            unsigned int k_issued = 0, v_issued = 0;
            bool ok = true;
            for (unsigned int c = 0; c < chunks && ok; c++)
            {
                const unsigned int s = c & 1u;
                const int y = (int)(start + c * MC_L);
                if (c >= 2 && !wait(k_empty + s, (c >> 1) - 1)) { ok = false; break; }
                mbar_expect_tx(k_full + s, blocks * MC_ROWS);
                for (unsigned int r = 0; r < 2; r++)    // 64 tokens by 64 tokens
                {
                    for (unsigned int b = 0; b < blocks; b++)
                    {
                        tma_load_2d(ks + ((s * 2 + r) * blocks + b) * MC_BLOCK, &tmX, xk + (int)b * 64, y + (int)r * 64, k_full + s);
                    }
                }
                mbar_arrive(k_full + s);
                k_issued++;
                if (is_n) { continue; }
                if (c >= 1 && !wait(v_empty, c - 1)) { ok = false; break; }
                mbar_expect_tx(v_full, MC_ROWS);
                for (unsigned int r = 0; r < 2; r++) { tma_load_2d(vs + r * MC_BLOCK, &tmX, xv, y + (int)r * 64, v_full); }
                mbar_arrive(v_full);
                v_issued++;
            }
            if (!ok)
            {
                give_up(0, k_issued);
                // wait (bounded) for the copies in flight before the CTA may leave
                auto drain = [&](uint64_t* bar, unsigned int parity) {
                    const unsigned long long t0 = global_timer_ns();
                    while (!mbar_try_wait(bar, parity & 1u) && global_timer_ns() - t0 < 100000ull) {}
                };
                for (unsigned int i = k_issued > 2 ? k_issued - 2 : 0; i < k_issued; i++) { drain(k_full + (i & 1u), i >> 1); }
                if (v_issued != 0) { drain(v_full, v_issued - 1); }
            }
        }
    }
    else if (warp == 1)
    {
        const uint32_t k_addr = smem_u32(ks);
        const uint64_t w_desc = umma_desc_mnmajor_sw128(smem_u32(ws));
        const uint32_t idesc = umma_idesc_bf16(128, MC_COLS) | (1u << 15) | (1u << 16);    // both operands lie with their k outermost
        bool ok = true;
        unsigned int c = 0;
        for (; c < chunks && ok; c++)
        {
            const unsigned int s = c & 1u;
            ok = wait(k_full + s, c >> 1) && wait(w_full, c) && wait(s_ready, c);
            if (!ok) { break; }
            tc_fence_after();
            if (elect_one())
            {
                for (unsigned int mb = 0; mb < (dp + 127) / 128; mb++)
                {
                    const uint64_t a = umma_desc_mnmajor_sw128(k_addr + (s * 2 * blocks + mb * 2) * MC_BLOCK), later = a + (blocks * MC_BLOCK >> 4);
#pragma unroll
                    for (unsigned int part = 0; part < 2; part++)
                    {
#pragma unroll
                        for (unsigned int k = 0; k < MC_L / 16; k++)
                        {
                            umma_bf16(tmem + mb * MC_COLS, (k < 4 ? a : later) + ((k % 4) * 2048 >> 4),
                                w_desc + (part * MC_ROWS + (k / 4) * MC_BLOCK + (k % 4) * 2048 >> 4), idesc, 1u);
                        }
                    }
                }
                umma_commit(k_empty + s);
                umma_commit(s_done);
            }
            __syncwarp();
        }
        if (!ok)
        {
            if (lane == 0) { give_up(1, c); }
            if (elect_one()) { umma_commit(s_done); }    // completes once the MMAs in flight have stopped reading shared memory
            __syncwarp();
        }
    }
    else if (warp < 10)
    {
        const unsigned int quarter = warp & 3u, mb = (warp - 2) >> 2, d = mb * 128 + quarter * 32 + lane;
        const uint32_t mine = tmem + ((quarter * 32u) << 16) + mb * MC_COLS;
        const bool some = mb * 128 + quarter * 32 < dp;    // does the warp have rows
        float m = m_start;
        bool ok = true;
        uint32_t S[MC_COLS];
#pragma unroll
        for (int j = 0; j < (int)MC_COLS; j++) { S[j] = 0u; }
        if (!fresh && d < p.dim)
        {
            if (is_n) { S[0] = __float_as_uint(st_n[d]); }
            else
            {
#pragma unroll
                for (int j = 0; j < (int)MC_COLS; j += 4)
                {
                    if (c0 + j < p.vdim)
                    {
                        const uint4 u = *reinterpret_cast<const uint4*>(st + (size_t)d * v_ld + c0 + j);
                        S[j] = u.x;
                        S[j + 1] = u.y;
                        S[j + 2] = u.z;
                        S[j + 3] = u.w;
                    }
                }
            }
        }
        float2 end = end_of(0);
        for (unsigned int c = 0; c < chunks; c++)
        {
            const float top = fmaxf(m, end.x), keep = expf(m - top), m_before = m;
            m = end.y + top;
            if (c + 1 < chunks) { end = end_of(c + 1); }
            if (c > 0)
            {
                ok = __all_sync(0xFFFFFFFFu, wait(s_done, c - 1));
                if (!ok) { break; }
                tc_fence_after();
                if (some)
                {
                    tmem_ld_32x32(mine, *reinterpret_cast<uint32_t(*)[32]>(S));
                    tmem_ld_32x32(mine + 32, *reinterpret_cast<uint32_t(*)[32]>(S + 32));
                    tmem_ld_wait();
                }
            }
            if (some)
            {
#pragma unroll
                for (int j = 0; j < (int)MC_COLS; j += 16)
                {
                    uint32_t scaled[16];
#pragma unroll
                    for (int i = 0; i < 16; i++) { scaled[i] = __float_as_uint(__uint_as_float(S[j + i]) * keep); }
                    tmem_st_32x16(mine + j, scaled);
                }
                tmem_st_wait();
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) { mbar_arrive(s_ready); }
            // the state ahead of the chunk, while the products run
            if (some && (is_n || !fresh || c > 0))
            {
                if (is_n)
                {
                    float* out = first.n + (size_t)c * p.heads * mc_record(p.dim);
                    out[d] = __uint_as_float(S[0]);
                    if (d == 0) { out[dp] = m_before; }
                }
                else
                {
                    // through shared memory, so that a store covers whole rows
                    __nv_bfloat16* out = first.S + (size_t)c * p.heads * 2 * mc_matrix(p.dim, p.vdim) + (size_t)(d - lane) * vp + c0;
                    unsigned char* stage = out_rows + (warp - 2) * 32 * 128;
#pragma unroll 1
                    for (int part = 0; part < 2; part++)
                    {
                        __syncwarp();
#pragma unroll
                        for (int q = 0; q < 8; q++)
                        {
                            uint32_t y[4];
#pragma unroll
                            for (int i = 0; i < 4; i++)
                            {
                                const float a = __uint_as_float(S[q * 8 + 2 * i]), b = __uint_as_float(S[q * 8 + 2 * i + 1]);
                                y[i] = pack_bf16x2(a, b);
                                if (part == 1) { y[i] = pack_bf16x2(a - __uint_as_float(y[i] << 16), b - __uint_as_float(y[i] & 0xFFFF0000u)); }
                            }
                            *reinterpret_cast<uint4*>(stage + lane * 128 + ((q ^ (lane & 7u)) * 16)) = make_uint4(y[0], y[1], y[2], y[3]);
                        }
                        __syncwarp();
#pragma unroll
                        for (unsigned int i = 0; i < 8; i++)
                        {
                            const unsigned int r = i * 4 + lane / 8, q = lane % 8;
                            *reinterpret_cast<uint4*>(out + (size_t)(part * dp + r) * vp + q * 8) =
                                *reinterpret_cast<const uint4*>(stage + r * 128 + ((q ^ (r & 7u)) * 16));
                        }
                    }
                }
            }
        }
        ok = ok && __all_sync(0xFFFFFFFFu, wait(s_done, chunks - 1));
        if (ok)
        {
            tc_fence_after();
            if (some)
            {
                tmem_ld_32x32(mine, *reinterpret_cast<uint32_t(*)[32]>(S));
                tmem_ld_32x32(mine + 32, *reinterpret_cast<uint32_t(*)[32]>(S + 32));
                tmem_ld_wait();
            }
            if (is_n)
            {
                // other column blocks may still have to read the old m: the last kernel puts the new n and m in place
                float* out = first.last + (size_t)(chunks - 1) * p.heads * mc_record(p.dim);
                if (d < dp) { out[d] = __uint_as_float(S[0]); }
                if (d == 0) { out[dp] = m; }
            }
            else if (d < p.dim)
            {
#pragma unroll
                for (int j = 0; j < (int)MC_COLS; j += 4)
                {
                    if (c0 + j < p.vdim) { *reinterpret_cast<uint4*>(st + (size_t)d * v_ld + c0 + j) = make_uint4(S[j], S[j + 1], S[j + 2], S[j + 3]); }
                }
            }
        }
        else if (lane == 0) { give_up(2 + quarter, mb); }
    }
    else
    {
        const unsigned int t = tid - 320;    // token of the chunk
        float m = m_start;
        bool ok = true;
        float2 end = end_of(0);
        float a = first.a[t];
        unsigned int c = 0;
        for (; c < chunks; c++)
        {
            const float top = fmaxf(m, end.x), w = expf(a - top);
            m = end.y + top;
            if (c + 1 < chunks)
            {
                end = end_of(c + 1);
                a = first.a[(size_t)(c + 1) * p.heads * mc_record(p.dim) + t];
            }
            ok = (is_n || wait(v_full, c)) && (c == 0 || wait(s_done, c - 1));    // the products have read the weighted values before
            ok = __all_sync(0xFFFFFFFFu, ok);
            if (!ok) { break; }
            const unsigned char* src = vs + t * 128;
            unsigned char* dst = ws + t * 128;
#pragma unroll
            for (unsigned int q = 0; q < 8; q++)
            {
                const unsigned int at = (q ^ (t & 7u)) * 16;
                float f[8];
                if (is_n)
                {
#pragma unroll
                    for (int i = 0; i < 8; i++) { f[i] = q == 0 && i == 0 ? w : 0.f; }
                }
                else
                {
                    const uint4 u = *reinterpret_cast<const uint4*>(src + at);
                    const uint32_t x[4] = { u.x, u.y, u.z, u.w };
#pragma unroll
                    for (int i = 0; i < 4; i++)
                    {
                        f[2 * i] = w * __uint_as_float(x[i] << 16);
                        f[2 * i + 1] = w * __uint_as_float(x[i] & 0xFFFF0000u);
                    }
                }
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int i = 0; i < 4; i++)
                {
                    hi[i] = pack_bf16x2(f[2 * i], f[2 * i + 1]);
                    lo[i] = pack_bf16x2(f[2 * i] - __uint_as_float(hi[i] << 16), f[2 * i + 1] - __uint_as_float(hi[i] & 0xFFFF0000u));
                }
                *reinterpret_cast<uint4*>(dst + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *reinterpret_cast<uint4*>(dst + MC_ROWS + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
            fence_proxy_async();
            __syncwarp();
            if (lane == 0)
            {
                mbar_arrive(w_full);
                if (!is_n) { mbar_arrive(v_empty); }
            }
        }
        if (!ok && lane == 0) { give_up(6, c); }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) { tmem_dealloc(tmem, MS_TMEM); }
}

// ---- outputs ---------------------------------------------------------------------------------------
constexpr int MO_THREADS = 32 * 10;
constexpr uint32_t MO_O = 128, MO_TMEM = 256;    // columns: scores, in their place weighted scores (64 keys: 32 high, 32 low), then the output
// a block of 64 elements: q, k, and 64 rows of S (high, low)
__host__ __device__ constexpr int mo_stage(int vb) { return 2 * MC_ROWS + 2 * (vb / 64) * MC_BLOCK; }
__host__ __device__ constexpr int mo_smem(int vb) { return 1024 + mo_stage(vb) + (vb / 64) * MC_ROWS + 1024; }

// grid (column blocks of VB = the cluster, heads, entries x chunks), two CTAs per SM.  A TMA lane fetches v, then q, k and S in blocks of
// 64 elements; the MMA lane adds up q k^T and q S over the blocks and, once eight warps (half a row of scores per thread) have weighted
// the scores and scaled what S gives, (weighted scores) v on top.  The results leave through shared memory, so that gates and
// outputs are read and written in whole rows.
template <int VB>
__global__ void __launch_bounds__(MO_THREADS, 2) mlstm_outputs_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ CUtensorMap tmS,
    const __grid_constant__ MlstmParams p, const unsigned int max_chunks, unsigned int* status)
{
    extern __shared__ unsigned char mo_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(mo_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ float F[MC_L], a[MC_L], M[MC_L], maxima[MC_L / 32], sq[2][MC_L], nq[2][MC_L], peers[MC_MAX_CLUSTER][MC_L];
    __shared__ __align__(16) float n0[MC_MAX_DIM];
    constexpr int HB = VB / 2;
    const unsigned int dp = mc_dp(p.dim), blocks = dp / 64;
    uint64_t* full = reinterpret_cast<uint64_t*>(smem);
    uint64_t *empty = full + 1, *v_full = full + 2, *s_full = full + 3, *p_ready = full + 4, *o_full = full + 5;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(full + 6);
    volatile unsigned int* abort_flag = reinterpret_cast<volatile unsigned int*>(tmem_slot + 1);
    unsigned char* qs = smem + 1024;
    unsigned char* ks = qs + MC_ROWS;
    unsigned char* ss = ks + MC_ROWS;
    unsigned char* vs = qs + mo_stage(VB);

    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const unsigned int rank = blockIdx.x, h = blockIdx.y, e = p.e0 + blockIdx.z / max_chunks, c = blockIdx.z % max_chunks, c0 = rank * VB;
    if (tid == 0)
    {
        for (int i = 0; i < 6; i++) { mbar_init(full + i, i == 4 ? 8 : 1); }
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
    const unsigned int steps = p.dim / 16;
    auto load_block = [&](unsigned int b) {
        const int y = (int)first, xq = (int)(h * p.dim + b * 64), xk = (int)(p.k_off + h * p.dim + b * 64);
        mbar_expect_tx(full, fresh ? 2 * MC_ROWS : mo_stage(VB));
        for (int r = 0; r < 2; r++)
        {
            tma_load_2d(qs + r * MC_BLOCK, &tmX, xq, y + r * 64, full);
            tma_load_2d(ks + r * MC_BLOCK, &tmX, xk, y + r * 64, full);
        }
        if (!fresh)
        {
            for (int part = 0; part < 2; part++)
            {
                for (int j = 0; j < VB / 64; j++)
                {
                    tma_load_2d(ss + (part * (VB / 64) + j) * MC_BLOCK, &tmS, (int)c0 + j * 64, (int)((rec.at * 2 + part) * dp + b * 64), full);
                }
            }
        }
        mbar_arrive(full);
    };
    if (tid == 0)
    {
        load_block(0);
        mbar_expect_tx(v_full, (VB / 64) * MC_ROWS);
        for (int r = 0; r < 2; r++)    // 64 rows by 64 rows
        {
            for (int j = 0; j < VB / 64; j++)
            {
                tma_load_2d(vs + (r * (VB / 64) + j) * MC_BLOCK, &tmX, (int)(p.v_off + h * p.vdim + c0) + j * 64, (int)first + r * 64, v_full);
            }
        }
        mbar_arrive(v_full);
    }
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
        note_timeout(status, WAIT_MLSTM_OUTPUTS, role, step);
        *abort_flag = 1;
    };
    auto wait = [&](uint64_t* bar, unsigned int parity) { return *abort_flag == 0 && mbar_wait_bounded(bar, parity & 1u); };
    const unsigned int quarter = warp & 3u, half = warp >= 2 ? (warp - 2u) >> 2 : 0u, t = quarter * 32 + lane;    // row of an epilogue thread
    const uint32_t lanes = tmem + ((quarter * 32u) << 16);
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg + (size_t)first * p.ld;
    float inv = 0.f;
    bool good = false;

    if (warp == 0)
    {
        if (lane == 0)
        {
            unsigned int b = 1;
            bool ok = true;
            for (; b < blocks && ok; b++)
            {
                ok = wait(empty, b - 1);
                if (ok) { load_block(b); }
                else { break; }
            }
            if (!ok)
            {
                give_up(0, b);
                // wait (bounded) for the copies in flight before the CTA may leave
                auto drain = [&](uint64_t* bar, unsigned int parity) {
                    const unsigned long long t0 = global_timer_ns();
                    while (!mbar_try_wait(bar, parity & 1u) && global_timer_ns() - t0 < 100000ull) {}
                };
                drain(v_full, 0);
                drain(full, b - 1);
            }
        }
    }
    else if (warp == 1)
    {
        const uint64_t q_desc = umma_desc_kmajor_sw128(smem_u32(qs)), k_desc = umma_desc_kmajor_sw128(smem_u32(ks)),
                       s_desc = umma_desc_mnmajor_sw128(smem_u32(ss)), v_desc = umma_desc_mnmajor_sw128(smem_u32(vs));
        const uint32_t idesc_s = umma_idesc_bf16(MC_L, MC_L), idesc_o = umma_idesc_bf16(MC_L, VB) | (1u << 16);    // B is MN-major
        bool ok = true;
        unsigned int b = 0;
        for (; b < blocks && ok; b++)
        {
            ok = wait(full, b);
            if (!ok) { break; }
            tc_fence_after();
            if (elect_one())
            {
#pragma unroll
                for (unsigned int k = 0; k < 4; k++)
                {
                    if (b * 4 + k < steps) { umma_bf16(tmem, q_desc + k * 2, k_desc + k * 2, idesc_s, (b | k) != 0 ? 1u : 0u); }
                }
#pragma unroll
                for (unsigned int part = 0; part < 2; part++)
                {
#pragma unroll
                    for (unsigned int k = 0; k < 4; k++)
                    {
                        if (!fresh && b * 4 + k < steps)
                        {
                            umma_bf16(tmem + MO_O, q_desc + k * 2, s_desc + (part * (VB / 64) * MC_BLOCK + k * 2048 >> 4), idesc_o, (b | part | k) != 0 ? 1u : 0u);
                        }
                    }
                }
                if (b + 1 < blocks) { umma_commit(empty); }
                else { umma_commit(s_full); }
            }
            __syncwarp();
        }
        if (ok) { ok = wait(v_full, 0) && wait(p_ready, 0); }
        if (ok)
        {
            tc_fence_after();
            if (elect_one())
            {
#pragma unroll
                for (unsigned int part = 0; part < 2; part++)
                {
#pragma unroll
                    for (unsigned int k = 0; k < MC_L / 16; k++)
                    {
                        umma_bf16_ts(tmem + MO_O, tmem + (k / 4) * 64 + part * 32 + (k % 4) * 8,
                            v_desc + ((k / 4) * (VB / 64) * MC_BLOCK + (k % 4) * 2048 >> 4), idesc_o, !fresh || (part | k) != 0 ? 1u : 0u);
                    }
                }
                umma_commit(o_full);
            }
            __syncwarp();
        }
        else
        {
            if (lane == 0) { give_up(1, b); }
            if (elect_one()) { umma_commit(o_full); }    // completes once the MMAs in flight have stopped reading shared memory
            __syncwarp();
        }
    }
    else
    {
        const float mt = M[t], mt2 = mt * 1.44269504088896341f, carry = p.q_scale * expf(m0 - mt);
        float sum = 0.f;
        if (!fresh && t < live)    // n0 . q over half of the eights
        {
            const __nv_bfloat16* q = x + (size_t)t * p.ld + h * p.dim;
#pragma unroll 4
            for (unsigned int d = half * 8; d < p.dim; d += 16)
            {
                const uint4 u = *reinterpret_cast<const uint4*>(q + d);
                const float4 g0 = *reinterpret_cast<const float4*>(n0 + d), g1 = *reinterpret_cast<const float4*>(n0 + d + 4);
                sum = fmaf(__uint_as_float(u.x << 16), g0.x, fmaf(__uint_as_float(u.x & 0xFFFF0000u), g0.y, sum));
                sum = fmaf(__uint_as_float(u.y << 16), g0.z, fmaf(__uint_as_float(u.y & 0xFFFF0000u), g0.w, sum));
                sum = fmaf(__uint_as_float(u.z << 16), g1.x, fmaf(__uint_as_float(u.z & 0xFFFF0000u), g1.y, sum));
                sum = fmaf(__uint_as_float(u.w << 16), g1.z, fmaf(__uint_as_float(u.w & 0xFFFF0000u), g1.w, sum));
            }
            sum *= carry;
        }
        good = __all_sync(0xFFFFFFFFu, wait(s_full, 0));
        if (good)
        {
            tc_fence_after();
            // this half's 64 keys, their weights in the place of their scores; none where the rows of the warp end before
            uint32_t hi[32], lo[32];
#pragma unroll
            for (int q = 0; q < 2; q++)
            {
                const unsigned int s0 = half * 64 + q * 32;
                uint32_t z[32];
#pragma unroll
                for (int j = 0; j < 16; j++) { hi[q * 16 + j] = lo[q * 16 + j] = 0u; }
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
                        const uint32_t u = pack_bf16x2(w[0], w[1]);
                        hi[q * 16 + j] = u;
                        lo[q * 16 + j] = pack_bf16x2(w[0] - __uint_as_float(u << 16), w[1] - __uint_as_float(u & 0xFFFF0000u));
                    }
                }
            }
#pragma unroll
            for (int q = 0; q < 2; q++)
            {
                tmem_st_32x16(lanes + half * 64 + q * 16, hi + q * 16);
                tmem_st_32x16(lanes + half * 64 + 32 + q * 16, lo + q * 16);
            }
            if (!fresh)
            {
#pragma unroll
                for (int d = 0; d < HB; d += 32)
                {
                    uint32_t o[32];
                    tmem_ld_32x32(lanes + MO_O + half * HB + d, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 32; j++) { o[j] = __float_as_uint(__uint_as_float(o[j]) * carry); }
                    tmem_st_32x16(lanes + MO_O + half * HB + d, o);
                    tmem_st_32x16(lanes + MO_O + half * HB + d + 16, o + 16);
                }
            }
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) { mbar_arrive(p_ready); }
        }
        nq[half][t] = sum;
        bar_sync_named(1, 256);
        inv = 1.0f / (fmaxf(fabsf(nq[0][t] + nq[1][t]), expf(-(F[t] + mt))) + 1e-6f);
        good = __all_sync(0xFFFFFFFFu, good && wait(o_full, 0)) && *abort_flag == 0;
        good = __all_sync(0xFFFFFFFFu, good);
        float s = 0.f;
        if (good)
        {
            tc_fence_after();
#pragma unroll
            for (int d = 0; d < HB; d += 32)
            {
                uint32_t o[32];
                tmem_ld_32x32(lanes + MO_O + half * HB + d, o);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; j++)
                {
                    const float v = __uint_as_float(o[j]) * inv;
                    if (c0 + half * HB + d + j < p.vdim) { s = fmaf(v, v, s); }
                }
            }
        }
        else if (lane == 0) { give_up(2 + quarter, half); }
        sq[half][t] = s;
    }
    __syncthreads();
    cg::cluster_group cluster = cg::this_cluster();
    const unsigned int ranks = cluster.num_blocks();
    for (unsigned int j = tid; j < ranks * MC_L; j += MO_THREADS)
    {
        const unsigned int r = j % MC_L;
        cluster.map_shared_rank(&peers[0][0], j / MC_L)[rank * MC_L + r] = sq[0][r] + sq[1][r];
    }
    cluster.sync();
    if (warp >= 2)
    {
        float* rows = reinterpret_cast<float*>(qs);    // [128][VB], sixteen bytes at a time in an order of the row's own
        if (good)
        {
            float s = 0.f;
            for (unsigned int r = 0; r < ranks; r++) { s += peers[r][t]; }
            const float unit = inv / sqrtf(s / (float)p.vdim + p.eps);
#pragma unroll
            for (int d = 0; d < HB; d += 32)
            {
                uint32_t o[32];
                tmem_ld_32x32(lanes + MO_O + half * HB + d, o);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; j += 4)
                {
                    const unsigned int q = (half * HB + d + j) / 4;
                    *reinterpret_cast<float4*>(rows + t * VB + ((q ^ (t & 15u)) * 4)) = make_float4(__uint_as_float(o[j]) * unit, __uint_as_float(o[j + 1]) * unit,
                        __uint_as_float(o[j + 2]) * unit, __uint_as_float(o[j + 3]) * unit);
                }
            }
        }
        const bool all_good = *abort_flag == 0;
        bar_sync_named(1, 256);
        const __nv_bfloat16* gate = x + p.g_off + h * p.vdim + c0;
        __nv_bfloat16* out = (__nv_bfloat16*)p.out + (size_t)first * p.ldo + h * p.vdim + c0;
        const float* w = p.norm + h * p.vdim + c0;
        constexpr unsigned int PER = VB / 8;
#pragma unroll 4
        for (unsigned int j = tid - 64; j < MC_L * PER; j += 256)
        {
            const unsigned int r = j / PER, col = j % PER * 8;
            if (r >= live || c0 + col >= p.vdim || !all_good) { continue; }
            const uint4 u = *reinterpret_cast<const uint4*>(gate + (size_t)r * p.ld + col);
            const float4 v0 = *reinterpret_cast<const float4*>(rows + r * VB + ((col / 4 ^ (r & 15u)) * 4));
            const float4 v1 = *reinterpret_cast<const float4*>(rows + r * VB + (((col / 4 + 1) ^ (r & 15u)) * 4));
            const float4 w0 = *reinterpret_cast<const float4*>(w + col), w1 = *reinterpret_cast<const float4*>(w + col + 4);
            const float v[8] = { v0.x * w0.x, v0.y * w0.y, v0.z * w0.z, v0.w * w0.w, v1.x * w1.x, v1.y * w1.y, v1.z * w1.z, v1.w * w1.w };
            const uint32_t g[4] = { u.x, u.y, u.z, u.w };
            uint32_t y[4];
#pragma unroll
            for (int k = 0; k < 4; k++)
            {
                y[k] = pack_bf16x2(v[2 * k] * sigmoid_f32(__uint_as_float(g[k] << 16)), v[2 * k + 1] * sigmoid_f32(__uint_as_float(g[k] & 0xFFFF0000u)));
            }
            *reinterpret_cast<uint4*>(out + (size_t)r * p.ldo + col) = make_uint4(y[0], y[1], y[2], y[3]);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) { tmem_dealloc(tmem, MO_TMEM); }
    if (rank == 0 && (c + 1) * MC_L >= n)
    {
        float* st_n = mlstm_state_of(p, e, h) + (size_t)p.dim * mlstm_v_ld(p.vdim);
        for (unsigned int d = tid; d < p.dim; d += MO_THREADS) { st_n[d] = rec.last[d]; }
        if (tid == 0) { st_n[mlstm_n_ld(p.dim)] = rec.last[dp]; }
    }
}

template <int VB>
static int run_outputs(const MlstmParams& p, const CUtensorMap& tx, unsigned int* status, cudaStream_t stream, bool pdl)
{
    const unsigned int ranks = (p.vdim + VB - 1) / VB, chunks = (p.max_n + MC_L - 1) / MC_L, dp = mc_dp(p.dim), vp = mc_vp(p.vdim);
    CUtensorMap ts;
    if (!make_map_2d(&ts, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.work, vp, (unsigned long long)mc_slots(p.tokens, p.entries) * p.heads * 2 * dp,
            (unsigned long long)vp * 2, 64, 64, true))
    {
        return -1;
    }
    return launch_cluster("mlstm_outputs", mlstm_outputs_kernel<VB>, dim3(ranks, p.heads, p.entries * chunks), dim3(MO_THREADS), (size_t)mo_smem(VB), ranks,
        stream, pdl, tx, ts, p, chunks, status);
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
    unsigned int* status = decoder_status_word();
    if (!status) { return 1; }
    CUtensorMap tx;
    if (!make_map_2d(&tx, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.qkvg, p.ld, (unsigned long long)p.t0 + p.tokens, (unsigned long long)p.ld * 2, 64, 64, true))
    {
        return -1;
    }
    int rc = launch_kernel("mlstm_gates", mlstm_gates_kernel, dim3(chunks, p.heads, entries), dim3(MC_L), 0, stream, pdl, p);
    if (rc) { return rc; }
    rc = launch_kernel("mlstm_states", mlstm_states_kernel, dim3(mc_vp(p.vdim) / MC_COLS + 1, p.heads, entries), dim3(MS_ROLES),
        (size_t)mc_states_smem((int)mc_dp(p.dim)), stream, pdl, tx, p, status);
    if (rc) { return rc; }
    return p.vdim <= 64 ? run_outputs<64>(p, tx, status, stream, pdl) : run_outputs<128>(p, tx, status, stream, pdl);
}

}    // namespace b200
