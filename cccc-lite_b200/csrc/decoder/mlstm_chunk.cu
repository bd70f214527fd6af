// The mLSTM recurrence over prompts, in chunks of 128 tokens on mma.sync.
//
// Inside a chunk, with F the running sum of the log forget gates, a_s = i_s - F_s and M_t = max(m_0, a_s up to t), the running
// maximum is m_t = F_t + M_t, and unrolled from the chunk's first token
//   o_t ~ e^(m_0 - M_t) S_0^T q_t + sum_{s <= t} e^(a_s - M_t) (q_t . k_s) v_s,   S_L = e^(m_0 - M_L) S_0 + sum_s e^(a_s - M_L) k_s v_s^T,
// no exponent above zero.  Three kernels:
//   gates  : F and a of every chunk.
//   states : a CTA per 32 value columns of a head walks an entry's chunks, its columns of S as float accumulators in registers;
//            it leaves the state ahead of every chunk in scratch memory.
//   outputs: a cluster per (chunk, head), a CTA per 64 or 128 value columns; the head's sum of squares meets in the cluster.
// One operand of every product is exact (q, k or v); the other - S, weighted values, weighted scores - enters as the sum of two
// BF16 numbers.
#include "attention_mma.cuh"
#include "mlstm.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace b200
{

constexpr unsigned int MC_L = 128, MC_WARPS = 16, MC_THREADS = 32 * MC_WARPS, MC_COLS = 32, MC_SLICE = 32, MC_MAX_DIM = 256, MC_MAX_CLUSTER = 8;

__host__ __device__ __forceinline__ unsigned int mc_dp(unsigned int dim) { return dim <= 64 ? 64 : (dim <= 128 ? 128 : 256); }
__host__ __device__ __forceinline__ unsigned int mc_vp(unsigned int vdim) { return (vdim + MC_COLS - 1) / MC_COLS * MC_COLS; }
// Scratch of a (chunk, head): S high [dp][vp], S low, then n and m ahead of the chunk, n and m behind the entry's last chunk, F, a,
// the largest a and the last F.
__host__ __device__ __forceinline__ size_t mc_record(unsigned int dim, unsigned int vdim)
{
    return (size_t)mc_dp(dim) * mc_vp(vdim) + 2 * (mc_dp(dim) + 4) + 2 * MC_L + 4;
}
struct ChunkRecord
{
    __nv_bfloat16* S;
    float *n, *last, *F, *a, *top;    // m behind n, the last m behind last
};
__device__ __forceinline__ ChunkRecord mc_record_of(const MlstmParams& p, unsigned int e, unsigned int chunk, unsigned int head)
{
    const unsigned int at = ((unsigned int)p.start[e] - p.t0) / MC_L + (e - p.e0) + chunk;    // entries' chunks one behind the other
    const unsigned int dp = mc_dp(p.dim);
    float* r = p.work + ((size_t)at * p.heads + head) * mc_record(p.dim, p.vdim);
    ChunkRecord c;
    c.S = reinterpret_cast<__nv_bfloat16*>(r);
    c.n = r + (size_t)dp * mc_vp(p.vdim);
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
    __shared__ __align__(16) __nv_bfloat16 hi[MC_L * (MC_COLS + 8)], lo[MC_L * (MC_COLS + 8)];
    const unsigned int vp = mc_vp(p.vdim);
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, gc = (lane & 3) * 2, d0 = warp * 16;
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
    float m = fresh ? 0.f : st_n[mlstm_n_ld(p.dim)], nn = !fresh && tid < p.dim ? st_n[tid] : 0.f;
    ChunkRecord rec = mc_record_of(p, e, 0, h);
    float a = tid < MC_L ? rec.a[tid] : 0.f;
    float2 end = *reinterpret_cast<const float2*>(rec.top);
    for (unsigned int c = 0; c < chunks; c++)
    {
        const unsigned int live = min(MC_L, n - c * MC_L);
        fetch(c + 1);
        const float top = fmaxf(m, end.x), keep = expf(m - top);    // M at the chunk's end
        if (tid < MC_L) { w[tid] = expf(a - top); }
        if (d0 < (unsigned int)DP && (!fresh || c > 0))
        {
#pragma unroll
            for (int j = 0; j < (int)MC_COLS / 8; j++)
            {
#pragma unroll
                for (int half = 0; half < 2; half++)
                {
                    const float s0 = S[j][2 * half], s1 = S[j][2 * half + 1];
                    const uint32_t high = pack_bf16x2(s0, s1);
                    uint32_t* y = reinterpret_cast<uint32_t*>(rec.S + (size_t)(d0 + gr + 8 * half) * vp + c0 + j * 8 + gc);
                    y[0] = high;
                    y[(size_t)DP * vp / 2] = pack_bf16x2(s0 - __uint_as_float(high << 16), s1 - __uint_as_float(high & 0xFFFF0000u));
                }
            }
        }
        if (blockIdx.x == 0)
        {
            if (tid < (unsigned int)DP) { rec.n[tid] = nn; }
            if (tid == 0) { rec.n[DP] = m; }
        }
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
        if (blockIdx.x == 0 && tid < p.dim)
        {
            const __nv_bfloat16* k = reinterpret_cast<const __nv_bfloat16*>(mc_raw + (c & 1u) * KBYTES) + tid;
            float part[4] = { 0.f, 0.f, 0.f, 0.f };
#pragma unroll 4
            for (unsigned int s = 0; s < MC_L; s += 4)
            {
#pragma unroll
                for (int i = 0; i < 4; i++) { part[i] = fmaf(w[s + i], __bfloat162float(k[(s + i) * (DP + 8)]), part[i]); }
            }
            nn = keep * nn + ((part[0] + part[1]) + (part[2] + part[3]));
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
#pragma unroll 4
            for (unsigned int s0 = 0; s0 < live; s0 += 16)
            {
                uint32_t b[2][MC_COLS / 16][4], k[4];
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
        if (blockIdx.x == 0 && c + 1 == chunks)
        {
            if (tid < p.dim) { now.last[tid] = nn; }
            if (tid == 0) { now.last[DP] = m; }
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
// q, k, v; two slices of S beside them
__host__ __device__ constexpr unsigned int mc_slice_bytes(unsigned int vb) { return 2 * MC_SLICE * (vb + 8) * 2; }
__host__ __device__ constexpr unsigned int mc_outputs_smem(unsigned int dp, unsigned int vb)
{
    return 2 * MC_L * (dp + 8) * 2 + MC_L * (vb + 8) * 2 + 2 * mc_slice_bytes(vb);
}

// grid (column blocks of VB = the cluster, heads, entries x chunks); a warp owns 16 tokens and half of the columns.  The chunk's own
// tokens come first; the slices of S then also take the place of k and v.
template <int DP, int VB>
__global__ void __launch_bounds__(MC_THREADS) mlstm_outputs_kernel(const MlstmParams p, const unsigned int max_chunks)
{
    extern __shared__ __align__(16) unsigned char mc_raw[];
    __shared__ float F[MC_L], a[MC_L], M[MC_L], maxima[MC_L / 32], sq[2][MC_L], peers[MC_MAX_CLUSTER][MC_L], n0[DP];
    constexpr unsigned int VS = (VB + 8) * 2, QS = (DP + 8) * 2, SLICE = mc_slice_bytes(VB), SLICES = DP / MC_SLICE, HB = VB / 2;
    constexpr unsigned int QBYTES = MC_L * QS, VBYTES = MC_L * VS;
    constexpr unsigned int PLACES = (QBYTES + VBYTES) / SLICE;    // of slices where k and v were
    const unsigned int vp = mc_vp(p.vdim);
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, gc = (lane & 3) * 2;
    const unsigned int rank = blockIdx.x, h = blockIdx.y, e = p.e0 + blockIdx.z / max_chunks, c = blockIdx.z % max_chunks, c0 = rank * VB;
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e];
    if (c * MC_L >= n) { return; }    // the whole cluster
    const unsigned int live = min(MC_L, n - c * MC_L), first = start + c * MC_L;
    const bool fresh = p.pos[e] == 0 && c == 0;
    const ChunkRecord rec = mc_record_of(p, e, c, h);
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg + (size_t)first * p.ld;
    const uint32_t qs = smem_u32(mc_raw), ks = qs + QBYTES, vs = ks + QBYTES, ss = vs + VBYTES;
    auto place = [&](unsigned int i) { return i < 2 ? ss + i * SLICE : (i - 2 < PLACES ? ks + (i - 2) * SLICE : ss + (i - 2 - PLACES) * SLICE); };
    auto fetch_slice = [&](unsigned int i) {
        if (i < SLICES && !fresh)
        {
            constexpr unsigned int PER = VB / 8, ALL = 2 * MC_SLICE * PER;
            const uint32_t to = place(i);
            for (unsigned int j = tid; j < ALL; j += MC_THREADS)
            {
                const unsigned int part = j / (MC_SLICE * PER), r = j / PER % MC_SLICE, d = j % PER, col = c0 + d * 8;
                const bool ok = col < vp;
                cp_async16(to + part * (SLICE / 2) + r * VS + d * 16, rec.S + (ok ? (size_t)part * DP * vp + (size_t)(i * MC_SLICE + r) * vp + col : 0), ok);
            }
        }
        cp_async_commit();
    };
    mc_fetch<DP>(qs, x + h * p.dim, p.ld, live, p.dim);
    mc_fetch<DP>(ks, x + p.k_off + h * p.dim, p.ld, live, p.dim);
    mc_fetch<VB>(vs, x + p.v_off + h * p.vdim + c0, p.ld, live, min((unsigned int)VB, p.vdim - c0));
    cp_async_commit();
    fetch_slice(0);
    fetch_slice(1);
    const float m0 = fresh ? 0.f : rec.n[DP];
    for (unsigned int d = tid; d < (unsigned int)DP; d += MC_THREADS) { n0[d] = fresh ? 0.f : rec.n[d]; }
    float t_max = -INFINITY;
    if (tid < MC_L)    // M: running maxima of a, with m0
    {
        F[tid] = rec.F[tid];
        t_max = rec.a[tid];
        a[tid] = t_max;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1)
        {
            const float y = __shfl_up_sync(0xFFFFFFFFu, t_max, o);
            if (lane >= (unsigned int)o) { t_max = fmaxf(t_max, y); }
        }
        if (lane == 31) { maxima[warp] = t_max; }
    }
    __syncthreads();
    if (tid < MC_L)
    {
        t_max = fmaxf(m0, t_max);
        for (unsigned int j = 0; j < warp; j++) { t_max = fmaxf(t_max, maxima[j]); }
        M[tid] = t_max;
    }
    cp_async_wait<2>();
    __syncthreads();
    const unsigned int r0 = (warp & 7u) * 16, ch = warp >> 3;    // tokens, half of the columns
    const uint32_t qa = qs + (r0 + (lane & 15)) * QS + (lane >> 4) * 16;
    float o[HB / 8][4], z2[HB / 8][4], nq[2] = { 0.f, 0.f }, mt[2], carry[2];
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
        mt[i] = M[r0 + gr + 8 * i];
        carry[i] = p.q_scale * expf(m0 - mt[i]);
    }
#pragma unroll
    for (int j = 0; j < (int)HB / 8; j++)
    {
#pragma unroll
        for (int i = 0; i < 4; i++) { o[j][i] = z2[j][i] = 0.f; }
    }
    {
        const uint32_t kb = ks + ((lane & 7) + ((lane >> 4) << 3)) * QS + ((lane >> 3) & 1) * 16;
        const uint32_t vb = vs + (lane & 15) * VS + (lane >> 4) * 16 + ch * HB * 2;
        for (unsigned int s0 = 0; s0 < r0 + 16; s0 += 32)
        {
            float z[4][4];
#pragma unroll
            for (int i = 0; i < 4; i++)
            {
#pragma unroll
                for (int j = 0; j < 4; j++) { z[i][j] = 0.f; }
            }
#pragma unroll 4
            for (int kk = 0; kk < DP / 16; kk++)
            {
                uint32_t q[4], b[2][4];
                ldmatrix_x4(q, qa + kk * 32);
                ldmatrix_x4(b[0], kb + s0 * QS + kk * 32);
                ldmatrix_x4(b[1], kb + (s0 + 16) * QS + kk * 32);
#pragma unroll
                for (int i = 0; i < 2; i++)
                {
                    mma_bf16_16816(z[2 * i], q[0], q[1], q[2], q[3], b[i][0], b[i][1]);
                    mma_bf16_16816(z[2 * i + 1], q[0], q[1], q[2], q[3], b[i][2], b[i][3]);
                }
            }
#pragma unroll
            for (int i = 0; i < 4; i++)
            {
#pragma unroll
                for (int j = 0; j < 4; j++)
                {
                    const unsigned int s = s0 + i * 8 + gc + (j & 1), t = r0 + gr + 8 * (j >> 1);
                    z[i][j] = s <= t ? z[i][j] * p.q_scale * expf(a[s] - mt[j >> 1]) : 0.f;
                    nq[j >> 1] += z[i][j];
                }
            }
#pragma unroll
            for (int i = 0; i < 2; i++)
            {
                uint32_t top[4], rest[4];
#pragma unroll
                for (int j = 0; j < 4; j++)
                {
                    // a0: row g, keys 0-7; a1: row g + 8, keys 0-7; a2, a3: keys 8-15
                    const float* f = &z[2 * i + (j >> 1)][(j & 1) * 2];
                    top[j] = pack_bf16x2(f[0], f[1]);
                    rest[j] = pack_bf16x2(f[0] - __uint_as_float(top[j] << 16), f[1] - __uint_as_float(top[j] & 0xFFFF0000u));
                }
#pragma unroll
                for (int j = 0; j < (int)HB / 16; j++)
                {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, vb + (s0 + i * 16) * VS + j * 32);
                    mma_bf16_16816(o[2 * j], top[0], top[1], top[2], top[3], b[0], b[1]);
                    mma_bf16_16816(o[2 * j + 1], top[0], top[1], top[2], top[3], b[2], b[3]);
                    mma_bf16_16816(o[2 * j], rest[0], rest[1], rest[2], rest[3], b[0], b[1]);
                    mma_bf16_16816(o[2 * j + 1], rest[0], rest[1], rest[2], rest[3], b[2], b[3]);
                }
            }
        }
    }
    nq[0] += __shfl_xor_sync(0xFFFFFFFFu, nq[0], 1);
    nq[1] += __shfl_xor_sync(0xFFFFFFFFu, nq[1], 1);
    nq[0] += __shfl_xor_sync(0xFFFFFFFFu, nq[0], 2);
    nq[1] += __shfl_xor_sync(0xFFFFFFFFu, nq[1], 2);
    if (!fresh)
    {
        __syncthreads();    // k and v have been read
#pragma unroll
        for (unsigned int i = 2; i < SLICES; i++)
        {
            if (i < 2 + PLACES) { fetch_slice(i); }
        }
        // n0 . q: the four lanes of a row share its elements
#pragma unroll
        for (int i = 0; i < 2; i++)
        {
            const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(mc_raw) + (size_t)(r0 + gr + 8 * i) * (DP + 8);
            float s = 0.f;
#pragma unroll 8
            for (int d = 0; d < DP; d += 8)
            {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q + d + gc)), g = *reinterpret_cast<const float2*>(n0 + d + gc);
                s = fmaf(f.x, g.x, fmaf(f.y, g.y, s));
            }
            s += __shfl_xor_sync(0xFFFFFFFFu, s, 1);
            s += __shfl_xor_sync(0xFFFFFFFFu, s, 2);
            nq[i] += carry[i] * s;
        }
        constexpr int ISSUED = (int)(SLICES < 2 + PLACES ? SLICES : 2 + PLACES);
#pragma unroll
        for (int i = 0; i < (int)SLICES; i++)
        {
            // groups behind slice i: those issued so far, and one more per slice of the second round
            constexpr int LATE = (int)SLICES - ISSUED;
            const int behind = i < ISSUED ? ISSUED - 1 - i + (i < LATE ? i : LATE) : (int)SLICES - 1 - i;
            switch (behind)
            {
            case 0: cp_async_wait<0>(); break;
            case 1: cp_async_wait<1>(); break;
            case 2: cp_async_wait<2>(); break;
            case 3: cp_async_wait<3>(); break;
            case 4: cp_async_wait<4>(); break;
            case 5: cp_async_wait<5>(); break;
            default: cp_async_wait<6>(); break;
            }
            __syncthreads();
            const uint32_t sb = place((unsigned int)i) + (lane & 15) * VS + (lane >> 4) * 16 + ch * HB * 2;
#pragma unroll
            for (int kk = 0; kk < (int)MC_SLICE / 16; kk++)
            {
                uint32_t q[4];
                ldmatrix_x4(q, qa + (i * MC_SLICE + kk * 16) * 2);
#pragma unroll
                for (int part = 0; part < 2; part++)
                {
#pragma unroll
                    for (int j = 0; j < (int)HB / 16; j++)
                    {
                        uint32_t b[4];
                        ldmatrix_x4_trans(b, sb + part * (SLICE / 2) + kk * 16 * VS + j * 32);
                        mma_bf16_16816(z2[2 * j], q[0], q[1], q[2], q[3], b[0], b[1]);
                        mma_bf16_16816(z2[2 * j + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
                    }
                }
            }
            if (i < LATE)
            {
                __syncthreads();    // the place of slice i is free
                fetch_slice((unsigned int)(ISSUED + i));
            }
        }
#pragma unroll
        for (int j = 0; j < (int)HB / 8; j++)
        {
#pragma unroll
            for (int i = 0; i < 4; i++) { o[j][i] = fmaf(carry[i >> 1], z2[j][i], o[j][i]); }
        }
    }
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
        const float inv = 1.0f / (fmaxf(fabsf(nq[i]), expf(-(F[r0 + gr + 8 * i] + mt[i]))) + 1e-6f);
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < (int)HB / 8; j++)
        {
            o[j][2 * i] *= inv;
            o[j][2 * i + 1] *= inv;
            s += o[j][2 * i] * o[j][2 * i] + o[j][2 * i + 1] * o[j][2 * i + 1];
        }
        s += __shfl_xor_sync(0xFFFFFFFFu, s, 1);
        s += __shfl_xor_sync(0xFFFFFFFFu, s, 2);
        if ((lane & 3) == 0) { sq[ch][r0 + gr + 8 * i] = s; }
    }
    __syncthreads();
    cg::cluster_group cluster = cg::this_cluster();
    const unsigned int ranks = cluster.num_blocks();
    for (unsigned int j = tid; j < ranks * MC_L; j += MC_THREADS)
    {
        const unsigned int t = j % MC_L;
        cluster.map_shared_rank(&peers[0][0], j / MC_L)[rank * MC_L + t] = sq[0][t] + sq[1][t];
    }
    cluster.sync();
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
        const unsigned int t = r0 + gr + 8 * i;
        if (t >= live) { continue; }
        float s = 0.f;
        for (unsigned int r = 0; r < ranks; r++) { s += peers[r][t]; }
        const float inv = 1.0f / sqrtf(s / (float)p.vdim + p.eps);
        const unsigned int at = h * p.vdim + c0 + ch * HB;
        const __nv_bfloat16* gate = x + (size_t)t * p.ld + p.g_off + at;
        __nv_bfloat16* out = (__nv_bfloat16*)p.out + (size_t)(first + t) * p.ldo + at;
        const float* w = p.norm + at;
#pragma unroll
        for (int j = 0; j < (int)HB / 8; j++)
        {
            const unsigned int col = j * 8 + gc;
            if (c0 + ch * HB + col < p.vdim)
            {
                const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + col));
                *reinterpret_cast<uint32_t*>(out + col) =
                    pack_bf16x2(o[j][2 * i] * inv * w[col] * sigmoid_f32(g.x), o[j][2 * i + 1] * inv * w[col + 1] * sigmoid_f32(g.y));
            }
        }
    }
    if (rank == 0 && (c + 1) * MC_L >= n)
    {
        float* st_n = mlstm_state_of(p, e, h) + (size_t)p.dim * mlstm_v_ld(p.vdim);
        for (unsigned int d = tid; d < p.dim; d += MC_THREADS) { st_n[d] = rec.last[d]; }
        if (tid == 0) { st_n[mlstm_n_ld(p.dim)] = rec.last[DP]; }
    }
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
    auto outputs = [&](auto kernel, unsigned int vb) {
        const unsigned int ranks = (p.vdim + vb - 1) / vb;
        return launch_cluster("mlstm_outputs", kernel, dim3(ranks, p.heads, entries * chunks), dim3(MC_THREADS), (size_t)mc_outputs_smem(DP, vb), ranks, stream, pdl,
            p, chunks);
    };
    return p.vdim <= 64 ? outputs(mlstm_outputs_kernel<DP, 64>, 64) : outputs(mlstm_outputs_kernel<DP, 128>, 128);
}

unsigned long long mlstm_chunk_floats(unsigned int tokens, unsigned int entries, unsigned int heads, unsigned int dim, unsigned int vdim)
{
    return (unsigned long long)(tokens / MC_L + entries) * heads * mc_record(dim, vdim);
}

bool mlstm_chunk_takes(unsigned int dim, unsigned int vdim) { return (dim % 8) == 0 && (vdim % 8) == 0 && dim <= MC_MAX_DIM && vdim <= 128 * MC_MAX_CLUSTER; }

int launch_mlstm_chunk(const MlstmParams& p, unsigned int entries, cudaStream_t stream, bool pdl)
{
    const unsigned int chunks = (p.max_n + MC_L - 1) / MC_L;
    if (!mlstm_chunk_takes(p.dim, p.vdim) || (p.ld % 8) || (p.k_off % 8) || (p.v_off % 8) || (p.g_off % 2) || (p.ldo % 2)
        || (unsigned long long)entries * chunks > 65535ull)
    {
        return -1;
    }
    if (p.dim <= 64) { return run_chunks<64>(p, entries, stream, pdl); }
    if (p.dim <= 128) { return run_chunks<128>(p, entries, stream, pdl); }
    return run_chunks<256>(p, entries, stream, pdl);
}

}    // namespace b200
