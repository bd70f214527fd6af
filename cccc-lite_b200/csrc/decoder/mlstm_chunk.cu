// The mLSTM recurrence over prompts, in chunks of 128 tokens on mma.sync.
//
// Inside a chunk, with F the running sum of the log forget gates, a_s = i_s - F_s and M_t = max(m_0, a_s up to t), the running
// maximum is m_t = F_t + M_t, and unrolled from the chunk's first token
//   o_t ~ e^(m_0 - M_t) S_0^T q_t + sum_{s <= t} e^(a_s - M_t) (q_t . k_s) v_s,   S_L = e^(m_0 - M_L) S_0 + sum_s e^(a_s - M_L) k_s v_s^T,
// no exponent above zero.  Two kernels:
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

constexpr unsigned int MC_L = 128, MC_WARPS = 8, MC_THREADS = 32 * MC_WARPS, MC_COLS = 32, MC_SLICE = 32, MC_MAX_DIM = 256, MC_MAX_CLUSTER = 8;

__host__ __device__ __forceinline__ unsigned int mc_dp(unsigned int dim) { return (dim + 31) / 32 * 32; }
__host__ __device__ __forceinline__ unsigned int mc_vp(unsigned int vdim) { return (vdim + MC_COLS - 1) / MC_COLS * MC_COLS; }
// Scratch of a (chunk, head): S high [dp][vp], S low, n [dp], m, and of an entry's last chunk the state behind it: n [dp], m.
__host__ __device__ __forceinline__ size_t mc_record(unsigned int dim, unsigned int vdim)
{
    return (size_t)mc_dp(dim) * mc_vp(vdim) + 2 * mc_dp(dim) + 8;
}
__device__ __forceinline__ float* mc_record_of(const MlstmParams& p, unsigned int e, unsigned int chunk, unsigned int head)
{
    const unsigned int at = ((unsigned int)p.start[e] - p.t0) / MC_L + (e - p.e0) + chunk;    // entries' chunks one behind the other
    return p.work + ((size_t)at * p.heads + head) * mc_record(p.dim, p.vdim);
}

// Gates of a chunk of `live` tokens from token `first` on: F (running sums) and a for every token, by all threads of the CTA.
// Tokens behind the last: F stays, a = -inf.  Returns with the arrays visible to all.
__device__ __forceinline__ void mc_gates(const MlstmParams& p, unsigned int first, unsigned int live, unsigned int head, float* F, float* a, float* sums)
{
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float in = -INFINITY, f = 0.f;
    if (tid < live) { mlstm_gates(p, first + tid, head, in, f); }
    if (tid < MC_L)
    {
#pragma unroll
        for (int o = 1; o < 32; o <<= 1)
        {
            const float x = __shfl_up_sync(0xFFFFFFFFu, f, o);
            if (lane >= (unsigned int)o) { f += x; }
        }
        if (lane == 31) { sums[warp] = f; }
    }
    __syncthreads();
    if (tid < MC_L)
    {
        for (unsigned int w = 0; w < warp; w++) { f += sums[w]; }
        F[tid] = f;
        a[tid] = tid < live ? in - f : -INFINITY;
    }
    __syncthreads();
}

// Rows [first, first + live) of a projection, `width` elements from `src` on, into padded shared rows; rows behind and columns up to
// `padded` are zero.
__device__ __forceinline__ void mc_fetch(uint32_t dst, unsigned int stride, const __nv_bfloat16* src, unsigned int ld, unsigned int live, unsigned int width,
    unsigned int padded)
{
    const unsigned int per = padded / 8;
    for (unsigned int c = threadIdx.x; c < MC_L * per; c += MC_THREADS)
    {
        const unsigned int r = c / per, d = c % per;
        const bool ok = r < live && d * 8 < width;
        cp_async16(dst + r * stride + d * 16, src + (ok ? (size_t)r * ld + d * 8 : 0), ok);
    }
}

// grid (column blocks of 32, heads, entries); RT: 16-row tiles of S per warp
template <int RT>
__global__ void __launch_bounds__(MC_THREADS) mlstm_states_kernel(const MlstmParams p)
{
    extern __shared__ __align__(16) unsigned char mc_raw[];
    constexpr unsigned int VS = (MC_COLS + 8) * 2;
    __shared__ float F[MC_L], a[MC_L], w[MC_L], sums[MC_WARPS];
    __shared__ __align__(16) __nv_bfloat16 hi[MC_L * (MC_COLS + 8)], lo[MC_L * (MC_COLS + 8)];
    const unsigned int dp = mc_dp(p.dim), vp = mc_vp(p.vdim), KS = (dp + 8) * 2;
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, gc = (lane & 3) * 2;
    const unsigned int c0 = blockIdx.x * MC_COLS, h = blockIdx.y, e = p.e0 + blockIdx.z;
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], chunks = (n + MC_L - 1) / MC_L;
    const bool fresh = p.pos[e] == 0;
    float* st = mlstm_state_of(p, e, h);
    const unsigned int v_ld = mlstm_v_ld(p.vdim);
    float* st_n = st + (size_t)p.dim * v_ld;
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg + (size_t)start * p.ld;
    const uint32_t ks = smem_u32(mc_raw), vs = ks + 2 * MC_L * KS, hs = smem_u32(hi), ls = smem_u32(lo);
    const __nv_bfloat16* v_raw = reinterpret_cast<const __nv_bfloat16*>(mc_raw + 2 * MC_L * KS);
    auto fetch = [&](unsigned int c) {
        if (c < chunks)
        {
            const unsigned int live = min(MC_L, n - c * MC_L), vw = p.vdim > c0 ? min(MC_COLS, p.vdim - c0) : 0u;
            mc_fetch(ks + (c & 1u) * MC_L * KS, KS, x + (size_t)c * MC_L * p.ld + p.k_off + h * p.dim, p.ld, live, p.dim, dp);
            mc_fetch(vs + (c & 1u) * MC_L * VS, VS, x + (size_t)c * MC_L * p.ld + p.v_off + h * p.vdim + c0, p.ld, live, vw, MC_COLS);
        }
        cp_async_commit();
    };
    fetch(0);
    float S[RT][MC_COLS / 8][4];
#pragma unroll
    for (int r = 0; r < RT; r++)
    {
#pragma unroll
        for (int j = 0; j < (int)MC_COLS / 8; j++)
        {
#pragma unroll
            for (int half = 0; half < 2; half++)
            {
                const unsigned int d = (warp + r * MC_WARPS) * 16 + gr + 8 * half, col = c0 + j * 8 + gc;
                float2 v = make_float2(0.f, 0.f);
                if (!fresh && d < p.dim && col < p.vdim) { v = *reinterpret_cast<const float2*>(st + (size_t)d * v_ld + col); }
                S[r][j][2 * half] = v.x;
                S[r][j][2 * half + 1] = v.y;
            }
        }
    }
    float m = fresh ? 0.f : st_n[mlstm_n_ld(p.dim)], nn = !fresh && tid < p.dim ? st_n[tid] : 0.f;
    for (unsigned int c = 0; c < chunks; c++)
    {
        const unsigned int live = min(MC_L, n - c * MC_L);
        fetch(c + 1);
        float* rec = mc_record_of(p, e, c, h);
        if (!fresh || c > 0)
        {
            __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(rec);
#pragma unroll
            for (int r = 0; r < RT; r++)
            {
#pragma unroll
                for (int j = 0; j < (int)MC_COLS / 8; j++)
                {
#pragma unroll
                    for (int half = 0; half < 2; half++)
                    {
                        const unsigned int d = (warp + r * MC_WARPS) * 16 + gr + 8 * half;
                        const float s0 = S[r][j][2 * half], s1 = S[r][j][2 * half + 1];
                        const uint32_t top = pack_bf16x2(s0, s1);
                        if (d < dp)
                        {
                            uint32_t* y = reinterpret_cast<uint32_t*>(out + (size_t)d * vp + c0 + j * 8 + gc);
                            y[0] = top;
                            y[(size_t)dp * vp / 2] = pack_bf16x2(s0 - __uint_as_float(top << 16), s1 - __uint_as_float(top & 0xFFFF0000u));
                        }
                    }
                }
            }
        }
        if (blockIdx.x == 0)
        {
            if (tid < dp) { rec[(size_t)dp * vp + tid] = nn; }
            if (tid == 0) { rec[(size_t)dp * vp + dp] = m; }
        }
        mc_gates(p, start + c * MC_L, live, h, F, a, sums);
        float top = m;    // M at the chunk's end
        for (unsigned int s = lane; s < MC_L; s += 32) { top = fmaxf(top, a[s]); }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) { top = fmaxf(top, __shfl_xor_sync(0xFFFFFFFFu, top, o)); }
        const float keep = expf(m - top);
        if (tid < MC_L) { w[tid] = expf(a[tid] - top); }
        m = F[MC_L - 1] + top;
        cp_async_wait<1>();
        __syncthreads();
        const __nv_bfloat16* v = v_raw + (c & 1u) * MC_L * (MC_COLS + 8);
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
            const __nv_bfloat16* k = reinterpret_cast<const __nv_bfloat16*>(mc_raw + (c & 1u) * MC_L * KS) + tid;
            nn *= keep;
#pragma unroll 8
            for (unsigned int s = 0; s < MC_L; s++) { nn = fmaf(w[s], __bfloat162float(k[s * (dp + 8)]), nn); }
        }
        __syncthreads();
        const uint32_t kb = ks + (c & 1u) * MC_L * KS + ((lane & 7) + ((lane >> 4) << 3)) * KS + ((lane >> 3) & 1) * 16;
        const uint32_t vb = (lane & 15) * VS + (lane >> 4) * 16;
#pragma unroll
        for (int r = 0; r < RT; r++)
        {
#pragma unroll
            for (int j = 0; j < (int)MC_COLS / 8; j++)
            {
#pragma unroll
                for (int i = 0; i < 4; i++) { S[r][j][i] *= keep; }
            }
        }
        for (unsigned int s0 = 0; s0 < live; s0 += 16)
        {
            uint32_t b[2][MC_COLS / 16][4];
#pragma unroll
            for (int j = 0; j < (int)MC_COLS / 16; j++)
            {
                ldmatrix_x4_trans(b[0][j], hs + vb + s0 * VS + j * 32);
                ldmatrix_x4_trans(b[1][j], ls + vb + s0 * VS + j * 32);
            }
#pragma unroll
            for (int r = 0; r < RT; r++)
            {
                const unsigned int d = (warp + r * MC_WARPS) * 16;
                if (d < dp)
                {
                    uint32_t k[4];
                    ldmatrix_x4_trans(k, kb + s0 * KS + d * 2);
#pragma unroll
                    for (int part = 0; part < 2; part++)
                    {
#pragma unroll
                        for (int j = 0; j < (int)MC_COLS / 16; j++)
                        {
                            mma_bf16_16816(S[r][2 * j], k[0], k[1], k[2], k[3], b[part][j][0], b[part][j][1]);
                            mma_bf16_16816(S[r][2 * j + 1], k[0], k[1], k[2], k[3], b[part][j][2], b[part][j][3]);
                        }
                    }
                }
            }
        }
        __syncthreads();    // the next chunk but one takes this one's place
    }
    cp_async_wait<0>();
#pragma unroll
    for (int r = 0; r < RT; r++)
    {
#pragma unroll
        for (int j = 0; j < (int)MC_COLS / 8; j++)
        {
#pragma unroll
            for (int half = 0; half < 2; half++)
            {
                const unsigned int d = (warp + r * MC_WARPS) * 16 + gr + 8 * half, col = c0 + j * 8 + gc;
                if (d < p.dim && col < p.vdim) { *reinterpret_cast<float2*>(st + (size_t)d * v_ld + col) = make_float2(S[r][j][2 * half], S[r][j][2 * half + 1]); }
            }
        }
    }
    // other column blocks may still have to read the old n and m: the second kernel puts the new ones in place
    if (blockIdx.x == 0 && chunks > 0)
    {
        float* last = mc_record_of(p, e, chunks - 1, h) + (size_t)dp * vp + dp + 4;
        if (tid < p.dim) { last[tid] = nn; }
        if (tid == 0) { last[dp] = m; }
    }
}

__host__ __device__ constexpr unsigned int mc_states_smem(unsigned int dp) { return 2 * MC_L * ((dp + 8) * 2 + (MC_COLS + 8) * 2); }
__host__ __device__ constexpr unsigned int mc_outputs_smem(unsigned int dp, unsigned int vb)
{
    return 2 * MC_L * (dp + 8) * 2 + MC_L * (vb + 8) * 2 + 4 * MC_SLICE * (vb + 8) * 2 + (dp + 4) * 4;
}

// grid (column blocks of VB = the cluster, heads, entries x chunks); a warp owns 16 tokens
template <int VB>
__global__ void __launch_bounds__(MC_THREADS) mlstm_outputs_kernel(const MlstmParams p, const unsigned int max_chunks)
{
    extern __shared__ __align__(16) unsigned char mc_raw[];
    __shared__ float F[MC_L], a[MC_L], M[MC_L], sums[MC_WARPS], sq[MC_L], peers[MC_MAX_CLUSTER][MC_L];
    constexpr unsigned int VS = (VB + 8) * 2, SLICE = MC_SLICE * VS;
    const unsigned int dp = mc_dp(p.dim), vp = mc_vp(p.vdim), QS = (dp + 8) * 2;
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, gc = (lane & 3) * 2;
    const unsigned int rank = blockIdx.x, h = blockIdx.y, e = p.e0 + blockIdx.z / max_chunks, c = blockIdx.z % max_chunks, c0 = rank * VB;
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e];
    if (c * MC_L >= n) { return; }    // the whole cluster
    const unsigned int live = min(MC_L, n - c * MC_L), first = start + c * MC_L;
    const bool fresh = p.pos[e] == 0 && c == 0;
    const float* rec = mc_record_of(p, e, c, h);
    const __nv_bfloat16* before = reinterpret_cast<const __nv_bfloat16*>(rec);
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg + (size_t)first * p.ld;
    const uint32_t qs = smem_u32(mc_raw), ks = qs + MC_L * QS, vs = ks + MC_L * QS, ss = vs + MC_L * VS;
    float* n0 = reinterpret_cast<float*>(mc_raw + 2 * MC_L * QS + MC_L * VS + 4 * SLICE);
    const unsigned int slices = fresh ? 0 : dp / MC_SLICE;
    auto fetch_slice = [&](unsigned int i) {
        if (i < slices)
        {
            for (unsigned int j = tid; j < 2 * MC_SLICE * (VB / 8); j += MC_THREADS)
            {
                const unsigned int part = j / (MC_SLICE * (VB / 8)), r = j / (VB / 8) % MC_SLICE, d = j % (VB / 8), col = c0 + d * 8;
                const bool ok = col < vp;
                cp_async16(ss + ((i & 1u) * 2 + part) * SLICE + r * VS + d * 16,
                    before + (ok ? (size_t)part * dp * vp + (size_t)(i * MC_SLICE + r) * vp + col : 0), ok);
            }
        }
        cp_async_commit();
    };
    mc_fetch(qs, QS, x + h * p.dim, p.ld, live, p.dim, dp);
    fetch_slice(0);
    fetch_slice(1);
    mc_fetch(ks, QS, x + p.k_off + h * p.dim, p.ld, live, p.dim, dp);
    mc_fetch(vs, VS, x + p.v_off + h * p.vdim + c0, p.ld, live, p.vdim > c0 ? min((unsigned int)VB, p.vdim - c0) : 0u, VB);
    cp_async_commit();
    for (unsigned int d = tid; d < dp; d += MC_THREADS) { n0[d] = fresh ? 0.f : rec[(size_t)dp * vp + d]; }
    const float m0 = fresh ? 0.f : rec[(size_t)dp * vp + dp];
    mc_gates(p, first, live, h, F, a, sums);
    if (tid < MC_L)    // M: running maxima, with m0
    {
        float t = a[tid];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1)
        {
            const float y = __shfl_up_sync(0xFFFFFFFFu, t, o);
            if (lane >= (unsigned int)o) { t = fmaxf(t, y); }
        }
        if (lane == 31) { sums[warp] = t; }
        M[tid] = t;
    }
    __syncthreads();
    if (tid < MC_L)
    {
        float t = fmaxf(m0, M[tid]);
        for (unsigned int j = 0; j < warp; j++) { t = fmaxf(t, sums[j]); }
        M[tid] = t;
    }
    const unsigned int r0 = warp * 16;
    float o[VB / 8][4], nq[2] = { 0.f, 0.f };
#pragma unroll
    for (int j = 0; j < VB / 8; j++)
    {
#pragma unroll
        for (int i = 0; i < 4; i++) { o[j][i] = 0.f; }
    }
    const uint32_t qa = qs + (r0 + (lane & 15)) * QS + (lane >> 4) * 16;
    for (unsigned int i = 0; i < slices; i++)
    {
        if (i < 2) { cp_async_wait<2>(); }
        else { cp_async_wait<1>(); }
        __syncthreads();
        const uint32_t sb = ss + (i & 1u) * 2 * SLICE + (lane & 15) * VS + (lane >> 4) * 16;
#pragma unroll
        for (int kk = 0; kk < (int)MC_SLICE / 16; kk++)
        {
            uint32_t q[4];
            ldmatrix_x4(q, qa + (i * MC_SLICE + kk * 16) * 2);
#pragma unroll
            for (int part = 0; part < 2; part++)
            {
#pragma unroll
                for (int j = 0; j < VB / 16; j++)
                {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, sb + part * SLICE + kk * 16 * VS + j * 32);
                    mma_bf16_16816(o[2 * j], q[0], q[1], q[2], q[3], b[0], b[1]);
                    mma_bf16_16816(o[2 * j + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
                }
            }
        }
        __syncthreads();
        fetch_slice(i + 2);
    }
    cp_async_wait<0>();
    __syncthreads();
    float mt[2], carry[2];
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
        mt[i] = M[r0 + gr + 8 * i];
        carry[i] = p.q_scale * expf(m0 - mt[i]);
    }
    if (!fresh)
    {
#pragma unroll
        for (int j = 0; j < VB / 8; j++)
        {
#pragma unroll
            for (int i = 0; i < 4; i++) { o[j][i] *= carry[i >> 1]; }
        }
        // n0 . q: the four lanes of a row share its elements
#pragma unroll
        for (int i = 0; i < 2; i++)
        {
            const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(mc_raw) + (size_t)(r0 + gr + 8 * i) * (dp + 8);
            float s = 0.f;
            for (unsigned int d = gc; d < dp; d += 8)
            {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q + d));
                s = fmaf(f.x, n0[d], s);
                s = fmaf(f.y, n0[d + 1], s);
            }
            nq[i] = carry[i] * s;
        }
    }
    const uint32_t kb = ks + ((lane & 7) + ((lane >> 4) << 3)) * QS + ((lane >> 3) & 1) * 16;
    const uint32_t vb = vs + (lane & 15) * VS + (lane >> 4) * 16;
    for (unsigned int s0 = 0; s0 < r0 + 16; s0 += 32)
    {
        float z[4][4];
#pragma unroll
        for (int i = 0; i < 4; i++)
        {
#pragma unroll
            for (int j = 0; j < 4; j++) { z[i][j] = 0.f; }
        }
        for (unsigned int kk = 0; kk < dp / 16; kk++)
        {
            uint32_t q[4];
            ldmatrix_x4(q, qa + kk * 32);
#pragma unroll
            for (int i = 0; i < 2; i++)
            {
                uint32_t b[4];
                ldmatrix_x4(b, kb + (s0 + i * 16) * QS + kk * 32);
                mma_bf16_16816(z[2 * i], q[0], q[1], q[2], q[3], b[0], b[1]);
                mma_bf16_16816(z[2 * i + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
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
            for (int j = 0; j < VB / 16; j++)
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
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
        nq[i] += __shfl_xor_sync(0xFFFFFFFFu, nq[i], 1);
        nq[i] += __shfl_xor_sync(0xFFFFFFFFu, nq[i], 2);
        const float inv = 1.0f / (fmaxf(fabsf(nq[i]), expf(-(F[r0 + gr + 8 * i] + mt[i]))) + 1e-6f);
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < VB / 8; j++)
        {
            o[j][2 * i] *= inv;
            o[j][2 * i + 1] *= inv;
            s += o[j][2 * i] * o[j][2 * i] + o[j][2 * i + 1] * o[j][2 * i + 1];
        }
        s += __shfl_xor_sync(0xFFFFFFFFu, s, 1);
        s += __shfl_xor_sync(0xFFFFFFFFu, s, 2);
        if ((lane & 3) == 0) { sq[r0 + gr + 8 * i] = s; }
    }
    __syncthreads();
    cg::cluster_group cluster = cg::this_cluster();
    const unsigned int ranks = cluster.num_blocks();
    for (unsigned int j = tid; j < ranks * MC_L; j += MC_THREADS) { cluster.map_shared_rank(&peers[0][0], j / MC_L)[rank * MC_L + j % MC_L] = sq[j % MC_L]; }
    cluster.sync();
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
        const unsigned int t = r0 + gr + 8 * i;
        if (t >= live) { continue; }
        float s = 0.f;
        for (unsigned int r = 0; r < ranks; r++) { s += peers[r][t]; }
        const float inv = 1.0f / sqrtf(s / (float)p.vdim + p.eps);
        const __nv_bfloat16* gate = x + (size_t)t * p.ld + p.g_off + h * p.vdim + c0;
        __nv_bfloat16* out = (__nv_bfloat16*)p.out + (size_t)(first + t) * p.ldo + h * p.vdim + c0;
        const float* w = p.norm + h * p.vdim + c0;
#pragma unroll
        for (int j = 0; j < VB / 8; j++)
        {
            const unsigned int col = j * 8 + gc;
            if (c0 + col < p.vdim)
            {
                const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + col));
                *reinterpret_cast<uint32_t*>(out + col) =
                    pack_bf16x2(o[j][2 * i] * inv * w[col] * sigmoid_f32(g.x), o[j][2 * i + 1] * inv * w[col + 1] * sigmoid_f32(g.y));
            }
        }
    }
    if (rank == 0 && (c + 1) * MC_L >= n)
    {
        const float* last = rec + (size_t)dp * vp + dp + 4;
        float* st_n = mlstm_state_of(p, e, h) + (size_t)p.dim * mlstm_v_ld(p.vdim);
        for (unsigned int d = tid; d < p.dim; d += MC_THREADS) { st_n[d] = last[d]; }
        if (tid == 0) { st_n[mlstm_n_ld(p.dim)] = last[dp]; }
    }
}

template <int RT>
static int run_states(const MlstmParams& p, unsigned int entries, cudaStream_t stream, bool pdl)
{
    return launch_kernel("mlstm_states", mlstm_states_kernel<RT>, dim3(mc_vp(p.vdim) / MC_COLS, p.heads, entries), dim3(MC_THREADS),
        (size_t)mc_states_smem(mc_dp(p.dim)), stream, pdl, p);
}
template <int VB>
static int run_outputs(const MlstmParams& p, unsigned int entries, cudaStream_t stream, bool pdl)
{
    const unsigned int ranks = (p.vdim + VB - 1) / VB, chunks = (p.max_n + MC_L - 1) / MC_L;
    return launch_cluster("mlstm_outputs", mlstm_outputs_kernel<VB>, dim3(ranks, p.heads, entries * chunks), dim3(MC_THREADS),
        (size_t)mc_outputs_smem(mc_dp(p.dim), VB), ranks, stream, pdl, p, chunks);
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
    const unsigned int dp = mc_dp(p.dim);
    int rc = dp <= 128 ? run_states<1>(p, entries, stream, pdl) : run_states<2>(p, entries, stream, pdl);
    if (rc) { return rc; }
    return p.vdim <= 64 ? run_outputs<64>(p, entries, stream, pdl) : run_outputs<128>(p, entries, stream, pdl);
}

}    // namespace b200
