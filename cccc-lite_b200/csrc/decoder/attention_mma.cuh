// BF16 attention on mma.sync: a warp holds 16 query rows (a row is one query head of one token; the heads that share a
// kv head are packed together) as A fragments and walks keys with a running softmax in float.  Keys arrive through
// cp.async into padded shared-memory rows; K is the B operand as it lies, V through transposed ldmatrix.  Softmax weights
// enter the value product as the sum of two BF16 numbers, so that they keep 16 significant bits.
//   split : few query rows.  A CTA's four warps take 16-key tiles of one split of the sequence in turn, each through a
//           ring of its own; their partial results meet in shared memory, the splits' in global memory, where the last
//           CTA to arrive adds them in split order.
//   tiled : prompts.  Four warps with 16 rows each share 64-key tiles, double buffered.
#pragma once

#include "attention.cuh"
#include "../gemv_decode.cuh"

namespace b200
{

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid)
{
    const int bytes = valid ? 16 : 0;    // 0: sixteen zero bytes
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait()
{
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}

// 16 query rows of one warp and their running softmax.
template <int DK, int DV>
struct RowTile
{
    uint32_t q[DK / 16][4];
    float o[DV / 8][4];
    float m[2], l[2];    // rows lane / 4 and lane / 4 + 8, in units of log2

    // r0: first packed row of the tile inside entry e
    __device__ __forceinline__ void init(const AttnParams& p, const __nv_bfloat16* qkvg, unsigned int start, unsigned int n, unsigned int kvh,
        unsigned int r0, unsigned int lane)
    {
        const unsigned int rows = n * p.G;
        const __nv_bfloat16* src[2];
        bool ok[2];
#pragma unroll
        for (int h = 0; h < 2; h++)
        {
            const unsigned int r = r0 + (lane >> 2) + 8 * h;
            ok[h] = r < rows;
            const unsigned int rr = ok[h] ? r : 0;
            src[h] = qkvg + (size_t)(start + rr / p.G) * p.ld + (size_t)(kvh * p.G + rr % p.G) * p.q_ld;
            m[h] = -INFINITY;
            l[h] = 0.f;
        }
#pragma unroll
        for (int kk = 0; kk < DK / 16; kk++)
        {
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                const int h = j & 1;
                const unsigned int d = kk * 16 + (lane & 3) * 2 + (j >> 1) * 8;
                uint32_t lo = 0, hi = 0;
                if (ok[h] && d < p.dim) { lo = __bfloat16_as_ushort(src[h][d]); }
                if (ok[h] && d + 1 < p.dim) { hi = __bfloat16_as_ushort(src[h][d + 1]); }
                q[kk][j] = lo | (hi << 16);
            }
        }
#pragma unroll
        for (int i = 0; i < DV / 8; i++)
        {
#pragma unroll
            for (int j = 0; j < 4; j++) { o[i][j] = 0.f; }
        }
    }

    // KT keys (a multiple of 16) at shared addresses ks / vs, the first being key k0 of the sequence; row h sees the keys
    // from low[h] on and below lim[h].  scale2 = scale * log2(e).
    template <int KT>
    __device__ __forceinline__ void step(uint32_t ks, uint32_t vs, unsigned int k0, const unsigned int (&low)[2], const unsigned int (&lim)[2], bool masked, float scale2,
        unsigned int dim, unsigned int vdim, unsigned int lane)
    {
        constexpr int KS = (DK + 8) * 2, VS = (DV + 8) * 2;
        float s[KT / 8][4];
#pragma unroll
        for (int i = 0; i < KT / 8; i++)
        {
#pragma unroll
            for (int j = 0; j < 4; j++) { s[i][j] = 0.f; }
        }
        // lanes 0-7: keys 0-7, k 0-7; 8-15: keys 0-7, k 8-15; 16-23: keys 8-15, k 0-7; 24-31: keys 8-15, k 8-15
        const uint32_t kb = ks + ((lane & 7) + ((lane >> 4) << 3)) * KS + ((lane >> 3) & 1) * 16;
#pragma unroll
        for (int kk = 0; kk < DK / 16; kk++)
        {
            if (kk * 16 < (int)dim)
            {
#pragma unroll
                for (int i = 0; i < KT / 16; i++)
                {
                    uint32_t b[4];
                    ldmatrix_x4(b, kb + i * 16 * KS + kk * 32);
                    mma_bf16_16816(s[2 * i], q[kk][0], q[kk][1], q[kk][2], q[kk][3], b[0], b[1]);
                    mma_bf16_16816(s[2 * i + 1], q[kk][0], q[kk][1], q[kk][2], q[kk][3], b[2], b[3]);
                }
            }
        }
        float mx[2] = { -INFINITY, -INFINITY };
#pragma unroll
        for (int i = 0; i < KT / 8; i++)
        {
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                s[i][j] *= scale2;
                const unsigned int key = k0 + i * 8 + (lane & 3) * 2 + (j & 1);
                if (masked && (key < low[j >> 1] || key >= lim[j >> 1])) { s[i][j] = -INFINITY; }
                mx[j >> 1] = fmaxf(mx[j >> 1], s[i][j]);
            }
        }
        float base[2];
#pragma unroll
        for (int h = 0; h < 2; h++)
        {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xFFFFFFFFu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xFFFFFFFFu, mx[h], 2));
            const float mn = fmaxf(m[h], mx[h]);
            base[h] = mn == -INFINITY ? 0.f : mn;
            const float c = exp2f(m[h] - base[h]);    // 0 while nothing has been seen
            m[h] = mn;
            l[h] *= c;
#pragma unroll
            for (int i = 0; i < DV / 8; i++)
            {
                o[i][2 * h] *= c;
                o[i][2 * h + 1] *= c;
            }
        }
        const uint32_t vb = vs + (lane & 15) * VS + (lane >> 4) * 16;
#pragma unroll
        for (int i = 0; i < KT / 16; i++)
        {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                // a0: row g, keys 0-7; a1: row g + 8, keys 0-7; a2, a3: keys 8-15
                float* c = &s[2 * i + (j >> 1)][(j & 1) * 2];
                const int h = j & 1;
                const float p0 = exp2f(c[0] - base[h]), p1 = exp2f(c[1] - base[h]);
                l[h] += p0 + p1;
                hi[j] = pack_bf16x2(p0, p1);
                lo[j] = pack_bf16x2(p0 - __uint_as_float(hi[j] << 16), p1 - __uint_as_float(hi[j] & 0xFFFF0000u));
            }
#pragma unroll
            for (int d = 0; d < DV / 16; d++)
            {
                if (d * 16 < (int)vdim)
                {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, vb + i * 16 * VS + d * 32);
                    mma_bf16_16816(o[2 * d], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                    mma_bf16_16816(o[2 * d + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                    mma_bf16_16816(o[2 * d], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
                    mma_bf16_16816(o[2 * d + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
                }
            }
        }
    }
    // the row sums are held per lane until here
    __device__ __forceinline__ void finish()
    {
#pragma unroll
        for (int h = 0; h < 2; h++)
        {
            l[h] += __shfl_xor_sync(0xFFFFFFFFu, l[h], 1);
            l[h] += __shfl_xor_sync(0xFFFFFFFFu, l[h], 2);
        }
    }
};

__device__ __forceinline__ void attention_store(const AttnParams& p, const __nv_bfloat16* qkvg, unsigned int start, unsigned int kvh, unsigned int r,
    unsigned int d, float v)
{
    const unsigned int col = (kvh * p.G + r % p.G) * p.vdim + d;
    const size_t tok = start + r / p.G;
    v *= head_factor<__nv_bfloat16>(p, tok, kvh * p.G + r % p.G);
    if (p.gate) { v *= sigmoid_f32(__bfloat162float(qkvg[tok * p.ld + p.g_off + col])); }
    ((__nv_bfloat16*)p.out)[tok * p.ldo + col] = __float2bfloat16_rn(v);
}

constexpr int AS_WARPS = 4, AS_KT = 16;
constexpr unsigned int kMaxSplits = 32;

// What the warps of a split CTA leave for each other, and the last CTA's weights of the splits.
struct SplitMeet
{
    float ml[AS_WARPS][16][2];    // maximum (log2) and sum of every row
    float weight[16][kMaxSplits];
    float inv[16];
    int last;
};

// Adds the four warps' results (om: [warp][RT][DV] floats, meet.ml) and, with several splits, the splits' - the last CTA of
// a unit to arrive does, in split order, so that the bits do not depend on who that is.  All 128 threads call.
template <int DV, int RT>
__device__ __forceinline__ void split_finish(const AttnParams& p, SplitMeet& meet, const float* om, const __nv_bfloat16* qkvg, unsigned int e,
    unsigned int start, unsigned int kvh, unsigned int rt, unsigned int r0, unsigned int rows)
{
    __syncthreads();
    const unsigned int tid = threadIdx.x, live = min((unsigned int)RT, rows - r0);
    if (tid < live)
    {
        float m = -INFINITY, l = 0.f;
#pragma unroll
        for (int w = 0; w < AS_WARPS; w++) { m = fmaxf(m, meet.ml[w][tid][0]); }
        float c[AS_WARPS];
#pragma unroll
        for (int w = 0; w < AS_WARPS; w++)
        {
            c[w] = m == -INFINITY ? 0.f : exp2f(meet.ml[w][tid][0] - m);
            l += c[w] * meet.ml[w][tid][1];
        }
#pragma unroll
        for (int w = 0; w < AS_WARPS; w++) { meet.ml[w][tid][0] = c[w]; }
        if (p.sink != nullptr && p.splits == 1) { l += exp2f(p.sink[kvh * p.G + (r0 + tid) % p.G] * 1.44269504088896341f - m); }
        meet.ml[0][tid][1] = m;
        meet.ml[1][tid][1] = l;
    }
    __syncthreads();
    auto sum = [&](unsigned int r, unsigned int d) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < AS_WARPS; w++) { o += meet.ml[w][r][0] * om[(w * RT + r) * DV + d]; }
        return o;
    };
    if (p.splits == 1)
    {
        for (unsigned int j = tid; j < live * p.vdim; j += 32 * AS_WARPS)
        {
            const unsigned int r = j / p.vdim, d = j % p.vdim;
            attention_store(p, qkvg, start, kvh, r0 + r, d, sum(r, d) / meet.ml[1][r][1]);
        }
        return;
    }
    const unsigned int vp = (p.vdim + 15) / 16 * 16, stride = 16 * (vp + 2), split = blockIdx.x;
    const unsigned int unit = ((e - p.e0) * p.row_tiles + rt) * p.Hkv + kvh;
    float* all = p.partial + (size_t)unit * p.splits * stride;
    float* mine = all + (size_t)split * stride;
    for (unsigned int j = tid; j < live * p.vdim; j += 32 * AS_WARPS)
    {
        const unsigned int r = j / p.vdim, d = j % p.vdim;
        mine[32 + r * vp + d] = sum(r, d);
    }
    if (tid < live)
    {
        mine[2 * tid] = meet.ml[0][tid][1];
        mine[2 * tid + 1] = meet.ml[1][tid][1];
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) { meet.last = atomicAdd(p.counter + unit, 1) == (int)p.splits - 1; }
    __syncthreads();
    if (!meet.last) { return; }
    __threadfence();
    for (unsigned int j = tid; j < live * p.splits; j += 32 * AS_WARPS)
    {
        const unsigned int r = j / p.splits, s = j % p.splits;
        meet.weight[r][s] = __ldcg(all + (size_t)s * stride + 2 * r);
    }
    __syncthreads();
    // a warp per row: the rows' maxima over the splits, then weights and sums
    for (unsigned int r = tid >> 5; r < live; r += AS_WARPS)
    {
        const unsigned int lane = tid & 31;
        float m = -INFINITY, l = 0.f;
        for (unsigned int s = lane; s < p.splits; s += 32) { m = fmaxf(m, meet.weight[r][s]); }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) { m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, o)); }
        for (unsigned int s = lane; s < p.splits; s += 32)
        {
            const float c = exp2f(meet.weight[r][s] - m);
            meet.weight[r][s] = c;
            l += c * __ldcg(all + (size_t)s * stride + 2 * r + 1);
        }
        l = warp_sum(l);
        if (p.sink != nullptr) { l += exp2f(p.sink[kvh * p.G + (r0 + r) % p.G] * 1.44269504088896341f - m); }
        if (lane == 0) { meet.inv[r] = 1.0f / l; }
    }
    __syncthreads();
    // four columns per thread (the rows are padded to sixteen)
    for (unsigned int j = tid; j < live * (vp / 4); j += 32 * AS_WARPS)
    {
        const unsigned int r = j / (vp / 4), d = (j % (vp / 4)) * 4;
        const float* src = all + 32 + r * vp + d;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 16
        for (unsigned int s = 0; s < p.splits; s++)
        {
            const float4 x = __ldcg(reinterpret_cast<const float4*>(src + (size_t)s * stride));
            const float c = meet.weight[r][s];
            o.x += c * x.x;
            o.y += c * x.y;
            o.z += c * x.z;
            o.w += c * x.w;
        }
        const float out[4] = { o.x, o.y, o.z, o.w };
#pragma unroll
        for (int i = 0; i < 4; i++)
        {
            if (d + i < p.vdim) { attention_store(p, qkvg, start, kvh, r0 + r, d + i, out[i] * meet.inv[r]); }
        }
    }
    if (tid == 0) { p.counter[unit] = 0; }
}

__host__ __device__ constexpr int as_stages(int dk, int dv) { return dk + dv <= 256 ? 4 : 3; }
__host__ __device__ constexpr int as_tile_bytes(int dk, int dv) { return AS_KT * ((dk + 8) + (dv + 8)) * 2; }
__host__ __device__ constexpr int as_smem(int dk, int dv)
{
    const int ring = AS_WARPS * as_stages(dk, dv) * as_tile_bytes(dk, dv), meet = AS_WARPS * 16 * (dv + 2) * 4;
    return ring > meet ? ring : meet;
}

// grid (splits, Hkv * row_tiles, entries)
template <int DK, int DV>
__global__ void __launch_bounds__(32 * AS_WARPS) attention_split_kernel(const AttnParams p)
{
    extern __shared__ __align__(16) unsigned char as_raw[];
    constexpr int ST = as_stages(DK, DV), TB = as_tile_bytes(DK, DV), KS = (DK + 8) * 2, VS = (DV + 8) * 2;
    __shared__ SplitMeet meet;
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const unsigned int split = blockIdx.x, kvh = blockIdx.y % p.Hkv, rt = blockIdx.y / p.Hkv, e = p.e0 + blockIdx.z;
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], pos = (unsigned int)p.pos[e], r0 = rt * 16;
    const unsigned int rows = n * p.G;
    if (r0 >= rows) { return; }
    const __nv_bfloat16* qkvg = (const __nv_bfloat16*)p.qkvg;
    const size_t seq = ((size_t)p.slot[e] * p.Hkv + kvh) * p.T_max;
    const __nv_bfloat16* K = (const __nv_bfloat16*)p.k_cache + seq * p.k_ld;
    const __nv_bfloat16* V = (const __nv_bfloat16*)p.v_cache + seq * p.v_ld;
    // keys that any row of the tile sees, cut into equal runs of whole tiles
    const unsigned int last_row = min(r0 + 15u, rows - 1);
    const unsigned int T = min(pos + last_row / p.G + 1, p.T_max);
    const unsigned int first_lim = pos + r0 / p.G + 1;    // no row ends before
    const unsigned int begin = first_key(p, e, first_lim) / AS_KT, last_low = first_key(p, e, pos + last_row / p.G + 1);
    const unsigned int tiles = (T + AS_KT - 1) / AS_KT, per = (tiles - begin + p.splits - 1) / p.splits;
    const unsigned int tile0 = min(begin + split * per, tiles), tile1 = min(tile0 + per, tiles);

    RowTile<DK, DV> w;
    w.init(p, qkvg, start, n, kvh, r0, lane);
    unsigned int low[2], lim[2];
#pragma unroll
    for (int h = 0; h < 2; h++)
    {
        const unsigned int end = pos + (r0 + (lane >> 2) + 8 * h) / p.G + 1;
        low[h] = first_key(p, e, end);
        lim[h] = min(end, T);
    }

    const uint32_t ring = smem_u32(as_raw) + warp * (ST * TB);
    auto fetch = [&](unsigned int i) {    // i-th tile of this warp
        const unsigned int tile = tile0 + warp + i * AS_WARPS;
        if (tile < tile1)
        {
            const uint32_t ks = ring + (i % ST) * TB, vs = ks + AS_KT * KS;
            for (unsigned int c = lane; c < AS_KT * (DK / 8); c += 32)
            {
                const unsigned int r = c / (DK / 8), d = c % (DK / 8), key = tile * AS_KT + r;
                const bool ok = key < T && d * 8 < p.k_ld;
                cp_async16(ks + r * KS + d * 16, K + (ok ? (size_t)key * p.k_ld + d * 8 : 0), ok);
            }
            for (unsigned int c = lane; c < AS_KT * (DV / 8); c += 32)
            {
                const unsigned int r = c / (DV / 8), d = c % (DV / 8), key = tile * AS_KT + r;
                const bool ok = key < T && d * 8 < p.v_ld;
                cp_async16(vs + r * VS + d * 16, V + (ok ? (size_t)key * p.v_ld + d * 8 : 0), ok);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < ST - 1; i++) { fetch(i); }
    const float scale2 = p.scale * 1.44269504088896341f;
    unsigned int i = 0;
    for (unsigned int tile = tile0 + warp; tile < tile1; tile += AS_WARPS, i++)
    {
        fetch(i + ST - 1);
        cp_async_wait<ST - 1>();
        __syncwarp();
        const uint32_t ks = ring + (i % ST) * TB;
        w.template step<AS_KT>(ks, ks + AS_KT * KS, tile * AS_KT, low, lim, (tile + 1) * AS_KT > first_lim || tile * AS_KT < last_low, scale2, p.dim, p.vdim, lane);
        __syncwarp();
    }
    cp_async_wait<0>();
    w.finish();
    __syncthreads();    // the rings become the meeting place
    float* om = reinterpret_cast<float*>(as_raw) + warp * 16 * DV;
    const unsigned int gr = lane >> 2, gc = (lane & 3) * 2;
#pragma unroll
    for (int d = 0; d < DV / 8; d++)
    {
        *reinterpret_cast<float2*>(om + gr * DV + d * 8 + gc) = make_float2(w.o[d][0], w.o[d][1]);
        *reinterpret_cast<float2*>(om + (gr + 8) * DV + d * 8 + gc) = make_float2(w.o[d][2], w.o[d][3]);
    }
    if ((lane & 3) == 0)
    {
#pragma unroll
        for (int h = 0; h < 2; h++)
        {
            meet.ml[warp][gr + 8 * h][0] = w.m[h];
            meet.ml[warp][gr + 8 * h][1] = w.l[h];
        }
    }
    split_finish<DV, 16>(p, meet, reinterpret_cast<float*>(as_raw), qkvg, e, start, kvh, rt, r0, rows);
}

constexpr int AT_WARPS = 4;
__host__ __device__ constexpr int at_kt(int dk, int dv) { return dk + dv <= 256 ? 64 : 32; }
__host__ __device__ constexpr int at_smem(int dk, int dv) { return 2 * at_kt(dk, dv) * ((dk + 8) + (dv + 8)) * 2; }

// grid (row tiles of 64, Hkv, entries); the last rows of a prompt see the most keys and start first
template <int DK, int DV>
__global__ void __launch_bounds__(32 * AT_WARPS) attention_tiled_kernel(const AttnParams p)
{
    extern __shared__ __align__(16) unsigned char at_raw[];
    constexpr int KT = at_kt(DK, DV), KS = (DK + 8) * 2, VS = (DV + 8) * 2, TB = KT * (KS + VS);
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const unsigned int kvh = blockIdx.y, e = p.e0 + blockIdx.z;
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], pos = (unsigned int)p.pos[e];
    const unsigned int rows = n * p.G, tiles_r = (rows + 16 * AT_WARPS - 1) / (16 * AT_WARPS);
    if (blockIdx.x >= tiles_r) { return; }
    const unsigned int t0 = (tiles_r - 1 - blockIdx.x) * 16 * AT_WARPS, r0 = t0 + warp * 16;
    const __nv_bfloat16* qkvg = (const __nv_bfloat16*)p.qkvg;
    const size_t seq = ((size_t)p.slot[e] * p.Hkv + kvh) * p.T_max;
    const __nv_bfloat16* K = (const __nv_bfloat16*)p.k_cache + seq * p.k_ld;
    const __nv_bfloat16* V = (const __nv_bfloat16*)p.v_cache + seq * p.v_ld;
    const unsigned int T = min(pos + min(t0 + 16u * AT_WARPS - 1, rows - 1) / p.G + 1, p.T_max);
    const unsigned int tiles = (T + KT - 1) / KT;

    RowTile<DK, DV> w;
    w.init(p, qkvg, start, n, kvh, r0, lane);
    unsigned int low[2], lim[2];
#pragma unroll
    for (int h = 0; h < 2; h++)
    {
        const unsigned int end = pos + (r0 + (lane >> 2) + 8 * h) / p.G + 1;
        low[h] = first_key(p, e, end);
        lim[h] = min(end, T);
    }
    const unsigned int first_lim = pos + r0 / p.G + 1, last_lim = pos + (r0 + 15) / p.G + 1;
    const unsigned int begin = first_key(p, e, pos + t0 / p.G + 1) / KT, first_low = first_key(p, e, first_lim), last_low = first_key(p, e, last_lim);

    const uint32_t ring = smem_u32(at_raw);
    auto fetch = [&](unsigned int tile) {
        if (tile < tiles)
        {
            const uint32_t ks = ring + (tile & 1u) * TB, vs = ks + KT * KS;
            for (unsigned int c = threadIdx.x; c < KT * (DK / 8); c += 32 * AT_WARPS)
            {
                const unsigned int r = c / (DK / 8), d = c % (DK / 8), key = tile * KT + r;
                const bool ok = key < T && d * 8 < p.k_ld;
                cp_async16(ks + r * KS + d * 16, K + (ok ? (size_t)key * p.k_ld + d * 8 : 0), ok);
            }
            for (unsigned int c = threadIdx.x; c < KT * (DV / 8); c += 32 * AT_WARPS)
            {
                const unsigned int r = c / (DV / 8), d = c % (DV / 8), key = tile * KT + r;
                const bool ok = key < T && d * 8 < p.v_ld;
                cp_async16(vs + r * VS + d * 16, V + (ok ? (size_t)key * p.v_ld + d * 8 : 0), ok);
            }
        }
        cp_async_commit();
    };
    fetch(begin);
    const float scale2 = p.scale * 1.44269504088896341f;
    for (unsigned int tile = begin; tile < tiles; tile++)
    {
        fetch(tile + 1);
        cp_async_wait<1>();
        __syncthreads();
        if (tile * KT < last_lim && (tile + 1) * KT > first_low)
        {
            const uint32_t ks = ring + (tile & 1u) * TB;
            w.template step<KT>(ks, ks + KT * KS, tile * KT, low, lim, (tile + 1) * KT > first_lim || tile * KT < last_low, scale2, p.dim, p.vdim, lane);
        }
        __syncthreads();
    }
    w.finish();
    const unsigned int gr = lane >> 2, gc = (lane & 3) * 2;
#pragma unroll
    for (int h = 0; h < 2; h++)
    {
        const unsigned int r = r0 + gr + 8 * h;
        if (r < rows)
        {
            float l = w.l[h];
            if (p.sink != nullptr) { l += exp2f(p.sink[kvh * p.G + r % p.G] * 1.44269504088896341f - w.m[h]); }
            const float inv = 1.0f / l;
#pragma unroll
            for (int d = 0; d < DV / 8; d++)
            {
#pragma unroll
                for (int j = 0; j < 2; j++)
                {
                    const unsigned int c = d * 8 + gc + j;
                    if (c < p.vdim) { attention_store(p, qkvg, start, kvh, r, c, w.o[d][2 * h + j] * inv); }
                }
            }
        }
    }
}

template <int DK, int DV>
int run_attention_split(const AttnParams& p, unsigned int entries, cudaStream_t stream, bool pdl)
{
    return launch_kernel("attention_split", attention_split_kernel<DK, DV>, dim3(p.splits, p.Hkv * p.row_tiles, entries), dim3(32 * AS_WARPS),
        (size_t)as_smem(DK, DV), stream, pdl, p);
}
template <int DK, int DV>
int run_attention_tiled(const AttnParams& p, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl)
{
    const unsigned int tiles = (max_n * p.G + 16 * AT_WARPS - 1) / (16 * AT_WARPS);
    return launch_kernel("attention_tiled", attention_tiled_kernel<DK, DV>, dim3(tiles, p.Hkv, entries), dim3(32 * AT_WARPS), (size_t)at_smem(DK, DV),
        stream, pdl, p);
}

// One translation unit per padded key size (64, 128, 256) instantiates these.
template <int DK>
int attention_split_dk(const AttnParams& p, unsigned int entries, cudaStream_t stream, bool pdl);
template <int DK>
int attention_tiled_dk(const AttnParams& p, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl);

#define B200_ATTENTION_DK(DK)                                                                                                       \
    template <>                                                                                                                     \
    int attention_split_dk<DK>(const AttnParams& p, unsigned int entries, cudaStream_t stream, bool pdl)                            \
    {                                                                                                                               \
        if (p.vdim <= 64) { return run_attention_split<DK, 64>(p, entries, stream, pdl); }                                          \
        if (p.vdim <= 128) { return run_attention_split<DK, 128>(p, entries, stream, pdl); }                                        \
        return run_attention_split<DK, 256>(p, entries, stream, pdl);                                                               \
    }                                                                                                                               \
    template <>                                                                                                                     \
    int attention_tiled_dk<DK>(const AttnParams& p, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl)        \
    {                                                                                                                               \
        if (p.vdim <= 64) { return run_attention_tiled<DK, 64>(p, entries, max_n, stream, pdl); }                                   \
        if (p.vdim <= 128) { return run_attention_tiled<DK, 128>(p, entries, max_n, stream, pdl); }                                 \
        return run_attention_tiled<DK, 256>(p, entries, max_n, stream, pdl);                                                        \
    }

}    // namespace b200
