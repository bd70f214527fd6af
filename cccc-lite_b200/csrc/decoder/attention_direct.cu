// BF16 attention of few query rows (decoding), HBM-bound: keys and values go from global memory straight into the
// fragments of mma.m16n8k16, no shared memory in between.
//
// A warp holds up to 8 (or 16) query rows and walks 16-key tiles.  Scores: a lane reads 32 bytes of key row lane / 4, the
// four lanes of a row 64 consecutive elements; the order of the elements inside the product is permuted, alike for
// the queries.  Values: lane (g, t) reads the columns g * DV / 8 ... of the rows 2t, 2t + 1, 2t + 8, 2t + 9, so that a warp
// reads whole rows and a register pair becomes a fragment with one byte permute; which columns a fragment's n stands
// for is permuted in turn, and undone when the result is stored.  The next tile's keys are requested as soon as the scores
// are out, its values as soon as the value product is.  Softmax weights enter the value product as the sum of two BF16 numbers.
// Decoding steps (one token per sequence) are fused: the CTA whose split holds the new position brings its key to unit
// RMS, mixes its value and appends both; every CTA brings its own queries to unit RMS.
#include "attention_mma.cuh"

namespace b200
{

__device__ __forceinline__ void ldg32(const void* p, uint32_t (&r)[8], bool ok)
{
#pragma unroll
    for (int i = 0; i < 8; i++) { r[i] = 0u; }
    if (ok)
    {
        asm volatile("ld.global.v8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                     : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                     : "l"(p)
                     : "memory");
    }
}
__device__ __forceinline__ void ldg16(const void* p, uint32_t (&r)[4], bool ok)
{
#pragma unroll
    for (int i = 0; i < 4; i++) { r[i] = 0u; }
    if (ok) { asm volatile("ld.global.v4.b32 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "l"(p) : "memory"); }
}

// rows 8-15 of the fragment do not exist: their inputs and results are zero
__device__ __forceinline__ void mma_bf16_top(float& c0, float& c1, uint32_t a0, uint32_t a2, uint32_t b0, uint32_t b1)
{
    [[maybe_unused]] float d2, d3;
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%5}, {%7,%8}, {%0,%1,%9,%9};"
        : "+f"(c0), "+f"(c1), "=f"(d2), "=f"(d3)
        : "r"(a0), "r"(0u), "r"(a2), "r"(b0), "r"(b1), "f"(0.f));
}

// grid (splits, Hkv * row_tiles, entries)
template <int DK, int DV, int NR>    // NR: row groups of eight (1 or 2)
__global__ void __launch_bounds__(32 * AS_WARPS, NR == 1 && DK + DV < 256 ? 3 : 2) attention_direct_kernel(const AttnParams p)
{
    constexpr int RT = 8 * NR, KB = DK / 64, C = DV / 8, VR = C / 2;    // VR: registers of a value row per lane
    __shared__ float om[AS_WARPS * RT * DV];
    __shared__ SplitMeet meet;
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const unsigned int split = blockIdx.x, kvh = blockIdx.y % p.Hkv, rt = blockIdx.y / p.Hkv, e = p.e0 + blockIdx.z;
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], pos = (unsigned int)p.pos[e], r0 = rt * RT;
    const unsigned int rows = n * p.G;
    if (r0 >= rows) { return; }
    const __nv_bfloat16* qkvg = (const __nv_bfloat16*)p.qkvg;
    const size_t seq = ((size_t)p.slot[e] * p.Hkv + kvh) * p.T_max;
    __nv_bfloat16* K = (__nv_bfloat16*)p.k_cache + seq * p.k_ld;
    __nv_bfloat16* V = (__nv_bfloat16*)p.v_cache + seq * p.v_ld;
    const unsigned int last_row = min(r0 + RT - 1u, rows - 1);
    const unsigned int T = min(pos + last_row / p.G + 1, p.T_max);
    const unsigned int first_lim = pos + r0 / p.G + 1, last_low = first_key(p, e, pos + last_row / p.G + 1);
    const unsigned int begin = first_key(p, e, first_lim) / 16;
    const unsigned int tiles = (T + 15) / 16, per = (tiles - begin + p.splits - 1) / p.splits;
    const unsigned int tile0 = min(begin + split * per, tiles), tile1 = min(tile0 + per, tiles);

    uint32_t k[2][KB][8], v[4][VR];
    auto load_k = [&](unsigned int tile) {
#pragma unroll
        for (int i = 0; i < 2; i++)
        {
            const unsigned int key = tile * 16 + i * 8 + g;
#pragma unroll
            for (int b = 0; b < KB; b++)
            {
                const unsigned int d = b * 64 + t * 16;
                ldg32(K + (size_t)key * p.k_ld + d, k[i][b], tile < tile1 && key < T && d < p.k_ld);
            }
        }
    };
    auto load_v = [&](unsigned int tile) {
#pragma unroll
        for (int i = 0; i < 4; i++)
        {
            const unsigned int key = tile * 16 + 2 * t + (i & 1) + (i >> 1) * 8, d = g * C;
            const bool ok = tile < tile1 && key < T && d < p.v_ld;
            if constexpr (VR == 8) { ldg32(V + (size_t)key * p.v_ld + d, v[i], ok); }
            else { ldg16(V + (size_t)key * p.v_ld + d, v[i], ok); }
        }
    };
    // Two tiles ahead of the registers, whole lines on their way to L2.
    auto prefetch = [&](unsigned int tile) {
        if (tile < tile1)
        {
            const unsigned int kl = p.k_ld * 32, vl = p.v_ld * 32;    // bytes of a tile
            const char* kp = reinterpret_cast<const char*>(K + (size_t)tile * 16 * p.k_ld) + lane * 128;
            const char* vp = reinterpret_cast<const char*>(V + (size_t)tile * 16 * p.v_ld) + lane * 128;
            if (lane * 128 < kl && (tile + 1) * 16 <= T) { asm volatile("prefetch.global.L2 [%0];" ::"l"(kp)); }
            if (lane * 128 < vl && (tile + 1) * 16 <= T) { asm volatile("prefetch.global.L2 [%0];" ::"l"(vp)); }
        }
    };
    // the step's own row is in the cache only after the append below
    const bool owner = p.fused && pos < p.T_max && pos / 16 >= tile0 && pos / 16 < tile1;
    const bool late = owner && tile0 + warp == pos / 16;
    if (!late)
    {
        load_k(tile0 + warp);
        load_v(tile0 + warp);
    }
    prefetch(tile0 + warp + AS_WARPS);
    prefetch(tile0 + warp + 2 * AS_WARPS);
    // (every row tile of the unit writes the same values: its own reads come after them)
    if (owner)
    {
        const __nv_bfloat16* x = qkvg + (size_t)start * p.ld;
        if (warp == 0)
        {
            const __nv_bfloat16* src = x + p.k_off + (size_t)kvh * p.dim;
            float inv = 1.f;
            if (p.qk_norm)
            {
                float sq = 0.f;
                for (unsigned int d = lane; d < p.dim; d += 32)
                {
                    const float v = __bfloat162float(src[d]);
                    sq += v * v;
                }
                inv = 1.0f / sqrtf(warp_sum(sq) / (float)p.dim + p.eps);
            }
            for (unsigned int d = lane; d < p.dim; d += 32) { K[(size_t)pos * p.k_ld + d] = __float2bfloat16_rn(__bfloat162float(src[d]) * inv); }
        }
        else if (warp == 1)
        {
            const __nv_bfloat16* src = x + p.v_off + (size_t)kvh * p.vdim;
            __nv_bfloat16* first = p.v_mix ? (__nv_bfloat16*)p.v_first + (size_t)start * p.v_first_ld + (size_t)kvh * p.vdim : nullptr;
            for (unsigned int d = lane; d < p.vdim; d += 32)
            {
                float v = __bfloat162float(src[d]);
                if (p.v_mix == 1) { first[d] = src[d]; }
                else if (p.v_mix == 2) { v = (1.0f - p.lambda) * v + p.lambda * __bfloat162float(first[d]); }
                V[(size_t)pos * p.v_ld + d] = __float2bfloat16_rn(v);
            }
        }
        __syncthreads();
    }

    if (late)
    {
        load_k(tile0 + warp);
        load_v(tile0 + warp);
    }

    // queries: the same permuted element order as the keys
    uint32_t q[NR][KB][8];
    unsigned int low[NR], lim[NR];
#pragma unroll
    for (int h = 0; h < NR; h++)
    {
        const unsigned int r = r0 + g + 8 * h;
        const bool ok = r < rows;
        const unsigned int rr = ok ? r : 0;
        const __nv_bfloat16* src = qkvg + (size_t)(start + rr / p.G) * p.ld + (size_t)(kvh * p.G + rr % p.G) * p.q_ld;
        low[h] = first_key(p, e, pos + r / p.G + 1);
        lim[h] = min(pos + r / p.G + 1, T);
        float f[KB][16], sq = 0.f;
#pragma unroll
        for (int b = 0; b < KB; b++)
        {
            const unsigned int d0 = b * 64 + t * 16;
            if ((p.dim % 16) == 0 && (p.q_ld % 16) == 0)
            {
                uint32_t x[8];
                ldg32(src + d0, x, ok && d0 < p.dim);
#pragma unroll
                for (int j = 0; j < 8; j++)
                {
                    f[b][2 * j] = __uint_as_float(x[j] << 16);
                    f[b][2 * j + 1] = __uint_as_float(x[j] & 0xFFFF0000u);
                }
            }
            else
            {
#pragma unroll
                for (int j = 0; j < 16; j++) { f[b][j] = ok && d0 + j < p.dim ? __bfloat162float(src[d0 + j]) : 0.f; }
            }
#pragma unroll
            for (int j = 0; j < 16; j++) { sq += f[b][j] * f[b][j]; }
        }
        float inv = 1.f;
        if (p.fused && p.qk_norm)
        {
            sq += __shfl_xor_sync(0xFFFFFFFFu, sq, 1);
            sq += __shfl_xor_sync(0xFFFFFFFFu, sq, 2);
            inv = 1.0f / sqrtf(sq / (float)p.dim + p.eps);
        }
#pragma unroll
        for (int b = 0; b < KB; b++)
        {
#pragma unroll
            for (int j = 0; j < 8; j++) { q[h][b][j] = pack_bf16x2(f[b][2 * j] * inv, f[b][2 * j + 1] * inv); }
        }
    }

    float o[C][2 * NR], m[NR], l[NR];
#pragma unroll
    for (int h = 0; h < NR; h++)
    {
        m[h] = -INFINITY;
        l[h] = 0.f;
    }
#pragma unroll
    for (int j = 0; j < C; j++)
    {
#pragma unroll
        for (int i = 0; i < 2 * NR; i++) { o[j][i] = 0.f; }
    }
    const float scale2 = p.scale * 1.44269504088896341f;
    for (unsigned int tile = tile0 + warp; tile < tile1; tile += AS_WARPS)
    {
        float s[2][2 * NR];
#pragma unroll
        for (int i = 0; i < 2; i++)
        {
#pragma unroll
            for (int j = 0; j < 2 * NR; j++) { s[i][j] = 0.f; }
#pragma unroll
            for (int b = 0; b < KB; b++)
            {
#pragma unroll
                for (int x = 0; x < 4; x++)
                {
                    if constexpr (NR == 1) { mma_bf16_top(s[i][0], s[i][1], q[0][b][2 * x], q[0][b][2 * x + 1], k[i][b][2 * x], k[i][b][2 * x + 1]); }
                    else
                    {
                        mma_bf16_16816(s[i], q[0][b][2 * x], q[NR - 1][b][2 * x], q[0][b][2 * x + 1], q[NR - 1][b][2 * x + 1], k[i][b][2 * x],
                            k[i][b][2 * x + 1]);
                    }
                }
            }
        }
        load_k(tile + AS_WARPS);
        prefetch(tile + 3 * AS_WARPS);
        const bool masked = (tile + 1) * 16 > first_lim || tile * 16 < last_low;
        uint32_t hi[2 * NR], lo[2 * NR];    // [key half][row group]
#pragma unroll
        for (int h = 0; h < NR; h++)
        {
            float mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < 2; i++)
            {
#pragma unroll
                for (int j = 0; j < 2; j++)
                {
                    float& z = s[i][2 * h + j];
                    z *= scale2;
                    const unsigned int key = tile * 16 + i * 8 + 2 * t + j;
                    if (masked && (key < low[h] || key >= lim[h])) { z = -INFINITY; }
                    mx = fmaxf(mx, z);
                }
            }
            mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, 2));
            const float mn = fmaxf(m[h], mx), base = mn == -INFINITY ? 0.f : mn;
            if (__any_sync(0xFFFFFFFFu, mn > m[h]))
            {
                const float c = exp2f(m[h] - base);
                m[h] = mn;
                l[h] *= c;
#pragma unroll
                for (int j = 0; j < C; j++)
                {
                    o[j][2 * h] *= c;
                    o[j][2 * h + 1] *= c;
                }
            }
#pragma unroll
            for (int i = 0; i < 2; i++)
            {
                const float p0 = exp2f(s[i][2 * h] - base), p1 = exp2f(s[i][2 * h + 1] - base);
                l[h] += p0 + p1;
                const uint32_t u = pack_bf16x2(p0, p1);
                hi[i * NR + h] = u;
                lo[i * NR + h] = pack_bf16x2(p0 - __uint_as_float(u << 16), p1 - __uint_as_float(u & 0xFFFF0000u));
            }
        }
#pragma unroll
        for (int j = 0; j < C; j++)
        {
            const uint32_t sel = (j & 1) ? 0x7632u : 0x5410u;
            const uint32_t b0 = prmt(v[0][j / 2], v[1][j / 2], sel), b1 = prmt(v[2][j / 2], v[3][j / 2], sel);
            if constexpr (NR == 1)
            {
                mma_bf16_top(o[j][0], o[j][1], hi[0], hi[1], b0, b1);
                mma_bf16_top(o[j][0], o[j][1], lo[0], lo[1], b0, b1);
            }
            else
            {
                mma_bf16_16816(o[j], hi[0], hi[NR - 1], hi[NR], hi[2 * NR - 1], b0, b1);
                mma_bf16_16816(o[j], lo[0], lo[NR - 1], lo[NR], lo[2 * NR - 1], b0, b1);
            }
        }
        load_v(tile + AS_WARPS);
    }
    // n index 2t (+ 1) of fragment j is column (2t (+ 1)) * C + j
#pragma unroll
    for (int h = 0; h < NR; h++)
    {
        l[h] += __shfl_xor_sync(0xFFFFFFFFu, l[h], 1);
        l[h] += __shfl_xor_sync(0xFFFFFFFFu, l[h], 2);
        float* dst = om + (warp * RT + g + 8 * h) * DV + 2 * t * C;
#pragma unroll
        for (int j = 0; j < C; j++)
        {
            dst[j] = o[j][2 * h];
            dst[C + j] = o[j][2 * h + 1];
        }
        if (t == 0)
        {
            meet.ml[warp][g + 8 * h][0] = m[h];
            meet.ml[warp][g + 8 * h][1] = l[h];
        }
    }
    split_finish<DV, RT>(p, meet, om, qkvg, e, start, kvh, rt, r0, rows);
}

template <int DK, int DV>
static int run_direct(const AttnParams& p, unsigned int entries, unsigned int nr, cudaStream_t stream, bool pdl)
{
    const dim3 grid(p.splits, p.Hkv * p.row_tiles, entries);
    return nr == 1 ? launch_kernel("attention_direct", attention_direct_kernel<DK, DV, 1>, grid, dim3(32 * AS_WARPS), 0, stream, pdl, p)
                   : launch_kernel("attention_direct", attention_direct_kernel<DK, DV, 2>, grid, dim3(32 * AS_WARPS), 0, stream, pdl, p);
}

int launch_attention_direct(const AttnParams& p0, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl)
{
    AttnParams p = p0;
    auto low = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 31u) != 0; };
    if (p.dim > 128 || p.vdim > 128 || (p.k_ld % 16) || (p.v_ld % 16) || low(p.k_cache) || low(p.v_cache) || low(p.qkvg) || (p.ld % 16) || entries > 65535u) { return -1; }
    const unsigned int nr = max_n * p.G <= 8 ? 1 : 2;
    p.row_tiles = (max_n * p.G + 8 * nr - 1) / (8 * nr);
    if ((unsigned long long)p.Hkv * p.row_tiles > 65535ull) { return -1; }
    if (!plan_splits(p, entries, max_n, max_len, nr == 1 && (p.dim <= 64 || p.vdim <= 64) ? 3 : 2)) { return 1; }
    if (p.dim <= 64) { return p.vdim <= 64 ? run_direct<64, 64>(p, entries, nr, stream, pdl) : run_direct<64, 128>(p, entries, nr, stream, pdl); }
    return p.vdim <= 64 ? run_direct<128, 64>(p, entries, nr, stream, pdl) : run_direct<128, 128>(p, entries, nr, stream, pdl);
}

}    // namespace b200
