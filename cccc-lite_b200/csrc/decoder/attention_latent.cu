// BF16 attention of few query rows over latent rows: one key/value head for all query heads, whose values are the first columns
// of the key rows, so that a cache row is read once for both products.
//
// A CTA holds 32 query rows (a row is one head of one token) against a split of the sequence, in tiles of 64 rows that arrive
// through cp.async, two deep.  Scores: sixteen warps share 4 quarters of the row elements x 2 x 16 query rows x 2 x 32 keys,
// their queries as fragments in registers; the quarters meet in shared memory.  Softmax: sixteen threads per query row, running
// maximum; the weights enter the value product as the sum of two BF16 numbers.  Values: a warp owns a sixteenth of the columns.
// Partial results of the splits are combined by a second kernel, in split order.
#include "attention_mma.cuh"

namespace b200
{

constexpr int AL_WARPS = 16, AL_THREADS = 32 * AL_WARPS, AL_ROWS = 32, AL_KT = 64, AL_PARTS = 4, AL_SS = AL_KT + 4, AL_PS = AL_KT + 8;
__host__ __device__ constexpr int al_stride(int dv) { return dv + 64 + 8; }    // elements of a shared row
// queries, then in their place partial scores and weights
__host__ __device__ constexpr int al_front(int dv)
{
    const int q = AL_ROWS * al_stride(dv) * 2, s = AL_PARTS * AL_ROWS * AL_SS * 4 + 2 * AL_ROWS * AL_PS * 2;
    return q > s ? q : s;
}
__host__ __device__ constexpr int al_smem(int dv) { return al_front(dv) + 2 * AL_KT * al_stride(dv) * 2; }

__device__ __forceinline__ void ldmatrix_x2_trans(uint32_t (&r)[4], uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}

__device__ __forceinline__ unsigned int al_value_ld(const AttnParams& p) { return (p.vdim + 15) / 16 * 16; }
// partial result of a (unit, split): maximum and sum of every row, then the rows
__device__ __forceinline__ float* al_partial(const AttnParams& p, unsigned int unit, unsigned int split)
{
    return p.partial + ((size_t)unit * p.splits + split) * AL_ROWS * (al_value_ld(p) + 2);
}

// grid (splits, row tiles, entries)
template <int DV>
__global__ void __launch_bounds__(AL_THREADS, 1) attention_latent_kernel(const AttnParams p)
{
    extern __shared__ __align__(16) unsigned char al_raw[];
    // k steps of a warp, column tiles of 8 per warp, in pairs
    constexpr int DK = DV + 64, KS = al_stride(DV) * 2, STEPS = DK / 64, CT = DV / 128, CP = CT > 1 ? CT / 2 : 1;
    __shared__ float corr[AL_ROWS], ml[AL_ROWS][2];
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, gc = (lane & 3) * 2;
    const unsigned int split = blockIdx.x, rt = blockIdx.y, e = p.e0 + blockIdx.z;
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], pos = (unsigned int)p.pos[e], rows = n * p.G, r0 = rt * AL_ROWS;
    if (r0 >= rows) { return; }
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg;
    const __nv_bfloat16* K = (const __nv_bfloat16*)p.k_cache + (size_t)p.slot[e] * p.T_max * p.k_ld;
    const unsigned int last_row = min(r0 + AL_ROWS - 1u, rows - 1);
    const unsigned int T = min(pos + last_row / p.G + 1, p.T_max), begin = first_key(p, e, pos + r0 / p.G + 1) / AL_KT;
    const unsigned int tiles = (T + AL_KT - 1) / AL_KT, per = (tiles - begin + p.splits - 1) / p.splits;
    const unsigned int tile0 = min(begin + split * per, tiles), tile1 = min(tile0 + per, tiles);
    const uint32_t qs = smem_u32(al_raw), ks = qs + al_front(DV);
    float* sc = reinterpret_cast<float*>(al_raw);                                               // [part][row][key]
    __nv_bfloat16* pw = reinterpret_cast<__nv_bfloat16*>(sc + AL_PARTS * AL_ROWS * AL_SS);      // [high, low][row][key]
    auto fetch = [&](unsigned int tile) {
        if (tile < tile1)
        {
            const uint32_t dst = ks + (tile & 1u) * AL_KT * KS;
            const __nv_bfloat16* src = K + (size_t)tile * AL_KT * p.k_ld;
#pragma unroll
            for (int c = 0; c < AL_KT * (DK / 8) / AL_THREADS; c++)
            {
                const unsigned int at = tid + c * AL_THREADS, r = at / (DK / 8), d = at % (DK / 8);
                const bool ok = tile * AL_KT + r < T && d * 8 < p.k_ld;
                cp_async16(dst + r * KS + d * 16, src + (ok ? r * p.k_ld + d * 8 : 0u), ok);
            }
        }
        cp_async_commit();
    };
    // a tile's lines on their way to L2
    auto prefetch = [&](unsigned int tile) {
        if (tile < tile1 && (tile + 1) * AL_KT <= T)
        {
            const char* src = reinterpret_cast<const char*>(K + (size_t)tile * AL_KT * p.k_ld);
            for (unsigned int line = tid; line * 128 < AL_KT * p.k_ld * 2; line += AL_THREADS) { asm volatile("prefetch.global.L2 [%0];" ::"l"(src + line * 128)); }
        }
    };
    if ((p.q_ld % 8) == 0 && (p.ld % 8) == 0)
    {
        for (unsigned int c = tid; c < AL_ROWS * (DK / 8); c += AL_THREADS)
        {
            const unsigned int r = c / (DK / 8), d = c % (DK / 8), row = r0 + r;
            const bool ok = row < rows && d * 8 < p.q_ld;
            cp_async16(qs + r * KS + d * 16, x + (ok ? (size_t)(start + row / p.G) * p.ld + (size_t)(row % p.G) * p.q_ld + d * 8 : 0), ok);
        }
    }
    else
    {
        for (unsigned int j = tid; j < AL_ROWS * DK; j += AL_THREADS)
        {
            const unsigned int r = j / DK, d = j % DK, row = r0 + r;
            __nv_bfloat16 v = __float2bfloat16_rn(0.f);
            if (row < rows && d < p.dim) { v = x[(size_t)(start + row / p.G) * p.ld + (size_t)(row % p.G) * p.q_ld + d]; }
            reinterpret_cast<__nv_bfloat16*>(al_raw)[r * al_stride(DV) + d] = v;
        }
    }
    cp_async_commit();
    fetch(tile0);
    prefetch(tile0 + 1);
    cp_async_wait<1>();
    __syncthreads();
    // scores: this warp's quarter of the elements, query rows, keys
    const unsigned int part = warp >> 2, mr = (warp >> 1) & 1u, kg = warp & 1u;
    uint32_t q[STEPS][4];
    {
        const uint32_t qa = qs + (mr * 16 + (lane & 15)) * KS + (lane >> 4) * 16 + part * STEPS * 32;
#pragma unroll
        for (int i = 0; i < STEPS; i++) { ldmatrix_x4(q[i], qa + i * 32); }
    }
    const uint32_t kb = (kg * 32 + (lane & 7) + ((lane >> 4) << 3)) * KS + ((lane >> 3) & 1) * 16 + part * STEPS * 32;
    // softmax: query row tid / 16, keys tid % 16 + 16 j
    const unsigned int sr = tid >> 4, sk = tid & 15u, end = pos + (r0 + sr) / p.G + 1;
    const bool real = r0 + sr < rows;
    const unsigned int low = first_key(p, e, end), lim = real ? min(end, T) : 0u;
    const float scale2 = p.scale * 1.44269504088896341f;
    float m = -INFINITY, l = 0.f;
    // values
    const uint32_t vb = (lane & 15) * KS + (CT > 1 ? (lane >> 4) * 16 : 0u) + warp * CT * 16;
    const uint32_t pa = smem_u32(pw) + (lane & 15) * (AL_PS * 2) + (lane >> 4) * 16;
    float o[2][CT][4];
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
#pragma unroll
        for (int j = 0; j < CT; j++)
        {
#pragma unroll
            for (int k = 0; k < 4; k++) { o[i][j][k] = 0.f; }
        }
    }
    for (unsigned int tile = tile0; tile < tile1; tile++)
    {
        cp_async_wait<0>();
        __syncthreads();
        fetch(tile + 1);
        prefetch(tile + 2);
        const uint32_t at = ks + (tile & 1u) * AL_KT * KS;
        {
            float s[4][4];
#pragma unroll
            for (int i = 0; i < 4; i++)
            {
#pragma unroll
                for (int j = 0; j < 4; j++) { s[i][j] = 0.f; }
            }
#pragma unroll
            for (int i = 0; i < STEPS; i++)
            {
#pragma unroll
                for (int j = 0; j < 2; j++)
                {
                    uint32_t b[4];
                    ldmatrix_x4(b, at + kb + j * 16 * KS + i * 32);
                    mma_bf16_16816(s[2 * j], q[i][0], q[i][1], q[i][2], q[i][3], b[0], b[1]);
                    mma_bf16_16816(s[2 * j + 1], q[i][0], q[i][1], q[i][2], q[i][3], b[2], b[3]);
                }
            }
            float* dst = sc + (part * AL_ROWS + mr * 16 + gr) * AL_SS + kg * 32 + gc;
#pragma unroll
            for (int i = 0; i < 4; i++)
            {
                *reinterpret_cast<float2*>(dst + i * 8) = make_float2(s[i][0], s[i][1]);
                *reinterpret_cast<float2*>(dst + 8 * AL_SS + i * 8) = make_float2(s[i][2], s[i][3]);
            }
        }
        __syncthreads();
        {
            float z[4], mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                const unsigned int key = tile * AL_KT + sk + 16 * j;
                const float* src = sc + sr * AL_SS + sk + 16 * j;
                z[j] = ((src[0] + src[AL_ROWS * AL_SS]) + (src[2 * AL_ROWS * AL_SS] + src[3 * AL_ROWS * AL_SS])) * scale2;
                if (key < low || key >= lim) { z[j] = -INFINITY; }
                mx = fmaxf(mx, z[j]);
            }
#pragma unroll
            for (int i = 1; i < 16; i *= 2) { mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, i)); }
            const float mn = fmaxf(m, mx), base = mn == -INFINITY ? 0.f : mn, c = exp2f(m - base);
            m = mn;
            l *= c;
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                const float w = exp2f(z[j] - base);
                l += w;
                const __nv_bfloat16 hi = __float2bfloat16_rn(w);
                pw[sr * AL_PS + sk + 16 * j] = hi;
                pw[(AL_ROWS + sr) * AL_PS + sk + 16 * j] = __float2bfloat16_rn(w - __bfloat162float(hi));
            }
            if (sk == 0) { corr[sr] = c; }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; i++)
        {
            const float c0 = corr[i * 16 + gr], c1 = corr[i * 16 + gr + 8];
#pragma unroll
            for (int j = 0; j < CT; j++)
            {
                o[i][j][0] *= c0;
                o[i][j][1] *= c0;
                o[i][j][2] *= c1;
                o[i][j][3] *= c1;
            }
        }
#pragma unroll
        for (int k = 0; k < AL_KT / 16; k++)
        {
            uint32_t b[CP][4];
#pragma unroll
            for (int j = 0; j < CP; j++)
            {
                if constexpr (CT > 1) { ldmatrix_x4_trans(b[j], at + vb + k * 16 * KS + j * 32); }
                else { ldmatrix_x2_trans(b[j], at + vb + k * 16 * KS); }
            }
#pragma unroll
            for (int i = 0; i < 2; i++)
            {
#pragma unroll
                for (int low = 0; low < 2; low++)
                {
                    uint32_t w[4];
                    ldmatrix_x4(w, pa + (low * AL_ROWS + i * 16) * (AL_PS * 2) + k * 32);
#pragma unroll
                    for (int j = 0; j < CP; j++)
                    {
                        mma_bf16_16816(o[i][2 * j], w[0], w[1], w[2], w[3], b[j][0], b[j][1]);
                        if constexpr (CT > 1) { mma_bf16_16816(o[i][2 * j + 1], w[0], w[1], w[2], w[3], b[j][2], b[j][3]); }
                    }
                }
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int i = 1; i < 16; i *= 2) { l += __shfl_xor_sync(0xFFFFFFFFu, l, i); }
    if (sk == 0)
    {
        if (p.splits == 1 && p.sink != nullptr && real) { l += exp2f(p.sink[(r0 + sr) % p.G] * 1.44269504088896341f - m); }
        ml[sr][0] = m;
        ml[sr][1] = l;
    }
    __syncthreads();
    const unsigned int vl = al_value_ld(p);
    float* mine = al_partial(p, blockIdx.z * gridDim.y + rt, split);
    if (p.splits > 1 && tid < AL_ROWS)
    {
        mine[2 * tid] = ml[tid][0];
        mine[2 * tid + 1] = ml[tid][1];
    }
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
#pragma unroll
        for (int hf = 0; hf < 2; hf++)
        {
            const unsigned int r = i * 16 + gr + 8 * hf;
            if (r0 + r >= rows) { continue; }
            const float inv = 1.0f / ml[r][1];
#pragma unroll
            for (int j = 0; j < CT; j++)
            {
                const unsigned int d = (warp * CT + j) * 8 + gc;
                if (p.splits > 1)
                {
                    if (d < vl) { *reinterpret_cast<float2*>(mine + 2 * AL_ROWS + (size_t)r * vl + d) = make_float2(o[i][j][2 * hf], o[i][j][2 * hf + 1]); }
                    continue;
                }
                if (d < p.vdim) { attention_store(p, x, start, 0, r0 + r, d, o[i][j][2 * hf] * inv); }
                if (d + 1 < p.vdim) { attention_store(p, x, start, 0, r0 + r, d + 1, o[i][j][2 * hf + 1] * inv); }
            }
        }
    }
}

// grid (rows of a tile, row tiles, entries); a thread per four columns
__global__ void __launch_bounds__(128) attention_latent_combine_kernel(const AttnParams p)
{
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int lane = threadIdx.x & 31, r = blockIdx.x, rt = blockIdx.y, e = p.e0 + blockIdx.z;
    const unsigned int row = rt * AL_ROWS + r, rows = (unsigned int)p.n[e] * p.G, start = (unsigned int)p.start[e], vl = al_value_ld(p);
    if (row >= rows) { return; }
    const unsigned int d = 4 * threadIdx.x;
    const float* first = al_partial(p, blockIdx.z * gridDim.y + rt, 0);
    const size_t step = (size_t)AL_ROWS * (vl + 2);
    float m = -INFINITY, l = 0.f;
    if (lane < p.splits)
    {
        m = __ldcg(first + lane * step + 2 * r);
        l = __ldcg(first + lane * step + 2 * r + 1);
    }
    float top = m;
#pragma unroll
    for (int i = 16; i > 0; i >>= 1) { top = fmaxf(top, __shfl_xor_sync(0xFFFFFFFFu, top, i)); }
    const float c = exp2f(m - top);
    l = warp_sum(c * l);
    if (p.sink != nullptr) { l += exp2f(p.sink[row % p.G] * 1.44269504088896341f - top); }
    const float weight = c / l;
    const float* src = first + 2 * AL_ROWS + (size_t)r * vl + (d < vl ? d : 0u);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (unsigned int s = 0; s < p.splits; s++)
    {
        const float4 y = __ldcg(reinterpret_cast<const float4*>(src + s * step));
        const float w = __shfl_sync(0xFFFFFFFFu, weight, s);
        o.x = fmaf(w, y.x, o.x);
        o.y = fmaf(w, y.y, o.y);
        o.z = fmaf(w, y.z, o.z);
        o.w = fmaf(w, y.w, o.w);
    }
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg;
    const float out[4] = { o.x, o.y, o.z, o.w };
#pragma unroll
    for (int i = 0; i < 4; i++)
    {
        if (d + i < p.vdim) { attention_store(p, x, start, 0, row, d + i, out[i]); }
    }
}

int launch_attention_latent(const AttnParams& p0, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream, bool pdl)
{
    AttnParams p = p0;
    const DecoderDevice* dev = decoder_device();
    if (!dev) { return 1; }
    const unsigned int row_tiles = (max_n * p.G + AL_ROWS - 1) / AL_ROWS;
    if (p.Hkv != 1 || p.k_cache != p.v_cache || p.k_ld != p.v_ld || p.dim > 576 || p.vdim > 512 || (p.k_ld % 8) || row_tiles > 65535u || entries > 65535u)
    {
        return -1;
    }
    if (p.window != 0 && max_len > p.window + max_n) { max_len = p.window + max_n; }
    const unsigned long long units = (unsigned long long)entries * row_tiles;
    const unsigned int tiles = (max_len + AL_KT - 1) / AL_KT + (p.window != 0 ? 1 : 0);
    // the fewest tiles in a row, over all waves of CTAs; a split costs its start and the combining
    double best = 1e30;
    p.splits = 1;
    for (unsigned int s = 1; s <= kMaxSplits && (s == 1 || (units * s * 2 <= kAttnPartials && s <= tiles)); s++)
    {
        const double waves = (double)((units * s + dev->sm_count - 1) / dev->sm_count);
        const double t = waves * ((double)((tiles + s - 1) / s) + 1.0) + (s > 1 ? 1.0 + 0.03 * s : 0.0);
        if (t < best)
        {
            best = t;
            p.splits = s;
        }
    }
    const dim3 grid(p.splits, row_tiles, entries);
    int rc;
    if (p.vdim <= 128 && p.dim <= 192) { rc = launch_kernel("attention_latent", attention_latent_kernel<128>, grid, dim3(AL_THREADS), (size_t)al_smem(128), stream, pdl, p); }
    else if (p.vdim <= 256 && p.dim <= 320) { rc = launch_kernel("attention_latent", attention_latent_kernel<256>, grid, dim3(AL_THREADS), (size_t)al_smem(256), stream, pdl, p); }
    else { rc = launch_kernel("attention_latent", attention_latent_kernel<512>, grid, dim3(AL_THREADS), (size_t)al_smem(512), stream, pdl, p); }
    if (rc || p.splits == 1) { return rc; }
    return launch_kernel("attention_latent_combine", attention_latent_combine_kernel, dim3(AL_ROWS, row_tiles, entries), dim3(128), 0, stream, pdl, p);
}

}    // namespace b200
