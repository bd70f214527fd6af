// BF16 attention of few query rows over latent rows (decoding), HBM-bound, on tcgen05: one key/value head for all query heads, whose
// values are the first columns of the key rows, so that a cache row is read once for both products.
//
// A CTA holds 32 query rows (a row is one head of one token) against a split of the sequence, in tiles of 64 cache rows that a TMA
// lane fetches, two deep.  Both products are turned so that the 32 query rows are the short side: scores = K Q^T (64 x 32) and
// O^T += K^T P^T (128 latent columns x 32, the tile as an operand with its keys outermost).  Eight warps turn scores into weights:
// scores go through shared memory, eight threads then own a query row; the weights enter as the sum of two BF16 numbers.  The
// running maximum only moves when it grows by more than 2^8, so that O is seldom rescaled.  Partial results of the splits are
// combined by a second kernel, in split order.
// Every wait is bounded; on expiry the status word is raised, the roles drain, tensor memory is freed and the CTA returns.
#include "attention_mma.cuh"
#include "tile_common.cuh"

namespace b200
{

constexpr int AL_THREADS = 32 * 10, AL_ROWS = 32, AL_KT = 64, AL_SS = AL_KT + 4;
constexpr int AL_BLOCK = AL_KT * 128, AL_QBLOCK = AL_ROWS * 128;    // 64 elements of 64 cache rows, of 32 query rows
constexpr uint32_t AL_O = 64, AL_TMEM = 256;                          // columns: two places of scores, then O^T (32 for each 128 columns)
// 64-element blocks of a cache row: what the scores take, and what the value product touches
__host__ __device__ constexpr int al_key_blocks(int dim) { return (dim + 63) / 64; }
__host__ __device__ constexpr int al_blocks(int dim, int vdim)
{
    const int k = al_key_blocks(dim), v = 2 * ((vdim + 127) / 128);
    return k > v ? k : v;
}
__host__ __device__ constexpr int al_smem(int dim, int vdim)
{
    return 1024 + al_key_blocks(dim) * AL_QBLOCK + 2 * al_blocks(dim, vdim) * AL_BLOCK + 2 * AL_QBLOCK + AL_ROWS * AL_SS * 4 + 1024;
}

__device__ __forceinline__ unsigned int al_value_ld(const AttnParams& p) { return (p.vdim + 15) / 16 * 16; }
// partial result of a (unit, split): maximum and sum of every row, then the rows
__device__ __forceinline__ float* al_partial(const AttnParams& p, unsigned int unit, unsigned int split)
{
    return p.partial + ((size_t)unit * p.splits + split) * AL_ROWS * (al_value_ld(p) + 2);
}

// grid (splits, row tiles, entries)
__global__ void __launch_bounds__(AL_THREADS) attention_latent_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ AttnParams p,
    unsigned int* status)
{
    extern __shared__ unsigned char al_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(al_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ float corr[AL_ROWS], ml[AL_ROWS][2];
    // by parity of the tile, so that a warp may be a barrier ahead of another: does any row rescale, has any wait run out
    __shared__ int moved[2], stop[2];
    const int kblocks = al_key_blocks((int)p.dim), tile_bytes = al_blocks((int)p.dim, (int)p.vdim) * AL_BLOCK, vparts = ((int)p.vdim + 127) / 128;
    uint64_t* k_full = reinterpret_cast<uint64_t*>(smem);
    uint64_t *k_empty = k_full + 2, *s_full = k_full + 4, *q_ready = k_full + 6, *p_ready = k_full + 7, *pv_done = k_full + 8, *o_full = k_full + 9;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(k_full + 10);
    volatile unsigned int* abort_flag = reinterpret_cast<volatile unsigned int*>(tmem_slot + 1);
    unsigned char* ks = smem + 1024;
    unsigned char* qs = ks + 2 * tile_bytes;
    unsigned char* pw = qs + kblocks * AL_QBLOCK;                              // [high, low][row][key]
    float* sc = reinterpret_cast<float*>(pw + 2 * AL_QBLOCK);                  // [row][key]

    const unsigned int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const unsigned int split = blockIdx.x, rt = blockIdx.y, e = p.e0 + blockIdx.z;
    if (tid == 0)
    {
        for (int i = 0; i < 10; i++) { mbar_init(k_full + i, i == 6 || i == 7 ? 8 : 1); }
        *abort_flag = 0;
        moved[0] = moved[1] = stop[0] = stop[1] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) { tmem_alloc(tmem_slot, AL_TMEM); }
    grid_dependency_launch();
    // (the batch's arrays are written before the step's first launch)
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], pos = (unsigned int)p.pos[e], rows = n * p.G, r0 = rt * AL_ROWS;
    const bool idle = r0 >= rows;    // a shorter entry than the longest one
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg;
    const unsigned int last_row = idle ? 0 : min(r0 + AL_ROWS - 1u, rows - 1);
    const unsigned int T = idle ? 0 : min(pos + last_row / p.G + 1, p.T_max), begin = idle ? 0 : first_key(p, e, pos + r0 / p.G + 1) / AL_KT;
    const unsigned int all = (T + AL_KT - 1) / AL_KT, per = (all - begin + p.splits - 1) / p.splits;
    const unsigned int tile0 = min(begin + split * per, all), tiles = min(tile0 + per, all) - tile0;
    const int seq_row = (int)((unsigned int)p.slot[e] * p.T_max + tile0 * AL_KT);
    // tiles on their way to L2
    auto prefetch = [&](unsigned int t) {
        for (int b = 0; b < kblocks && t < tiles; b++)
        {
            asm volatile("cp.async.bulk.prefetch.tensor.2d.L2.global.tile [%0, {%1, %2}];" ::"l"(&tmK), "r"(b * 64), "r"(seq_row + (int)t * AL_KT) : "memory");
        }
    };
    if (tid == 0)
    {
        prefetch(0);
        prefetch(1);
    }
    grid_dependency_wait();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    auto give_up = [&](unsigned int role, unsigned int step) {
        note_timeout(status, WAIT_ATTENTION_LATENT, role, step);
        *abort_flag = 1;
    };
    auto wait = [&](uint64_t* bar, unsigned int parity) { return *abort_flag == 0 && mbar_wait_bounded(bar, parity & 1u); };

    if (warp == 0)
    {
        if (lane == 0)
        {
            unsigned int i = 0;
            bool ok = true;
            for (; i < tiles; i++)
            {
                const unsigned int s = i & 1u;
                if (i >= 2 && !wait(k_empty + s, (i >> 1) - 1)) { ok = false; break; }
                mbar_expect_tx(k_full + s, (unsigned int)kblocks * AL_BLOCK);
                for (int b = 0; b < kblocks; b++) { tma_load_2d(ks + s * tile_bytes + b * AL_BLOCK, &tmK, b * 64, seq_row + (int)i * AL_KT, k_full + s); }
                mbar_arrive(k_full + s);
                prefetch(i + 2);
            }
            if (!ok)
            {
                give_up(0, i);
                // wait (bounded) for the copies in flight before the CTA may leave
                for (unsigned int j = i > 2 ? i - 2 : 0; j < i; j++)
                {
                    const unsigned long long t = global_timer_ns();
                    while (!mbar_try_wait(k_full + (j & 1u), (j >> 1) & 1u) && global_timer_ns() - t < 100000ull) {}
                }
            }
        }
    }
    else if (warp == 1)
    {
        const uint32_t idesc_s = umma_idesc_bf16(AL_KT, AL_ROWS), idesc_o = umma_idesc_bf16(128, AL_ROWS) | (1u << 15);    // A has its keys outermost
        const uint32_t k_addr = smem_u32(ks);
        const uint64_t q_desc = umma_desc_kmajor_sw128(smem_u32(qs)), p_desc = umma_desc_kmajor_sw128(smem_u32(pw));
        const int steps = ((int)p.dim + 15) / 16;
        // whatever is ready first: the scores of a tile that has arrived, or the value product of one whose weights are there (the
        // scores two tiles on take the place of scores that have been read by then)
        unsigned int si = 0, i = 0;
        bool ok = tiles == 0 || wait(q_ready, 0);
        unsigned long long since = global_timer_ns();
        while (ok && i < tiles)
        {
            if (si < tiles && si < i + 2 && mbar_test(k_full + (si & 1u), (si >> 1) & 1u))
            {
                tc_fence_after();
                if (elect_one())
                {
                    uint64_t a = umma_desc_kmajor_sw128(k_addr + (si & 1u) * tile_bytes), b = q_desc;
                    for (int k0 = 0; k0 < steps; k0 += 4, a += AL_BLOCK >> 4, b += AL_QBLOCK >> 4)
                    {
#pragma unroll
                        for (int k = 0; k < 4; k++)
                        {
                            if (k0 + k < steps) { umma_bf16(tmem + (si & 1u) * AL_ROWS, a + k * 2, b + k * 2, idesc_s, (k0 | k) != 0 ? 1u : 0u); }
                        }
                    }
                    umma_commit(s_full + (si & 1u));
                }
                __syncwarp();
                si++;
                since = global_timer_ns();
                continue;
            }
            if (i < si && mbar_test(p_ready, i & 1u))
            {
                tc_fence_after();
                if (elect_one())
                {
                    uint64_t a = umma_desc_mnmajor_sw128(k_addr + (i & 1u) * tile_bytes);
                    for (int v = 0; v < vparts; v++, a += 2 * AL_BLOCK >> 4)
                    {
#pragma unroll
                        for (int part = 0; part < 2; part++)    // the high halves of the weights, then the low ones
                        {
#pragma unroll
                            for (int k = 0; k < AL_KT / 16; k++)
                            {
                                umma_bf16(tmem + AL_O + v * AL_ROWS, a + (k * 2048 >> 4), p_desc + (part * AL_QBLOCK + k * 32 >> 4), idesc_o,
                                    (i | (unsigned int)part | (unsigned int)k) != 0 ? 1u : 0u);
                            }
                        }
                    }
                    umma_commit(k_empty + (i & 1u));
                    umma_commit(pv_done);
                    if (i + 1 == tiles) { umma_commit(o_full); }
                }
                __syncwarp();
                i++;
                since = global_timer_ns();
                continue;
            }
            ok = __all_sync(0xFFFFFFFFu, *abort_flag == 0 && global_timer_ns() - since < kWaitLimitNs);
        }
        if (!ok)
        {
            if (lane == 0) { give_up(1, i); }
            if (elect_one()) { umma_commit(o_full); }    // completes once the MMAs in flight have stopped reading shared memory
            __syncwarp();
        }
    }
    else
    {
        const unsigned int st = tid - 64, sw = warp - 2, quarter = warp & 3u, side = sw >> 2;
        // queries in eights, four rows per warp
        if (!idle)
        {
            const bool vec = (p.q_ld % 8) == 0 && (p.ld % 8) == 0 && (p.dim % 8) == 0;
            uint4 u[4][3];
#pragma unroll
            for (unsigned int r = 0; r < 4; r++)
            {
                const unsigned int row = r0 + sw * 4 + r;
                const __nv_bfloat16* src = x + (size_t)(start + (row < rows ? row / p.G : 0u)) * p.ld + (size_t)(row < rows ? row % p.G : 0u) * p.q_ld;
#pragma unroll
                for (unsigned int j = 0; j < 3; j++)
                {
                    const unsigned int d = (lane + j * 32) * 8;
                    u[r][j] = make_uint4(0, 0, 0, 0);
                    if (row >= rows || d >= p.dim) { continue; }
                    if (vec) { u[r][j] = *reinterpret_cast<const uint4*>(src + d); }
                    else
                    {
                        uint32_t w[8];
#pragma unroll
                        for (int k = 0; k < 8; k++) { w[k] = d + k < p.dim ? __bfloat16_as_ushort(src[d + k]) : 0u; }
                        u[r][j] = make_uint4(w[0] | (w[1] << 16), w[2] | (w[3] << 16), w[4] | (w[5] << 16), w[6] | (w[7] << 16));
                    }
                }
            }
#pragma unroll
            for (unsigned int r = 0; r < 4; r++)
            {
#pragma unroll
                for (unsigned int j = 0; j < 3; j++)
                {
                    const unsigned int q = lane + j * 32, at = sw * 4 + r;
                    if (q < (unsigned int)kblocks * 8) { *reinterpret_cast<uint4*>(qs + (q / 8) * AL_QBLOCK + at * 128 + (((q % 8) ^ (at & 7u)) * 16)) = u[r][j]; }
                }
            }
        }
        fence_proxy_async();
        __syncwarp();
        if (lane == 0) { mbar_arrive(q_ready); }
        // softmax: query row st / 8, keys 8 (st % 8) ..
        const unsigned int sr = st >> 3, sk = st & 7u, end = pos + (r0 + sr) / p.G + 1;
        const bool real = r0 + sr < rows;
        const unsigned int low = first_key(p, e, end), lim = real ? min(end, T) : 0u;
        const float scale2 = p.scale * 1.44269504088896341f;
        const uint32_t lanes = tmem + ((quarter * 32u) << 16);
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        unsigned int i = 0;
        for (; i < tiles; i++)
        {
            ok = __all_sync(0xFFFFFFFFu, wait(s_full + (i & 1u), i >> 1));
            // sixteen keys per quarter of tensor memory; half of the query rows for each of its two warps
            if (ok)
            {
                tc_fence_after();
                uint32_t z[16];
                tmem_ld_32x16(lanes + (i & 1u) * AL_ROWS + side * 16, z);
                tmem_ld_wait();
                if (lane < 16)
                {
#pragma unroll
                    for (int j = 0; j < 16; j++) { sc[(side * 16 + j) * AL_SS + quarter * 16 + lane] = __uint_as_float(z[j]); }
                }
            }
            bar_sync_named(1, 256);    // also: every warp is past the tile before
            if (st == 0) { moved[(i + 1) & 1u] = 0; }
            float w[8], mx = -INFINITY;
            const unsigned int key0 = (tile0 + i) * AL_KT + sk * 8;
            const float4 z0 = *reinterpret_cast<const float4*>(sc + sr * AL_SS + sk * 8), z1 = *reinterpret_cast<const float4*>(sc + sr * AL_SS + sk * 8 + 4);
            w[0] = z0.x, w[1] = z0.y, w[2] = z0.z, w[3] = z0.w, w[4] = z1.x, w[5] = z1.y, w[6] = z1.z, w[7] = z1.w;
#pragma unroll
            for (int j = 0; j < 8; j++)
            {
                w[j] = key0 + j < low || key0 + j >= lim ? -INFINITY : w[j] * scale2;
                mx = fmaxf(mx, w[j]);
            }
#pragma unroll
            for (int k = 1; k < 8; k *= 2) { mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, k)); }
            float c = 1.f;
            if (mx > m + 8.f)
            {
                c = exp2_f32(m - mx);    // 0 at the first keys
                m = mx;
                l *= c;
                if (i > 0) { moved[i & 1u] = 1; }
            }
            if (sk == 0) { corr[sr] = c; }
            const float base = m == -INFINITY ? 0.f : m;
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                const float a = exp2_f32(w[2 * j] - base), b = exp2_f32(w[2 * j + 1] - base);
                l += a + b;
                hi[j] = pack_bf16x2(a, b);
                lo[j] = pack_bf16x2(a - __uint_as_float(hi[j] << 16), b - __uint_as_float(hi[j] & 0xFFFF0000u));
            }
            // the product before has read its weights (and left O alone) before they are written over
            if (i > 0) { ok = __all_sync(0xFFFFFFFFu, ok && wait(pv_done, i - 1)); }
            unsigned char* dst = pw + sr * 128 + ((sk ^ (sr & 7u)) * 16);
            *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(dst + AL_QBLOCK) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            fence_proxy_async();
            if (!ok && lane == 0) { stop[i & 1u] = 1; }
            bar_sync_named(1, 256);
            if (stop[i & 1u] != 0)    // all eight warps or none
            {
                ok = false;
                break;
            }
            if (moved[i & 1u] != 0)
            {
                tc_fence_after();
                for (int v = (int)side; v < vparts; v += 2)
                {
                    uint32_t o[32];
                    tmem_ld_32x32(lanes + AL_O + v * AL_ROWS, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 32; j++) { o[j] = __float_as_uint(__uint_as_float(o[j]) * corr[j]); }
                    tmem_st_32x16(lanes + AL_O + v * AL_ROWS, o);
                    tmem_st_32x16(lanes + AL_O + v * AL_ROWS + 16, o + 16);
                }
                tmem_st_wait();
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) { mbar_arrive(p_ready); }
        }
        ok = ok && (tiles == 0 || wait(o_full, 0));
        ok = __all_sync(0xFFFFFFFFu, ok);
#pragma unroll
        for (int k = 1; k < 8; k *= 2) { l += __shfl_xor_sync(0xFFFFFFFFu, l, k); }
        if (sk == 0)
        {
            if (p.splits == 1 && p.sink != nullptr && real) { l += exp2f(p.sink[(r0 + sr) % p.G] * 1.44269504088896341f - m); }
            ml[sr][0] = m;
            ml[sr][1] = l;
        }
        bar_sync_named(1, 256);
        if (!ok)
        {
            if (lane == 0) { give_up(2 + quarter, i); }
        }
        else if (!idle)
        {
            const unsigned int vl = al_value_ld(p), live = min((unsigned int)AL_ROWS, rows - r0);
            float* mine = al_partial(p, blockIdx.z * gridDim.y + rt, split);
            if (p.splits > 1 && st < AL_ROWS)
            {
                mine[2 * st] = ml[st][0];
                mine[2 * st + 1] = ml[st][1];
            }
            tc_fence_after();
            for (int v = (int)side; v < vparts; v += 2)
            {
                const unsigned int d = v * 128 + quarter * 32 + lane;
                uint32_t o[32];
#pragma unroll
                for (int j = 0; j < 32; j++) { o[j] = 0u; }
                if (tiles != 0)
                {
                    tmem_ld_32x32(lanes + AL_O + v * AL_ROWS, o);
                    tmem_ld_wait();
                }
                if (p.splits > 1)
                {
                    float* out = mine + 2 * AL_ROWS + d;
#pragma unroll
                    for (unsigned int r = 0; r < AL_ROWS; r++)
                    {
                        if (r < live && d < vl) { out[r * vl] = __uint_as_float(o[r]); }
                    }
                    continue;
                }
#pragma unroll 1
                for (unsigned int r = 0; r < live; r++)
                {
                    float y = 0.f;
#pragma unroll
                    for (unsigned int k = 0; k < AL_ROWS; k++) { y = k == r ? __uint_as_float(o[k]) : y; }
                    if (d < p.vdim) { attention_store(p, x, start, 0, r0 + r, d, y / ml[r][1]); }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) { tmem_dealloc(tmem, AL_TMEM); }
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

int launch_attention_latent(const AttnParams& p0, unsigned int slots, unsigned int entries, unsigned int max_n, unsigned int max_len, cudaStream_t stream,
    bool pdl)
{
    AttnParams p = p0;
    const DecoderDevice* dev = decoder_device();
    unsigned int* status = decoder_status_word();
    if (!dev || !status) { return 1; }
    const unsigned int row_tiles = (max_n * p.G + AL_ROWS - 1) / AL_ROWS;
    const unsigned long long cache_rows = (unsigned long long)slots * p.T_max;
    if (p.Hkv != 1 || p.k_cache != p.v_cache || p.k_ld != p.v_ld || p.dim > 576 || p.vdim > 512 || (p.k_ld % 8) || slots == 0 || cache_rows > 0x7FFFFFFFull
        || row_tiles > 65535u || entries > 65535u)
    {
        return -1;
    }
    CUtensorMap tk;
    if (!make_map_2d(&tk, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.k_cache, p.k_ld, cache_rows, (unsigned long long)p.k_ld * 2, 64, AL_KT, true)) { return -1; }
    if (p.window != 0 && max_len > p.window + max_n) { max_len = p.window + max_n; }
    const size_t smem = (size_t)al_smem((int)p.dim, (int)p.vdim);
    const unsigned int per_sm = smem > 100 * 1024 ? 1u : 2u;    // tensor memory holds two
    const unsigned long long units = (unsigned long long)entries * row_tiles, places = (unsigned long long)dev->sm_count * per_sm;
    const unsigned int tiles = (max_len + AL_KT - 1) / AL_KT + (p.window != 0 ? 1 : 0);
    // the fewest tiles in a row, over all waves of CTAs; a CTA costs its start, splits the combining
    double best = 1e30;
    p.splits = 1;
    for (unsigned int s = 1; s <= kMaxSplits && (s == 1 || (units * s * 2 <= kAttnPartials && s <= tiles)); s++)
    {
        const double waves = (double)((units * s + places - 1) / places);
        const double t = waves * ((double)((tiles + s - 1) / s) + 2.0) + (s > 1 ? 2.0 + 0.05 * s : 0.0);
        if (t < best)
        {
            best = t;
            p.splits = s;
        }
    }
    const int rc = launch_kernel("attention_latent", attention_latent_kernel, dim3(p.splits, row_tiles, entries), dim3(AL_THREADS), smem, stream, pdl, tk, p, status);
    if (rc || p.splits == 1) { return rc; }
    return launch_kernel("attention_latent_combine", attention_latent_combine_kernel, dim3(AL_ROWS, row_tiles, entries), dim3(128), 0, stream, pdl, p);
}

}    // namespace b200
