// Linears of many rows with BF16 weights: tcgen05 tiles, dense or grouped by expert, tensor-bound.
//
// A persistent CTA per SM walks tiles of 128 rows x BN weight rows.  A TMA lane streams the [128][64 k] piece of X and two
// halves of the [BN][64 k] piece of W (128-byte swizzle; for a gated MLP the halves are the gate rows and the up rows of the
// same features) through a ring that never drains between tiles; one lane issues tcgen05.mma (M = 128, N = BN, K = 16) into
// one of two accumulators in tensor memory; eight warps turn the other one into results: a thread owns one row, so gate and
// up of a feature meet in its registers.  Grouped: the tiles of group g start at its first row, the tile list is derived
// from the group offsets on the device.
// Every wait is bounded; on expiry the status word is raised, the roles drain, tensor memory is freed and the CTA returns.
#include "decoder_common.cuh"
#include "../gemm_prefill.cuh"
#include "linear.cuh"

#include <type_traits>

namespace b200
{

constexpr int LT_M = 128, LT_BK = 64;
constexpr int LT_EPI_WARPS = 8;
constexpr int LT_THREADS = 32 * (2 + LT_EPI_WARPS);
constexpr int LT_X_BYTES = LT_M * LT_BK * 2;
constexpr unsigned int LT_MAX_GROUPS = 1024;
__host__ __device__ constexpr int lt_stages(int bn) { return bn == 256 ? 4 : (bn == 128 ? 6 : 8); }
__host__ __device__ constexpr int lt_stage_bytes(int bn) { return LT_X_BYTES + bn * LT_BK * 2; }
constexpr int LT_HEADER = 1024 + (LT_MAX_GROUPS + 1) * 4;
__host__ __device__ constexpr int lt_header(void) { return (LT_HEADER + 1023) / 1024 * 1024; }
__host__ __device__ constexpr int lt_smem(int bn) { return lt_header() + lt_stages(bn) * lt_stage_bytes(bn) + 1024; }

// 32 result columns of one row
__device__ __forceinline__ void store_row32(const LinearMember& m, unsigned int row, unsigned int block, unsigned int f, const float (&v)[32], bool vec)
{
    const float s = linear_row_factor<__nv_bfloat16>(m, row, block);
    const unsigned int ycol = block * m.y_step;
    const size_t i = (size_t)row * m.ldy + ycol + f;
    if (f + 32 <= m.N && ycol + f + 32 <= m.tail && vec)
    {
        if (m.out_type == DT_BF16)
        {
            uint4* y = reinterpret_cast<uint4*>((__nv_bfloat16*)m.Y + i);
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                y[j] = make_uint4(pack_bf16x2(s * v[8 * j], s * v[8 * j + 1]), pack_bf16x2(s * v[8 * j + 2], s * v[8 * j + 3]),
                    pack_bf16x2(s * v[8 * j + 4], s * v[8 * j + 5]), pack_bf16x2(s * v[8 * j + 6], s * v[8 * j + 7]));
            }
        }
        else
        {
            float4* y = reinterpret_cast<float4*>((float*)m.Y + i);
#pragma unroll
            for (int j = 0; j < 8; j++)
            {
                float4 o = make_float4(s * v[4 * j], s * v[4 * j + 1], s * v[4 * j + 2], s * v[4 * j + 3]);
                if (m.accumulate)
                {
                    const float4 c = y[j];
                    o.x += c.x;
                    o.y += c.y;
                    o.z += c.z;
                    o.w += c.w;
                }
                y[j] = o;
            }
        }
        return;
    }
#pragma unroll
    for (int j = 0; j < 32; j++)
    {
        if (f + j < m.N) { linear_store(m, row, ycol + f + j, s * v[j]); }
    }
}

template <int BN>
__global__ void __launch_bounds__(LT_THREADS, 1) linear_tile_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ CUtensorMap tmW,
    const __grid_constant__ LinearMember m, const unsigned int ftiles, const int vec, unsigned int* status)
{
    extern __shared__ unsigned char lt_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~(uintptr_t)1023);
    constexpr unsigned int NS = lt_stages(BN);
    constexpr int STAGE = lt_stage_bytes(BN);
    constexpr int TMEM_COLS = 2 * BN;
    uint64_t* full = reinterpret_cast<uint64_t*>(smem);    // [8]
    uint64_t* empty = full + 8;                            // [8]
    uint64_t* acc_full = empty + 8;                        // [2]
    uint64_t* acc_empty = acc_full + 2;                    // [2]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    volatile unsigned int* abort_flag = reinterpret_cast<volatile unsigned int*>(tmem_slot + 1);
    int* first_tile = reinterpret_cast<int*>(smem + 1024);    // [groups + 1]: row tiles of the groups before
    unsigned char* stages = smem + lt_header();

    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool gated = activation_gated(m.activation);
    const unsigned int FT = gated ? BN / 2 : BN;    // result features per tile
    const unsigned int kblocks = (m.K + LT_BK - 1) / LT_BK;

    if (threadIdx.x == 0)
    {
        for (unsigned int s = 0; s < NS; s++)
        {
            mbar_init(full + s, 1);
            mbar_init(empty + s, 1);
        }
        for (unsigned int a = 0; a < 2; a++)
        {
            mbar_init(acc_full + a, 1);
            mbar_init(acc_empty + a, LT_EPI_WARPS);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) { tmem_alloc(tmem_slot, TMEM_COLS); }
    grid_dependency_launch();
    grid_dependency_wait();
    if (m.group_offset != nullptr && warp == 2)
    {
        int base = 0;
        for (unsigned int g0 = 0; g0 < m.groups; g0 += 32)
        {
            int c = 0;
            if (g0 + lane < m.groups) { c = (m.group_offset[g0 + lane + 1] - m.group_offset[g0 + lane] + LT_M - 1) / LT_M; }
            int inc = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1)
            {
                const int v = __shfl_up_sync(0xFFFFFFFFu, inc, o);
                if (lane >= (unsigned int)o) { inc += v; }
            }
            if (g0 + lane < m.groups) { first_tile[g0 + lane] = base + inc - c; }
            base += __shfl_sync(0xFFFFFFFFu, inc, 31);
        }
        if (lane == 0) { first_tile[m.groups] = base; }
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    const unsigned int row_tiles = m.group_offset != nullptr ? (unsigned int)first_tile[m.groups] : (m.rows + LT_M - 1) / LT_M;
    const unsigned int total = row_tiles * ftiles * m.blocks;

    // tile -> block, first weight row, first feature, first X / Y row, live rows.  Row tiles run fastest inside a group.
    auto coords = [&](unsigned int t, unsigned int& block, unsigned int& w0, unsigned int& f0, unsigned int& r0, unsigned int& live) {
        block = m.blocks > 1 ? t / (row_tiles * ftiles) : 0u;
        t -= block * row_tiles * ftiles;
        unsigned int g = block, tiles = row_tiles, rel = t, base = 0, rows = m.rows;
        if (m.group_offset != nullptr)
        {
            unsigned int lo = 0, hi = m.groups;    // the last group whose tiles start at or before t
            while (hi - lo > 1)
            {
                const unsigned int mid = (lo + hi) / 2;
                if ((unsigned int)first_tile[mid] * ftiles <= t) { lo = mid; }
                else { hi = mid; }
            }
            g = lo;
            rel = t - (unsigned int)first_tile[g] * ftiles;
            tiles = (unsigned int)(first_tile[g + 1] - first_tile[g]);
            base = (unsigned int)m.group_offset[g];
            rows = (unsigned int)m.group_offset[g + 1] - base;
        }
        const unsigned int rt = rel % tiles;
        f0 = rel / tiles * FT;
        w0 = g * m.group_rows + f0;
        r0 = base + rt * LT_M;
        live = min((unsigned int)LT_M, rows - rt * LT_M);
    };

    if (warp == 0)
    {
        if (lane == 0)
        {
            bool ok = true;
            unsigned int it = 0;
            for (unsigned int t = blockIdx.x; t < total && ok; t += gridDim.x)
            {
                unsigned int block, w0, f0, r0, live;
                coords(t, block, w0, f0, r0, live);
                const unsigned int xcol = block * m.x_step;
                const unsigned int w1 = gated ? w0 + m.up_row : w0 + BN / 2;
                for (unsigned int kb = 0; kb < kblocks; kb++, it++)
                {
                    const unsigned int s = it % NS;
                    if (it >= NS && (*abort_flag != 0 || !mbar_wait_bounded(empty + s, ((it / NS) - 1u) & 1u)))
                    {
                        ok = false;
                        note_timeout(status, WAIT_LINEAR_TILE, 0, it);
                        *abort_flag = 1;
                        break;
                    }
                    unsigned char* st = stages + s * STAGE;
                    mbar_expect_tx(full + s, STAGE);
                    tma_load_2d(st, &tmX, (int)(xcol + kb * LT_BK), (int)r0, full + s);
                    tma_load_2d(st + LT_X_BYTES, &tmW, (int)(kb * LT_BK), (int)w0, full + s);
                    tma_load_2d(st + LT_X_BYTES + BN * LT_BK, &tmW, (int)(kb * LT_BK), (int)w1, full + s);
                    mbar_arrive(full + s);
                }
            }
            if (!ok)
            {
                // wait (bounded) for the copies in flight before the CTA may leave
                for (unsigned int j = it > NS ? it - NS : 0; j < it; j++)
                {
                    const unsigned long long t0 = global_timer_ns();
                    while (!mbar_try_wait(full + (j % NS), (j / NS) & 1u) && global_timer_ns() - t0 < 100000ull) {}
                }
            }
        }
    }
    else if (warp == 1)
    {
        bool ok = true;
        unsigned int it = 0, n = 0;
        const uint32_t idesc = umma_idesc_bf16(LT_M, BN);
        for (unsigned int t = blockIdx.x; t < total && ok; t += gridDim.x, n++)
        {
            const unsigned int a = n & 1u;
            if (n >= 2 && (*abort_flag != 0 || !mbar_wait_bounded(acc_empty + a, ((n >> 1) - 1u) & 1u))) { ok = false; }
            for (unsigned int kb = 0; kb < kblocks && ok; kb++, it++)
            {
                const unsigned int s = it % NS;
                if (*abort_flag != 0 || !mbar_wait_bounded(full + s, (it / NS) & 1u))
                {
                    ok = false;
                    break;
                }
                tc_fence_after();
                const uint32_t x_addr = smem_u32(stages + s * STAGE), w_addr = x_addr + LT_X_BYTES;
                if (elect_one())
                {
#pragma unroll
                    for (int k = 0; k < LT_BK / 16; k++)
                    {
                        umma_bf16(tmem + a * BN, umma_desc_kmajor_sw128(x_addr + k * 32), umma_desc_kmajor_sw128(w_addr + k * 32), idesc,
                            (kb | (unsigned int)k) != 0 ? 1u : 0u);
                    }
                    umma_commit(empty + s);
                }
                __syncwarp();
            }
            if (ok && elect_one()) { umma_commit(acc_full + a); }
            __syncwarp();
        }
        if (!ok)
        {
            if (lane == 0)
            {
                note_timeout(status, WAIT_LINEAR_TILE, 1, it);
                *abort_flag = 1;
            }
            // the barrier completes once the MMAs in flight have stopped reading shared memory
            if (elect_one()) { umma_commit(acc_full + (n & 1u)); }
            __syncwarp();
        }
    }
    else
    {
        const unsigned int quarter = warp & 3u, half = (warp - 2u) >> 2;
        bool ok = true;
        unsigned int n = 0;
        for (unsigned int t = blockIdx.x; t < total && ok; t += gridDim.x, n++)
        {
            unsigned int block, w0, f0, r0, live;
            coords(t, block, w0, f0, r0, live);
            const unsigned int a = n & 1u;
            ok = *abort_flag == 0 && mbar_wait_bounded(acc_full + a, (n >> 1) & 1u);
            ok = __all_sync(0xFFFFFFFFu, ok) && *abort_flag == 0;
            ok = __all_sync(0xFFFFFFFFu, ok);
            if (!ok)
            {
                if (lane == 0)
                {
                    note_timeout(status, WAIT_LINEAR_TILE, 2, n);
                    *abort_flag = 1;
                }
                break;
            }
            tc_fence_after();
            const unsigned int rl = quarter * 32 + lane;
            const uint32_t lanes = tmem + ((quarter * 32u) << 16) + a * BN;
            const unsigned int per = FT >= 64 ? FT / 2 : FT;    // result columns of this half
            for (unsigned int c = half * per; c < (half + 1) * per && c < FT && f0 + c < m.N; c += 32)
            {
                uint32_t r[32];
                float v[32];
                tmem_ld_32x32(lanes + c, r);
                tmem_ld_wait();
                // one activation's code for all columns at a time
                auto plain = [&](auto act) {
#pragma unroll
                    for (int j = 0; j < 32; j++) { v[j] = activate<decltype(act)::value, true>(m.alpha * __uint_as_float(r[j]), 0.f, m.cap); }
                };
                if (gated)
                {
                    uint32_t u[32];
                    tmem_ld_32x32(lanes + BN / 2 + c, u);
                    tmem_ld_wait();
                    auto both = [&](auto act) {
#pragma unroll
                        for (int j = 0; j < 32; j++)
                        {
                            v[j] = activate<decltype(act)::value, true>(m.alpha * __uint_as_float(r[j]), m.alpha * __uint_as_float(u[j]), m.cap);
                        }
                    };
                    if (m.activation == B200_ACT_SILU_GATE) { both(std::integral_constant<int, B200_ACT_SILU_GATE>()); }
                    else { both(std::integral_constant<int, B200_ACT_GELU_GATE>()); }
                }
                else if (m.activation == B200_ACT_NONE) { plain(std::integral_constant<int, B200_ACT_NONE>()); }
                else if (m.activation == B200_ACT_RELU2) { plain(std::integral_constant<int, B200_ACT_RELU2>()); }
                else { plain(std::integral_constant<int, B200_ACT_SOFTCAP>()); }
                if (rl < live) { store_row32(m, r0 + rl, block, f0 + c, v, vec != 0); }
                __syncwarp();
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) { mbar_arrive(acc_empty + a); }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) { tmem_dealloc(tmem, TMEM_COLS); }
}

template <int BN>
static int launch_tile(const LinearMember& m, const DecoderDevice& dev, cudaStream_t stream, bool pdl)
{
    unsigned int* status = decoder_status_word();
    if (!status) { return 1; }
    const bool gated = activation_gated(m.activation);
    const unsigned int FT = gated ? BN / 2 : BN;
    const unsigned int ftiles = (m.N + FT - 1) / FT;
    // weight rows of all groups; rows past the end read as zeros, rows of a neighbouring group give results nobody stores
    const unsigned long long wrows = (unsigned long long)((m.blocks > 1 ? m.blocks : m.groups) - 1) * m.group_rows + (gated ? m.up_row : 0u) + m.N;
    CUtensorMap tx, tw;
    if (!make_map_2d(&tx, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, m.X, (unsigned long long)(m.blocks - 1) * m.x_step + m.K, m.rows, (unsigned long long)m.ldx * 2, LT_BK, LT_M, true)
        || !make_map_2d(&tw, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, m.W, m.K, wrows, (unsigned long long)m.ldw * 2, LT_BK, BN / 2, true))
    {
        return -1;
    }
    const bool vec = (reinterpret_cast<uintptr_t>(m.Y) & 15u) == 0 && (m.ldy % 8) == 0 && (m.y_step % 8) == 0;
    unsigned long long tiles = (unsigned long long)((m.rows + LT_M - 1) / LT_M + (m.groups > 1 ? m.groups : 0)) * ftiles * m.blocks;    // an upper bound
    const unsigned int grid = (unsigned int)(tiles < (unsigned long long)dev.sm_count ? tiles : dev.sm_count);
    return launch_kernel("linear_tile", linear_tile_kernel<BN>, dim3(grid), dim3(LT_THREADS), (size_t)lt_smem(BN), stream, pdl, tx, tw, m, ftiles,
        vec ? 1 : 0, status);
}

int launch_linear_tile(const LinearMember& m, cudaStream_t stream, bool pdl)
{
    if (m.x_row != nullptr || m.groups > LT_MAX_GROUPS) { return -1; }
    const DecoderDevice* dev = decoder_device();
    if (!dev) { return 1; }
    // the widest tile that still gives every SM one
    const bool gated = activation_gated(m.activation);
    const unsigned long long rt = (m.rows + LT_M - 1) / LT_M;
    auto tiles = [&](unsigned int bn) -> unsigned long long {
        const unsigned int ft = gated ? bn / 2 : bn;
        if (m.blocks > 1 && bn > 64 && m.N <= ft / 2) { return 0; }    // a block would not fill half of it
        return rt * m.blocks * ((m.N + ft - 1) / ft);
    };
    if (tiles(256) >= (unsigned long long)dev->sm_count * 8 / 10) { return launch_tile<256>(m, *dev, stream, pdl); }
    if (tiles(128) >= (unsigned long long)dev->sm_count * 8 / 10) { return launch_tile<128>(m, *dev, stream, pdl); }
    return launch_tile<64>(m, *dev, stream, pdl);
}

}    // namespace b200
