// BF16 attention of prompts on tcgen05, tensor-bound: 128 packed query rows per CTA (a row is one query head of one token;
// heads that share a kv head are packed together) against 64-key tiles, two CTAs per SM (one where keys and values are larger
// than 128).
//
// A TMA lane streams keys and values from the cache (128-byte swizzle) through two-deep rings; the MMA lane issues
// S = Q K^T (M = 128, N = 64) into tensor memory and, once the softmax warps have turned S into weights, O += P V with P as
// the operand in tensor memory and V as it lies ([key][element], an MN-major operand).  The weights enter as the sum of two
// BF16 numbers and take the place of their scores.  There are two such places: the scores of the next tile are ready when the
// softmax warps get to them.  Four softmax warps own one row per thread; the running maximum only moves when it grows by more
// than 2^8, so that O is seldom rescaled.
// Every wait is bounded; on expiry the status word is raised, the roles drain, tensor memory is freed and the CTA returns.
#include "attention.cuh"
#include "tile_common.cuh"

#include <type_traits>

namespace b200
{

constexpr int TA_KT = 64, TA_ROWS = 128;
constexpr int TA_THREADS = 192;
constexpr int TA_BLOCK = TA_KT * 128;          // 64 keys x 64 elements
constexpr int TA_QBLOCK = TA_ROWS * 128;       // 128 rows x 64 elements
__host__ __device__ constexpr int ta_smem(int dk, int dv) { return 1024 + (dk / 64) * TA_QBLOCK + 2 * (dk / 64 + dv / 64) * TA_BLOCK + 1024; }
constexpr uint32_t TA_O = 128;    // columns: two places of S (64) or P (32 high, 32 low), then O
__host__ __device__ constexpr uint32_t ta_tmem(int dv) { return dv <= 128 ? 256 : 512; }
__host__ __device__ constexpr int ta_ctas(int dk, int dv) { return ta_smem(dk, dv) <= 113 * 1024 && dv <= 128 ? 2 : 1; }

// A BF16 gate's sigmoid, by the hardware's exponential and reciprocal.
__device__ __forceinline__ float gate_sigmoid(float z) { return __fdividef(1.0f, 1.0f + exp2_f32(-1.44269504088896341f * z)); }

template <int DK, int DV>
__global__ void __launch_bounds__(TA_THREADS, ta_ctas(DK, DV)) attention_tile_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
    const __grid_constant__ AttnParams p, unsigned int* status)
{
    extern __shared__ unsigned char ta_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(ta_raw) + 1023) & ~(uintptr_t)1023);
    constexpr int KBY = (DK / 64) * TA_BLOCK, VBY = (DV / 64) * TA_BLOCK;
    uint64_t* k_full = reinterpret_cast<uint64_t*>(smem);
    uint64_t *k_empty = k_full + 2, *v_full = k_full + 4, *v_empty = k_full + 6;
    uint64_t *s_full = k_full + 8, *p_ready = k_full + 10, *q_ready = k_full + 12, *pv_done = k_full + 13, *o_full = k_full + 14;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(k_full + 15);
    volatile unsigned int* abort_flag = reinterpret_cast<volatile unsigned int*>(tmem_slot + 1);
    unsigned char* qs = smem + 1024;
    unsigned char* ks = qs + (DK / 64) * TA_QBLOCK;
    unsigned char* vs = ks + 2 * KBY;

    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0)
    {
        for (int i = 0; i < 10; i++) { mbar_init(k_full + i, 1); }
        mbar_init(q_ready, 4);
        mbar_init(p_ready, 4);    // one per place: a warp may be a tile ahead of another
        mbar_init(p_ready + 1, 4);
        mbar_init(pv_done, 1);
        mbar_init(o_full, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) { tmem_alloc(tmem_slot, ta_tmem(DV)); }
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int kvh = blockIdx.y, e = p.e0 + blockIdx.z;
    const unsigned int n = (unsigned int)p.n[e], start = (unsigned int)p.start[e], pos = (unsigned int)p.pos[e];
    const unsigned int rows = n * p.G, row_tiles = (rows + TA_ROWS - 1) / TA_ROWS;
    const bool idle = blockIdx.x >= row_tiles;    // a shorter entry than the longest one
    const unsigned int t0 = idle ? 0 : (row_tiles - 1 - blockIdx.x) * TA_ROWS;    // the rows that see the most keys first
    const unsigned int T = idle ? 0 : min(pos + min(t0 + TA_ROWS - 1u, rows - 1) / p.G + 1, p.T_max);
    const unsigned int begin = idle ? 0 : first_key(p, e, pos + t0 / p.G + 1) / TA_KT;    // key tile the first row's window starts in
    const unsigned int tiles = (T + TA_KT - 1) / TA_KT - begin;
    const unsigned int seq = ((unsigned int)p.slot[e] * p.Hkv + kvh) * p.T_max;
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    auto give_up = [&](unsigned int role, unsigned int step) {
        note_timeout(status, WAIT_ATTENTION_TILE, role, step);
        *abort_flag = 1;
    };
    auto wait = [&](uint64_t* bar, unsigned int parity) { return *abort_flag == 0 && mbar_wait_bounded(bar, parity & 1u); };

    if (warp == 0)
    {
        if (lane == 0)
        {
            unsigned int k_issued = 0, v_issued = 0;
            bool ok = true;
            for (unsigned int i = 0; i < tiles && ok; i++)
            {
                const unsigned int s = i & 1u;
                const int y = (int)(seq + (begin + i) * TA_KT);
                if (i >= 2 && !wait(k_empty + s, (i >> 1) - 1)) { ok = false; break; }
                mbar_expect_tx(k_full + s, KBY);
#pragma unroll
                for (int b = 0; b < DK / 64; b++) { tma_load_2d(ks + s * KBY + b * TA_BLOCK, &tmK, b * 64, y, k_full + s); }
                mbar_arrive(k_full + s);
                k_issued++;
                if (i >= 2 && !wait(v_empty + s, (i >> 1) - 1)) { ok = false; break; }
                mbar_expect_tx(v_full + s, VBY);
#pragma unroll
                for (int b = 0; b < DV / 64; b++) { tma_load_2d(vs + s * VBY + b * TA_BLOCK, &tmV, b * 64, y, v_full + s); }
                mbar_arrive(v_full + s);
                v_issued++;
            }
            if (!ok)
            {
                give_up(0, k_issued);
                // wait (bounded) for the copies in flight before the CTA may leave
                auto drain = [&](uint64_t* full, unsigned int issued) {
                    for (unsigned int j = issued > 2 ? issued - 2 : 0; j < issued; j++)
                    {
                        const unsigned long long t = global_timer_ns();
                        while (!mbar_try_wait(full + (j & 1u), (j >> 1) & 1u) && global_timer_ns() - t < 100000ull) {}
                    }
                };
                drain(k_full, k_issued);
                drain(v_full, v_issued);
            }
        }
    }
    else if (warp == 1)
    {
        const uint32_t idesc_s = umma_idesc_bf16(TA_ROWS, TA_KT);
        const uint32_t idesc_o = umma_idesc_bf16(TA_ROWS, DV) | (1u << 16);    // B is MN-major
        const uint32_t q_addr = smem_u32(qs), k_addr = smem_u32(ks), v_addr = smem_u32(vs);
        auto scores = [&](unsigned int i) {
            if (!wait(k_full + (i & 1u), i >> 1)) { return false; }
            tc_fence_after();
            if (elect_one())
            {
#pragma unroll
                for (int k = 0; k < DK / 16; k++)
                {
                    if (k * 16 < (int)p.dim)
                    {
                        umma_bf16(tmem + (i & 1u) * 64, umma_desc_kmajor_sw128(q_addr + (k / 4) * TA_QBLOCK + (k % 4) * 32),
                            umma_desc_kmajor_sw128(k_addr + (i & 1u) * KBY + (k / 4) * TA_BLOCK + (k % 4) * 32), idesc_s, k != 0 ? 1u : 0u);
                    }
                }
                umma_commit(k_empty + (i & 1u));
                umma_commit(s_full + (i & 1u));
            }
            __syncwarp();
            return true;
        };
        unsigned int at = 0;    // product the lane is at
        bool ok = tiles == 0 || (wait(q_ready, 0) && scores(0) && (tiles == 1 || scores(1)));
        for (unsigned int i = 0; i < tiles && ok; i++)
        {
            at = i + 1;
            ok = wait(p_ready + (i & 1u), i >> 1);
            if (!ok) { break; }
            tc_fence_after();
            if (!wait(v_full + (i & 1u), i >> 1)) { ok = false; break; }
            tc_fence_after();
            if (elect_one())
            {
#pragma unroll
                for (int part = 0; part < 2; part++)    // the high halves of the weights, then the low ones
                {
#pragma unroll
                    for (int k = 0; k < TA_KT / 16; k++)
                    {
                        umma_bf16_ts(tmem + TA_O, tmem + (i & 1u) * 64 + part * 32 + k * 8, umma_desc_mnmajor_sw128(v_addr + (i & 1u) * VBY + k * 2048), idesc_o,
                            (i | (unsigned int)part | (unsigned int)k) != 0 ? 1u : 0u);
                    }
                }
                umma_commit(v_empty + (i & 1u));
                umma_commit(pv_done);
                if (i + 1 == tiles) { umma_commit(o_full); }
            }
            __syncwarp();
            // into the place of the weights just issued: products of one thread run in the order of their issue
            if (i + 2 < tiles && !scores(i + 2)) { ok = false; }
        }
        if (!ok)
        {
            if (lane == 0) { give_up(1, at); }
            if (elect_one()) { umma_commit(pv_done); }    // completes once the MMAs in flight have stopped reading shared memory
            __syncwarp();
        }
    }
    else if (!idle)
    {
        const unsigned int quarter = warp & 3u, rl = quarter * 32 + lane, r = t0 + rl;
        const uint32_t lanes = tmem + ((quarter * 32u) << 16);
        const bool real = r < rows;
        const unsigned int tok = start + (real ? r / p.G : 0), head = kvh * p.G + (real ? r % p.G : 0);
        const __nv_bfloat16* x = (const __nv_bfloat16*)p.qkvg + (size_t)tok * p.ld;
        {
            const __nv_bfloat16* src = x + (size_t)head * p.q_ld;
            const bool vec = (p.dim % 8) == 0 && (p.q_ld % 8) == 0;
            const uint32_t flip = p.scale < 0.f ? 0x80008000u : 0u;    // the maximum is taken before scaling
#pragma unroll
            for (int c = 0; c < DK / 8; c++)
            {
                uint4 v = make_uint4(0, 0, 0, 0);
                if (real && c * 8 < (int)p.dim)
                {
                    if (vec) { v = *reinterpret_cast<const uint4*>(src + c * 8); }
                    else
                    {
                        uint32_t u[8];
#pragma unroll
                        for (int j = 0; j < 8; j++) { u[j] = c * 8 + j < (int)p.dim ? __bfloat16_as_ushort(src[c * 8 + j]) : 0u; }
                        v = make_uint4(u[0] | (u[1] << 16), u[2] | (u[3] << 16), u[4] | (u[5] << 16), u[6] | (u[7] << 16));
                    }
                }
                v.x ^= flip;
                v.y ^= flip;
                v.z ^= flip;
                v.w ^= flip;
                sts128(smem_u32(qs) + (c / 8) * TA_QBLOCK + rl * 128 + (((c % 8) ^ (rl & 7u)) * 16), v.x, v.y, v.z, v.w);
            }
            fence_proxy_async();
            __syncwarp();
            if (lane == 0) { mbar_arrive(q_ready); }
        }
        const unsigned int low = first_key(p, e, pos + r / p.G + 1), lim = min(pos + r / p.G + 1, T);
        const unsigned int first_lim = pos + t0 / p.G + 1, last_low = first_key(p, e, pos + (t0 + TA_ROWS - 1) / p.G + 1);
        const float scale2 = fmaxf(fabsf(p.scale) * 1.44269504088896341f, 1e-30f);    // 0 times a masked -inf would be no number
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        for (unsigned int i = 0; i < tiles; i++)
        {
            const uint32_t place = lanes + (i & 1u) * 64;
            ok = __all_sync(0xFFFFFFFFu, wait(s_full + (i & 1u), i >> 1));
            if (!ok) { break; }
            tc_fence_after();
            uint32_t s[TA_KT];
            tmem_ld_32x32(place, *reinterpret_cast<uint32_t(*)[32]>(s));
            tmem_ld_32x32(place + 32, *reinterpret_cast<uint32_t(*)[32]>(s + 32));
            tmem_ld_wait();
            const unsigned int key0 = (begin + i) * TA_KT;
            if (key0 + TA_KT > first_lim || key0 < last_low)
            {
#pragma unroll
                for (int j = 0; j < TA_KT; j++)
                {
                    if (key0 + j < low || key0 + j >= lim) { s[j] = 0xFF800000u; }    // -inf
                }
            }
            float mx[4] = { -INFINITY, -INFINITY, -INFINITY, -INFINITY };    // four maxima in flight
#pragma unroll
            for (int j = 0; j < TA_KT; j++) { mx[j & 3] = fmaxf(mx[j & 3], __uint_as_float(s[j])); }
            const float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * scale2;
            float c = 1.f;
            if (top > m + 8.f)
            {
                c = exp2_f32(m - top);    // 0 at the first tile
                m = top;
                l *= c;
            }
            const float base = m == -INFINITY ? 0.f : m;    // a window may start after this tile
            uint32_t hi[TA_KT / 2], lo[TA_KT / 2];
            float sum[2] = { 0.f, 0.f };
#pragma unroll
            for (int j = 0; j < TA_KT / 2; j++)
            {
                const float a = exp2_f32(fmaf(__uint_as_float(s[2 * j]), scale2, -base)), b = exp2_f32(fmaf(__uint_as_float(s[2 * j + 1]), scale2, -base));
                sum[0] += a;
                sum[1] += b;
                hi[j] = pack_bf16x2(a, b);
                lo[j] = pack_bf16x2(a - __uint_as_float(hi[j] << 16), b - __uint_as_float(hi[j] & 0xFFFF0000u));
            }
            l += sum[0] + sum[1];
            if (i > 0 && __any_sync(0xFFFFFFFFu, c != 1.f))
            {
                // the product before leaves O alone (the one before that has: the scores of this tile came after it)
                ok = __all_sync(0xFFFFFFFFu, wait(pv_done, i - 1));
                if (!ok) { break; }
                tc_fence_after();
#pragma unroll
                for (int d = 0; d < DV; d += 32)
                {
                    uint32_t o[32];
                    tmem_ld_32x32(lanes + TA_O + d, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 32; j++) { o[j] = __float_as_uint(__uint_as_float(o[j]) * c); }
                    tmem_st_32x16(lanes + TA_O + d, o);
                    tmem_st_32x16(lanes + TA_O + d + 16, o + 16);
                }
            }
            tmem_st_32x16(place, hi);
            tmem_st_32x16(place + 16, hi + 16);
            tmem_st_32x16(place + 32, lo);
            tmem_st_32x16(place + 48, lo + 16);
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) { mbar_arrive(p_ready + (i & 1u)); }
        }
        // a barrier of its own: a wait tells only neighbouring phases apart, and pv_done may be one or two further by now
        ok = ok && __all_sync(0xFFFFFFFFu, wait(o_full, 0));
        if (ok)
        {
            tc_fence_after();
            if (p.sink != nullptr) { l += exp2_f32(fmaf(p.sink[head], 1.44269504088896341f, -m)); }
            const float inv = head_factor<__nv_bfloat16>(p, tok, head) / l;
            const __nv_bfloat16* gate = x + p.g_off + (size_t)head * p.vdim;
            __nv_bfloat16* out = (__nv_bfloat16*)p.out + (size_t)tok * p.ldo + (size_t)head * p.vdim;
            const bool vec = (p.vdim % 8) == 0 && (p.g_off % 8) == 0;
#pragma unroll
            for (int d = 0; d < DV; d += 32)
            {
                if (d >= (int)p.vdim) { break; }
                uint32_t o[32];
                tmem_ld_32x32(lanes + TA_O + d, o);
                tmem_ld_wait();
                if (real)
                {
#pragma unroll
                    for (int q = 0; q < 32; q += 8)
                    {
                        if (d + q >= (int)p.vdim) { continue; }
                        float v[8];
#pragma unroll
                        for (int j = 0; j < 8; j++) { v[j] = __uint_as_float(o[q + j]) * inv; }
                        if (vec)
                        {
                            if (p.gate)
                            {
                                const uint4 gv = *reinterpret_cast<const uint4*>(gate + d + q);
                                const uint32_t gw[4] = { gv.x, gv.y, gv.z, gv.w };
#pragma unroll
                                for (int j = 0; j < 4; j++)
                                {
                                    v[2 * j] *= gate_sigmoid(__uint_as_float(gw[j] << 16));
                                    v[2 * j + 1] *= gate_sigmoid(__uint_as_float(gw[j] & 0xFFFF0000u));
                                }
                            }
                            *reinterpret_cast<uint4*>(out + d + q) =
                                make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
                        }
                        else
                        {
#pragma unroll
                            for (int j = 0; j < 8; j++)
                            {
                                if (d + q + j < (int)p.vdim)
                                {
                                    const float w = p.gate ? sigmoid_f32(__bfloat162float(gate[d + q + j])) : 1.f;
                                    out[d + q + j] = __float2bfloat16_rn(v[j] * w);
                                }
                            }
                        }
                    }
                }
                __syncwarp();
            }
        }
        else if (lane == 0) { give_up(2 + quarter, tiles); }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) { tmem_dealloc(tmem, ta_tmem(DV)); }
}

template <int DK, int DV>
static int run_tile(const AttnParams& p, const CUtensorMap& tk, const CUtensorMap& tv, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl)
{
    unsigned int* status = decoder_status_word();
    if (!status) { return 1; }
    const dim3 grid((max_n * p.G + TA_ROWS - 1) / TA_ROWS, p.Hkv, entries);
    return launch_kernel("attention_tile", attention_tile_kernel<DK, DV>, grid, dim3(TA_THREADS), (size_t)ta_smem(DK, DV), stream, pdl, tk, tv, p, status);
}

int launch_attention_tile(const AttnParams& p, unsigned int slots, unsigned int entries, unsigned int max_n, cudaStream_t stream, bool pdl)
{
    const unsigned long long rows = (unsigned long long)slots * p.Hkv * p.T_max;
    auto low = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) != 0; };
    if (p.dim > 256 || p.vdim > 256 || slots == 0 || rows > 0x7FFFFFFFull || low(p.k_cache) || low(p.v_cache) || low(p.qkvg) || low(p.out) || (p.ld % 8)
        || (p.ldo % 8) || entries > 65535u || p.Hkv > 65535u)
    {
        return -1;
    }
    CUtensorMap tk, tv;
    if (!make_map_2d(&tk, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.k_cache, p.k_ld, rows, (unsigned long long)p.k_ld * 2, 64, TA_KT, true)
        || !make_map_2d(&tv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.v_cache, p.v_ld, rows, (unsigned long long)p.v_ld * 2, 64, TA_KT, true))
    {
        return -1;
    }
    auto by_values = [&](auto dk) {
        constexpr int DK = decltype(dk)::value;
        if (p.vdim <= 64) { return run_tile<DK, 64>(p, tk, tv, entries, max_n, stream, pdl); }
        if (p.vdim <= 128) { return run_tile<DK, 128>(p, tk, tv, entries, max_n, stream, pdl); }
        if (p.vdim <= 192) { return run_tile<DK, 192>(p, tk, tv, entries, max_n, stream, pdl); }
        return run_tile<DK, 256>(p, tk, tv, entries, max_n, stream, pdl);
    };
    if (p.dim <= 64) { return by_values(std::integral_constant<int, 64>()); }
    if (p.dim <= 128) { return by_values(std::integral_constant<int, 128>()); }
    if (p.dim <= 192) { return by_values(std::integral_constant<int, 192>()); }
    return by_values(std::integral_constant<int, 256>());
}

}    // namespace b200
