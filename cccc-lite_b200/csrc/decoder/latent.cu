// The row operations around latent attention: norms of the two latents, rotated parts of keys and queries, the key part that
// all heads share beside expanded keys.
#include "decoder_common.cuh"

namespace b200
{

struct LatentParams
{
    const void* down;
    void *cq, *cache;
    const float *q_norm, *kv_norm;
    const float2* rotary;
    const int *slot, *pos, *start, *token_entry;
    unsigned int ld, ld_cq, kv_off, q_rank, kv_rank, rot_dim, c_ld, T_max, t0;
    float eps;
};

// A CTA per token and part (0: query latent, 1: cache row); the row lives in shared memory as floats.
template <class T>
__global__ void __launch_bounds__(512) latent_down_kernel(const LatentParams p)
{
    extern __shared__ float ld_row[];
    __shared__ float sums[16];
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int i = p.t0 + blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    const bool is_q = blockIdx.y == 0;
    const int e = p.token_entry[i];
    const unsigned int row = (unsigned int)(p.pos[e] + ((int)i - p.start[e]));
    if (row >= p.T_max) { return; }
    const unsigned int rank = is_q ? p.q_rank : p.kv_rank, all = is_q ? rank : rank + p.rot_dim;
    const T* src = (const T*)p.down + (size_t)i * p.ld + (is_q ? 0u : p.kv_off);
    float sq = 0.f;
    for (unsigned int d = tid; d < all; d += blockDim.x)
    {
        const float v = Elem<T>::get(src[d]);
        ld_row[d] = v;
        if (d < rank) { sq += v * v; }
    }
    sq = warp_sum(sq);
    if (lane == 0) { sums[warp] = sq; }
    __syncthreads();
    const float inv = 1.0f / sqrtf(warp_sum(lane < warps ? sums[lane] : 0.f) / (float)rank + p.eps);
    const float* w = is_q ? p.q_norm : p.kv_norm;
    T* dst = is_q ? (T*)p.cq + (size_t)i * p.ld_cq : (T*)p.cache + ((size_t)p.slot[e] * p.T_max + row) * p.c_ld;
    const float2* rot = p.rotary + (size_t)row * (p.rot_dim / 2);
    for (unsigned int d = tid; d < all; d += blockDim.x)
    {
        dst[d] = Elem<T>::put(d < rank ? ld_row[d] * inv * w[d] : rotated(ld_row + rank, d - rank, p.rot_dim, true, rot));
    }
}

// The same in BF16 by eights, a thread per eight: ranks, offsets and the rotated part are whole eights.
__global__ void __launch_bounds__(512) latent_down8_kernel(const LatentParams p)
{
    __shared__ float sums[16];
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int i = p.t0 + blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    const bool is_q = blockIdx.y == 0;
    const int e = p.token_entry[i];
    const unsigned int row = (unsigned int)(p.pos[e] + ((int)i - p.start[e]));
    if (row >= p.T_max) { return; }
    const unsigned int rank = is_q ? p.q_rank : p.kv_rank, all = is_q ? rank : rank + p.rot_dim, d = tid * 8;
    float f[8], sq = 0.f;
#pragma unroll
    for (int j = 0; j < 8; j++) { f[j] = 0.f; }
    if (d < all)
    {
        const uint4 u = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)p.down + (size_t)i * p.ld + (is_q ? 0u : p.kv_off) + d);
        const uint32_t w[4] = { u.x, u.y, u.z, u.w };
#pragma unroll
        for (int j = 0; j < 4; j++)
        {
            f[2 * j] = __uint_as_float(w[j] << 16);
            f[2 * j + 1] = __uint_as_float(w[j] & 0xFFFF0000u);
        }
    }
    if (d < rank)
    {
#pragma unroll
        for (int j = 0; j < 8; j++) { sq += f[j] * f[j]; }
    }
    sq = warp_sum(sq);
    if (lane == 0) { sums[warp] = sq; }
    __syncthreads();
    const float inv = 1.0f / sqrtf(warp_sum(lane < warps ? sums[lane] : 0.f) / (float)rank + p.eps);
    if (d >= all) { return; }
    if (d < rank)
    {
        const float* w = (is_q ? p.q_norm : p.kv_norm) + d;
#pragma unroll
        for (int j = 0; j < 8; j++) { f[j] *= inv * w[j]; }
    }
    else
    {
        const float2* rot = p.rotary + (size_t)row * (p.rot_dim / 2) + (d - rank) / 2;
#pragma unroll
        for (int j = 0; j < 4; j++)
        {
            const float2 cs = rot[j];
            const float u = f[2 * j], v = f[2 * j + 1];
            f[2 * j] = u * cs.x - v * cs.y;
            f[2 * j + 1] = v * cs.x + u * cs.y;
        }
    }
    __nv_bfloat16* dst = (is_q ? (__nv_bfloat16*)p.cq + (size_t)i * p.ld_cq : (__nv_bfloat16*)p.cache + ((size_t)p.slot[e] * p.T_max + row) * p.c_ld) + d;
    store4(dst, make_float4(f[0], f[1], f[2], f[3]));
    store4(dst + 4, make_float4(f[4], f[5], f[6], f[7]));
}

// A CTA per token, a thread per pair.
template <class T>
__global__ void __launch_bounds__(256) latent_query_kernel(const T* src, unsigned int ld_src, unsigned int src_step, unsigned int src_off, T* dst,
    unsigned int ld_dst, unsigned int dst_step, unsigned int dst_off, unsigned int heads, unsigned int pairs, const float2* rotary, unsigned int T_max,
    const int* pos, const int* start, const int* token_entry, unsigned int t0)
{
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int i = t0 + blockIdx.x;
    const int e = token_entry[i];
    const unsigned int row = (unsigned int)(pos[e] + ((int)i - start[e]));
    if (row >= T_max) { return; }
    for (unsigned int j = threadIdx.x; j < heads * pairs; j += blockDim.x)
    {
        const unsigned int h = j / pairs, k = j % pairs;
        const T* s = src + (size_t)i * ld_src + (size_t)h * src_step + src_off + 2 * k;
        T* d = dst + (size_t)i * ld_dst + (size_t)h * dst_step + dst_off + 2 * k;
        const float u = Elem<T>::get(s[0]), v = Elem<T>::get(s[1]);
        const float2 cs = rotary[(size_t)row * pairs + k];
        d[0] = Elem<T>::put(u * cs.x - v * cs.y);
        d[1] = Elem<T>::put(v * cs.x + u * cs.y);
    }
}

struct ExpandParams
{
    const void* cache;
    void *c, *K;
    const int *slot, *pos, *n, *floor, *pos2;
    unsigned int c_ld, T_max, kv_rank, rot_dim, ld_c, k_ld, T, dim, heads, e0;
};

// grid (rows, entries)
template <class T>
__global__ void __launch_bounds__(256) latent_expand_kernel(const ExpandParams p)
{
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int e = p.e0 + blockIdx.y, r = blockIdx.x;
    const unsigned int before = (unsigned int)(p.pos2[e] - p.floor[e]), to = (unsigned int)p.floor[e] + r;    // rows ahead of the entry's own
    if (r >= before + (unsigned int)p.n[e] || to >= p.T) { return; }
    const T* src = (const T*)p.cache + ((size_t)p.slot[e] * p.T_max + (unsigned int)p.pos[e] - before + r) * p.c_ld;
    T* c = (T*)p.c + (size_t)to * p.ld_c;
    for (unsigned int d = threadIdx.x; d < p.kv_rank; d += blockDim.x) { c[d] = src[d]; }
    for (unsigned int j = threadIdx.x; j < p.heads * p.rot_dim; j += blockDim.x)
    {
        const unsigned int h = j / p.rot_dim, d = j % p.rot_dim;
        ((T*)p.K)[((size_t)h * p.T + to) * p.k_ld + p.dim + d] = src[p.kv_rank + d];
    }
}

template <class T>
static int latent_down(const LatentParams& p, unsigned int tokens, void* stream, bool pdl)
{
    const unsigned int most = p.q_rank > p.kv_rank + p.rot_dim ? p.q_rank : p.kv_rank + p.rot_dim;
    unsigned int threads = 512;
    if (Elem<T>::type == DT_BF16 && (p.q_rank % 8) == 0 && (p.kv_rank % 8) == 0 && (p.rot_dim % 8) == 0 && (p.ld % 8) == 0 && (p.kv_off % 8) == 0
        && (p.ld_cq % 4) == 0 && (p.c_ld % 4) == 0 && (reinterpret_cast<uintptr_t>(p.down) & 15u) == 0 && most <= 8 * threads)
    {
        while (threads > 64 && most <= 8 * (threads / 2)) { threads /= 2; }
        return launch_kernel("latent_down8", latent_down8_kernel, dim3(tokens, 2), dim3(threads), 0, stream, pdl, p);
    }
    while (threads > 64 && threads / 2 * 2 >= most) { threads /= 2; }
    const DecoderDevice* dev = decoder_device();
    if (!dev || (size_t)most * 4 > (size_t)dev->max_smem - 1024) { return -1; }
    return launch_kernel("latent_down", latent_down_kernel<T>, dim3(tokens, 2), dim3(threads), (size_t)most * 4, stream, pdl, p);
}

}    // namespace b200

using namespace b200;

C_EXPORT int cuda_b200_latent_down(int dtype, const cuda_b200_latent* a, const cuda_b200_batch* b, void* stream, unsigned int flags)
{
    if (!a || !b || (dtype != DT_BF16 && dtype != DT_FLOAT)) { return -1; }
    if (b->tokens == 0) { return 0; }
    if (!a->down || !a->cq || !a->cache || !a->q_norm || !a->kv_norm || !a->rotary || !b->slot || !b->pos || !b->start || !b->token_entry || a->q_rank == 0
        || a->kv_rank == 0 || (a->rot_dim % 2) || a->c_ld < a->kv_rank + a->rot_dim || a->T_max == 0)
    {
        return -1;
    }
    LatentParams p;
    p.down = a->down;
    p.cq = a->cq;
    p.cache = a->cache;
    p.q_norm = (const float*)a->q_norm;
    p.kv_norm = (const float*)a->kv_norm;
    p.rotary = (const float2*)a->rotary;
    p.slot = (const int*)b->slot;
    p.pos = (const int*)b->pos;
    p.start = (const int*)b->start;
    p.token_entry = (const int*)b->token_entry;
    p.ld = a->ld;
    p.ld_cq = a->ld_cq;
    p.kv_off = a->kv_off;
    p.q_rank = a->q_rank;
    p.kv_rank = a->kv_rank;
    p.rot_dim = a->rot_dim;
    p.c_ld = a->c_ld;
    p.T_max = a->T_max;
    p.t0 = b->first_token;
    p.eps = a->eps;
    const bool pdl = (flags & 1u) != 0;
    return dtype == DT_BF16 ? latent_down<__nv_bfloat16>(p, b->tokens, stream, pdl) : latent_down<float>(p, b->tokens, stream, pdl);
}

C_EXPORT int cuda_b200_latent_query(int dtype, const void* src, unsigned int ld_src, unsigned int src_step, unsigned int src_off, void* dst,
    unsigned int ld_dst, unsigned int dst_step, unsigned int dst_off, unsigned int heads, unsigned int rot_dim, const void* rotary, unsigned int T_max,
    const cuda_b200_batch* b, void* stream, unsigned int flags)
{
    if (!src || !dst || !b || (rot_dim % 2) || (dtype != DT_BF16 && dtype != DT_FLOAT)) { return -1; }
    if (b->tokens == 0 || heads == 0 || rot_dim == 0) { return 0; }
    if (!rotary || !b->pos || !b->start || !b->token_entry) { return -1; }
    const bool pdl = (flags & 1u) != 0;
    auto run = [&](auto zero) {
        using T = decltype(zero);
        return launch_kernel("latent_query", latent_query_kernel<T>, dim3(b->tokens), dim3(256), 0, stream, pdl, (const T*)src, ld_src, src_step, src_off, (T*)dst,
            ld_dst, dst_step, dst_off, heads, rot_dim / 2, (const float2*)rotary, T_max, (const int*)b->pos, (const int*)b->start, (const int*)b->token_entry,
            b->first_token);
    };
    return dtype == DT_BF16 ? run(__nv_bfloat16()) : run(0.f);
}

C_EXPORT int cuda_b200_latent_expand(int dtype, const cuda_b200_expand* a, const cuda_b200_batch* b, void* stream, unsigned int flags)
{
    if (!a || !b || (dtype != DT_BF16 && dtype != DT_FLOAT)) { return -1; }
    if (b->entries == 0 || a->max_rows == 0) { return 0; }
    if (!a->cache || !a->c || !a->K || !a->floor || !a->pos2 || !b->slot || !b->pos || !b->n || a->k_ld < a->dim + a->rot_dim
        || a->c_ld < a->kv_rank + a->rot_dim || a->ld_c < a->kv_rank || b->entries > 65535u)
    {
        return -1;
    }
    ExpandParams p;
    p.cache = a->cache;
    p.c = a->c;
    p.K = a->K;
    p.slot = (const int*)b->slot;
    p.pos = (const int*)b->pos;
    p.n = (const int*)b->n;
    p.floor = (const int*)a->floor;
    p.pos2 = (const int*)a->pos2;
    p.c_ld = a->c_ld;
    p.T_max = a->T_max;
    p.kv_rank = a->kv_rank;
    p.rot_dim = a->rot_dim;
    p.ld_c = a->ld_c;
    p.k_ld = a->k_ld;
    p.T = a->T;
    p.dim = a->dim;
    p.heads = a->heads;
    p.e0 = b->first_entry;
    const bool pdl = (flags & 1u) != 0;
    auto run = [&](auto kernel) { return launch_kernel("latent_expand", kernel, dim3(a->max_rows, b->entries), dim3(256), 0, stream, pdl, p); };
    return dtype == DT_BF16 ? run(latent_expand_kernel<__nv_bfloat16>) : run(latent_expand_kernel<float>);
}
