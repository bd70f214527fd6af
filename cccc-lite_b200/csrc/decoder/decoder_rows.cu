// Row operations of a decoder layer: scaled embedding, branch addition + norm, table of rotations, routing to experts, row
// gather, greedy choice over float logits.
#include "decoder_common.cuh"

#include <cfloat>

namespace b200
{

// Row strides are multiples of four elements: quads of columns, the last one possibly into the padding.
template <class T>
__global__ void __launch_bounds__(256) embed_f32_kernel(const int* __restrict__ ids, const T* __restrict__ table, unsigned int ldt,
    float* __restrict__ X, unsigned int ldx, unsigned int width, unsigned int vocab, float scale)
{
    grid_dependency_launch();
    grid_dependency_wait();
    const int id = ids[blockIdx.x];
    const bool ok = id >= 0 && (unsigned int)id < vocab;
    const T* src = table + (size_t)(ok ? id : 0) * ldt;
    float* dst = X + (size_t)blockIdx.x * ldx;
#pragma unroll 4
    for (unsigned int i = threadIdx.x; i < (width + 3) / 4; i += blockDim.x)
    {
        float4 v = ok ? load4(src + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        v.x *= scale;
        v.y *= scale;
        v.z *= scale;
        v.w *= scale;
        store4(dst + 4 * i, v);
    }
}

// ---- branch addition + norm ------------------------------------------------------------------------
__device__ __forceinline__ float block_sum(float v, float* part)
{
    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    v = warp_sum(v);
    __syncthreads();    // part may still be read from the previous sum
    if (lane == 0) { part[warp] = v; }
    __syncthreads();
    return warp_sum(lane < warps ? part[lane] : 0.f);
}

struct NormParams
{
    float* X;
    const float *weight, *bias;
    void* out;
    const void* Y;
    const int* slot_row;
    const float* slot_weight;
    const int* rows;
    const float *branch, *branch_weight;
    unsigned int width, ldx, ldo, ldy, slots, ldb;
    int kind;
    float eps;
};

// One CTA per row.  The row lives in shared memory as floats; quads of columns per thread (row strides are multiples
// of four elements, so the last quad may cover padding columns, which take no part in the sums and are not stored).
enum
{
    ADD_NOTHING,
    ADD_SLOTS,     // experts' outputs
    ADD_BRANCH     // a branch that is normalised itself
};

template <class T, int ADD>
__global__ void __launch_bounds__(1024) norm_rows_kernel(const NormParams p)
{
    extern __shared__ __align__(16) float nr_row[];
    __shared__ float part[32];
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int r = p.rows ? (unsigned int)p.rows[blockIdx.x] : blockIdx.x;
    float* x = p.X + (size_t)r * p.ldx;
    const unsigned int quads = (p.width + 3) / 4;
    const T* Y = (const T*)p.Y;
    float bmean = 0.f, binv = 0.f;
    if (ADD == ADD_BRANCH)
    {
        const float* b = p.branch + (size_t)r * p.ldb;
        auto live = [&](unsigned int i, int j) { return 4 * i + j < p.width; };
        float s = 0.f;
#pragma unroll 4
        for (unsigned int i = threadIdx.x; i < quads; i += blockDim.x)
        {
            const float4 v = load4(b + 4 * i);
            *reinterpret_cast<float4*>(nr_row + 4 * i) = v;
            s += v.x + (live(i, 1) ? v.y : 0.f) + (live(i, 2) ? v.z : 0.f) + (live(i, 3) ? v.w : 0.f);
        }
        if (p.kind == B200_NORM_LAYER) { bmean = block_sum(s, part) / (float)p.width; }
        s = 0.f;
        for (unsigned int i = threadIdx.x; i < quads; i += blockDim.x)
        {
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                const float v = nr_row[4 * i + j] - bmean;
                if (live(i, j)) { s += v * v; }
            }
        }
        binv = 1.0f / sqrtf(block_sum(s, part) / (float)p.width + p.eps);
    }
    float sum = 0.f;
#pragma unroll 4
    for (unsigned int i = threadIdx.x; i < quads; i += blockDim.x)
    {
        float4 v = load4(x + 4 * i);
        if (ADD == ADD_BRANCH)
        {
            const float4 b = *reinterpret_cast<float4*>(nr_row + 4 * i);
            auto w = [&](int j) { return p.branch_weight && 4 * i + j < p.width ? p.branch_weight[4 * i + j] : 1.f; };
            v.x += (b.x - bmean) * binv * w(0);
            v.y += (b.y - bmean) * binv * w(1);
            v.z += (b.z - bmean) * binv * w(2);
            v.w += (b.w - bmean) * binv * w(3);
            store4(x + 4 * i, v);
        }
        if (ADD == ADD_SLOTS)
        {
#pragma unroll 4
            for (unsigned int s = 0; s < p.slots; s++)
            {
                const float w = p.slot_weight[(size_t)blockIdx.x * p.slots + s];
                const float4 y = load4(Y + (size_t)p.slot_row[(size_t)blockIdx.x * p.slots + s] * p.ldy + 4 * i);
                v.x += w * y.x;
                v.y += w * y.y;
                v.z += w * y.z;
                v.w += w * y.w;
            }
            store4(x + 4 * i, v);
        }
        if (4 * i + 3 < p.width) { sum += (v.x + v.y) + (v.z + v.w); }
        else
        {
            sum += v.x + (4 * i + 1 < p.width ? v.y : 0.f) + (4 * i + 2 < p.width ? v.z : 0.f);
        }
        *reinterpret_cast<float4*>(nr_row + 4 * i) = v;
    }
    if (!p.out) { return; }
    float mean = 0.f;
    if (p.kind == B200_NORM_LAYER) { mean = block_sum(sum, part) / (float)p.width; }
    float sq = 0.f;
    for (unsigned int i = threadIdx.x; i < quads; i += blockDim.x)
    {
        const float4 v = *reinterpret_cast<float4*>(nr_row + 4 * i);
        const float a[4] = { v.x - mean, v.y - mean, v.z - mean, v.w - mean };
#pragma unroll
        for (int j = 0; j < 4; j++)
        {
            if (4 * i + j < p.width) { sq += a[j] * a[j]; }
        }
    }
    const float inv = 1.0f / sqrtf(block_sum(sq, part) / (float)p.width + p.eps);
    T* out = (T*)p.out + (size_t)blockIdx.x * p.ldo;
    for (unsigned int i = threadIdx.x; i < quads; i += blockDim.x)
    {
        const float4 v = *reinterpret_cast<float4*>(nr_row + 4 * i);
        float a[4] = { v.x, v.y, v.z, v.w };
        const bool whole = 4 * i + 3 < p.width;
#pragma unroll
        for (int j = 0; j < 4; j++)
        {
            const unsigned int c = 4 * i + j;
            if (c < p.width)
            {
                a[j] = (a[j] - mean) * inv * (p.weight ? p.weight[c] : 1.f);
                if (p.kind == B200_NORM_LAYER && p.bias) { a[j] += p.bias[c]; }
                if (!whole) { out[c] = Elem<T>::put(a[j]); }
            }
        }
        if (whole) { store4(out + 4 * i, make_float4(a[0], a[1], a[2], a[3])); }
    }
}

// ---- rotations -------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) rotary_table_kernel(float2* __restrict__ table, unsigned int pairs, unsigned int dims, double base)
{
    const unsigned int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= pairs) { return; }
    double s, c;
    sincos((double)blockIdx.x * pow(base, -2.0 * (double)i / (double)dims), &s, &c);
    table[(size_t)blockIdx.x * pairs + i] = make_float2((float)c, (float)s);
}

// ---- routing ---------------------------------------------------------------------------------------
struct RouteParams
{
    const float* logits;
    int* pair_row;
    float* pair_weight;
    int* row_token;
    int* group_offset;
    int* active;
    float* shared_weight;
    int* choice;
    int* counters;    // [experts] pairs per expert
    unsigned int n, ldl, experts, top, active_cap;
    int sg_col;
};

// One warp chooses for token t: z holds its logits (clobbered), chosen / weight receive `top` entries.  All lanes return
// with both visible to the warp.
__device__ __forceinline__ void warp_choose(float* z, int* chosen, float* weight, const float* logits, unsigned int experts, unsigned int top,
    unsigned int lane)
{
    for (unsigned int e = lane; e < experts; e += 32)
    {
        const float v = logits[e];
        z[e] = v >= -FLT_MAX ? v : -FLT_MAX;    // NaN and -inf rank last but stay choosable
    }
    __syncwarp();
    float z0 = 0.f, total = 0.f;
    for (unsigned int s = 0; s < top; s++)
    {
        float best = -INFINITY;
        int bi = 0x7FFFFFFF;
        for (unsigned int e = lane; e < experts; e += 32)
        {
            if (z[e] > best)
            {
                best = z[e];
                bi = (int)e;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
        {
            const float ob = __shfl_xor_sync(0xFFFFFFFFu, best, o);
            const int oi = __shfl_xor_sync(0xFFFFFFFFu, bi, o);
            if (ob > best || (ob == best && oi < bi))
            {
                best = ob;
                bi = oi;
            }
        }
        if (s == 0) { z0 = best; }
        const float ex = expf(best - z0);
        total += ex;
        if (lane == 0)
        {
            z[bi] = -INFINITY;
            chosen[s] = bi;
            weight[s] = ex;
        }
        __syncwarp();
    }
    for (unsigned int s = lane; s < top; s += 32) { weight[s] = weight[s] / total; }
    __syncwarp();
}

// Exclusive offsets of counts[0..experts) into off[0..experts], by one warp; optionally the list of non-empty groups.
__device__ __forceinline__ void warp_offsets(const int* counts, int* off, int* active, unsigned int active_cap, unsigned int experts, unsigned int lane)
{
    int base = 0;
    unsigned int live = 0;
    for (unsigned int e0 = 0; e0 < experts; e0 += 32)
    {
        const int c = e0 + lane < experts ? counts[e0 + lane] : 0;
        int inc = c;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1)
        {
            const int v = __shfl_up_sync(0xFFFFFFFFu, inc, o);
            if (lane >= (unsigned int)o) { inc += v; }
        }
        if (e0 + lane < experts) { off[e0 + lane] = base + inc - c; }
        const unsigned int m = __ballot_sync(0xFFFFFFFFu, c > 0);
        if (active != nullptr && c > 0)
        {
            const unsigned int at = live + __popc(m & ((1u << lane) - 1u));
            if (at < active_cap) { active[at] = (int)(e0 + lane); }
        }
        live += __popc(m);
        base += __shfl_sync(0xFFFFFFFFu, inc, 31);
    }
    if (lane == 0) { off[experts] = base; }
    if (active != nullptr)
    {
        for (unsigned int i = live + lane; i < active_cap; i += 32) { active[i] = -1; }
    }
}

// Few tokens: everything in one CTA.  Shared memory: per warp experts floats + top floats + top ints; then the counts
// and offsets.
__global__ void __launch_bounds__(1024) route_small_kernel(const RouteParams p)
{
    extern __shared__ __align__(16) float rs_smem[];
    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    float* z = rs_smem + (size_t)warp * (p.experts + 2 * p.top);
    float* weight = z + p.experts;
    int* chosen = reinterpret_cast<int*>(weight + p.top);
    int* counts = reinterpret_cast<int*>(rs_smem + (size_t)warps * (p.experts + 2 * p.top));
    int* off = counts + p.experts;
    for (unsigned int e = threadIdx.x; e < p.experts; e += blockDim.x) { counts[e] = 0; }
    grid_dependency_launch();
    grid_dependency_wait();
    __syncthreads();
    for (unsigned int t = warp; t < p.n; t += warps)
    {
        const float* l = p.logits + (size_t)t * p.ldl;
        warp_choose(z, chosen, weight, l, p.experts, p.top, lane);
        for (unsigned int s = lane; s < p.top; s += 32)
        {
            const size_t i = (size_t)t * p.top + s;
            p.pair_weight[i] = weight[s];
            p.choice[i] = chosen[s];
            p.pair_row[i] = atomicAdd(counts + chosen[s], 1);    // rank within the expert
        }
        if (p.sg_col >= 0 && lane == 0) { p.shared_weight[t] = sigmoid_f32(l[p.sg_col]); }
    }
    __syncthreads();
    if (warp == 0) { warp_offsets(counts, off, p.active, p.active_cap, p.experts, lane); }
    __syncthreads();
    for (unsigned int e = threadIdx.x; e <= p.experts; e += blockDim.x) { p.group_offset[e] = off[e]; }
    for (unsigned int i = threadIdx.x; i < p.n * p.top; i += blockDim.x)
    {
        const int row = off[p.choice[i]] + p.pair_row[i];
        p.pair_row[i] = row;
        p.row_token[row] = (int)(i / p.top);
    }
}

constexpr unsigned int kRouteTokens = 8;    // tokens per CTA of the two-kernel form

__global__ void __launch_bounds__(256) route_choose_kernel(const RouteParams p)
{
    extern __shared__ __align__(16) float rc_smem[];
    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    float* z = rc_smem + (size_t)warp * (p.experts + 2 * p.top);
    float* weight = z + p.experts;
    int* chosen = reinterpret_cast<int*>(weight + p.top);
    int* counts = reinterpret_cast<int*>(rc_smem + (size_t)warps * (p.experts + 2 * p.top));
    int* base = counts + p.experts;
    for (unsigned int e = threadIdx.x; e < p.experts; e += blockDim.x) { counts[e] = 0; }
    grid_dependency_launch();
    grid_dependency_wait();
    __syncthreads();
    const unsigned int t0 = blockIdx.x * kRouteTokens, t1 = min(t0 + kRouteTokens, p.n);
    for (unsigned int t = t0 + warp; t < t1; t += warps)
    {
        const float* l = p.logits + (size_t)t * p.ldl;
        warp_choose(z, chosen, weight, l, p.experts, p.top, lane);
        for (unsigned int s = lane; s < p.top; s += 32)
        {
            const size_t i = (size_t)t * p.top + s;
            p.pair_weight[i] = weight[s];
            p.choice[i] = chosen[s];
            p.pair_row[i] = atomicAdd(counts + chosen[s], 1);
        }
        if (p.sg_col >= 0 && lane == 0) { p.shared_weight[t] = sigmoid_f32(l[p.sg_col]); }
    }
    __syncthreads();
    for (unsigned int e = threadIdx.x; e < p.experts; e += blockDim.x) { base[e] = counts[e] ? atomicAdd(p.counters + e, counts[e]) : 0; }
    __syncthreads();
    for (unsigned int i = t0 * p.top + threadIdx.x; i < t1 * p.top; i += blockDim.x) { p.pair_row[i] += base[p.choice[i]]; }
}

__global__ void __launch_bounds__(256) route_place_kernel(const RouteParams p)
{
    extern __shared__ __align__(16) int rp_off[];    // experts + 1
    grid_dependency_launch();
    grid_dependency_wait();
    if (threadIdx.x < 32)
    {
        warp_offsets(p.counters, rp_off, blockIdx.x == 0 ? p.active : nullptr, p.active_cap, p.experts, threadIdx.x);
    }
    __syncthreads();
    if (blockIdx.x == 0)
    {
        for (unsigned int e = threadIdx.x; e <= p.experts; e += blockDim.x) { p.group_offset[e] = rp_off[e]; }
    }
    for (unsigned int i = blockIdx.x * blockDim.x + threadIdx.x; i < p.n * p.top; i += gridDim.x * blockDim.x)
    {
        const int row = rp_off[p.choice[i]] + p.pair_row[i];
        p.pair_row[i] = row;
        p.row_token[row] = (int)(i / p.top);
    }
}

// ---- gather, argmax ----------------------------------------------------------------------------------
__global__ void __launch_bounds__(128) gather_rows_kernel(const uint4* __restrict__ X, unsigned int ldx4, const int* __restrict__ row_token,
    uint4* __restrict__ out, unsigned int ldo4, unsigned int cols4)
{
    grid_dependency_launch();
    grid_dependency_wait();
    const uint4* src = X + (size_t)row_token[blockIdx.x] * ldx4;
    uint4* dst = out + (size_t)blockIdx.x * ldo4;
    for (unsigned int i = threadIdx.x; i < cols4; i += blockDim.x) { dst[i] = src[i]; }
}

__global__ void __launch_bounds__(1024) argmax_f32_kernel(const float* __restrict__ logits, unsigned int cols, unsigned int ld, int* __restrict__ idx,
    float* __restrict__ val)
{
    __shared__ float bv[32];
    __shared__ int bi[32];
    grid_dependency_launch();
    grid_dependency_wait();
    const float* row = logits + (size_t)blockIdx.x * ld;
    float best = -INFINITY;
    int at = 0x7FFFFFFF;
    auto see = [&](float v, unsigned int i) {
        if (v > best || (v == best && at == 0x7FFFFFFF))    // the second case: a leading -inf
        {
            best = v;
            at = (int)i;
        }
    };
    unsigned int done = 0;
    if ((ld % 4) == 0 && (reinterpret_cast<uintptr_t>(logits) & 15u) == 0)
    {
        // four quads of a thread in flight; its indices still grow, so that the first of equal values stays
        const float4* quad = reinterpret_cast<const float4*>(row);
        for (; done + 16 * blockDim.x <= cols; done += 16 * blockDim.x)
        {
            float4 v[4];
#pragma unroll
            for (int j = 0; j < 4; j++) { v[j] = quad[done / 4 + j * blockDim.x + threadIdx.x]; }
#pragma unroll
            for (int j = 0; j < 4; j++)
            {
                const unsigned int i = done + 4 * (j * blockDim.x + threadIdx.x);
                see(v[j].x, i);
                see(v[j].y, i + 1);
                see(v[j].z, i + 2);
                see(v[j].w, i + 3);
            }
        }
    }
    for (unsigned int i = done + threadIdx.x; i < cols; i += blockDim.x) { see(row[i], i); }
    auto take = [&](float ov, int oi) {
        if (ov > best || (ov == best && oi < at))
        {
            best = ov;
            at = oi;
        }
    };
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) { take(__shfl_xor_sync(0xFFFFFFFFu, best, o), __shfl_xor_sync(0xFFFFFFFFu, at, o)); }
    if ((threadIdx.x & 31) == 0)
    {
        bv[threadIdx.x >> 5] = best;
        bi[threadIdx.x >> 5] = at;
    }
    __syncthreads();
    if (threadIdx.x < 32)
    {
        best = threadIdx.x < blockDim.x / 32 ? bv[threadIdx.x] : -INFINITY;
        at = threadIdx.x < blockDim.x / 32 ? bi[threadIdx.x] : 0x7FFFFFFF;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) { take(__shfl_xor_sync(0xFFFFFFFFu, best, o), __shfl_xor_sync(0xFFFFFFFFu, at, o)); }
        if (threadIdx.x == 0)
        {
            idx[blockIdx.x] = at == 0x7FFFFFFF ? -1 : at;
            if (val) { val[blockIdx.x] = best; }
        }
    }
}

}    // namespace b200

using namespace b200;

C_EXPORT int cuda_b200_embed_f32(int dtype, const void* ids, const void* table, unsigned int ld_table, void* X, unsigned int ldx, unsigned int n,
    unsigned int width, unsigned int vocab, float scale, void* stream, unsigned int flags)
{
    if (n == 0) { return 0; }
    if (!ids || !table || !X || (ld_table % 4) || (ldx % 4)) { return -1; }
    const bool pdl = (flags & 1u) != 0;
    if (dtype == DT_BF16)
    {
        return launch_kernel("embed_f32", embed_f32_kernel<__nv_bfloat16>, dim3(n), dim3(256), 0, stream, pdl, (const int*)ids,
            (const __nv_bfloat16*)table, ld_table, (float*)X, ldx, width, vocab, scale);
    }
    if (dtype == DT_FLOAT)
    {
        return launch_kernel("embed_f32", embed_f32_kernel<float>, dim3(n), dim3(256), 0, stream, pdl, (const int*)ids, (const float*)table, ld_table,
            (float*)X, ldx, width, vocab, scale);
    }
    return -1;
}

C_EXPORT int cuda_b200_rotary_table(void* table, unsigned int rows, unsigned int dims, double base, void* stream)
{
    if (rows == 0 || dims == 0) { return 0; }
    if (!table || (dims % 2) || !(base > 0.0)) { return -1; }
    const unsigned int pairs = dims / 2, threads = pairs < 256 ? (pairs + 31) / 32 * 32 : 256;
    return launch_kernel("rotary_table", rotary_table_kernel, dim3(rows, (pairs + threads - 1) / threads), dim3(threads), 0, stream, false, (float2*)table, pairs,
        dims, base);
}

C_EXPORT int cuda_b200_norm_rows(int dtype, const cuda_b200_norm* a, void* stream, unsigned int flags)
{
    if (!a || a->n == 0) { return a ? 0 : -1; }
    if (!a->X || a->width == 0 || (a->ldx % 4) || (a->out && (a->ldo % 4)) || (dtype != DT_BF16 && dtype != DT_FLOAT)) { return -1; }
    if (a->kind != B200_NORM_RMS && a->kind != B200_NORM_LAYER) { return -1; }
    if (a->slots && (!a->Y || !a->slot_row || !a->slot_weight || a->rows || (a->ldy % 4))) { return -1; }
    if (a->branch && (a->slots || a->rows || (a->ldb % 4) || a->ldb < a->width)) { return -1; }
    const DecoderDevice* dev = decoder_device();
    const size_t smem = ((size_t)a->width + 3) / 4 * 16;
    if (!dev || smem > (size_t)dev->max_smem - 1024) { return -1; }
    NormParams p;
    p.X = (float*)a->X;
    p.weight = (const float*)a->weight;
    p.bias = (const float*)a->bias;
    p.out = a->out;
    p.Y = a->Y;
    p.slot_row = (const int*)a->slot_row;
    p.slot_weight = (const float*)a->slot_weight;
    p.rows = (const int*)a->rows;
    p.branch = (const float*)a->branch;
    p.branch_weight = (const float*)a->branch_weight;
    p.ldb = a->ldb;
    p.width = a->width;
    p.ldx = a->ldx;
    p.ldo = a->ldo;
    p.ldy = a->ldy;
    p.slots = a->slots;
    p.kind = a->kind;
    p.eps = a->eps;
    // a few rows: the whole SM on one row; many: smaller CTAs, several per SM
    unsigned int threads = a->n <= 64 ? 1024u : 256u;
    while (threads > 64 && threads / 2 * 4 >= a->width) { threads /= 2; }
    const bool pdl = (flags & 1u) != 0;
    auto run = [&](auto kernel) { return launch_kernel("norm_rows", kernel, dim3(a->n), dim3(threads), smem, stream, pdl, p); };
    auto pick = [&](auto zero) {
        using T = decltype(zero);
        if (p.branch) { return run(norm_rows_kernel<T, ADD_BRANCH>); }
        return p.slots ? run(norm_rows_kernel<T, ADD_SLOTS>) : run(norm_rows_kernel<T, ADD_NOTHING>);
    };
    return dtype == DT_BF16 ? pick(__nv_bfloat16()) : pick(0.f);
}

C_EXPORT int cuda_b200_route_rows(const cuda_b200_route* a, void* stream, unsigned int flags)
{
    if (!a || a->n == 0) { return a ? 0 : -1; }
    if (!a->logits || !a->pair_row || !a->pair_weight || !a->row_token || !a->group_offset || !a->choice || !a->counters || a->top == 0
        || a->top > a->experts || a->experts > 4096 || (a->sg_col >= 0 && !a->shared_weight))
    {
        return -1;
    }
    RouteParams p;
    p.logits = (const float*)a->logits;
    p.pair_row = (int*)a->pair_row;
    p.pair_weight = (float*)a->pair_weight;
    p.row_token = (int*)a->row_token;
    p.group_offset = (int*)a->group_offset;
    p.active = (int*)a->active;
    p.shared_weight = (float*)a->shared_weight;
    p.choice = (int*)a->choice;
    p.counters = (int*)a->counters;
    p.n = a->n;
    p.ldl = a->ldl;
    p.experts = a->experts;
    p.top = a->top;
    p.active_cap = a->active ? a->active_cap : 0;
    p.sg_col = a->sg_col;
    const bool pdl = (flags & 1u) != 0;
    const DecoderDevice* dev = decoder_device();
    if (!dev) { return 1; }
    auto smem_for = [&](unsigned int warps) { return ((size_t)warps * (p.experts + 2 * p.top) + 2 * p.experts + 1) * 4; };
    if (a->n <= 64)
    {
        unsigned int warps = a->n < 32 ? a->n : 32;
        if (warps < 4) { warps = 4; }    // the tail loops want a few warps
        while (warps > 1 && smem_for(warps) > 160 * 1024) { warps /= 2; }
        if (smem_for(warps) > (size_t)dev->max_smem) { return -1; }
        return launch_kernel("route_small", route_small_kernel, dim3(1), dim3(32 * warps), smem_for(warps), stream, pdl, p);
    }
    if (smem_for(8) > (size_t)dev->max_smem) { return -1; }
    if (cudaMemsetAsync(p.counters, 0, (size_t)p.experts * 4, (cudaStream_t)stream) != cudaSuccess) { return report_launch("route_rows") ? 1 : 1; }
    int rc = launch_kernel("route_choose", route_choose_kernel, dim3((p.n + kRouteTokens - 1) / kRouteTokens), dim3(256), smem_for(8), stream, false, p);
    if (rc) { return rc; }
    const unsigned int grid = (p.n * p.top + 1023) / 1024;
    return launch_kernel("route_place", route_place_kernel, dim3(grid < 512 ? grid : 512), dim3(256), ((size_t)p.experts + 1) * 4, stream, pdl, p);
}

C_EXPORT int cuda_b200_gather_rows(int dtype, const void* X, unsigned int ldx, const void* row_token, void* out, unsigned int ldo, unsigned int n,
    unsigned int width, void* stream, unsigned int flags)
{
    if (n == 0) { return 0; }
    const unsigned int per = dtype == DT_BF16 ? 8 : 4;
    if (!X || !row_token || !out || (dtype != DT_BF16 && dtype != DT_FLOAT) || (ldx % per) || (ldo % per)) { return -1; }
    return launch_kernel("gather_rows", gather_rows_kernel, dim3(n), dim3(128), 0, stream, (flags & 1u) != 0, (const uint4*)X, ldx / per,
        (const int*)row_token, (uint4*)out, ldo / per, (width + per - 1) / per);
}

C_EXPORT int cuda_b200_argmax_f32(const void* logits, unsigned int rows, unsigned int cols, unsigned int ld, void* idx, void* val, void* stream,
    unsigned int flags)
{
    if (rows == 0) { return 0; }
    if (!logits || !idx || cols == 0) { return -1; }
    return launch_kernel("argmax_f32", argmax_f32_kernel, dim3(rows), dim3(1024), 0, stream, (flags & 1u) != 0, (const float*)logits, cols, ld,
        (int*)idx, (float*)val);
}
