// What precedes attention (norms and rotation of q and k, value mixing, cache append) and the plain attention kernel of the
// float mode.
#include "attention.cuh"

namespace b200
{

// A warp per (token, head): q heads, then k heads, then v heads.
template <class T>
__global__ void __launch_bounds__(256) attention_append_kernel(const AttnParams p)
{
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int i = p.t0 + blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int e = p.token_entry[i];
    const unsigned int row = (unsigned int)(p.pos[e] + ((int)i - p.start[e]));
    if (row >= p.T_max) { return; }
    T* x = (T*)p.qkvg + (size_t)i * p.ld;
    const size_t kv0 = (size_t)p.slot[e] * p.Hkv;
    const unsigned int h = blockIdx.y * warps + warp;
    if (h < p.H + 2 * p.Hkv)
    {
        if (h < p.H + p.Hkv)
        {
            const bool is_q = h < p.H;
            const unsigned int kh = h - p.H;
            T* src = is_q ? x + (size_t)h * p.dim : x + p.k_off + (size_t)kh * p.dim;
            T* dst = is_q ? src : (T*)p.k_cache + ((kv0 + kh) * p.T_max + row) * p.k_ld;
            if (is_q && !p.qk_norm) { return; }
            float inv = 1.f;
            // rows of up to 128 elements in whole quads: one load and one store per lane
            if ((p.dim % 4) == 0 && p.dim <= 128 && (p.ld % 4) == 0 && (p.k_off % 4) == 0)
            {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (4 * lane < p.dim) { v = load4(src + 4 * lane); }
                if (p.qk_norm)
                {
                    inv = 1.0f / sqrtf(warp_sum((v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w)) / (float)p.dim + p.eps);
                }
                if (4 * lane < p.dim) { store4(dst + 4 * lane, make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv)); }
                return;
            }
            if (p.qk_norm)
            {
                float sq = 0.f;
                for (unsigned int d = lane; d < p.dim; d += 32)
                {
                    const float v = Elem<T>::get(src[d]);
                    sq += v * v;
                }
                inv = 1.0f / sqrtf(warp_sum(sq) / (float)p.dim + p.eps);
            }
            for (unsigned int d = lane; d < p.dim; d += 32) { dst[d] = Elem<T>::put(Elem<T>::get(src[d]) * inv); }
        }
        else
        {
            const unsigned int vh = h - p.H - p.Hkv;
            const T* src = x + p.v_off + (size_t)vh * p.vdim;
            T* dst = (T*)p.v_cache + ((kv0 + vh) * p.T_max + row) * p.v_ld;
            T* first = p.v_mix ? (T*)p.v_first + (size_t)i * p.v_first_ld + (size_t)vh * p.vdim : nullptr;
            for (unsigned int d = lane; d < p.vdim; d += 32)
            {
                float v = Elem<T>::get(src[d]);
                if (p.v_mix == 1) { first[d] = src[d]; }
                else if (p.v_mix == 2) { v = (1.0f - p.lambda) * v + p.lambda * Elem<T>::get(first[d]); }
                dst[d] = Elem<T>::put(v);
            }
        }
    }
}

// A CTA per token and part (0: q, 1: k and v), for norms over a whole projection and rotations.  The part's row lives in shared
// memory as floats.
template <class T>
__global__ void __launch_bounds__(512) attention_prepare_kernel(const AttnParams p)
{
    extern __shared__ float ar_row[];
    __shared__ float sums[16];
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int i = p.t0 + blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    const bool is_q = blockIdx.y == 0;
    const int e = p.token_entry[i];
    const unsigned int row = (unsigned int)(p.pos[e] + ((int)i - p.start[e]));
    if (row >= p.T_max) { return; }
    T* x = (T*)p.qkvg + (size_t)i * p.ld;
    const size_t kv0 = (size_t)p.slot[e] * p.Hkv;
    const unsigned int heads = is_q ? p.H : p.Hkv, all = heads * p.dim;
    const T* src = is_q ? x : x + p.k_off;
    const float* w = is_q ? p.q_norm : p.k_norm;
    float sq = 0.f;
    for (unsigned int d = tid; d < all; d += blockDim.x)
    {
        const float v = Elem<T>::get(src[d]);
        ar_row[d] = v;
        sq += v * v;
    }
    if (w != nullptr)
    {
        sq = warp_sum(sq);
        if (lane == 0) { sums[warp] = sq; }
        __syncthreads();
        const float inv = 1.0f / sqrtf(warp_sum(lane < warps ? sums[lane] : 0.f) / (float)all + p.eps);
        for (unsigned int d = tid; d < all; d += blockDim.x) { ar_row[d] *= inv * w[d]; }
    }
    __syncthreads();
    if (p.qk_norm)
    {
        for (unsigned int h = warp; h < heads; h += warps)
        {
            float* r = ar_row + h * p.dim;
            float s = 0.f;
            for (unsigned int d = lane; d < p.dim; d += 32) { s += r[d] * r[d]; }
            const float inv = 1.0f / sqrtf(warp_sum(s) / (float)p.dim + p.eps);
            for (unsigned int d = lane; d < p.dim; d += 32) { r[d] *= inv; }
        }
        __syncthreads();
    }
    const float2* rot = p.rotary + (size_t)row * (p.rot_dims / 2);
    for (unsigned int j = tid; j < all; j += blockDim.x)
    {
        const unsigned int h = j / p.dim, d = j % p.dim;
        const float v = rotated(ar_row + h * p.dim, d, p.rot_dims, p.rot_interleaved != 0, rot);
        T* dst = is_q ? x + j : (T*)p.k_cache + ((kv0 + h) * p.T_max + row) * p.k_ld + d;
        *dst = Elem<T>::put(v);
    }
    if (is_q) { return; }
    for (unsigned int j = tid; j < p.Hkv * p.vdim; j += blockDim.x)
    {
        const T raw = x[p.v_off + j];
        float v = Elem<T>::get(raw);
        if (p.v_mix == 1) { ((T*)p.v_first)[(size_t)i * p.v_first_ld + j] = raw; }
        else if (p.v_mix == 2) { v = (1.0f - p.lambda) * v + p.lambda * Elem<T>::get(((const T*)p.v_first)[(size_t)i * p.v_first_ld + j]); }
        ((T*)p.v_cache)[((kv0 + j / p.vdim) * p.T_max + row) * p.v_ld + j % p.vdim] = Elem<T>::put(v);
    }
}

__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8])
{
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = { u.x, u.y, u.z, u.w };
#pragma unroll
    for (int i = 0; i < 4; i++)
    {
        f[2 * i] = __uint_as_float(w[i] << 16);
        f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
}
__device__ __forceinline__ void load8(const float* p, float (&f)[8])
{
    const float4 a = load4(p), b = load4(p + 4);
    const float v[8] = { a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w };
#pragma unroll
    for (int i = 0; i < 8; i++) { f[i] = v[i]; }
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8])
{
    store4(p, make_float4(f[0], f[1], f[2], f[3]));
    store4(p + 4, make_float4(f[4], f[5], f[6], f[7]));
}

// The same in BF16 by eights, where sizes and offsets allow it: heads and, for pairs that lie apart, half of the rotated part are
// whole eights.  Without unit RMS of single heads.
__global__ void __launch_bounds__(512) attention_prepare8_kernel(const AttnParams p)
{
    __shared__ float sums[16];
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int i = p.t0 + blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    const bool is_q = blockIdx.y == 0;
    const int e = p.token_entry[i];
    const unsigned int row = (unsigned int)(p.pos[e] + ((int)i - p.start[e]));
    if (row >= p.T_max) { return; }
    __nv_bfloat16* x = (__nv_bfloat16*)p.qkvg + (size_t)i * p.ld;
    const size_t kv0 = (size_t)p.slot[e] * p.Hkv;
    const unsigned int per = p.dim / 8, all = (is_q ? p.H : p.Hkv) * per, half = p.rot_dims / 2;
    const __nv_bfloat16* src = is_q ? x : x + p.k_off;
    const float* w = is_q ? p.q_norm : p.k_norm;
    const float2* rot = p.rotary + (size_t)row * half;
    // the eights of the row that a thread turns, with the ones they are turned with (two rounds keep everything in registers)
    constexpr int R = 2;
    float own[R][8], other[R][8], sq = 0.f;
#pragma unroll
    for (int r = 0; r < R; r++)
    {
        const unsigned int c = tid + r * blockDim.x, d = (c % per) * 8;
        if (c < all)
        {
            load8(src + c * 8, own[r]);
            if (d < p.rot_dims && !p.rot_interleaved)
            {
                const unsigned int o = d < half ? c * 8 + half : c * 8 - half;
                load8(src + o, other[r]);
                if (w != nullptr)
                {
                    float wo[8];
                    load8(w + o, wo);
#pragma unroll
                    for (int j = 0; j < 8; j++) { other[r][j] *= wo[j]; }
                }
            }
#pragma unroll
            for (int j = 0; j < 8; j++) { sq += own[r][j] * own[r][j]; }
            if (w != nullptr)
            {
                float wc[8];
                load8(w + c * 8, wc);
#pragma unroll
                for (int j = 0; j < 8; j++) { own[r][j] *= wc[j]; }
            }
        }
    }
    sq = warp_sum(sq);
    if (lane == 0) { sums[warp] = sq; }
    __syncthreads();    // q: also, every eight has been read
    const float inv = w != nullptr ? 1.0f / sqrtf(warp_sum(lane < warps ? sums[lane] : 0.f) / (float)(all * 8) + p.eps) : 1.f;
#pragma unroll
    for (int r = 0; r < R; r++)
    {
        const unsigned int c = tid + r * blockDim.x, h = c / per, d = (c % per) * 8;
        if (c >= all) { continue; }
        float out[8];
#pragma unroll
        for (int j = 0; j < 8; j++) { out[j] = own[r][j] * inv; }
        if (d < p.rot_dims)
        {
            if (p.rot_interleaved)
            {
#pragma unroll
                for (int j = 0; j < 4; j++)
                {
                    const float2 cs = rot[d / 2 + j];
                    const float u = out[2 * j], v = out[2 * j + 1];
                    out[2 * j] = u * cs.x - v * cs.y;
                    out[2 * j + 1] = v * cs.x + u * cs.y;
                }
            }
            else
            {
                const bool second = d >= half;
#pragma unroll
                for (int j = 0; j < 8; j++)
                {
                    const float2 cs = rot[(second ? d - half : d) + j];
                    const float o = other[r][j] * inv;
                    out[j] = second ? out[j] * cs.x + o * cs.y : out[j] * cs.x - o * cs.y;
                }
            }
        }
        store8(is_q ? x + c * 8 : (__nv_bfloat16*)p.k_cache + ((kv0 + h) * p.T_max + row) * p.k_ld + d, out);
    }
    if (is_q) { return; }
    for (unsigned int c = tid; c < p.Hkv * (p.vdim / 8); c += blockDim.x)
    {
        const unsigned int h = c / (p.vdim / 8), d = (c % (p.vdim / 8)) * 8;
        float v[8];
        load8(x + p.v_off + c * 8, v);
        if (p.v_mix)
        {
            __nv_bfloat16* first = (__nv_bfloat16*)p.v_first + (size_t)i * p.v_first_ld + c * 8;
            if (p.v_mix == 1) { store8(first, v); }
            else
            {
                float f[8];
                load8(first, f);
#pragma unroll
                for (int j = 0; j < 8; j++) { v[j] = (1.0f - p.lambda) * v[j] + p.lambda * f[j]; }
            }
        }
        store8((__nv_bfloat16*)p.v_cache + ((kv0 + h) * p.T_max + row) * p.v_ld + d, v);
    }
}

constexpr unsigned int AP_KEYS = 128;

// One CTA per (token, kv head, group of GB query heads): the heads against the cache in chunks of 128 keys with a running
// softmax.
template <class T>
__global__ void __launch_bounds__(128) attention_plain_kernel(const AttnParams p, const unsigned int GB)
{
    extern __shared__ float ap_smem[];
    grid_dependency_launch();
    grid_dependency_wait();
    const unsigned int i = p.t0 + blockIdx.x, kvh = blockIdx.y, g0 = blockIdx.z * GB, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int e = p.token_entry[i];
    const unsigned int row = (unsigned int)(p.pos[e] + ((int)i - p.start[e]));
    const unsigned int keys = min(row + 1u, p.T_max), G = min(GB, p.G - g0), h0 = kvh * p.G + g0;
    float* q = ap_smem;                     // [G][dim]
    float* sc = q + G * p.dim;              // [G][128]
    float* acc = sc + G * AP_KEYS;          // [G][vdim]
    float* ml = acc + G * p.vdim;           // [G][3]: maximum, sum, correction
    const T* x = (const T*)p.qkvg + (size_t)i * p.ld;
    const T* K = (const T*)p.k_cache + (((size_t)p.slot[e] * p.Hkv + kvh) * p.T_max) * p.k_ld;
    const T* V = (const T*)p.v_cache + (((size_t)p.slot[e] * p.Hkv + kvh) * p.T_max) * p.v_ld;
    for (unsigned int j = tid; j < G * p.dim; j += 128) { q[j] = Elem<T>::get(x[(size_t)(h0 + j / p.dim) * p.q_ld + j % p.dim]); }
    for (unsigned int j = tid; j < G * p.vdim; j += 128) { acc[j] = 0.f; }
    for (unsigned int g = tid; g < G; g += 128)
    {
        ml[3 * g] = -INFINITY;
        ml[3 * g + 1] = 0.f;
    }
    __syncthreads();
    for (unsigned int k0 = first_key(p, (unsigned int)e, row + 1u); k0 < keys; k0 += AP_KEYS)
    {
        const unsigned int nk = min(AP_KEYS, keys - k0);
        if (tid < nk)
        {
            const T* kr = K + (size_t)(k0 + tid) * p.k_ld;
            for (unsigned int g = 0; g < G; g++)
            {
                float s = 0.f;
                for (unsigned int d = 0; d < p.dim; d++) { s = fmaf(q[g * p.dim + d], Elem<T>::get(kr[d]), s); }
                sc[g * AP_KEYS + tid] = s * p.scale;
            }
        }
        __syncthreads();
        for (unsigned int g = warp; g < G; g += 4)
        {
            float* s = sc + g * AP_KEYS;
            float m = -INFINITY;
            for (unsigned int j = lane; j < nk; j += 32) { m = fmaxf(m, s[j]); }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) { m = fmaxf(m, __shfl_xor_sync(0xFFFFFFFFu, m, o)); }
            const float mo = ml[3 * g], mn = fmaxf(mo, m);
            float l = 0.f;
            for (unsigned int j = lane; j < nk; j += 32)
            {
                const float w = expf(s[j] - mn);
                s[j] = w;
                l += w;
            }
            l = warp_sum(l);
            __syncwarp();
            if (lane == 0)
            {
                const float c = expf(mo - mn);
                ml[3 * g] = mn;
                ml[3 * g + 1] = ml[3 * g + 1] * c + l;
                ml[3 * g + 2] = c;
            }
        }
        __syncthreads();
        for (unsigned int j = tid; j < G * p.vdim; j += 128)
        {
            const unsigned int g = j / p.vdim, d = j % p.vdim;
            const float* s = sc + g * AP_KEYS;
            float o = acc[j] * ml[3 * g + 2];
            for (unsigned int k = 0; k < nk; k++) { o = fmaf(s[k], Elem<T>::get(V[(size_t)(k0 + k) * p.v_ld + d]), o); }
            acc[j] = o;
        }
        __syncthreads();
    }
    T* out = (T*)p.out + (size_t)i * p.ldo + (size_t)h0 * p.vdim;
    for (unsigned int j = tid; j < G * p.vdim; j += 128)
    {
        const unsigned int g = j / p.vdim;
        float l = ml[3 * g + 1];
        if (p.sink != nullptr) { l += expf(p.sink[h0 + g] - ml[3 * g]); }
        float o = acc[j] / l * head_factor<T>(p, i, h0 + g);
        if (p.gate) { o *= sigmoid_f32(Elem<T>::get(x[p.g_off + (size_t)h0 * p.vdim + j])); }
        out[j] = Elem<T>::put(o);
    }
}

template <class T>
static int attention_append(const AttnParams& p, unsigned int tokens, void* stream, bool pdl)
{
    if (p.q_norm || p.k_norm || p.rot_dims)
    {
        const unsigned int most = (p.H > p.Hkv ? p.H : p.Hkv) * p.dim;
        unsigned int threads = 512;
        const bool eights = Elem<T>::type == DT_BF16 && !p.qk_norm && (p.dim % 8) == 0 && (p.vdim % 8) == 0 && (p.rot_dims % (p.rot_interleaved ? 8 : 16)) == 0
            && (p.ld % 8) == 0 && (p.k_off % 8) == 0 && (p.v_off % 8) == 0 && (p.v_first_ld % 8) == 0 && most <= 2 * 8 * threads;
        if (eights)
        {
            while (threads > 64 && most <= 2 * 8 * (threads / 2)) { threads /= 2; }
            return launch_kernel("attention_prepare8", attention_prepare8_kernel, dim3(tokens, 2), dim3(threads), 0, stream, pdl, p);
        }
        while (threads > 64 && threads / 2 * 4 >= most) { threads /= 2; }
        const DecoderDevice* dev = decoder_device();
        if (!dev || (size_t)most * 4 > (size_t)dev->max_smem - 1024) { return -1; }
        return launch_kernel("attention_prepare", attention_prepare_kernel<T>, dim3(tokens, 2), dim3(threads), (size_t)most * 4, stream, pdl, p);
    }
    const unsigned int heads = p.H + 2 * p.Hkv;
    const unsigned int warps = heads < 8 ? heads : 8;
    return launch_kernel("attention_append", attention_append_kernel<T>, dim3(tokens, (heads + warps - 1) / warps), dim3(32 * warps), 0, stream, pdl, p);
}

template <class T>
static int attention_plain(const AttnParams& p, unsigned int tokens, void* stream, bool pdl)
{
    const DecoderDevice* dev = decoder_device();
    if (!dev) { return 1; }
    const size_t head = (size_t)(p.dim + p.vdim + AP_KEYS + 3) * 4, fit = (size_t)dev->max_smem / head;
    if (fit == 0) { return -1; }
    const unsigned int GB = p.G < fit ? p.G : (unsigned int)fit;
    return launch_kernel("attention_plain", attention_plain_kernel<T>, dim3(tokens, p.Hkv, (p.G + GB - 1) / GB), dim3(128), head * GB, stream, pdl, p, GB);
}

}    // namespace b200

using namespace b200;

static unsigned int vdim_padded(unsigned int vdim) { return (vdim + 15) / 16 * 16; }

C_EXPORT unsigned long long cuda_b200_attention_work_bytes(unsigned int vdim)
{
    return kAttnCounters * 4ull + (unsigned long long)kAttnPartials * 16 * (vdim_padded(vdim) + 2) * 4;
}

C_EXPORT int cuda_b200_attention_rows(int dtype, const cuda_b200_attention* a, const cuda_b200_batch* b, void* stream, unsigned int flags, int kernel)
{
    if (!a || !b) { return -1; }
    if (b->tokens == 0 || b->entries == 0) { return 0; }
    if (!a->qkvg || !a->out || !a->k_cache || !a->v_cache || !a->work || !b->slot || !b->pos || !b->start || !b->n || !b->token_entry) { return -1; }
    auto low = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) != 0; };
    if (low(a->qkvg) || low(a->k_cache) || low(a->v_cache) || low(a->work)) { return -1; }
    if ((dtype != DT_BF16 && dtype != DT_FLOAT) || a->H == 0 || a->Hkv == 0 || (a->H % a->Hkv) || a->dim == 0 || a->vdim == 0 || a->k_ld < a->dim
        || a->v_ld < a->vdim || (a->k_ld % 8) || (a->v_ld % 8) || a->T_max == 0 || (a->v_mix && !a->v_first) || (a->rot_dims % 2) || a->rot_dims > a->dim
        || (a->rot_dims && !a->rotary) || (!a->no_append && a->q_ld != 0 && a->q_ld != a->dim) || (a->q_ld != 0 && a->q_ld < a->dim))
    {
        return -1;
    }
    AttnParams p;
    p.qkvg = a->qkvg;
    p.out = a->out;
    p.k_cache = a->k_cache;
    p.v_cache = a->v_cache;
    p.v_first = a->v_first;
    p.counter = (int*)a->work;
    p.partial = (float*)a->work + kAttnCounters;
    p.slot = (const int*)b->slot;
    p.pos = (const int*)b->pos;
    p.start = (const int*)b->start;
    p.n = (const int*)b->n;
    p.token_entry = (const int*)b->token_entry;
    p.floor = (const int*)b->floor;
    p.q_norm = (const float*)a->q_norm;
    p.k_norm = (const float*)a->k_norm;
    p.sink = (const float*)a->sink;
    p.rotary = (const float2*)a->rotary;
    p.head_gate = a->head_gate;
    p.ld_gate = a->ld_gate;
    p.rot_dims = a->rot_dims;
    p.rot_interleaved = a->rot_interleaved;
    p.window = a->window;
    p.q_ld = a->q_ld ? a->q_ld : a->dim;
    p.e0 = b->first_entry;
    p.t0 = b->first_token;
    p.ld = a->ld;
    p.ldo = a->ldo;
    p.k_off = a->k_off;
    p.v_off = a->v_off;
    p.g_off = a->g_off;
    p.v_first_ld = a->v_first_ld;
    p.H = a->H;
    p.Hkv = a->Hkv;
    p.G = a->H / a->Hkv;
    p.dim = a->dim;
    p.vdim = a->vdim;
    p.k_ld = a->k_ld;
    p.v_ld = a->v_ld;
    p.T_max = a->T_max;
    p.splits = p.row_tiles = 1;
    p.v_mix = a->v_mix;
    p.qk_norm = a->qk_norm;
    p.gate = a->gate;
    p.lambda = a->mix;
    p.eps = a->eps;
    p.scale = a->scale;
    p.fused = 0;
    const bool pdl = (flags & 1u) != 0;
    cudaStream_t st = (cudaStream_t)stream;
    const bool direct = p.dim <= 128 && p.vdim <= 128 && (p.k_ld % 16) == 0 && (p.v_ld % 16) == 0;
    if (dtype == DT_FLOAT) { kernel = 3; }
    if (kernel == 0)
    {
        if (p.k_cache == p.v_cache && p.Hkv == 1 && p.k_ld == p.v_ld && p.dim <= 576 && p.vdim <= 512 && a->slots != 0) { kernel = 6; }
        else if (p.dim > 256 || p.vdim > 256) { kernel = 3; }
        else if (b->max_n * p.G <= 64 || b->max_n <= 4) { kernel = direct ? 4 : 1; }
        else { kernel = a->slots != 0 ? 5 : 2; }
    }
    const bool ready = a->no_append != 0, simple = !p.q_norm && !p.k_norm && p.rot_dims == 0;
    if (kernel == 4 && b->max_n == 1 && !ready && simple)
    {
        p.fused = 1;
        return launch_attention_direct(p, b->entries, 1, b->max_len, st, pdl);
    }
    int rc = ready ? 0 : dtype == DT_BF16 ? attention_append<__nv_bfloat16>(p, b->tokens, st, pdl) : attention_append<float>(p, b->tokens, st, pdl);
    if (rc) { return rc; }
    switch (kernel)
    {
    case 1: return launch_attention_split(p, b->entries, b->max_n, b->max_len, st, pdl);
    case 2: return launch_attention_tiled(p, b->entries, b->max_n, st, pdl);
    case 6: return launch_attention_latent(p, a->slots, b->entries, b->max_n, b->max_len, st, pdl);
    case 5: return launch_attention_tile(p, a->slots, b->entries, b->max_n, st, pdl);
    case 4: return launch_attention_direct(p, b->entries, b->max_n, b->max_len, st, pdl);
    default: return dtype == DT_BF16 ? attention_plain<__nv_bfloat16>(p, b->tokens, st, pdl) : attention_plain<float>(p, b->tokens, st, pdl);
    }
}
