// Linears of a few rows with BF16 weights (weight streaming, HBM-bound), and the linears of the float mode.
//
// The streaming kernel: eight warps, WK of which share 16 (or 2 x 16) output features and take the 64-wide k chunks in turn
// (all eight, or two where k is short).  A lane loads 32 bytes of weight row g and of row g + 8 straight into the A fragments of mma.m16n8k16 - the k order
// inside a chunk is permuted, identically for both operands, so that fragments are whole pieces of a row - and the rows of X
// are the eight B columns.  The next chunks' weights are requested before the current ones are consumed, the first ones of
// a dense member before the previous kernel of the stream has finished.  The warps' partial sums meet in shared memory.
#include "decoder_common.cuh"
#include "../gemv_decode.cuh"
#include "linear.cuh"

namespace b200
{

constexpr int LS_WARPS = 8;

struct LinearLaunch
{
    LinearMember m[LINEAR_MAX_MEMBERS];
    unsigned int count;
};

// 32 bytes of a weight row, read once
__device__ __forceinline__ void ldg_stream(const void* p, uint4& a, uint4& b)
{
    asm volatile("ld.global.nc.L1::no_allocate.L2::evict_first.v8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(a.x), "=r"(a.y), "=r"(a.z), "=r"(a.w), "=r"(b.x), "=r"(b.y), "=r"(b.z), "=r"(b.w)
                 : "l"(p));
}

// NT: row groups of eight; RT: 16-feature tiles per warp; U: chunks per loop turn; WK: warps that share features
template <int NT, int RT, int U, int WK>
__global__ void __launch_bounds__(32 * LS_WARPS, NT == 4 ? 1 : 2) linear_stream_kernel(const __grid_constant__ LinearLaunch L)
{
    constexpr int R = 16 * RT, C = 8 * NT;
    __shared__ float red[LS_WARPS][C][R + 1];
    unsigned int mi = 0;
    if (L.count > 1 && blockIdx.x >= L.m[1].block0) { mi = 1; }
    if (L.count > 2 && blockIdx.x >= L.m[2].block0) { mi = 2; }
    const LinearMember& m = L.m[mi];
    const unsigned int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const unsigned int b = blockIdx.x - m.block0;
    const bool gated = activation_gated(m.activation);
    const unsigned int F = gated ? R / 2 : R;    // output features of a warp
    const unsigned int wk = warp % WK, wf = warp / WK;
    const unsigned int fb = b % m.fblocks, slot = b / m.fblocks;
    const unsigned int fc = fb * F * (LS_WARPS / WK), f0 = fc + wf * F;    // first feature of the CTA, of the warp
    const bool grouped = m.group_offset != nullptr;
    grid_dependency_launch();
    unsigned int group = 0, row0 = 0, count = m.rows;
    if (grouped)
    {
        grid_dependency_wait();
        if (m.active != nullptr)
        {
            const int id = m.active[slot];
            if (id < 0) { return; }
            group = (unsigned int)id;
        }
        else { group = slot; }
        row0 = (unsigned int)m.group_offset[group];
        count = (unsigned int)m.group_offset[group + 1] - row0;
        if (count == 0) { return; }
    }
    if (m.blocks > 1) { group = slot; }
    const __nv_bfloat16* W = (const __nv_bfloat16*)m.W + (size_t)group * m.group_rows * m.ldw;
    const unsigned int xcol = m.blocks > 1 ? group * m.x_step : 0u, ycol = m.blocks > 1 ? group * m.y_step : 0u;
    const __nv_bfloat16* wr[RT][2];
#pragma unroll
    for (int r = 0; r < RT; r++)
    {
#pragma unroll
        for (int h = 0; h < 2; h++)
        {
            unsigned int f = f0 + (gated ? 0 : r * 16) + g + h * 8;
            f = min(f, m.N - 1);    // rows past N: any valid row, the result is not stored
            wr[r][h] = W + (size_t)(f + (gated && r == 1 ? m.up_row : 0u)) * m.ldw + t * 16;
        }
    }
    const unsigned int chunks = (m.K + 63) / 64;
    uint4 a[U][RT][2][2], an[U][RT][2][2];
    auto load = [&](uint4 (&d)[U][RT][2][2], unsigned int c0) {
#pragma unroll
        for (int u = 0; u < U; u++)
        {
            const unsigned int c = c0 + u * WK;
            if (c < chunks)
            {
#pragma unroll
                for (int r = 0; r < RT; r++)
                {
#pragma unroll
                    for (int h = 0; h < 2; h++)
                    {
                        ldg_stream(wr[r][h] + c * 64, d[u][r][h][0], d[u][r][h][1]);
                    }
                }
            }
        }
    };
    load(a, wk);
    if (!grouped) { grid_dependency_wait(); }
    for (unsigned int n0 = 0; n0 < count; n0 += C)
    {
        if (n0 != 0) { load(a, wk); }
        const __nv_bfloat16* xr[NT];
        bool live[NT];
#pragma unroll
        for (int nt = 0; nt < NT; nt++)
        {
            const unsigned int n = n0 + nt * 8 + g;
            live[nt] = n < count;
            unsigned int r = row0 + (live[nt] ? n : 0u);
            if (m.x_row != nullptr) { r = (unsigned int)m.x_row[r]; }
            xr[nt] = (const __nv_bfloat16*)m.X + (size_t)r * m.ldx + xcol + t * 16;
        }
        float acc[RT][NT][4];
#pragma unroll
        for (int r = 0; r < RT; r++)
        {
#pragma unroll
            for (int nt = 0; nt < NT; nt++)
            {
#pragma unroll
                for (int j = 0; j < 4; j++) { acc[r][nt][j] = 0.f; }
            }
        }
        for (unsigned int c0 = wk; c0 < chunks; c0 += U * WK)
        {
            load(an, c0 + U * WK);
#pragma unroll
            for (int u = 0; u < U; u++)
            {
                const unsigned int c = c0 + u * WK;
                if (c >= chunks) { break; }
                uint4 x[NT][2];
#pragma unroll
                for (int nt = 0; nt < NT; nt++)
                {
#pragma unroll
                    for (int k = 0; k < 2; k++)
                    {
                        x[nt][k] = make_uint4(0, 0, 0, 0);
                        if (live[nt]) { x[nt][k] = *reinterpret_cast<const uint4*>(xr[nt] + c * 64 + k * 8); }
                    }
                }
#pragma unroll
                for (int nt = 0; nt < NT; nt++)
                {
#pragma unroll
                    for (int k = 0; k < 2; k++)
                    {
#pragma unroll
                        for (int r = 0; r < RT; r++)
                        {
                            mma_bf16_16816(acc[r][nt], a[u][r][0][k].x, a[u][r][1][k].x, a[u][r][0][k].y, a[u][r][1][k].y, x[nt][k].x, x[nt][k].y);
                            mma_bf16_16816(acc[r][nt], a[u][r][0][k].z, a[u][r][1][k].z, a[u][r][0][k].w, a[u][r][1][k].w, x[nt][k].z, x[nt][k].w);
                        }
                    }
                }
            }
#pragma unroll
            for (int u = 0; u < U; u++)
            {
#pragma unroll
                for (int r = 0; r < RT; r++)
                {
#pragma unroll
                    for (int h = 0; h < 2; h++)
                    {
                        a[u][r][h][0] = an[u][r][h][0];
                        a[u][r][h][1] = an[u][r][h][1];
                    }
                }
            }
        }
        if (n0 != 0) { __syncthreads(); }
#pragma unroll
        for (int r = 0; r < RT; r++)
        {
#pragma unroll
            for (int nt = 0; nt < NT; nt++)
            {
                red[warp][nt * 8 + 2 * t][r * 16 + g] = acc[r][nt][0];
                red[warp][nt * 8 + 2 * t + 1][r * 16 + g] = acc[r][nt][1];
                red[warp][nt * 8 + 2 * t][r * 16 + g + 8] = acc[r][nt][2];
                red[warp][nt * 8 + 2 * t + 1][r * 16 + g + 8] = acc[r][nt][3];
            }
        }
        __syncthreads();
        const unsigned int cols = min((unsigned int)C, count - n0);
        const unsigned int all = F * (LS_WARPS / WK);
        for (unsigned int i = threadIdx.x; i < cols * all; i += 32 * LS_WARPS)
        {
            const unsigned int f = i % all, n = i / all, w0 = f / F * WK, fl = f % F;
            if (fc + f >= m.N) { continue; }
            float v = 0.f, up = 0.f;
#pragma unroll
            for (int w = 0; w < WK; w++) { v += red[w0 + w][n][fl]; }
            if (gated)
            {
#pragma unroll
                for (int w = 0; w < WK; w++) { up += red[w0 + w][n][16 + fl]; }
            }
            const float y = linear_activation<true>(m.activation, m.alpha * v, m.alpha * up, m.cap);
            linear_store(m, row0 + n0 + n, ycol + fc + f, y * linear_row_factor<__nv_bfloat16>(m, row0 + n0 + n, group));
        }
    }
}

// ---- the float mode: a plain tiled product in true float -------------------------------------------
constexpr int LF_F = 64, LF_R = 32, LF_K = 32;

template <bool GATED>
__global__ void __launch_bounds__(256) linear_f32_kernel(const LinearMember m)
{
    __shared__ float ws[GATED ? 2 : 1][LF_K][LF_F + 1];
    __shared__ float xs[LF_K][LF_R + 1];
    grid_dependency_launch();
    grid_dependency_wait();
    unsigned int group = 0, row0 = 0, count = m.rows;
    if (m.group_offset != nullptr)
    {
        group = blockIdx.z;
        row0 = (unsigned int)m.group_offset[group];
        count = (unsigned int)m.group_offset[group + 1] - row0;
    }
    const unsigned int f0 = blockIdx.x * LF_F, r0 = blockIdx.y * LF_R;
    if (r0 >= count) { return; }
    if (m.blocks > 1) { group = blockIdx.z; }
    const float* W = (const float*)m.W + (size_t)group * m.group_rows * m.ldw;
    const unsigned int xcol = m.blocks > 1 ? group * m.x_step : 0u, ycol = m.blocks > 1 ? group * m.y_step : 0u;
    const unsigned int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;    // 16 x 16 threads: 4 features x 2 rows each
    float acc[GATED ? 2 : 1][2][4] = {};
    for (unsigned int k0 = 0; k0 < m.K; k0 += LF_K)
    {
        for (unsigned int i = threadIdx.x; i < LF_F * LF_K; i += 256)
        {
            const unsigned int k = i % LF_K, f = i / LF_K;
            const bool ok = k0 + k < m.K && f0 + f < m.N;
            ws[0][k][f] = ok ? W[(size_t)(f0 + f) * m.ldw + k0 + k] : 0.f;
            if (GATED) { ws[GATED ? 1 : 0][k][f] = ok ? W[(size_t)(m.up_row + f0 + f) * m.ldw + k0 + k] : 0.f; }
        }
        for (unsigned int i = threadIdx.x; i < LF_R * LF_K; i += 256)
        {
            const unsigned int k = i % LF_K, r = i / LF_K;
            float v = 0.f;
            if (k0 + k < m.K && r0 + r < count)
            {
                unsigned int xr = row0 + r0 + r;
                if (m.x_row != nullptr) { xr = (unsigned int)m.x_row[xr]; }
                v = ((const float*)m.X)[(size_t)xr * m.ldx + xcol + k0 + k];
            }
            xs[k][r] = v;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < LF_K; k++)
        {
#pragma unroll
            for (int i = 0; i < 2; i++)
            {
                const float x = xs[k][ty + 16 * i];
#pragma unroll
                for (int j = 0; j < 4; j++)
                {
                    acc[0][i][j] = fmaf(ws[0][k][tx + 16 * j], x, acc[0][i][j]);
                    if (GATED) { acc[GATED ? 1 : 0][i][j] = fmaf(ws[GATED ? 1 : 0][k][tx + 16 * j], x, acc[GATED ? 1 : 0][i][j]); }
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; i++)
    {
#pragma unroll
        for (int j = 0; j < 4; j++)
        {
            const unsigned int r = r0 + ty + 16 * i, f = f0 + tx + 16 * j;
            if (r < count && f < m.N)
            {
                const float y = linear_activation<false>(m.activation, m.alpha * acc[0][i][j], GATED ? m.alpha * acc[GATED ? 1 : 0][i][j] : 0.f, m.cap);
                linear_store(m, row0 + r, ycol + f, y * linear_row_factor<float>(m, row0 + r, group));
            }
        }
    }
}

template <int NT, int RT, int U, int WK>
static int launch_stream_wk(LinearLaunch& L, cudaStream_t st, bool pdl)
{
    unsigned int blocks = 0;
    for (unsigned int j = 0; j < L.count; j++)
    {
        LinearMember& m = L.m[j];
        const unsigned int F = (activation_gated(m.activation) ? 8 * RT : 16 * RT) * (LS_WARPS / WK);
        m.fblocks = (m.N + F - 1) / F;
        m.block0 = blocks;
        blocks += m.fblocks * m.slots;
    }
    // The rows of X are read through L1, of which a kernel with much shared memory just before would otherwise leave little.
    static std::atomic<unsigned long long> done{ 0 };
    prefer_l1(linear_stream_kernel<NT, RT, U, WK>, done);
    return launch_kernel("linear_stream", linear_stream_kernel<NT, RT, U, WK>, dim3(blocks), dim3(32 * LS_WARPS), 0, st, pdl, L);
}

template <int NT, int RT, int U>
static int launch_stream(LinearLaunch& L, cudaStream_t st, bool pdl)
{
    // eight warps over few chunks would leave some without any; the members of a launch take one form
    unsigned int longest = 0;
    for (unsigned int j = 0; j < L.count; j++) { longest = L.m[j].K > longest ? L.m[j].K : longest; }
    return longest <= 1024 ? launch_stream_wk<NT, RT, U, 2>(L, st, pdl) : launch_stream_wk<NT, RT, U, 8>(L, st, pdl);
}

}    // namespace b200

using namespace b200;

C_EXPORT int cuda_b200_linear_rows(int dtype, unsigned int count, const cuda_b200_linear* members, void* stream, unsigned int flags, int kernel)
{
    if (count == 0) { return 0; }
    if (!members || count > LINEAR_MAX_MEMBERS || (dtype != DT_BF16 && dtype != DT_FLOAT)) { return -1; }
    LinearLaunch L;
    memset(&L, 0, sizeof(L));
    unsigned int most = 0, group_max[LINEAR_MAX_MEMBERS] = {};
    for (unsigned int j = 0; j < count; j++)
    {
        const cuda_b200_linear& a = members[j];
        if (a.rows == 0 || a.N == 0) { continue; }
        auto bad_align = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 31u) != 0; };
        if (!a.W || !a.X || !a.Y || a.K == 0 || bad_align(a.W) || bad_align(a.X)) { return -1; }
        if (a.activation < B200_ACT_NONE || a.activation > B200_ACT_SOFTCAP || (a.out_type != DT_FLOAT && a.out_type != DT_BF16)) { return -1; }
        if (a.accumulate && a.out_type != DT_FLOAT) { return -1; }
        if (dtype == DT_FLOAT && a.out_type != DT_FLOAT) { return -1; }
        const unsigned int kp = (a.K + 63) / 64 * 64;
        if ((a.ldw % 64) || (a.ldx % 64) || a.ldw < kp || a.ldx < kp) { return -1; }
        if (a.group_offset && (a.groups == 0 || a.group_max == 0 || a.blocks > 1)) { return -1; }
        if (a.blocks > 1 && ((a.x_step % 8) || a.x_row)) { return -1; }
        if (a.activation == B200_ACT_SOFTCAP && !(a.cap > 0.f)) { return -1; }
        if (a.tail && (!a.Y_tail || a.accumulate || a.blocks > 1 || a.group_offset || a.activation != B200_ACT_NONE)) { return -1; }
        LinearMember& m = L.m[L.count++];
        m.W = a.W;
        m.X = a.X;
        m.Y = a.Y;
        m.row_scale = (const float*)a.row_scale;
        m.group_offset = (const int*)a.group_offset;
        m.x_row = (const int*)a.x_row;
        m.active = (const int*)a.active;
        m.rows = a.rows;
        m.N = a.N;
        m.K = a.K;
        m.ldw = a.ldw;
        m.ldx = a.ldx;
        m.ldy = a.ldy;
        m.groups = a.group_offset ? a.groups : 1;
        m.group_rows = a.group_rows;
        m.up_row = a.up_row;
        m.blocks = a.blocks > 1 ? a.blocks : 1;
        m.x_step = a.x_step;
        m.y_step = a.y_step;
        m.head_gate = a.head_gate;
        m.ld_gate = a.ld_gate;
        m.Y_tail = (float*)a.Y_tail;
        m.tail = a.tail ? a.tail : 0xFFFFFFFFu;
        m.ld_tail = a.ld_tail;
        m.cap = a.cap;
        m.slots = a.group_offset ? (a.active ? a.active_cap : a.groups) : m.blocks;
        m.out_type = a.out_type;
        m.activation = a.activation;
        m.accumulate = a.accumulate;
        m.alpha = a.alpha;
        if (m.slots == 0) { return -1; }
        group_max[L.count - 1] = a.group_max;
        const unsigned int rows = a.group_offset ? a.group_max : a.rows;
        most = rows > most ? rows : most;
    }
    if (L.count == 0) { return 0; }
    const bool pdl = (flags & 1u) != 0;
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == DT_FLOAT)
    {
        for (unsigned int j = 0; j < L.count; j++)
        {
            const LinearMember& m = L.m[j];
            const unsigned int rows = m.group_offset ? (most < m.rows ? most : m.rows) : m.rows;
            const dim3 grid((m.N + LF_F - 1) / LF_F, (rows + LF_R - 1) / LF_R, m.blocks > 1 ? m.blocks : m.groups);
            if (grid.y > 65535u || grid.z > 65535u) { return -1; }
            const int rc = activation_gated(m.activation) ? launch_kernel("linear_f32", linear_f32_kernel<true>, grid, dim3(256), 0, st, pdl, m)
                                                              : launch_kernel("linear_f32", linear_f32_kernel<false>, grid, dim3(256), 0, st, pdl, m);
            if (rc) { return rc; }
        }
        return 0;
    }
    // a dense linear of 17 to 32 rows with a tile for every SM (a head over a vocabulary): tiles stream weights as fast
    if (kernel == 0 && L.count == 1 && most > 16 && L.m[0].blocks == 1 && !L.m[0].group_offset && !L.m[0].x_row)
    {
        const DecoderDevice* dev = decoder_device();
        if (dev && L.m[0].N >= 256u * (unsigned int)dev->sm_count) { kernel = 2; }
    }
    if (kernel == 1 || (kernel == 0 && most <= 32))
    {
        // Members whose groups hold about as many rows share a launch: 8, 16 or 32 rows at a time.  A group with more rows
        // than that reads its weights again, so experts go by twice their mean.
        for (unsigned int width = 8; width <= 32; width *= 2)
        {
            LinearLaunch part;
            memset(&part, 0, sizeof(part));
            bool gated = false;
            for (unsigned int j = 0; j < L.count; j++)
            {
                const LinearMember& m = L.m[j];
                unsigned int rows = m.rows;
                if (m.group_offset)
                {
                    rows = 2 * ((m.rows + m.slots - 1) / m.slots);
                    if (rows > group_max[j]) { rows = group_max[j]; }
                }
                if (width < 32 ? rows > width : false) { continue; }
                if (width > 8 && rows <= width / 2) { continue; }
                part.m[part.count++] = m;
                gated = gated || activation_gated(m.activation);
            }
            if (part.count == 0) { continue; }
            int rc;
            if (width == 8) { rc = gated ? launch_stream<1, 2, 1>(part, st, pdl) : launch_stream<1, 1, 2>(part, st, pdl); }
            else if (width == 16) { rc = gated ? launch_stream<2, 2, 1>(part, st, pdl) : launch_stream<2, 1, 2>(part, st, pdl); }
            else { rc = launch_stream<4, 2, 1>(part, st, pdl); }
            if (rc) { return rc; }
        }
        return 0;
    }
    for (unsigned int j = 0; j < L.count; j++)
    {
        const int rc = launch_linear_tile(L.m[j], st, pdl);
        if (rc) { return rc; }
    }
    return 0;
}
