// The Mamba-2 recurrence of long portions, in chunks of MC tokens.  Per head, with dt = softplus(raw + bias), a = e^(-e^(A_log) dt),
// B and C (N features, of the head's group) and x (P features) of a token:  S <- a S + dt B x^T,  y = S^T C + D x.  With S the
// state at a chunk's start and t, j counting the chunk's r tokens from 0:
//     y_t    = (a_0 .. a_t) S^T C_t + sum_{j <= t} (a_{j+1} .. a_t) dt_j (C_t . B_j) x_j + D x_t
//     S_next = (a_0 .. a_{r-1}) S + sum_j (a_{j+1} .. a_{r-1}) dt_j B_j x_j^T
// ssm_chunk_scores_kernel   C_t . B_j of every chunk and group (shared by the group's heads)
// ssm_chunk_sum_kernel      the chunks' own sums, [N][P] per head and chunk
// ssm_chunk_scan_kernel     a thread per element of the state walks its request's chunks: sums become the states at the starts
// ssm_chunk_out_kernel      y of every chunk
// A decay between two tokens is a product of the a's between them (running products of numbers in [0, 1], cut at the middle of
// the chunk), never a quotient or a difference of sums, so that nothing cancels after a token with a large step.
// Everything is float.  N and P are multiples of 4.  The slot's layout is that of ssm_scan_kernel: [H][P][N].
#include "common.cuh"

namespace bg {

constexpr int MC = 64;                     // tokens of a chunk
constexpr int MPT = 64;                    // columns p of a block
constexpr int MCP = MC + 4;                // row stride of the score tile
constexpr int MBATCH = 8;                  // chunks of the walk fetched at a time

struct SsmChunkParams {
    const float* xbc; int channels;        // [T][x: H P | B: G N | C: G N]
    const void* src; int src_stride, dt_col;
    const void* dt_bias; const void* A_log; const void* D;
    float* state; size_t slot_stride; const int* slots;
    const int* chunks;                     // [n_chunks][4] = (request, first row, rows, -)
    const int* longs;                      // [n_long][4]   = (request, first row, rows, first chunk)
    float* scores;                         // [n_chunks][G][MC (t)][MC (j)]
    float* work;                           // [n_chunks][H][N][P]
    float* decay;                          // [n_chunks][H]
    float* y;                              // [T][H P]
    int H, P, N, G;
};

__device__ __forceinline__ float sc_softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ void sc_async16(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void sc_async_wait() { asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;\n" ::: "memory"); }

// rows [0, MC) of `w` floats (a multiple of 4) into a tile of row stride `ld`; rows from `rows` on become zeros
__device__ __forceinline__ void sc_rows(float* dst, int ld, const float* src, size_t stride, int rows, int w) {
    const int w4 = w >> 2;
    for (int idx = threadIdx.x; idx < MC * w4; idx += blockDim.x) {
        const int r = idx / w4, c = (idx - r * w4) * 4;
        if (r < rows) sc_async16(dst + r * ld + c, src + (size_t)r * stride + c);
        else *reinterpret_cast<float4*>(dst + r * ld + c) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
}

// Step sizes and decays of the chunk's tokens for head h, and the decays' running products inside each half of the chunk:
// pre[t] = product from the half's start up to and with t, suf[j] = product behind j to the half's end.  Tokens from `rows` on
// have a step of nought and a decay of one.  Warps 0 and 1 work; the caller synchronises.
template <typename TI, typename TW>
__device__ __forceinline__ void sc_steps(const SsmChunkParams& p, int h, int row0, int rows, float* dt_s, float* a_s, float* pre, float* suf) {
    if (threadIdx.x >= MC) return;
    const int t = threadIdx.x, lane = t & 31;
    float dt = 0.0f, a = 1.0f;
    if (t < rows) {
        dt = sc_softplus(to_float(((const TI*)p.src)[(size_t)(row0 + t) * p.src_stride + p.dt_col + h]) + to_float(((const TW*)p.dt_bias)[h]));
        a = expf(-expf(to_float(((const TW*)p.A_log)[h])) * dt);
    }
    float up = a, down = a;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float u = __shfl_up_sync(0xffffffffu, up, o), d = __shfl_down_sync(0xffffffffu, down, o);
        if (lane >= o) up *= u;
        if (lane + o < 32) down *= d;
    }
    const float behind = __shfl_down_sync(0xffffffffu, down, 1);
    dt_s[t] = dt; a_s[t] = a; pre[t] = up; suf[t] = lane == 31 ? 1.0f : behind;
}

__global__ void __launch_bounds__(256) ssm_chunk_scores_kernel(SsmChunkParams p) {
    extern __shared__ __align__(16) float sc_s[];
    const int ld = p.N + 4;
    float* Cs = sc_s;                      // [MC][N + 4]
    float* Bs = Cs + MC * ld;              // [MC][N + 4]
    pdl_launch();
    pdl_wait();
    const int g = blockIdx.x, ch = blockIdx.y;
    const int row0 = p.chunks[ch * 4 + 1], rows = p.chunks[ch * 4 + 2];
    const float* base = p.xbc + (size_t)row0 * p.channels + (size_t)p.H * p.P + (size_t)g * p.N;
    sc_rows(Bs, ld, base, p.channels, rows, p.N);
    sc_rows(Cs, ld, base + (size_t)p.G * p.N, p.channels, rows, p.N);
    sc_async_wait();
    __syncthreads();
    // a thread takes queries ty, ty + 16, .. and keys tx, tx + 16, ..
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
#pragma unroll 2
    for (int n = 0; n < p.N; n += 4) {
        float4 c[4], b[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            c[u] = *reinterpret_cast<const float4*>(Cs + (ty + 16 * u) * ld + n);
            b[u] = *reinterpret_cast<const float4*>(Bs + (tx + 16 * u) * ld + n);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int v = 0; v < 4; ++v)
                acc[u][v] = fmaf(c[u].x, b[v].x, fmaf(c[u].y, b[v].y, fmaf(c[u].z, b[v].z, fmaf(c[u].w, b[v].w, acc[u][v]))));
    }
    float* out = p.scores + ((size_t)ch * p.G + g) * MC * MC;
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int v = 0; v < 4; ++v) out[(ty + 16 * u) * MC + tx + 16 * v] = acc[u][v];
}

template <typename TI, typename TW>
__global__ void __launch_bounds__(256) ssm_chunk_sum_kernel(SsmChunkParams p) {
    extern __shared__ __align__(16) float sc_s[];
    __shared__ float dt_s[MC], a_s[MC], pre[MC], suf[MC];
    const int N = p.N, P = p.P;
    float* Bs = sc_s;                      // [MC][N]
    float* Xs = Bs + (size_t)MC * N;       // [MC][MPT]
    pdl_launch();
    pdl_wait();
    const int h = blockIdx.x, ch = blockIdx.y, p0 = blockIdx.z * MPT, tid = threadIdx.x;
    const int pw = min(MPT, P - p0);
    const int row0 = p.chunks[ch * 4 + 1], rows = p.chunks[ch * 4 + 2];
    const float* row = p.xbc + (size_t)row0 * p.channels;
    sc_rows(Bs, N, row + (size_t)p.H * P + (size_t)(h / (p.H / p.G)) * N, p.channels, rows, N);
    sc_rows(Xs, MPT, row + (size_t)h * P + p0, p.channels, rows, pw);
    sc_steps<TI, TW>(p, h, row0, rows, dt_s, a_s, pre, suf);
    sc_async_wait();
    __syncthreads();
    if (tid == 0 && blockIdx.z == 0) p.decay[(size_t)ch * p.H + h] = pre[MC / 2 - 1] * pre[MC - 1];
    {                                      // x_j times its step and the decay behind it
        const float second = pre[MC - 1];
        for (int idx = tid; idx < MC * (pw >> 2); idx += blockDim.x) {
            const int j = idx / (pw >> 2), c = (idx - j * (pw >> 2)) * 4;
            const float w = dt_s[j] * (j < MC / 2 ? suf[j] * second : suf[j]);
            float4* x = reinterpret_cast<float4*>(Xs + j * MPT + c);
            float4 v = *x;
            v.x *= w; v.y *= w; v.z *= w; v.w *= w;
            *x = v;
        }
    }
    __syncthreads();
    float* A = p.work + ((size_t)ch * p.H + h) * N * P;
    const int tp = pw >> 2, tn = (N + 7) >> 3;
    for (int tile = tid; tile < tn * tp; tile += blockDim.x) {
        const int n0 = (tile / tp) * 8, c0 = (tile % tp) * 4;
        const bool two = n0 + 4 < N;       // (N is a multiple of 4)
        float acc[8][4] = {};
#pragma unroll 4
        for (int j = 0; j < MC; ++j) {
            const float4 x = *reinterpret_cast<const float4*>(Xs + j * MPT + c0);
            const float4 b0 = *reinterpret_cast<const float4*>(Bs + (size_t)j * N + n0);
            const float4 b1 = two ? *reinterpret_cast<const float4*>(Bs + (size_t)j * N + n0 + 4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            const float b[8] = {b0.x, b0.y, b0.z, b0.w, b1.x, b1.y, b1.z, b1.w};
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                acc[u][0] = fmaf(b[u], x.x, acc[u][0]); acc[u][1] = fmaf(b[u], x.y, acc[u][1]);
                acc[u][2] = fmaf(b[u], x.z, acc[u][2]); acc[u][3] = fmaf(b[u], x.w, acc[u][3]);
            }
        }
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (n0 + u < N) *reinterpret_cast<float4*>(A + (size_t)(n0 + u) * P + p0 + c0) = make_float4(acc[u][0], acc[u][1], acc[u][2], acc[u][3]);
    }
}

__global__ void __launch_bounds__(256) ssm_chunk_scan_kernel(SsmChunkParams p) {
    pdl_launch();
    pdl_wait();
    const int e = blockIdx.x * blockDim.x + threadIdx.x, h = blockIdx.y, l = blockIdx.z;
    const int sz = p.N * p.P;
    if (e >= sz) return;
    const int req = p.longs[l * 4 + 0], rows = p.longs[l * 4 + 2], c0 = p.longs[l * 4 + 3];
    const int n_chunks = (rows + MC - 1) / MC;
    const int n = e / p.P, col = e - n * p.P;
    float* st = p.state + (size_t)p.slots[req] * p.slot_stride + (size_t)h * sz + (size_t)col * p.N + n;
    float* a0 = p.work + ((size_t)c0 * p.H + h) * sz + e;
    const float* d0 = p.decay + (size_t)c0 * p.H + h;
    const size_t step = (size_t)p.H * sz;
    float S = *st;
    for (int c = 0; c < n_chunks; c += MBATCH) {
        float A[MBATCH], D[MBATCH];
#pragma unroll
        for (int u = 0; u < MBATCH; ++u) {
            A[u] = c + u < n_chunks ? a0[(size_t)(c + u) * step] : 0.0f;
            D[u] = c + u < n_chunks ? d0[(size_t)(c + u) * p.H] : 0.0f;
        }
#pragma unroll
        for (int u = 0; u < MBATCH; ++u)
            if (c + u < n_chunks) {
                a0[(size_t)(c + u) * step] = S;
                S = fmaf(D[u], S, A[u]);
            }
    }
    *st = S;
}

// The token that a thread's row u (of eight) stands for: a warp holds sixteen tokens, a half of it four neighbours and the four
// eight further on, so that the two halves' reads of a tile of rows fall on different banks.
__device__ __forceinline__ int sc_token(int u) {
    return ((int)threadIdx.x >> 5) * 16 + (((int)threadIdx.x >> 4) & 1) * 4 + (u & 3) + (u >> 2) * 8;
}

// acc[u][v] += sum over k of a[token of row u][k] b[k][v], k in steps of 4 up to `k_end`
__device__ __forceinline__ void sc_product(float (&acc)[8][4], const float* a, int lda, const float* b, int k_end) {
#pragma unroll 1
    for (int k = 0; k < k_end; k += 4) {
        float4 bb[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) bb[i] = *reinterpret_cast<const float4*>(b + (size_t)(k + i) * MPT);
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const float4 aa = *reinterpret_cast<const float4*>(a + sc_token(u) * lda + k);
            acc[u][0] = fmaf(aa.x, bb[0].x, acc[u][0]); acc[u][1] = fmaf(aa.x, bb[0].y, acc[u][1]);
            acc[u][2] = fmaf(aa.x, bb[0].z, acc[u][2]); acc[u][3] = fmaf(aa.x, bb[0].w, acc[u][3]);
            acc[u][0] = fmaf(aa.y, bb[1].x, acc[u][0]); acc[u][1] = fmaf(aa.y, bb[1].y, acc[u][1]);
            acc[u][2] = fmaf(aa.y, bb[1].z, acc[u][2]); acc[u][3] = fmaf(aa.y, bb[1].w, acc[u][3]);
            acc[u][0] = fmaf(aa.z, bb[2].x, acc[u][0]); acc[u][1] = fmaf(aa.z, bb[2].y, acc[u][1]);
            acc[u][2] = fmaf(aa.z, bb[2].z, acc[u][2]); acc[u][3] = fmaf(aa.z, bb[2].w, acc[u][3]);
            acc[u][0] = fmaf(aa.w, bb[3].x, acc[u][0]); acc[u][1] = fmaf(aa.w, bb[3].y, acc[u][1]);
            acc[u][2] = fmaf(aa.w, bb[3].z, acc[u][2]); acc[u][3] = fmaf(aa.w, bb[3].w, acc[u][3]);
        }
    }
}

template <typename TI, typename TW>
__global__ void __launch_bounds__(128) ssm_chunk_out_kernel(SsmChunkParams p) {
    extern __shared__ __align__(16) float sc_s[];
    __shared__ float dt_s[MC], a_s[MC], pre[MC], suf[MC];
    const int N = p.N, P = p.P, ldc = N + 4;
    float* Cs = sc_s;                      // [MC][N + 4]
    float* Ss = Cs + (size_t)MC * ldc;     // [N][MPT]
    float* Xs = Ss + (size_t)N * MPT;      // [MC][MPT]
    float* Ws = Xs + (size_t)MC * MPT;     // [MC (t)][MCP]: scores, then times decay and step
    pdl_launch();
    pdl_wait();
    const int h = blockIdx.x, ch = blockIdx.y, p0 = blockIdx.z * MPT, tid = threadIdx.x;
    const int pw = min(MPT, P - p0), g = h / (p.H / p.G);
    const int row0 = p.chunks[ch * 4 + 1], rows = p.chunks[ch * 4 + 2];
    const float* row = p.xbc + (size_t)row0 * p.channels;
    sc_rows(Ws, MCP, p.scores + ((size_t)ch * p.G + g) * MC * MC, MC, MC, MC);
    sc_rows(Cs, ldc, row + (size_t)p.H * P + (size_t)(p.G + g) * N, p.channels, rows, N);
    sc_rows(Xs, MPT, row + (size_t)h * P + p0, p.channels, rows, pw);
    {
        const float* S0 = p.work + ((size_t)ch * p.H + h) * N * P + p0;
        const int w4 = pw >> 2;
        for (int idx = tid; idx < N * w4; idx += blockDim.x) {
            const int r = idx / w4, c = (idx - r * w4) * 4;
            sc_async16(Ss + r * MPT + c, S0 + (size_t)r * P + c);
        }
    }
    sc_steps<TI, TW>(p, h, row0, rows, dt_s, a_s, pre, suf);
    sc_async_wait();
    __syncthreads();
    {
        // the weight of key j at query t: score x (product of the decays behind j up to t) x step.  Threads 0 .. 63: the queries
        // of the key's own half of the chunk, one decay after the other; 64 .. 127: those of the second half for keys of the first
        const int j = tid & (MC - 1), half = j / (MC / 2);
        const float dt = dt_s[j];
        if (tid < MC) {
            const int t_begin = half * (MC / 2);
            float l = dt;
            for (int t = t_begin; t < t_begin + MC / 2; ++t) {
                if (t > j) l *= a_s[t];
                Ws[t * MCP + j] = t < j ? 0.0f : Ws[t * MCP + j] * l;
            }
        } else if (half == 0) {
            const float l = suf[j] * dt;
            for (int t = MC / 2; t < MC; ++t) Ws[t * MCP + j] *= l * pre[t];
        }
        // (the first half's queries never read a key of the second)
    }
    __syncthreads();
    const int t0 = (tid >> 5) * 16, c0 = (tid & 15) * 4;        // the warp's first token
    if (t0 >= rows || c0 >= pw) return;
    float acc[8][4] = {};
    sc_product(acc, Cs, ldc, Ss + c0, N);
    const float first = t0 >= MC / 2 ? pre[MC / 2 - 1] : 1.0f;
#pragma unroll
    for (int u = 0; u < 8; ++u) {
        const float f = first * pre[sc_token(u)];
#pragma unroll
        for (int v = 0; v < 4; ++v) acc[u][v] *= f;
    }
    sc_product(acc, Ws, MCP, Xs + c0, t0 + 16);
    const float Dh = to_float(((const TW*)p.D)[h]);
#pragma unroll
    for (int u = 0; u < 8; ++u) {
        const int t = sc_token(u);
        if (t >= rows) continue;
        const float4 x = *reinterpret_cast<const float4*>(Xs + t * MPT + c0);
        *reinterpret_cast<float4*>(p.y + (size_t)(row0 + t) * p.H * P + (size_t)h * P + p0 + c0) =
            make_float4(fmaf(Dh, x.x, acc[u][0]), fmaf(Dh, x.y, acc[u][1]), fmaf(Dh, x.z, acc[u][2]), fmaf(Dh, x.w, acc[u][3]));
    }
}

static size_t sc_smem_scores(int N) { return (size_t)2 * MC * (N + 4) * sizeof(float); }
static size_t sc_smem_sum(int N) { return ((size_t)MC * N + (size_t)MC * MPT) * sizeof(float); }
static size_t sc_smem_out(int N) { return ((size_t)MC * (N + 4) + (size_t)N * MPT + (size_t)MC * MPT + (size_t)MC * MCP) * sizeof(float); }

}  // namespace bg

using namespace bg;

// 0 when the chunked kernels take these sizes, else BG_ERR_UNSUPPORTED; `chunk` receives the tokens of a chunk.
extern "C" int bg_ssm_chunk_plan(int H, int P, int N, int G, int* chunk) {
    if (H <= 0 || P <= 0 || N <= 0 || G <= 0 || H % G) return BG_ERR_SHAPE;
    if (chunk) *chunk = MC;
    if (P % 4 || N % 4 || H > 65535 || sc_smem_out(N) > 220 * 1024 || sc_smem_scores(N) > 220 * 1024) return BG_ERR_UNSUPPORTED;
    return BG_OK;
}

// The recurrence of requests of many rows.  xbc [T][channels] float; chunks, longs as in decay_attention.cu; scores float
// [n_chunks][G][64 * 64], work float [n_chunks][H][N * P], decay float [n_chunks][H].
extern "C" int bg_ssm_chunked(const float* xbc, int channels, const void* src, int src_dtype, int src_stride, int dt_col,
                              const void* dt_bias, const void* A_log, const void* D, int w_dtype, float* state, long long slot_stride,
                              const int* slots, const int* chunks, int n_chunks, const int* longs, int n_long, float* scores, float* work,
                              float* decay, float* y, int H, int P, int N, int G, cudaStream_t stream) {
    if (n_chunks <= 0 || n_long <= 0) return BG_OK;
    const int rc = bg_ssm_chunk_plan(H, P, N, G, nullptr);
    if (rc != BG_OK) return rc;
    if (n_chunks > 65535 || n_long > 65535 || (P + MPT - 1) / MPT > 65535) return BG_ERR_SHAPE;
    if (channels != H * P + 2 * G * N) return BG_ERR_SHAPE;
    if ((uintptr_t)xbc % 16 || (uintptr_t)y % 16 || (uintptr_t)work % 16 || (uintptr_t)scores % 16) return BG_ERR_ALIGN;
    SsmChunkParams p;
    p.xbc = xbc; p.channels = channels; p.src = src; p.src_stride = src_stride; p.dt_col = dt_col; p.dt_bias = dt_bias; p.A_log = A_log;
    p.D = D; p.state = state; p.slot_stride = (size_t)slot_stride; p.slots = slots; p.chunks = chunks; p.longs = longs; p.scores = scores;
    p.work = work; p.decay = decay; p.y = y; p.H = H; p.P = P; p.N = N; p.G = G;
    const size_t s_scores = sc_smem_scores(N), s_sum = sc_smem_sum(N), s_out = sc_smem_out(N);
    const unsigned tiles = (unsigned)((P + MPT - 1) / MPT);
    if (s_scores > BG_SMEM_OPT_IN) {
        cudaError_t e = cudaFuncSetAttribute(ssm_chunk_scores_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s_scores);
        if (e != cudaSuccess) return (int)e;
    }
    launch(ssm_chunk_scores_kernel, dim3(G, n_chunks), dim3(256), s_scores, stream, p);
    BG_LAUNCH_CHECK();
    BG_DISPATCH_DTYPE(src_dtype, TI, BG_DISPATCH_DTYPE(w_dtype, TW, {
        auto ksum = ssm_chunk_sum_kernel<TI, TW>;
        auto kout = ssm_chunk_out_kernel<TI, TW>;
        if (s_sum > BG_SMEM_OPT_IN) {
            cudaError_t e = cudaFuncSetAttribute(ksum, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s_sum);
            if (e != cudaSuccess) return (int)e;
        }
        if (s_out > BG_SMEM_OPT_IN) {
            cudaError_t e = cudaFuncSetAttribute(kout, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s_out);
            if (e != cudaSuccess) return (int)e;
        }
        launch(ksum, dim3(H, n_chunks, tiles), dim3(256), s_sum, stream, p);
        BG_LAUNCH_CHECK();
        launch(ssm_chunk_scan_kernel, dim3((N * P + 255) / 256, H, n_long), dim3(256), 0, stream, p);
        BG_LAUNCH_CHECK();
        launch(kout, dim3(H, n_chunks, tiles), dim3(128), s_out, stream, p);
    }));
    BG_LAUNCH_CHECK();
    return BG_OK;
}
