// Linear attention with a decay per key channel.  Per head, with q, k, a (n features) and v (nv features) of a token:
//     S <- diag(a) S + k v^T        (S is n x nv, float, one per request and head, zero when the request starts)
//     o  = S^T q
// and the head's result o is RMS-normed by itself with a weight vector shared by the heads, and multiplied by silu of a
// further product of the token's row when there is a gate.  Two ways from the product's rows to q, k and a:
//   FORGET   a = l + (1 - l) sigmoid(f + b), k = 1 - a: the forget gate also decides what is written (l in [0, 1] per channel)
//   DECAY    k a product of its own, a = sigmoid(z)^(1/tau) with z = W r + b for a short row r of the token
// with q = silu(product) or product times a constant.  The state is carried from step to step in a slot of the cache
// manager's slab.  Everything behind the products is float: gates, decays, state, readout, norm.
//
//   gla_walk_kernel      a block per (head, request) walks the request's tokens in turn with the whole state in registers,
//                        and norms and gates the head's result itself.  Steps of single tokens and short portions.
//   gla_walk_mem_kernel  the same with the state in global memory: heads of any size.
//   gla_alpha_kernel     DECAY, long portions: the decays of all rows and channels.
//   gla_chunk_*          long portions in chunks of GC tokens: the chunks' own decayed sums of k v^T in parallel, a pass over
//                        the chunks that turns them into the states at the chunks' starts, the chunks' outputs in parallel.
//
// A decay between two tokens is a PRODUCT of the a's between them; it is never formed as a quotient of products from a
// chunk's start (which underflow) nor from logarithms (a may be 0).  A chunk is cut into blocks of GB tokens, and a product
// over tokens of several blocks is split at the blocks' borders: (from the key's token to its block's end) x (whole blocks
// between) x (from the start of the query's block to its token), each a running product of numbers in [0, 1].
#include "common.cuh"

namespace bg {

__device__ __forceinline__ float gla_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gla_silu(float z) { return z / (1.0f + expf(-z)); }
// sigmoid(z)^p through the logarithm log sigmoid(z) = min(z, 0) - log1p(e^-|z|)
__device__ __forceinline__ float gla_root(float z, float p) { return expf(p * (fminf(z, 0.0f) - log1pf(expf(-fabsf(z))))); }

struct GlaParams {
    const float* src; int src_stride;           // rows of the product(s)
    int q_col, k_col, v_col, g_col;             // k_col: the forget gate's (FORGET) or the key's columns; g_col < 0: no gate
    int forget;                                 // FORGET or DECAY
    int q_silu; float q_scale;
    const float* bias;                          // [H n] b
    const float* lower;                         // FORGET: [H n] l
    int r_col, rank;                            // DECAY: the short row's columns
    const float* wa;                            // DECAY: [H n][rank]
    float power;                                // DECAY: 1 / tau
    const float* alpha;                         // DECAY, chunks: [T][H n] made by gla_alpha_kernel
    const float* norm_w; float eps;             // [nv]
    float* state; size_t slot_stride;           // slab [slots][>= H n nv]
    const int* slots;
    const int* reqs;                            // [n_req][3] = (request, first row, rows)
    void* out; int out_float;                   // [T][H nv]
    int H, n, nv;
    // chunks
    const int* chunks;                          // [n_chunks][4] = (request, first row, rows, -)
    const int* longs;                           // [n_long][4]   = (request, first row, rows, first chunk)
    float* work;                                // [n_chunks][H][n nv]
    float* decay;                               // [n_chunks][H][n] the chunk's whole decay
    int np, nvp;                                // n, nv rounded up to multiples of 4
};

__device__ __forceinline__ float gla_query(const GlaParams& p, float raw) { return p.q_silu ? gla_silu(raw) * p.q_scale : raw * p.q_scale; }
// FORGET: (a, k) from the gate's product z of channel c
__device__ __forceinline__ void gla_forget(const GlaParams& p, int c, float raw, float* a, float* k) {
    const float z = raw + p.bias[c], l = p.lower[c];
    *a = fmaf(1.0f - l, gla_sigmoid(z), l);
    *k = (1.0f - l) * gla_sigmoid(-z);
}
// DECAY: a of channel c from the token's row
__device__ __forceinline__ float gla_decay(const GlaParams& p, int c, const float* row) {
    float z = p.bias[c];
    const float* w = p.wa + (size_t)c * p.rank;
    for (int r = 0; r < p.rank; ++r) z = fmaf(w[r], row[p.r_col + r], z);
    return gla_root(z, p.power);
}
__device__ __forceinline__ void gla_store(const GlaParams& p, size_t at, float v) {
    if (p.out_float) ((float*)p.out)[at] = v; else ((__nv_bfloat16*)p.out)[at] = __float2bfloat16_rn(v);
}
__device__ __forceinline__ float gla_gate(const GlaParams& p, const float* row, int h, int c) {
    return p.g_col >= 0 ? gla_silu(row[p.g_col + h * p.nv + c]) : 1.0f;
}

// q, k, a (n values each) and v (nv) of a token's head into shared memory.
__device__ __forceinline__ void gla_load_token(const GlaParams& p, const float* row, int h, float* qs, float* ks, float* as, float* vs) {
    const int n = p.n, nv = p.nv, tid = threadIdx.x;
    for (int i = tid; i < n; i += blockDim.x) {
        const int c = h * n + i;
        qs[i] = gla_query(p, row[p.q_col + c]);
        if (p.forget) gla_forget(p, c, row[p.k_col + c], as + i, ks + i);
        else { ks[i] = row[p.k_col + c]; as[i] = gla_decay(p, c, row); }
    }
    for (int i = tid; i < nv; i += blockDim.x) vs[i] = row[p.v_col + h * nv + i];
}

// The state in registers: thread (slice, column) holds the R rows from slice R on of its column; `slices` threads share a
// column (blockDim.x / nv of them, whole columns only, slices R >= n).  q, k and a are padded with zeros up to slices R, so
// that a thread reads them four at a time and without a condition.
template <int R>
__global__ void __launch_bounds__(512) gla_walk_kernel(GlaParams p, int slices) {
    extern __shared__ __align__(16) float ga_s[];
    __shared__ float scratch[32];
    const int n = p.n, nv = p.nv, np = slices * R;
    float* qs = ga_s;                      // [np]
    float* ks = qs + np;                   // [np]
    float* as = ks + np;                   // [np]
    float* vs = as + np;                   // [nv]
    float* red = vs + nv;                  // [slices][nv]
    pdl_launch();
    const int h = blockIdx.x, r = blockIdx.y;
    const int req = p.reqs[r * 3 + 0], row0 = p.reqs[r * 3 + 1], rows = p.reqs[r * 3 + 2];
    const int tid = threadIdx.x;
    const int sl = tid / nv, c = tid - sl * nv, i0 = sl * R;
    const bool own = sl < slices && rows > 0;
    // the state was left by an earlier step: it is on its way while the product ahead still runs
    float* st = p.state + (size_t)p.slots[req] * p.slot_stride + (size_t)h * n * nv + (size_t)i0 * nv + c;
    float S[R];
#pragma unroll
    for (int k = 0; k < R; ++k) S[k] = (own && i0 + k < n) ? st[(size_t)k * nv] : 0.0f;
    for (int i = n + tid; i < np; i += blockDim.x) { qs[i] = 0.0f; ks[i] = 0.0f; as[i] = 0.0f; }
    pdl_wait();
    if (rows <= 0) return;
    for (int t = 0; t < rows; ++t) {
        const float* row = p.src + (size_t)(row0 + t) * p.src_stride;
        __syncthreads();
        gla_load_token(p, row, h, qs, ks, as, vs);
        __syncthreads();
        if (own) {
            const float v = vs[c];
            float acc0 = 0.0f, acc1 = 0.0f;
#pragma unroll
            for (int k = 0; k < R; k += 4) {
                const float4 a = *reinterpret_cast<const float4*>(as + i0 + k), kk = *reinterpret_cast<const float4*>(ks + i0 + k);
                const float4 q = *reinterpret_cast<const float4*>(qs + i0 + k);
                S[k + 0] = fmaf(a.x, S[k + 0], kk.x * v); acc0 = fmaf(S[k + 0], q.x, acc0);
                S[k + 1] = fmaf(a.y, S[k + 1], kk.y * v); acc1 = fmaf(S[k + 1], q.y, acc1);
                S[k + 2] = fmaf(a.z, S[k + 2], kk.z * v); acc0 = fmaf(S[k + 2], q.z, acc0);
                S[k + 3] = fmaf(a.w, S[k + 3], kk.w * v); acc1 = fmaf(S[k + 3], q.w, acc1);
            }
            red[sl * nv + c] = acc0 + acc1;
        }
        __syncthreads();
        float o = 0.0f;
        if (tid < nv) for (int q = 0; q < slices; ++q) o += red[q * nv + tid];
        const float ss = block_sum(o * o, scratch);
        if (tid < nv)
            gla_store(p, (size_t)(row0 + t) * p.H * nv + (size_t)h * nv + tid,
                      o * (1.0f / sqrtf(ss / (float)nv + p.eps)) * p.norm_w[tid] * gla_gate(p, row, h, tid));
    }
    if (own) {
        int stride = nv;
        asm volatile("" : "+r"(stride));   // the addresses are worked out again here: kept from the loads, they would fill the registers
#pragma unroll
        for (int k = 0; k < R; ++k)
            if (i0 + k < n) st[(size_t)k * stride] = S[k];
    }
}

// The same with the state in place: a thread walks whole columns.
__global__ void __launch_bounds__(256) gla_walk_mem_kernel(GlaParams p) {
    extern __shared__ float ga_s[];
    __shared__ float scratch[32];
    const int n = p.n, nv = p.nv;
    float* qs = ga_s; float* ks = qs + n; float* as = ks + n; float* vs = as + n; float* os = vs + nv;
    pdl_launch();
    pdl_wait();
    const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x;
    const int req = p.reqs[r * 3 + 0], row0 = p.reqs[r * 3 + 1], rows = p.reqs[r * 3 + 2];
    if (rows <= 0) return;
    float* st = p.state + (size_t)p.slots[req] * p.slot_stride + (size_t)h * n * nv;
    for (int t = 0; t < rows; ++t) {
        const float* row = p.src + (size_t)(row0 + t) * p.src_stride;
        __syncthreads();
        gla_load_token(p, row, h, qs, ks, as, vs);
        __syncthreads();
        float ss = 0.0f;
        for (int c = tid; c < nv; c += blockDim.x) {
            const float v = vs[c];
            float acc = 0.0f;
            for (int i = 0; i < n; ++i) {
                const float s = fmaf(as[i], st[(size_t)i * nv + c], ks[i] * v);
                st[(size_t)i * nv + c] = s;
                acc = fmaf(s, qs[i], acc);
            }
            os[c] = acc;
            ss += acc * acc;
        }
        const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)nv + p.eps);
        for (int c = tid; c < nv; c += blockDim.x)
            gla_store(p, (size_t)(row0 + t) * p.H * nv + (size_t)h * nv + c, os[c] * inv * p.norm_w[c] * gla_gate(p, row, h, c));
    }
}

// alpha[t][c] = sigmoid(W_c . r_t + b_c)^power: GA_ROWS rows a block, a thread per channel.
constexpr int GA_ROWS = 16, GA_RANK = 16;
__global__ void __launch_bounds__(256) gla_alpha_kernel(GlaParams p, float* __restrict__ alpha, int T) {
    __shared__ float r_s[GA_ROWS][GA_RANK];
    pdl_launch();
    pdl_wait();
    const int C = p.H * p.n, t0 = blockIdx.y * GA_ROWS;
    const int c = blockIdx.x * 256 + threadIdx.x;
    const bool live = c < C;
    float z[GA_ROWS];
    const float b = live ? p.bias[c] : 0.0f;
#pragma unroll
    for (int t = 0; t < GA_ROWS; ++t) z[t] = b;
    for (int r0 = 0; r0 < p.rank; r0 += GA_RANK) {
        __syncthreads();
        {
            const int t = threadIdx.x / GA_RANK, r = threadIdx.x % GA_RANK;
            r_s[t][r] = (t0 + t < T && r0 + r < p.rank) ? p.src[(size_t)(t0 + t) * p.src_stride + p.r_col + r0 + r] : 0.0f;
        }
        float w[GA_RANK];
#pragma unroll
        for (int r = 0; r < GA_RANK; ++r) w[r] = (live && r0 + r < p.rank) ? p.wa[(size_t)c * p.rank + r0 + r] : 0.0f;
        __syncthreads();
#pragma unroll
        for (int t = 0; t < GA_ROWS; ++t)
#pragma unroll
            for (int r = 0; r < GA_RANK; ++r) z[t] = fmaf(w[r], r_s[t][r], z[t]);
    }
    if (!live) return;
#pragma unroll
    for (int t = 0; t < GA_ROWS; ++t)
        if (t0 + t < T) alpha[(size_t)(t0 + t) * C + c] = gla_root(z[t], p.power);
}

// ---------------------------------------------------------------------------------------------------------------
// Chunks of GC tokens in blocks of GB.  Rows of a chunk beyond its last token have q = k = v = 0 and a = 1.
constexpr int GC = 64, GB = 16, GNB = GC / GB;
constexpr int GCP = GC + 4;               // row stride of the tiles [feature][token]
constexpr int GC_THREADS = 512;
constexpr int GC_BATCH = 8;               // loads a thread has on their way at a time

#define GLA_FMA44(acc, a, b)                                                                                     \
    do {                                                                                                         \
        acc[0][0] = fmaf(a.x, b.x, acc[0][0]); acc[0][1] = fmaf(a.x, b.y, acc[0][1]); acc[0][2] = fmaf(a.x, b.z, acc[0][2]); acc[0][3] = fmaf(a.x, b.w, acc[0][3]); \
        acc[1][0] = fmaf(a.y, b.x, acc[1][0]); acc[1][1] = fmaf(a.y, b.y, acc[1][1]); acc[1][2] = fmaf(a.y, b.z, acc[1][2]); acc[1][3] = fmaf(a.y, b.w, acc[1][3]); \
        acc[2][0] = fmaf(a.z, b.x, acc[2][0]); acc[2][1] = fmaf(a.z, b.y, acc[2][1]); acc[2][2] = fmaf(a.z, b.z, acc[2][2]); acc[2][3] = fmaf(a.z, b.w, acc[2][3]); \
        acc[3][0] = fmaf(a.w, b.x, acc[3][0]); acc[3][1] = fmaf(a.w, b.y, acc[3][1]); acc[3][2] = fmaf(a.w, b.z, acc[3][2]); acc[3][3] = fmaf(a.w, b.w, acc[3][3]); \
    } while (0)

// The (row, column) of element tid + k * blockDim.x of a [rows][w] tile, stepped without a division per element.
struct GlaWalk {
    int j, i, dj, di, w;
    __device__ __forceinline__ GlaWalk(int w_) : w(w_) {
        j = (int)threadIdx.x / w; i = (int)threadIdx.x - j * w;
        dj = (int)blockDim.x / w; di = (int)blockDim.x - dj * w;
    }
    __device__ __forceinline__ void next() { i += di; j += dj; if (i >= w) { i -= w; ++j; } }
};

// Calls put(token, feature, x, y) for every element of a [GC][width] tile of which `rows` x `cols` are real; x = a[...], y =
// b[...] (b may be null) are fetched a batch at a time; elements that are not real get live = false.
template <typename Put>
__device__ __forceinline__ void gla_fill(int width, int rows, int cols, const float* a, size_t a_stride, const float* b, size_t b_stride,
                                         Put put) {
    for (GlaWalk w(width); w.j < GC;) {
        float x[GC_BATCH], y[GC_BATCH];
        int jj[GC_BATCH], ii[GC_BATCH];
#pragma unroll
        for (int u = 0; u < GC_BATCH; ++u) {
            jj[u] = w.j; ii[u] = w.i; w.next();
            const bool live = jj[u] < rows && ii[u] < cols;
            x[u] = live ? a[(size_t)jj[u] * a_stride + ii[u]] : 0.0f;
            y[u] = (live && b) ? b[(size_t)jj[u] * b_stride + ii[u]] : 0.0f;
        }
#pragma unroll
        for (int u = 0; u < GC_BATCH; ++u)
            if (jj[u] < GC) put(jj[u], ii[u], jj[u] < rows && ii[u] < cols, x[u], y[u]);
    }
}

__global__ void __launch_bounds__(GC_THREADS) gla_chunk_sum_kernel(GlaParams p) {
    extern __shared__ __align__(16) float gc_s[];
    const int n = p.n, nv = p.nv, np = p.np, nvp = p.nvp;
    float* Ks = gc_s;                          // [GC][np] k_j, then k_j times the decay from j to the chunk's end
    float* Vs = Ks + (size_t)GC * np;          // [GC][nvp]
    float* As = Vs + (size_t)GC * nvp;         // [GC][np]
    float* F = As + (size_t)GC * np;           // [GNB][np] a block's whole decay
    pdl_launch();
    pdl_wait();
    const int h = blockIdx.x, ch = blockIdx.y, tid = threadIdx.x;
    const int row0 = p.chunks[ch * 4 + 1], rows = p.chunks[ch * 4 + 2];
    const float* src = p.src + (size_t)row0 * p.src_stride;
    const size_t C = (size_t)p.H * n;
    gla_fill(np, rows, n, src + p.k_col + h * n, p.src_stride, p.forget ? nullptr : p.alpha + (size_t)row0 * C + h * n, C,
             [&](int j, int i, bool live, float x, float y) {
                 float a = 1.0f, k = 0.0f;
                 if (live) { if (p.forget) gla_forget(p, h * n + i, x, &a, &k); else { k = x; a = y; } }
                 Ks[j * np + i] = k;
                 As[j * np + i] = a;
             });
    gla_fill(nvp, rows, nv, src + p.v_col + h * nv, p.src_stride, nullptr, 0,
             [&](int j, int i, bool live, float x, float) { Vs[j * nvp + i] = x; });
    __syncthreads();
    for (int e = tid; e < GNB * np; e += blockDim.x) {           // a block's products from its end backwards
        const int b = e / np, i = e - b * np;
        float w = 1.0f;
#pragma unroll
        for (int j = GB - 1; j >= 0; --j) {
            const int at = (b * GB + j) * np + i;
            Ks[at] *= w;
            w *= As[at];
        }
        F[b * np + i] = w;
    }
    __syncthreads();
    for (int e = tid; e < GNB * np; e += blockDim.x) {           // ... and the whole blocks behind it
        const int b = e / np, i = e - b * np;
        float w = 1.0f;
        for (int m = b + 1; m < GNB; ++m) w *= F[m * np + i];
        if (b < GNB - 1)
#pragma unroll
            for (int j = 0; j < GB; ++j) Ks[(b * GB + j) * np + i] *= w;
        if (b == 0 && i < n) p.decay[((size_t)ch * p.H + h) * n + i] = w * F[i];
    }
    __syncthreads();
    float* A = p.work + ((size_t)ch * p.H + h) * n * nv;
    const int tc = nvp / 4, tiles = (np / 4) * tc;
    for (int tile = tid; tile < tiles; tile += blockDim.x) {
        const int i0 = (tile / tc) * 4, c0 = (tile % tc) * 4;
        float acc[4][4] = {};
#pragma unroll 4
        for (int j = 0; j < rows; ++j) {
            const float4 kk = *(const float4*)(Ks + (size_t)j * np + i0);
            const float4 vv = *(const float4*)(Vs + (size_t)j * nvp + c0);
            GLA_FMA44(acc, kk, vv);
        }
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b)
                if (i0 + a < n && c0 + b < nv) A[(size_t)(i0 + a) * nv + c0 + b] = acc[a][b];
    }
}

// A thread per element of the state walks its request's chunks: the chunk's sum is replaced by the state at its start, the
// slot gets the state behind the last.  Eight chunks' sums and decays are fetched at a time.
__global__ void __launch_bounds__(256) gla_chunk_scan_kernel(GlaParams p) {
    pdl_launch();
    pdl_wait();
    const int e = blockIdx.x * blockDim.x + threadIdx.x, h = blockIdx.y, l = blockIdx.z;
    const int sz = p.n * p.nv;
    if (e >= sz) return;
    const int req = p.longs[l * 4 + 0], rows = p.longs[l * 4 + 2], c0 = p.longs[l * 4 + 3];
    const int n_chunks = (rows + GC - 1) / GC;
    float* st = p.state + (size_t)p.slots[req] * p.slot_stride + (size_t)h * sz + e;
    float* a0 = p.work + ((size_t)c0 * p.H + h) * sz + e;
    const float* d0 = p.decay + ((size_t)c0 * p.H + h) * p.n + e / p.nv;
    const size_t step = (size_t)p.H * sz, dstep = (size_t)p.H * p.n;
    float S = *st;
    for (int c = 0; c < n_chunks; c += GC_BATCH) {
        float A[GC_BATCH], D[GC_BATCH];
#pragma unroll
        for (int u = 0; u < GC_BATCH; ++u) {
            A[u] = c + u < n_chunks ? a0[(size_t)(c + u) * step] : 0.0f;
            D[u] = c + u < n_chunks ? d0[(size_t)(c + u) * dstep] : 0.0f;
        }
#pragma unroll
        for (int u = 0; u < GC_BATCH; ++u)
            if (c + u < n_chunks) {
                a0[(size_t)(c + u) * step] = S;
                S = fmaf(D[u], S, A[u]);
            }
    }
    *st = S;
}

// o of every chunk.  Shared memory: q and k [feature][token]; a in a region that the values take over; the state; the
// scores of the chunk's own tokens [key][query]; the blocks' decays.  The keys' region ends as the outputs [token][column].
__global__ void __launch_bounds__(GC_THREADS) gla_chunk_out_kernel(GlaParams p) {
    extern __shared__ __align__(16) float gc_s[];
    const int n = p.n, nv = p.nv, np = p.np, nvp = p.nvp;
    const int k_floats = max(np * GCP, GC * nvp);
    float* Qt = gc_s;                          // [np][GCP]
    float* Kt = Qt + (size_t)np * GCP;         // [np][GCP], later [GC][nvp]
    float* At = Kt + k_floats;                 // [np][GCP], later [GC][nvp]
    float* Ss = At + k_floats;                 // [np][nvp]
    float* Pt = Ss + (size_t)np * nvp;         // [GC (key)][GCP (query)]
    float* F = Pt + (size_t)GC * GCP;          // [GNB][np]
    pdl_launch();
    pdl_wait();
    const int h = blockIdx.x, ch = blockIdx.y, tid = threadIdx.x;
    const int row0 = p.chunks[ch * 4 + 1], rows = p.chunks[ch * 4 + 2];
    const float* src = p.src + (size_t)row0 * p.src_stride;
    const size_t C = (size_t)p.H * n;
    gla_fill(np, rows, n, src + p.q_col + h * n, p.src_stride, src + p.k_col + h * n, p.src_stride,
             [&](int j, int i, bool live, float x, float y) {
                 float a = 1.0f, k = 0.0f;
                 if (live) { if (p.forget) gla_forget(p, h * n + i, y, &a, &k); else k = y; }
                 Qt[(size_t)i * GCP + j] = live ? gla_query(p, x) : 0.0f;
                 Kt[(size_t)i * GCP + j] = k;
                 if (p.forget) At[(size_t)i * GCP + j] = a;
             });
    if (!p.forget)
        gla_fill(np, rows, n, p.alpha + (size_t)row0 * C + h * n, C, nullptr, 0,
                 [&](int j, int i, bool live, float x, float) { At[(size_t)i * GCP + j] = live ? x : 1.0f; });
    {
        const float* S0 = p.work + ((size_t)ch * p.H + h) * n * nv;
        for (GlaWalk w(nvp); w.j < np;) {
            float raw[GC_BATCH];
            int jj[GC_BATCH], ii[GC_BATCH];
#pragma unroll
            for (int u = 0; u < GC_BATCH; ++u) {
                jj[u] = w.j; ii[u] = w.i; w.next();
                raw[u] = (jj[u] < n && ii[u] < nv) ? S0[(size_t)jj[u] * nv + ii[u]] : 0.0f;
            }
#pragma unroll
            for (int u = 0; u < GC_BATCH; ++u)
                if (jj[u] < np) Ss[jj[u] * nvp + ii[u]] = raw[u];
        }
    }
    __syncthreads();
    // scores inside a block of GB tokens: eight threads per key j share the channels; each carries k_j times the decay from j
    // to t along as t moves on, so a score is one sum per query
    {
        const int g = tid & 7, jb = (tid >> 3) & (GB - 1), b = tid >> 7;            // 4 blocks x 16 keys x 8 threads
        const int j = b * GB + jb;
        float w[32];                                                                // channels g, g + 8, ...: up to 256
        const int per = (np + 7) / 8;
#pragma unroll
        for (int m = 0; m < 32; ++m) w[m] = (m < per && g + 8 * m < np) ? Kt[(size_t)(g + 8 * m) * GCP + j] : 0.0f;
        for (int s = 0; s < GB; ++s) {
            const int t = j + s;
            const bool on = jb + s < GB;
            float acc = 0.0f;
            if (on) {
#pragma unroll
                for (int m = 0; m < 32; ++m) {
                    const int i = g + 8 * m;
                    if (m < per && i < np) {
                        if (s > 0) w[m] *= At[(size_t)i * GCP + t];
                        acc = fmaf(w[m], Qt[(size_t)i * GCP + t], acc);
                    }
                }
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            if (g == 0) {
                if (on) Pt[(size_t)j * GCP + t] = acc;
                else Pt[(size_t)j * GCP + b * GB + (jb + s - GB)] = 0.0f;           // queries in front of the key
            }
        }
    }
    __syncthreads();
    // q_t times the decay from its block's start up to t, k_j times the decay behind j to its block's end, the block's decay
    for (int e = tid; e < GNB * np; e += blockDim.x) {
        const int b = e / np, i = e - b * np;
        float* q = Qt + (size_t)i * GCP + b * GB;
        float* k = Kt + (size_t)i * GCP + b * GB;
        const float* a = At + (size_t)i * GCP + b * GB;
        float w = 1.0f;
#pragma unroll
        for (int t = 0; t < GB; ++t) { w *= a[t]; q[t] *= w; }
        F[b * np + i] = w;
        w = 1.0f;
#pragma unroll
        for (int t = GB - 1; t >= 0; --t) { k[t] *= w; w *= a[t]; }
    }
    __syncthreads();
    // the values take the decays' place; meanwhile scores across blocks: a 4 x 4 tile (queries, keys) per four threads, which
    // share the channels
    gla_fill(nvp, rows, nv, src + p.v_col + h * nv, p.src_stride, nullptr, 0,
             [&](int j, int i, bool live, float x, float) { At[(size_t)j * nvp + i] = x; });
    {
        constexpr int PAIRS = GNB * (GNB - 1) / 2, PER_PAIR = (GB / 4) * (GB / 4);
        for (int e = tid; e < PAIRS * PER_PAIR * 4; e += blockDim.x) {               // (a multiple of 32 threads takes part)
            const int part = e & 3, tile = e >> 2;
            const int pair = tile / PER_PAIR, in = tile % PER_PAIR;
            int I = 1, J = pair;                                                     // pairs (1,0) (2,0) (2,1) (3,0) ...
            while (J >= I) { J -= I; ++I; }
            const int t0 = I * GB + (in / (GB / 4)) * 4, j0 = J * GB + (in % (GB / 4)) * 4;
            float acc[4][4] = {};
            for (int i = part; i < np; i += 4) {
                float4 qq = *(const float4*)(Qt + (size_t)i * GCP + t0);
                const float4 kk = *(const float4*)(Kt + (size_t)i * GCP + j0);
                float mid = 1.0f;
                for (int m = J + 1; m < I; ++m) mid *= F[m * np + i];
                qq.x *= mid; qq.y *= mid; qq.z *= mid; qq.w *= mid;
                GLA_FMA44(acc, qq, kk);
            }
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
                for (int b = 0; b < 4; ++b) {
                    acc[a][b] += __shfl_xor_sync(0xffffffffu, acc[a][b], 1);
                    acc[a][b] += __shfl_xor_sync(0xffffffffu, acc[a][b], 2);
                }
            // thread `part` of the four stores the tile's key j0 + part
#pragma unroll
            for (int b = 0; b < 4; ++b)
                if (b == part)
                    *(float4*)(Pt + (size_t)(j0 + b) * GCP + t0) = make_float4(acc[0][b], acc[1][b], acc[2][b], acc[3][b]);
        }
    }
    __syncthreads();
    // q_t times the decay from the CHUNK's start: the whole blocks in front of its own
    for (int e = tid; e < (GNB - 1) * np; e += blockDim.x) {
        const int b = 1 + e / np, i = e - (b - 1) * np;
        float w = 1.0f;
        for (int m = 0; m < b; ++m) w *= F[m * np + i];
        float* q = Qt + (size_t)i * GCP + b * GB;
#pragma unroll
        for (int t = 0; t < GB; ++t) q[t] *= w;
    }
    __syncthreads();
    const float* Vs = At;
    float* Os = Kt;
    const int tc = nvp / 4, tiles = (GC / 4) * tc;
    for (int tile = tid; tile < tiles; tile += blockDim.x) {
        const int t0 = (tile / tc) * 4, c0 = (tile % tc) * 4;
        if (t0 >= rows) continue;
        float acc[4][4] = {};
#pragma unroll 4
        for (int i = 0; i < n; ++i) {
            const float4 qq = *(const float4*)(Qt + (size_t)i * GCP + t0);
            const float4 ss = *(const float4*)(Ss + (size_t)i * nvp + c0);
            GLA_FMA44(acc, qq, ss);
        }
        const int jend = min(rows, t0 + 4);
#pragma unroll 4
        for (int j = 0; j < jend; ++j) {
            const float4 pp = *(const float4*)(Pt + (size_t)j * GCP + t0);
            const float4 vv = *(const float4*)(Vs + (size_t)j * nvp + c0);
            GLA_FMA44(acc, pp, vv);
        }
#pragma unroll
        for (int a = 0; a < 4; ++a)
            *(float4*)(Os + (size_t)(t0 + a) * nvp + c0) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
    }
    __syncthreads();
    // the norm over a head's columns, its weight, the gate: a warp per token
    const int warp = tid >> 5, lane = tid & 31;
    for (int t = warp; t < rows; t += GC_THREADS / 32) {
        const float* o = Os + (size_t)t * nvp;
        float ss = 0.0f;
        for (int c = lane; c < nv; c += 32) ss += o[c] * o[c];
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)nv + p.eps);
        const float* row = src + (size_t)t * p.src_stride;
        for (int c = lane; c < nv; c += 32)
            gla_store(p, (size_t)(row0 + t) * p.H * nv + (size_t)h * nv + c, o[c] * inv * p.norm_w[c] * gla_gate(p, row, h, c));
    }
}

static size_t gla_out_smem(int np, int nvp) {
    const size_t k = (size_t)np * GCP > (size_t)GC * nvp ? (size_t)np * GCP : (size_t)GC * nvp;
    return ((size_t)np * GCP + 2 * k + (size_t)np * nvp + (size_t)GC * GCP + (size_t)GNB * np) * sizeof(float);
}
static size_t gla_sum_smem(int np, int nvp) { return ((size_t)2 * GC * np + (size_t)GC * nvp + (size_t)GNB * np) * sizeof(float); }
constexpr size_t GLA_SMEM_MAX = 224 * 1024;

}  // namespace bg

using namespace bg;

// What all entries share, as one struct of plain fields that the host side fills by name.
struct GlaArgs {
    const float* src; long long src_stride;
    int q_col, k_col, v_col, g_col, forget, q_silu, r_col, rank;
    float q_scale, power, eps, pad;
    const float* bias; const float* lower; const float* wa; const float* norm_w;
    float* state; long long slot_stride; const int* slots;
    void* out; int out_dtype, H, n, nv;
};

static int gla_params(GlaParams& p, const GlaArgs* a) {
    if (a->H <= 0 || a->n <= 0 || a->nv <= 0 || a->H > 65535 || (a->forget ? !a->lower : (!a->wa || a->rank < 1)) || !a->bias || !a->norm_w) return BG_ERR_SHAPE;
    if (a->out_dtype != BG_DTYPE_F32 && a->out_dtype != BG_DTYPE_BF16) return BG_ERR_DTYPE;
    p.src = a->src; p.src_stride = (int)a->src_stride; p.q_col = a->q_col; p.k_col = a->k_col; p.v_col = a->v_col; p.g_col = a->g_col;
    p.forget = a->forget; p.q_silu = a->q_silu; p.q_scale = a->q_scale; p.bias = a->bias; p.lower = a->lower; p.r_col = a->r_col;
    p.rank = a->rank; p.wa = a->wa; p.power = a->power; p.alpha = nullptr; p.norm_w = a->norm_w; p.eps = a->eps; p.state = a->state;
    p.slot_stride = (size_t)a->slot_stride; p.slots = a->slots; p.reqs = nullptr; p.out = a->out; p.out_float = a->out_dtype == BG_DTYPE_F32;
    p.H = a->H; p.n = a->n; p.nv = a->nv; p.chunks = nullptr; p.longs = nullptr; p.work = nullptr; p.decay = nullptr;
    p.np = (a->n + 3) / 4 * 4; p.nvp = (a->nv + 3) / 4 * 4;
    return BG_OK;
}

extern "C" int bg_gla_walk(const GlaArgs* args, const int* reqs, int n_req, cudaStream_t stream) {
    if (n_req <= 0) return BG_OK;
    GlaParams p;
    const int rc = gla_params(p, args);
    if (rc != BG_OK) return rc;
    if (n_req > 65535) return BG_ERR_SHAPE;
    p.reqs = reqs;
    const dim3 grid(p.H, n_req);
    // whole columns per block of up to 512 threads, four to 64 rows of its column a thread
    if (p.nv <= 512) {
        int slices = 512 / p.nv, R = 4;
        while (R < 64 && slices * R < p.n) R *= 2;
        slices = (p.n + R - 1) / R < slices ? (p.n + R - 1) / R : slices;
        const int threads = (slices * p.nv + 31) / 32 * 32;
        const size_t smem = ((size_t)3 * slices * R + p.nv + (size_t)slices * p.nv) * sizeof(float);
        if (slices * R >= p.n && smem <= BG_SMEM_OPT_IN) {
            switch (R) {
                case 4: launch(gla_walk_kernel<4>, grid, dim3(threads), smem, stream, p, slices); break;
                case 8: launch(gla_walk_kernel<8>, grid, dim3(threads), smem, stream, p, slices); break;
                case 16: launch(gla_walk_kernel<16>, grid, dim3(threads), smem, stream, p, slices); break;
                case 32: launch(gla_walk_kernel<32>, grid, dim3(threads), smem, stream, p, slices); break;
                default: launch(gla_walk_kernel<64>, grid, dim3(threads), smem, stream, p, slices); break;
            }
            BG_LAUNCH_CHECK();
            return BG_OK;
        }
    }
    const size_t smem = ((size_t)3 * p.n + 2 * p.nv) * sizeof(float);
    if (smem > 200 * 1024) return BG_ERR_UNSUPPORTED;
    if (smem > BG_SMEM_OPT_IN) {
        cudaError_t e = cudaFuncSetAttribute(gla_walk_mem_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    launch(gla_walk_mem_kernel, grid, dim3(256), smem, stream, p);
    BG_LAUNCH_CHECK();
    return BG_OK;
}

// 0 when the chunked kernels take heads of n x nv values (their tiles fit in shared memory), else BG_ERR_UNSUPPORTED.
extern "C" int bg_gla_chunk_plan(int n, int nv, int* chunk) {
    if (n <= 0 || nv <= 0) return BG_ERR_SHAPE;
    const int np = (n + 3) / 4 * 4, nvp = (nv + 3) / 4 * 4;
    if (chunk) *chunk = GC;
    return np <= 256 && gla_out_smem(np, nvp) <= GLA_SMEM_MAX && gla_sum_smem(np, nvp) <= GLA_SMEM_MAX ? BG_OK : BG_ERR_UNSUPPORTED;
}

// Requests of many rows: chunks [n_chunks][4] and longs [n_long][4] as in decay_attention.cu; work float [n_chunks][H][n nv],
// decay float [n_chunks][H][n], alpha float [T][H n] (DECAY only; n_rows = T).
extern "C" int bg_gla_chunked(const GlaArgs* args, int n_rows, const int* chunks, int n_chunks, const int* longs, int n_long, float* work,
                              float* decay, float* alpha, cudaStream_t stream) {
    if (n_chunks <= 0 || n_long <= 0) return BG_OK;
    GlaParams p;
    const int rc = gla_params(p, args);
    if (rc != BG_OK) return rc;
    if (n_chunks > 65535 || n_long > 65535 || (!p.forget && !alpha)) return BG_ERR_SHAPE;
    if (bg_gla_chunk_plan(p.n, p.nv, nullptr) != BG_OK) return BG_ERR_UNSUPPORTED;
    p.chunks = chunks; p.longs = longs; p.work = work; p.decay = decay; p.alpha = alpha;
    const size_t smem_sum = gla_sum_smem(p.np, p.nvp), smem_out = gla_out_smem(p.np, p.nvp);
    if (smem_sum > BG_SMEM_OPT_IN) {
        cudaError_t e = cudaFuncSetAttribute(gla_chunk_sum_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_sum);
        if (e != cudaSuccess) return (int)e;
    }
    if (smem_out > BG_SMEM_OPT_IN) {
        cudaError_t e = cudaFuncSetAttribute(gla_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_out);
        if (e != cudaSuccess) return (int)e;
    }
    if (!p.forget) {
        const int row_blocks = (n_rows + GA_ROWS - 1) / GA_ROWS;
        if (row_blocks > 65535) return BG_ERR_SHAPE;
        launch(gla_alpha_kernel, dim3((p.H * p.n + 255) / 256, row_blocks), dim3(256), 0, stream, p, alpha, n_rows);
        BG_LAUNCH_CHECK();
    }
    launch(gla_chunk_sum_kernel, dim3(p.H, n_chunks), dim3(GC_THREADS), smem_sum, stream, p);
    BG_LAUNCH_CHECK();
    launch(gla_chunk_scan_kernel, dim3((p.n * p.nv + 255) / 256, p.H, n_long), dim3(256), 0, stream, p);
    BG_LAUNCH_CHECK();
    launch(gla_chunk_out_kernel, dim3(p.H, n_chunks), dim3(GC_THREADS), smem_out, stream, p);
    BG_LAUNCH_CHECK();
    return BG_OK;
}
