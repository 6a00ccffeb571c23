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
//   gla_chunk_*          long portions in chunks of GC tokens: per chunk the gates, the decayed queries and keys and the scores
//                        of the chunk's own tokens; the chunks' decayed sums of k v^T; a pass over the chunks that turns them
//                        into the states at the chunks' starts; the chunks' outputs, normed and gated.
//
// A decay between two tokens is a PRODUCT of the a's between them; it is never formed as a quotient of products from a
// chunk's start (which underflow) nor from logarithms (a may be 0).  A chunk is cut into blocks of GB tokens, and a product
// over tokens of several blocks is split at the blocks' borders: (from the key's token to its block's end) x (whole blocks
// between) x (from the start of the query's block to its token), each a running product of numbers in [0, 1].
#include "common.cuh"

namespace bg {

// (sigmoid(z), sigmoid(-z)) from one exponential of a number that is not positive
__device__ __forceinline__ float2 gla_sigmoids(float z) {
    const float e = expf(-fabsf(z)), big = __frcp_rn(1.0f + e), small = e * big;
    return z >= 0.0f ? make_float2(big, small) : make_float2(small, big);
}
__device__ __forceinline__ float gla_silu(float z) { return z * gla_sigmoids(z).x; }
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
    const float* norm_w; float eps;             // [nv]
    float* state; size_t slot_stride;           // slab [slots][>= H n nv]
    const int* slots;
    const int* reqs;                            // [n_req][3] = (request, first row, rows)
    void* out; int out_float;                   // [T][H nv]
    int H, n, nv;
    // chunks
    const int* chunks;                          // [n_chunks][4] = (request, first row, rows, -)
    const int* longs;                           // [n_long][4]   = (request, first row, rows, first chunk)
    float* qd; float* kd;                       // [T][H np] queries times the decay from the chunk's start, keys times that to its end
    float* scores;                              // [n_chunks][H][GC (t)][GC (j)], j <= t (and noughts up to the end of t's block)
    float* work;                                // [n_chunks][H][np nvp]
    float* decay;                               // [n_chunks][H][n] the chunk's whole decay
    int np, nvp;                                // n, nv rounded up to multiples of 4
    int vec, vec_qk;                            // rows of values, and of q and k, lie on 16-byte boundaries
};

__device__ __forceinline__ float gla_query(const GlaParams& p, float raw) { return p.q_silu ? gla_silu(raw) * p.q_scale : raw * p.q_scale; }
// FORGET: (a, k) from the gate's product z of channel c
__device__ __forceinline__ void gla_forget(const GlaParams& p, int c, float raw, float* a, float* k) {
    const float l = p.lower[c];
    const float2 g = gla_sigmoids(raw + p.bias[c]);
    *a = fmaf(1.0f - l, g.x, l);
    *k = (1.0f - l) * g.y;
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

// ---------------------------------------------------------------------------------------------------------------
// Chunks of GC tokens in blocks of GB.  Rows of a chunk beyond its last token have q = k = v = 0 and a = 1.
constexpr int GC = 64, GB = 16, GNB = GC / GB;
constexpr int GCP = GC + 4;               // row stride of the score tile
constexpr int GPT = 64;                   // value columns of a block
constexpr int GC_BATCH = 8;               // loads (of 16 bytes: half as many) a thread has on their way at a time
constexpr int GLA_RANK = 16;              // features of the short row taken at a time

// The (row, column) of element tid + k * blockDim.x of a [rows][w] tile, stepped without a division per element.
struct GlaWalk {
    int j, i, dj, di, w;
    __device__ __forceinline__ GlaWalk(int w_) : w(w_) {
        j = (int)threadIdx.x / w; i = (int)threadIdx.x - j * w;
        dj = (int)blockDim.x / w; di = (int)blockDim.x - dj * w;
    }
    __device__ __forceinline__ void next() { i += di; j += dj; if (i >= w) { i -= w; ++j; } }
};

__device__ __forceinline__ void gla_async16(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void gla_async_wait() { asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;\n" ::: "memory"); }

// `n_rows` rows of `w` floats into a tile of row stride `ld` whose rows are `wp` wide (a multiple of 4); what lies beyond `rows`
// and `w` becomes nought.  16 bytes at a time when `vec` (rows on 16-byte boundaries, w a multiple of 4).
__device__ __forceinline__ void gla_rows(float* dst, int ld, const float* src, size_t stride, int n_rows, int rows, int w, int wp, int vec) {
    if (vec) {
        const int w4 = wp >> 2;
        for (int idx = threadIdx.x; idx < n_rows * w4; idx += blockDim.x) {
            const int r = idx / w4, c = (idx - r * w4) * 4;
            if (r < rows && c < w) gla_async16(dst + (size_t)r * ld + c, src + (size_t)r * stride + c);
            else *reinterpret_cast<float4*>(dst + (size_t)r * ld + c) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    } else {
        for (int idx = threadIdx.x; idx < n_rows * wp; idx += blockDim.x) {
            const int r = idx / wp, c = idx - r * wp;
            dst[(size_t)r * ld + c] = (r < rows && c < w) ? src[(size_t)r * stride + c] : 0.0f;
        }
    }
}

// (M groups of 32 channels cover np; a block of 256 threads)
template <int M>
__device__ __forceinline__ void gla_block_scores(const float* Qs, const float* Ks, const float* As, float* sc, int np, int ld) {
    for (int pass = 0; pass < 2; ++pass) {
        const int slot = (int)threadIdx.x + pass * 256;
        const int g = slot & 7, jb = (slot >> 3) & (GB - 1), b = slot >> 7;         // 4 blocks x 16 keys x 8 threads
        const int j = b * GB + jb, steps = GB - (jb & ~3);                          // a warp's four keys are neighbours
        float4 w[M];
#pragma unroll
        for (int m = 0; m < M; ++m) {
            const int i = 4 * g + 32 * m;
            w[m] = i < np ? *reinterpret_cast<const float4*>(Ks + j * ld + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        for (int s = 0; s < steps; ++s) {
            const int t = j + s;
            const bool on = jb + s < GB;
            float acc = 0.0f;
            if (on) {
#pragma unroll
                for (int m = 0; m < M; ++m) {
                    const int i = 4 * g + 32 * m;
                    if (i < np) {
                        if (s > 0) {
                            const float4 a = *reinterpret_cast<const float4*>(As + t * ld + i);
                            w[m].x *= a.x; w[m].y *= a.y; w[m].z *= a.z; w[m].w *= a.w;
                        }
                        const float4 q = *reinterpret_cast<const float4*>(Qs + t * ld + i);
                        acc = fmaf(w[m].x, q.x, fmaf(w[m].y, q.y, fmaf(w[m].z, q.z, fmaf(w[m].w, q.w, acc))));
                    }
                }
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            if (g == 0 && on) sc[t * GC + j] = acc;
        }
        for (int t = g; t < jb; t += 8) sc[(b * GB + t) * GC + j] = 0.0f;           // queries in front of the key
    }
}

__global__ void __launch_bounds__(256) gla_chunk_prep_kernel(GlaParams p) {
    extern __shared__ __align__(16) float gc_s[];
    const int n = p.n, np = p.np, ld = np + 8;
    float* Qs = gc_s;                          // [GC][ld]
    float* Ks = Qs + (size_t)GC * ld;          // [GC][ld]
    float* As = Ks + (size_t)GC * ld;          // [GC][ld]
    float* F = As + (size_t)GC * ld;           // [GNB][np] a block's whole decay
    pdl_launch();
    pdl_wait();
    const int h = blockIdx.x, ch = blockIdx.y, tid = threadIdx.x;
    const int row0 = p.chunks[ch * 4 + 1], rows = p.chunks[ch * 4 + 2];
    const float* src = p.src + (size_t)row0 * p.src_stride;
    {
        // four channels of a token at a time; GC_BATCH / 2 such groups' loads on their way together
        const int n4 = np >> 2;
        for (GlaWalk w(n4); w.j < GC;) {
            float4 x[GC_BATCH / 2], y[GC_BATCH / 2];
            int jj[GC_BATCH / 2], ii[GC_BATCH / 2];
#pragma unroll
            for (int u = 0; u < GC_BATCH / 2; ++u) {
                jj[u] = w.j; ii[u] = 4 * w.i; w.next();
                x[u] = y[u] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (jj[u] < rows) {
                    const float* r = src + (size_t)jj[u] * p.src_stride + h * n + ii[u];
                    if (p.vec_qk) {
                        x[u] = *reinterpret_cast<const float4*>(r + p.q_col);
                        y[u] = *reinterpret_cast<const float4*>(r + p.k_col);
                    } else {
                        const int m = n - ii[u];
                        x[u] = make_float4(r[p.q_col], m > 1 ? r[p.q_col + 1] : 0.0f, m > 2 ? r[p.q_col + 2] : 0.0f, m > 3 ? r[p.q_col + 3] : 0.0f);
                        y[u] = make_float4(r[p.k_col], m > 1 ? r[p.k_col + 1] : 0.0f, m > 2 ? r[p.k_col + 2] : 0.0f, m > 3 ? r[p.k_col + 3] : 0.0f);
                    }
                }
            }
#pragma unroll
            for (int u = 0; u < GC_BATCH / 2; ++u) {
                if (jj[u] >= GC) continue;
                const float xs[4] = {x[u].x, x[u].y, x[u].z, x[u].w}, ys[4] = {y[u].x, y[u].y, y[u].z, y[u].w};
                float q[4], k[4], a[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    q[e] = k[e] = 0.0f; a[e] = 1.0f;
                    if (jj[u] < rows && ii[u] + e < n) {
                        q[e] = gla_query(p, xs[e]);
                        if (p.forget) gla_forget(p, h * n + ii[u] + e, ys[e], &a[e], &k[e]); else k[e] = ys[e];
                    }
                }
                const int at = jj[u] * ld + ii[u];
                *reinterpret_cast<float4*>(Qs + at) = make_float4(q[0], q[1], q[2], q[3]);
                *reinterpret_cast<float4*>(Ks + at) = make_float4(k[0], k[1], k[2], k[3]);
                if (p.forget) *reinterpret_cast<float4*>(As + at) = make_float4(a[0], a[1], a[2], a[3]);
            }
        }
    }
    if (!p.forget) {
        // z = W r + b: the short rows in F's place (a few features at a time), a thread per channel and every tokens-th token
        float* Rs = F;                         // [GC][GLA_RANK]
        for (int r0 = 0; r0 < p.rank; r0 += GLA_RANK) {
            __syncthreads();
            for (int idx = tid; idx < GC * GLA_RANK; idx += blockDim.x) {
                const int t = idx / GLA_RANK, r = idx % GLA_RANK;
                Rs[idx] = (t < rows && r0 + r < p.rank) ? src[(size_t)t * p.src_stride + p.r_col + r0 + r] : 0.0f;
            }
            __syncthreads();
            const int lanes = np < 256 ? 256 / np : 1;                       // threads that share a channel
            for (int i = lanes > 1 ? tid % np : tid; i < np; i += 256) {
                const int part = lanes > 1 ? tid / np : 0;
                if (part >= lanes) break;
                const int c = h * n + (i < n ? i : 0);
                float w[GLA_RANK];
#pragma unroll
                for (int r = 0; r < GLA_RANK; ++r) w[r] = (i < n && r0 + r < p.rank) ? p.wa[(size_t)c * p.rank + r0 + r] : 0.0f;
                const float b = i < n ? p.bias[c] : 0.0f;
                const bool last = r0 + GLA_RANK >= p.rank;
                for (int t = part; t < GC; t += lanes) {
                    float z = r0 == 0 ? b : As[t * ld + i];
#pragma unroll
                    for (int r = 0; r < GLA_RANK; r += 4) {
                        const float4 v = *reinterpret_cast<const float4*>(Rs + t * GLA_RANK + r);
                        z = fmaf(w[r], v.x, z); z = fmaf(w[r + 1], v.y, z); z = fmaf(w[r + 2], v.z, z); z = fmaf(w[r + 3], v.w, z);
                    }
                    if (last) z = (t < rows && i < n) ? gla_root(z, p.power) : 1.0f;
                    As[t * ld + i] = z;
                }
                if (lanes > 1) break;
            }
        }
    }
    __syncthreads();
    float* sc = p.scores + ((size_t)ch * p.H + h) * GC * GC;
    // scores inside a block of GB tokens: eight threads per key j share the channels, four neighbours at a time; each carries k_j
    // times the decay from j to t along as t moves on, so a score is one sum per query
    if (np <= 32) gla_block_scores<1>(Qs, Ks, As, sc, np, ld);
    else if (np <= 64) gla_block_scores<2>(Qs, Ks, As, sc, np, ld);
    else if (np <= 128) gla_block_scores<4>(Qs, Ks, As, sc, np, ld);
    else gla_block_scores<8>(Qs, Ks, As, sc, np, ld);
    __syncthreads();
    // q_t times the decay from its block's start up to t, k_j times the decay behind j to its block's end, the block's decay
    for (int e = tid; e < GNB * np; e += blockDim.x) {
        const int b = e / np, i = e - b * np;
        const int at = b * GB * ld + i;
        float w = 1.0f;
#pragma unroll
        for (int t = 0; t < GB; ++t) { w *= As[at + t * ld]; Qs[at + t * ld] *= w; }
        F[b * np + i] = w;
        w = 1.0f;
#pragma unroll
        for (int t = GB - 1; t >= 0; --t) { Ks[at + t * ld] *= w; w *= As[at + t * ld]; }
    }
    __syncthreads();
    // scores across blocks: a tile of 4 x 4 (queries tq + 4 u, keys jq + 4 v of their blocks) per two threads, which share the
    // channels; a warp's tiles are those of one pair of blocks
    constexpr int PAIRS = GNB * (GNB - 1) / 2, PER_PAIR = (GB / 4) * (GB / 4);
    if (tid < PAIRS * PER_PAIR * 2) {
        const int part = tid & 1, tile = tid >> 1;
        const int pair = tile / PER_PAIR, in = tile % PER_PAIR;
        int I = 1, J = pair;                                                         // pairs (1,0) (2,0) (2,1) (3,0) ...
        while (J >= I) { J -= I; ++I; }
        const int t0 = I * GB + in / (GB / 4), j0 = J * GB + in % (GB / 4);
        float acc[4][4] = {};
        for (int i = 4 * part; i < np; i += 8) {
            float4 k[4];
#pragma unroll
            for (int v = 0; v < 4; ++v) k[v] = *reinterpret_cast<const float4*>(Ks + (j0 + 4 * v) * ld + i);
            for (int b = J + 1; b < I; ++b) {
                const float4 f = *reinterpret_cast<const float4*>(F + b * np + i);
#pragma unroll
                for (int v = 0; v < 4; ++v) { k[v].x *= f.x; k[v].y *= f.y; k[v].z *= f.z; k[v].w *= f.w; }
            }
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float4 q = *reinterpret_cast<const float4*>(Qs + (t0 + 4 * u) * ld + i);
#pragma unroll
                for (int v = 0; v < 4; ++v)
                    acc[u][v] = fmaf(q.x, k[v].x, fmaf(q.y, k[v].y, fmaf(q.z, k[v].z, fmaf(q.w, k[v].w, acc[u][v]))));
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int v = 0; v < 4; ++v) {
                acc[u][v] += __shfl_xor_sync(0xffffffffu, acc[u][v], 1);
                if ((u >> 1) == part) sc[(t0 + 4 * u) * GC + j0 + 4 * v] = acc[u][v];
            }
    }
    __syncthreads();
    // the queries with the whole blocks in front of theirs, the keys with those behind
    const int n4 = np >> 2;
    for (int idx = tid; idx < rows * n4; idx += blockDim.x) {
        const int t = idx / n4, i = (idx - t * n4) * 4, b = t / GB;
        float4 q = *reinterpret_cast<const float4*>(Qs + t * ld + i), k = *reinterpret_cast<const float4*>(Ks + t * ld + i);
#pragma unroll
        for (int m = 0; m < GNB; ++m) {
            const float4 f = *reinterpret_cast<const float4*>(F + m * np + i);
            if (m < b) { q.x *= f.x; q.y *= f.y; q.z *= f.z; q.w *= f.w; }
            if (m > b) { k.x *= f.x; k.y *= f.y; k.z *= f.z; k.w *= f.w; }
        }
        const size_t at = ((size_t)(row0 + t) * p.H + h) * np + i;
        *reinterpret_cast<float4*>(p.qd + at) = q;
        *reinterpret_cast<float4*>(p.kd + at) = k;
    }
    for (int i = tid; i < n; i += blockDim.x) {
        float w = F[i];
#pragma unroll
        for (int m = 1; m < GNB; ++m) w *= F[m * np + i];
        p.decay[((size_t)ch * p.H + h) * n + i] = w;
    }
}

__global__ void __launch_bounds__(256) gla_chunk_sum_kernel(GlaParams p) {
    extern __shared__ __align__(16) float gc_s[];
    const int np = p.np, nvp = p.nvp;
    float* Ks = gc_s;                          // [GC][np]
    float* Vs = Ks + (size_t)GC * np;          // [GC][GPT]
    pdl_launch();
    pdl_wait();
    const int h = blockIdx.x, ch = blockIdx.y, c_first = blockIdx.z * GPT, tid = threadIdx.x;
    const int wp = min(GPT, nvp - c_first), w = min(GPT, p.nv - c_first);
    const int row0 = p.chunks[ch * 4 + 1], rows = p.chunks[ch * 4 + 2];
    gla_rows(Ks, np, p.kd + ((size_t)row0 * p.H + h) * np, (size_t)p.H * np, GC, rows, np, np, 1);
    gla_rows(Vs, GPT, p.src + (size_t)row0 * p.src_stride + p.v_col + h * p.nv + c_first, p.src_stride, GC, rows, w, wp, p.vec);
    gla_async_wait();
    __syncthreads();
    float* A = p.work + ((size_t)ch * p.H + h) * np * nvp + c_first;
    const int tp = wp >> 2, tn = (np + 7) >> 3;
    for (int tile = tid; tile < tn * tp; tile += blockDim.x) {
        const int i0 = (tile / tp) * 8, c0 = (tile % tp) * 4;
        const bool two = i0 + 4 < np;
        float acc[8][4] = {};
#pragma unroll 4
        for (int j = 0; j < GC; ++j) {
            const float4 v = *reinterpret_cast<const float4*>(Vs + j * GPT + c0);
            const float4 k0 = *reinterpret_cast<const float4*>(Ks + (size_t)j * np + i0);
            const float4 k1 = two ? *reinterpret_cast<const float4*>(Ks + (size_t)j * np + i0 + 4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            const float k[8] = {k0.x, k0.y, k0.z, k0.w, k1.x, k1.y, k1.z, k1.w};
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                acc[u][0] = fmaf(k[u], v.x, acc[u][0]); acc[u][1] = fmaf(k[u], v.y, acc[u][1]);
                acc[u][2] = fmaf(k[u], v.z, acc[u][2]); acc[u][3] = fmaf(k[u], v.w, acc[u][3]);
            }
        }
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (i0 + u < np) *reinterpret_cast<float4*>(A + (size_t)(i0 + u) * nvp + c0) = make_float4(acc[u][0], acc[u][1], acc[u][2], acc[u][3]);
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
    const int i = e / p.nv, c_at = e - i * p.nv;
    float* st = p.state + (size_t)p.slots[req] * p.slot_stride + (size_t)h * sz + e;
    const size_t pad = (size_t)p.np * p.nvp;
    float* a0 = p.work + ((size_t)c0 * p.H + h) * pad + (size_t)i * p.nvp + c_at;
    const float* d0 = p.decay + ((size_t)c0 * p.H + h) * p.n + i;
    const size_t step = (size_t)p.H * pad, dstep = (size_t)p.H * p.n;
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

// The token that a thread's row u (of eight) stands for: a warp holds sixteen tokens, a half of it four neighbours and the four
// eight further on, so that the two halves' reads of a tile of rows fall on different banks.
__device__ __forceinline__ int gla_token(int u) {
    return ((int)threadIdx.x >> 5) * 16 + (((int)threadIdx.x >> 4) & 1) * 4 + (u & 3) + (u >> 2) * 8;
}

// acc[u][v] += sum over k of a[token of row u][k] b[k][v], k in steps of 4 up to `k_end`
__device__ __forceinline__ void gla_product(float (&acc)[8][4], const float* a, int lda, const float* b, int k_end) {
#pragma unroll 1
    for (int k = 0; k < k_end; k += 4) {
        float4 bb[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) bb[i] = *reinterpret_cast<const float4*>(b + (size_t)(k + i) * GPT);
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const float4 aa = *reinterpret_cast<const float4*>(a + gla_token(u) * lda + k);
            const float ak[4] = {aa.x, aa.y, aa.z, aa.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                acc[u][0] = fmaf(ak[i], bb[i].x, acc[u][0]); acc[u][1] = fmaf(ak[i], bb[i].y, acc[u][1]);
                acc[u][2] = fmaf(ak[i], bb[i].z, acc[u][2]); acc[u][3] = fmaf(ak[i], bb[i].w, acc[u][3]);
            }
        }
    }
}

// o of GPT columns of a head in a chunk, its norm and gate.  The blocks of a head's columns form a cluster along z (of 1, 2, 4 or
// 8: those beyond the columns only take part in its barriers) and add up their rows' sums of squares in one another's shared
// memory.
__global__ void __launch_bounds__(128) gla_chunk_out_kernel(GlaParams p) {
    extern __shared__ __align__(16) float gc_s[];
    __shared__ float ssq[8][GC];               // [rank in the cluster][token]
    const int np = p.np, nvp = p.nvp, ldq = np + 4;
    float* Qs = gc_s;                          // [GC][np + 4]
    float* Ss = Qs + (size_t)GC * ldq;         // [np][GPT]
    float* Vs = Ss + (size_t)np * GPT;         // [GC][GPT]
    float* Ws = Vs + (size_t)GC * GPT;         // [GC (t)][GCP] scores
    const int h = blockIdx.x, ch = blockIdx.y, rank = blockIdx.z, n_rank = gridDim.z, c_first = rank * GPT, tid = threadIdx.x;
    const int wp = max(0, min(GPT, nvp - c_first)), w = max(0, min(GPT, p.nv - c_first));
    if (n_rank > 1) cluster_arrive_relaxed();  // waited for before the first store to a peer: every peer runs by then
    pdl_launch();
    pdl_wait();
    const int row0 = p.chunks[ch * 4 + 1], rows = p.chunks[ch * 4 + 2];
    const float* src = p.src + (size_t)row0 * p.src_stride;
    gla_rows(Qs, ldq, p.qd + ((size_t)row0 * p.H + h) * np, (size_t)p.H * np, GC, rows, np, np, 1);
    gla_rows(Ss, GPT, p.work + ((size_t)ch * p.H + h) * np * nvp + c_first, nvp, np, np, wp, wp, 1);
    gla_rows(Ws, GCP, p.scores + ((size_t)ch * p.H + h) * GC * GC, GC, GC, GC, GC, GC, 1);
    gla_rows(Vs, GPT, src + p.v_col + h * p.nv + c_first, p.src_stride, GC, rows, w, wp, p.vec);
    gla_async_wait();
    __syncthreads();
    const int t0 = (tid >> 5) * 16, c0 = (tid & 15) * 4;        // the warp's first token
    float acc[8][4] = {};
    if (t0 < rows && c0 < wp) {
        gla_product(acc, Qs, ldq, Ss + c0, np);
        gla_product(acc, Ws, GCP, Vs + c0, t0 + GB);            // (a warp's tokens are one block of GB)
    }
    if (n_rank > 1) { __syncwarp(); cluster_wait(); }
    // (columns beyond the head's own are noughts: the values and the state hold noughts there)
#pragma unroll
    for (int u = 0; u < 8; ++u) {
        float s = acc[u][0] * acc[u][0] + acc[u][1] * acc[u][1] + acc[u][2] * acc[u][2] + acc[u][3] * acc[u][3];
#pragma unroll
        for (int o = 1; o < 16; o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if ((tid & 15) == 0) {
            const int t = gla_token(u);
            if (n_rank == 1) ssq[0][t] = s;
            else for (int q = 0; q < n_rank; ++q) st_cluster(peer_addr((unsigned)__cvta_generic_to_shared(&ssq[rank][t]), (unsigned)q), s);
        }
    }
    __syncwarp();
    if (n_rank > 1) cluster_sync_all(); else __syncthreads();
    if (c0 >= w) return;
#pragma unroll
    for (int u = 0; u < 8; ++u) {
        const int t = gla_token(u);
        if (t >= rows) continue;
        float total = 0.0f;
        for (int q = 0; q < n_rank; ++q) total += ssq[q][t];
        const float inv = 1.0f / sqrtf(total / (float)p.nv + p.eps);
        const float* row = src + (size_t)t * p.src_stride;
        const size_t at = (size_t)(row0 + t) * p.H * p.nv + (size_t)h * p.nv + c_first + c0;
#pragma unroll
        for (int v = 0; v < 4; ++v)
            if (c0 + v < w)
                gla_store(p, at + v, acc[u][v] * inv * p.norm_w[c_first + c0 + v] * gla_gate(p, row, h, c_first + c0 + v));
    }
}

static size_t gla_prep_smem(int np, int rank) {
    const size_t tail = (size_t)GNB * np > (size_t)GC * GLA_RANK || rank == 0 ? (size_t)GNB * np : (size_t)GC * GLA_RANK;
    return ((size_t)3 * GC * (np + 8) + tail) * sizeof(float);
}
static size_t gla_sum_smem(int np) { return ((size_t)GC * np + (size_t)GC * GPT) * sizeof(float); }
static size_t gla_out_smem(int np) { return ((size_t)GC * (np + 4) + (size_t)np * GPT + (size_t)GC * GPT + (size_t)GC * GCP) * sizeof(float); }
constexpr size_t GLA_SMEM_MAX = 222 * 1024;

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
    p.rank = a->rank; p.wa = a->wa; p.power = a->power; p.norm_w = a->norm_w; p.eps = a->eps; p.state = a->state;
    p.slot_stride = (size_t)a->slot_stride; p.slots = a->slots; p.reqs = nullptr; p.out = a->out; p.out_float = a->out_dtype == BG_DTYPE_F32;
    p.H = a->H; p.n = a->n; p.nv = a->nv; p.chunks = nullptr; p.longs = nullptr; p.work = nullptr; p.decay = nullptr; p.qd = nullptr; p.kd = nullptr; p.scores = nullptr;
    const bool rows16 = a->src_stride % 4 == 0 && (uintptr_t)a->src % 16 == 0;
    p.vec = rows16 && a->nv % 4 == 0 && a->v_col % 4 == 0;
    p.vec_qk = rows16 && a->n % 4 == 0 && a->q_col % 4 == 0 && a->k_col % 4 == 0;
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
    // (the blocks of a head's columns are a cluster of at most eight)
    return np <= 256 && nvp <= 8 * GPT && gla_prep_smem(np, 1) <= GLA_SMEM_MAX && gla_out_smem(np) <= GLA_SMEM_MAX ? BG_OK : BG_ERR_UNSUPPORTED;
}

// Requests of many rows: chunks [n_chunks][4] and longs [n_long][4] as in decay_attention.cu.  Scratch, float, np and nvp being n
// and nv rounded up to multiples of 4: qd and kd [T][H np], scores [n_chunks][H][64 * 64], work [n_chunks][H][np nvp], decay
// [n_chunks][H][n].
extern "C" int bg_gla_chunked(const GlaArgs* args, const int* chunks, int n_chunks, const int* longs, int n_long, float* qd, float* kd,
                              float* scores, float* work, float* decay, cudaStream_t stream) {
    if (n_chunks <= 0 || n_long <= 0) return BG_OK;
    GlaParams p;
    const int rc = gla_params(p, args);
    if (rc != BG_OK) return rc;
    if (n_chunks > 65535 || n_long > 65535) return BG_ERR_SHAPE;
    if (bg_gla_chunk_plan(p.n, p.nv, nullptr) != BG_OK) return BG_ERR_UNSUPPORTED;
    if ((uintptr_t)qd % 16 || (uintptr_t)kd % 16 || (uintptr_t)scores % 16 || (uintptr_t)work % 16) return BG_ERR_ALIGN;
    p.chunks = chunks; p.longs = longs; p.qd = qd; p.kd = kd; p.scores = scores; p.work = work; p.decay = decay;
    const size_t s_prep = gla_prep_smem(p.np, p.rank), s_sum = gla_sum_smem(p.np), s_out = gla_out_smem(p.np);
    const unsigned tiles = (unsigned)((p.nvp + GPT - 1) / GPT);
    cudaError_t e = cudaSuccess;
    if (s_prep > BG_SMEM_OPT_IN) e = cudaFuncSetAttribute(gla_chunk_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s_prep);
    if (e == cudaSuccess && s_sum > BG_SMEM_OPT_IN) e = cudaFuncSetAttribute(gla_chunk_sum_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s_sum);
    if (e == cudaSuccess && s_out > BG_SMEM_OPT_IN) e = cudaFuncSetAttribute(gla_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s_out);
    if (e != cudaSuccess) return (int)e;
    launch(gla_chunk_prep_kernel, dim3(p.H, n_chunks), dim3(256), s_prep, stream, p);
    BG_LAUNCH_CHECK();
    launch(gla_chunk_sum_kernel, dim3(p.H, n_chunks, tiles), dim3(256), s_sum, stream, p);
    BG_LAUNCH_CHECK();
    launch(gla_chunk_scan_kernel, dim3((p.n * p.nv + 255) / 256, p.H, n_long), dim3(256), 0, stream, p);
    BG_LAUNCH_CHECK();
    const unsigned cluster = tiles <= 2 ? tiles : tiles <= 4 ? 4 : 8;
    launch_cluster(gla_chunk_out_kernel, dim3(p.H, n_chunks, cluster), dim3(128), s_out, stream, (int)cluster, p);
    BG_LAUNCH_CHECK();
    return BG_OK;
}
