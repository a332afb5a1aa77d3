// Linear recurrences of a matrix state S [D][VD] per head, carried in per-request state slots:
//
//   time mixing (RWKV)   o_t = S^T r + (r . (u k)) v,   then S = diag(w) S + k v^T
//   state space (SSD)    S = a S + k (dt v)^T,           then o_t = S^T r + d v
//
// with a decay per key channel (w [D]) or one per head (a).  Both are one scan kernel; around
// it stand the input kernels of the two mixers.
//
//   time_mix     five mixes of a token's row with the row before it, x + (x' - x) mu_s; the row
//                before an entry's first token comes from the slot, the entry's last row goes
//                there (by the block that has read the slot).
//   mix_prepare  decay = exp(-exp(z + w0)) per head and channel, z a product's float output or,
//                for few tokens, made here as W_w2 tanh(low) (a block per token and head, eight
//                lanes along a row of W_w2); and the current token's weight r . (u k) per head.
//   ssd_prepare  causal convolution (bias) and SiLU of the x | B | C channels, dt = softplus(dt +
//                bias), a = exp(-exp(A_log) dt).
//   scan         below.
//
// Everything here is float whatever the activation type; a token's arithmetic does not depend
// on the rest of the batch.
#include "common.cuh"
#include "mma_util.cuh"

// ------------------------------------------------------------------ time_mix
#define TM_MIXES 5

template <int V, typename T> __device__ __forceinline__ void lr_load(const T* p, float (&v)[V]) {
    if constexpr (V == 8) load8(p, v);
    else v[0] = to_float(p[0]);
}
template <int V, typename T> __device__ __forceinline__ void lr_store(T* p, const float (&v)[V]) {
    if constexpr (V == 8) store8(p, v);
    else p[0] = from_float<T>(v[0]);
}

template <typename A, int V>
__global__ void time_mix_kernel(const A* x, int ldx, const float* __restrict__ mu, A* __restrict__ out,
                                const int* __restrict__ token_req, const int* __restrict__ qo_indptr,
                                const int* __restrict__ slots, float* state, long long state_stride,
                                int tokens, int width) {
    const int t = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    const unsigned long long waited = pdl_wait();
    x = pdl_after(x, waited);
    state = pdl_after(state, waited);
    if (c >= width) return;
    const int e = token_req[t], first = qo_indptr[e];
    float cur[V], before[V];
    lr_load<V>(x + (size_t)t * ldx + c, cur);
    if (t == first) {
        float* slot = state + (size_t)slots[e] * state_stride + c;
#pragma unroll
        for (int i = 0; i < V; ++i) before[i] = slot[i];
        float last[V];
        lr_load<V>(x + (size_t)(qo_indptr[e + 1] - 1) * ldx + c, last);
#pragma unroll
        for (int i = 0; i < V; ++i) slot[i] = last[i];
    } else {
        lr_load<V>(x + (size_t)(t - 1) * ldx + c, before);
    }
#pragma unroll
    for (int s = 0; s < TM_MIXES; ++s) {
        float m[V], y[V];
        lr_load<V>(mu + (size_t)s * width + c, m);
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = fmaf(before[i] - cur[i], m[i], cur[i]);
        lr_store<V>(out + ((size_t)s * tokens + t) * width + c, y);
    }
}

// x: [tokens] rows of ldx elements; mu: float [5][width]; out: [5][tokens][width]; the slot's row is
// `width` floats at state + slot * state_stride.
MSTAR_API int mstar_time_mix(const void* x, int ldx, const float* mu, void* out, const int* token_req,
                             const int* qo_indptr, const int* slots, float* state,
                             long long state_stride, int act_dtype, int tokens, int width,
                             void* stream) {
    if (tokens <= 0) return 0;
    if (width <= 0) return -1;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = width % 8 == 0 && ldx % 8 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)out % 16 == 0 &&
                     (uintptr_t)mu % 16 == 0;
    const int lanes = vec ? width / 8 : width;
    const int threads = lanes >= 128 ? 128 : ((lanes + 31) / 32) * 32;
    const dim3 grid(tokens, (lanes + threads - 1) / threads);
#define GO(A, V)                                                                                  \
    mstar_launch((time_mix_kernel<A, V>), grid, dim3(threads), 0, s, (const A*)x, ldx, mu, (A*)out, \
                 token_req, qo_indptr, slots, state, state_stride, tokens, width)
    if (act_dtype == MSTAR_F32) { if (vec) GO(float, 8); else GO(float, 1); }
    else { if (vec) GO(bf16, 8); else GO(bf16, 1); }
#undef GO
    return launch_status();
}

// ------------------------------------------------------------------ tanh of a float product
template <typename A>
__global__ void tanh_rows_kernel(const float* x, int ldx, A* __restrict__ out, int cols, size_t total) {
    x = pdl_after(x, pdl_wait());
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total;
         i += (size_t)gridDim.x * blockDim.x)
        out[i] = from_float<A>(tanhf(x[i / cols * ldx + i % cols]));
}

MSTAR_API int mstar_tanh_rows(const float* x, int ldx, void* out, int act_dtype, int rows, int cols,
                              void* stream) {
    const size_t total = (size_t)rows * cols;
    if (total == 0) return 0;
    size_t blocks = (total + 255) / 256;
    const size_t most = (size_t)device_sm_count() * 8;
    if (blocks > most) blocks = most;
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == MSTAR_F32)
        mstar_launch((tanh_rows_kernel<float>), dim3((int)blocks), dim3(256), 0, s, x, ldx, (float*)out, cols, total);
    else
        mstar_launch((tanh_rows_kernel<bf16>), dim3((int)blocks), dim3(256), 0, s, x, ldx, (bf16*)out, cols, total);
    return launch_status();
}

// ------------------------------------------------------------------ mix_prepare
struct MixPrepArgs {
    const float* rows;          // [tokens] of ld floats: r at 0, k at H*D
    int ld;
    const float* z;             // [tokens][H*D] of ldz, or null
    int ldz;
    const float* low;           // [tokens] of ld_low floats (before the tanh), with w2 [H*D][rank]
    int ld_low, rank;
    const void* w2;
    const float* w0;            // [H*D]
    const float* u;             // [H*D]
    float* decay;               // [tokens][H*D]
    float* direct;              // [tokens][H]
    int H, D;
};

// Many tokens: a warp per (token, head).
__global__ void __launch_bounds__(128) mix_prepare_kernel(MixPrepArgs a, int pairs) {
    const int lane = threadIdx.x & 31;
    const unsigned long long waited = pdl_wait();
    const int pair = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (pair >= pairs) return;
    const int t = pair / a.H, h = pair - t * a.H, hd = a.H * a.D;
    const float* row = pdl_after(a.rows, waited) + (size_t)t * a.ld;
    const float* z = pdl_after(a.z, waited) + (size_t)t * a.ldz;
    float sum = 0.f;
    for (int d = lane; d < a.D; d += 32) {
        const int i = h * a.D + d;
        a.decay[(size_t)t * hd + i] = expf(-expf(z[i] + a.w0[i]));
        sum = fmaf(row[i] * a.u[i], row[hd + i], sum);
    }
    sum = warp_sum(sum);
    if (lane == 0) a.direct[(size_t)t * a.H + h] = sum;
}

// Few tokens: a block per (token, head); eight lanes take a row of W_w2, so that a warp reads
// four whole rows at a time.
template <typename W>
__global__ void __launch_bounds__(128) mix_prepare_few_kernel(MixPrepArgs a) {
    extern __shared__ float sm[];             // tanh of the token's low row [rank]
    const int t = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int sub = lane & 7, hd = a.H * a.D;
    const unsigned long long waited = pdl_wait();
    const float* low = pdl_after(a.low, waited) + (size_t)t * a.ld_low;
    for (int i = threadIdx.x; i < a.rank; i += blockDim.x) sm[i] = tanhf(low[i]);
    __syncthreads();
    const float* row = pdl_after(a.rows, waited) + (size_t)t * a.ld + h * a.D;
    const bool vec = a.rank % 8 == 0 && ((uintptr_t)a.w2 & 15) == 0;
    const W* w2 = (const W*)a.w2 + (size_t)h * a.D * a.rank;
#pragma unroll 4
    for (int d0 = warp * 4; d0 < a.D; d0 += (blockDim.x >> 5) * 4) {
        const int d = d0 + (lane >> 3);
        float z = 0.f;
        if (d < a.D) {
            const W* w = w2 + (size_t)d * a.rank;
            if (vec) {
                for (int c = sub * 8; c < a.rank; c += 64) {
                    float w8[8];
                    load8(w + c, w8);
#pragma unroll
                    for (int q = 0; q < 8; ++q) z = fmaf(w8[q], sm[c + q], z);
                }
            } else {
                for (int c = sub; c < a.rank; c += 8) z = fmaf(to_float(w[c]), sm[c], z);
            }
        }
        z += __shfl_xor_sync(0xffffffffu, z, 1);
        z += __shfl_xor_sync(0xffffffffu, z, 2);
        z += __shfl_xor_sync(0xffffffffu, z, 4);
        if (sub == 0 && d < a.D)
            a.decay[(size_t)t * hd + h * a.D + d] = expf(-expf(z + a.w0[h * a.D + d]));
    }
    if (warp == 0) {
        float sum = 0.f;
        for (int d = lane; d < a.D; d += 32) sum = fmaf(row[d] * a.u[h * a.D + d], row[hd + d], sum);
        sum = warp_sum(sum);
        if (lane == 0) a.direct[(size_t)t * a.H + h] = sum;
    }
}

MSTAR_API int mstar_mix_prepare(const float* rows, int ld, const float* z, int ldz, const float* low,
                                int ld_low, int rank, const void* w2, int w2_dtype, const float* w0,
                                const float* u, float* decay, float* direct, int tokens, int H, int D,
                                void* stream) {
    if (tokens <= 0) return 0;
    if (H <= 0 || D <= 0 || ld < 2 * H * D) return -1;
    if (z == nullptr && (low == nullptr || w2 == nullptr || rank <= 0 || rank > 8192)) return -1;
    MixPrepArgs a{rows, ld, z, ldz, low, ld_low, rank, w2, w0, u, decay, direct, H, D};
    cudaStream_t s = (cudaStream_t)stream;
    if (z != nullptr) {
        const int pairs = tokens * H;
        mstar_launch(mix_prepare_kernel, dim3((pairs + 3) / 4), dim3(128), 0, s, a, pairs);
        return launch_status();
    }
    if (H > 65535) return -1;
    const size_t smem = sizeof(float) * rank;
    if (w2_dtype == MSTAR_F32)
        mstar_launch((mix_prepare_few_kernel<float>), dim3(tokens, H), dim3(128), smem, s, a);
    else
        mstar_launch((mix_prepare_few_kernel<bf16>), dim3(tokens, H), dim3(128), smem, s, a);
    return launch_status();
}

// ------------------------------------------------------------------ ssd_prepare
struct SsdPrepArgs {
    const float* proj;          // [tokens] rows of ld floats: [z: inner | x | B | C | dt: H]
    int ld, inner, channels, taps, H;
    const float* conv_wt;       // [taps][channels]
    const float* conv_b;        // [channels]
    const float* dt_bias;       // [H]
    const float* a_exp;         // [H]: exp(A_log)
    const int* token_req;
    const int* qo_indptr;
    const int* slots;
    const float* state;         // slot: the convolution's last inputs [taps - 1][channels] come first
    long long state_stride;
    float* xbc;                 // [tokens][channels]
    float* dt;                  // [tokens][H]
    float* decay;               // [tokens][H]
};

template <int V> struct LrVec;
template <> struct LrVec<1> { typedef float T; };
template <> struct LrVec<4> { typedef float4 T; };
template <int V> __device__ __forceinline__ void lr_fetch(const float* p, float (&v)[V]) {
    const typename LrVec<V>::T x = *reinterpret_cast<const typename LrVec<V>::T*>(p);
    const float* f = reinterpret_cast<const float*>(&x);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = f[i];
}

template <int V>
__global__ void ssd_prepare_kernel(SsdPrepArgs a) {
    const int t = blockIdx.x;
    const unsigned long long waited = pdl_wait();
    const float* proj = pdl_after(a.proj, waited);
    const float* state = pdl_after(a.state, waited);
    if (blockIdx.y == gridDim.y - 1) {         // the last block row: step sizes and decays
        for (int h = threadIdx.x; h < a.H; h += blockDim.x) {
            const float q = proj[(size_t)t * a.ld + a.inner + a.channels + h] + a.dt_bias[h];
            const float d = fmaxf(q, 0.f) + log1pf(expf(-fabsf(q)));
            a.dt[(size_t)t * a.H + h] = d;
            a.decay[(size_t)t * a.H + h] = expf(-a.a_exp[h] * d);
        }
        return;
    }
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    if (c >= a.channels) return;
    const int e = a.token_req[t], local = t - a.qo_indptr[e], keep = a.taps - 1;
    const float* row = proj + (size_t)t * a.ld + a.inner + c;
    const float* slot = keep > 0 ? state + (size_t)a.slots[e] * a.state_stride + c : nullptr;
    float acc[V];
    lr_fetch<V>(a.conv_b + c, acc);
    for (int j = 0; j < a.taps; ++j) {
        const int back = keep - j;
        float x[V], w[V];
        if (back <= local) lr_fetch<V>(row - (ptrdiff_t)back * a.ld, x);
        else lr_fetch<V>(slot + (size_t)(keep + local - back) * a.channels, x);
        lr_fetch<V>(a.conv_wt + (size_t)j * a.channels + c, w);
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(w[i], x[i], acc[i]);
    }
    typename LrVec<V>::T y;
#pragma unroll
    for (int i = 0; i < V; ++i) reinterpret_cast<float*>(&y)[i] = acc[i] / (1.f + expf(-acc[i]));
    *reinterpret_cast<typename LrVec<V>::T*>(a.xbc + (size_t)t * a.channels + c) = y;
}

MSTAR_API int mstar_ssd_prepare(const float* proj, int ld, int inner, int channels, int taps, int H,
                                const float* conv_wt, const float* conv_b, const float* dt_bias,
                                const float* a_exp, const int* token_req, const int* qo_indptr,
                                const int* slots, const float* state, long long state_stride,
                                float* xbc, float* dt, float* decay, int tokens, void* stream) {
    if (tokens <= 0) return 0;
    if (inner <= 0 || channels <= 0 || taps < 1 || H <= 0 || ld < inner + channels + H) return -1;
    if (taps > 1 && (slots == nullptr || state == nullptr)) return -1;
    SsdPrepArgs a{proj, ld, inner, channels, taps, H, conv_wt, conv_b, dt_bias, a_exp, token_req, qo_indptr,
                  slots, state, state_stride, xbc, dt, decay};
    const bool vec = ld % 4 == 0 && inner % 4 == 0 && channels % 4 == 0 && state_stride % 4 == 0 &&
                     (uintptr_t)proj % 16 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)conv_wt % 16 == 0 &&
                     (uintptr_t)conv_b % 16 == 0 && (uintptr_t)xbc % 16 == 0;
    const int lanes = vec ? channels / 4 : channels;
    const int threads = lanes >= 128 ? 128 : ((lanes + 31) / 32) * 32;
    const dim3 grid(tokens, (lanes + threads - 1) / threads + 1);
    cudaStream_t s = (cudaStream_t)stream;
    if (vec) mstar_launch((ssd_prepare_kernel<4>), grid, dim3(threads), 0, s, a);
    else mstar_launch((ssd_prepare_kernel<1>), grid, dim3(threads), 0, s, a);
    return launch_status();
}

// ------------------------------------------------------------------ scan
// A block owns columns of one head of one entry; a thread CT = 4 neighbouring columns, whose D
// rows lie on the L lanes of the columns' group: lane l keeps rows 4 l .. 4 l + 3 of every 4 L
// rows, R of them.  What the block's columns share of a token (its r, k and decay rows) and
// their values are staged in shared memory, `chunk` tokens at a time, the next chunk on its way
// (cp.async) while this one is walked; a row read from shared memory serves four columns.  The
// rows are taken in pairs (two floats an instruction), so a token costs a thread 3 R CT / 2
// multiply-adds; the only chain from token to token is one of them per row, and the read-out's
// sums over the lanes hang off it.
//
// Long entries are cut into pieces that run side by side (the recurrence is linear in S): pass 1
// walks every piece but the last from a zero state and leaves its end state and the product of
// its decays in scratch, scan_join turns those into the state before each piece, pass 2 walks
// every piece from there and makes the outputs.
#define LR_CT 4
#define LR_CHUNK 16

struct ScanArgs {
    const float* r;             // + token * ld_r + (h / rk_share) * D
    const float* k;
    const float* v;             // + token * ld_v + h * VD
    int ld_r, ld_k, ld_v, rk_share;
    const float* decay;         // [tokens][H*D], or [tokens][H]
    const float* direct;        // weight of the token's own values: [tokens][H], or [H] (one decay a head)
    const float* dt;            // [tokens][H] or null: multiplies the values that enter the state
    const int* qo_indptr;
    const int* slots;
    float* state;               // the slot's S^T [H][VD][D] at state_offset
    long long state_stride, state_offset;
    float* out;                 // [tokens][H*VD]
    int H, D, VD, chunk, zblocks;
    int piece, max_pieces;      // piece 0: entries are not cut
    float* piece_state;         // [entries][max_pieces][H][VD][D]
    float* piece_decay;         // [entries][max_pieces][H][D] or [entries][max_pieces][H]
    // with taps > 1: the slot's convolution rows [taps - 1][channels] at its start move on by
    // the entry's raw rows (+ token * raw_ld)
    const float* raw;
    int raw_ld, channels, taps;
};

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
    f32x2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ void lr_copy4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(
                     (uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void lr_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(
                     (uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// rows of a token in shared memory: r, k, (decays,) values, then decay (one a head), direct, dt
__host__ __device__ constexpr int lr_token_floats(bool vecdecay, int dp, int cols) {
    return (vecdecay ? 3 : 2) * dp + cols + 4;
}

// PASS 0: whole entries, 1: pieces without outputs, 2: pieces with outputs.
// VECDECAY: a decay per key channel and the read before the update, else one a head and the read
// after it.  VEC: rows are whole 16-byte pieces.
template <bool VECDECAY, int PASS, int L, int R, bool VEC>
__global__ void __launch_bounds__(128) linear_scan_kernel(ScanArgs a) {
    extern __shared__ __align__(16) float stage[];
    constexpr int DP = L * R, RV = R / 4;
    constexpr bool OUT = PASS != 1;
    const int threads = blockDim.x, cols = threads / L * LR_CT;
    const int per_tok = lr_token_floats(VECDECAY, DP, cols);
    float* prod = stage + 2 * a.chunk * per_tok;          // [D] or [1]: product of the decays (pass 1)
    const int e = blockIdx.x, h = blockIdx.y;
    const int zb = blockIdx.z % a.zblocks, piece = blockIdx.z / a.zblocks;
    const int tid = threadIdx.x, lane = tid % L, group = tid / L;
    const int D = a.D, VD = a.VD;
    const int col0 = zb * cols, mycol = col0 + group * LR_CT;
    const unsigned long long waited = pdl_wait();
    const int e_start = a.qo_indptr[e], e_n = a.qo_indptr[e + 1] - e_start;
    if (e_n <= 0) return;
    const int pieces = PASS == 0 ? 1 : (e_n + a.piece - 1) / a.piece;
    if (piece >= pieces || (PASS == 1 && piece == pieces - 1)) return;
    const int start = e_start + (PASS == 0 ? 0 : piece * a.piece);
    const int n = PASS == 0 ? e_n : min(a.piece, e_n - piece * a.piece);
    const int rk = h / a.rk_share;
    const float* r = pdl_after(a.r, waited) + (size_t)rk * D;
    const float* k = pdl_after(a.k, waited) + (size_t)rk * D;
    const float* v = pdl_after(a.v, waited) + (size_t)h * VD;
    const float* decay = pdl_after(a.decay, waited);
    const float* direct = pdl_after(a.direct, waited);
    const float* dt = pdl_after(a.dt, waited);
    float* slot = pdl_after(a.state, waited) + (size_t)a.slots[e] * a.state_stride;
    const size_t hcols = (size_t)h * VD;                  // first column of the head
    float* scratch = PASS == 0 ? nullptr
        : pdl_after(a.piece_state, waited) + (((size_t)e * a.max_pieces + piece) * a.H * VD + hcols) * D;

    const int ncols = min(cols, VD - col0);
    auto fetch = [&](int buf, int base) {
        const int here = min(a.chunk, n - base);
        float* dst0 = stage + (size_t)buf * a.chunk * per_tok;
        // a thread takes a piece of a token's rows (k, then decays, then r, then the values) and
        // copies it for every token of the chunk: its addresses move on by fixed steps
        const int unit = VEC ? 4 : 1, per_row = D / unit;
        const int all_rows = ((VECDECAY ? 2 : 1) + (OUT ? 1 : 0)) * per_row;
        const int pieces_tok = all_rows + ncols / unit;
        const size_t tok = (size_t)(start + base);
        for (int p = tid; p < pieces_tok; p += threads) {
            const float* src;
            float* dst = dst0;
            size_t step;
            if (p >= all_rows) {
                const int c = (p - all_rows) * unit;
                src = v + tok * a.ld_v + col0 + c;
                step = a.ld_v;
                dst += (VECDECAY ? 3 : 2) * DP + c;
            } else {
                const int which = p / per_row, d = (p - which * per_row) * unit;
                if (which == 0) {
                    src = k + tok * a.ld_k + d;
                    step = a.ld_k;
                    dst += DP + d;
                } else if (VECDECAY && which == 1) {
                    step = (size_t)a.H * D;
                    src = decay + tok * step + (size_t)h * D + d;
                    dst += 2 * DP + d;
                } else {
                    src = r + tok * a.ld_r + d;
                    step = a.ld_r;
                    dst += d;
                }
            }
#pragma unroll 4
            for (int j = 0; j < here; ++j, src += step, dst += per_tok) {
                if constexpr (VEC) lr_copy16(dst, src); else lr_copy4(dst, src);
            }
        }
        float* vdst = dst0 + (VECDECAY ? 3 : 2) * DP;
        for (int t = tid; t < here; t += threads) {
            const size_t at = (size_t)(start + base + t) * a.H + h;
            float* sc = vdst + (size_t)t * per_tok + cols;
            if (!VECDECAY) lr_copy4(sc, decay + at);
            if (VECDECAY && OUT) lr_copy4(sc + 1, direct + at);
            if (a.dt != nullptr) lr_copy4(sc + 2, dt + at);
        }
    };

    // rows past D and columns past the head's read as zeros whatever the chunk
    if (DP > D || ncols < cols)
        for (int i = tid; i < 2 * a.chunk * per_tok; i += threads) stage[i] = 0.f;
    if (PASS == 1)
        for (int i = tid; i < (VECDECAY ? D : 1); i += threads) prod[i] = 1.f;
    __syncthreads();
    fetch(0, 0);
    cp_async_commit();

    f32x2 S[LR_CT][R / 2];
    bool live[LR_CT];
#pragma unroll
    for (int c = 0; c < LR_CT; ++c) {
        live[c] = mycol + c < VD;
        const float* src = PASS == 0 ? slot + a.state_offset + (hcols + mycol + c) * D
                                     : scratch + (size_t)(mycol + c) * D;
#pragma unroll
        for (int i = 0; i < RV; ++i) {
            const int row = 4 * lane + 4 * L * i;
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (PASS != 1 && live[c]) {
                if (VEC) {
                    if (row < D) x = *reinterpret_cast<const float4*>(src + row);
                } else {
                    if (row < D) x.x = src[row];
                    if (row + 1 < D) x.y = src[row + 1];
                    if (row + 2 < D) x.z = src[row + 2];
                    if (row + 3 < D) x.w = src[row + 3];
                }
            }
            S[c][2 * i] = pack2(x.x, x.y);
            S[c][2 * i + 1] = pack2(x.z, x.w);
        }
    }
    const float skip = VECDECAY ? 0.f : direct[h];
    // after the exchange below, the lane's own column of the four
    const int keep = (lane & 1) * 2 + ((lane >> 1) & 1);
    int buf = 0;
    for (int base = 0; base < n; base += a.chunk, buf ^= 1) {
        if (base + a.chunk < n) fetch(buf ^ 1, base + a.chunk);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const int here = min(a.chunk, n - base);
        const float* tok = stage + (size_t)buf * a.chunk * per_tok;
        if (PASS == 1 && zb == 0) {
            if (VECDECAY) {
                for (int d = tid; d < D; d += threads) {
                    float p = prod[d];
                    for (int j = 0; j < here; ++j) p *= tok[(size_t)j * per_tok + 2 * DP + d];
                    prod[d] = p;
                }
            } else if (tid == 0) {
                float p = prod[0];
                for (int j = 0; j < here; ++j) p *= tok[(size_t)j * per_tok + 2 * DP + cols];
                prod[0] = p;
            }
        }
#pragma unroll 2
        for (int j = 0; j < here; ++j, tok += per_tok) {
            const float* vs = tok + (VECDECAY ? 3 : 2) * DP;
            const float4 v4 = *reinterpret_cast<const float4*>(vs + group * LR_CT);
            const float4 sc = *reinterpret_cast<const float4*>(vs + cols);    // decay, direct, dt
            const float in = a.dt != nullptr ? sc.z : 1.f;
            const f32x2 vv[LR_CT] = {pack2(v4.x * in, v4.x * in), pack2(v4.y * in, v4.y * in),
                                     pack2(v4.z * in, v4.z * in), pack2(v4.w * in, v4.w * in)};
            const f32x2 one = pack2(sc.x, sc.x);
            f32x2 acc[LR_CT];
#pragma unroll
            for (int c = 0; c < LR_CT; ++c) acc[c] = 0ull;
#pragma unroll
            for (int i = 0; i < RV; ++i) {
                const int row = 4 * lane + 4 * L * i;
                const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(tok + DP + row);
                ulonglong2 rr = make_ulonglong2(0ull, 0ull), ww = make_ulonglong2(one, one);
                if (OUT) rr = *reinterpret_cast<const ulonglong2*>(tok + row);
                if (VECDECAY) ww = *reinterpret_cast<const ulonglong2*>(tok + 2 * DP + row);
#pragma unroll
                for (int c = 0; c < LR_CT; ++c) {
                    f32x2& s0 = S[c][2 * i];
                    f32x2& s1 = S[c][2 * i + 1];
                    if (VECDECAY && OUT) {
                        acc[c] = fma2(rr.x, s0, acc[c]);
                        acc[c] = fma2(rr.y, s1, acc[c]);
                    }
                    s0 = fma2(ww.x, s0, mul2(kk.x, vv[c]));
                    s1 = fma2(ww.y, s1, mul2(kk.y, vv[c]));
                    if (!VECDECAY && OUT) {
                        acc[c] = fma2(rr.x, s0, acc[c]);
                        acc[c] = fma2(rr.y, s1, acc[c]);
                    }
                }
            }
            if (OUT) {
                float y[LR_CT];
#pragma unroll
                for (int c = 0; c < LR_CT; ++c) {
                    const float2 p = unpack2(acc[c]);
                    y[c] = p.x + p.y;
                }
                // four sums over L lanes: two lanes exchange two of them, then one, then the
                // rest of the lanes add up
                const bool odd = lane & 1, second = (lane >> 1) & 1;
                const float g0 = __shfl_xor_sync(0xffffffffu, odd ? y[0] : y[2], 1);
                const float g1 = __shfl_xor_sync(0xffffffffu, odd ? y[1] : y[3], 1);
                const float k0 = (odd ? y[2] : y[0]) + g0, k1 = (odd ? y[3] : y[1]) + g1;
                const float g2 = __shfl_xor_sync(0xffffffffu, second ? k0 : k1, 2);
                float o = (second ? k1 : k0) + g2;
#pragma unroll
                for (int w = 4; w < L; w <<= 1) o += __shfl_xor_sync(0xffffffffu, o, w);
                const int col = mycol + keep;
                if (lane < 4 && col < VD)
                    a.out[(size_t)(start + base + j) * a.H * VD + hcols + col] =
                        fmaf(VECDECAY ? sc.y : skip, vs[group * LR_CT + keep], o);
            }
        }
        __syncthreads();                       // the buffer is free for the chunk after next
    }
    cp_async_wait<0>();

    const bool last_piece = piece == pieces - 1;
    if (PASS == 1 || last_piece) {
#pragma unroll
        for (int c = 0; c < LR_CT; ++c) {
            if (!live[c]) continue;
            float* dst = PASS == 1 ? scratch + (size_t)(mycol + c) * D
                                   : slot + a.state_offset + (hcols + mycol + c) * D;
#pragma unroll
            for (int i = 0; i < RV; ++i) {
                const int row = 4 * lane + 4 * L * i;
                const float2 lo = unpack2(S[c][2 * i]), hi = unpack2(S[c][2 * i + 1]);
                if (VEC) {
                    if (row < D) *reinterpret_cast<float4*>(dst + row) = make_float4(lo.x, lo.y, hi.x, hi.y);
                } else {
                    if (row < D) dst[row] = lo.x;
                    if (row + 1 < D) dst[row + 1] = lo.y;
                    if (row + 2 < D) dst[row + 2] = hi.x;
                    if (row + 3 < D) dst[row + 3] = hi.y;
                }
            }
        }
    }
    if (PASS == 1 && zb == 0) {                // (the loop's last barrier lies behind the products)
        const int wide = VECDECAY ? D : 1;
        float* dst = pdl_after(a.piece_decay, waited) + (((size_t)e * a.max_pieces + piece) * a.H + h) * wide;
        for (int i = tid; i < wide; i += threads) dst[i] = prod[i];
    }
    if (PASS != 1 && last_piece && zb == 0 && a.taps > 1) {
        // the convolution's window moves on: this head's share of the channels, oldest row first
        // (row s is read from s + n, which is written later or not at all)
        const float* raw = pdl_after(a.raw, waited);
        const int c_end = (int)((long long)(h + 1) * a.channels / a.H), kept = a.taps - 1;
        for (int c = (int)((long long)h * a.channels / a.H) + tid; c < c_end; c += threads)
            for (int s = 0; s < kept; ++s) {
                const int src = e_n - kept + s;
                slot[(size_t)s * a.channels + c] = src >= 0 ? raw[(size_t)(e_start + src) * a.raw_ld + c]
                                                            : slot[(size_t)(s + e_n) * a.channels + c];
            }
    }
}

// The state before every piece, in place of the pieces' own end states: a thread per element.
__global__ void scan_join_kernel(ScanArgs a, int wide) {
    const int e = blockIdx.y;
    const unsigned long long waited = pdl_wait();
    const int n = a.qo_indptr[e + 1] - a.qo_indptr[e];
    const int pieces = (n + a.piece - 1) / a.piece;
    const long long size = (long long)a.H * a.VD * a.D;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= size || pieces <= 0) return;
    const int h = (int)(i / ((long long)a.VD * a.D)), d = (int)(i % a.D);
    float S = pdl_after(a.state, waited)[(size_t)a.slots[e] * a.state_stride + a.state_offset + i];
    float* at = pdl_after(a.piece_state, waited) + (size_t)e * a.max_pieces * size + i;
    const float* dec = pdl_after(a.piece_decay, waited) +
                       ((size_t)e * a.max_pieces * a.H + h) * wide + (wide > 1 ? d : 0);
    const size_t step = (size_t)a.H * wide;
    int p = 0;
    for (; p + 4 < pieces; p += 4) {           // four pieces' loads in flight
        float E[4], w[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            E[q] = at[(size_t)(p + q) * size];
            w[q] = dec[(size_t)(p + q) * step];
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            at[(size_t)(p + q) * size] = S;
            S = fmaf(w[q], S, E[q]);
        }
    }
    for (; p < pieces - 1; ++p) {
        const float E = at[(size_t)p * size];
        at[(size_t)p * size] = S;
        S = fmaf(dec[(size_t)p * step], S, E);
    }
    at[(size_t)(pieces - 1) * size] = S;
}

template <bool VECDECAY, int PASS, int L, int R, bool VEC>
static int launch_scan(ScanArgs a, int entries, int threads, cudaStream_t s) {
    const int cols = threads / L * LR_CT;
    const int per_tok = lr_token_floats(VECDECAY, L * R, cols);
    while (a.chunk > 1 && (size_t)2 * a.chunk * per_tok * sizeof(float) > 96 * 1024) a.chunk /= 2;
    const size_t smem = ((size_t)2 * a.chunk * per_tok + a.D) * sizeof(float);
    static size_t configured = 0;
    if (smem > 48 * 1024 && smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(linear_scan_kernel<VECDECAY, PASS, L, R, VEC>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = smem;
    }
    mstar_launch((linear_scan_kernel<VECDECAY, PASS, L, R, VEC>),
                 dim3(entries, a.H, a.zblocks * (PASS == 0 ? 1 : a.max_pieces)), dim3(threads), smem, s, a);
    return launch_status();
}

template <bool VECDECAY, int L, int R, bool VEC>
static int scan_passes(ScanArgs& a, int entries, cudaStream_t s) {
    // threads: enough for the head's columns, at most 128; whole warps
    int threads = (a.VD + LR_CT - 1) / LR_CT * L;
    threads = threads >= 128 ? 128 : (threads + 31) / 32 * 32;
    const int cols = threads / L * LR_CT;
    a.zblocks = (a.VD + cols - 1) / cols;
    if ((long long)a.zblocks * a.max_pieces > 65535) return -1;
    if (a.piece == 0) return launch_scan<VECDECAY, 0, L, R, VEC>(a, entries, threads, s);
    int code = launch_scan<VECDECAY, 1, L, R, VEC>(a, entries, threads, s);
    if (code != 0) return code;
    const long long size = (long long)a.H * a.VD * a.D;
    mstar_launch(scan_join_kernel, dim3((unsigned)((size + 255) / 256), entries), dim3(256), 0, s, a,
                 VECDECAY ? a.D : 1);
    code = launch_status();
    if (code != 0) return code;
    return launch_scan<VECDECAY, 2, L, R, VEC>(a, entries, threads, s);
}

// r, k, v: float rows (strides in floats); decay: [tokens][H*D] with `vector_decay`, else
// [tokens][H]; direct: [tokens][H] / [H]; dt: [tokens][H] or null.  piece > 0: entries are cut into
// pieces of that many tokens; piece_state is float scratch [entries, max_pieces, H, VD, D],
// piece_decay [entries, max_pieces, H, D or 1].  Returns 0, a CUDA error code, or -1 when the
// shape is refused (D above 512).
MSTAR_API int mstar_linear_scan(const float* r, const float* k, const float* v, int ld_r, int ld_k,
                                int ld_v, int rk_share, const float* decay, int vector_decay,
                                const float* direct, const float* dt, const int* qo_indptr,
                                const int* slots, float* state, long long state_stride,
                                long long state_offset, float* out, int entries, int max_q_len, int H,
                                int D, int VD, int piece, int max_pieces, float* piece_state,
                                float* piece_decay, const float* raw, int raw_ld, int channels, int taps,
                                void* stream) {
    if (entries <= 0) return 0;
    if (H <= 0 || H > 65535 || D <= 0 || D > 512 || VD <= 0 || rk_share <= 0) return -1;
    if (piece < 0 || (piece > 0 && (max_pieces < 1 || !piece_state || !piece_decay || entries > 65535))) return -1;
    if (taps > 1 && (raw == nullptr || channels <= 0)) return -1;
    int chunk = LR_CHUNK;
    while (chunk > 1 && chunk / 2 >= max_q_len) chunk /= 2;
    ScanArgs a{r, k, v, ld_r, ld_k, ld_v, rk_share, decay, direct, dt, qo_indptr, slots, state, state_stride,
               state_offset, out, H, D, VD, chunk, 1, piece, piece > 0 ? max_pieces : 1, piece_state,
               piece_decay, raw, raw_ld, channels, taps};
    auto aligned = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
    const bool vec = D % 4 == 0 && VD % 4 == 0 && ld_r % 4 == 0 && ld_k % 4 == 0 && ld_v % 4 == 0 &&
                     state_stride % 4 == 0 && state_offset % 4 == 0 && aligned(r) && aligned(k) && aligned(v) &&
                     aligned(state) && aligned(piece_state) && (!vector_decay || aligned(decay));
    cudaStream_t s = (cudaStream_t)stream;
#define GO(L, R)                                                                                  \
    do {                                                                                          \
        if (vector_decay)                                                                         \
            return vec ? scan_passes<true, L, R, true>(a, entries, s)                             \
                       : scan_passes<true, L, R, false>(a, entries, s);                           \
        return vec ? scan_passes<false, L, R, true>(a, entries, s)                                \
                   : scan_passes<false, L, R, false>(a, entries, s);                              \
    } while (0)
    if (D <= 32) GO(4, 8);
    if (D <= 64) GO(4, 16);
    if (D <= 128) GO(8, 16);
    if (D <= 256) GO(16, 16);
    GO(32, 16);
#undef GO
}
