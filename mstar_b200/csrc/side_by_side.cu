// What lies between two layers whose sublayers stand side by side on one norm,
//   x_new = x + (mixer output + feed-forward output),   n = rms(x_new) * w,
//   shifted = n + (n' - n) * shift,  n' the previous token's n,
// as one kernel: the sum, the norm and the token shift.
//
// The mixer's output is a row y0, or the mean of two branches, (rms(y0) w0 + rms(y1) w1) / 2;
// the feed-forward's output f joins it.  Optional results: the new residual (float, written to
// another buffer than the one read), n and the shifted n in the activation type, the residual
// itself in the activation type, or (with `rows`) the residual of some rows only.
//
// A block takes a run of consecutive tokens and keeps n of the token before in registers; for
// the run's first token it makes the row before it once more (the residual is read from one
// buffer and written to another, so the neighbours' rows may be read at any time), or, where
// the token is the first of its entry, takes it from the request's state slot.  The block that
// has read an entry's slot is the one that writes its last n there (making that row once more
// if it lies outside its run), so no two blocks touch a slot.
//
// All arithmetic is float; a row's sums do not depend on what else is in the batch.
#include "common.cuh"

struct SideArgs {
    const float* resid;         // [tokens][width]
    const void* y0;             // [tokens][width] or null; float or activation type
    const void* y1;             // second branch (activation type), or null
    const void* f;              // feed-forward output (activation type), or null
    const float* w0;            // branch weights (with y1)
    const float* w1;
    float branch_eps;
    float* resid_out;           // [tokens][width] / [rows][width], or null
    void* raw_out;              // [tokens][width] activation type, or null
    const void* norm_w;         // or null: no norm
    float eps;
    void* normed;               // [tokens][width] activation type, or null
    void* shifted;              // likewise; needs shift and the slot arguments
    const void* shift;
    float* prev;                // state slots: row of slot s at prev + s * prev_stride
    long long prev_stride;
    const int* token_req;
    const int* qo_indptr;
    const int* slots;
    const int* rows;            // or null
    int width, tokens, per_block;
};

// Two sums over the block at once.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    __syncthreads();
    if (lane == 0) scratch[warp] = make_float2(a, b);
    __syncthreads();
    const float2 r = lane < nwarps ? scratch[lane] : make_float2(0.f, 0.f);
    return make_float2(warp_sum(r.x), warp_sum(r.y));
}

template <int V, typename T> __device__ __forceinline__ void sb_load(const T* p, float (&v)[V]) {
    if constexpr (V == 8) load8(p, v);
    else v[0] = to_float(p[0]);
}
template <int V, typename T> __device__ __forceinline__ void sb_put(T* p, const float (&v)[V]) {
    if constexpr (V == 8) store8(p, v);
    else p[0] = from_float<T>(v[0]);
}

// V elements an access, NC accesses a thread.  A: activation type, Y: type of y0, W: of the
// norm and shift weights.
#define SD_THREADS 512
template <typename A, typename Y, typename W, int V, int NC>
__global__ void __launch_bounds__(SD_THREADS) side_step_kernel(SideArgs a) {
    __shared__ float scratch[32];
    __shared__ float2 scratch2[32];
    const int chunks = a.width / V;
    int at[NC];
    bool has[NC];
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        at[c] = (threadIdx.x + c * blockDim.x) * V;
        has[c] = threadIdx.x + c * blockDim.x < chunks;
    }
    // with one access a thread the parameters are asked for while the kernel before is still
    // draining, and kept; wider rows read them where they are used
    constexpr bool HOLD = NC == 1;
    float nw[V], sw[V], w0[V], w1[V];
    auto branch_weights = [&](int c) {
        sb_load<V>(a.w0 + at[c], w0);
        sb_load<V>(a.w1 + at[c], w1);
    };
    auto norm_weight = [&](int c) { sb_load<V>((const W*)a.norm_w + at[c], nw); };
    auto shift_weight = [&](int c) { sb_load<V>((const W*)a.shift + at[c], sw); };
    if (HOLD && has[0]) {
        if (a.norm_w != nullptr) norm_weight(0);
        if (a.shifted != nullptr) shift_weight(0);
        if (a.y1 != nullptr) branch_weights(0);
    }
    const unsigned long long waited = pdl_wait();
    const float* resid = pdl_after(a.resid, waited);
    const Y* y0 = pdl_after((const Y*)a.y0, waited);
    const A* y1 = pdl_after((const A*)a.y1, waited);
    const A* f = pdl_after((const A*)a.f, waited);
    float* prev = pdl_after(a.prev, waited);
    float v[NC][V], hp[NC][V];

    // the new residual of a token in v
    auto residual = [&](int tok) {
        const size_t base = (size_t)tok * a.width;
        if (y1 != nullptr) {
            float b0[NC][V], b1[NC][V], s0 = 0.f, s1 = 0.f;
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (has[c]) {
                    sb_load<V>(y0 + base + at[c], b0[c]);
                    sb_load<V>(y1 + base + at[c], b1[c]);
                    sb_load<V>(resid + base + at[c], v[c]);
#pragma unroll
                    for (int i = 0; i < V; ++i) {
                        s0 = fmaf(b0[c][i], b0[c][i], s0);
                        s1 = fmaf(b1[c][i], b1[c][i], s1);
                    }
                }
            const float2 ss = block_sum2(s0, s1, scratch2);
            const float i0 = 0.5f * rsqrtf(ss.x / (float)a.width + a.branch_eps);
            const float i1 = 0.5f * rsqrtf(ss.y / (float)a.width + a.branch_eps);
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (has[c]) {
                    if (!HOLD) branch_weights(c);
#pragma unroll
                    for (int i = 0; i < V; ++i)
                        v[c][i] += b0[c][i] * i0 * w0[i] + b1[c][i] * i1 * w1[i];
                }
        } else {
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (has[c]) {
                    sb_load<V>(resid + base + at[c], v[c]);
                    if (y0 != nullptr) {
                        float d[V];
                        sb_load<V>(y0 + base + at[c], d);
#pragma unroll
                        for (int i = 0; i < V; ++i) v[c][i] += d[i];
                    }
                }
        }
        if (f != nullptr) {
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (has[c]) {
                    float d[V];
                    sb_load<V>(f + base + at[c], d);
#pragma unroll
                    for (int i = 0; i < V; ++i) v[c][i] += d[i];
                }
        }
    };
    // v -> its norm, in place
    auto norm = [&]() {
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (has[c])
#pragma unroll
                for (int i = 0; i < V; ++i) ss = fmaf(v[c][i], v[c][i], ss);
        const float inv = rsqrtf(block_sum(ss, scratch) / (float)a.width + a.eps);
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (has[c]) {
                if (!HOLD) norm_weight(c);
#pragma unroll
                for (int i = 0; i < V; ++i) v[c][i] *= inv * nw[i];
            }
    };

    if (a.rows != nullptr) {                   // some rows of the residual, nothing else
        const int tok = a.rows[blockIdx.x];
        residual(tok);
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (has[c]) sb_put<V>(a.resid_out + (size_t)blockIdx.x * a.width + at[c], v[c]);
        return;
    }
    const int t0 = blockIdx.x * a.per_block, t1 = min(t0 + a.per_block, a.tokens);
    const bool shifting = a.shifted != nullptr;
    int owned = -1;                            // the entry whose slot this block has read last
    for (int t = t0; t < t1; ++t) {
        int e = 0, last = -1;
        if (shifting) {
            e = a.token_req[t];
            const int first = a.qo_indptr[e];
            last = a.qo_indptr[e + 1] - 1;
            if (t == first) {
                owned = e;
                const float* p = prev + (size_t)a.slots[e] * a.prev_stride;
#pragma unroll
                for (int c = 0; c < NC; ++c)
                    if (has[c])
#pragma unroll
                        for (int i = 0; i < V; ++i) hp[c][i] = p[at[c] + i];
            } else if (t == t0) {              // the row before the run, once more
                residual(t - 1);
                norm();
#pragma unroll
                for (int c = 0; c < NC; ++c)
                    if (has[c])
#pragma unroll
                        for (int i = 0; i < V; ++i) hp[c][i] = v[c][i];
            }
        }
        const size_t base = (size_t)t * a.width;
        residual(t);
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (has[c]) {
                if (a.resid_out != nullptr) sb_put<V>(a.resid_out + base + at[c], v[c]);
                if (a.raw_out != nullptr) sb_put<V>((A*)a.raw_out + base + at[c], v[c]);
            }
        if (a.norm_w == nullptr) continue;
        norm();
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (has[c]) {
                if (a.normed != nullptr) sb_put<V>((A*)a.normed + base + at[c], v[c]);
                if (shifting) {
                    float s[V];
                    if (!HOLD) shift_weight(c);
#pragma unroll
                    for (int i = 0; i < V; ++i) s[i] = fmaf(hp[c][i] - v[c][i], sw[i], v[c][i]);
                    sb_put<V>((A*)a.shifted + base + at[c], s);
#pragma unroll
                    for (int i = 0; i < V; ++i) hp[c][i] = v[c][i];
                }
            }
        // this block has read the entry's slot, so it also leaves the entry's last n there
        if (shifting && owned == e && (t == last || t == t1 - 1)) {
            if (t != last) {
                residual(last);
                norm();
            }
            float* p = prev + (size_t)a.slots[e] * a.prev_stride;
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (has[c])
#pragma unroll
                    for (int i = 0; i < V; ++i) p[at[c] + i] = v[c][i];
        }
    }
}

// Returns 0, a CUDA error code, or -1 when the shape is refused (a width above 16,384, or
// above 8,192 where rows are no whole 16-byte pieces).
// `y_dtype`: type of y0 (the activation type, or float); two branches are of the activation type.
MSTAR_API int mstar_side_step(const float* resid, const void* y0, int y_dtype, const void* y1,
                              const void* f, const float* w0, const float* w1, float branch_eps,
                              float* resid_out, void* raw_out, const void* norm_w, const void* shift,
                              int weight_dtype, float eps, void* normed, void* shifted, float* prev,
                              long long prev_stride, const int* token_req, const int* qo_indptr,
                              const int* slots, const int* rows, int num_rows, int tokens, int width,
                              int act_dtype, void* stream) {
    const int work = rows != nullptr ? num_rows : tokens;
    if (work <= 0) return 0;
    if (width <= 0 || resid == resid_out) return -1;
    if (y1 != nullptr && (y0 == nullptr || w0 == nullptr || w1 == nullptr || y_dtype != act_dtype)) return -1;
    if (act_dtype == MSTAR_F32 && y_dtype != MSTAR_F32) return -1;
    if (shifted != nullptr && (!norm_w || !shift || !prev || !token_req || !qo_indptr || !slots)) return -1;
    if (rows != nullptr && (resid_out == nullptr || norm_w != nullptr)) return -1;
    // a run of tokens per block where tokens are many: four blocks an SM still
    int per_block = 1;
    if (rows == nullptr && shifted != nullptr) {
        per_block = tokens / (device_sm_count() * 4);
        if (per_block < 1) per_block = 1;
        if (per_block > 8) per_block = 8;
    }
    SideArgs a{resid, y0, y1, f, w0, w1, branch_eps, resid_out, raw_out, norm_w, eps, normed, shifted,
               shift, prev, prev_stride, token_req, qo_indptr, slots, rows, width, tokens, per_block};
    auto aligned = [](const void* p, size_t n) { return ((uintptr_t)p % n) == 0; };
    const bool vec = width % 8 == 0 && aligned(resid, 16) && aligned(y0, 16) && aligned(y1, 16) &&
                     aligned(f, 16) && aligned(w0, 16) && aligned(w1, 16) && aligned(resid_out, 16) &&
                     aligned(raw_out, 16) && aligned(norm_w, 16) && aligned(shift, 16) &&
                     aligned(normed, 16) && aligned(shifted, 16);
    const int chunks = vec ? width / 8 : width;
    const int most = SD_THREADS;
    int nc = vec ? 1 : 4;
    if (vec) while (nc < 4 && chunks > most * nc) nc *= 2;
    else if (chunks > most * nc) nc = 16;
    if (chunks > most * nc) return -1;
    const int threads = (((chunks + nc - 1) / nc + 31) / 32) * 32;
    const dim3 grid((work + per_block - 1) / per_block);
    cudaStream_t s = (cudaStream_t)stream;
#define GO(A, Y, W, V, NC)                                                                        \
    mstar_launch((side_step_kernel<A, Y, W, V, NC>), grid, dim3(threads), 0, s, a)
#define SIZES(A, Y, W)                                                                            \
    do {                                                                                          \
        if (vec) {                                                                                \
            if (nc == 1) GO(A, Y, W, 8, 1);                                                       \
            else if (nc == 2) GO(A, Y, W, 8, 2);                                                  \
            else GO(A, Y, W, 8, 4);                                                               \
        } else if (nc == 4) GO(A, Y, W, 1, 4);                                                    \
        else GO(A, Y, W, 1, 16);                                                                  \
    } while (0)
    if (act_dtype == MSTAR_F32) {
        if (weight_dtype == MSTAR_F32) SIZES(float, float, float); else SIZES(float, float, bf16);
    } else if (y_dtype == MSTAR_F32 && y0 != nullptr) {
        if (weight_dtype == MSTAR_F32) SIZES(bf16, float, float); else SIZES(bf16, float, bf16);
    } else {
        if (weight_dtype == MSTAR_F32) SIZES(bf16, bf16, float); else SIZES(bf16, bf16, bf16);
    }
#undef SIZES
#undef GO
    return launch_status();
}
