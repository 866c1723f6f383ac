// A residual of several streams, and what stands between two sublayers of a model that has one.  Per token the streams
// x_1 .. x_S are FP32 rows of D; a sublayer reads one combination of them and its result goes into all of them:
//
//   x_t <- sum_s mix[s, t] x_s + out[t] y      (mix[s, t]: what stream s gives to stream t)
//   u    = sum_t in[t] x_t                      with the weights of the sublayer that comes next
//   n    = T(u * rsqrt(mean(u^2) + eps) * w)    its norm, in the operand dtype
//
// in ONE pass over the row: the streams are read once and written once.  The first part is left out when there is no y (before
// the first sublayer), the last two when no norm is asked for; with all in[t] equal to one and no `dst` the kernel closes
// the model (the sum of the streams through the last norm, for picked rows).  While all streams are still equal (the
// embedding output) `src` is ONE row per token, read for every stream.
//
// y is one of
//   * a (+ bias) + sum_j pw[t, j] py[row(t, j)]: FP32 [T, D] or split-K slices of it, a projection's bias, a routed
//     feed-forward's rows with their weights, or
//   * m (norm(a + bias) wa + norm(b) wb): two results side by side, each over its root mean square over D times a stored
//     weight (`wb` given); the row's two results wait in shared memory between their sums of squares and the add.
//
// normed_pair_kernel is that second form alone, for a block that adds plain FP32 results.
#include "common.cuh"

namespace {

constexpr int HYPER_MAX_STREAMS = 32;
constexpr int HYPER_PAIRS = 64;                   // routed rows of a token whose places and weights the 16-byte kernel keeps at hand

struct HyperArgs {
    const float* src; int broadcast;              // [T, S, D], or [T, D] for all streams
    float* dst;                                   // [T, S, D] or null; may be src
    const float* a; int a_slices; size_t slice_stride; const float* bias;
    const float* py; const int* pair_row; const float* pw; int pairs;
    const float* b; int b_slices; const float* wa; const float* wb; float m;
    const float* mix; const float* out_w; const float* in_w; const float* norm_w; float eps;
    void* out; const int* rows; int S, D;
};

__device__ __forceinline__ float4 f4(float v) { return make_float4(v, v, v, v); }
__device__ __forceinline__ float4 fma4(float s, float4 x, float4 acc) {
    return make_float4(fmaf(s, x.x, acc.x), fmaf(s, x.y, acc.y), fmaf(s, x.z, acc.z), fmaf(s, x.w, acc.w));
}
__device__ __forceinline__ float4 add4(float4 x, float4 y) { return make_float4(x.x + y.x, x.y + y.y, x.z + y.z, x.w + y.w); }
__device__ __forceinline__ float dot4(float4 x, float acc) { return fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, acc)))); }
__device__ __forceinline__ float4 ld4(const float* p, size_t i) { return reinterpret_cast<const float4*>(p)[i]; }

__device__ __forceinline__ void put4(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* dst, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const unsigned*>(&lo);
    u.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(dst) = u;
}

// a sublayer's result in one column (or four): the slices in order
__device__ __forceinline__ float summed(const float* x, int slices, size_t stride, size_t at) {
    float v = x[at];
    for (int s = 1; s < slices; ++s) v += x[s * stride + at];
    return v;
}
__device__ __forceinline__ float4 summed4(const float* x, int slices, size_t stride, size_t at4) {
    float4 v = ld4(x, at4);
    for (int s = 1; s < slices; ++s) v = add4(v, ld4(x + s * stride, at4));
    return v;
}

// S known, D a multiple of 4 and every operand on 16 bytes.  One block per row.  Shared memory: D floats for u, 2 D more
// for the second form of y.
template <typename T, int S>
__global__ void __launch_bounds__(256, S <= 4 ? 3 : 1) hyper_vec_kernel(const HyperArgs g) {
    pdl_enter();
    extern __shared__ __align__(16) float us[];
    __shared__ float red[32], pair_w[HYPER_PAIRS];
    __shared__ int pair_at[HYPER_PAIRS];
    const int r = blockIdx.x, t = g.rows ? g.rows[r] : r, D = g.D, D4 = D >> 2;
    const size_t row4 = (size_t)t * D4;
    const bool adds = g.a || g.py || g.bias, pair = g.wb != nullptr;
    float mix[S][S], ow[S], iw[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        ow[s] = adds ? g.out_w[s] : 0.0f;
        iw[s] = g.in_w ? g.in_w[s] : 0.0f;
#pragma unroll
        for (int q = 0; q < S; ++q) mix[s][q] = adds ? g.mix[s * S + q] : 0.0f;
    }
    if (g.py) {                                                   // the token's routed rows: where they lie and their weights
        for (int j = threadIdx.x; j < g.pairs; j += blockDim.x) {
            pair_at[j] = g.pair_row ? g.pair_row[t * g.pairs + j] : t * g.pairs + j;
            pair_w[j] = g.pw[t * g.pairs + j];
        }
        __syncthreads();
    }
    float4* ya = reinterpret_cast<float4*>(us + D);
    float4* yb = ya + D4;
    float ca = 0.0f, cb = 0.0f;
    if (pair) {                                                   // both results of the row, then their norms
        float sa = 0.0f, sb = 0.0f;
        for (int i = threadIdx.x; i < D4; i += blockDim.x) {
            float4 va = summed4(g.a, g.a_slices, g.slice_stride, row4 + i);
            if (g.bias) va = add4(va, ld4(g.bias, i));
            const float4 vb = summed4(g.b, g.b_slices, g.slice_stride, row4 + i);
            ya[i] = va, yb[i] = vb;
            sa = dot4(va, sa), sb = dot4(vb, sb);
        }
        ca = rsqrtf(block_sum(sa, red) / (float)D + g.eps) * g.m;
        cb = rsqrtf(block_sum(sb, red) / (float)D + g.eps) * g.m;
    }
    float ss = 0.0f;
    for (int i = threadIdx.x; i < D4; i += blockDim.x) {
        float4 x[S];
        if (g.broadcast) {
            x[0] = ld4(g.src, row4 + i);
#pragma unroll
            for (int s = 1; s < S; ++s) x[s] = x[0];
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) x[s] = ld4(g.src, ((size_t)t * S + s) * D4 + i);
        }
        if (adds) {
            float4 y = f4(0.0f);
            if (pair) {
                const float4 va = ya[i], vb = yb[i], wa = ld4(g.wa, i), wb = ld4(g.wb, i);
                y = make_float4(va.x * ca * wa.x + vb.x * cb * wb.x, va.y * ca * wa.y + vb.y * cb * wb.y,
                                va.z * ca * wa.z + vb.z * cb * wb.z, va.w * ca * wa.w + vb.w * cb * wb.w);
            } else {
                if (g.a) y = summed4(g.a, g.a_slices, g.slice_stride, row4 + i);
                if (g.bias) y = add4(y, ld4(g.bias, i));
                if (g.py) {
                    float4 sp = f4(0.0f);
#pragma unroll 4
                    for (int j = 0; j < g.pairs; ++j) sp = fma4(pair_w[j], ld4(g.py, (size_t)pair_at[j] * D4 + i), sp);
                    y = add4(y, sp);
                }
            }
            float4 n[S];
#pragma unroll
            for (int q = 0; q < S; ++q) {
                float4 v = f4(0.0f);
#pragma unroll
                for (int s = 0; s < S; ++s) v = fma4(mix[s][q], x[s], v);
                n[q] = fma4(ow[q], y, v);
            }
#pragma unroll
            for (int q = 0; q < S; ++q) {
                x[q] = n[q];
                if (g.dst) reinterpret_cast<float4*>(g.dst)[((size_t)t * S + q) * D4 + i] = n[q];
            }
        }
        if (g.out) {
            float4 u = f4(0.0f);
#pragma unroll
            for (int s = 0; s < S; ++s) u = fma4(iw[s], x[s], u);
            reinterpret_cast<float4*>(us)[i] = u;
            ss = dot4(u, ss);
        }
    }
    if (!g.out) return;
    const float inv = rsqrtf(block_sum(ss, red) / (float)D + g.eps);
    for (int i = threadIdx.x; i < D4; i += blockDim.x) {
        const float4 u = reinterpret_cast<const float4*>(us)[i], w = ld4(g.norm_w, i);
        put4((T*)g.out + (size_t)r * D + 4 * i, make_float4(u.x * inv * w.x, u.y * inv * w.y, u.z * inv * w.z, u.w * inv * w.w));
    }
}

// Any number of streams up to HYPER_MAX_STREAMS, any D, no alignment.
template <typename T>
__global__ void __launch_bounds__(256) hyper_any_kernel(const HyperArgs g) {
    pdl_enter();
    extern __shared__ __align__(16) float us[];
    __shared__ float red[32];
    const int r = blockIdx.x, t = g.rows ? g.rows[r] : r, D = g.D, S = g.S;
    const size_t row = (size_t)t * D;
    const bool adds = g.a || g.py || g.bias, pair = g.wb != nullptr;
    float *ya = us + D, *yb = us + 2 * D;
    float ca = 0.0f, cb = 0.0f;
    if (pair) {
        float sa = 0.0f, sb = 0.0f;
        for (int i = threadIdx.x; i < D; i += blockDim.x) {
            float va = summed(g.a, g.a_slices, g.slice_stride, row + i);
            if (g.bias) va += g.bias[i];
            const float vb = summed(g.b, g.b_slices, g.slice_stride, row + i);
            ya[i] = va, yb[i] = vb;
            sa = fmaf(va, va, sa), sb = fmaf(vb, vb, sb);
        }
        ca = rsqrtf(block_sum(sa, red) / (float)D + g.eps) * g.m;
        cb = rsqrtf(block_sum(sb, red) / (float)D + g.eps) * g.m;
    }
    float ss = 0.0f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float x[HYPER_MAX_STREAMS], y = 0.0f, u = 0.0f;
        for (int s = 0; s < S; ++s) x[s] = g.src[g.broadcast ? row + i : ((size_t)t * S + s) * D + i];
        if (adds) {
            if (pair) {
                y = ya[i] * ca * g.wa[i] + yb[i] * cb * g.wb[i];
            } else {
                if (g.a) y = summed(g.a, g.a_slices, g.slice_stride, row + i);
                if (g.bias) y += g.bias[i];
                if (g.py) {
                    float sp = 0.0f;
                    for (int j = 0; j < g.pairs; ++j) {
                        const int at = t * g.pairs + j;
                        sp = fmaf(g.pw[at], g.py[(size_t)(g.pair_row ? g.pair_row[at] : at) * D + i], sp);
                    }
                    y += sp;
                }
            }
        }
        for (int q = 0; q < S; ++q) {
            float v = x[q];
            if (adds) {
                v = 0.0f;
                for (int s = 0; s < S; ++s) v = fmaf(g.mix[s * S + q], x[s], v);
                v = fmaf(g.out_w[q], y, v);
                if (g.dst) g.dst[((size_t)t * S + q) * D + i] = v;
            }
            if (g.out) u = fmaf(g.in_w[q], v, u);
        }
        us[i] = u;
        ss = fmaf(u, u, ss);
    }
    if (!g.out) return;
    const float inv = rsqrtf(block_sum(ss, red) / (float)D + g.eps);
    for (int i = threadIdx.x; i < D; i += blockDim.x) ((T*)g.out)[(size_t)r * D + i] = from_f32<T>(us[i] * inv * g.norm_w[i]);
}

// out[t] = m (norm(a[t] + bias) wa + norm(b[t]) wb), FP32.
__global__ void __launch_bounds__(256) normed_pair_kernel(const float* a, int a_slices, const float* bias, const float* b, int b_slices, size_t slice_stride,
                                                          const float* wa, const float* wb, float m, float eps, float* out, int D) {
    pdl_enter();
    extern __shared__ __align__(16) float ys[];            // 2 D floats
    __shared__ float red[32];
    const size_t row = (size_t)blockIdx.x * D;
    float sa = 0.0f, sb = 0.0f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float va = summed(a, a_slices, slice_stride, row + i);
        if (bias) va += bias[i];
        const float vb = summed(b, b_slices, slice_stride, row + i);
        ys[i] = va, ys[D + i] = vb;
        sa = fmaf(va, va, sa), sb = fmaf(vb, vb, sb);
    }
    const float ca = rsqrtf(block_sum(sa, red) / (float)D + eps) * m;
    const float cb = rsqrtf(block_sum(sb, red) / (float)D + eps) * m;
    for (int i = threadIdx.x; i < D; i += blockDim.x) out[row + i] = ys[i] * ca * wa[i] + ys[D + i] * cb * wb[i];
}

}  // namespace

Q6K_API int q6k_hyper_max_streams() { return HYPER_MAX_STREAMS; }

// R rows (picked by `rows`, or all).  slice_stride: floats between two slices of a and of b.
Q6K_API int q6k_hyper_step(const float* src, int broadcast, float* dst, const float* a, int a_slices, long long slice_stride, const float* bias,
                           const float* py, const int* pair_row, const float* pw, int pairs, const float* b, int b_slices, const float* wa,
                           const float* wb, float m, const float* mix, const float* out_w, const float* in_w, const float* norm_w, float eps,
                           void* out, const int* rows, int R, int S, int D, int dtype, cudaStream_t st) {
    if (R == 0) return 0;
    Q6K_REQUIRE(R > 0 && D > 0 && S > 0 && S <= HYPER_MAX_STREAMS, "hyper_step: bad sizes R=%d D=%d streams=%d (at most %d)", R, D, S, HYPER_MAX_STREAMS);
    Q6K_REQUIRE(a_slices >= 1 && b_slices >= 1, "hyper_step: %d and %d slices", a_slices, b_slices);
    const bool adds = a || py || bias;
    Q6K_REQUIRE(!adds || (mix && out_w), "hyper_step: an add needs its weights");
    Q6K_REQUIRE(!py || (pw && pairs > 0), "hyper_step: weighted rows need their weights");
    Q6K_REQUIRE((wb == nullptr) == (b == nullptr) && (!wb || (wa && a && !py)), "hyper_step: two normed results come with both weights and without routed rows");
    Q6K_REQUIRE(!out || (in_w && norm_w), "hyper_step: a norm needs the streams' weights and its own");
    Q6K_REQUIRE(!dst || (adds && !rows), "hyper_step: streams are written when something is added, for all rows");
    HyperArgs g{src, broadcast, dst, a, a_slices, (size_t)slice_stride, bias, py, pair_row, pw, pairs, b, b_slices, wa, wb, m, mix, out_w, in_w, norm_w, eps, out, rows, S, D};
    const size_t smem = (size_t)D * (wb ? 3 : 1) * sizeof(float);
    Q6K_REQUIRE(smem <= 200 * 1024, "hyper_step: rows of %d do not fit shared memory", D);
    auto on16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    // which kernel runs depends on the row width, the stream count and the buffers' alignment alone, never on the step
    const bool vec = S <= 8 && pairs <= HYPER_PAIRS && D % 4 == 0 && slice_stride % 4 == 0 && on16(src) && on16(dst) && on16(a) && on16(bias) && on16(py) && on16(b) &&
                     on16(wa) && on16(wb) && on16(norm_w) && on16(out);
#define HYPER_GO(KERNEL)                                                                                               \
    do {                                                                                                               \
        auto kernel = KERNEL;                                                                                          \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
        q6k_launch(kernel, R, 256, smem, st, g);                                                                       \
    } while (0)
#define HYPER_CASE(N) case N: HYPER_GO((hyper_vec_kernel<T, N>)); break
    Q6K_DISPATCH(dtype, {
        if (!vec) HYPER_GO((hyper_any_kernel<T>));
        else switch (S) {
            HYPER_CASE(1); HYPER_CASE(2); HYPER_CASE(3); HYPER_CASE(4); HYPER_CASE(5); HYPER_CASE(6); HYPER_CASE(7); HYPER_CASE(8);
        }
    });
#undef HYPER_CASE
#undef HYPER_GO
    return q6k_check_launch("hyper_step");
}

Q6K_API int q6k_normed_pair(const float* a, int a_slices, const float* bias, const float* b, int b_slices, long long slice_stride, const float* wa,
                            const float* wb, float m, float eps, float* out, int T_, int D, cudaStream_t st) {
    if (T_ == 0) return 0;
    Q6K_REQUIRE(T_ > 0 && D > 0 && a_slices >= 1 && b_slices >= 1 && a && b && wa && wb, "normed_pair: bad sizes T=%d D=%d", T_, D);
    const size_t smem = 2 * (size_t)D * sizeof(float);
    Q6K_REQUIRE(smem <= 200 * 1024, "normed_pair: rows of %d do not fit shared memory", D);
    if (smem > 48 * 1024) cudaFuncSetAttribute(normed_pair_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    q6k_launch(normed_pair_kernel, T_, 256, smem, st, a, a_slices, bias, b, b_slices, (size_t)slice_stride, wa, wb, m, eps, out, D);
    return q6k_check_launch("normed_pair");
}
