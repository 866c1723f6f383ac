// Layer norm with weight and bias over rows of the FP32 residual stream, in the places a block with norms on both sides of a
// sublayer needs it, as one kernel.  For row t (t = r, or rows[r]):
//
//   u[t] = gate[t] * y[t] + sum_s pw[t, s] * py[row(t, s)] + xw[t] * x[t]        what the sublayer before left, unsummed
//   1. "after":   h[t] += LN(u[t]; wa, ba)        or, "replace":   h[t] = u[t] + vec
//   2. "plus":    h[t] += extra[t]                (the embedding output re-entering a repeated span of layers)
//   3. "before":  out[r] = T(LN(h[t]; w, b))      the next sublayer's input in the operand dtype,
//      or "raw":  out[r] = T(h[t])                the stream as it stands
//
// y: a sublayer's FP32 result, or [splits, R, D] partial sums added in order; gate: one number per row (null: 1).  py, pair_row,
// pw: a routed feed-forward's results and weights (row(t, s) = pair_row[t*S + s], or t*S + s); a row whose weight is zero is not
// read (experts that answer their input have no row: their part is xw[t] * x[t], x in the operand dtype).
//
// Any subset may be asked for in one launch; 1 and 3 together close one sublayer and open the next with a single pass
// over the row.  With picked rows h itself is left as it is.  LN(x) = (x - mean) / sqrt(var + eps) * w + b with the mean
// first and the variance as the mean of squared deviations from it, all in FP32, summed in a fixed order.
#include "common.cuh"

namespace {

struct LayerNormArgs {
    float* h;
    const float* y; int splits; size_t split_stride; const float* gate;
    const float* py; const int* pair_row; const float* pw; int S;
    const void* x; const float* xw;
    const float* wa; const float* ba; int replace; const float* vec;
    const float* extra;
    const float* w; const float* b; const int* rows;
    void* out; long long ldo; int D; float eps;
};

template <typename T>
__global__ void __launch_bounds__(256) layernorm_kernel(const LayerNormArgs a) {
    pdl_enter();
    extern __shared__ float row[];            // D floats
    __shared__ float red[32];
    const int r = blockIdx.x, D = a.D, t = a.rows ? a.rows[r] : r;
    const size_t at = (size_t)t * D;
    float* hr = a.h + at;
    const bool add = a.y || a.py || a.x, store = !a.rows;
    auto stats = [&](float& mean, float& inv) {           // a thread reads back only what it wrote itself
        float s = 0.0f;
        for (int i = threadIdx.x; i < D; i += blockDim.x) s += row[i];
        mean = block_sum(s, red) / (float)D;
        float q = 0.0f;
        for (int i = threadIdx.x; i < D; i += blockDim.x) {
            const float d = row[i] - mean;
            q = fmaf(d, d, q);
        }
        inv = rsqrtf(block_sum(q, red) / (float)D + a.eps);
    };
    float mean = 0.0f, inv = 1.0f;
    if (add) {
        for (int i = threadIdx.x; i < D; i += blockDim.x) {
            float v = 0.0f;
            if (a.y) {
                v = a.y[at + i];
                for (int k = 1; k < a.splits; ++k) v += a.y[k * a.split_stride + at + i];
                if (a.gate) v *= a.gate[t];
            }
            if (a.py) {
                float sp = 0.0f;
                for (int s = 0; s < a.S; ++s) {
                    const float g = a.pw[(size_t)t * a.S + s];
                    if (g != 0.0f) sp = fmaf(g, a.py[(size_t)(a.pair_row ? a.pair_row[(size_t)t * a.S + s] : t * a.S + s) * D + i], sp);
                }
                v += sp;
            }
            if (a.x) v = fmaf(a.xw[t], to_f32(((const T*)a.x)[at + i]), v);
            row[i] = v;
        }
        if (!a.replace) stats(mean, inv);
    }
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float v;
        if (!add) v = hr[i];
        else if (a.replace) v = row[i] + (a.vec ? a.vec[i] : 0.0f);
        else v = hr[i] + ((row[i] - mean) * inv * a.wa[i] + a.ba[i]);
        if (a.extra) v += a.extra[at + i];
        if (store && (add || a.extra)) hr[i] = v;
        row[i] = v;
    }
    if (!a.out) return;
    T* o = (T*)a.out + (size_t)r * a.ldo;
    if (!a.w) {
        for (int i = threadIdx.x; i < D; i += blockDim.x) o[i] = from_f32<T>(row[i]);
        return;
    }
    stats(mean, inv);
    for (int i = threadIdx.x; i < D; i += blockDim.x) o[i] = from_f32<T>((row[i] - mean) * inv * a.w[i] + a.b[i]);
}

__device__ __forceinline__ void store4(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* dst, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const unsigned*>(&lo);
    u.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(dst) = u;
}
__device__ __forceinline__ float4 load4(const float* src) { return *reinterpret_cast<const float4*>(src); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* src) {
    const uint2 u = *reinterpret_cast<const uint2*>(src);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}

// The same with the row in registers (D a multiple of 4, at most 1024 * V4; every operand on 16 bytes, `out` and x on 8 in
// bfloat16): one read of every input, 16-byte accesses.  MIX: there are routed rows, a gate or x (their places and weights
// wait in shared memory, S of them at most MIX_SLOTS).
constexpr int MIX_SLOTS = 64;

// Sum over the 256 threads in a fixed order; `red` holds 8 floats that nothing else uses in this kernel.
__device__ __forceinline__ float block_sum_once(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) t += red[i];
    return t;
}

template <typename T, int V4, bool MIX>
__global__ void __launch_bounds__(256) layernorm_reg_kernel(const LayerNormArgs a) {
    pdl_enter();
    __shared__ float red[4][8];
    __shared__ float slot_w[MIX ? MIX_SLOTS : 1];
    __shared__ int slot_row[MIX ? MIX_SLOTS : 1];
    __shared__ int slots_live;
    const int r = blockIdx.x, D = a.D, t = a.rows ? a.rows[r] : r;
    const size_t at = (size_t)t * D;
    float* h = a.h + at;
    const bool add = a.y || (MIX && (a.py || a.x)), store = !a.rows;
    float4 v[V4];
    bool has[V4];
#pragma unroll
    for (int j = 0; j < V4; ++j) has[j] = (threadIdx.x + 256 * j) * 4 < D;
    auto stats = [&](float& mean, float& inv, int which) {
        float s = 0.0f;
#pragma unroll
        for (int j = 0; j < V4; ++j)
            if (has[j]) s += (v[j].x + v[j].y) + (v[j].z + v[j].w);
        mean = block_sum_once(s, red[which]) / (float)D;
        float q = 0.0f;
#pragma unroll
        for (int j = 0; j < V4; ++j)
            if (has[j]) {
                const float a0 = v[j].x - mean, a1 = v[j].y - mean, a2 = v[j].z - mean, a3 = v[j].w - mean;
                q += fmaf(a0, a0, a1 * a1) + fmaf(a2, a2, a3 * a3);
            }
        inv = rsqrtf(block_sum_once(q, red[which + 1]) / (float)D + a.eps);
    };
    float mean = 0.0f, inv = 1.0f;
    // everything whose place is known is asked of memory before the first wait
    float4 was[V4];
#pragma unroll
    for (int j = 0; j < V4; ++j)
        if (has[j] && !(add && a.replace)) was[j] = load4(h + (threadIdx.x + 256 * j) * 4);
    if (add) {
        float gate = 1.0f, xw = 0.0f;
        int live = 0;
#pragma unroll
        for (int j = 0; j < V4; ++j) {
            v[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (has[j] && a.y) v[j] = load4(a.y + at + (threadIdx.x + 256 * j) * 4);
        }
        if (MIX) {
            if (a.gate) gate = a.gate[t];
            if (a.x) xw = a.xw[t];
            if (a.py) {
                if (threadIdx.x < 32) {                      // the slots whose weight is not zero, in their order
                    int n = 0;
                    for (int s0 = 0; s0 < a.S; s0 += 32) {
                        const int s = s0 + (int)threadIdx.x;
                        const float g = s < a.S ? a.pw[(size_t)t * a.S + s] : 0.0f;
                        const int place = s < a.S && a.pair_row ? a.pair_row[(size_t)t * a.S + s] : t * a.S + s;
                        const unsigned on = __ballot_sync(0xffffffffu, g != 0.0f);
                        if (g != 0.0f) {
                            const int i = n + __popc(on & ((1u << threadIdx.x) - 1u));
                            slot_w[i] = g, slot_row[i] = place;
                        }
                        n += __popc(on);
                    }
                    if (threadIdx.x == 0) slots_live = n;
                }
                __syncthreads();
                live = slots_live;
            }
        }
#pragma unroll
        for (int j = 0; j < V4; ++j)
            if (has[j]) {
                const int c = (threadIdx.x + 256 * j) * 4;
                if (a.y) {
                    for (int k = 1; k < a.splits; ++k) {
                        const float4 o = load4(a.y + k * a.split_stride + at + c);
                        v[j].x += o.x, v[j].y += o.y, v[j].z += o.z, v[j].w += o.w;
                    }
                    if (MIX) v[j].x *= gate, v[j].y *= gate, v[j].z *= gate, v[j].w *= gate;
                }
                if (MIX) {
                    float4 sp = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 4
                    for (int s = 0; s < live; ++s) {         // four rows' loads on the way at a time
                        const float g = slot_w[s];
                        const float4 o = load4(a.py + (size_t)slot_row[s] * D + c);
                        sp.x = fmaf(g, o.x, sp.x), sp.y = fmaf(g, o.y, sp.y), sp.z = fmaf(g, o.z, sp.z), sp.w = fmaf(g, o.w, sp.w);
                    }
                    v[j].x += sp.x, v[j].y += sp.y, v[j].z += sp.z, v[j].w += sp.w;
                    if (xw != 0.0f) {
                        const float4 o = load4((const T*)a.x + at + c);
                        v[j].x = fmaf(xw, o.x, v[j].x), v[j].y = fmaf(xw, o.y, v[j].y), v[j].z = fmaf(xw, o.z, v[j].z), v[j].w = fmaf(xw, o.w, v[j].w);
                    }
                }
            }
        if (!a.replace) stats(mean, inv, 0);
    }
#pragma unroll
    for (int j = 0; j < V4; ++j)
        if (has[j]) {
            const int c = (threadIdx.x + 256 * j) * 4;
            if (!add) {
                v[j] = was[j];
            } else if (a.replace) {
                if (a.vec) {
                    const float4 e = load4(a.vec + c);
                    v[j].x += e.x, v[j].y += e.y, v[j].z += e.z, v[j].w += e.w;
                }
            } else {
                const float4 hv = was[j], ww = load4(a.wa + c), bb = load4(a.ba + c);
                v[j].x = hv.x + ((v[j].x - mean) * inv * ww.x + bb.x), v[j].y = hv.y + ((v[j].y - mean) * inv * ww.y + bb.y);
                v[j].z = hv.z + ((v[j].z - mean) * inv * ww.z + bb.z), v[j].w = hv.w + ((v[j].w - mean) * inv * ww.w + bb.w);
            }
            if (a.extra) {
                const float4 e = load4(a.extra + at + c);
                v[j].x += e.x, v[j].y += e.y, v[j].z += e.z, v[j].w += e.w;
            }
            if (store && (add || a.extra)) store4(h + c, v[j]);
        }
    if (!a.out) return;
    T* o = (T*)a.out + (size_t)r * a.ldo;
    if (a.w) stats(mean, inv, 2);
#pragma unroll
    for (int j = 0; j < V4; ++j)
        if (has[j]) {
            const int c = (threadIdx.x + 256 * j) * 4;
            float4 n = v[j];
            if (a.w) {
                const float4 ww = load4(a.w + c), bb = load4(a.b + c);
                n.x = (n.x - mean) * inv * ww.x + bb.x, n.y = (n.y - mean) * inv * ww.y + bb.y;
                n.z = (n.z - mean) * inv * ww.z + bb.z, n.w = (n.w - mean) * inv * ww.w + bb.w;
            }
            store4(o + c, n);
        }
}

}  // namespace

// h: FP32 [*, D], updated in place when there is something to add (and rows is null).  y: FP32 [R, D] or [splits, R, D] (slices
// split_stride floats apart) or null; gate: FP32 [*] or null.  py, pair_row, pw (S a token), x (operand dtype [*, D]), xw (FP32 [*]): see
// above, or null.  wa, ba: the weight and bias of the norm applied to the sum, unless replace (vec: FP32 [D] or null).  extra:
// FP32 like h, or null.  out: rows ldo elements apart in `dtype`, the norm of w and b or (w null) the stream itself, or null.
// rows: int32 [R] picks the rows (h is not updated then), or null.
Q6K_API int q6k_layernorm(float* h, const float* y, int splits, long long split_stride, const float* gate, const float* py, const int* pair_row,
                          const float* pw, int S, const void* x, const float* xw, const float* wa, const float* ba, int replace, const float* vec,
                          const float* extra, const float* w, const float* b, const int* rows, void* out, long long ldo, int R, int D, float eps,
                          int dtype, cudaStream_t st) {
    if (R == 0) return 0;
    Q6K_REQUIRE(R > 0 && D > 0 && D <= 12000, "layernorm: bad sizes R=%d D=%d (rows of at most 12000)", R, D);
    const bool add = y || py || x;
    Q6K_REQUIRE(!add || replace || (wa && ba), "layernorm: a sublayer result needs the weight and bias of its norm");
    Q6K_REQUIRE(!replace || add, "layernorm: nothing to replace the stream with");
    Q6K_REQUIRE(splits >= 1 && (!gate || y), "layernorm: bad sublayer result (%d slices)", splits);
    Q6K_REQUIRE(!py || (pw && S > 0), "layernorm: routed rows need their weights");
    Q6K_REQUIRE((x == nullptr) == (xw == nullptr), "layernorm: an input that joins the sum needs its weights");
    Q6K_REQUIRE(!w || (b && out), "layernorm: an output needs weight, bias and a buffer");
    Q6K_REQUIRE(!out || ldo >= D, "layernorm: output rows %lld apart for %d columns", ldo, D);
    const LayerNormArgs a{h, y, splits, (size_t)split_stride, gate, py, pair_row, pw, S, x, xw, wa, ba, replace, vec, extra, w, b, rows, out, ldo, D, eps};
    auto on = [](const void* p, int bytes) { return ((uintptr_t)p & (bytes - 1)) == 0; };
    const int narrow = dtype == Q6K_BF16 ? 8 : 16;
    const bool aligned = D % 4 == 0 && D <= 4096 && (!y || split_stride % 4 == 0) && on(h, 16) && on(y, 16) && on(py, 16) && on(x, narrow) && on(wa, 16) &&
                         on(ba, 16) && on(vec, 16) && on(extra, 16) && on(w, 16) && on(b, 16) && on(out, narrow) && (!out || ldo % 4 == 0) && (!py || S <= MIX_SLOTS);
    const bool mix = py || x || gate;
#define LN_REG(V4)                                                                                                \
    do {                                                                                                          \
        if (mix) Q6K_DISPATCH(dtype, q6k_launch(layernorm_reg_kernel<T, V4, true>, dim3(R), 256, 0, st, a););    \
        else Q6K_DISPATCH(dtype, q6k_launch(layernorm_reg_kernel<T, V4, false>, dim3(R), 256, 0, st, a););       \
    } while (0)
    if (aligned && D <= 1024) LN_REG(1);
    else if (aligned && D <= 2048) LN_REG(2);
    else if (aligned) LN_REG(4);
    else Q6K_DISPATCH(dtype, q6k_launch(layernorm_kernel<T>, dim3(R), 256, (size_t)D * sizeof(float), st, a););
#undef LN_REG
    return q6k_check_launch("layernorm");
}
