// Retention: linear attention with one fixed decay per head and neither softmax nor denominator.  Per head, with a
// state S [dk, dv] that starts at zero and is carried from token to token in the request's state slot:
//
//     S <- decay S + k v^T;      o = S^T q
//
//  * retention_prep_kernel turns the first `rd` dimensions of every head of q and k by position * inv_freq[pair] (pairs by
//    halves, or of neighbours) and multiplies k by a scale, in place on the FP32 result of the projection; a block per token.
//    Before that it may pass the row's first `act_cols` columns (q, k and v of a mixer that activates them) through silu.
//  * retention_kernel walks a request's tokens in order.  A block owns 16 columns of one head of one request; a thread holds
//    a stretch of consecutive rows of ONE column in registers (lane = column and one of two stretches, eight warps = sixteen
//    stretches), so k and q of its rows come as 16-byte reads every lane of a half-warp shares and a token costs three
//    floating-point instructions per element of the state and little else.  A token's sum over the rows is the thread's own
//    (in row order), then the two stretches of a warp (one shuffle), then the eight warps' through shared memory, in the
//    warps' order: the same tree for every token wherever a prompt was cut.  q, k and v of eight tokens at a time are
//    copied to shared memory asynchronously, three tiles ahead of the one that is walked (a tile's first read is a miss in
//    L2 for one block of a head, and its latency is several times a tile's work).
//
// The same walk serves a second recurrence (TM below): a decay per token and key channel, the read-out before the write, and
// the current token entering the read-out through a bonus vector u per head,
//
//     o = S^T r + (sum_x u[x] k[x] r[x]) v;      S <- diag(w) S + k v^T
//
//  * token_shift_kernel makes what its projections read: per token n mixes x + (x' - x) mu_j of the token's row with the row
//    before it (x' = 0 for a sequence's first token; the row before a portion is kept in the request's state slot).
//  * time_mix_prep_kernel makes the decays w = exp(-exp(z + w0)) in place and the token's bonus number per head.
//
// Everything is FP32: angles, the rotation, decays and their powers, the state and every sum.
#include "common.cuh"

namespace {

constexpr int RET_WARPS = 8, RET_THREADS = RET_WARPS * 32, RET_COLS = 16, RET_CHUNKS = 2 * RET_WARPS, RET_TILE = 8, RET_STAGES = 4, RET_MAX_DK = 256;

// One block per token: the sines and cosines of its rd / 2 angles are made once (they are the same for every head, for q
// and for k), then every pair of q and of k is turned in place and the rest of k scaled; what neither turns nor scales
// is not touched.
__global__ void __launch_bounds__(256) retention_prep_kernel(float* p, int ld, int H, int dk, int q_col, int k_col,
                                                             const float* inv_freq, int rd, int neighbours, float k_scale,
                                                             const int* positions, int act_cols) {
    pdl_enter();
    extern __shared__ float xs[];            // cos [rd / 2] | sin [rd / 2]
    const int t = blockIdx.x, half = rd / 2;
    const float pos = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * inv_freq[i], &xs[half + i], &xs[i]);
    float* row = p + (size_t)t * ld;
    for (int c = threadIdx.x; c < act_cols; c += blockDim.x) {             // silu on the projections, before anything else
        const float z = row[c];
        row[c] = z / (1.0f + expf(-z));
    }
    __syncthreads();
    for (int w = threadIdx.x; w < 2 * H * half; w += blockDim.x) {          // (q or k, head, pair)
        const int i = w % half, h = (w / half) % H, is_k = w / (half * H);
        float* x = row + (is_k ? k_col : q_col) + (size_t)h * dk;
        const int a = neighbours ? 2 * i : i, b = neighbours ? 2 * i + 1 : i + half;
        const float u = x[a], v = x[b], cs = xs[i], sn = xs[half + i], mul = is_k ? k_scale : 1.0f;
        x[a] = (u * cs - v * sn) * mul;
        x[b] = (v * cs + u * sn) * mul;
    }
    if (k_scale != 1.0f) {
        const int rest = dk - rd;
        for (int w = threadIdx.x; w < H * rest; w += blockDim.x) {
            float* x = row + k_col + (size_t)(w / rest) * dk + rd + w % rest;
            *x *= k_scale;
        }
    }
}

// Four bytes from global to shared memory without passing registers; `in` false writes a zero and reads nothing.
__device__ __forceinline__ void ret_copy(float* dst, const float* src, bool in) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    const int bytes = in ? 4 : 0;
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}

__device__ __forceinline__ void ret_copy16(float* dst, const float* src, bool in) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    const int bytes = in ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}

// grid (R, H, ceil(dv / 16)), 256 threads.  qp, kp (prepared), vp: FP32, a token's heads side by side, rows ld apart; state: FP32
// [slots, H, dk, dv]; o: FP32 [T, H dv].  RPT: rows per thread (dk <= 16 RPT).  STAGES tiles are in flight or in use.
// WIDE: every head's q and k (and decays) start on 16 bytes in every row and dk is a multiple of 4 (copies of 16 bytes).
// TM: the second recurrence; q is r, wt: FP32 [T, ld_w] with the decays of head h from column h dk on, bonus: FP32 [T, H].
template <int RPT, int STAGES, bool WIDE, bool TM>
__global__ void __launch_bounds__(RET_THREADS) retention_kernel(const float* qp, const float* kp, const float* vp, int ld, const float* decay,
                                                                const float* wt, int ld_w, const float* bonus, float* state, const int* q_start,
                                                                const int* slot_ids, float* o, int H, int dk, int dv) {
    pdl_enter();
    constexpr int DKP = RET_CHUNKS * RPT;                                // rows, padded
    constexpr int PER_THREAD = RET_TILE * DKP / RET_THREADS;             // elements of q (and of k) a thread stages per tile
    static_assert(RPT % 4 == 0 && RET_TILE * DKP % RET_THREADS == 0 && RET_TILE * RET_COLS <= RET_THREADS, "16-byte reads; a tile divides among the threads");
    // q [STAGES][TILE][DKP] | k likewise | (TM: decays likewise) | v [STAGES][TILE][COLS] | sums [2][TILE][WARPS][COLS] | (TM: bonus [STAGES][TILE])
    extern __shared__ __align__(16) float sm[];
    float* qs = sm;
    float* ks = qs + STAGES * RET_TILE * DKP;
    float* ws = ks + STAGES * RET_TILE * DKP;
    float* vs = ws + (TM ? STAGES * RET_TILE * DKP : 0);
    float* red = vs + STAGES * RET_TILE * RET_COLS;
    float* bs = red + 2 * RET_TILE * RET_WARPS * RET_COLS;
    const int r = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * RET_COLS;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, cl = lane % RET_COLS, col = c0 + cl;
    const int row0 = (warp * 2 + lane / RET_COLS) * RPT;                 // this thread's first row
    const int t0 = q_start[r], t1 = q_start[r + 1];
    if (t0 >= t1) return;
    const float d = TM ? 0.0f : decay[head];
    float* mine = state + ((size_t)slot_ids[r] * H + head) * dk * dv + (col < dv ? col : 0);
    float s[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) s[i] = (col < dv && row0 + i < dk) ? mine[(size_t)(row0 + i) * dv] : 0.0f;
    auto fetch = [&](int ta, int b) {         // this thread's share of the tile that starts at token ta, on its way to buffer b
        const int n = min(RET_TILE, t1 - ta);
        if (n > 0) {
            if (WIDE) {
#pragma unroll
                for (int e = 0; e < (PER_THREAD + 3) / 4; ++e) {
                    const int i = (threadIdx.x + e * RET_THREADS) * 4, tt = i / DKP, row = i % DKP;
                    if (PER_THREAD >= 4 || i < RET_TILE * DKP) {
                        const bool in = tt < n && row < dk;
                        const size_t at = in ? (size_t)(ta + tt) * ld + (size_t)head * dk + row : 0;
                        ret_copy16(qs + b * RET_TILE * DKP + i, qp + at, in);
                        ret_copy16(ks + b * RET_TILE * DKP + i, kp + at, in);
                        if (TM) ret_copy16(ws + b * RET_TILE * DKP + i, in ? wt + (size_t)(ta + tt) * ld_w + (size_t)head * dk + row : wt, in);
                    }
                }
            } else {
#pragma unroll
                for (int e = 0; e < PER_THREAD; ++e) {
                    const int i = threadIdx.x + e * RET_THREADS, tt = i / DKP, row = i % DKP;
                    const bool in = tt < n && row < dk;
                    const size_t at = in ? (size_t)(ta + tt) * ld + (size_t)head * dk + row : 0;
                    ret_copy(qs + b * RET_TILE * DKP + i, qp + at, in);
                    ret_copy(ks + b * RET_TILE * DKP + i, kp + at, in);
                    if (TM) ret_copy(ws + b * RET_TILE * DKP + i, in ? wt + (size_t)(ta + tt) * ld_w + (size_t)head * dk + row : wt, in);
                }
            }
            if (threadIdx.x < RET_TILE * RET_COLS) {
                const int tt = threadIdx.x / RET_COLS, cc = c0 + threadIdx.x % RET_COLS;
                const bool in = tt < n && cc < dv;
                ret_copy(vs + b * RET_TILE * RET_COLS + threadIdx.x, in ? vp + (size_t)(ta + tt) * ld + (size_t)head * dv + cc : vp, in);
            }
            if (TM && threadIdx.x >= RET_THREADS - RET_TILE) {
                const int tt = threadIdx.x - (RET_THREADS - RET_TILE);
                ret_copy(bs + b * RET_TILE + tt, tt < n ? bonus + (size_t)(ta + tt) * H + head : bonus, tt < n);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto finish = [&](int ta, int b2) {       // the warps' sums of one (token, column), in the warps' order
        if (threadIdx.x < RET_TILE * RET_COLS) {
            const int tt = threadIdx.x / RET_COLS, cc = threadIdx.x % RET_COLS;
            if (ta + tt < t1 && c0 + cc < dv) {
                const float* src = red + (b2 * RET_TILE + tt) * RET_WARPS * RET_COLS + cc;
                float sum = src[0];
#pragma unroll
                for (int w = 1; w < RET_WARPS; ++w) sum += src[w * RET_COLS];
                o[((size_t)(ta + tt) * H + head) * dv + c0 + cc] = sum;
            }
        }
    };
#pragma unroll
    for (int st = 0; st < STAGES - 1; ++st) fetch(t0 + st * RET_TILE, st);
    int b = 0, b2 = 0;
    for (int ta = t0; ta < t1; ta += RET_TILE, b = b + 1 == STAGES ? 0 : b + 1, b2 ^= 1) {
        const int n = min(RET_TILE, t1 - ta);
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
        __syncthreads();                      // this tile has landed for everyone; the tile before it is done with
        if (ta > t0) finish(ta - RET_TILE, b2 ^ 1);
        fetch(ta + (STAGES - 1) * RET_TILE, b == 0 ? STAGES - 1 : b - 1);
        const float* qb = qs + b * RET_TILE * DKP + row0;
        const float* kb = ks + b * RET_TILE * DKP + row0;
        const float* wb = ws + b * RET_TILE * DKP + row0;
        const float* vb = vs + b * RET_TILE * RET_COLS + cl;
        const float* bb = bs + b * RET_TILE;
        const bool starts = warp == 0 && lane < RET_COLS;    // TM: the thread whose sum starts with the bonus
        auto element = [&](float& st, float kx, float qx, float wx, float v, float& acc) {
            if (TM) {
                acc = fmaf(st, qx, acc);
                st = fmaf(wx, st, kx * v);
            } else {
                st = fmaf(d, st, kx * v);
                acc = fmaf(st, qx, acc);
            }
        };
        float* rb = red + (b2 * RET_TILE * RET_WARPS + warp) * RET_COLS + cl;
        auto token = [&](int tt) {
            const float v = vb[tt * RET_COLS];
            float acc = TM && starts ? bb[tt] * v : 0.0f;
#pragma unroll
            for (int i = 0; i < RPT; i += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(kb + tt * DKP + i);
                const float4 q4 = *reinterpret_cast<const float4*>(qb + tt * DKP + i);
                const float4 w4 = TM ? *reinterpret_cast<const float4*>(wb + tt * DKP + i) : k4;
                element(s[i], k4.x, q4.x, w4.x, v, acc);
                element(s[i + 1], k4.y, q4.y, w4.y, v, acc);
                element(s[i + 2], k4.z, q4.z, w4.z, v, acc);
                element(s[i + 3], k4.w, q4.w, w4.w, v, acc);
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, RET_COLS);       // the lane with the same column and the warp's other rows
            if (lane < RET_COLS) rb[tt * RET_WARPS * RET_COLS] = acc;
        };
        if (n == RET_TILE) {                  // a full tile: the next token's rows are read while this one's are summed
            float4 kk[2][RPT / 4], qq[2][RPT / 4], ww[2][TM ? RPT / 4 : 1];
            float vv[RET_TILE];
#pragma unroll
            for (int tt = 0; tt < RET_TILE; ++tt) vv[tt] = vb[tt * RET_COLS];
#pragma unroll
            for (int i = 0; i < RPT / 4; ++i) {
                kk[0][i] = *reinterpret_cast<const float4*>(kb + 4 * i);
                qq[0][i] = *reinterpret_cast<const float4*>(qb + 4 * i);
                if (TM) ww[0][TM ? i : 0] = *reinterpret_cast<const float4*>(wb + 4 * i);
            }
#pragma unroll
            for (int tt = 0; tt < RET_TILE; ++tt) {
                if (tt + 1 < RET_TILE) {
#pragma unroll
                    for (int i = 0; i < RPT / 4; ++i) {
                        kk[(tt + 1) & 1][i] = *reinterpret_cast<const float4*>(kb + (tt + 1) * DKP + 4 * i);
                        qq[(tt + 1) & 1][i] = *reinterpret_cast<const float4*>(qb + (tt + 1) * DKP + 4 * i);
                        if (TM) ww[(tt + 1) & 1][TM ? i : 0] = *reinterpret_cast<const float4*>(wb + (tt + 1) * DKP + 4 * i);
                    }
                }
                const float v = vv[tt];
                float acc = TM && starts ? bb[tt] * v : 0.0f;
#pragma unroll
                for (int i = 0; i < RPT / 4; ++i) {
                    const float4 k4 = kk[tt & 1][i], q4 = qq[tt & 1][i], w4 = TM ? ww[tt & 1][TM ? i : 0] : k4;
                    element(s[4 * i], k4.x, q4.x, w4.x, v, acc);
                    element(s[4 * i + 1], k4.y, q4.y, w4.y, v, acc);
                    element(s[4 * i + 2], k4.z, q4.z, w4.z, v, acc);
                    element(s[4 * i + 3], k4.w, q4.w, w4.w, v, acc);
                }
                acc += __shfl_xor_sync(0xffffffffu, acc, RET_COLS);
                if (lane < RET_COLS) rb[tt * RET_WARPS * RET_COLS] = acc;
            }
        } else {
#pragma unroll
            for (int tt = 0; tt < RET_TILE; ++tt)
                if (tt < n) token(tt);
        }
    }
    __syncthreads();
    finish(t0 + (t1 - t0 - 1) / RET_TILE * RET_TILE, b2 ^ 1);
    if (col < dv) {
#pragma unroll
        for (int i = 0; i < RPT; ++i)
            if (row0 + i < dk) mine[(size_t)(row0 + i) * dv] = s[i];
    }
}

template <int RPT, int STAGES, bool WIDE, bool TM>
int launch_retention(dim3 grid, cudaStream_t st, const float* q, const float* k, const float* v, int ld, const float* decay, const float* wt, int ld_w,
                     const float* bonus, float* state, const int* q_start, const int* slot_ids, float* o, int H, int dk, int dv) {
    const size_t smem = (size_t)(STAGES * RET_TILE * ((TM ? 3 : 2) * RET_CHUNKS * RPT + RET_COLS + (TM ? 1 : 0)) + 2 * RET_TILE * RET_WARPS * RET_COLS) * sizeof(float);
    auto kernel = retention_kernel<RPT, STAGES, WIDE, TM>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    q6k_launch(kernel, grid, RET_THREADS, smem, st, q, k, v, ld, decay, wt, ld_w, bonus, state, q_start, slot_ids, o, H, dk, dv);
    return 0;
}

// One block per token: the n mixes of its row with the row before it, out[j, t] = T(x + (x' - x) mu[j]).  prev: FP32 [slots, D], the
// last row of the request's earlier portions (zeros at its start); the block of a portion's first row reads it, then leaves
// the portion's last row there.
template <typename T>
__global__ void __launch_bounds__(256) token_shift_kernel(const T* x, const float* mu, int n, float* prev, const int* req_of_token, const int* q_start,
                                                          const int* slot_ids, T* out, int T_, int D) {
    pdl_enter();
    const int t = blockIdx.x, r = req_of_token[t], first = q_start[r], last = q_start[r + 1] - 1;
    float* mine = prev + (size_t)slot_ids[r] * D;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        const float v = to_f32(x[(size_t)t * D + i]);
        float before;
        if (t == first) {
            before = mine[i];
            mine[i] = to_f32(x[(size_t)last * D + i]);
        } else {
            before = to_f32(x[(size_t)(t - 1) * D + i]);
        }
        for (int j = 0; j < n; ++j) out[((size_t)j * T_ + t) * D + i] = from_f32<T>(fmaf(before - v, mu[(size_t)j * D + i], v));
    }
}

// Eight values at a time as FP32 (16 bytes of bfloat16, 32 of FP32), and back.
template <typename T> __device__ __forceinline__ void load8(const T* p, float* v);
template <> __device__ __forceinline__ void load8<float>(const float* p, float* v) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float* v) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const unsigned w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) v[2 * i] = __uint_as_float(w[i] << 16), v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
}
__device__ __forceinline__ void store8(float* p, const float* v) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* v) {
    unsigned w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        w[i] = *reinterpret_cast<const unsigned*>(&h);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

// The same for rows of a multiple of eight entries that start on 16 bytes: grid (T, ceil(D / 8 / 128)), eight entries a thread.
template <typename T>
__global__ void __launch_bounds__(128) token_shift8_kernel(const T* x, const float* mu, int n, float* prev, const int* req_of_token, const int* q_start,
                                                           const int* slot_ids, T* out, int T_, int D) {
    pdl_enter();
    const int t = blockIdx.x, i = (blockIdx.y * 128 + threadIdx.x) * 8;
    if (i >= D) return;
    const int r = req_of_token[t], first = q_start[r];
    float v[8], before[8];
    load8<T>(x + (size_t)t * D + i, v);
    if (t == first) {
        float* mine = prev + (size_t)slot_ids[r] * D + i;
        float last[8];
        load8<float>(mine, before);
        load8<T>(x + (size_t)(q_start[r + 1] - 1) * D + i, last);
        store8(mine, last);
    } else {
        load8<T>(x + (size_t)(t - 1) * D + i, before);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) before[e] -= v[e];
    for (int j = 0; j < n; ++j) {
        float m[8], o[8];
        load8<float>(mu + (size_t)j * D + i, m);
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = fmaf(before[e], m[e], v[e]);
        store8(out + ((size_t)j * T_ + t) * D + i, o);
    }
}

// A warp per (token, head): w <- exp(-exp(w + w0)) in place, bonus = sum_x u[x] k[x] r[x].
__global__ void __launch_bounds__(128) time_mix_prep_kernel(const float* r, const float* k, int ld, float* w, const float* w0, const float* u, float* bonus,
                                                            int rows, int H, int dk) {
    pdl_enter();
    const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= rows) return;
    const int t = row / H, h = row % H;
    const float* rr = r + (size_t)t * ld + h * dk;
    const float* kr = k + (size_t)t * ld + h * dk;
    float* wr = w + ((size_t)t * H + h) * dk;
    float sum = 0.0f;
    for (int x = lane; x < dk; x += 32) {
        sum = fmaf(u[h * dk + x] * kr[x], rr[x], sum);
        wr[x] = expf(-expf(wr[x] + w0[h * dk + x]));
    }
    sum = warp_sum(sum);
    if (lane == 0) bonus[row] = sum;
}

}  // namespace

Q6K_API int q6k_retention_max_dim() { return RET_MAX_DK; }

// Rotates q and k of every head in place and scales k.
Q6K_API int q6k_retention_prep(float* p, int ld, int T_, int H, int dk, int q_col, int k_col,
                               const float* inv_freq, int rd, int neighbours, float k_scale, const int* positions, int act_cols,
                               cudaStream_t st) {
    if (T_ == 0) return 0;
    Q6K_REQUIRE(T_ > 0 && H > 0 && dk > 0 && 2 * H <= 65535, "retention_prep: bad sizes T=%d H=%d dk=%d", T_, H, dk);
    Q6K_REQUIRE(rd >= 0 && rd % 2 == 0 && rd <= dk && (rd == 0 || inv_freq), "retention_prep: %d turning dimensions of %d", rd, dk);
    Q6K_REQUIRE(act_cols >= 0 && act_cols <= ld, "retention_prep: %d activated columns of %d", act_cols, ld);
    if (rd == 0 && k_scale == 1.0f && act_cols == 0) return 0;
    q6k_launch(retention_prep_kernel, dim3(T_), 256, (size_t)rd * sizeof(float), st, p, ld, H, dk, q_col, k_col,
               inv_freq, rd, neighbours, k_scale, positions, act_cols);
    return q6k_check_launch("retention_prep");
}

Q6K_API int q6k_retention(const float* p, int ld, int q_col, int k_col, int v_col, const float* decay, float* state, const int* q_start,
                          const int* slot_ids, int R, float* o, int H, int dk, int dv, cudaStream_t st) {
    if (R == 0) return 0;
    Q6K_REQUIRE(R > 0 && H > 0 && dk > 0 && dv > 0 && dk <= RET_MAX_DK, "retention: bad sizes R=%d H=%d dk=%d (at most %d) dv=%d", R, H, dk, RET_MAX_DK, dv);
    const int zb = (dv + RET_COLS - 1) / RET_COLS;
    Q6K_REQUIRE(H <= 65535 && zb <= 65535, "retention: grid too large");
    const dim3 grid(R, H, zb);
    auto on16 = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
    const bool wide = dk % 4 == 0 && ld % 4 == 0 && on16(p + q_col) && on16(p + k_col);
#define RET_LAUNCH(RPT)                                                                                                               \
    do {                                                                                                                              \
        if (wide) launch_retention<RPT, RET_STAGES, true, false>(grid, st, p + q_col, p + k_col, p + v_col, ld, decay, nullptr, 0, nullptr, state, q_start, slot_ids, o, H, dk, dv); \
        else launch_retention<RPT, RET_STAGES, false, false>(grid, st, p + q_col, p + k_col, p + v_col, ld, decay, nullptr, 0, nullptr, state, q_start, slot_ids, o, H, dk, dv);     \
    } while (0)
    if (dk <= 64) RET_LAUNCH(4);
    else if (dk <= 128) RET_LAUNCH(8);
    else RET_LAUNCH(16);
#undef RET_LAUNCH
    return q6k_check_launch("retention");
}

// x: [T, D] in the storage type; mu: FP32 [n, D]; prev: FP32 [slots, D]; out: [n, T, D] in the storage type.
Q6K_API int q6k_token_shift(const void* x, const float* mu, int n, float* prev, const int* req_of_token, const int* q_start, const int* slot_ids, void* out,
                            int T_, int D, int dtype, cudaStream_t st) {
    if (T_ == 0) return 0;
    Q6K_REQUIRE(T_ > 0 && D > 0 && n > 0, "token_shift: bad sizes T=%d D=%d n=%d", T_, D, n);
    auto on16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (D % 8 == 0 && on16(x) && on16(mu) && on16(prev) && on16(out)) {
        Q6K_DISPATCH(dtype, q6k_launch(token_shift8_kernel<T>, dim3(T_, (D / 8 + 127) / 128), 128, 0, st, (const T*)x, mu, n, prev, req_of_token, q_start, slot_ids,
                                       (T*)out, T_, D););
        return q6k_check_launch("token_shift");
    }
    Q6K_DISPATCH(dtype, q6k_launch(token_shift_kernel<T>, dim3(T_), 256, 0, st, (const T*)x, mu, n, prev, req_of_token, q_start, slot_ids, (T*)out, T_, D););
    return q6k_check_launch("token_shift");
}

// r, k: FP32, a token's heads side by side, rows ld apart; w: FP32 [T, H dk] (in: the decay projection, out: the decays); w0, u: FP32 [H dk];
// bonus: FP32 [T, H].
Q6K_API int q6k_time_mix_prep(const float* r, const float* k, int ld, float* w, const float* w0, const float* u, float* bonus, int T_, int H, int dk, cudaStream_t st) {
    if (T_ == 0) return 0;
    Q6K_REQUIRE(T_ > 0 && H > 0 && dk > 0 && (long long)T_ * H <= 0x7fffffffLL, "time_mix_prep: bad sizes T=%d H=%d dk=%d", T_, H, dk);
    q6k_launch(time_mix_prep_kernel, dim3((unsigned)(((long long)T_ * H + 3) / 4)), 128, 0, st, r, k, ld, w, w0, u, bonus, T_ * H, H, dk);
    return q6k_check_launch("time_mix_prep");
}

// The second recurrence: r, k, v FP32, rows ld apart; w: FP32 [T, H dk] decays; bonus: FP32 [T, H]; state: FP32 [slots, H, dk, dv]; o: FP32 [T, H dv].
Q6K_API int q6k_time_mix(const float* r, const float* k, const float* v, int ld, const float* w, const float* bonus, float* state, const int* q_start,
                         const int* slot_ids, int R, float* o, int H, int dk, int dv, cudaStream_t st) {
    if (R == 0) return 0;
    Q6K_REQUIRE(R > 0 && H > 0 && dk > 0 && dv > 0 && dk <= RET_MAX_DK, "time_mix: bad sizes R=%d H=%d dk=%d (at most %d) dv=%d", R, H, dk, RET_MAX_DK, dv);
    const int zb = (dv + RET_COLS - 1) / RET_COLS;
    Q6K_REQUIRE(H <= 65535 && zb <= 65535, "time_mix: grid too large");
    const dim3 grid(R, H, zb);
    auto on16 = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
    const bool wide = dk % 4 == 0 && ld % 4 == 0 && on16(r) && on16(k) && on16(w);
#define RET_LAUNCH(RPT)                                                                                                               \
    do {                                                                                                                              \
        if (wide) launch_retention<RPT, RET_STAGES, true, true>(grid, st, r, k, v, ld, nullptr, w, H * dk, bonus, state, q_start, slot_ids, o, H, dk, dv); \
        else launch_retention<RPT, RET_STAGES, false, true>(grid, st, r, k, v, ld, nullptr, w, H * dk, bonus, state, q_start, slot_ids, o, H, dk, dv);     \
    } while (0)
    if (dk <= 64) RET_LAUNCH(4);
    else if (dk <= 128) RET_LAUNCH(8);
    else RET_LAUNCH(16);
#undef RET_LAUNCH
    return q6k_check_launch("time_mix");
}
