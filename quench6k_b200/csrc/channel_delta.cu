// The gated delta rule with one decay per head AND key channel.  Per head, with a state S [dk, dv] in FP32:
//
//     S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// with q and k made unit vectors per head first (q also times dk^-1/2), beta = sigmoid(b) and the decays
// g[x] = exp(-exp(A_log) softplus(a[x] + dt_bias[x])), everything FP32.
//
// Tokens are taken CH at a time (four; one in a step of single tokens), counted from the start of the request's portion.  With S the state before the chunk,
// P_i = g_1 ... g_i (per channel, products within the chunk), k'_i = P_i k_i, q'_i = P_i q_i and k''_m = (g_(m+1) ... g_CH) k_m,
//
//     u_i = beta_i (v_i - S^T k'_i - sum_(m<i) u_m kk[m, i]),     kk[m, i] = sum_x k_m[x] k_i[x] g_(m+1)[x] ... g_i[x]
//     o_i = S^T q'_i + sum_(m<=i) u_m kq[m, i],                   kq[m, i] likewise with q_i
//     S  <- diag(P_CH) S + sum_m k''_m u_m^T
//
// (no quotient of decays is ever formed: every product of decays is made going forward, so a channel that forgets at once is
// as exact as one that keeps everything).  The columns of S do not meet, and nothing but u, v and o depends on the column:
// the vectors k', q', k'', P_CH and the numbers kk, kq, beta of a chunk are made once per head by delta_channel_prepare_kernel
// for steps with long portions; the recurrence copies them to shared memory ahead of its walk, and for steps of a few
// tokens makes them itself.  A block owns COLS columns of one head of one request, LANES lanes share a column; lane l holds
// rows 4 (l + LANES j) .. + 3.  One pass over the state gives the eight sums of a chunk, one butterfly over the lanes reduces
// them, a few scalar steps per column give u and o in order, one more pass writes the state.
// The state is kept column-major, [slots, heads, dv, dk]: a column's rows lie together.
#include "common.cuh"

namespace {

constexpr int CHUNK = 4;              // tokens of a chunk (one in steps that bring one token per request)
constexpr int NUM = 12;               // numbers kept per token: kk [CHUNK], kq [CHUNK] (index: the earlier token), beta, padding
constexpr int LANES = 8, COLS = 16, THREADS = LANES * COLS;
constexpr int TILE = 16, STAGES = 2;  // prepared inputs: tokens staged at a time, tiles in flight or in use
constexpr int MAX_DK = 256;

__device__ __forceinline__ float softplus_of(float v) { return v > 20.0f ? v : log1pf(expf(v)); }

__device__ __forceinline__ void copy16(float* dst, const float* src, bool in) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    const int bytes = in ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void copy4(float* dst, const float* src, bool in) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    const int bytes = in ? 4 : 0;
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}

// One warp makes a chunk's vectors and numbers for one head.  q, k: the first token's raw vectors, rows ldu apart; a: its dk
// decay inputs, rows lda apart; b: its beta logit, rows ldb apart.  Tokens from cnt on read as zero vectors with decays of
// one.  Results: vec + token * vec_stride + {0, 1, 2} * width (k', q', k''), cum (P), num + token * num_stride; entries from dk
// to `padded` are zero.
template <int CH>
__device__ __forceinline__ void prepare_chunk(int cnt, const float* q, const float* k, size_t ldu, const float* a, size_t lda, const float* b, size_t ldb,
                                              const float* dt_bias, float rate, int dk, int padded, float* vec, size_t vec_stride, int width,
                                              float* cum, float* num, size_t num_stride) {
    const int lane = threadIdx.x & 31;
    float kinv[CH], qinv[CH];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        float kk = 0.0f, qq = 0.0f;
        if (c < cnt)
            for (int x = lane; x < dk; x += 32) {
                const float kv = k[c * ldu + x], qv = q[c * ldu + x];
                kk = fmaf(kv, kv, kk), qq = fmaf(qv, qv, qq);
            }
        kinv[c] = rsqrtf(warp_sum(kk) + 1e-6f), qinv[c] = rsqrtf(warp_sum(qq) + 1e-6f) * rsqrtf((float)dk);
    }
    float kk[CH][CH], kq[CH][CH];
#pragma unroll
    for (int m = 0; m < CH; ++m)
#pragma unroll
        for (int i = 0; i < CH; ++i) kk[m][i] = 0.0f, kq[m][i] = 0.0f;
    for (int x = lane; x < dk; x += 32) {
        float kc[CH], qc[CH], g[CH];
        const float bias = dt_bias[x];
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const bool live = c < cnt;
            kc[c] = live ? k[c * ldu + x] * kinv[c] : 0.0f;
            qc[c] = live ? q[c * ldu + x] * qinv[c] : 0.0f;
            g[c] = live ? expf(rate * softplus_of(a[c * lda + x] + bias)) : 1.0f;
        }
        float P = 1.0f, later = 1.0f;
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            P *= g[c];
            vec[c * vec_stride + x] = P * kc[c];
            vec[c * vec_stride + width + x] = P * qc[c];
        }
        cum[x] = P;
#pragma unroll
        for (int c = CH - 1; c >= 0; --c) {
            vec[c * vec_stride + 2 * width + x] = later * kc[c];
            later *= g[c];
        }
#pragma unroll
        for (int m = 0; m < CH; ++m) {
            float w = kc[m];                                         // k_m times the decays after token m
            kq[m][m] = fmaf(w, qc[m], kq[m][m]);
#pragma unroll
            for (int i = m + 1; i < CH; ++i) {
                w *= g[i];
                kk[m][i] = fmaf(w, kc[i], kk[m][i]);
                kq[m][i] = fmaf(w, qc[i], kq[m][i]);
            }
        }
    }
    for (int x = dk + lane; x < padded; x += 32) {
#pragma unroll
        for (int c = 0; c < CH; ++c) vec[c * vec_stride + x] = vec[c * vec_stride + width + x] = vec[c * vec_stride + 2 * width + x] = 0.0f;
        cum[x] = 0.0f;
    }
#pragma unroll
    for (int i = 0; i < CH; ++i) {
        float beta = 0.0f;
        if (lane == 0 && i < cnt) beta = 1.0f / (1.0f + expf(-b[i * ldb]));
#pragma unroll
        for (int m = 0; m < CH; ++m) {
            const float x = m < i ? warp_sum(kk[m][i]) : 0.0f, y = m <= i ? warp_sum(kq[m][i]) : 0.0f;
            if (lane == 0) num[i * num_stride + m] = x, num[i * num_stride + CHUNK + m] = y;
        }
        if (lane == 0) num[i * num_stride + 2 * CHUNK] = beta;
    }
}

// grid (T, ceil(H / 4)), a warp per head; the block of a chunk's first token does the chunk.  vec: FP32 [T, H, 4, dkp]
// (k', q', k'' of the token, and P in the row of a chunk's first token), num: FP32 [T, H, NUM]; dkp = dk rounded up to 4.
__global__ void __launch_bounds__(128) delta_channel_prepare_kernel(const float* u, int ldu, const float* p, int ldp, int b_col, const float* a, int lda,
                                                                    int a_col, const float* A_log, const float* dt_bias, const int* req_of_token,
                                                                    const int* q_start, float* vec, float* num, int H, int G, int dk, int dkp) {
    pdl_enter();
    constexpr int CH = CHUNK;
    const int t = blockIdx.x, r = req_of_token[t], i = t - q_start[r], head = blockIdx.y * 4 + (threadIdx.x >> 5);
    if (i % CH || head >= H) return;
    const int cnt = min(CH, q_start[r + 1] - t), kvh = head / (H / G);
    const float* ur = u + (size_t)t * ldu;
    float* mine = vec + ((size_t)t * H + head) * 4 * dkp;
    float* nums = num + ((size_t)t * H + head) * NUM;
    // rows of tokens beyond the portion belong to other requests: they are written for `cnt` tokens only, through a copy
    // of the arithmetic that stops there
    const float rate = -expf(A_log[head]);
    if (cnt == CH) {
        prepare_chunk<CH>(CH, ur + kvh * dk, ur + G * dk + kvh * dk, ldu, a + (size_t)t * lda + a_col + head * dk, lda, p + (size_t)t * ldp + b_col + head, ldp,
                      dt_bias + head * dk, rate, dk, dkp, mine, (size_t)H * 4 * dkp, dkp, mine + 3 * dkp, nums, (size_t)H * NUM);
        return;
    }
    // an unfinished chunk at a portion's end: its tokens beyond the end go to shared memory
    extern __shared__ float spill[];                   // per warp CH * 3 * dkp + dkp + CH * NUM floats
    float* sv = spill + (size_t)(threadIdx.x >> 5) * (CH * 3 * dkp + dkp + CH * NUM);
    float* sc = sv + CH * 3 * dkp;
    float* sn = sc + dkp;
    prepare_chunk<CH>(cnt, ur + kvh * dk, ur + G * dk + kvh * dk, ldu, a + (size_t)t * lda + a_col + head * dk, lda, p + (size_t)t * ldp + b_col + head, ldp,
                  dt_bias + head * dk, rate, dk, dkp, sv, 3 * dkp, dkp, sc, sn, NUM);
    __syncwarp();
    const int lane = threadIdx.x & 31;
    for (int c = 0; c < cnt; ++c) {
        for (int x = lane; x < dkp; x += 32)
            for (int j = 0; j < 3; ++j) mine[(size_t)c * H * 4 * dkp + j * dkp + x] = sv[(c * 3 + j) * dkp + x];
        if (lane < NUM) nums[(size_t)c * H * NUM + lane] = sn[c * NUM + lane];
    }
    for (int x = lane; x < dkp; x += 32) mine[3 * dkp + x] = sc[x];
}

// grid (H * ceil(dv / COLS), R), THREADS threads.  RPL: rows of the state per lane, a multiple of 4 (dk <= RPL LANES).
template <int RPL, int CH, bool PREPARED>
__global__ void __launch_bounds__(THREADS) delta_channel_kernel(const float* u, int ldu, const float* p, int ldp, int b_col, const float* a, int lda,
                                                                int a_col, const float* A_log, const float* dt_bias, const float* vec, const float* num,
                                                                float* state, const int* q_start, const int* slot_ids, float* o, int H, int G, int dk,
                                                                int dkp, int dv) {
    pdl_enter();
    // without prepared inputs a chunk is made and walked at a time
    constexpr int KS = RPL * LANES, TILE = PREPARED ? ::TILE : CH, STAGES = PREPARED ? ::STAGES : 1, CHUNKS = TILE / CH;
    constexpr int STAGE = TILE * 3 * KS + CHUNKS * KS + TILE * NUM + TILE * COLS;      // floats of a stage
    static_assert(TILE % CH == 0 && NUM >= 2 * CHUNK + 1 && NUM % 4 == 0 && CH <= CHUNK, "whole chunks");
    extern __shared__ __align__(16) float sm[];
    const int col_blocks = (dv + COLS - 1) / COLS;
    const int head = blockIdx.x / col_blocks, col0 = (blockIdx.x % col_blocks) * COLS, r = blockIdx.y, kvh = head / (H / G);
    const int sub = threadIdx.x % LANES, cl = threadIdx.x / LANES, col = col0 + cl, warp = threadIdx.x >> 5;
    const int first = q_start[r], n = q_start[r + 1] - first;
    if (n <= 0) return;
    const int v_at = 2 * G * dk + head * dv;
    float* mine = state + (((size_t)slot_ids[r] * H + head) * dv + (col < dv ? col : 0)) * dk;
    const bool by4 = dk % 4 == 0;
    float S[RPL];
#pragma unroll
    for (int j = 0; j < RPL / 4; ++j) {
        const int row = 4 * (sub + LANES * j);
        float4 s4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (col < dv && row < dk) {
            if (by4) {
                s4 = *reinterpret_cast<const float4*>(mine + row);
            } else {
                s4.x = mine[row];
                if (row + 1 < dk) s4.y = mine[row + 1];
                if (row + 2 < dk) s4.z = mine[row + 2];
                if (row + 3 < dk) s4.w = mine[row + 3];
            }
        }
        S[4 * j] = s4.x, S[4 * j + 1] = s4.y, S[4 * j + 2] = s4.z, S[4 * j + 3] = s4.w;
    }
    if (PREPARED) {                                   // rows beyond dk read as zero
        for (int i = threadIdx.x; i < STAGES * STAGE; i += THREADS) sm[i] = 0.0f;
        __syncthreads();
    }
    auto fetch = [&](int t0, int b) {                 // PREPARED: the tile at t0 on its way to buffer b
        const int nt = min(TILE, n - t0);
        if (nt > 0) {
            float* sv = sm + b * STAGE;
            float* sp = sv + TILE * 3 * KS;
            float* sn = sp + CHUNKS * KS;
            float* sval = sn + TILE * NUM;
            constexpr int K4 = KS / 4;                // a power of two
            const int x = threadIdx.x % K4;           // the thread's place in a row of 16-byte pieces, the same in every turn
            static_assert(THREADS % K4 == 0 || K4 % THREADS == 0, "whole rows per turn");
            const float* src = vec + ((size_t)(first + t0) * H + head) * 4 * dkp + 4 * x;
            if (K4 <= THREADS ? 4 * x < dkp : true) {
#pragma unroll
                for (int i = threadIdx.x; i < (TILE * 3 + CHUNKS) * K4; i += THREADS) {
                    const int row = i / K4, xx = K4 <= THREADS ? x : i % K4;
                    if (K4 > THREADS && 4 * xx >= dkp) continue;
                    const bool cum = row >= TILE * 3;
                    const int t = cum ? (row - TILE * 3) * CH : row / 3, j = cum ? 3 : row % 3;
                    const bool in = t < nt;
                    copy16((cum ? sp + (row - TILE * 3) * KS : sv + row * KS) + 4 * xx, in ? src + ((size_t)t * H * 4 + j) * dkp + 4 * (xx - x) : vec, in);
                }
            }
            for (int i = threadIdx.x; i < TILE * NUM / 4; i += THREADS) {
                const int t = i / (NUM / 4), x = i % (NUM / 4);
                const bool in = t < nt;
                copy16(sn + t * NUM + 4 * x, in ? num + ((size_t)(first + t0 + t) * H + head) * NUM + 4 * x : num, in);
            }
            for (int i = threadIdx.x; i < TILE * COLS; i += THREADS) {
                const int t = i / COLS, c = col0 + i % COLS;
                const bool in = t < nt && c < dv;
                copy4(sval + i, in ? u + (size_t)(first + t0 + t) * ldu + v_at + c : u, in);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (PREPARED) {
#pragma unroll
        for (int s = 0; s < STAGES - 1; ++s) fetch(s * TILE, s);
    }
    int b = 0;
    for (int t0 = 0; t0 < n; t0 += TILE) {
        const int nt = min(TILE, n - t0);
        float* sv = sm + b * STAGE;
        float* sp = sv + TILE * 3 * KS;
        float* sn = sp + CHUNKS * KS;
        float* sval = sn + TILE * NUM;
        if (PREPARED) {
            asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
            __syncthreads();                          // this tile has landed for everyone; the one before it is done with
            fetch(t0 + (STAGES - 1) * TILE, b == 0 ? STAGES - 1 : b - 1);
        } else {
            __syncthreads();
            if (warp == 0) {
                const int t = first + t0;
                const float* ur = u + (size_t)t * ldu;
                prepare_chunk<CH>(nt, ur + kvh * dk, ur + G * dk + kvh * dk, ldu, a + (size_t)t * lda + a_col + head * dk, lda,
                              p + (size_t)t * ldp + b_col + head, ldp, dt_bias + head * dk, -expf(A_log[head]), dk, KS, sv, 3 * KS, KS, sp, sn, NUM);
            }
            for (int i = threadIdx.x - 32; i >= 0 && i < nt * COLS; i += THREADS - 32) {
                const int t = i / COLS, c = col0 + i % COLS;
                sval[i] = c < dv ? u[(size_t)(first + t0 + t) * ldu + v_at + c] : 0.0f;
            }
            __syncthreads();
        }
        for (int c0 = 0; c0 < nt; c0 += CH) {
            const int cnt = min(CH, nt - c0);
            const float4* v4 = reinterpret_cast<const float4*>(sv + c0 * 3 * KS) + sub;
            float sk[CH], sq[CH];
#pragma unroll
            for (int c = 0; c < CH; ++c) sk[c] = 0.0f, sq[c] = 0.0f;
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j)
#pragma unroll
                for (int c = 0; c < CH; ++c) {
                    const float4 k4 = v4[(c * 3) * (KS / 4) + LANES * j], q4 = v4[(c * 3 + 1) * (KS / 4) + LANES * j];
                    sk[c] = fmaf(S[4 * j], k4.x, sk[c]), sk[c] = fmaf(S[4 * j + 1], k4.y, sk[c]);
                    sk[c] = fmaf(S[4 * j + 2], k4.z, sk[c]), sk[c] = fmaf(S[4 * j + 3], k4.w, sk[c]);
                    sq[c] = fmaf(S[4 * j], q4.x, sq[c]), sq[c] = fmaf(S[4 * j + 1], q4.y, sq[c]);
                    sq[c] = fmaf(S[4 * j + 2], q4.z, sq[c]), sq[c] = fmaf(S[4 * j + 3], q4.w, sq[c]);
                }
#pragma unroll
            for (int off = LANES / 2; off > 0; off >>= 1)
#pragma unroll
                for (int c = 0; c < CH; ++c) {
                    sk[c] += __shfl_xor_sync(0xffffffffu, sk[c], off);
                    sq[c] += __shfl_xor_sync(0xffffffffu, sq[c], off);
                }
            float uu[CH];
#pragma unroll
            for (int i = 0; i < CH; ++i) {
                const float* nu = sn + (c0 + i) * NUM;
                float x = sk[i], y = sq[i];
#pragma unroll
                for (int m = 0; m < i; ++m) x = fmaf(uu[m], nu[m], x), y = fmaf(uu[m], nu[CHUNK + m], y);
                uu[i] = i < cnt ? nu[2 * CHUNK] * (sval[(c0 + i) * COLS + cl] - x) : 0.0f;
                y = fmaf(uu[i], nu[CHUNK + i], y);
                if (i < cnt && sub == 0 && col < dv) o[((size_t)(first + t0 + c0 + i) * H + head) * dv + col] = y;
            }
            const float4* p4 = reinterpret_cast<const float4*>(sp + c0 / CH * KS) + sub;
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) {
                const float4 P = p4[LANES * j];
                float s0 = P.x * S[4 * j], s1 = P.y * S[4 * j + 1], s2 = P.z * S[4 * j + 2], s3 = P.w * S[4 * j + 3];
#pragma unroll
                for (int c = 0; c < CH; ++c) {
                    const float4 k4 = v4[(c * 3 + 2) * (KS / 4) + LANES * j];
                    s0 = fmaf(uu[c], k4.x, s0), s1 = fmaf(uu[c], k4.y, s1), s2 = fmaf(uu[c], k4.z, s2), s3 = fmaf(uu[c], k4.w, s3);
                }
                S[4 * j] = s0, S[4 * j + 1] = s1, S[4 * j + 2] = s2, S[4 * j + 3] = s3;
            }
        }
        if (PREPARED) b = b + 1 == STAGES ? 0 : b + 1;
    }
    if (PREPARED) asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (col >= dv) return;
#pragma unroll
    for (int j = 0; j < RPL / 4; ++j) {
        const int row = 4 * (sub + LANES * j);
        if (row >= dk) continue;
        if (by4) {
            *reinterpret_cast<float4*>(mine + row) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (row + e < dk) mine[row + e] = S[4 * j + e];
        }
    }
}

template <int RPL, int CH, bool PREPARED>
void launch_delta(dim3 grid, cudaStream_t st, const float* u, int ldu, const float* p, int ldp, int b_col, const float* a, int lda, int a_col,
                  const float* A_log, const float* dt_bias, const float* vec, const float* num, float* state, const int* q_start,
                  const int* slot_ids, float* o, int H, int G, int dk, int dkp, int dv) {
    constexpr int KS = RPL * LANES;
    constexpr int T_ = PREPARED ? TILE : CH;
    const size_t smem = (size_t)(PREPARED ? STAGES : 1) * (T_ * 3 * KS + T_ / CH * KS + T_ * NUM + T_ * COLS) * sizeof(float);
    auto kernel = delta_channel_kernel<RPL, CH, PREPARED>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    q6k_launch(kernel, grid, THREADS, smem, st, u, ldu, p, ldp, b_col, a, lda, a_col, A_log, dt_bias, vec, num, state, q_start, slot_ids, o, H, G, dk, dkp, dv);
}

}  // namespace

Q6K_API int q6k_delta_channel_max_dim() { return MAX_DK; }
// floats of scratch per token (a token's vectors and numbers) for steps with long portions
Q6K_API long long q6k_delta_channel_scratch(int H, int dk) { return (long long)H * (4 * ((dk + 3) / 4 * 4) + NUM); }

// u: FP32 [T, ldu] = [q (G heads of dk) | k | v (H heads of dv)]; p: FP32 [T, ldp] with the H beta logits from b_col; a: FP32 [T, lda]
// with the H dk decay inputs from a_col; dt_bias: FP32 [H dk]; state: FP32 [slots, H, dv, dk]; o: FP32 [T, H dv].
// scratch: null, or T * q6k_delta_channel_scratch(H, dk) floats on 16 bytes.  single: no request brings more than one token (chunks
// of one token then).
Q6K_API int q6k_delta_channel(const float* u, int ldu, const float* p, int ldp, int b_col, const float* a, int lda, int a_col, const float* A_log,
                              const float* dt_bias, float* scratch, float* state, const int* req_of_token, const int* q_start, const int* slot_ids,
                              float* o, int T_, int R, int H, int G, int dk, int dv, int single, cudaStream_t st) {
    if (R == 0 || T_ == 0) return 0;
    Q6K_REQUIRE(R > 0 && T_ > 0 && H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0, "delta_channel: bad sizes R=%d H=%d G=%d dk=%d dv=%d", R, H, G, dk, dv);
    Q6K_REQUIRE(dk <= MAX_DK, "delta_channel: keys of %d entries exceed the supported %d", dk, MAX_DK);
    Q6K_REQUIRE(R <= 65535 && (H + 3) / 4 <= 65535, "delta_channel: %d requests or %d heads exceed the grid limit", R, H);
    const int dkp = (dk + 3) / 4 * 4;
    float *vec = nullptr, *num = nullptr;
    if (scratch) {
        Q6K_REQUIRE((reinterpret_cast<uintptr_t>(scratch) & 15) == 0, "delta_channel: scratch must start on 16 bytes");
        vec = scratch, num = scratch + (size_t)T_ * H * 4 * dkp;
        const size_t smem = 4 * (size_t)(CHUNK * 3 * dkp + dkp + CHUNK * NUM) * sizeof(float);
        if (smem > 48 * 1024) cudaFuncSetAttribute(delta_channel_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        q6k_launch(delta_channel_prepare_kernel, dim3(T_, (H + 3) / 4), 128, smem, st, u, ldu, p, ldp, b_col, a, lda, a_col, A_log, dt_bias, req_of_token,
                   q_start, vec, num, H, G, dk, dkp);
        if (int rc = q6k_check_launch("delta_channel_prepare")) return rc;
    }
    const dim3 grid(H * ((dv + COLS - 1) / COLS), R);
#define DELTA_GO(R_)                                                                                                                               \
    do {                                                                                                                                           \
        if (scratch) launch_delta<R_, CHUNK, true>(grid, st, u, ldu, p, ldp, b_col, a, lda, a_col, A_log, dt_bias, vec, num, state, q_start, slot_ids, o, H, G, dk, dkp, dv); \
        else if (single) launch_delta<R_, 1, false>(grid, st, u, ldu, p, ldp, b_col, a, lda, a_col, A_log, dt_bias, vec, num, state, q_start, slot_ids, o, H, G, dk, dkp, dv); \
        else launch_delta<R_, CHUNK, false>(grid, st, u, ldu, p, ldp, b_col, a, lda, a_col, A_log, dt_bias, vec, num, state, q_start, slot_ids, o, H, G, dk, dkp, dv);     \
    } while (0)
    if (dk <= 4 * LANES) DELTA_GO(4);
    else if (dk <= 8 * LANES) DELTA_GO(8);
    else if (dk <= 16 * LANES) DELTA_GO(16);
    else DELTA_GO(MAX_DK / LANES);
#undef DELTA_GO
    return q6k_check_launch("delta_channel");
}
