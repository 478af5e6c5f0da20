// Linear recurrences whose per-request state is a matrix per head, S [d, e], and whose decay is one factor per key channel
// and token: gated linear attention, time mixing with a bonus for the current token, and the delta rule.
//
//   z = W2 low + b             [H * d], a product of low rank; what W1 h gives comes in as float32 rows `low` [T, rank], which
//                              pass tanh first where the rule says so
//   la = logsigmoid(z) / tau,  -exp(z)  or  -exp(a_log_head) softplus(z)             the decay's logarithm, never above zero
//   D_t = diag(exp(la_t))
//   add     S_t = D_t S_(t-1) + k_t v_t^T,                          o_t = S_t^T (q_t * q_scale)
//   bonus   S_t = D_t S_(t-1) + k_t v_t^T,                          o_t = (S_(t-1) + diag(u) k_t v_t^T)^T (q_t * q_scale)
//   delta   S' = D_t S_(t-1);  u_t = sigmoid(b_t) (v_t - S'^T k_t);  S_t = S' + k_t u_t^T,  o_t = S_t^T (q_t * q_scale)
//
// (gated_linear.h states the rules as the entry points take them.)  Query and key heads may be fewer than heads.
// Everything here is float32 arithmetic whatever the engine's compute type; q, k and v are read in the projection's type.
// The state lives in the request's slot, transposed: [H][e][d], so that a column's rows are consecutive.  The columns of S
// never meet, so every kernel spreads the work over (request, head, block of SANDY_MATRIX_STATE_COLS columns).
//
// Token by token (`sandy_fade_scan`): decode steps and short portions.  A warp owns four columns, a lane the rows lane,
// lane + 32, ...; the decays of the staged tokens are formed by the block itself (rank multiplications a channel), so a
// decode step is one launch.
//
// A chunk of 32 tokens at a time, in two launches.  With A_t the running sum of la inside the chunk and S0 the state
// before it,
//   o_t = (q_t exp(A_t))^T S0 + sum_{j<=t} P(t, j) v_j,   P(t, j) = sum_i q_t[i] k_j[i] exp(A_t[i] - A_j[i])
//   S   = diag(exp(A_31)) S0 + sum_j (k_j exp(A_31 - A_j)) v_j^T
// Splitting exp(A_t - A_j) into exp(A_t) exp(-A_j) would overflow where a channel fades fast, so the chunk is cut into
// four parts of 8 tokens and only exponents that are never positive are formed.  With L the running sum inside a part and
// D_r a part's whole sum: inside a part exp(L_t - L_j) is formed pair by pair; between parts r < s
// exp(L_t) * exp(D_(r+1) + .. + D_(s-1)) * exp(D_r - L_j).
// With the bonus a token reads the state before it: A_(t-1) in place of A_t for its query, and P(t, t) = sum_i q_t[i] u[i] k_t[i].
// The delta rule's u replace the v:
//   u_t = beta_t (v_t - (k_t exp(A_t))^T S0 - sum_{j<t} R(t, j) u_j),   R(t, j) = sum_i k_t[i] k_j[i] exp(A_t[i] - A_j[i])
// a unit lower triangular system with diag(beta) R below the diagonal.  It is solved for the e columns of beta v (U) and the d
// columns of beta k exp(A) (W) before the state is known; then u = U - W S0.
//   fade_chunk_prepare_kernel   one block a (chunk, head, request), all chunks side by side: P, q exp(A_t), k exp(A_31 - A_j)
//                               and exp(A_31), for the delta rule U and W, in float32
//   fade_chunk_scan_kernel      one block a (request, head, 16 columns) walks the chunks with S in shared memory; nothing
//                               that does not need the state is left in it.  The next chunk's rows come by cp.async while
//                               this one is computed.
#include "common.cuh"
#include "gated_linear.h"
#include "matrix_state.h"

namespace {

constexpr int WARPS = 4;
constexpr int CPW = 4;                                   // columns per warp
constexpr int COLS = SANDY_MATRIX_STATE_COLS;            // columns per block
static_assert(COLS == WARPS * CPW, "a block's columns are its warps' columns");
constexpr int THREADS = WARPS * 32;
constexpr int STAGE = 8;                                 // tokens staged at a time, token by token

constexpr int ADD = SANDY_FADE_ADD, BONUS = SANDY_FADE_BONUS, DELTA = SANDY_FADE_DELTA;

__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

// The decay's logarithm; `rate` is exp(a_log) of the head (softplus form).  exp(-104) is zero in float32: a channel that fades
// faster fades to nothing just the same, and sums of logarithms stay small and exact.
__device__ __forceinline__ float log_decay(const SandyFadeRule& rule, float z, float rate) {
    float la;
    if (rule.decay == SANDY_DECAY_EXP) la = -expf(z);
    else if (rule.decay == SANDY_DECAY_SOFTPLUS) la = -rate * softplus_f(z);
    else la = log_sigmoid_f(z) * rule.inv_tau;
    return fmaxf(la, -104.0f);
}

__device__ __forceinline__ void cp16(void* smem, const void* gmem, bool valid) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(gmem), "r"(bytes) : "memory");
}

// ---- token by token ------------------------------------------------------------------------------------------
// Shared memory per staged token: q [d], k [d], decay [d], v [COLS], beta (delta); then the staged tokens' rows of `low` [rank]; then,
// with w_staged, the head's columns of w2t [rank][d]: weights, on their way before the kernel in front has finished.
template <typename T, int R, int MODE>
__global__ void __launch_bounds__(THREADS)
fade_scan_kernel(const T* __restrict__ proj, int ld, int q_off, int k_off, int v_off, const float* __restrict__ low, int ld_low,
                 int rank, const float* __restrict__ w2t, const float* __restrict__ bias, const SandyFadeRule rule, float q_scale,
                 float* __restrict__ state, long long state_stride, const int* __restrict__ q_start,
                 const int* __restrict__ seq_slots, float* __restrict__ out, int ld_out, int n_heads, int d, int e, int long_from,
                 int w_staged) {
    extern __shared__ __align__(16) float stage[];
    const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * COLS;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int hq = h / (n_heads / rule.n_qk_heads);
    const int per = 3 * d + COLS + (MODE == DELTA ? 1 : 0);
    float* slow = stage + STAGE * per;                   // [STAGE][rank]
    float* sw = slow + (STAGE * rank + 3) / 4 * 4;       // [rank][d]; STAGE * per is a multiple of 4
    const int t0 = q_start[s], t1 = q_start[s + 1];
    if (long_from > 0 && t1 - t0 >= long_from) {
        pdl_wait();                                      // a kernel ends only after the one before it has
        return;
    }
    float* S = state + (long long)seq_slots[s] * state_stride + (long long)h * e * d;    // [e][d]
    if (w_staged) {
        const int pieces = d / 4;
        for (int x = threadIdx.x; x < rank * pieces; x += THREADS) {
            const int r = x / pieces, i = (x % pieces) * 4;
            cp16(sw + r * d + i, w2t + (size_t)r * n_heads * d + h * d + i, true);
        }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    const float rate = rule.decay == SANDY_DECAY_SOFTPLUS ? expf(rule.a_log[h]) : 0.0f;
    float bonus[R];
    if (MODE == BONUS)
#pragma unroll
        for (int r = 0; r < R; r++) bonus[r] = lane + 32 * r < d ? rule.bonus[h * d + lane + 32 * r] : 0.0f;
    pdl_wait();
    float st[R][CPW];
#pragma unroll
    for (int c = 0; c < CPW; c++) {
        const int col = col0 + warp * CPW + c;
#pragma unroll
        for (int r = 0; r < R; r++) {
            const int i = lane + 32 * r;
            st[r][c] = (col < e && i < d) ? S[(size_t)col * d + i] : 0.0f;
        }
    }
    for (int tc = t0; tc < t1; tc += STAGE) {
        const int n_tok = min(STAGE, t1 - tc);
        __syncthreads();
        for (int f = threadIdx.x; f < n_tok * rank; f += THREADS) {
            const float z = low[(size_t)(tc + f / rank) * ld_low + f % rank];
            slow[f] = rule.tanh_low ? tanhf(z) : z;
        }
        for (int f = threadIdx.x; f < n_tok * d; f += THREADS) {
            const int tok = f / d, i = f % d;
            const T* row = proj + (size_t)(tc + tok) * ld;
            float* dst = stage + tok * per;
            dst[i] = to_f32(row[q_off + hq * d + i]) * q_scale;
            dst[d + i] = to_f32(row[k_off + hq * d + i]);
        }
        for (int f = threadIdx.x; f < n_tok * COLS; f += THREADS) {
            const int tok = f / COLS, c = f % COLS;
            stage[tok * per + 3 * d + c] = col0 + c < e ? to_f32(proj[(size_t)(tc + tok) * ld + v_off + h * e + col0 + c]) : 0.0f;
        }
        if (MODE == DELTA && threadIdx.x < n_tok)
            stage[threadIdx.x * per + 3 * d + COLS] = sigmoid_f(rule.beta[(size_t)(tc + threadIdx.x) * rule.ld_beta + h]);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        for (int f = threadIdx.x; f < n_tok * d; f += THREADS) {      // the decays: rank multiplications each, in four sums
            const int tok = f / d, i = f % d, ch = h * d + i;
            const float* lo = slow + tok * rank;
            const float* w = w_staged ? sw + i : w2t + ch;
            const size_t pitch = w_staged ? d : (size_t)n_heads * d;
            float z[4] = {bias[ch], 0.0f, 0.0f, 0.0f};
            int r = 0;
#pragma unroll 4
            for (; r + 4 <= rank; r += 4)
#pragma unroll
                for (int c = 0; c < 4; c++) z[c] = fmaf(w[(r + c) * pitch], lo[r + c], z[c]);
            for (; r < rank; r++) z[0] = fmaf(w[r * pitch], lo[r], z[0]);
            stage[tok * per + 2 * d + i] = expf(log_decay(rule, (z[0] + z[1]) + (z[2] + z[3]), rate));
        }
        __syncthreads();
        for (int tok = 0; tok < n_tok; tok++) {
            const float* in = stage + tok * per;
            constexpr int NR = MODE == ADD ? CPW : (MODE == BONUS ? CPW + 1 : 2 * CPW + 1);
            float v[CPW], red[NR];
#pragma unroll
            for (int c = 0; c < CPW; c++) v[c] = in[3 * d + warp * CPW + c];
#pragma unroll
            for (int c = 0; c < NR; c++) red[c] = 0.0f;
#pragma unroll
            for (int r = 0; r < R; r++) {
                const int i = lane + 32 * r;
                if (i < d) {
                    const float q = in[i], k = in[d + i], a = in[2 * d + i];
                    if (MODE == BONUS) red[NR - 1] = fmaf(q * bonus[r], k, red[NR - 1]);
                    if (MODE == DELTA) red[NR - 1] = fmaf(q, k, red[NR - 1]);
#pragma unroll
                    for (int c = 0; c < CPW; c++) {
                        if (MODE == ADD) {
                            st[r][c] = fmaf(k, v[c], a * st[r][c]);
                            red[c] = fmaf(st[r][c], q, red[c]);
                        } else if (MODE == BONUS) {
                            red[c] = fmaf(st[r][c], q, red[c]);
                            st[r][c] = fmaf(k, v[c], a * st[r][c]);
                        } else {
                            st[r][c] *= a;
                            red[c] = fmaf(st[r][c], q, red[c]);
                            red[CPW + c] = fmaf(st[r][c], k, red[CPW + c]);
                        }
                    }
                }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int c = 0; c < NR; c++) red[c] += __shfl_xor_sync(0xffffffffu, red[c], o);
            if (MODE == BONUS)
#pragma unroll
                for (int c = 0; c < CPW; c++) red[c] = fmaf(red[NR - 1], v[c], red[c]);
            if (MODE == DELTA) {
                const float beta = in[3 * d + COLS];
                float u[CPW];
#pragma unroll
                for (int c = 0; c < CPW; c++) {
                    u[c] = beta * (v[c] - red[CPW + c]);
                    red[c] = fmaf(red[NR - 1], u[c], red[c]);
                }
#pragma unroll
                for (int r = 0; r < R; r++) {
                    const int i = lane + 32 * r;
                    if (i < d)
#pragma unroll
                        for (int c = 0; c < CPW; c++) st[r][c] = fmaf(in[d + i], u[c], st[r][c]);
                }
            }
            float mine = red[0];
#pragma unroll
            for (int c = 1; c < CPW; c++)
                if (lane == c) mine = red[c];
            const int col = col0 + warp * CPW + lane;
            if (lane < CPW && col < e) out[(size_t)(tc + tok) * ld_out + h * e + col] = mine;
        }
    }
    pdl_launch_dependents();
    if (t0 < t1) {
#pragma unroll
        for (int c = 0; c < CPW; c++) {
            const int col = col0 + warp * CPW + c;
#pragma unroll
            for (int r = 0; r < R; r++) {
                const int i = lane + 32 * r;
                if (col < e && i < d) S[(size_t)col * d + i] = st[r][c];
            }
        }
    }
}

// ---- chunks: what does not need the state --------------------------------------------------------------------
constexpr int CC = 32;                 // tokens per chunk
constexpr int CT = 256;                // threads
constexpr int PART = 8;                // tokens per part
constexpr int PARTS = CC / PART;
static_assert(PART == 8, "a part's tokens are two float4");
static_assert(CT == PARTS * PART * PART, "inside the parts a thread a pair");

// Place of chunk c of request s among all chunks of the step (a request brings ceil(n / CC) of them).
__device__ __forceinline__ int chunk_slot(int t0, int s, int c) { return t0 / CC + s + c; }

__device__ __forceinline__ float dot4(const float* __restrict__ x, const float* __restrict__ y, int n) {
    float a = 0.0f, b = 0.0f;
    for (int i = 0; i < n; i += 4) {
        const float4 u = *reinterpret_cast<const float4*>(x + i), v = *reinterpret_cast<const float4*>(y + i);
        a = fmaf(u.x, v.x, a);
        b = fmaf(u.y, v.y, b);
        a = fmaf(u.z, v.z, a);
        b = fmaf(u.w, v.w, b);
    }
    return a + b;
}

constexpr int LM = CC + 4;             // pitch of the triangular system's columns

// qs, ks: float32 [T, H * dp]; P: float32 [T, H * CC]; dec: float32 [slots, H * dp]; dp = d rounded up to 4, zeros behind d.
// Delta rule: W float32 [T, H * dp], U float32 [T, H * e].
template <typename T, int MODE>
__global__ void __launch_bounds__(CT, MODE == DELTA ? 2 : 3)       // left alone the triangular system takes 248 registers, one block an SM
fade_chunk_prepare_kernel(const T* __restrict__ proj, int ld, int q_off, int k_off, int v_off, const float* __restrict__ low,
                          int ld_low, int rank, const float* __restrict__ w2t, const float* __restrict__ bias,
                          const SandyFadeRule rule, float q_scale, const int* __restrict__ q_start, float* __restrict__ qs,
                          float* __restrict__ ks, float* __restrict__ P, float* __restrict__ dec, float* __restrict__ W,
                          float* __restrict__ U, int n_heads, int d, int e, int long_from) {
    extern __shared__ __align__(16) float smem[];
    const int c = blockIdx.x, h = blockIdx.y, s = blockIdx.z, tid = threadIdx.x;
    const int t0 = q_start[s], n = q_start[s + 1] - t0;
    const int hq = h / (n_heads / rule.n_qk_heads);
    const float rate = rule.decay == SANDY_DECAY_SOFTPLUS ? expf(rule.a_log[h]) : 0.0f;
    pdl_wait();
    if (n < long_from || c * CC >= n) return;
    const int tc = t0 + c * CC, n_tok = min(CC, n - c * CC);
    const int dp = (d + 3) / 4 * 4, lds = dp + 4;
    float* sq = smem;                     // [CC][lds]
    float* sk = sq + CC * lds;            // [CC][lds]
    float* sl = sk + CC * lds;            // [CC][lds]: L
    float* sp = sl + CC * lds;            // [CC][CC]
    float* slow = sp + CC * CC;           // [rank][CC]
    float* sbeta = slow + CC * rank;      // delta rule: [CC]
    float* sw = sbeta + CC;               // delta rule: [CC][lds], k exp(L)
    float* sm = sw + CC * lds;            // delta rule: [CC][LM], column j of the system: beta_t R(t, j), t > j
    const int warp = tid >> 5, lane = tid & 31;
    constexpr int NW = CT / 32;
    for (int i = lane; i < dp; i += 32)          // a warp a row of a token, all its rows of four loads on their way at once
#pragma unroll
        for (int u = 0; u < CC / NW; u++) {
            const int t = warp + u * NW;
            const bool live = t < n_tok && i < d;
            const T* row = proj + (size_t)(tc + (live ? t : 0)) * ld;
            sq[t * lds + i] = live ? to_f32(row[q_off + hq * d + i]) * q_scale : 0.0f;
            sk[t * lds + i] = live ? to_f32(row[k_off + hq * d + i]) : 0.0f;
        }
    for (int r = lane; r < rank; r += 32)
#pragma unroll
        for (int u = 0; u < CC / NW; u++) {
            const int t = warp + u * NW;
            float z = t < n_tok ? low[(size_t)(tc + t) * ld_low + r] : 0.0f;
            if (rule.tanh_low) z = tanhf(z);
            slow[r * CC + t] = z;
        }
    for (int x = tid; x < CC * CC; x += CT) sp[x] = 0.0f;
    if (MODE == DELTA && tid < CC) sbeta[tid] = tid < n_tok ? sigmoid_f(rule.beta[(size_t)(tc + tid) * rule.ld_beta + h]) : 0.0f;
    __syncthreads();
    // the decays' logarithms and their running sums inside a part: a thread a (channel, part)
    for (int x = tid; x < PARTS * dp; x += CT) {
        const int part = x / dp, i = x % dp;
        float z[PART];
        if (i < d) {
            const float b = bias[h * d + i];
#pragma unroll
            for (int t = 0; t < PART; t++) z[t] = b;
#pragma unroll 8
            for (int r = 0; r < rank; r++) {
                const float w = w2t[(size_t)r * n_heads * d + h * d + i];
                const float4 a = *reinterpret_cast<const float4*>(slow + r * CC + part * PART);
                const float4 c4 = *reinterpret_cast<const float4*>(slow + r * CC + part * PART + 4);
                z[0] = fmaf(w, a.x, z[0]); z[1] = fmaf(w, a.y, z[1]); z[2] = fmaf(w, a.z, z[2]); z[3] = fmaf(w, a.w, z[3]);
                z[4] = fmaf(w, c4.x, z[4]); z[5] = fmaf(w, c4.y, z[5]); z[6] = fmaf(w, c4.z, z[6]); z[7] = fmaf(w, c4.w, z[7]);
            }
        }
        float run = 0.0f;
#pragma unroll
        for (int t = 0; t < PART; t++) {
            if (i < d && part * PART + t < n_tok) run += log_decay(rule, z[t], rate);
            sl[(part * PART + t) * lds + i] = run;
        }
    }
    __syncthreads();
    // pairs inside a part, a thread a pair
    {
        const int part = tid / (PART * PART), tt = part * PART + (tid / PART) % PART, jj = part * PART + tid % PART;
        if (jj <= tt) {
            // a query behind the bonus sees the state before its token: its decay ends one token earlier
            const float *q = sq + tt * lds, *k = sk + jj * lds, *w = sk + tt * lds;
            const float *lt = sl + (tt - (MODE == BONUS ? 1 : 0)) * lds, *lj = sl + jj * lds;
            float a = 0.0f, r = 0.0f;
            if (jj == tt) {
                if (MODE == BONUS)
                    for (int i = 0; i < d; i++) a = fmaf(q[i] * rule.bonus[h * d + i], k[i], a);
                else a = dot4(q, k, dp);
            } else {
                for (int i = 0; i < dp; i += 4) {
                    const float4 qv = *reinterpret_cast<const float4*>(q + i), kv = *reinterpret_cast<const float4*>(k + i);
                    const float4 u = *reinterpret_cast<const float4*>(lt + i), v = *reinterpret_cast<const float4*>(lj + i);
                    const float4 f = make_float4(kv.x * expf(u.x - v.x), kv.y * expf(u.y - v.y), kv.z * expf(u.z - v.z), kv.w * expf(u.w - v.w));
                    a = fmaf(qv.x, f.x, a);
                    a = fmaf(qv.y, f.y, a);
                    a = fmaf(qv.z, f.z, a);
                    a = fmaf(qv.w, f.w, a);
                    if (MODE == DELTA) {
                        const float4 wv = *reinterpret_cast<const float4*>(w + i);
                        r = fmaf(wv.x, f.x, r);
                        r = fmaf(wv.y, f.y, r);
                        r = fmaf(wv.z, f.z, r);
                        r = fmaf(wv.w, f.w, r);
                    }
                }
                if (MODE == DELTA) sm[jj * LM + tt] = sbeta[tt] * r;
            }
            sp[tt * CC + jj] = a;
        }
    }
    __syncthreads();
    for (int t = warp; t < CC; t += NW) {                 // q exp(L), k exp(D - L)
        const int last = (t / PART) * PART + PART - 1;
        for (int i = lane; i < dp; i += 32) {
            const float l = sl[t * lds + i], k = sk[t * lds + i];
            const float lq = MODE == BONUS ? (t % PART ? sl[(t - 1) * lds + i] : 0.0f) : l;
            sq[t * lds + i] *= expf(lq);
            sk[t * lds + i] = k * expf(sl[last * lds + i] - l);
            if (MODE == DELTA) sw[t * lds + i] = k * expf(l);
        }
    }
    __syncthreads();
    // pairs between parts: the keys of earlier parts fade on by one part's sum a round
    for (int p = 1; p < PARTS; p++) {
        if (p > 1) {
            for (int i = lane; i < dp; i += 32) {         // a warp one row of every part: PART warps
                const float f = expf(sl[(p * PART - 1) * lds + i]);
                for (int r = 0; r < p - 1; r++) sk[(r * PART + warp) * lds + i] *= f;
            }
            __syncthreads();
        }
        const int keys = p * PART;
        if (tid < PART * keys) {
            const int t = p * PART + tid / keys, j = tid % keys;
            sp[t * CC + j] = dot4(sq + t * lds, sk + j * lds, dp);
            if (MODE == DELTA) sm[j * LM + t] = sbeta[t] * dot4(sw + t * lds, sk + j * lds, dp);
        }
        __syncthreads();
    }
    // out: queries as seen from the chunk's start, keys as seen from its end, the whole chunk's fading, P
    const int ldw = n_heads * dp;
    static_assert(NW == PART, "a warp writes one row of every part");
    for (int i = lane; i < dp; i += 32) {
        const float last = expf(sl[(CC - 1) * lds + i]);
        float before = 0.0f;
#pragma unroll
        for (int p = 0; p < PARTS; p++) {
            const int t = p * PART + warp;
            if (t < n_tok) {
                qs[(size_t)(tc + t) * ldw + h * dp + i] = sq[t * lds + i] * expf(before);
                const float k = sk[t * lds + i];
                ks[(size_t)(tc + t) * ldw + h * dp + i] = p < PARTS - 1 ? k * last : k;
            }
            before += sl[(p * PART + PART - 1) * lds + i];
        }
    }
    for (int i = tid; i < dp; i += CT) {
        float all = 0.0f;
#pragma unroll
        for (int p = 0; p < PARTS; p++) all += sl[(p * PART + PART - 1) * lds + i];
        dec[(size_t)chunk_slot(t0, s, c) * ldw + h * dp + i] = expf(all);
    }
    for (int x = tid; x < n_tok * CC; x += CT) P[((size_t)(tc + x / CC) * n_heads + h) * CC + x % CC] = sp[x];
    if (MODE == DELTA) {
        // The triangular system, a thread a column of the right-hand side [beta k exp(A) | beta v], the column in registers;
        // a solved row is taken out of all rows behind it at once.
        for (int x = tid; x < dp + e; x += CT) {
            float u[CC];
            if (x < dp) {
                float before = 0.0f;
#pragma unroll
                for (int p = 0; p < PARTS; p++) {
                    const float f = expf(before);
#pragma unroll
                    for (int t = 0; t < PART; t++) u[p * PART + t] = sbeta[p * PART + t] * f * sw[(p * PART + t) * lds + x];
                    before += sl[(p * PART + PART - 1) * lds + x];
                }
            } else {
                const T* v = proj + (size_t)tc * ld + v_off + h * e + (x - dp);
#pragma unroll
                for (int t = 0; t < CC; t++) {
                    u[t] = t < n_tok ? sbeta[t] * to_f32(*v) : 0.0f;
                    v += ld;
                }
            }
#pragma unroll
            for (int j = 0; j < CC - 1; j++) {
#pragma unroll
                for (int b = (j + 1) / 4; b < CC / 4; b++) {
                    const float4 m = *reinterpret_cast<const float4*>(sm + j * LM + 4 * b);
                    if (4 * b > j) u[4 * b] = fmaf(-m.x, u[j], u[4 * b]);
                    if (4 * b + 1 > j) u[4 * b + 1] = fmaf(-m.y, u[j], u[4 * b + 1]);
                    if (4 * b + 2 > j) u[4 * b + 2] = fmaf(-m.z, u[j], u[4 * b + 2]);
                    u[4 * b + 3] = fmaf(-m.w, u[j], u[4 * b + 3]);
                }
                asm volatile("" ::: "memory");       // a column's loads stay with it: hoisted, they took every register there is
            }
            float* dst = x < dp ? W + (size_t)tc * ldw + h * dp + x : U + ((size_t)tc * n_heads + h) * e + (x - dp);
            const size_t pitch = x < dp ? (size_t)ldw : (size_t)n_heads * e;
#pragma unroll
            for (int t = 0; t < CC; t++) {
                if (t < n_tok) *dst = u[t];
                dst += pitch;
            }
        }
    }
    pdl_launch_dependents();
}

// ---- chunks: the recurrence ------------------------------------------------------------------------------------
// q, k, P, dec, (delta) W; rows of q, k and W lie dp + 4 apart, so that a warp's four tokens meet different banks.
__host__ __device__ constexpr int scan_buffer_floats(int dp, bool delta) { return (delta ? 3 : 2) * CC * (dp + 4) + CC * CC + dp; }

// MAXR: rows of the state a thread owns (d <= 32 * MAXR).  With DELTA `proj` is U ([T, H * e], v_off 0) and a token's row of it
// becomes u = U - W S0 before it is used.
template <typename T, int MAXR, bool DELTA_RULE>
__global__ void __launch_bounds__(CT)
fade_chunk_scan_kernel(const T* __restrict__ proj, int ld, int v_off, const float* __restrict__ qs, const float* __restrict__ ks,
                       const float* __restrict__ P, const float* __restrict__ dec, const float* __restrict__ W,
                       float* __restrict__ state, long long state_stride, const int* __restrict__ q_start,
                       const int* __restrict__ seq_slots, float* __restrict__ out, int ld_out, int n_heads, int d, int e,
                       int long_from) {
    extern __shared__ __align__(16) float smem[];
    const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * COLS, tid = threadIdx.x;
    const int t0 = q_start[s], t1 = q_start[s + 1];
    pdl_wait();
    if (t1 - t0 < long_from) return;
    const int dp = (d + 3) / 4 * 4, lds = dp + 4, ldw = n_heads * dp, buf_floats = scan_buffer_floats(dp, DELTA_RULE);
    float* buf = smem;                              // two of (q [CC][lds], k [CC][lds], P [CC][CC], dec [dp], W [CC][lds])
    float* sv = buf + 2 * buf_floats;               // [CC][COLS]
    float* S0 = sv + CC * COLS;                     // [dp][COLS]
    float* S = state + (long long)seq_slots[s] * state_stride + (long long)h * e * d;
    for (int x = tid; x < dp * COLS; x += CT) {
        const int c = x / dp, i = x % dp;            // consecutive threads read consecutive rows of a column
        S0[i * COLS + c] = (i < d && col0 + c < e) ? S[(size_t)(col0 + c) * d + i] : 0.0f;
    }
    T pre_v[CC * COLS / CT];                         // as loaded: a conversion here would make the warp wait for it
    auto fetch = [&](int tc, int b) {                // chunk at token tc into buffer b; nothing behind the last token
        float* dst = buf + b * buf_floats;
        const int n_tok = t1 - tc, pieces = dp / 4;
        for (int x = tid; x < CC * pieces; x += CT) {
            const int t = x / pieces, i = (x % pieces) * 4;
            const bool live = t < n_tok;
            const size_t at = (size_t)(live ? tc + t : t0) * ldw + h * dp + i;
            cp16(dst + t * lds + i, qs + at, live);
            cp16(dst + CC * lds + t * lds + i, ks + at, live);
            if (DELTA_RULE) cp16(dst + 2 * CC * lds + CC * CC + dp + t * lds + i, W + at, live);
        }
        for (int x = tid; x < CC * CC / 4; x += CT) {
            const int t = x / (CC / 4), j = (x % (CC / 4)) * 4;
            const bool live = t < n_tok;
            cp16(dst + 2 * CC * lds + t * CC + j, P + ((size_t)(live ? tc + t : t0) * n_heads + h) * CC + j, live);
        }
        for (int x = tid; x < pieces; x += CT)
            cp16(dst + 2 * CC * lds + CC * CC + x * 4, dec + (size_t)chunk_slot(t0, s, n_tok > 0 ? (tc - t0) / CC : 0) * ldw + h * dp + x * 4, true);
        asm volatile("cp.async.commit_group;" ::: "memory");
#pragma unroll
        for (int u = 0; u < CC * COLS / CT; u++) {
            const int x = tid + u * CT, t = x / COLS, c = x % COLS;
            T v = from_f32<T>(0.0f);
            if (t < n_tok && col0 + c < e) v = proj[(size_t)(tc + t) * ld + v_off + h * e + col0 + c];
            pre_v[u] = v;
        }
    };
    const int ot = tid / 8, oc = (tid % 8) * 2;      // this thread's token (and first state row) and two columns
    fetch(t0, 0);
    for (int tc = t0, b = 0; tc < t1; tc += CC, b ^= 1) {
        const int n_tok = min(CC, t1 - tc);
        __syncthreads();                             // everyone is done with sv and the other buffer
#pragma unroll
        for (int u = 0; u < CC * COLS / CT; u++) sv[tid + u * CT] = to_f32(pre_v[u]);
        const bool more = tc + CC < t1;
        if (more) fetch(tc + CC, b ^ 1);
        if (more) asm volatile("cp.async.wait_group 1;" ::: "memory");
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const float* q = buf + b * buf_floats;
        const float* k = q + CC * lds;
        const float* p = k + CC * lds;
        const float* fade = p + CC * CC;
        float o[2] = {0.0f, 0.0f};
        {
            const float* qrow = q + ot * lds;
            const float* wrow = fade + dp + ot * lds;
            float ws[2] = {0.0f, 0.0f};
#pragma unroll 4
            for (int i = 0; i < dp; i += 4) {
                const float4 x = *reinterpret_cast<const float4*>(qrow + i);
                const float2 a0 = *reinterpret_cast<const float2*>(S0 + (i + 0) * COLS + oc), a1 = *reinterpret_cast<const float2*>(S0 + (i + 1) * COLS + oc);
                const float2 a2 = *reinterpret_cast<const float2*>(S0 + (i + 2) * COLS + oc), a3 = *reinterpret_cast<const float2*>(S0 + (i + 3) * COLS + oc);
                o[0] = fmaf(x.x, a0.x, o[0]); o[1] = fmaf(x.x, a0.y, o[1]);
                o[0] = fmaf(x.y, a1.x, o[0]); o[1] = fmaf(x.y, a1.y, o[1]);
                o[0] = fmaf(x.z, a2.x, o[0]); o[1] = fmaf(x.z, a2.y, o[1]);
                o[0] = fmaf(x.w, a3.x, o[0]); o[1] = fmaf(x.w, a3.y, o[1]);
                if (DELTA_RULE) {
                    const float4 y = *reinterpret_cast<const float4*>(wrow + i);
                    ws[0] = fmaf(y.x, a0.x, ws[0]); ws[1] = fmaf(y.x, a0.y, ws[1]);
                    ws[0] = fmaf(y.y, a1.x, ws[0]); ws[1] = fmaf(y.y, a1.y, ws[1]);
                    ws[0] = fmaf(y.z, a2.x, ws[0]); ws[1] = fmaf(y.z, a2.y, ws[1]);
                    ws[0] = fmaf(y.w, a3.x, ws[0]); ws[1] = fmaf(y.w, a3.y, ws[1]);
                }
            }
            if (DELTA_RULE) {                        // each thread reads and writes its own two numbers
                float2 u = *reinterpret_cast<const float2*>(sv + ot * COLS + oc);
                u.x -= ws[0]; u.y -= ws[1];
                *reinterpret_cast<float2*>(sv + ot * COLS + oc) = u;
                __syncthreads();
            }
            const float* prow = p + ot * CC;
#pragma unroll 2
            for (int j = 0; j <= ot; j += 4) {       // P is zero behind the diagonal, v behind the last token
                const float4 x = *reinterpret_cast<const float4*>(prow + j);
                const float2 a0 = *reinterpret_cast<const float2*>(sv + (j + 0) * COLS + oc), a1 = *reinterpret_cast<const float2*>(sv + (j + 1) * COLS + oc);
                const float2 a2 = *reinterpret_cast<const float2*>(sv + (j + 2) * COLS + oc), a3 = *reinterpret_cast<const float2*>(sv + (j + 3) * COLS + oc);
                o[0] = fmaf(x.x, a0.x, o[0]); o[1] = fmaf(x.x, a0.y, o[1]);
                o[0] = fmaf(x.y, a1.x, o[0]); o[1] = fmaf(x.y, a1.y, o[1]);
                o[0] = fmaf(x.z, a2.x, o[0]); o[1] = fmaf(x.z, a2.y, o[1]);
                o[0] = fmaf(x.w, a3.x, o[0]); o[1] = fmaf(x.w, a3.y, o[1]);
            }
            if (ot < n_tok)
#pragma unroll
                for (int c = 0; c < 2; c++)
                    if (col0 + oc + c < e) out[(size_t)(tc + ot) * ld_out + h * e + col0 + oc + c] = o[c];
        }
        // the state after the chunk, kept in registers until everyone has read S0
        float sn[MAXR][2];
#pragma unroll
        for (int r = 0; r < MAXR; r++) {
            const int i = ot + 32 * r;
            if (i < dp) {
                const float2 x = *reinterpret_cast<const float2*>(S0 + i * COLS + oc);
                const float f = fade[i];
                sn[r][0] = f * x.x; sn[r][1] = f * x.y;
            }
        }
#pragma unroll 8
        for (int j = 0; j < CC; j++) {               // k and v are zero behind the last token
            const float2 v = *reinterpret_cast<const float2*>(sv + j * COLS + oc);
#pragma unroll
            for (int r = 0; r < MAXR; r++) {
                const int i = ot + 32 * r;
                if (i < dp) {
                    const float x = k[j * lds + i];
                    sn[r][0] = fmaf(x, v.x, sn[r][0]); sn[r][1] = fmaf(x, v.y, sn[r][1]);
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < MAXR; r++) {
            const int i = ot + 32 * r;
            if (i < dp) *reinterpret_cast<float2*>(S0 + i * COLS + oc) = make_float2(sn[r][0], sn[r][1]);
        }
    }
    __syncthreads();
    pdl_launch_dependents();
    for (int x = tid; x < dp * COLS; x += CT) {
        const int c = x / dp, i = x % dp;
        if (i < d && col0 + c < e) S[(size_t)(col0 + c) * d + i] = S0[i * COLS + c];
    }
}

size_t prepare_smem(int d, int rank, bool delta) {
    const int dp = (d + 3) / 4 * 4;
    size_t n = (size_t)3 * CC * (dp + 4) + CC * CC + CC * rank;
    if (delta) n += (size_t)CC + CC * (dp + 4) + CC * LM;
    return n * sizeof(float);
}
size_t scan_smem(int d, bool delta) {
    const int dp = (d + 3) / 4 * 4;
    return (size_t)(2 * scan_buffer_floats(dp, delta) + CC * COLS + dp * COLS) * sizeof(float);
}

constexpr int MAX_DIM = 256, MAX_RANK = 512;

template <typename K>
int allow_smem(K kernel, size_t smem, size_t& configured) {
    if (smem <= 48 * 1024 || smem <= configured) return SANDY_OK;
    const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
    configured = smem;
    return SANDY_OK;
}

// What a rule needs beside the shapes; n_qk_heads 0 becomes as many as heads.
int check_rule(SandyFadeRule& rule, int n_heads) {
    if (rule.n_qk_heads == 0) rule.n_qk_heads = n_heads;
    if (rule.n_qk_heads < 0 || n_heads % rule.n_qk_heads) return SANDY_ERR_UNSUPPORTED;
    if (rule.kind == SANDY_FADE_BONUS ? !rule.bonus : rule.kind == SANDY_FADE_DELTA ? !rule.beta : rule.kind != SANDY_FADE_ADD)
        return SANDY_ERR_ARGUMENT;
    if (rule.decay == SANDY_DECAY_SOFTPLUS ? !rule.a_log : (rule.decay != SANDY_DECAY_EXP && rule.decay != SANDY_DECAY_LOGSIGMOID))
        return SANDY_ERR_ARGUMENT;
    return SANDY_OK;
}

// What the calls of a scan have in common.
struct FadeCall {
    const void* proj;
    int ld, q_off, k_off, v_off;
    const float* low;
    int ld_low, rank;
    const float *w2t, *bias;
    SandyFadeRule rule;
    float q_scale;
    float* state;
    long long state_stride;
    const int *q_start, *seq_slots;
    float* out;
    int ld_out, n_tokens, n_seqs, max_q_len, n_heads, d, e, long_from;
    cudaStream_t stream;
};

template <typename T, int MODE>
int scan_tokens(const FadeCall& f) {
    const dim3 grid(f.n_seqs, f.n_heads, (f.e + COLS - 1) / COLS);
    size_t smem = ((size_t)STAGE * (3 * f.d + COLS + 1) + (STAGE * f.rank + 3) / 4 * 4) * sizeof(float);
    const size_t w_bytes = (size_t)f.rank * f.d * sizeof(float);
    const int w_staged = f.d % 4 == 0 && w_bytes <= 64 * 1024 && !((uintptr_t)f.w2t & 15);
    if (w_staged) smem += w_bytes;
#define CASE(RR)                                                                                                         \
    if (f.d <= 32 * RR) {                                                                                                \
        static size_t have = 0;                                                                                          \
        if (int err = allow_smem(fade_scan_kernel<T, RR, MODE>, smem, have)) return err;                                 \
        return sandy_launch(fade_scan_kernel<T, RR, MODE>, grid, dim3(THREADS), smem, f.stream, (const T*)f.proj, f.ld,   \
                            f.q_off, f.k_off, f.v_off, f.low, f.ld_low, f.rank, f.w2t, f.bias, f.rule, f.q_scale, f.state, \
                            f.state_stride, f.q_start, f.seq_slots, f.out, f.ld_out, f.n_heads, f.d, f.e, f.long_from,    \
                            w_staged);                                                                                   \
    }
    CASE(1); CASE(2); CASE(3); CASE(4); CASE(6); CASE(8);
#undef CASE
    return SANDY_ERR_UNSUPPORTED;
}

template <typename T, int MAXR, bool DELTA_RULE>
int scan_chunks(const FadeCall& f, const T* v, int ld_v, int v_off, const float* qs, const float* ks, const float* P,
                const float* dec, const float* W) {
    static size_t have = 0;
    const size_t smem = scan_smem(f.d, DELTA_RULE);
    if (int err = allow_smem(fade_chunk_scan_kernel<T, MAXR, DELTA_RULE>, smem, have)) return err;
    return sandy_launch(fade_chunk_scan_kernel<T, MAXR, DELTA_RULE>, dim3(f.n_seqs, f.n_heads, (f.e + COLS - 1) / COLS), dim3(CT), smem,
                        f.stream, v, ld_v, v_off, qs, ks, P, dec, W, f.state, f.state_stride, f.q_start, f.seq_slots, f.out, f.ld_out,
                        f.n_heads, f.d, f.e, f.long_from);
}

template <typename T, int MODE>
int chunks(const FadeCall& f, float* scratch) {
    const long long dp = (f.d + 3) / 4 * 4, rows = (long long)f.n_tokens * f.n_heads;
    const long long slots = (long long)f.n_tokens / CC + f.n_seqs + 1;
    float* qs = scratch;
    float* ks = qs + rows * dp;
    float* P = ks + rows * dp;
    float* dec = P + rows * CC;
    float* W = dec + slots * f.n_heads * dp;
    float* U = W + rows * dp;
    const size_t smem = prepare_smem(f.d, f.rank, MODE == DELTA);
    static size_t have = 0;
    if (int err = allow_smem(fade_chunk_prepare_kernel<T, MODE>, smem, have)) return err;
    if (int err = sandy_launch(fade_chunk_prepare_kernel<T, MODE>, dim3((f.max_q_len + CC - 1) / CC, f.n_heads, f.n_seqs), dim3(CT), smem,
                               f.stream, (const T*)f.proj, f.ld, f.q_off, f.k_off, f.v_off, f.low, f.ld_low, f.rank, f.w2t, f.bias,
                               f.rule, f.q_scale, f.q_start, qs, ks, P, dec, W, U, f.n_heads, f.d, f.e, f.long_from))
        return err;
#define CASE(MAXR)                                                                                                              \
    if (f.d <= 32 * MAXR) {                                                                                                     \
        if constexpr (MODE == DELTA) return scan_chunks<float, MAXR, true>(f, U, f.n_heads * f.e, 0, qs, ks, P, dec, W);        \
        else return scan_chunks<T, MAXR, false>(f, (const T*)f.proj, f.ld, f.v_off, qs, ks, P, dec, nullptr);                   \
    }
    CASE(1); CASE(2); CASE(4); CASE(8);
#undef CASE
    return SANDY_ERR_UNSUPPORTED;
}

}  // namespace

// proj: [T, ld] of dtype with q at q_off + h * qk_dim (h a query/key head), k at k_off + h * qk_dim, v at v_off + h * v_dim; low:
// float32 [T, rank] with pitch ld_low; w2t: float32 [rank, n_heads * qk_dim]; bias: float32 [n_heads * qk_dim]; state: float32, a
// request's S [n_heads][v_dim][qk_dim] at the start of its slot; out: float32 [T, n_heads * v_dim].  Requests that bring
// `long_from` tokens or more are left to the chunked kernels (0: none are).
SANDY_API int sandy_fade_scan(const void* proj, int ld, int dtype, int q_off, int k_off, int v_off, const float* low, int ld_low,
                              int rank, const float* w2t, const float* bias, const SandyFadeRule* rule, float q_scale, float* state,
                              long long state_stride, const int* q_start, const int* seq_slots, float* out, int ld_out, int n_seqs,
                              int n_heads, int qk_dim, int v_dim, int long_from, cudaStream_t stream) {
    if (n_seqs == 0) return SANDY_OK;
    if (!proj || !low || !w2t || !bias || !rule || !state || !q_start || !seq_slots || !out) return SANDY_ERR_ARGUMENT;
    if (qk_dim <= 0 || qk_dim > MAX_DIM || v_dim <= 0 || n_heads <= 0 || rank < 1 || rank > MAX_RANK || n_heads > 65535) return SANDY_ERR_UNSUPPORTED;
    FadeCall f{proj, ld, q_off, k_off, v_off, low, ld_low, rank, w2t, bias, *rule, q_scale, state, state_stride, q_start, seq_slots,
               out, ld_out, 0, n_seqs, 0, n_heads, qk_dim, v_dim, long_from, stream};
    if (int err = check_rule(f.rule, n_heads)) return err;
#define MODES(TT)                                                                  \
    do {                                                                           \
        if (f.rule.kind == SANDY_FADE_BONUS) return scan_tokens<TT, BONUS>(f);     \
        if (f.rule.kind == SANDY_FADE_DELTA) return scan_tokens<TT, DELTA>(f);     \
        return scan_tokens<TT, ADD>(f);                                            \
    } while (0)
    if (dtype == SANDY_F32) MODES(float);
    if (dtype == SANDY_BF16) MODES(bf16);
#undef MODES
    return SANDY_ERR_UNSUPPORTED;
}

// Floats of the chunked kernels' scratch for a step of n_tokens tokens of n_seqs requests: q, k, P, the chunks' fading, and for
// the delta rule W and U.
SANDY_API long long sandy_fade_scratch_floats(int kind, int n_tokens, int n_seqs, int n_heads, int qk_dim, int v_dim) {
    const long long dp = (qk_dim + 3) / 4 * 4;
    return (long long)n_tokens * n_heads * (2 * dp + CC) + ((long long)n_tokens / CC + n_seqs + 1) * n_heads * dp +
           (kind == SANDY_FADE_DELTA ? (long long)n_tokens * n_heads * (dp + v_dim) : 0);
}

// The chunked form, two launches, for requests that bring at least `long_from` tokens; max_q_len: the step's longest
// portion.  scratch: float32, 16-byte aligned, as many floats as sandy_fade_scratch_floats says.
SANDY_API int sandy_fade_chunk_scan(const void* proj, int ld, int dtype, int q_off, int k_off, int v_off, const float* low,
                                    int ld_low, int rank, const float* w2t, const float* bias, const SandyFadeRule* rule,
                                    float q_scale, float* state, long long state_stride, const int* q_start, const int* seq_slots,
                                    float* out, int ld_out, float* scratch, int n_tokens, int n_seqs, int max_q_len, int n_heads,
                                    int qk_dim, int v_dim, int long_from, cudaStream_t stream) {
    if (n_seqs == 0 || n_tokens == 0) return SANDY_OK;
    if (!proj || !low || !w2t || !bias || !rule || !state || !q_start || !seq_slots || !out || !scratch) return SANDY_ERR_ARGUMENT;
    if (qk_dim <= 0 || qk_dim > MAX_DIM || v_dim <= 0 || n_heads <= 0 || n_heads > 65535 || n_seqs > 65535 || rank < 1 ||
        rank > MAX_RANK || long_from < 1 || ((uintptr_t)scratch & 15))
        return SANDY_ERR_UNSUPPORTED;
    FadeCall f{proj, ld, q_off, k_off, v_off, low, ld_low, rank, w2t, bias, *rule, q_scale, state, state_stride, q_start, seq_slots,
               out, ld_out, n_tokens, n_seqs, max_q_len, n_heads, qk_dim, v_dim, long_from, stream};
    if (int err = check_rule(f.rule, n_heads)) return err;
    if (prepare_smem(qk_dim, rank, f.rule.kind == SANDY_FADE_DELTA) > 227 * 1024) return SANDY_ERR_UNSUPPORTED;
#define MODES(TT)                                                                          \
    do {                                                                                   \
        if (f.rule.kind == SANDY_FADE_BONUS) return chunks<TT, BONUS>(f, scratch);         \
        if (f.rule.kind == SANDY_FADE_DELTA) return chunks<TT, DELTA>(f, scratch);         \
        return chunks<TT, ADD>(f, scratch);                                                \
    } while (0)
    if (dtype == SANDY_F32) MODES(float);
    if (dtype == SANDY_BF16) MODES(bf16);
#undef MODES
    return SANDY_ERR_UNSUPPORTED;
}

// Gated linear attention by itself: the rule `add` with decays sigmoid(z)^inv_tau.
SANDY_API int sandy_gla_scan(const void* proj, int ld, int dtype, int q_off, int k_off, int v_off, const float* low, int ld_low,
                             int rank, const float* w2t, const float* bias, float inv_tau, float q_scale, float* state,
                             long long state_stride, const int* q_start, const int* seq_slots, float* out, int ld_out, int n_seqs,
                             int n_heads, int qk_dim, int v_dim, int long_from, cudaStream_t stream) {
    SandyFadeRule rule = {};
    rule.inv_tau = inv_tau;
    return sandy_fade_scan(proj, ld, dtype, q_off, k_off, v_off, low, ld_low, rank, w2t, bias, &rule, q_scale, state, state_stride,
                           q_start, seq_slots, out, ld_out, n_seqs, n_heads, qk_dim, v_dim, long_from, stream);
}

SANDY_API long long sandy_gla_scratch_floats(int n_tokens, int n_seqs, int n_heads, int qk_dim) {
    return sandy_fade_scratch_floats(SANDY_FADE_ADD, n_tokens, n_seqs, n_heads, qk_dim, 0);
}

SANDY_API int sandy_gla_chunk_scan(const void* proj, int ld, int dtype, int q_off, int k_off, int v_off, const float* low,
                                   int ld_low, int rank, const float* w2t, const float* bias, float inv_tau, float q_scale,
                                   float* state, long long state_stride, const int* q_start, const int* seq_slots, float* out,
                                   int ld_out, float* scratch, int n_tokens, int n_seqs, int max_q_len, int n_heads, int qk_dim,
                                   int v_dim, int long_from, cudaStream_t stream) {
    SandyFadeRule rule = {};
    rule.inv_tau = inv_tau;
    return sandy_fade_chunk_scan(proj, ld, dtype, q_off, k_off, v_off, low, ld_low, rank, w2t, bias, &rule, q_scale, state,
                                 state_stride, q_start, seq_slots, out, ld_out, scratch, n_tokens, n_seqs, max_q_len, n_heads,
                                 qk_dim, v_dim, long_from, stream);
}
