// The gated delta rule with one decay per head:  S <- g S;  d = beta (v - S^T k);  S <- S + k d^T;  o = S^T q.
//
//   head_delta_prep     from the rows of one packed projection, per token: the short convolution over the channels of q, k and v
//                       and its silu, q and k as unit vectors (q also times key_dim^-1/2), beta = sigmoid(b),
//                       log g = -exp(A_log) softplus(a + dt_bias), q . k of every key head
//   head_delta_chunks   the recurrence over prompts, chunks of 64 tokens at a time.  Inside a chunk, with L_i = log g_1 + .. + log g_i and
//                       S the state before it, the writes are the rows of
//                           U = (I + M)^-1 (diag(beta) V - diag(beta e^L) K S),   M_ij = beta_i e^(L_i - L_j) k_i . k_j  (j < i),
//                       the outputs  o_i = e^(L_i) S^T q_i + sum_(j <= i) e^(L_i - L_j) (q_i . k_j) u_j,  and the state after the chunk
//                       e^(L_n) S + sum_j e^(L_n - L_j) k_j u_j^T.  What does not need the state (the two triangular systems' solutions
//                       W = (I + M)^-1 diag(beta e^L) K and (I + M)^-1 diag(beta) V, the matrix of the read-out) is made for all chunks
//                       side by side; the walk over the chunks then touches the state once a chunk instead of once a token
//   head_delta_step     steps of a few tokens (single decoded tokens above all) in one launch: all of the preparation, the
//                       recurrence, each head's RMSNorm and the gate silu(z)
//
// A step's sequences are given as in csrc/recurrent.cu: sequence s owns token rows [cu_q[s], cu_q[s+1]), its state lies in slot
// state_slots[s] (-1: none), rows beyond cu_q[n_seqs] and sequences without tokens are skipped.  A state row is
// [S (heads x key_dim x value_dim) | the convolution's last taps - 1 inputs over the channels of q, k, v, oldest first], float32.
#define LLMK_MODULE_NAME "head_delta"
#include "common.cuh"
#include <algorithm>

LLMK_DEFINE_LAST_ERROR()

constexpr int MAX_TAPS = 8;

__device__ __forceinline__ int seq_of_row(const int* __restrict__ cu_q, int n_seqs, int t) {
    if (t >= cu_q[n_seqs]) return -1;
    int lo = 0, hi = n_seqs;
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (cu_q[mid] <= t) lo = mid; else hi = mid;
    }
    return lo;
}

__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }
// The activation behind the short convolution, and the inverse lengths of q and k: with rows of bfloat16 through the special-function unit (a few units in the last place of
// a float32, far below the rounding of what went in).
template <typename T>
__device__ __forceinline__ float inverse_root(float x) {
    if constexpr (sizeof(T) == 2) return rsqrtf(x);
    else return 1.0f / sqrtf(x);
}
template <typename T>
__device__ __forceinline__ float conv_silu(float x) {
    if constexpr (sizeof(T) == 2) return __fdividef(x, 1.0f + __expf(-x));
    else return x / (1.0f + expf(-x));
}
__device__ __forceinline__ float softplusf_(float x) { return x > 20.f ? x : log1pf(expf(x)); }

struct PrepParams {
    float* qkv;              // [n_tokens, C] prepared: q, k (unit vectors), v
    float* gates;            // [n_tokens, 2 H + G]: beta, log g, q . k
    const void* x;           // packed projection [n_tokens, x_ld]: q, k, v at column 0
    long long x_ld;
    int beta_off, decay_off; // columns of b and a in it
    const float* taps;       // [C, K]
    const float* dt_bias;    // [H]
    const float* a_log;      // [H]
    float* state;            // the convolution's part of slot 0's row
    long long state_ld;
    const int* cu_q;
    const int* state_slots;
    int n_seqs, n_tokens, H, G, D, E, K;
    float unit_eps, q_scale;
};

// A block per TB token rows: a thread walks its channels over the rows with the last K - 1 inputs in registers, the convolved
// rows go through shared memory to the warps that norm the heads.
template <typename T, int TB>
__global__ void __launch_bounds__(256) head_delta_prep_kernel(PrepParams p) {
    extern __shared__ float rows[];       // [TB][C]
    __shared__ int seq[TB];
    const int C = 2 * p.G * p.D + p.H * p.E, K = p.K;
    const int t0 = blockIdx.x * TB;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const T* x = static_cast<const T*>(p.x);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x < TB) seq[threadIdx.x] = t0 + (int)threadIdx.x < p.n_tokens ? seq_of_row(p.cu_q, p.n_seqs, t0 + threadIdx.x) : -1;
    __syncthreads();
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
        float tp[MAX_TAPS], w[MAX_TAPS];
#pragma unroll
        for (int i = 0; i < MAX_TAPS; ++i) {
            tp[i] = i < K ? p.taps[(size_t)c * K + i] : 0.f;
            w[i] = 0.f;
        }
        int held = -1;                    // whose last inputs w holds
#pragma unroll
        for (int tt = 0; tt < TB; ++tt) {
            const int s = seq[tt];
            if (s < 0) continue;
            const int q_beg = p.cu_q[s], j = t0 + tt - q_beg;
            if (s != held) {
                const int slot = p.state_slots[s];
#pragma unroll
                for (int i = 0; i < MAX_TAPS - 1; ++i) {
                    if (i >= K - 1) break;
                    const int r = j - (K - 1) + i;
                    w[i] = r >= 0 ? to_float(x[(size_t)(q_beg + r) * p.x_ld + c])
                                  : slot >= 0 ? p.state[(size_t)slot * p.state_ld + (size_t)(K - 1 + r) * C + c] : 0.f;
                }
                held = s;
            }
            const float v = to_float(x[(size_t)(t0 + tt) * p.x_ld + c]);
            float acc = 0.f;
#pragma unroll
            for (int i = 0; i < MAX_TAPS; ++i) {
                if (i < K - 1) acc = fmaf(tp[i], w[i], acc);
                else if (i == K - 1) acc = fmaf(tp[i], v, acc);
            }
            rows[tt * C + c] = conv_silu<T>(acc);
#pragma unroll
            for (int i = 0; i < MAX_TAPS - 1; ++i)
                if (i < K - 1) w[i] = i + 1 < K - 1 ? w[i + 1] : v;
        }
    }
    __syncthreads();
    const int GD = p.G * p.D, HE = p.H * p.E, width = 2 * p.H + p.G;
    for (int idx = warp; idx < TB * p.G; idx += warps) {
        const int tt = idx / p.G, head = idx % p.G;
        if (seq[tt] < 0) continue;
        const float* xq = rows + tt * C + head * p.D;
        const float* xk = xq + GD;
        float sq = 0.f, sk = 0.f;
        for (int d = lane; d < p.D; d += 32) {
            sq += xq[d] * xq[d];
            sk += xk[d] * xk[d];
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        const float fq = p.q_scale / sqrtf(sq + p.unit_eps), fk = 1.0f / sqrtf(sk + p.unit_eps);
        float dot = 0.f;
        float* out = p.qkv + (size_t)(t0 + tt) * C + head * p.D;
        for (int d = lane; d < p.D; d += 32) {
            const float qv = xq[d] * fq, kv = xk[d] * fk;
            out[d] = qv;
            out[GD + d] = kv;
            dot = fmaf(qv, kv, dot);
        }
        dot = warp_sum(dot);
        if (lane == 0) p.gates[(size_t)(t0 + tt) * width + 2 * p.H + head] = dot;
    }
    for (int idx = threadIdx.x; idx < TB * HE; idx += blockDim.x) {
        const int tt = idx / HE, c = 2 * GD + idx % HE;
        if (seq[tt] >= 0) p.qkv[(size_t)(t0 + tt) * C + c] = rows[tt * C + c];
    }
    for (int idx = threadIdx.x; idx < TB * p.H; idx += blockDim.x) {
        const int tt = idx / p.H, h = idx % p.H;
        if (seq[tt] < 0) continue;
        const T* row = x + (size_t)(t0 + tt) * p.x_ld;
        float* out = p.gates + (size_t)(t0 + tt) * width;
        out[h] = sigmoidf_(to_float(row[p.beta_off + h]));
        out[p.H + h] = -expf(p.a_log[h]) * softplusf_(to_float(row[p.decay_off + h]) + p.dt_bias[h]);
    }
}

// The same where rows of q, k and v are whole vectors of four channels and a key head has at most 128 * NB of them: a warp takes one key
// head (q and k) or one value head over WTB token rows, four channels a lane (NB times), with the last KT - 1 inputs and the taps in
// registers; a convolution of fewer taps has zeros in front.
constexpr int WTB = 8;

template <typename T>
__device__ __forceinline__ float4 load_four(const T* p) {
    if constexpr (sizeof(T) == 4) return *reinterpret_cast<const float4*>(p);
    else {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
}

template <int KT>
struct ConvLane {                 // four channels of one lane
    float tp[KT][4], w[KT - 1][4];
    __device__ __forceinline__ void taps(const float* src, int K) {
        if (KT == 4 && K == 4 && aligned16(src)) {
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const float4 v = *reinterpret_cast<const float4*>(src + c * 4);
                tp[0][c] = v.x; tp[1][c] = v.y; tp[KT - 2][c] = v.z; tp[KT - 1][c] = v.w;
            }
            return;
        }
#pragma unroll
        for (int i = 0; i < KT; ++i)
#pragma unroll
            for (int c = 0; c < 4; ++c) tp[i][c] = i >= KT - K ? src[(size_t)c * K + i - (KT - K)] : 0.f;
    }
    template <typename T>
    __device__ __forceinline__ void history(const T* x, long long x_ld, int q_beg, int j, const float* st, int C, int K, size_t gc) {
#pragma unroll
        for (int i = 0; i < KT - 1; ++i) {
            const int r = j - (KT - 1) + i;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r >= 0) v = load_four(x + (size_t)(q_beg + r) * x_ld + gc);
            else if (st && r >= -(K - 1)) {
                const float* p = st + (size_t)(K - 1 + r) * C + gc;
                v = make_float4(p[0], p[1], p[2], p[3]);
            }
            w[i][0] = v.x; w[i][1] = v.y; w[i][2] = v.z; w[i][3] = v.w;
        }
    }
    template <typename T>
    __device__ __forceinline__ void next(const float4& v, float (&out)[4]) {
        const float in[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            float acc = 0.f;
#pragma unroll
            for (int i = 0; i < KT - 1; ++i) acc = fmaf(tp[i][c], w[i][c], acc);
            acc = fmaf(tp[KT - 1][c], in[c], acc);
            out[c] = conv_silu<T>(acc);
#pragma unroll
            for (int i = 0; i < KT - 1; ++i) w[i][c] = i + 1 < KT - 1 ? w[i + 1][c] : in[c];
        }
    }
};

template <typename T, int KT, int NB>
__global__ void __launch_bounds__(128, NB == 1 && KT == 4 ? 4 : 2) head_delta_prep_warp_kernel(PrepParams p, int tiles) {
    const int lane = threadIdx.x & 31;
    const int items = p.G + p.H + 1;
    const int id = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int item = id % items, t0 = id / items * WTB;
    if (id >= tiles * items) return;
    const int D = p.D, E = p.E, K = p.K, GD = p.G * D, C = 2 * GD + p.H * E, width = 2 * p.H + p.G;
    const T* x = static_cast<const T*>(p.x);
    pdl_launch_dependents();
    pdl_wait();
    const int t1 = min(t0 + WTB, min(p.n_tokens, p.cu_q[p.n_seqs]));
    if (item == p.G + p.H) {                  // beta and the decays
        for (int idx = lane; idx < (t1 - t0) * p.H; idx += 32) {
            const int t = t0 + idx / p.H, h = idx % p.H;
            const T* row = x + (size_t)t * p.x_ld;
            float* out = p.gates + (size_t)t * width;
            out[h] = sigmoidf_(to_float(row[p.beta_off + h]));
            out[p.H + h] = -expf(p.a_log[h]) * softplusf_(to_float(row[p.decay_off + h]) + p.dt_bias[h]);
        }
        return;
    }
    int held = -1, s = t0 < t1 ? seq_of_row(p.cu_q, p.n_seqs, t0) : 0;
    if (item < p.G) {
        ConvLane<KT> cq[NB], ck[NB];
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            const int d = b * 128 + lane * 4;
            if (d < D) {
                cq[b].taps(p.taps + (size_t)(item * D + d) * K, K);
                ck[b].taps(p.taps + (size_t)(GD + item * D + d) * K, K);
            }
        }
        auto begin = [&](int t) {             // the history of token t's sequence
            const int slot = p.state_slots[s], q_beg = p.cu_q[s];
            const float* st = slot >= 0 && K > 1 ? p.state + (size_t)slot * p.state_ld : nullptr;
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                const int d = b * 128 + lane * 4;
                if (d < D) {
                    cq[b].history(x, p.x_ld, q_beg, t - q_beg, st, C, K, (size_t)item * D + d);
                    ck[b].history(x, p.x_ld, q_beg, t - q_beg, st, C, K, (size_t)GD + item * D + d);
                }
            }
        };
        auto token = [&](int t, const float4 (&xq)[NB], const float4 (&xk)[NB]) {
            float q[NB][4], k[NB][4];
            float sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                if (b * 128 + lane * 4 < D) {
                    cq[b].template next<T>(xq[b], q[b]);
                    ck[b].template next<T>(xk[b], k[b]);
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        sq = fmaf(q[b][c], q[b][c], sq);
                        sk = fmaf(k[b][c], k[b][c], sk);
                        qk = fmaf(q[b][c], k[b][c], qk);
                    }
                }
            }
            sq = warp_sum(sq);
            sk = warp_sum(sk);
            qk = warp_sum(qk);
            const float fq = p.q_scale * inverse_root<T>(sq + p.unit_eps), fk = inverse_root<T>(sk + p.unit_eps);
            float* out = p.qkv + (size_t)t * C + (size_t)item * D;
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                const int d = b * 128 + lane * 4;
                if (d < D) {
                    *reinterpret_cast<float4*>(out + d) = make_float4(q[b][0] * fq, q[b][1] * fq, q[b][2] * fq, q[b][3] * fq);
                    *reinterpret_cast<float4*>(out + GD + d) = make_float4(k[b][0] * fk, k[b][1] * fk, k[b][2] * fk, k[b][3] * fk);
                }
            }
            if (lane == 0) p.gates[(size_t)t * width + 2 * p.H + item] = fq * fk * qk;
        };
        auto load = [&](int t, float4 (&xq)[NB], float4 (&xk)[NB]) {
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                const int d = b * 128 + lane * 4;
                if (d < D) {
                    const T* row = x + (size_t)t * p.x_ld + (size_t)item * D + d;
                    xq[b] = load_four(row);
                    xk[b] = load_four(row + GD);
                }
            }
        };
        if (t0 + WTB <= p.cu_q[s + 1] && t1 == t0 + WTB) {     // one sequence: all rows asked for at once
            float4 xq[WTB][NB], xk[WTB][NB];
#pragma unroll
            for (int i = 0; i < WTB; ++i) load(t0 + i, xq[i], xk[i]);
            begin(t0);
#pragma unroll
            for (int i = 0; i < WTB; ++i) token(t0 + i, xq[i], xk[i]);
            return;
        }
        for (int t = t0; t < t1; ++t) {
            while (t >= p.cu_q[s + 1]) ++s;
            if (s != held) begin(t);
            held = s;
            float4 xq[NB], xk[NB];
            load(t, xq, xk);
            token(t, xq, xk);
        }
        return;
    }
    const size_t v0 = (size_t)2 * GD + (size_t)(item - p.G) * E;
    const int s_first = s;
    for (int e0 = 0; e0 < E; e0 += 128) {      // a value head's columns need not be held together
        const int e = e0 + lane * 4;
        if (e >= E) continue;
        ConvLane<KT> cv;
        cv.taps(p.taps + (v0 + e) * K, K);
        s = s_first;
        auto begin = [&](int t) {
            const int slot = p.state_slots[s], q_beg = p.cu_q[s];
            cv.history(x, p.x_ld, q_beg, t - q_beg, slot >= 0 && K > 1 ? p.state + (size_t)slot * p.state_ld : nullptr, C, K, v0 + e);
        };
        auto token = [&](int t, const float4& in) {
            float v[4];
            cv.template next<T>(in, v);
            *reinterpret_cast<float4*>(p.qkv + (size_t)t * C + v0 + e) = make_float4(v[0], v[1], v[2], v[3]);
        };
        if (t0 + WTB <= p.cu_q[s + 1] && t1 == t0 + WTB) {
            float4 in[WTB];
#pragma unroll
            for (int i = 0; i < WTB; ++i) in[i] = load_four(x + (size_t)(t0 + i) * p.x_ld + v0 + e);
            begin(t0);
#pragma unroll
            for (int i = 0; i < WTB; ++i) token(t0 + i, in[i]);
            continue;
        }
        held = -1;
        for (int t = t0; t < t1; ++t) {
            while (t >= p.cu_q[s + 1]) ++s;
            if (s != held) begin(t);
            held = s;
            token(t, load_four(x + (size_t)t * p.x_ld + v0 + e));
        }
    }
}

// The last K - 1 inputs of every sequence into its state, behind the preparation that read the old ones.
template <typename T>
__global__ void conv_tail_kernel(PrepParams p) {
    const int s = blockIdx.y, C = 2 * p.G * p.D + p.H * p.E, K = p.K;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (c >= C) return;
    const int q_beg = p.cu_q[s], n = p.cu_q[s + 1] - q_beg, slot = p.state_slots[s];
    if (n <= 0 || slot < 0) return;
    float* st = p.state + (size_t)slot * p.state_ld + c;
    float old[MAX_TAPS];
#pragma unroll
    for (int i = 0; i < MAX_TAPS - 1; ++i) old[i] = i < K - 1 ? st[(size_t)i * C] : 0.f;
#pragma unroll
    for (int i = 0; i < MAX_TAPS - 1; ++i) {
        if (i >= K - 1) break;
        const int idx = n + i - (K - 1);
        float v = 0.f;
        if (idx >= 0) v = to_float(static_cast<const T*>(p.x)[(size_t)(q_beg + idx) * p.x_ld + c]);
        else {
#pragma unroll
            for (int o = 0; o < MAX_TAPS - 1; ++o)
                if (o == n + i) v = old[o];
        }
        st[(size_t)i * C] = v;
    }
}

template <typename T>
static cudaError_t launch_prep(const PrepParams& p, cudaStream_t s) {
    constexpr int TB = 4;
    const int C = 2 * p.G * p.D + p.H * p.E;
    const size_t smem = (size_t)TB * C * sizeof(float);
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(head_delta_prep_kernel<T, TB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    cudaError_t e;
    const bool vec = p.D % 4 == 0 && p.E % 4 == 0 && p.x_ld % 4 == 0 && (reinterpret_cast<uintptr_t>(p.x) & (4 * sizeof(T) - 1)) == 0 && host_aligned16(p.qkv);
    const int tiles = ceil_div(p.n_tokens, WTB);
    const dim3 wgrid(ceil_div(tiles * (p.G + p.H + 1), 4));
    if (vec && p.D <= 128 && p.K <= 4) e = llmk_launch(head_delta_prep_warp_kernel<T, 4, 1>, wgrid, dim3(128), 0, s, true, p, tiles);
    else if (vec && p.D <= 128) e = llmk_launch(head_delta_prep_warp_kernel<T, 8, 1>, wgrid, dim3(128), 0, s, true, p, tiles);
    else if (vec && p.D <= 256 && p.K <= 4) e = llmk_launch(head_delta_prep_warp_kernel<T, 4, 2>, wgrid, dim3(128), 0, s, true, p, tiles);
    else e = llmk_launch(head_delta_prep_kernel<T, TB>, dim3(ceil_div(p.n_tokens, TB)), dim3(256), smem, s, true, p);
    if (e == cudaSuccess && p.K > 1)
        e = llmk_launch(conv_tail_kernel<T>, dim3(ceil_div(C, 128), p.n_seqs), dim3(128), 0, s, true, p);
    return e;
}

// x: packed rows of the storage dtype; conv_state: the convolution's part of slot 0's state row (K > 1), rewritten.
LLMK_EXPORT int llmk_head_delta_prep(float* qkv, float* gates, const void* x, long long x_ld, int beta_off, int decay_off, const float* taps,
                                     const float* dt_bias, const float* a_log, float* conv_state, long long state_ld, const int* cu_q,
                                     const int* state_slots, int n_seqs, int n_tokens, int H, int G, int D, int E, int K, float unit_eps,
                                     float q_scale, int dtype, void* stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return LLMK_OK;
    if (H <= 0 || G <= 0 || H % G != 0 || D <= 0 || E <= 0) LLMK_FAIL("head_delta_prep: heads %d on %d, widths %d and %d", H, G, D, E);
    if (K < 1 || K > MAX_TAPS) LLMK_FAIL("head_delta_prep: %d taps (1 to %d are built)", K, MAX_TAPS);
    if (!qkv || !gates || !x || !taps || !dt_bias || !a_log || (!conv_state && K > 1) || !cu_q || !state_slots) LLMK_FAIL("head_delta_prep: bad arguments");
    if (((size_t)2 * G * D + (size_t)H * E) * 16 > 220 * 1024) LLMK_FAIL("head_delta_prep: rows of %d channels do not fit shared memory", 2 * G * D + H * E);
    if (n_seqs > 65535) LLMK_FAIL("head_delta_prep: %d sequences", n_seqs);
    PrepParams p = {qkv, gates, x, x_ld, beta_off, decay_off, taps, dt_bias, a_log, conv_state, state_ld, cu_q, state_slots,
                    n_seqs, n_tokens, H, G, D, E, K, unit_eps, q_scale};
    cudaError_t e;
    if (dtype == LLMK_F32) e = launch_prep<float>(p, (cudaStream_t)stream);
    else if (dtype == LLMK_BF16) e = launch_prep<bf16>(p, (cudaStream_t)stream);
    else LLMK_FAIL("head_delta_prep: unknown dtype %d", dtype);
    LLMK_CHECK_LAUNCH_RC("head_delta_prep", e);
    return LLMK_OK;
}

// ------------------------------------------------------------------------------------------------ chunks
// A chunk of a sequence has a place of its own in the scratch: chunk c of sequence s lies at cu_q[s] / CHUNK + s + c.
constexpr int CHUNK = 64;
constexpr int CTHREADS = 256;

struct ChunkParams {
    float* out;              // [n_tokens, H * E]
    const float* qkv;        // [n_tokens, C]: prepared q, k, v
    const float* gates;      // [n_tokens, 2 H + G]: beta, log g, q . k
    float* state;            // [slots, state_ld]: S [H][D][E]
    long long state_ld;
    const int* cu_q;
    const int* state_slots;
    float* qs;               // [places][G][CHUNK][DP]
    float* ks;               // [places][G][CHUNK * DP], in the order the walk's threads read it: see `key_place`
    float* w;                // [places][H][CHUNK][DP]
    float* uv;               // [places][H][CHUNK][EP]
    float* p;                // [places][H][CHUNK][CHUNK]
    float* dec;              // [places][H][2][CHUNK]: e^(L_i), e^(L_n - L_i)
    int n_seqs, n_tokens, H, G, D, E, EP, vec_ok;
};

// Where four key channels d .. d + 3 of token i lie in a chunk's keys: the walk's thread (d / 4) * TS + i % TS reads its i / TS-th
// vector there, so a warp reads 512 bytes side by side.
template <int DP>
__device__ __forceinline__ int key_place(int i, int d) {
    constexpr int TS = CTHREADS / (DP / 4);
    return (((i / TS) * (DP / 4) + d / 4) * TS + i % TS) * 4;
}

__device__ __forceinline__ unsigned long long pack2(float a, float b) {
    unsigned long long r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpack2(unsigned long long v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
// two float32 multiply-adds at a time
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
    unsigned long long r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

constexpr int CHUNK_VALUES = 128;          // columns of v that a block holds in shared memory

__device__ __forceinline__ void cp_async16(float* smem_dst, const float* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(smem_dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// Everything of one (chunk, head) that does not need the state.
template <int DP>
__global__ void __launch_bounds__(CTHREADS, 2) chunk_prep_kernel(ChunkParams p) {
    constexpr int MLD = CHUNK, TILES = CHUNK / 4, LOWER = TILES * (TILES + 1) / 2;
    extern __shared__ __align__(16) float csm[];
    float* Ks = csm;                        // [CHUNK][DP], vectors of four swizzled by the row's tile
    float* Qs = Ks + CHUNK * DP;            // the same
    float* M = Qs + CHUNK * DP;             // [CHUNK][MLD]: minus the lower triangle, zeros from the diagonal on
    float* bet = M + CHUNK * MLD;           // [CHUNK]
    float* L = bet + CHUNK;                 // [CHUNK]
    float* bel = L + CHUNK;                 // [CHUNK] beta e^L
    float* Vs = bel + CHUNK;                // [CHUNK][VC] the first columns of v
    const int place = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int kvh = h / (p.H / p.G);
    const bool writes_qk = h % (p.H / p.G) == 0;
    pdl_launch_dependents();
    pdl_wait();
    // the last sequence whose first chunk lies at or before this place
    int lo = 0, hi = p.n_seqs;
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (p.cu_q[mid] / CHUNK + mid <= place) lo = mid; else hi = mid;
    }
    const int q_beg = p.cu_q[lo], first = (place - q_beg / CHUNK - lo) * CHUNK;
    const int n = min(CHUNK, p.cu_q[lo + 1] - q_beg - first);
    if (n <= 0) return;
    const int t0 = q_beg + first;
    const int D = p.D, E = p.E, GD = p.G * D, C = 2 * GD + p.H * E;
    auto at = [](int i, int d) { return i * DP + ((((d >> 2) ^ (i >> 2)) & (DP / 4 < 8 ? DP / 4 - 1 : 7)) | ((d >> 2) & ~7)) * 4 + (d & 3); };
    float* kout = p.ks + (size_t)(place * p.G + kvh) * CHUNK * DP;
    float* qout = p.qs + (size_t)(place * p.G + kvh) * CHUNK * DP;
    const int VC = min(p.EP, CHUNK_VALUES);
    const float* vsrc = p.qkv + (size_t)t0 * C + 2 * GD + (size_t)h * E;
    for (int idx = tid; idx < CHUNK * DP / 4; idx += CTHREADS) {
        const int i = idx / (DP / 4), d = idx % (DP / 4) * 4;
        const float* row = p.qkv + (size_t)(t0 + i) * C + (size_t)kvh * D + d;
        float4 kv = make_float4(0.f, 0.f, 0.f, 0.f), qv = kv;
        if (i < n && d < D) {
            if (p.vec_ok) {
                cp_async16(Ks + at(i, d), row + GD);
                cp_async16(Qs + at(i, d), row);
                continue;
            }
            qv.x = row[0]; kv.x = row[GD];
            if (d + 1 < D) { qv.y = row[1]; kv.y = row[GD + 1]; }
            if (d + 2 < D) { qv.z = row[2]; kv.z = row[GD + 2]; }
            if (d + 3 < D) { qv.w = row[3]; kv.w = row[GD + 3]; }
        }
        *reinterpret_cast<float4*>(Ks + at(i, d)) = kv;
        *reinterpret_cast<float4*>(Qs + at(i, d)) = qv;
    }
    for (int idx = tid; idx < CHUNK * VC / 4; idx += CTHREADS) {
        const int i = idx / (VC / 4), e = idx % (VC / 4) * 4;
        if (p.vec_ok && i < n && e < E) cp_async16(Vs + i * VC + e, vsrc + (size_t)i * C + e);
        else
            for (int u = 0; u < 4; ++u) Vs[i * VC + e + u] = (i < n && e + u < E) ? vsrc[(size_t)i * C + e + u] : 0.f;
    }
    for (int idx = tid; idx < CHUNK * MLD; idx += CTHREADS) M[idx] = 0.f;
    float* P = p.p + (size_t)(place * p.H + h) * CHUNK * CHUNK;
    for (int idx = tid; idx < CHUNK * TILES; idx += CTHREADS) {      // the read-out's tiles above the diagonal
        const int i = idx / TILES, tj = idx % TILES;
        if (tj > i / 4) *reinterpret_cast<float4*>(P + i * CHUNK + tj * 4) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (tid < 32) {           // running sums of log g, two rows a lane
        const float* g0 = p.gates + (size_t)t0 * (2 * p.H + p.G);
        const int a = 2 * tid, b = a + 1, width = 2 * p.H + p.G;
        const float la = a < n ? g0[(size_t)a * width + p.H + h] : 0.f, lb = b < n ? g0[(size_t)b * width + p.H + h] : 0.f;
        bet[a] = a < n ? g0[(size_t)a * width + h] : 0.f;
        bet[b] = b < n ? g0[(size_t)b * width + h] : 0.f;
        float sum = la + lb;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, sum, o);
            if (tid >= o) sum += up;
        }
        L[a] = sum - lb;
        L[b] = sum;
        const float all = __shfl_sync(0xffffffffu, sum, 31);
        float* dec = p.dec + (size_t)(place * p.H + h) * 2 * CHUNK;
        dec[a] = expf(sum - lb);
        dec[b] = expf(sum);
        dec[CHUNK + a] = expf(all - (sum - lb));
        dec[CHUNK + b] = expf(all - sum);
        bel[a] = bet[a] * expf(sum - lb);
        bel[b] = bet[b] * expf(sum);
    }
    cp_async_wait_all();
    __syncthreads();
    if (writes_qk) {
        for (int idx = tid; idx < CHUNK * DP / 4; idx += CTHREADS) {
            const int i = idx / (DP / 4), d = idx % (DP / 4) * 4;
            *reinterpret_cast<float4*>(kout + key_place<DP>(i, d)) = *reinterpret_cast<const float4*>(Ks + at(i, d));
            *reinterpret_cast<float4*>(qout + i * DP + d) = *reinterpret_cast<const float4*>(Qs + at(i, d));
        }
    }
    // k_i . k_j, then q_i . k_j: the tiles of 4 x 4 on and below the diagonal, a thread a tile
    for (int idx = tid; idx < 2 * LOWER; idx += CTHREADS) {
        const bool read = idx >= LOWER;
        const int tile = read ? idx - LOWER : idx;
        int ti = (int)((sqrtf(8.f * tile + 1.f) - 1.f) * 0.5f);
        ti += (ti + 1) * (ti + 2) / 2 <= tile ? 1 : 0;
        ti -= ti * (ti + 1) / 2 > tile ? 1 : 0;
        const int tj = tile - ti * (ti + 1) / 2;
        const float* A = read ? Qs : Ks;
        unsigned long long acc[4][4];
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) acc[a][b] = 0ull;
#pragma unroll 2
        for (int d = 0; d < DP; d += 4) {
            ulonglong2 av[4], bv[4];
#pragma unroll
            for (int a = 0; a < 4; ++a) {
                av[a] = *reinterpret_cast<const ulonglong2*>(A + at(ti * 4 + a, d));
                bv[a] = *reinterpret_cast<const ulonglong2*>(Ks + at(tj * 4 + a, d));
            }
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
                for (int b = 0; b < 4; ++b) acc[a][b] = fma2(av[a].y, bv[b].y, fma2(av[a].x, bv[b].x, acc[a][b]));
        }
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            const int i = ti * 4 + a;
            float r[4];
#pragma unroll
            for (int b = 0; b < 4; ++b) {
                const int j = tj * 4 + b;
                const float2 two = unpack2(acc[a][b]);
                r[b] = (read ? j <= i : j < i) ? (two.x + two.y) * expf(L[i] - L[j]) : 0.f;
                if (!read) r[b] *= -bet[i];
            }
            *reinterpret_cast<float4*>((read ? P + i * CHUNK : M + i * MLD) + tj * 4) = make_float4(r[0], r[1], r[2], r[3]);
        }
    }
    __syncthreads();
    // (I + M) x = b, a column a thread, two rows of it in a register pair: the columns of diag(beta e^L) K, then those of diag(beta) V
    float* W = p.w + (size_t)(place * p.H + h) * CHUNK * DP;
    float* U = p.uv + (size_t)(place * p.H + h) * CHUNK * p.EP;
    for (int c = tid; c < DP + p.EP; c += CTHREADS) {
        const bool key = c < DP;
        const int e = c - DP;
        float* dst = key ? W + c : U + e;
        const int ld = key ? DP : p.EP;
        unsigned long long x[CHUNK / 2];
#pragma unroll
        for (int i = 0; i < CHUNK; i += 2) {
            float b0, b1;
            if (key) {
                b0 = bel[i] * Ks[at(i, c)];
                b1 = bel[i + 1] * Ks[at(i + 1, c)];
            } else if (e < VC) {
                b0 = bet[i] * Vs[i * VC + e];
                b1 = bet[i + 1] * Vs[(i + 1) * VC + e];
            } else {
                b0 = (i < n && e < E) ? bet[i] * vsrc[(size_t)i * C + e] : 0.f;
                b1 = (i + 1 < n && e < E) ? bet[i + 1] * vsrc[(size_t)(i + 1) * C + e] : 0.f;
            }
            x[i / 2] = pack2(b0, b1);
        }
#pragma unroll
        for (int i = 0; i < CHUNK; i += 2) {
            // rows i and i + 1; what lies right of the diagonal in M is zero, so whole groups of four are added
            unsigned long long p0 = 0ull, p1 = 0ull, r0 = 0ull, r1 = 0ull;
#pragma unroll
            for (int j = 0; j < i; j += 4) {
                const ulonglong2 m0 = *reinterpret_cast<const ulonglong2*>(M + i * MLD + j);
                const ulonglong2 m1 = *reinterpret_cast<const ulonglong2*>(M + (i + 1) * MLD + j);
                p0 = fma2(m0.x, x[j / 2], p0);
                r0 = fma2(m1.x, x[j / 2], r0);
                if (j + 2 < i) {
                    p1 = fma2(m0.y, x[j / 2 + 1], p1);
                    r1 = fma2(m1.y, x[j / 2 + 1], r1);
                }
            }
            const float2 b = unpack2(x[i / 2]), a0 = unpack2(p0), a1 = unpack2(p1), c0 = unpack2(r0), c1 = unpack2(r1);
            const float x0 = b.x + ((a0.x + a1.x) + (a0.y + a1.y));
            const float x1 = fmaf(M[(i + 1) * MLD + i], x0, b.y + ((c0.x + c1.x) + (c0.y + c1.y)));
            x[i / 2] = pack2(x0, x1);
            dst[(size_t)i * ld] = x0;
            dst[(size_t)(i + 1) * ld] = x1;
        }
    }
}

// The sums over LANES neighbouring lanes of N values each, scattered: lane l of the group ends with values [l * N / LANES, ...) in v[0 ..].
template <int N, int LANES>
__device__ __forceinline__ void reduce_scatter(float (&v)[N], int lane) {
    int n = N;
#pragma unroll
    for (int bit = LANES / 2; bit > 0; bit >>= 1) {
        n /= 2;
        const bool up = (lane & bit) != 0;
#pragma unroll
        for (int i = 0; i < N / 2; ++i) {
            if (i >= n) break;
            const float send = up ? v[i] : v[i + n];
            const float keep = up ? v[i + n] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
        }
    }
}

// The walk: block (sequence, head, COLS value columns), the state's columns in shared memory.  A chunk takes three steps:
//   1  rows of W and of Q times S: a thread has 4 rows, all columns, and one of 8 slices of the key channels; warps 0 .. 3 hold W's rows
//      and leave U, warps 4 .. 7 hold Q's
//   2  S <- e^(L_n) S + K^T (U scaled): a thread has 4 key channels, all columns, and one slice of the chunk's tokens
//   3  (warps 4 .. 7) the outputs: e^(L_i) times the rows of step 1 + P U
// Operands of W, Q, K and P are used by one thread each and go from global memory straight into registers, asked for a step ahead.
template <int DP, int COLS>
__global__ void __launch_bounds__(CTHREADS) chunk_scan_kernel(ChunkParams p) {
    constexpr int KR = DP / 32;                    // runs of four key channels a thread has in step 1
    constexpr int TS = CTHREADS / (DP / 4);        // slices of tokens in step 2
    constexpr int TR = CHUNK / TS;                 // tokens of one
    constexpr int SQ = 4 * COLS + 4;               // four rows of S side by side, padded: slices read different banks
    constexpr int UL = COLS + 4;                   // a row of U
    constexpr int NV = 4 * COLS;                   // outputs of a thread before the slices are summed up
    __shared__ __align__(16) float S[DP / 4 * SQ];
    __shared__ __align__(16) float U[2][CHUNK / 4 * SQ];   // as the outputs read it (four rows side by side), two chunks in turn
    __shared__ __align__(16) float Ud[CHUNK * UL];         // times e^(L_n - L_j)
    const int s = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * COLS, tid = threadIdx.x;
    const int lane = tid & 31, warp = tid >> 5;
    const int kvh = h / (p.H / p.G);
    const int ks = lane & 7, rt = warp * 4 + (lane >> 3);  // slice of key channels, row tile (0 .. 15: W, 16 .. 31: Q)
    const bool reads_out = rt >= 16;
    const int row0 = (reads_out ? rt - 16 : rt) * 4;
    const int ts = tid & (TS - 1), d0 = tid / TS * 4;
    pdl_launch_dependents();
    pdl_wait();
    const int q_beg = p.cu_q[s], n = p.cu_q[s + 1] - q_beg;
    if (n <= 0) return;
    const int slot = p.state_slots[s], D = p.D, E = p.E;
    float* st = slot >= 0 ? p.state + (size_t)slot * p.state_ld + (size_t)h * D * E : nullptr;
    for (int idx = tid; idx < DP * COLS; idx += CTHREADS) {
        const int d = idx / COLS, c = idx % COLS;
        S[(d >> 2) * SQ + (d & 3) * COLS + c] = (st && d < D && e0 + c < E) ? st[(size_t)d * E + e0 + c] : 0.f;
    }
    const int place0 = q_beg / CHUNK + s, chunks = ceil_div(n, CHUNK);
    float4 a4[4][KR], k4[TR], p4[4][2];
    auto load_rows = [&](int c) {
        const size_t place = place0 + c;
        const float* src = reads_out ? p.qs + ((place * p.G + kvh) * CHUNK + row0) * DP : p.w + ((place * p.H + h) * CHUNK + row0) * DP;
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int i = 0; i < KR; ++i) a4[r][i] = *reinterpret_cast<const float4*>(src + r * DP + i * 32 + ks * 4);
    };
    auto load_keys = [&](int c) {
        const float* src = p.ks + ((size_t)(place0 + c) * p.G + kvh) * CHUNK * DP + tid * 4;
#pragma unroll
        for (int j = 0; j < TR; ++j) k4[j] = *reinterpret_cast<const float4*>(src + j * CTHREADS * 4);
    };
    load_rows(0);
    load_keys(0);
    __syncthreads();
    for (int c = 0; c < chunks; ++c) {
        const size_t ph = (size_t)(place0 + c) * p.H + h;
        const float* dec = p.dec + ph * 2 * CHUNK;
        float v[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) v[i] = 0.f;
#pragma unroll
        for (int i = 0; i < KR; ++i) {
            const float* sr = S + (i * 8 + ks) * SQ;
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                float4 sv[COLS / 4];
#pragma unroll
                for (int u = 0; u < COLS / 4; ++u) sv[u] = *reinterpret_cast<const float4*>(sr + q * COLS + 4 * u);
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    const float w = q == 0 ? a4[r][i].x : q == 1 ? a4[r][i].y : q == 2 ? a4[r][i].z : a4[r][i].w;
#pragma unroll
                    for (int u = 0; u < COLS / 4; ++u) {
                        v[r * COLS + 4 * u] = fmaf(w, sv[u].x, v[r * COLS + 4 * u]);
                        v[r * COLS + 4 * u + 1] = fmaf(w, sv[u].y, v[r * COLS + 4 * u + 1]);
                        v[r * COLS + 4 * u + 2] = fmaf(w, sv[u].z, v[r * COLS + 4 * u + 2]);
                        v[r * COLS + 4 * u + 3] = fmaf(w, sv[u].w, v[r * COLS + 4 * u + 3]);
                    }
                }
            }
        }
        // what the slices add up to: this lane keeps NV / 8 values of one row
        constexpr int KEEP = NV / 8;
        const int at = ks * KEEP, row = row0 + at / COLS, col = at % COLS;
        float4 uv[KEEP / 4];
        if (!reads_out) {
#pragma unroll
            for (int u = 0; u < KEEP / 4; ++u) uv[u] = *reinterpret_cast<const float4*>(p.uv + (ph * CHUNK + row) * p.EP + e0 + col + 4 * u);
        }
        const float scale = reads_out ? dec[row] : dec[CHUNK + row], keep = dec[CHUNK - 1];
        reduce_scatter<NV, 8>(v, ks);
        float* ur = U[c & 1];
        if (!reads_out) {
#pragma unroll
            for (int u = 0; u < KEEP / 4; ++u) {
                const float4 x = make_float4(uv[u].x - v[4 * u], uv[u].y - v[4 * u + 1], uv[u].z - v[4 * u + 2], uv[u].w - v[4 * u + 3]);
                *reinterpret_cast<float4*>(ur + (row >> 2) * SQ + (row & 3) * COLS + col + 4 * u) = x;
                *reinterpret_cast<float4*>(Ud + row * UL + col + 4 * u) = make_float4(scale * x.x, scale * x.y, scale * x.z, scale * x.w);
            }
        }
        float o[KEEP];
#pragma unroll
        for (int i = 0; i < KEEP; ++i) o[i] = scale * v[i];
        __syncthreads();                     // U is there, and S has been read
        if (c + 1 < chunks) load_rows(c + 1);
        if (reads_out) {
            const float* src = p.p + (ph * CHUNK + row0) * CHUNK;
#pragma unroll
            for (int r = 0; r < 4; ++r)
#pragma unroll
                for (int i = 0; i < 2; ++i) p4[r][i] = *reinterpret_cast<const float4*>(src + r * CHUNK + i * 32 + ks * 4);
        }
#pragma unroll
        for (int i = 0; i < NV; ++i) v[i] = 0.f;
#pragma unroll
        for (int j = 0; j < TR; ++j) {
            float4 u4[COLS / 4];
#pragma unroll
            for (int u = 0; u < COLS / 4; ++u) u4[u] = *reinterpret_cast<const float4*>(Ud + (j * TS + ts) * UL + 4 * u);
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                const float k = r == 0 ? k4[j].x : r == 1 ? k4[j].y : r == 2 ? k4[j].z : k4[j].w;
#pragma unroll
                for (int u = 0; u < COLS / 4; ++u) {
                    v[r * COLS + 4 * u] = fmaf(k, u4[u].x, v[r * COLS + 4 * u]);
                    v[r * COLS + 4 * u + 1] = fmaf(k, u4[u].y, v[r * COLS + 4 * u + 1]);
                    v[r * COLS + 4 * u + 2] = fmaf(k, u4[u].z, v[r * COLS + 4 * u + 2]);
                    v[r * COLS + 4 * u + 3] = fmaf(k, u4[u].w, v[r * COLS + 4 * u + 3]);
                }
            }
        }
        if (c + 1 < chunks) load_keys(c + 1);
        reduce_scatter<NV, TS>(v, ts);
        {
            constexpr int KEEP2 = NV / TS;
            float* sr = S + (d0 >> 2) * SQ + ts * KEEP2;
            if (KEEP2 % 4 == 0) {
#pragma unroll
                for (int u = 0; u < KEEP2 / 4; ++u) {
                    float4 x = *reinterpret_cast<float4*>(sr + 4 * u);
                    x.x = fmaf(keep, x.x, v[4 * u]);
                    x.y = fmaf(keep, x.y, v[4 * u + 1]);
                    x.z = fmaf(keep, x.z, v[4 * u + 2]);
                    x.w = fmaf(keep, x.w, v[4 * u + 3]);
                    *reinterpret_cast<float4*>(sr + 4 * u) = x;
                }
            } else {
#pragma unroll
                for (int i = 0; i < KEEP2; ++i) sr[i] = fmaf(keep, sr[i], v[i]);
            }
        }
        __syncthreads();                     // S is the state after the chunk
        if (reads_out) {
#pragma unroll
            for (int i = 0; i < NV; ++i) v[i] = 0.f;
#pragma unroll
            for (int i = 0; i < 2; ++i) {
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const float* uj = ur + (i * 8 + ks) * SQ + q * COLS;
                    float4 u4[COLS / 4];
#pragma unroll
                    for (int u = 0; u < COLS / 4; ++u) u4[u] = *reinterpret_cast<const float4*>(uj + 4 * u);
#pragma unroll
                    for (int r = 0; r < 4; ++r) {
                        const float w = q == 0 ? p4[r][i].x : q == 1 ? p4[r][i].y : q == 2 ? p4[r][i].z : p4[r][i].w;
#pragma unroll
                        for (int u = 0; u < COLS / 4; ++u) {
                            v[r * COLS + 4 * u] = fmaf(w, u4[u].x, v[r * COLS + 4 * u]);
                            v[r * COLS + 4 * u + 1] = fmaf(w, u4[u].y, v[r * COLS + 4 * u + 1]);
                            v[r * COLS + 4 * u + 2] = fmaf(w, u4[u].z, v[r * COLS + 4 * u + 2]);
                            v[r * COLS + 4 * u + 3] = fmaf(w, u4[u].w, v[r * COLS + 4 * u + 3]);
                        }
                    }
                }
            }
            reduce_scatter<NV, 8>(v, ks);
            if (c * CHUNK + row < n) {
                float* dst = p.out + (size_t)(q_beg + c * CHUNK + row) * ((size_t)p.H * E) + (size_t)h * E + e0 + col;
#pragma unroll
                for (int i = 0; i < KEEP; ++i)
                    if (e0 + col + i < E) dst[i] = o[i] + v[i];
            }
        }
    }
    if (st) {
        for (int idx = tid; idx < DP * COLS; idx += CTHREADS) {
            const int d = idx / COLS, c = idx % COLS;
            if (d < D && e0 + c < E) st[(size_t)d * E + e0 + c] = S[(d >> 2) * SQ + (d & 3) * COLS + c];
        }
    }
}

static int chunk_width(int D) { return D <= 32 ? 32 : D <= 64 ? 64 : 128; }
static int chunk_places(int n_tokens, int n_seqs) { return n_tokens / CHUNK + std::min(n_seqs, n_tokens); }

// Floats of scratch for a step of n_tokens rows in n_seqs sequences; 0: the kernels do not take these sizes.
LLMK_EXPORT long long llmk_head_delta_chunk_floats(int n_tokens, int n_seqs, int H, int G, int D, int E) {
    if (n_tokens <= 0 || n_seqs <= 0 || D <= 0 || D > 128 || E <= 0 || H <= 0 || G <= 0) return 0;
    const long long dp = chunk_width(D), ep = ceil_div(E, 16) * 16;
    return (long long)chunk_places(n_tokens, n_seqs) * CHUNK * (2 * G * dp + H * (dp + ep + CHUNK + 2));
}

template <int DP>
static cudaError_t launch_chunks(const ChunkParams& p, int places, cudaStream_t s) {
    const size_t smem = ((size_t)2 * CHUNK * DP + CHUNK * CHUNK + 3 * CHUNK + (size_t)CHUNK * std::min(p.EP, CHUNK_VALUES)) * sizeof(float);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(chunk_prep_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             (2 * CHUNK * DP + CHUNK * CHUNK + 3 * CHUNK + CHUNK * CHUNK_VALUES) * (int)sizeof(float));
        if (e != cudaSuccess) return e;
        configured = true;
    }
    cudaError_t e = llmk_launch(chunk_prep_kernel<DP>, dim3(places, p.H), dim3(CTHREADS), smem, s, true, p);
    if (e != cudaSuccess) return e;
    // sixteen columns a block where eight would not fit the SMs side by side
    if (p.H * ceil_div(p.E, 8) <= device_sm_count())
        return llmk_launch(chunk_scan_kernel<DP, 8>, dim3(p.n_seqs, p.H, ceil_div(p.E, 8)), dim3(CTHREADS), 0, s, true, p);
    return llmk_launch(chunk_scan_kernel<DP, 16>, dim3(p.n_seqs, p.H, ceil_div(p.E, 16)), dim3(CTHREADS), 0, s, true, p);
}

// scratch: llmk_head_delta_chunk_floats(...) floats on a 16-byte boundary.  qkv and gates as `head_delta_prep` leaves them.
LLMK_EXPORT int llmk_head_delta_chunks(float* out, const float* qkv, const float* gates, float* state, long long state_ld, const int* cu_q,
                                       const int* state_slots, float* scratch, int n_seqs, int n_tokens, int H, int G, int D, int E,
                                       void* stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return LLMK_OK;
    if (H <= 0 || G <= 0 || H % G != 0) LLMK_FAIL("head_delta_chunks: %d heads are not a multiple of %d key heads", H, G);
    if (llmk_head_delta_chunk_floats(n_tokens, n_seqs, H, G, D, E) == 0) LLMK_FAIL("head_delta_chunks: key width %d (at most 128), value width %d", D, E);
    if (!out || !qkv || !gates || !state || !cu_q || !state_slots || !scratch || !host_aligned16(scratch)) LLMK_FAIL("head_delta_chunks: bad arguments");
    if (H > 65535 || ceil_div(E, 8) > 65535) LLMK_FAIL("head_delta_chunks: grid too large");
    const int places = chunk_places(n_tokens, n_seqs);
    const long long dp = chunk_width(D), ep = ceil_div(E, 16) * 16, rows = (long long)places * CHUNK;
    ChunkParams p;
    p.out = out; p.qkv = qkv; p.gates = gates; p.state = state; p.state_ld = state_ld; p.cu_q = cu_q; p.state_slots = state_slots;
    p.qs = scratch;
    p.ks = p.qs + rows * G * dp;
    p.w = p.ks + rows * G * dp;
    p.uv = p.w + rows * H * dp;
    p.p = p.uv + rows * H * ep;
    p.dec = p.p + rows * H * CHUNK;
    p.n_seqs = n_seqs; p.n_tokens = n_tokens; p.H = H; p.G = G; p.D = D; p.E = E; p.EP = (int)ep;
    p.vec_ok = (D % 4 == 0 && E % 4 == 0 && (2 * G * D + H * E) % 4 == 0 && host_aligned16(qkv)) ? 1 : 0;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e = dp == 32 ? launch_chunks<32>(p, places, s) : dp == 64 ? launch_chunks<64>(p, places, s) : launch_chunks<128>(p, places, s);
    LLMK_CHECK_LAUNCH_RC("head_delta_chunks", e);
    return LLMK_OK;
}

// ------------------------------------------------------------------------------------------------ a few tokens
// Block (head, sequence), the heads of one key head a cluster: they all read the key head's history of the convolution, and only then
// does the first of them write it anew.  The state stays in registers: thread (e, slice) holds NR rows of column e.
constexpr int STHREADS = 512;

struct StepParams {
    void* y;                 // [n_tokens, y_ld], head h at column h * E
    long long y_ld;
    PrepParams prep;         // x, its columns, taps, gates' constants, state (of the convolution), sequences, sizes; qkv and gates unused
    int gate_off;            // column of the output gate in x
    const float* norm_gain;  // [E]
    float norm_eps;
    float* state;            // [slots, state_ld]: S [H][D][E]
    int EP;                  // E rounded up to a power of two, 32 at least
};

template <typename T, int NR>
__global__ void __launch_bounds__(STHREADS) head_delta_step_kernel(StepParams sp) {
    extern __shared__ float ssm[];
    const PrepParams& p = sp.prep;
    const int D = p.D, E = p.E, K = p.K, GD = p.G * D, C = 2 * GD + p.H * E, Ch = 2 * D + E, EP = sp.EP, NS = STHREADS / EP;
    float* hist = ssm;                        // [K - 1][Ch]
    float* tap = hist + (K - 1) * Ch;         // [K][Ch]
    const int DR = NR * NS;                   // key channels with those that pad them (zeros)
    float* row = tap + K * Ch;                // [DR] q, [DR] k, [EP] v after the convolution
    row += (4 - ((2 * K - 1) * Ch & 3)) & 3;  // on 16 bytes
    float* red = row + 2 * DR + EP;           // [2][STHREADS]
    float* scal = red + 2 * STHREADS;         // |q|^2, |k|^2, q . k, beta, 1 - g, the norm's warp sums [8]
    const int h = blockIdx.x, s = blockIdx.y, R = p.H / p.G, kvh = h / R;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int e = tid & (EP - 1), sl = tid / EP;
    const T* x = static_cast<const T*>(p.x);
    auto channel = [&](int c) { return c < D ? kvh * D + c : c < 2 * D ? GD + kvh * D + c - D : 2 * GD + h * E + c - 2 * D; };
    auto place = [&](int c) { return c < D ? c : c < 2 * D ? DR + c - D : 2 * DR + c - 2 * D; };
    pdl_launch_dependents();
    for (int i = tid; i < 2 * DR + EP; i += STHREADS) row[i] = 0.f;
    // weights, before the wait for the kernel that makes x
    for (int c = tid; c < Ch; c += STHREADS) {
        const float* src = p.taps + (size_t)channel(c) * K;
        for (int i = 0; i < K; ++i) tap[i * Ch + c] = src[i];
    }
    const float gain = e < E ? sp.norm_gain[e] : 0.f, rate = -expf(p.a_log[h]), dt = p.dt_bias[h];
    pdl_wait();
    const int q_beg = p.cu_q[s], n = p.cu_q[s + 1] - q_beg, slot = p.state_slots[s];
    if (n <= 0) return;                       // the whole cluster
    float* st = slot >= 0 ? sp.state + (size_t)slot * p.state_ld + (size_t)h * D * E + e : nullptr;
    float* cst = slot >= 0 && K > 1 ? p.state + (size_t)slot * p.state_ld : nullptr;
    for (int c = tid; c < Ch; c += STHREADS) {
        const int gc = channel(c);
        for (int i = 0; i < K - 1; ++i) hist[i * Ch + c] = cst ? cst[(size_t)i * C + gc] : 0.f;
    }
    float S[NR];
    const int d0 = sl * NR, live = e < E ? min(NR, D - d0) : 0;       // rows that exist
    float* own = st ? st + (size_t)d0 * E : nullptr;
    if (own && live == NR) {
#pragma unroll
        for (int i = 0; i < NR; ++i) S[i] = own[i * E];
    } else {
#pragma unroll
        for (int i = 0; i < NR; ++i) S[i] = (own && i < live) ? own[i * E] : 0.f;
    }
    if (R > 1) cluster_sync_all();            // every head of the key head has read its history
    else __syncthreads();
    for (int j = 0; j < n; ++j) {
        const T* xr = x + (size_t)(q_beg + j) * p.x_ld;
        const float gate = (sl == 0 && e < E) ? to_float(xr[sp.gate_off + h * E + e]) : 0.f;
#pragma unroll 1
        for (int c = tid; c < Ch; c += STHREADS) {
            const float v = to_float(xr[channel(c)]);
            float acc = 0.f;
#pragma unroll 1
            for (int i = 0; i < K - 1; ++i) {
                acc = fmaf(tap[i * Ch + c], hist[i * Ch + c], acc);
                hist[i * Ch + c] = i + 1 < K - 1 ? hist[(i + 1) * Ch + c] : v;
            }
            acc = fmaf(tap[(K - 1) * Ch + c], v, acc);
            row[place(c)] = conv_silu<T>(acc);
        }
        if (warp == 3 && lane == 0) {
            scal[3] = sigmoidf_(to_float(xr[p.beta_off + h]));
            scal[4] = -expm1f(rate * softplusf_(to_float(xr[p.decay_off + h]) + dt));
        }
        __syncthreads();
        if (warp < 3) {                       // |q|^2, |k|^2, q . k
            const float* a = warp == 1 ? row + DR : row;
            const float* b = warp == 0 ? row : row + DR;
            float sum = 0.f;
            for (int d = lane; d < D; d += 32) sum = fmaf(a[d], b[d], sum);
            sum = warp_sum(sum);
            if (lane == 0) scal[warp] = sum;
        }
        const float lost = scal[4];
        float ks[4] = {0.f, 0.f, 0.f, 0.f}, qs[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < NR; i += 4) {
            const float4 k4 = *reinterpret_cast<const float4*>(row + DR + d0 + i), q4 = *reinterpret_cast<const float4*>(row + d0 + i);
            const float kv[4] = {k4.x, k4.y, k4.z, k4.w}, qv[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                S[i + u] = fmaf(-lost, S[i + u], S[i + u]);
                ks[u] = fmaf(kv[u], S[i + u], ks[u]);
                qs[u] = fmaf(qv[u], S[i + u], qs[u]);
            }
        }
        red[tid] = (ks[0] + ks[1]) + (ks[2] + ks[3]);
        red[STHREADS + tid] = (qs[0] + qs[1]) + (qs[2] + qs[3]);
        __syncthreads();
        const float fq = p.q_scale * inverse_root<T>(scal[0] + p.unit_eps), fk = inverse_root<T>(scal[1] + p.unit_eps), dot = fq * fk * scal[2], beta = scal[3];
        float kS = 0.f, qS = 0.f;
        for (int i = 0; i < NS; ++i) {
            kS += red[i * EP + e];
            qS += red[STHREADS + i * EP + e];
        }
        const float write = beta * (row[2 * DR + e] - fk * kS);      // columns beyond E: zero
        const float o = fmaf(dot, write, fq * qS), kw = fk * write;
#pragma unroll
        for (int i = 0; i < NR; i += 4) {
            const float4 k4 = *reinterpret_cast<const float4*>(row + DR + d0 + i);
            S[i] = fmaf(k4.x, kw, S[i]);
            S[i + 1] = fmaf(k4.y, kw, S[i + 1]);
            S[i + 2] = fmaf(k4.z, kw, S[i + 2]);
            S[i + 3] = fmaf(k4.w, kw, S[i + 3]);
        }
        if (sl == 0) {                        // whole warps: EP is a multiple of 32
            const float ss = warp_sum(e < E ? o * o : 0.f);
            if (lane == 0) scal[8 + warp] = ss;
        }
        __syncthreads();
        if (sl == 0 && e < E) {
            float ss = 0.f;
            for (int i = 0; i < EP / 32; ++i) ss += scal[8 + i];
            const float rinv = 1.0f / sqrtf(ss / (float)E + sp.norm_eps);
            static_cast<T*>(sp.y)[(size_t)(q_beg + j) * sp.y_ld + (size_t)h * E + e] =
                from_float<T>(o * rinv * gain * (gate * sigmoidf_(gate)));
        }
    }
    if (own && live == NR) {
#pragma unroll
        for (int i = 0; i < NR; ++i) own[i * E] = S[i];
    } else if (own) {
#pragma unroll
        for (int i = 0; i < NR; ++i)
            if (i < live) own[i * E] = S[i];
    }
    if (cst) {
        const int from = h % R == 0 ? 0 : 2 * D;          // the key head's channels are its first head's to write
        for (int c = from + tid; c < Ch; c += STHREADS) {
            const int gc = channel(c);
            for (int i = 0; i < K - 1; ++i) cst[(size_t)i * C + gc] = hist[i * Ch + c];
        }
    }
}

// Rows of the state a thread holds; 0: the kernel does not take these sizes.
static int step_rows(int H, int G, int D, int E) {
    if (D <= 0 || E <= 0 || E > 256 || G <= 0 || H % G != 0 || H / G > 8) return 0;
    int ep = 32;
    while (ep < E) ep *= 2;
    const int nr = ceil_div(D, STHREADS / ep);
    return nr > 64 ? 0 : nr;
}
LLMK_EXPORT int llmk_head_delta_step_usable(int H, int G, int D, int E) { return step_rows(H, G, D, E) > 0 ? 1 : 0; }

template <typename T>
static cudaError_t launch_step(const StepParams& p, size_t smem, int rows, cudaStream_t s) {
    const dim3 grid(p.prep.H, p.prep.n_seqs), block(STHREADS), cluster(p.prep.H / p.prep.G, 1, 1);
#define HEAD_DELTA_STEP(NR)                                                                                                        \
    do {                                                                                                                           \
        if (smem > 48 * 1024) {                                                                                                    \
            cudaError_t e = cudaFuncSetAttribute(head_delta_step_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return e;                                                                                        \
        }                                                                                                                          \
        return llmk_launch_clusters(head_delta_step_kernel<T, NR>, grid, block, smem, s, true, cluster, p);                        \
    } while (0)
    if (rows <= 4) HEAD_DELTA_STEP(4);
    if (rows <= 8) HEAD_DELTA_STEP(8);
    if (rows <= 16) HEAD_DELTA_STEP(16);
    if (rows <= 32) HEAD_DELTA_STEP(32);
    HEAD_DELTA_STEP(64);
#undef HEAD_DELTA_STEP
}

// y [n_tokens, y_ld] of the storage dtype: RMSNorm(o) * norm_gain * silu(gate) per head.  state: slot 0's S; the convolution's part of the
// row begins behind it at conv_state.  Everything else as for head_delta_prep.
LLMK_EXPORT int llmk_head_delta_step(void* y, long long y_ld, const void* x, long long x_ld, int beta_off, int decay_off, int gate_off,
                                     const float* taps, const float* dt_bias, const float* a_log, const float* norm_gain, float norm_eps,
                                     float* state, float* conv_state, long long state_ld, const int* cu_q, const int* state_slots, int n_seqs,
                                     int n_tokens, int H, int G, int D, int E, int K, float unit_eps, float q_scale, int dtype, void* stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return LLMK_OK;
    const int rows = step_rows(H, G, D, E);
    if (rows == 0) LLMK_FAIL("head_delta_step: heads %d on %d, widths %d and %d are not taken", H, G, D, E);
    if (K < 1 || K > MAX_TAPS) LLMK_FAIL("head_delta_step: %d taps (1 to %d are built)", K, MAX_TAPS);
    if (!y || !x || !taps || !dt_bias || !a_log || !norm_gain || !state || (!conv_state && K > 1) || !cu_q || !state_slots) LLMK_FAIL("head_delta_step: bad arguments");
    if (n_seqs > 65535) LLMK_FAIL("head_delta_step: %d sequences", n_seqs);
    StepParams p;
    p.y = y; p.y_ld = y_ld;
    p.prep = {nullptr, nullptr, x, x_ld, beta_off, decay_off, taps, dt_bias, a_log, conv_state, state_ld, cu_q, state_slots,
              n_seqs, n_tokens, H, G, D, E, K, unit_eps, q_scale};
    p.gate_off = gate_off; p.norm_gain = norm_gain; p.norm_eps = norm_eps; p.state = state;
    p.EP = 32;
    while (p.EP < E) p.EP *= 2;
    const int held = rows <= 4 ? 4 : rows <= 8 ? 8 : rows <= 16 ? 16 : rows <= 32 ? 32 : 64;
    const size_t smem = ((size_t)(2 * K - 1) * (2 * D + E) + 4 + 2 * held * (STHREADS / p.EP) + p.EP + 2 * STHREADS + 16) * sizeof(float);
    cudaError_t e;
    if (dtype == LLMK_F32) e = launch_step<float>(p, smem, rows, (cudaStream_t)stream);
    else if (dtype == LLMK_BF16) e = launch_step<bf16>(p, smem, rows, (cudaStream_t)stream);
    else LLMK_FAIL("head_delta_step: unknown dtype %d", dtype);
    LLMK_CHECK_LAUNCH_RC("head_delta_step", e);
    return LLMK_OK;
}
