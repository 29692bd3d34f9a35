// The gated delta rule with one decay per head:  S <- g S;  d = beta (v - S^T k);  S <- S + k d^T;  o = S^T q.
//
//   head_delta_prep     from the rows of one packed projection, per token: the short convolution over the channels of q, k and v
//                       and its silu, q and k as unit vectors (q also times key_dim^-1/2), beta = sigmoid(b),
//                       1 - g = -expm1(-exp(A_log) softplus(a + dt_bias)), q . k of every key head
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
__device__ __forceinline__ float softplusf_(float x) { return x > 20.f ? x : log1pf(expf(x)); }

struct PrepParams {
    float* qkv;              // [n_tokens, C] prepared: q, k (unit vectors), v
    float* gates;            // [n_tokens, 2 H + G]: beta, 1 - g, q . k
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
            rows[tt * C + c] = acc / (1.0f + expf(-acc));
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
        out[p.H + h] = -expm1f(-expf(p.a_log[h]) * softplusf_(to_float(row[p.decay_off + h]) + p.dt_bias[h]));
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
    cudaError_t e = llmk_launch(head_delta_prep_kernel<T, TB>, dim3(ceil_div(p.n_tokens, TB)), dim3(256), smem, s, true, p);
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
