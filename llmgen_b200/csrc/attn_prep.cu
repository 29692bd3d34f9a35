// Between the QKV projection and attention, in one pass over the packed rows:
// per-head RMSNorm of q and k, rotary position encoding of q and k, and the write of k and v
// into the paged cache at this step's slots.
//
// It replaces five launches of the reference: `rmsnorm_head_kernel` on q and on k
// (src/backend/cuda/norm/norm_final.cu:28-45), `rope_kernel` on q and on k
// (src/backend/cuda/rope/rope_v1.cu:11-45) and `store_kv_kernel`
// (src/backend/cuda/attention/attention.cu:18-33).  Those fix head_dim = 128 and at most 32
// heads; here any head_dim up to 512 that is a multiple of 2, any head counts, and a rotary
// width below the head width (src/module/rope.zig:86-88) are taken.
//
// Layouts: qkv[t] = [q heads | k heads | v heads], each head `hd` values (value heads `vd`, where that differs), row
// stride given; an optional float32 bias over the packed columns is added first (the projections' biases);
// q is normalised and rotated into `q_out` (which may be the packed rows themselves).  The packed
// rows are of the storage type T, or (splits > 0) `splits` float32 slices [splits][n][row_stride],
// `split_stride` floats apart, added in slice order: the partial sums of a projection cut along K.
// Cache arrays are [page][kv_head][page_size][hd]
// (src/memory/page_atten.zig:2) and slot = page * page_size + offset, slot < 0 = do not store.
// cos/sin tables are float32 [max_positions, rot/2], computed on the host in float64.
#define LLMK_MODULE_NAME "attn_prep"
#include "common.cuh"

LLMK_DEFINE_LAST_ERROR()

constexpr int MAX_PAIRS = 8;   // rot/2 <= 256 per lane-strided loop of 32
constexpr int MAX_TAIL = 16;   // hd - rot <= 512

template <typename T>
struct PackedRow {
    const T* x;
    const float* p;
    int splits;
    long long split_stride;
    __device__ __forceinline__ float operator[](int e) const {
        if (splits == 0) return to_float(x[e]);
        float acc = p[e];
        for (int sp = 1; sp < splits; ++sp) acc += p[(size_t)sp * split_stride + e];
        return acc;
    }
};

template <typename T>
__global__ void attn_prep_kernel(const void* __restrict__ qkv, long long row_stride, int splits, long long split_stride,
                                 T* __restrict__ q_out, long long q_stride, T* __restrict__ kcache,
                                 T* __restrict__ vcache, const int* __restrict__ positions,
                                 const int* __restrict__ slots, const float* __restrict__ cos_tab,
                                 const float* __restrict__ sin_tab, const float* __restrict__ q_gain,
                                 const float* __restrict__ k_gain, int n_tokens, int nq, int nk, int nkv_cache,
                                 int hd, int rot, int page_size, float eps, float q_off, float k_off,
                                 const float* __restrict__ bias, int vd, int interleaved, int norm_after) {
    const int lane = threadIdx.x & 31;
    const int warps_per_block = blockDim.x >> 5;
    const int heads = nq + 2 * nk;
    const long long item = (long long)blockIdx.x * warps_per_block + (threadIdx.x >> 5);
    if (item >= (long long)n_tokens * heads) return;
    const int t = (int)(item / heads);
    const int h = (int)(item % heads);
    pdl_launch_dependents();
    pdl_wait();
    // where the head's values begin in a packed row (and in the bias): value heads are `vd` wide and come last
    const size_t col0 = h < nq + nk ? (size_t)h * hd : (size_t)(nq + nk) * hd + (size_t)(h - nq - nk) * vd;
    PackedRow<T> x;
    x.x = static_cast<const T*>(qkv) + (size_t)t * row_stride + col0;
    x.p = static_cast<const float*>(qkv) + (size_t)t * row_stride + col0;
    x.splits = splits;
    x.split_stride = split_stride;
    const float* hb = bias ? bias + col0 : nullptr;
    const int slot = slots ? slots[t] : -1;

    if (h >= nq + nk) {  // a value head: copy into the cache
        if (slot < 0 || !vcache) return;
        const int kvh = h - nq - nk;
        T* dst = vcache + (((size_t)(slot / page_size) * nkv_cache + kvh) * page_size + slot % page_size) * vd;
        if (splits == 0) {
            if (hb) for (int i = lane; i < vd; i += 32) dst[i] = from_float<T>(to_float(x.x[i]) + hb[i]);
            else for (int i = lane; i < vd; i += 32) dst[i] = x.x[i];
            return;
        }
        float vv[MAX_TAIL];
#pragma unroll
        for (int i = 0; i < MAX_TAIL; ++i) vv[i] = 0.f;
#pragma unroll 4
        for (int sp = 0; sp < splits; ++sp) {
            const float* ps = x.p + (size_t)sp * split_stride;
#pragma unroll
            for (int i = 0; i < MAX_TAIL; ++i)
                if (lane + 32 * i < vd) vv[i] += __ldcg(ps + lane + 32 * i);
        }
#pragma unroll
        for (int i = 0; i < MAX_TAIL; ++i)
            if (lane + 32 * i < vd) dst[lane + 32 * i] = from_float<T>(vv[i] + (hb ? hb[lane + 32 * i] : 0.f));
        return;
    }
    const bool is_q = h < nq;
    const float* gain = is_q ? q_gain : k_gain;
    const float goff = is_q ? q_off : k_off;
    const int half = rot / 2;

    float a[MAX_PAIRS], b[MAX_PAIRS], tail[MAX_TAIL];
    float ss = 0.f;
    if (splits == 0) {
#pragma unroll
        for (int i = 0; i < MAX_PAIRS; ++i) {
            const int p = lane + 32 * i, pa = interleaved ? 2 * p : p, pb = interleaved ? 2 * p + 1 : p + half;
            if (p < half) {
                a[i] = to_float(x.x[pa]);
                b[i] = to_float(x.x[pb]);
            }
        }
#pragma unroll
        for (int i = 0; i < MAX_TAIL; ++i) {
            const int e = rot + lane + 32 * i;
            if (e < hd) tail[i] = to_float(x.x[e]);
        }
    } else {
        // partial sums: the loads of one slice are independent, slices are added in order
#pragma unroll
        for (int i = 0; i < MAX_PAIRS; ++i) a[i] = b[i] = 0.f;
#pragma unroll
        for (int i = 0; i < MAX_TAIL; ++i) tail[i] = 0.f;
#pragma unroll 4
        for (int sp = 0; sp < splits; ++sp) {
            const float* ps = x.p + (size_t)sp * split_stride;
#pragma unroll
            for (int i = 0; i < MAX_PAIRS; ++i) {
                const int p = lane + 32 * i, pa = interleaved ? 2 * p : p, pb = interleaved ? 2 * p + 1 : p + half;
                if (p < half) {
                    a[i] += __ldcg(ps + pa);
                    b[i] += __ldcg(ps + pb);
                }
            }
#pragma unroll
            for (int i = 0; i < MAX_TAIL; ++i) {
                const int e = rot + lane + 32 * i;
                if (e < hd) tail[i] += __ldcg(ps + e);
            }
        }
    }
    if (hb) {
#pragma unroll
        for (int i = 0; i < MAX_PAIRS; ++i) {
            const int p = lane + 32 * i, pa = interleaved ? 2 * p : p, pb = interleaved ? 2 * p + 1 : p + half;
            if (p < half) {
                a[i] += hb[pa];
                b[i] += hb[pb];
            }
        }
#pragma unroll
        for (int i = 0; i < MAX_TAIL; ++i) {
            const int e = rot + lane + 32 * i;
            if (e < hd) tail[i] += hb[e];
        }
    }
#pragma unroll
    for (int i = 0; i < MAX_PAIRS; ++i)
        if (lane + 32 * i < half) ss += a[i] * a[i] + b[i] * b[i];
#pragma unroll
    for (int i = 0; i < MAX_TAIL; ++i)
        if (rot + lane + 32 * i < hd) ss += tail[i] * tail[i];
    if (gain) {
        ss = warp_sum(ss);
        const float rinv = 1.0f / sqrtf(ss / (float)hd + eps);
#pragma unroll
        for (int i = 0; i < MAX_PAIRS; ++i) {
            const int p = lane + 32 * i, pa = interleaved ? 2 * p : p, pb = interleaved ? 2 * p + 1 : p + half;
            if (p < half) {
                a[i] = a[i] * rinv * (gain[pa] + goff);
                b[i] = b[i] * rinv * (gain[pb] + goff);
            }
        }
#pragma unroll
        for (int i = 0; i < MAX_TAIL; ++i) {
            const int e = rot + lane + 32 * i;
            if (e < hd) tail[i] = tail[i] * rinv * (gain[e] + goff);
        }
    }
    if (cos_tab) {
        const int pos = positions[t];
        const float* c = cos_tab + (size_t)pos * half;
        const float* s = sin_tab + (size_t)pos * half;
#pragma unroll
        for (int i = 0; i < MAX_PAIRS; ++i) {
            const int p = lane + 32 * i;
            if (p < half) {
                const float x0 = a[i], x1 = b[i], cs = c[p], sn = s[p];
                a[i] = x0 * cs - x1 * sn;
                b[i] = x1 * cs + x0 * sn;
            }
        }
    }
    if (norm_after) {
        // no gains: the rotated head divided by its root mean square
        float s2 = 0.f;
#pragma unroll
        for (int i = 0; i < MAX_PAIRS; ++i)
            if (lane + 32 * i < half) s2 += a[i] * a[i] + b[i] * b[i];
#pragma unroll
        for (int i = 0; i < MAX_TAIL; ++i)
            if (rot + lane + 32 * i < hd) s2 += tail[i] * tail[i];
        s2 = warp_sum(s2);
        const float rinv = 1.0f / sqrtf(s2 / (float)hd + eps);
#pragma unroll
        for (int i = 0; i < MAX_PAIRS; ++i) {
            a[i] *= rinv;
            b[i] *= rinv;
        }
#pragma unroll
        for (int i = 0; i < MAX_TAIL; ++i) tail[i] *= rinv;
    }
    T* dst;
    if (is_q) {
        dst = q_out + (size_t)t * q_stride + (size_t)h * hd;
    } else {
        if (slot < 0 || !kcache) return;
        const int kvh = h - nq;
        dst = kcache + (((size_t)(slot / page_size) * nkv_cache + kvh) * page_size + slot % page_size) * hd;
    }
#pragma unroll
    for (int i = 0; i < MAX_PAIRS; ++i) {
        const int p = lane + 32 * i, pa = interleaved ? 2 * p : p, pb = interleaved ? 2 * p + 1 : p + half;
        if (p < half) {
            dst[pa] = from_float<T>(a[i]);
            dst[pb] = from_float<T>(b[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < MAX_TAIL; ++i) {
        const int e = rot + lane + 32 * i;
        if (e < hd) dst[e] = from_float<T>(tail[i]);
    }
}

// The same for whole prompts, with 16-byte accesses: `LPR` lanes share one (token, head) row, each
// holding one 16-byte vector of it, so a warp works on 32 / LPR rows at a time; the rotary partner of
// a value sits LPR / 2 lanes away.  Taken when the rotary width is the head width, the rows are not
// partial sums, and everything is 16-byte aligned.
template <typename T, int LPR>
__global__ void __launch_bounds__(256)
attn_prep_vec_kernel(const T* __restrict__ qkv, long long row_stride, T* __restrict__ q_out, long long q_stride,
                     T* __restrict__ kcache, T* __restrict__ vcache, const int* __restrict__ positions,
                     const int* __restrict__ slots, const float* __restrict__ cos_tab,
                     const float* __restrict__ sin_tab, const float* __restrict__ q_gain,
                     const float* __restrict__ k_gain, int n_tokens, int nq, int nk, int nkv_cache, int hd,
                     int page_size, float eps, float q_off, float k_off) {
    constexpr int EPL = Vec16<T>::N;            // elements per lane
    constexpr int RPW = 32 / LPR;               // rows per warp
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const int sub = lane % LPR;                 // which vector of the row
    // 32-bit row numbers (the launcher refuses more rows): divisions of 64-bit numbers by `heads` were
    // a quarter of the kernel's instructions
    const unsigned heads = (unsigned)(nq + 2 * nk);
    const unsigned n_rows = (unsigned)n_tokens * heads;
    const unsigned warp_id = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const unsigned n_warps = gridDim.x * (blockDim.x >> 5);
    const int half_lanes = LPR / 2;
    const float inv_hd = 1.0f / (float)hd;
    for (unsigned row0 = warp_id * RPW; row0 < n_rows; row0 += n_warps * RPW) {
        const unsigned row = row0 + lane / LPR;
        const bool live = row < n_rows;
        const int t = live ? (int)(row / heads) : 0;
        const int h = live ? (int)(row - (unsigned)t * heads) : 0;
        const int slot = slots ? slots[t] : -1;
        const int pos = cos_tab ? positions[t] : 0;        // asked for here, with the row: its cos and sin follow it
        Vec16<T> x;
        x.raw = *reinterpret_cast<const decltype(x.raw)*>(qkv + (size_t)t * row_stride + (size_t)h * hd + sub * EPL);
        float f[EPL];
        x.unpack(f);
        const bool is_v = h >= nq + nk;
        const bool is_q = h < nq;
        const float* gain = is_q ? q_gain : k_gain;
        const float goff = is_q ? q_off : k_off;
        // every lane takes part in the shuffles, whatever kind of row it holds
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < EPL; ++i) ss += f[i] * f[i];
#pragma unroll
        for (int o = LPR / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (!is_v && gain) {
            // bfloat16 rows: the reciprocal root of the special-function unit (2 ulp, far below the rounding
            // of the result); the exact root and division are calls with slow paths that a row would wait for
            float rinv;
            if constexpr (sizeof(T) == 2) rinv = rsqrtf(fmaf(ss, inv_hd, eps));
            else rinv = 1.0f / sqrtf(ss / (float)hd + eps);
            float g[EPL];
#pragma unroll
            for (int i = 0; i < EPL; i += 4) {
                const float4 gv = *reinterpret_cast<const float4*>(gain + sub * EPL + i);
                g[i] = gv.x; g[i + 1] = gv.y; g[i + 2] = gv.z; g[i + 3] = gv.w;
            }
#pragma unroll
            for (int i = 0; i < EPL; ++i) f[i] = f[i] * rinv * (g[i] + goff);
        }
        float partner[EPL];
#pragma unroll
        for (int i = 0; i < EPL; ++i) partner[i] = __shfl_xor_sync(0xffffffffu, f[i], half_lanes);
        if (!is_v && cos_tab) {
            const int p0 = (sub % half_lanes) * EPL;          // index of the pair inside the half
            const float* c = cos_tab + (size_t)pos * (hd / 2) + p0;
            const float* sn = sin_tab + (size_t)pos * (hd / 2) + p0;
            const float sign = sub < half_lanes ? -1.f : 1.f;  // low half: x cos - y sin; high half: x cos + y sin
#pragma unroll
            for (int i = 0; i < EPL; i += 4) {
                const float4 cv = *reinterpret_cast<const float4*>(c + i);
                const float4 sv = *reinterpret_cast<const float4*>(sn + i);
                f[i] = f[i] * cv.x + sign * partner[i] * sv.x;
                f[i + 1] = f[i + 1] * cv.y + sign * partner[i + 1] * sv.y;
                f[i + 2] = f[i + 2] * cv.z + sign * partner[i + 2] * sv.z;
                f[i + 3] = f[i + 3] * cv.w + sign * partner[i + 3] * sv.w;
            }
        }
        if (!live) continue;
        T* dst = nullptr;
        if (is_q) {
            dst = q_out + (size_t)t * q_stride + (size_t)h * hd;
        } else if (slot >= 0) {
            T* cache = is_v ? vcache : kcache;
            const int kvh = is_v ? h - nq - nk : h - nq;
            const int page = slot / page_size;
            if (cache) dst = cache + (((size_t)page * nkv_cache + kvh) * page_size + (slot - page * page_size)) * hd;
        }
        if (dst) {
            Vec16<T> y;
            y.pack(f);
            *reinterpret_cast<decltype(y.raw)*>(dst + sub * EPL) = is_v ? x.raw : y.raw;
        }
    }
}

// The same, a warp taking `U` rounds of rows of ONE token at a time: position, slot, the lane's cos and
// sin values and its gains are read once for U * 32 / LPR rows (16 heads of 128 in bfloat16) instead of
// once a row, and the U loads of the rows are in flight together.
template <typename T, int LPR, int U>
__global__ void __launch_bounds__(256)
attn_prep_token_kernel(const T* __restrict__ qkv, long long row_stride, T* __restrict__ q_out, long long q_stride,
                       T* __restrict__ kcache, T* __restrict__ vcache, const int* __restrict__ positions,
                       const int* __restrict__ slots, const float* __restrict__ cos_tab,
                       const float* __restrict__ sin_tab, const float* __restrict__ q_gain,
                       const float* __restrict__ k_gain, int n_tokens, int nq, int nk, int nkv_cache, int hd,
                       int page_size, float eps, float q_off, float k_off) {
    constexpr int EPL = Vec16<T>::N;            // elements per lane
    constexpr int RPW = 32 / LPR;               // rows per round
    constexpr int RC = U * RPW;                 // rows per item
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int sub = lane % LPR;                 // which vector of the row
    const int half_lanes = LPR / 2;
    const int heads = nq + 2 * nk;
    const int chunks = (heads + RC - 1) / RC;
    const unsigned n_items = (unsigned)n_tokens * (unsigned)chunks;
    const unsigned warp_id = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const unsigned n_warps = gridDim.x * (blockDim.x >> 5);
    const float inv_hd = 1.0f / (float)hd;
    // the gains are weights: read before the wait
    float gq[EPL], gk[EPL];
#pragma unroll
    for (int i = 0; i < EPL; i += 4) {
        const float4 a = q_gain ? *reinterpret_cast<const float4*>(q_gain + sub * EPL + i) : make_float4(1.f, 1.f, 1.f, 1.f);
        const float4 b = k_gain ? *reinterpret_cast<const float4*>(k_gain + sub * EPL + i) : make_float4(1.f, 1.f, 1.f, 1.f);
        gq[i] = a.x + q_off; gq[i + 1] = a.y + q_off; gq[i + 2] = a.z + q_off; gq[i + 3] = a.w + q_off;
        gk[i] = b.x + k_off; gk[i + 1] = b.y + k_off; gk[i + 2] = b.z + k_off; gk[i + 3] = b.w + k_off;
    }
    const float sign = sub < half_lanes ? -1.f : 1.f;      // low half: x cos - y sin; high half: x cos + y sin
    pdl_wait();
    for (unsigned item = warp_id; item < n_items; item += n_warps) {
        const int t = (int)(item / (unsigned)chunks);
        const int h0 = (int)(item - (unsigned)t * (unsigned)chunks) * RC + lane / LPR;
        const T* src = qkv + (size_t)t * row_stride + sub * EPL;
        Vec16<T> x[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int h = h0 + u * RPW;
            if (h < heads) x[u].raw = *reinterpret_cast<const decltype(x[u].raw)*>(src + (size_t)h * hd);
            else x[u].raw = decltype(x[u].raw){};
        }
        const int slot = slots ? slots[t] : -1;
        float cv[EPL], sv[EPL];
        if (cos_tab) {
            const int pos = positions[t];
            const int p0 = (sub % half_lanes) * EPL;          // index of the pair inside the half
            const float* c = cos_tab + (size_t)pos * (hd / 2) + p0;
            const float* sn = sin_tab + (size_t)pos * (hd / 2) + p0;
#pragma unroll
            for (int i = 0; i < EPL; i += 4) {
                const float4 a = *reinterpret_cast<const float4*>(c + i);
                const float4 b = *reinterpret_cast<const float4*>(sn + i);
                cv[i] = a.x; cv[i + 1] = a.y; cv[i + 2] = a.z; cv[i + 3] = a.w;
                sv[i] = sign * b.x; sv[i + 1] = sign * b.y; sv[i + 2] = sign * b.z; sv[i + 3] = sign * b.w;
            }
        }
        const int page = slot >= 0 ? slot / page_size : 0;
        const int in_page = slot - page * page_size;
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int h = h0 + u * RPW;
            const bool live = h < heads;
            const bool is_q = h < nq;
            const bool is_v = h >= nq + nk;
            float f[EPL];
            x[u].unpack(f);
            // every lane takes part in the shuffles, whatever kind of row it holds
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < EPL; ++i) ss += f[i] * f[i];
#pragma unroll
            for (int o = LPR / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            if (!is_v && (is_q ? q_gain != nullptr : k_gain != nullptr)) {
                float rinv;
                if constexpr (sizeof(T) == 2) rinv = rsqrtf(fmaf(ss, inv_hd, eps));
                else rinv = 1.0f / sqrtf(ss / (float)hd + eps);
#pragma unroll
                for (int i = 0; i < EPL; ++i) f[i] = f[i] * rinv * (is_q ? gq[i] : gk[i]);
            }
            float partner[EPL];
#pragma unroll
            for (int i = 0; i < EPL; ++i) partner[i] = __shfl_xor_sync(0xffffffffu, f[i], half_lanes);
            if (!is_v && cos_tab) {
#pragma unroll
                for (int i = 0; i < EPL; ++i) f[i] = f[i] * cv[i] + partner[i] * sv[i];
            }
            if (!live) continue;
            T* dst = nullptr;
            if (is_q) {
                dst = q_out + (size_t)t * q_stride + (size_t)h * hd;
            } else if (slot >= 0) {
                T* cache = is_v ? vcache : kcache;
                const int kvh = is_v ? h - nq - nk : h - nq;
                if (cache) dst = cache + (((size_t)page * nkv_cache + kvh) * page_size + in_page) * hd;
            }
            if (dst) {
                Vec16<T> y;
                y.pack(f);
                *reinterpret_cast<decltype(y.raw)*>(dst + sub * EPL) = is_v ? x[u].raw : y.raw;
            }
        }
    }
}

static bool g_prep_by_token = true;
LLMK_EXPORT void llmk_attn_prep_set_by_token(int on) { g_prep_by_token = on != 0; }

template <typename T>
static bool launch_vec(const void* qkv, long long row_stride, void* q_out, long long q_stride, void* kcache, void* vcache,
                       const int* positions, const int* slots, const float* cos_tab, const float* sin_tab,
                       const float* q_gain, const float* k_gain, int n_tokens, int nq, int nk, int nkv_cache, int hd,
                       int rot, int page_size, float eps, float q_off, float k_off, cudaStream_t s, cudaError_t* err) {
    constexpr int EPL = Vec16<T>::N;
    if (hd % EPL != 0 || (cos_tab && rot != hd)) return false;
    const int lpr = hd / EPL;
    if (lpr != 8 && lpr != 16 && lpr != 32) return false;
    if (row_stride % EPL != 0 || q_stride % EPL != 0 || !host_aligned16(qkv) || !host_aligned16(q_out) ||
        (kcache && !host_aligned16(kcache)) || (vcache && !host_aligned16(vcache)))
        return false;
    // gains and rotary tables are read four floats at a time
    if ((q_gain && !host_aligned16(q_gain)) || (k_gain && !host_aligned16(k_gain)) || (cos_tab && !host_aligned16(cos_tab)) ||
        (sin_tab && !host_aligned16(sin_tab)) || (hd / 2) % 4 != 0)
        return false;
    const long long rows = (long long)n_tokens * (nq + 2 * nk);
    if (rows >= (1LL << 31) - (1LL << 20)) return false;       // the kernel counts rows in 32 bits
    const int rpw = 32 / lpr;
    if (g_prep_by_token) {
#define LAUNCH_TOKEN(L, U)                                                                                                  \
    do {                                                                                                                    \
        const int chunks = (nq + 2 * nk + U * rpw - 1) / (U * rpw);                                                         \
        long long tblocks = ((long long)n_tokens * chunks + 7) / 8;                                                         \
        if (tblocks > device_sm_count() * 8) tblocks = device_sm_count() * 8;                                                                           \
        *err = llmk_launch(attn_prep_token_kernel<T, L, U>, dim3((unsigned)tblocks), dim3(256), 0, s, true, (const T*)qkv,  \
                           row_stride, (T*)q_out, q_stride, (T*)kcache, (T*)vcache, positions, slots, cos_tab, sin_tab,     \
                           q_gain, k_gain, n_tokens, nq, nk, nkv_cache, hd, page_size, eps, q_off, k_off);                  \
    } while (0)
        // eight rounds of rows in flight per warp: 13.3 us on 2,048 tokens of 32 heads of 128 in bfloat16,
        // 15.2 us with four, 14.5 us a row at a time
        if (lpr == 8) LAUNCH_TOKEN(8, 8);
        else if (lpr == 16) LAUNCH_TOKEN(16, 8);
        else LAUNCH_TOKEN(32, 8);
#undef LAUNCH_TOKEN
        return true;
    }
    long long blocks = (rows + 8 * rpw - 1) / (8 * rpw);
    if (blocks > device_sm_count() * 8) blocks = device_sm_count() * 8;
#define LAUNCH_VEC(L)                                                                                                   \
    *err = llmk_launch(attn_prep_vec_kernel<T, L>, dim3((unsigned)blocks), dim3(256), 0, s, true, (const T*)qkv, row_stride, \
                       (T*)q_out, q_stride, (T*)kcache, (T*)vcache, positions, slots, cos_tab, sin_tab, q_gain, k_gain,  \
                       n_tokens, nq, nk, nkv_cache, hd, page_size, eps, q_off, k_off)
    if (lpr == 8) LAUNCH_VEC(8);
    else if (lpr == 16) LAUNCH_VEC(16);
    else LAUNCH_VEC(32);
#undef LAUNCH_VEC
    return true;
}

// The general kernel's arithmetic with 16-byte accesses for pairs (2i, 2i + 1): a pair never leaves its lane's vector, so any
// rotary width, biases and values of their own width are taken, where all of them are whole vectors.  `LPR` lanes share one
// (token, head) row.
template <typename T, int LPR>
__global__ void __launch_bounds__(256)
attn_prep_pairs_kernel(const T* __restrict__ qkv, long long row_stride, T* __restrict__ q_out, long long q_stride, T* __restrict__ kcache,
                       T* __restrict__ vcache, const int* __restrict__ positions, const int* __restrict__ slots,
                       const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, const float* __restrict__ q_gain,
                       const float* __restrict__ k_gain, int n_tokens, int nq, int nk, int nkv_cache, int hd, int rot, int page_size,
                       float eps, float q_off, float k_off, const float* __restrict__ bias, int vd) {
    constexpr int EPL = Vec16<T>::N;
    const unsigned heads = (unsigned)(nq + 2 * nk);
    const unsigned row = (blockIdx.x * blockDim.x + threadIdx.x) / LPR;
    const int at = (int)(threadIdx.x % LPR) * EPL;
    pdl_launch_dependents();
    pdl_wait();
    const bool live = row < (unsigned)n_tokens * heads;
    const int t = live ? (int)(row / heads) : 0;
    const int h = live ? (int)(row - (unsigned)t * heads) : 0;
    const bool is_q = h < nq, is_v = h >= nq + nk;
    const int width = is_v ? vd : hd;
    const bool on = live && at < width;
    const size_t col0 = is_v ? (size_t)(nq + nk) * hd + (size_t)(h - nq - nk) * vd : (size_t)h * hd;
    const int slot = slots ? slots[t] : -1;
    const int pos = cos_tab ? positions[t] : 0;
    float f[EPL];
#pragma unroll
    for (int i = 0; i < EPL; ++i) f[i] = 0.f;
    if (on) {
        Vec16<T> x;
        x.raw = *reinterpret_cast<const decltype(x.raw)*>(qkv + (size_t)t * row_stride + col0 + at);
        x.unpack(f);
        if (bias) {
#pragma unroll
            for (int i = 0; i < EPL; i += 4) {
                const float4 b = *reinterpret_cast<const float4*>(bias + col0 + at + i);
                f[i] += b.x; f[i + 1] += b.y; f[i + 2] += b.z; f[i + 3] += b.w;
            }
        }
    }
    const float* gain = is_v ? nullptr : is_q ? q_gain : k_gain;
    const float goff = is_q ? q_off : k_off;
    float ss = 0.f;                           // every lane takes part in the shuffles
#pragma unroll
    for (int i = 0; i < EPL; ++i) ss = fmaf(f[i], f[i], ss);
#pragma unroll
    for (int o = LPR / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!on) return;
    if (gain) {
        const float rinv = 1.0f / sqrtf(ss / (float)hd + eps);
#pragma unroll
        for (int i = 0; i < EPL; i += 4) {
            const float4 g = *reinterpret_cast<const float4*>(gain + at + i);
            f[i] *= rinv * (g.x + goff); f[i + 1] *= rinv * (g.y + goff); f[i + 2] *= rinv * (g.z + goff); f[i + 3] *= rinv * (g.w + goff);
        }
    }
    if (!is_v && cos_tab && at < rot) {
        const float* c = cos_tab + (size_t)pos * (rot / 2) + at / 2;
        const float* s = sin_tab + (size_t)pos * (rot / 2) + at / 2;
#pragma unroll
        for (int i = 0; i < EPL; i += 4) {
            const float2 cv = *reinterpret_cast<const float2*>(c + i / 2), sv = *reinterpret_cast<const float2*>(s + i / 2);
            const float a0 = f[i], b0 = f[i + 1], a1 = f[i + 2], b1 = f[i + 3];
            f[i] = a0 * cv.x - b0 * sv.x;
            f[i + 1] = b0 * cv.x + a0 * sv.x;
            f[i + 2] = a1 * cv.y - b1 * sv.y;
            f[i + 3] = b1 * cv.y + a1 * sv.y;
        }
    }
    T* dst = nullptr;
    if (is_q) {
        dst = q_out + (size_t)t * q_stride + (size_t)h * hd;
    } else if (slot >= 0) {
        T* cache = is_v ? vcache : kcache;
        const int kvh = is_v ? h - nq - nk : h - nq, page = slot / page_size;
        if (cache) dst = cache + (((size_t)page * nkv_cache + kvh) * page_size + (slot - page * page_size)) * width;
    }
    if (!dst) return;
    Vec16<T> y;
    y.pack(f);
    *reinterpret_cast<decltype(y.raw)*>(dst + at) = y.raw;
}

template <typename T>
static bool launch_pairs(const void* qkv, long long row_stride, void* q_out, long long q_stride, void* kcache, void* vcache, const int* positions,
                         const int* slots, const float* cos_tab, const float* sin_tab, const float* q_gain, const float* k_gain, int n_tokens,
                         int nq, int nk, int nkv_cache, int hd, int rot, int page_size, float eps, float q_off, float k_off,
                         const float* bias, int vd, cudaStream_t s, cudaError_t* e) {
    constexpr int EPL = Vec16<T>::N;
    const int most = (nk > 0 && vd > hd ? vd : hd) / EPL;
    if (hd % EPL || vd % EPL || rot % EPL || row_stride % EPL || q_stride % EPL || most > 32 || !host_aligned16(qkv) || !host_aligned16(q_out) ||
        !host_aligned16(kcache) || !host_aligned16(vcache) || !host_aligned16(cos_tab) || !host_aligned16(sin_tab) || !host_aligned16(bias) ||
        !host_aligned16(q_gain) || !host_aligned16(k_gain) || (long long)n_tokens * (nq + 2 * nk) * 32 > 2000000000LL)
        return false;
    const long long rows = (long long)n_tokens * (nq + 2 * nk);
#define ATTN_PREP_PAIRS(LPR)                                                                                                            \
    *e = llmk_launch(attn_prep_pairs_kernel<T, LPR>, dim3((unsigned)((rows * LPR + 255) / 256)), dim3(256), 0, s, true, (const T*)qkv,  \
                     row_stride, (T*)q_out, q_stride, (T*)kcache, (T*)vcache, positions, slots, cos_tab, sin_tab, q_gain, k_gain,       \
                     n_tokens, nq, nk, nkv_cache, hd, rot, page_size, eps, q_off, k_off, bias, vd)
    if (most <= 4) ATTN_PREP_PAIRS(4);
    else if (most <= 8) ATTN_PREP_PAIRS(8);
    else if (most <= 16) ATTN_PREP_PAIRS(16);
    else ATTN_PREP_PAIRS(32);
#undef ATTN_PREP_PAIRS
    return true;
}

// nk = number of k (and v) heads present in the packed rows: num_kv_heads for a layer that
// writes its cache, 0 for a layer that only reads another layer's cache.
LLMK_EXPORT int llmk_attn_prep(const void* qkv, long long row_stride, int splits, long long split_stride, void* q_out,
                               long long q_stride, void* kcache, void* vcache, const int* positions,
                               const int* slots, const float* cos_tab, const float* sin_tab, const float* q_gain,
                               const float* k_gain, int n_tokens, int nq, int nk, int nkv_cache, int hd, int rot,
                               int page_size, float eps, float q_off, float k_off, int pairing, int head_norm,
                               const float* bias, int vd, int dtype, void* stream) {
    if (n_tokens <= 0) return LLMK_OK;
    if (vd <= 0) vd = hd;
    if (vd > 32 * MAX_TAIL) LLMK_FAIL("attn_prep: value width %d too large", vd);
    if (pairing != LLMK_PAIR_HALF_SPLIT && pairing != LLMK_PAIR_INTERLEAVED)
        LLMK_FAIL("attn_prep: rotary pairing %d is not built (0: half-split, pairs (i, i + rot / 2); 1: pairs (2i, 2i + 1))", pairing);
    if (head_norm != LLMK_HEAD_NORM_RMS && head_norm != LLMK_HEAD_NORM_UNIT_AFTER)
        LLMK_FAIL("attn_prep: per-head norm kind %d is not built (0: RMSNorm before the rotation; 1: without gains, after it)", head_norm);
    if (head_norm == LLMK_HEAD_NORM_UNIT_AFTER && (q_gain || k_gain)) LLMK_FAIL("attn_prep: the norm after the rotation has no gains");
    // the 16-byte variants pair values half a head apart and norm before they rotate
    const bool general_only = pairing != LLMK_PAIR_HALF_SPLIT || head_norm != LLMK_HEAD_NORM_RMS;
    const int interleaved = pairing == LLMK_PAIR_INTERLEAVED ? 1 : 0, norm_after = head_norm == LLMK_HEAD_NORM_UNIT_AFTER ? 1 : 0;
    if (hd <= 0 || hd % 2 != 0 || hd > 512) LLMK_FAIL("attn_prep: head_dim %d must be even and at most 512", hd);
    if (rot < 0 || rot > hd || rot % 2 != 0) LLMK_FAIL("attn_prep: rotary width %d must be even and at most head_dim %d", rot, hd);
    if (rot / 2 > 32 * MAX_PAIRS || hd - rot > 32 * MAX_TAIL) LLMK_FAIL("attn_prep: head_dim %d / rotary width %d too large", hd, rot);
    if (nq < 0 || nk < 0 || nq + nk <= 0) LLMK_FAIL("attn_prep: bad head counts nq=%d nk=%d", nq, nk);
    if (nk > 0 && (page_size <= 0 || nkv_cache < nk)) LLMK_FAIL("attn_prep: bad cache geometry page_size=%d kv heads=%d", page_size, nkv_cache);
    if (splits < 0 || (splits > 0 && split_stride <= 0)) LLMK_FAIL("attn_prep: bad partial sums (%d slices)", splits);
    if (!q_out && nq > 0) LLMK_FAIL("attn_prep: no place for q");
    if (!cos_tab) rot = 0;
    if (cos_tab && (!sin_tab || !positions)) LLMK_FAIL("attn_prep: rotary tables need sin and positions");
    cudaStream_t s = (cudaStream_t)stream;
    const int warps = 4;
    const long long items = (long long)n_tokens * (nq + 2 * nk);
    const long long blocks = (items + warps - 1) / warps;
    if (blocks > 2147483647LL) LLMK_FAIL("attn_prep: too many rows");
    cudaError_t e;
    if (splits == 0 && n_tokens >= 32 && !bias && vd == hd && !general_only) {
        bool taken = false;
        if (dtype == LLMK_F32)
            taken = launch_vec<float>(qkv, row_stride, q_out, q_stride, kcache, vcache, positions, slots, cos_tab, sin_tab,
                                      q_gain, k_gain, n_tokens, nq, nk, nkv_cache, hd, rot, page_size, eps, q_off, k_off, s, &e);
        else if (dtype == LLMK_BF16)
            taken = launch_vec<bf16>(qkv, row_stride, q_out, q_stride, kcache, vcache, positions, slots, cos_tab, sin_tab,
                                     q_gain, k_gain, n_tokens, nq, nk, nkv_cache, hd, rot, page_size, eps, q_off, k_off, s, &e);
        if (taken) {
            LLMK_CHECK_LAUNCH_RC("attn_prep", e);
            return LLMK_OK;
        }
    }
    if (splits == 0 && interleaved && !norm_after) {
        bool taken = false;
        if (dtype == LLMK_F32)
            taken = launch_pairs<float>(qkv, row_stride, q_out, q_stride, kcache, vcache, positions, slots, cos_tab, sin_tab, q_gain, k_gain,
                                        n_tokens, nq, nk, nkv_cache, hd, rot, page_size, eps, q_off, k_off, bias, vd, s, &e);
        else if (dtype == LLMK_BF16)
            taken = launch_pairs<bf16>(qkv, row_stride, q_out, q_stride, kcache, vcache, positions, slots, cos_tab, sin_tab, q_gain, k_gain,
                                       n_tokens, nq, nk, nkv_cache, hd, rot, page_size, eps, q_off, k_off, bias, vd, s, &e);
        if (taken) {
            LLMK_CHECK_LAUNCH_RC("attn_prep", e);
            return LLMK_OK;
        }
    }
    if (dtype == LLMK_F32)
        e = llmk_launch(attn_prep_kernel<float>, dim3((unsigned)blocks), dim3(warps * 32), 0, s, true, qkv, row_stride,
                        splits, split_stride, (float*)q_out, q_stride, (float*)kcache, (float*)vcache, positions, slots,
                        cos_tab, sin_tab, q_gain, k_gain, n_tokens, nq, nk, nkv_cache, hd, rot, page_size, eps, q_off,
                        k_off, bias, vd, interleaved, norm_after);
    else if (dtype == LLMK_BF16)
        e = llmk_launch(attn_prep_kernel<bf16>, dim3((unsigned)blocks), dim3(warps * 32), 0, s, true, qkv, row_stride,
                        splits, split_stride, (bf16*)q_out, q_stride, (bf16*)kcache, (bf16*)vcache, positions, slots,
                        cos_tab, sin_tab, q_gain, k_gain, n_tokens, nq, nk, nkv_cache, hd, rot, page_size, eps, q_off,
                        k_off, bias, vd, interleaved, norm_after);
    else
        LLMK_FAIL("attn_prep: unknown dtype %d", dtype);
    LLMK_CHECK_LAUNCH_RC("attn_prep", e);
    return LLMK_OK;
}

// ------------------------------------------------------------------------------------------------ norms over whole projections
// For layers whose q and k are normed over the whole projection (all heads of a token at once, gains of that size) and
// whose values are rotated too.  x [n, ld] float32 holds [q | k | v] of a token (nq hd, nk hd, nk vd values): q and k are
// divided by the root mean square of their whole row (eps inside the root) and multiplied by their gains, the first `rot`
// values of each head are turned in half-split pairs (i, i + rot / 2) by the position's angles; v is turned over all of
// its vd values in pairs (m, m + vd / 2) by angles of its own table (vcos / vsin [max_positions, vd / 2]; none: v as it is).
// q goes to q_out, k and v to the cache at the token's slot (slot < 0: not stored).  A block per token.
template <typename T>
__global__ void attn_prep_rows_kernel(const float* __restrict__ x, long long ld, T* __restrict__ q_out, long long q_stride,
                                      T* __restrict__ kcache, T* __restrict__ vcache, const int* __restrict__ positions,
                                      const int* __restrict__ slots, const float* __restrict__ cos_tab,
                                      const float* __restrict__ sin_tab, const float* __restrict__ vcos,
                                      const float* __restrict__ vsin, const float* __restrict__ q_gain,
                                      const float* __restrict__ k_gain, int nq, int nk, int nkv_cache, int hd, int vd, int rot,
                                      int page_size, float eps) {
    __shared__ float scratch[33];
    const size_t t = blockIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const float* row = x + t * ld;
    const int nQ = nq * hd, nK = nk * hd, nV = nk * vd;
    const int pos = positions ? positions[t] : 0;
    const int slot = slots ? slots[t] : -1;
    const int half = rot / 2;
    float ssq = 0.f, ssk = 0.f;
    for (int i = threadIdx.x; i < nQ; i += blockDim.x) ssq = fmaf(row[i], row[i], ssq);
    for (int i = threadIdx.x; i < nK; i += blockDim.x) ssk = fmaf(row[nQ + i], row[nQ + i], ssk);
    ssq = block_sum(ssq, scratch);
    ssk = nK > 0 ? block_sum(ssk, scratch) : 0.f;
    const float rq = 1.0f / sqrtf(ssq / (float)max(nQ, 1) + eps), rk = 1.0f / sqrtf(ssk / (float)max(nK, 1) + eps);
    for (int i = threadIdx.x; i < nQ + nK; i += blockDim.x) {
        const bool is_q = i < nQ;
        const int c = is_q ? i : i - nQ;
        const int d = c % hd;
        const float* g = is_q ? q_gain : k_gain;
        const float r = is_q ? rq : rk;
        float val = row[i] * r * (g ? g[c] : 1.f);
        if (d < rot) {
            const int other = d < half ? i + half : i - half;
            const int oc = d < half ? c + half : c - half;
            const float pv = row[other] * r * (g ? g[oc] : 1.f);
            const int f = d < half ? d : d - half;
            const float cs = cos_tab[(size_t)pos * half + f], sn = sin_tab[(size_t)pos * half + f];
            val = d < half ? val * cs - pv * sn : val * cs + pv * sn;
        }
        if (is_q) {
            q_out[t * q_stride + c] = from_float<T>(val);
        } else if (slot >= 0 && kcache) {
            const int kvh = c / hd;
            kcache[(((size_t)(slot / page_size) * nkv_cache + kvh) * page_size + slot % page_size) * hd + d] = from_float<T>(val);
        }
    }
    if (slot < 0 || !vcache) return;
    const int vhalf = vd / 2;
    for (int i = threadIdx.x; i < nV; i += blockDim.x) {
        const int kvh = i / vd, d = i % vd;
        float val = row[nQ + nK + i];
        if (vcos) {
            const float pv = row[nQ + nK + (d < vhalf ? i + vhalf : i - vhalf)];
            const int f = d < vhalf ? d : d - vhalf;
            const float cs = vcos[(size_t)pos * vhalf + f], sn = vsin[(size_t)pos * vhalf + f];
            val = d < vhalf ? val * cs - pv * sn : val * cs + pv * sn;
        }
        vcache[(((size_t)(slot / page_size) * nkv_cache + kvh) * page_size + slot % page_size) * vd + d] = from_float<T>(val);
    }
}

LLMK_EXPORT int llmk_attn_prep_rows(const float* x, long long ld, void* q_out, long long q_stride, void* kcache, void* vcache,
                                    const int* positions, const int* slots, const float* cos_tab, const float* sin_tab,
                                    const float* vcos, const float* vsin, const float* q_gain, const float* k_gain, int n_tokens,
                                    int nq, int nk, int nkv_cache, int hd, int vd, int rot, int page_size, float eps, int dtype,
                                    void* stream) {
    if (n_tokens <= 0) return LLMK_OK;
    if (nq <= 0 || nk < 0 || hd <= 0 || vd <= 0 || !q_out) LLMK_FAIL("attn_prep_rows: bad sizes (nq %d, nk %d, hd %d, vd %d)", nq, nk, hd, vd);
    if (!cos_tab) rot = 0;
    if (rot < 0 || rot > hd || rot % 2 != 0) LLMK_FAIL("attn_prep_rows: rotary width %d must be even and at most head_dim %d", rot, hd);
    if (rot > 0 && (!sin_tab || !positions)) LLMK_FAIL("attn_prep_rows: rotary tables need sin and positions");
    if (vcos && (!vsin || !positions || vd % 2 != 0)) LLMK_FAIL("attn_prep_rows: rotated values need sin, positions and an even width");
    if (nk > 0 && (page_size <= 0 || nkv_cache < nk)) LLMK_FAIL("attn_prep_rows: bad cache geometry page_size=%d kv heads=%d", page_size, nkv_cache);
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (dtype == LLMK_F32)
        e = llmk_launch(attn_prep_rows_kernel<float>, dim3(n_tokens), dim3(256), 0, s, true, x, ld, (float*)q_out, q_stride, (float*)kcache,
                        (float*)vcache, positions, slots, cos_tab, sin_tab, vcos, vsin, q_gain, k_gain, nq, nk, nkv_cache, hd, vd, rot,
                        page_size, eps);
    else if (dtype == LLMK_BF16)
        e = llmk_launch(attn_prep_rows_kernel<bf16>, dim3(n_tokens), dim3(256), 0, s, true, x, ld, (bf16*)q_out, q_stride, (bf16*)kcache,
                        (bf16*)vcache, positions, slots, cos_tab, sin_tab, vcos, vsin, q_gain, k_gain, nq, nk, nkv_cache, hd, vd, rot,
                        page_size, eps);
    else
        LLMK_FAIL("attn_prep_rows: unknown dtype %d", dtype);
    LLMK_CHECK_LAUNCH_RC("attn_prep_rows", e);
    return LLMK_OK;
}

// Attention whose values are its projected keys: a token's entry is stored once, as projected, and what the key's norm does to it
// is one number beside it.  With q = x[0 : nQ] + b and k = x[nQ : nQ + nK] + b of a token's packed row, rq and rk the inverse root
// mean squares of the two whole rows:
//   cache[slot, g, :]  = k of key head g                        (storage dtype; keys and values of the attention)
//   k_scale[slot]      = rk                                     (float32; multiplies the token's scores)
//   q_out[t, h, :]     = q rq * gains[h, :] * temperature       (gains: q's times those of the key head that h reads, folded at load)
// temperature = 1 + coef ln(floor((position + 1) / every) + 1), or 1 with coef 0.  The packed row is an array of T or float32
// slices of a product.  A block per token; the row passes through shared memory, V values a thread at a time.
template <typename T>
__device__ __forceinline__ float packed_sum(const void* x, size_t at, int splits, long long split_stride) {
    if (splits == 0) return to_float(static_cast<const T*>(x)[at]);
    const float* p = static_cast<const float*>(x) + at;
    float acc = p[0];
    for (int s = 1; s < splits; ++s) acc += p[(size_t)s * split_stride];
    return acc;
}

template <typename T>
__global__ void __launch_bounds__(512) attn_prep_shared_rows_kernel(const void* __restrict__ x, long long ld, int splits, long long split_stride,
                                                                    const float* __restrict__ bias, T* __restrict__ q_out, long long q_stride,
                                                                    T* __restrict__ cache, float* __restrict__ k_scale,
                                                                    const int* __restrict__ positions, const int* __restrict__ slots,
                                                                    const float* __restrict__ gains, int nq, int nk, int nkv_cache, int hd,
                                                                    int page_size, float eps, float coef, float every) {
    extern __shared__ __align__(16) float prow[];     // nQ + nK floats, 33 scratch
    const int nQ = nq * hd, nK = nk * hd, n = nQ + nK;
    float* scratch = prow + n;
    const size_t t = blockIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const size_t base = t * ld;
    float ssq = 0.f, ssk = 0.f;
    const bool vec = sizeof(T) == 2 && splits == 0 && (nQ & 7) == 0 && (nK & 7) == 0 && (ld & 7) == 0 && aligned16(x);
    if (vec) {
        for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {
            Vec16<bf16> raw;
            raw.raw = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(x) + base + i);
            float v[8];
            raw.unpack(v);
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                if (bias) v[e] += bias[i + e];
                ss = fmaf(v[e], v[e], ss);
            }
            *reinterpret_cast<float4*>(prow + i) = make_float4(v[0], v[1], v[2], v[3]);
            *reinterpret_cast<float4*>(prow + i + 4) = make_float4(v[4], v[5], v[6], v[7]);
            if (i < nQ) ssq += ss; else ssk += ss;
        }
    } else if (splits > 0 && (nQ & 3) == 0 && (nK & 3) == 0 && (ld & 3) == 0 && (split_stride & 3) == 0 && aligned16(x) && (!bias || aligned16(bias))) {
        // slices, four values a thread at a time, the loads of four slices in flight together
        for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
            const float* p = static_cast<const float*>(x) + base + i;
            float4 v = *reinterpret_cast<const float4*>(p);
#pragma unroll 4
            for (int s = 1; s < splits; ++s) {
                const float4 f = *reinterpret_cast<const float4*>(p + (size_t)s * split_stride);
                v.x += f.x; v.y += f.y; v.z += f.z; v.w += f.w;
            }
            if (bias) {
                const float4 b = *reinterpret_cast<const float4*>(bias + i);
                v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
            }
            *reinterpret_cast<float4*>(prow + i) = v;
            const float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
            if (i < nQ) ssq += ss; else ssk += ss;
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) {
            const float v = packed_sum<T>(x, base + i, splits, split_stride) + (bias ? bias[i] : 0.f);
            prow[i] = v;
            if (i < nQ) ssq = fmaf(v, v, ssq); else ssk = fmaf(v, v, ssk);
        }
    }
    ssq = block_sum(ssq, scratch);
    ssk = nK > 0 ? block_sum(ssk, scratch) : 0.f;       // block_sum also orders the row in shared memory
    const int pos = positions[t];
    float rq = 1.0f / sqrtf(ssq / (float)nQ + eps);
    if (coef != 0.f) rq *= 1.0f + coef * logf(floorf((float)(pos + 1) / every) + 1.0f);
    T* qo = q_out + t * q_stride;
    if (vec && (q_stride & 7) == 0 && aligned16(q_out)) {
        for (int i = threadIdx.x * 8; i < nQ; i += blockDim.x * 8) {
            float v[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = prow[i + e] * rq * gains[i + e];
            Vec16<bf16> raw;
            raw.pack(v);
            *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(qo) + i) = raw.raw;
        }
    } else {
        for (int i = threadIdx.x; i < nQ; i += blockDim.x) qo[i] = from_float<T>(prow[i] * rq * gains[i]);
    }
    const int slot = slots ? slots[t] : -1;
    if (slot < 0 || nK == 0) return;
    const int page = slot / page_size, off = slot % page_size;
    for (int i = threadIdx.x; i < nK; i += blockDim.x) {
        const int g = i / hd, d = i % hd;
        cache[(((size_t)page * nkv_cache + g) * page_size + off) * hd + d] = from_float<T>(prow[nQ + i]);
    }
    if (threadIdx.x == 0) k_scale[slot] = 1.0f / sqrtf(ssk / (float)nK + eps);
}

LLMK_EXPORT int llmk_attn_prep_shared_rows(const void* x, long long ld, int splits, long long split_stride, const float* bias, void* q_out,
                                           long long q_stride, void* cache, float* k_scale, const int* positions, const int* slots,
                                           const float* gains, int n_tokens, int nq, int nk, int nkv_cache, int hd, int page_size, float eps,
                                           float coef, float every, int dtype, void* stream) {
    if (n_tokens <= 0) return LLMK_OK;
    if (nq <= 0 || nk < 0 || hd <= 0 || !x || !q_out || !gains || !positions) LLMK_FAIL("attn_prep_shared_rows: bad arguments (nq %d, nk %d, hd %d)", nq, nk, hd);
    if (nk > 0 && (!cache || !k_scale || page_size <= 0 || nkv_cache < nk)) LLMK_FAIL("attn_prep_shared_rows: bad cache geometry page_size=%d kv heads=%d", page_size, nkv_cache);
    if (coef != 0.f && !(every > 0.f)) LLMK_FAIL("attn_prep_shared_rows: a temperature every %g positions", (double)every);
    const size_t smem = ((size_t)(nq + nk) * hd + 33) * sizeof(float);
    if (smem > 200 * 1024) LLMK_FAIL("attn_prep_shared_rows: a row of %d values does not fit shared memory", (nq + nk) * hd);
    const int threads = splits > 0 && (nq + nk) * hd >= 2048 ? 512 : 256;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (dtype == LLMK_F32) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(attn_prep_shared_rows_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        e = llmk_launch(attn_prep_shared_rows_kernel<float>, dim3(n_tokens), dim3(threads), smem, s, true, x, ld, splits, split_stride, bias, (float*)q_out,
                        q_stride, (float*)cache, k_scale, positions, slots, gains, nq, nk, nkv_cache, hd, page_size, eps, coef, every);
    } else if (dtype == LLMK_BF16) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(attn_prep_shared_rows_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        e = llmk_launch(attn_prep_shared_rows_kernel<bf16>, dim3(n_tokens), dim3(threads), smem, s, true, x, ld, splits, split_stride, bias, (bf16*)q_out,
                        q_stride, (bf16*)cache, k_scale, positions, slots, gains, nq, nk, nkv_cache, hd, page_size, eps, coef, every);
    } else
        LLMK_FAIL("attn_prep_shared_rows: unknown dtype %d", dtype);
    LLMK_CHECK_LAUNCH_RC("attn_prep_shared_rows", e);
    return LLMK_OK;
}

// The attention's rows on their way to the output projection: each head's vd values turned back in pairs (m, m + vd / 2) by
// minus the position's angles (vcos / vsin [max_positions, vd / 2]; none: as they are), then multiplied by sigmoid(gate[t, h]),
// one number per head (gate rows `gate_stride` apart; none: no gate).  In place; a thread per pair.
template <typename T>
__global__ void unrotate_gate_kernel(T* __restrict__ o, long long o_stride, const T* __restrict__ gate, long long gate_stride,
                                     const int* __restrict__ positions, const float* __restrict__ vcos,
                                     const float* __restrict__ vsin, long long n, int nq, int vd) {
    pdl_launch_dependents();
    pdl_wait();
    const int vhalf = vd / 2;
    const long long total = n * nq * vhalf;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const int m = (int)(i % vhalf);
        const int h = (int)((i / vhalf) % nq);
        const size_t t = (size_t)(i / ((long long)vhalf * nq));
        T* p = o + t * o_stride + (size_t)h * vd;
        float a = to_float(p[m]), b = to_float(p[m + vhalf]);
        if (vcos) {
            const int pos = positions[t];
            const float cs = vcos[(size_t)pos * vhalf + m], sn = vsin[(size_t)pos * vhalf + m];
            const float a2 = a * cs + b * sn, b2 = b * cs - a * sn;
            a = a2;
            b = b2;
        }
        if (gate) {
            const float g = 1.0f / (1.0f + expf(-to_float(gate[t * gate_stride + h])));
            a *= g;
            b *= g;
        }
        p[m] = from_float<T>(a);
        p[m + vhalf] = from_float<T>(b);
    }
}

LLMK_EXPORT int llmk_unrotate_gate(void* o, long long o_stride, const void* gate, long long gate_stride, const int* positions,
                                   const float* vcos, const float* vsin, int n_tokens, int nq, int vd, int dtype, void* stream) {
    if (n_tokens <= 0) return LLMK_OK;
    if (nq <= 0 || vd <= 0 || vd % 2 != 0) LLMK_FAIL("unrotate_gate: %d heads of %d values (an even width)", nq, vd);
    if (vcos && (!vsin || !positions)) LLMK_FAIL("unrotate_gate: the tables need sin and positions");
    long long blocks = ((long long)n_tokens * nq * (vd / 2) + 255) / 256;
    if (blocks > device_sm_count() * 16) blocks = device_sm_count() * 16;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (dtype == LLMK_F32)
        e = llmk_launch(unrotate_gate_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, s, true, (float*)o, o_stride, (const float*)gate,
                        gate_stride, positions, vcos, vsin, (long long)n_tokens, nq, vd);
    else if (dtype == LLMK_BF16)
        e = llmk_launch(unrotate_gate_kernel<bf16>, dim3((unsigned)blocks), dim3(256), 0, s, true, (bf16*)o, o_stride, (const bf16*)gate,
                        gate_stride, positions, vcos, vsin, (long long)n_tokens, nq, vd);
    else
        LLMK_FAIL("unrotate_gate: unknown dtype %d", dtype);
    LLMK_CHECK_LAUNCH_RC("unrotate_gate", e);
    return LLMK_OK;
}
