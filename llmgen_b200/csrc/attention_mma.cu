// Causal grouped-query attention over the paged cache for prompts and prompt portions in bfloat16 whose softmax
// weights must stay 32-bit: the products run on the tensor cores (`mma.sync.m16n8k16`, bfloat16 operands, float32
// accumulators), everything between them on the CUDA cores in float32.
//
//   S = Q K^T      Q and K are the cache's bfloat16 values, every product exact, sums float32
//   scores         s * scale, then (softcap > 0) softcap * tanh(s / softcap), the causal (and window, or block) mask, the row's
//                  running maximum and sum, the weights exp(s - m): float32 (powers of two of scores times log2(e))
//   O += P V       a float32 weight enters as THREE bfloat16 terms p = p1 + p2 + p3 (24 bits of mantissa), so every
//                  product with a bfloat16 value is what float32 arithmetic would give; three MMAs a step
//   finish         the sink (one more term exp(0) in the denominator), the division, the output gate sigmoid(g)
//
// Block = 64 queries of one sequence x one query head, four warps of 16 rows; keys in tiles of 64 through shared
// memory: 16-byte `cp.async` copies out of the pages into two buffers, the next tile on its way while this one is used.  Semantics as in csrc/attention.cu (which takes float32, single tokens in
// parts, and every size this kernel refuses): query j of a portion sits at position ctx - q_len + j.
// Entries that are key and value at once (SHARED: `k_scale`, a factor on the scores per cached token; no value array): a tile of
// keys is copied once and serves both products, its tokens' factors beside it.
// Taken: key width and value width 64 or 128 each.
//
// `attention_mma_parts` is the same arithmetic for steps of single tokens: the rows of a block are the query heads of one key head
// (up to 16), its keys one part of what the token sees; four warps take 16 keys each of a tile of 64, with a softmax of their own
// that is merged at the end, and the blocks of one (token, key head) are a cluster that merges the parts through each other's
// shared memory, in part order.  No gate and no turn back there.
#define LLMK_MODULE_NAME "attention_mma"
#include "common.cuh"

LLMK_DEFINE_LAST_ERROR()

namespace {

constexpr int BM = 64, BN = 64, WARPS = 4;

struct Params {
    const bf16* q;
    const bf16* kcache;
    const bf16* vcache;
    bf16* out;
    const bf16* gate;
    const float* sink_values;     // with `sink`: the sink's score per query head [nq]; null: 0
    const float* turn_cos;        // [positions, VD / 2] (with turn_sin): every head's row is turned back in pairs (m, m + VD / 2) by minus
    const float* turn_sin;        // its query's position before the gate; null: rows leave as they are
    const float* k_scale;         // SHARED: [pages, page_size]
    int gate_heads;               // 1: the gate is one number per head, [tokens, nq]
    const int* block_tables;
    const int* ctx_len;
    const int* cu_q;
    const int* tile_seq;
    const int* tile_q0;
    long long q_stride, o_stride, gate_stride;
    int max_blocks, nq, nkv, page_size, window, sink, chunk;     // chunk > 0: a query sees the keys of its own block of that many positions
    float scale, softcap;
};

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem_row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem_row) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem_row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(void* smem_dst, const void* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(smem_dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(void* smem_dst, const void* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(smem_dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_but_one() { asm volatile("cp.async.wait_group 1;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }
// tanh(x) = 1 - 2 / (1 + e^(2x)): an absolute error of a few 1e-7, which is what a score needs (it is an exponent)
__device__ __forceinline__ float tanh_abs(float x) { return 1.0f - __fdividef(2.0f, 1.0f + exp2f(x * 2.8853900817779268f)); }
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
// 2^x (the hardware's approximation: 2 ulp; results below the smallest normal number are zero)
__device__ __forceinline__ float pow2(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}
// x / d where d's shift is known (d a power of two), else by division
__device__ __forceinline__ int quotient(int x, int d, int shift) { return shift >= 0 ? x >> shift : x / d; }
__device__ __forceinline__ int shift_of(int d) { return (d & (d - 1)) == 0 ? __ffs(d) - 1 : -1; }
// two float32 as three pairs of bfloat16: x = w1 + w2 + w3, the most significant pieces first
__device__ __forceinline__ void split3(float x0, float x1, uint32_t& w1, uint32_t& w2, uint32_t& w3) {
    w1 = pack2(x0, x1);
    const float r0 = x0 - __uint_as_float(w1 << 16), r1 = x1 - __uint_as_float(w1 & 0xffff0000u);
    w2 = pack2(r0, r1);
    w3 = pack2(r0 - __uint_as_float(w2 << 16), r1 - __uint_as_float(w2 & 0xffff0000u));
}

template <int HD, int VD, bool SHARED>
__global__ void __launch_bounds__(WARPS * 32, SHARED || VD == 64 ? 3 : 2) attention_mma_kernel(Params p) {
    static_assert(!SHARED || HD == VD, "keys that are values have one width");
    constexpr int QLD = HD + 8, VLD = VD + 8;      // rows 16 bytes longer: the eight rows of an ldmatrix fall on different banks
    extern __shared__ __align__(16) uint8_t smem_raw[];
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);      // [BM][QLD]
    bf16* Kbuf = Qs + BM * QLD;                         // 2 x [BN][QLD]
    bf16* Vbuf = SHARED ? Kbuf : Kbuf + 2 * BN * QLD;   // 2 x [BN][VLD] (SHARED: the keys' own rows)
    float* Sbuf = reinterpret_cast<float*>(Kbuf + 2 * BN * QLD);      // SHARED: 2 x [BN] factors
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int g = lane >> 2, tq = lane & 3;
    const int s = p.tile_seq[blockIdx.x];
    pdl_launch_dependents();
    pdl_wait();
    if (s < 0) return;
    const int q0 = p.tile_q0[blockIdx.x];
    const int head = blockIdx.y;
    const int kvh = head / (p.nq / p.nkv);
    const int q_beg = p.cu_q[s], q_len = p.cu_q[s + 1] - q_beg, ctx = p.ctx_len[s];
    const int nq_tile = min(BM, q_len - q0);
    if (nq_tile <= 0 || ctx < q_len) {
        // rows of padding: zeros
        for (int idx = threadIdx.x; idx < max(nq_tile, 0) * VD; idx += blockDim.x)
            p.out[(size_t)(q_beg + q0 + idx / VD) * p.o_stride + (size_t)head * VD + idx % VD] = __float2bfloat16_rn(0.f);
        return;
    }
    const int first_pos = ctx - q_len + q0;
    const int k_end = first_pos + nq_tile;
    int k_beg = p.window > 0 ? max(0, first_pos - p.window + 1) / BN * BN : 0;
    if (p.chunk > 0) k_beg = max(k_beg, first_pos / p.chunk * p.chunk / BN * BN);
    const int* bt = p.block_tables + (size_t)s * p.max_blocks;
    const int page_shift = shift_of(p.page_size);

    for (int idx = threadIdx.x; idx < BM * (HD / 8); idx += blockDim.x) {
        const int r = idx / (HD / 8), v = idx % (HD / 8);
        uint4 val = make_uint4(0, 0, 0, 0);
        if (r < nq_tile) val = *reinterpret_cast<const uint4*>(p.q + (size_t)(q_beg + q0 + r) * p.q_stride + (size_t)head * HD + v * 8);
        *reinterpret_cast<uint4*>(Qs + r * QLD + v * 8) = val;
    }
    __syncthreads();
    uint32_t qf[HD / 16][4];
#pragma unroll
    for (int j = 0; j < HD / 16; ++j)
        ldmatrix_x4(qf[j], Qs + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * QLD + j * 16 + (lane >> 4) * 8);

    float o[VD / 8][4];
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    const int qpos[2] = {first_pos + warp * 16 + g, first_pos + warp * 16 + g + 8};
    const int kmin[2] = {p.chunk > 0 ? qpos[0] / p.chunk * p.chunk : 0, p.chunk > 0 ? qpos[1] / p.chunk * p.chunk : 0};
    constexpr float LOG2E = 1.4426950408889634f;
    // the bound on the scores, as they are: cap2 tanh(s2 / cap2) with s2 = s log2(e), cap2 = cap log2(e)
    const float scale2 = p.scale * LOG2E, cap2 = p.softcap * LOG2E, inv_cap2 = p.softcap > 0.f ? 1.0f / cap2 : 0.f;

    constexpr int VECS = HD / 8 + (SHARED ? 0 : VD / 8);
    auto load_tile = [&](int t0, int buf) {
        bf16* Kd = Kbuf + buf * BN * QLD;
        bf16* Vd = Vbuf + buf * BN * VLD;
#pragma unroll 4
        for (int idx = threadIdx.x; idx < BN * VECS; idx += WARPS * 32) {
            const int key = idx / VECS, v = idx % VECS;
            const int kpos = t0 + key;
            bf16* dst = v < HD / 8 ? Kd + key * QLD + v * 8 : Vd + key * VLD + (v - HD / 8) * 8;
            const int at = quotient(kpos, p.page_size, page_shift);
            const int page = kpos < k_end ? bt[at] : -1;      // -1 too: a page the window has passed
            if (page >= 0) {
                const size_t row = ((size_t)page * p.nkv + kvh) * p.page_size + (kpos - at * p.page_size);
                cp_async16(dst, v < HD / 8 ? p.kcache + row * HD + v * 8 : p.vcache + row * VD + (v - HD / 8) * 8);
            } else {
                *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
            }
        }
        if constexpr (SHARED) {
            for (int key = threadIdx.x; key < BN; key += WARPS * 32) {
                const int kpos = t0 + key;
                const int at = quotient(kpos, p.page_size, page_shift);
                const int page = kpos < k_end ? bt[at] : -1;
                if (page >= 0) cp_async4(Sbuf + buf * BN + key, p.k_scale + (size_t)page * p.page_size + (kpos - at * p.page_size));
                else Sbuf[buf * BN + key] = 0.f;
            }
        }
    };
    load_tile(k_beg, 0);
    int turn = 0;
    for (int t0 = k_beg; t0 < k_end; t0 += BN, turn ^= 1) {
        cp_async_wait_all();
        __syncthreads();          // this tile has arrived, and the tile before is consumed by every warp
        if (t0 + BN < k_end) load_tile(t0 + BN, turn ^ 1);
        const bf16* Ks = Kbuf + turn * BN * QLD;
        const bf16* Vs = Vbuf + turn * BN * VLD;
        // a warp whose rows all lie before this tile's first key has nothing to do in it (causal)
        if (first_pos + warp * 16 + 15 < t0) continue;

        float sc[BN / 8][4];
#pragma unroll
        for (int n = 0; n < BN / 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
        for (int j = 0; j < HD / 16; ++j) {
#pragma unroll
            for (int n2 = 0; n2 < BN / 16; ++n2) {
                uint32_t kb[4];
                ldmatrix_x4(kb, Ks + (n2 * 16 + (lane >> 4) * 8 + (lane & 7)) * QLD + j * 16 + ((lane >> 3) & 1) * 8);
                mma_bf16(sc[2 * n2], qf[j], kb[0], kb[1]);
                mma_bf16(sc[2 * n2 + 1], qf[j], kb[2], kb[3]);
            }
        }
        // scores as powers of two, s log2(e), and the rows' maxima; the mask where a tile is not wholly visible to these rows
        const bool whole = t0 + BN - 1 <= first_pos + warp * 16 && t0 + BN <= k_end && (p.window <= 0 || t0 > first_pos + warp * 16 + 15 - p.window) &&
                           t0 >= kmin[1];
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < BN / 8; ++n) {
            float2 f = make_float2(scale2, scale2);
            if constexpr (SHARED) {
                const float2 ks = *reinterpret_cast<const float2*>(Sbuf + turn * BN + n * 8 + 2 * tq);
                f.x *= ks.x;
                f.y *= ks.y;
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[n][e] *= (e & 1) ? f.y : f.x;
        }
        if (p.softcap > 0.f) {
#pragma unroll
            for (int n = 0; n < BN / 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) sc[n][e] = cap2 * tanh_abs(sc[n][e] * inv_cap2);
        }
        if (!whole) {
#pragma unroll
            for (int n = 0; n < BN / 8; ++n) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = e >> 1;
                    const int kpos = t0 + n * 8 + 2 * tq + (e & 1);
                    const bool vis = kpos <= qpos[r] && kpos < k_end && (p.window <= 0 || kpos > qpos[r] - p.window) && kpos >= kmin[r];
                    sc[n][e] = vis ? sc[n][e] : -INFINITY;
                }
            }
        }
#pragma unroll
        for (int n = 0; n < BN / 8; ++n) {
            mx[0] = fmaxf(mx[0], fmaxf(sc[n][0], sc[n][1]));
            mx[1] = fmaxf(mx[1], fmaxf(sc[n][2], sc[n][3]));
        }
        float alpha[2], base[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float m_new = fmaxf(m[r], mx[r]);
            base[r] = m_new > -INFINITY ? m_new : 0.f;        // a row that has seen nothing: every weight 2^-inf
            alpha[r] = pow2(m[r] - base[r]);
            m[r] = m_new;
            l[r] *= alpha[r];
        }
        if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
            for (int n = 0; n < VD / 8; ++n) {
                o[n][0] *= alpha[0]; o[n][1] *= alpha[0];
                o[n][2] *= alpha[1]; o[n][3] *= alpha[1];
            }
        }
#pragma unroll
        for (int n = 0; n < BN / 8; ++n) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float pv = pow2(sc[n][e] - base[e >> 1]);
                sc[n][e] = pv;
                l[e >> 1] += pv;
            }
        }
        // O += P V, sixteen keys a step, the weights in three bfloat16 terms
#pragma unroll
        for (int j = 0; j < BN / 16; ++j) {
            uint32_t pa[3][4];
#pragma unroll
            for (int q4 = 0; q4 < 4; ++q4) {
                const int n = 2 * j + (q4 >> 1), e = (q4 & 1) * 2;
                split3(sc[n][e], sc[n][e + 1], pa[0][q4], pa[1][q4], pa[2][q4]);
            }
            // four steps of 16 columns at a time, a term over all of them before the next: consecutive products on one
            // accumulator would wait for each other
#pragma unroll
            for (int n4 = 0; n4 < VD / 16; n4 += 4) {
                uint32_t vb[4][4];
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    ldmatrix_x4_trans(vb[u], Vs + (j * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * VLD + (n4 + u) * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int term = 2; term >= 0; --term) {          // smallest terms first
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        mma_bf16(o[2 * (n4 + u)], pa[term], vb[u][0], vb[u][1]);
                        mma_bf16(o[2 * (n4 + u) + 1], pa[term], vb[u][2], vb[u][3]);
                    }
                }
            }
        }
    }
    // the rows' sums over the four threads that share a row, the sink, the gate, the division
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = warp * 16 + g + r * 8;
        if (row >= nq_tile) continue;
        float inv = l[r] > 0.f ? 1.0f / l[r] : 0.f;
        if (p.sink && l[r] > 0.f) {
            const float z = p.sink_values ? p.sink_values[head] : 0.f;
            const float mr = m[r] * 0.6931471805599453f;          // as a power of e
            const float M = fmaxf(mr, z);
            const float w = expf(mr - M);
            inv = w / (l[r] * w + expf(z - M));
        }
        const size_t tok = (size_t)(q_beg + q0 + row);
        bf16* dst = p.out + tok * p.o_stride + (size_t)head * VD;
        const bf16* gt = p.gate ? p.gate + tok * p.gate_stride + (size_t)head * (p.gate_heads ? 1 : VD) : nullptr;
        const float head_gate = (gt && p.gate_heads) ? 1.0f / (1.0f + expf(-__bfloat162float(gt[0]))) : 1.f;
        if (p.turn_cos) {
            // the thread holds columns n * 8 + 2 tq (+ 1) for every n: a column and the one half a head on are both its own
            const float* cs = p.turn_cos + (size_t)qpos[r] * (VD / 2);
            const float* sn = p.turn_sin + (size_t)qpos[r] * (VD / 2);
#pragma unroll
            for (int n = 0; n < VD / 16; ++n) {
                const int col = n * 8 + 2 * tq;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float lo = o[n][2 * r + e], hi = o[n + VD / 16][2 * r + e];
                    const float c = cs[col + e], sv = sn[col + e];
                    o[n][2 * r + e] = lo * c + hi * sv;
                    o[n + VD / 16][2 * r + e] = hi * c - lo * sv;
                }
            }
        }
#pragma unroll
        for (int n = 0; n < VD / 8; ++n) {
            const int col = n * 8 + 2 * tq;
            float v0 = o[n][2 * r] * inv * head_gate, v1 = o[n][2 * r + 1] * inv * head_gate;
            if (gt && !p.gate_heads) {
                v0 *= 1.0f / (1.0f + expf(-__bfloat162float(gt[col])));
                v1 *= 1.0f / (1.0f + expf(-__bfloat162float(gt[col + 1])));
            }
            *reinterpret_cast<__nv_bfloat162*>(dst + col) = __floats2bfloat162_rn(v0, v1);
        }
    }
}

template <int HD, int VD, bool SHARED = false>
int launch(const Params& p, dim3 grid, cudaStream_t s) {
    const size_t smem = ((size_t)(BM + 2 * BN) * (HD + 8) + (SHARED ? 0 : (size_t)2 * BN * (VD + 8))) * sizeof(bf16) + (SHARED ? 2 * BN * sizeof(float) : 0);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(attention_mma_kernel<HD, VD, SHARED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) LLMK_FAIL("attention_mma: cannot raise shared memory to %zu: %s", smem, cudaGetErrorString(e));
        configured = true;
    }
    LLMK_CHECK_LAUNCH_RC("attention_mma", llmk_launch(attention_mma_kernel<HD, VD, SHARED>, grid, dim3(WARPS * 32), smem, s, true, p));
    return LLMK_OK;
}

// ------------------------------------------------------------------------------------- single tokens, keys in parts
constexpr int PROWS = 16;
constexpr int PSTAGES = 3;           // tiles of keys on their way
constexpr int PPAGES = 512;          // page ids of a part that are looked up once, in front of the first tile (longer parts: as they go)

template <int HD, int VD, bool SHARED>
struct PartsSmem {
    static constexpr int QLD = HD + 8, VLD = VD + 8, OLD = VD + 4;
    static constexpr size_t Q = (size_t)PROWS * QLD * sizeof(bf16);
    static constexpr size_t KV = ((size_t)PSTAGES * BN * QLD + (SHARED ? 0 : (size_t)PSTAGES * BN * VLD)) * sizeof(bf16);
    static constexpr size_t FACTORS = SHARED ? PSTAGES * BN * sizeof(float) : 0;
    static constexpr size_t OUT = ((size_t)PROWS * OLD + 2 * PROWS + 2 * WARPS * PROWS + 3 * 8 * PROWS) * sizeof(float);
    static constexpr size_t PAGES = PPAGES * sizeof(int);
    static constexpr size_t TOTAL = Q + KV + FACTORS + OUT + PAGES;
};

template <int HD, int VD, bool SHARED>
__global__ void __launch_bounds__(WARPS * 32) attention_mma_parts_kernel(Params p, int gc, int chunks, int parts) {
    using L = PartsSmem<HD, VD, SHARED>;
    constexpr int QLD = L::QLD, VLD = SHARED ? L::QLD : L::VLD, OLD = L::OLD;
    static_assert(!SHARED || HD == VD, "keys that are values have one width");
    extern __shared__ __align__(16) uint8_t smem_raw[];
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);
    bf16* Kbuf = Qs + PROWS * QLD;
    bf16* Vbuf = SHARED ? Kbuf : Kbuf + PSTAGES * BN * QLD;
    float* Sbuf = reinterpret_cast<float*>(smem_raw + L::Q + L::KV);
    float* Os = reinterpret_cast<float*>(smem_raw + L::Q + L::KV + L::FACTORS);      // [PROWS][OLD]
    float* Ml = Os + PROWS * OLD;                                                    // [PROWS] maxima, [PROWS] sums
    float* Wm = Ml + 2 * PROWS;                                                      // [WARPS][PROWS]
    float* Wl = Wm + WARPS * PROWS;
    float* Rm = Wl + WARPS * PROWS;                                                  // [8 parts][2 PROWS] the parts' maxima and sums
    float* Rw = Rm + 8 * 2 * PROWS;                                                  // [8 parts][PROWS] their weights
    int* pages = reinterpret_cast<int*>(smem_raw + L::Q + L::KV + L::FACTORS + L::OUT);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int g = lane >> 2, tq = lane & 3;
    pdl_launch_dependents();
    pdl_wait();
    const int s = blockIdx.x, part = blockIdx.z;
    const int G = p.nq / p.nkv;
    const int kvh = blockIdx.y / chunks, chunk = blockIdx.y % chunks;
    const int heads = min(gc, G - chunk * gc);                  // rows of this block
    const int head0 = kvh * G + chunk * gc;
    const int q_beg = p.cu_q[s], q_len = p.cu_q[s + 1] - q_beg, ctx = p.ctx_len[s];
    const bool live = q_len == 1 && ctx >= 1;
    const int qpos = ctx - 1;
    int k_beg = 0, k_end = 0;
    if (live) {
        int first = p.window > 0 ? max(0, qpos - p.window + 1) : 0;
        if (p.chunk > 0) first = max(first, qpos / p.chunk * p.chunk);
        const int size = ceil_div(ceil_div(qpos + 1 - first, parts), BN) * BN;       // whole tiles a part
        k_beg = first + part * size;
        k_end = min(qpos + 1, k_beg + size);
    }
    const int* bt = p.block_tables + (size_t)s * p.max_blocks;
    const int page_shift = shift_of(p.page_size);
    const int page0 = k_beg / p.page_size;
    const int n_pages = k_beg < k_end ? (k_end - 1) / p.page_size - page0 + 1 : 0;
    const bool staged = n_pages <= PPAGES;
    if (staged) {
        for (int i = threadIdx.x; i < n_pages; i += WARPS * 32) pages[i] = bt[page0 + i];
        __syncthreads();
    }

    constexpr int VECS = HD / 8 + (SHARED ? 0 : VD / 8);
    auto load_tile = [&](int t0, int buf) {
        bf16* Kd = Kbuf + buf * BN * QLD;
        bf16* Vd = Vbuf + buf * BN * VLD;
#pragma unroll 4
        for (int idx = threadIdx.x; idx < BN * VECS; idx += WARPS * 32) {
            const int key = idx / VECS, v = idx % VECS;
            const int kpos = t0 + key;
            bf16* dst = v < HD / 8 ? Kd + key * QLD + v * 8 : Vd + key * VLD + (v - HD / 8) * 8;
            const int at = quotient(kpos, p.page_size, page_shift);
            const int page = kpos < k_end ? (staged ? pages[at - page0] : bt[at]) : -1;
            if (page >= 0) {
                const int off = kpos - at * p.page_size;
                const size_t row = ((size_t)page * p.nkv + kvh) * p.page_size + off;
                cp_async16(dst, v < HD / 8 ? p.kcache + row * HD + v * 8 : p.vcache + row * VD + (v - HD / 8) * 8);
                if constexpr (SHARED) {
                    if (v == 0) cp_async4(Sbuf + buf * BN + key, p.k_scale + (size_t)page * p.page_size + off);
                }
            } else {
                *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
                if constexpr (SHARED) {
                    if (v == 0) Sbuf[buf * BN + key] = 0.f;
                }
            }
        }
        cp_async_commit();
    };
    // every turn asks for the tile two ahead; a group is committed for every turn, also where there is no tile left
#pragma unroll
    for (int i = 0; i < PSTAGES - 1; ++i) {
        if (k_beg + i * BN < k_end) load_tile(k_beg + i * BN, i);
        else cp_async_commit();
    }
    for (int idx = threadIdx.x; idx < PROWS * (HD / 8); idx += blockDim.x) {
        const int r = idx / (HD / 8), v = idx % (HD / 8);
        uint4 val = make_uint4(0, 0, 0, 0);
        if (live && r < heads) val = *reinterpret_cast<const uint4*>(p.q + (size_t)q_beg * p.q_stride + (size_t)(head0 + r) * HD + v * 8);
        *reinterpret_cast<uint4*>(Qs + r * QLD + v * 8) = val;
    }
    __syncthreads();
    uint32_t qf[HD / 16][4];
#pragma unroll
    for (int j = 0; j < HD / 16; ++j) ldmatrix_x4(qf[j], Qs + ((lane & 7) + ((lane >> 3) & 1) * 8) * QLD + j * 16 + (lane >> 4) * 8);

    float o[VD / 8][4];
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    constexpr float LOG2E = 1.4426950408889634f;
    const float scale2 = p.scale * LOG2E, cap2 = p.softcap * LOG2E, inv_cap2 = p.softcap > 0.f ? 1.0f / cap2 : 0.f;
    int turn = 0;
    for (int t0 = k_beg; t0 < k_end; t0 += BN, turn = turn + 1 == PSTAGES ? 0 : turn + 1) {
        cp_async_wait_but_one();  // this tile has arrived (the one after it may still be on its way) ...
        __syncthreads();          // ... for every thread, and the buffer of the tile before is free
        const int ahead = t0 + (PSTAGES - 1) * BN;
        if (ahead < k_end) load_tile(ahead, turn == 0 ? PSTAGES - 1 : turn - 1);
        else cp_async_commit();
        const int kw = warp * 16;                               // this warp's keys of the tile
        if (t0 + kw < k_end) {
            const bf16* Ks = Kbuf + turn * BN * QLD + kw * QLD;
            const bf16* Vs = Vbuf + turn * BN * VLD + kw * VLD;
            float sc[2][4];
#pragma unroll
            for (int n = 0; n < 2; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
            for (int j = 0; j < HD / 16; ++j) {
                uint32_t kb[4];
                ldmatrix_x4(kb, Ks + ((lane >> 4) * 8 + (lane & 7)) * QLD + j * 16 + ((lane >> 3) & 1) * 8);
                mma_bf16(sc[0], qf[j], kb[0], kb[1]);
                mma_bf16(sc[1], qf[j], kb[2], kb[3]);
            }
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int n = 0; n < 2; ++n) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int key = kw + n * 8 + 2 * tq + (e & 1);
                    float v = sc[n][e] * scale2;
                    if constexpr (SHARED) v *= Sbuf[turn * BN + key];
                    if (p.softcap > 0.f) v = cap2 * tanh_abs(v * inv_cap2);
                    v = t0 + key < k_end ? v : -INFINITY;
                    sc[n][e] = v;
                    mx[e >> 1] = fmaxf(mx[e >> 1], v);
                }
            }
            float alpha[2], base[2];
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                const float m_new = fmaxf(m[r], mx[r]);
                base[r] = m_new > -INFINITY ? m_new : 0.f;
                alpha[r] = pow2(m[r] - base[r]);
                m[r] = m_new;
                l[r] *= alpha[r];
            }
            if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
                for (int n = 0; n < VD / 8; ++n) {
                    o[n][0] *= alpha[0]; o[n][1] *= alpha[0];
                    o[n][2] *= alpha[1]; o[n][3] *= alpha[1];
                }
            }
            uint32_t pa[3][4];
#pragma unroll
            for (int q4 = 0; q4 < 4; ++q4) {
                const int n = q4 >> 1, e = (q4 & 1) * 2, r = e >> 1;
                const float p0 = pow2(sc[n][e] - base[r]), p1 = pow2(sc[n][e + 1] - base[r]);
                l[r] += p0 + p1;
                split3(p0, p1, pa[0][q4], pa[1][q4], pa[2][q4]);
            }
#pragma unroll
            for (int n4 = 0; n4 < VD / 16; n4 += 4) {
                uint32_t vb[4][4];
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    ldmatrix_x4_trans(vb[u], Vs + (((lane >> 3) & 1) * 8 + (lane & 7)) * VLD + (n4 + u) * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int term = 2; term >= 0; --term) {
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        mma_bf16(o[2 * (n4 + u)], pa[term], vb[u][0], vb[u][1]);
                        mma_bf16(o[2 * (n4 + u) + 1], pa[term], vb[u][2], vb[u][3]);
                    }
                }
            }
        }
    }
    // the warps' sums: one maximum per row over the block, the warps add up in their order
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        if (tq == 0) {
            Wm[warp * PROWS + g + 8 * r] = m[r];
            Wl[warp * PROWS + g + 8 * r] = l[r];
        }
    }
    __syncthreads();
    float fac[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        float M = -INFINITY;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) M = fmaxf(M, Wm[w * PROWS + g + 8 * r]);
        fac[r] = (m[r] == -INFINITY) ? 0.f : pow2(m[r] - M);
    }
    for (int w = 0; w < WARPS; ++w) {
        if (warp == w) {
#pragma unroll
            for (int n = 0; n < VD / 8; ++n) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    float* dst = Os + (g + 8 * (e >> 1)) * OLD + n * 8 + 2 * tq + (e & 1);
                    const float v = o[n][e] * fac[e >> 1];
                    *dst = w == 0 ? v : *dst + v;
                }
            }
        }
        __syncthreads();
    }
    if (threadIdx.x < PROWS) {
        float M = -INFINITY, sum = 0.f;
        for (int w = 0; w < WARPS; ++w) M = fmaxf(M, Wm[w * PROWS + threadIdx.x]);
        for (int w = 0; w < WARPS; ++w) {
            const float mw = Wm[w * PROWS + threadIdx.x];
            if (mw != -INFINITY) sum += pow2(mw - M) * Wl[w * PROWS + threadIdx.x];
        }
        Ml[threadIdx.x] = M;
        Ml[PROWS + threadIdx.x] = sum;
    }
    // the parts of this (token, key head) merge through each other's shared memory; every block finishes a share of the values
    cluster_sync_all();
    const uint32_t os = (uint32_t)__cvta_generic_to_shared(Os), ml = (uint32_t)__cvta_generic_to_shared(Ml);
    for (int i = threadIdx.x; i < parts * 2 * PROWS; i += WARPS * 32)
        Rm[i] = cluster_ld_f32(cluster_map_shared(ml + (i % (2 * PROWS)) * 4, i / (2 * PROWS)));
    __syncthreads();
    if (threadIdx.x < PROWS) {
        // a row's weights of the parts: 2^(m_part - M) over the sum of all of them (the sink among them)
        const int r = threadIdx.x;
        float M = -INFINITY;
        for (int pt = 0; pt < parts; ++pt) M = fmaxf(M, Rm[pt * 2 * PROWS + r]);
        const bool seen = M > -INFINITY;
        const float z = (p.sink && p.sink_values && r < heads) ? p.sink_values[head0 + r] * LOG2E : 0.f;
        if (p.sink && seen) M = fmaxf(M, z);
        float den = (p.sink && seen) ? pow2(z - M) : 0.f;
        for (int pt = 0; pt < parts; ++pt) {
            const float mp = Rm[pt * 2 * PROWS + r];
            const float w = mp == -INFINITY ? 0.f : pow2(mp - M);
            Rw[pt * PROWS + r] = w;
            den = fmaf(w, Rm[pt * 2 * PROWS + PROWS + r], den);
        }
        const float inv = den > 0.f ? 1.0f / den : 0.f;
        for (int pt = 0; pt < parts; ++pt) Rw[pt * PROWS + r] *= inv;
    }
    __syncthreads();
    if (q_len == 1) {
        for (int idx = part * (WARPS * 32) + threadIdx.x; idx < heads * VD; idx += parts * (WARPS * 32)) {
            const int r = idx / VD, d = idx % VD;
            float v[8];
#pragma unroll
            for (int pt = 0; pt < 8; ++pt) v[pt] = pt < parts ? cluster_ld_f32(cluster_map_shared(os + (r * OLD + d) * 4, pt)) : 0.f;
            float sum = 0.f;
#pragma unroll
            for (int pt = 0; pt < 8; ++pt)
                if (pt < parts) sum = fmaf(Rw[pt * PROWS + r], v[pt], sum);
            p.out[(size_t)q_beg * p.o_stride + (size_t)(head0 + r) * VD + d] = __float2bfloat16_rn(sum);
        }
    }
    cluster_sync_all();           // nobody leaves while its shared memory is read
}

template <int HD, int VD, bool SHARED>
int launch_parts(const Params& p, int n_seqs, int parts, cudaStream_t s) {
    const int G = p.nq / p.nkv;
    const int gc = G < PROWS ? G : PROWS;
    const int chunks = (G + gc - 1) / gc;
    constexpr size_t smem = PartsSmem<HD, VD, SHARED>::TOTAL;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(attention_mma_parts_kernel<HD, VD, SHARED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) LLMK_FAIL("attention_mma_parts: cannot raise shared memory to %zu: %s", smem, cudaGetErrorString(e));
        configured = true;
    }
    LLMK_CHECK_LAUNCH_RC("attention_mma_parts", llmk_launch_clusters(attention_mma_parts_kernel<HD, VD, SHARED>, dim3(n_seqs, p.nkv * chunks, parts),
                                                                     dim3(WARPS * 32), smem, s, true, dim3(1, 1, parts), p, gc, chunks, parts));
    return LLMK_OK;
}

}  // namespace

// Queries per tile (0: the kernel does not take these sizes).
LLMK_EXPORT int llmk_attention_mma_tile_queries(int nq, int nkv, int hd, int vd) {
    if (nkv <= 0 || nq <= 0 || nq % nkv != 0) return 0;
    if ((hd != 64 && hd != 128) || (vd != 64 && vd != 128)) return 0;
    return BM;
}

// out[t, nq*vd] (bfloat16) = attention of q[t] (bfloat16) over the paged cache [pages, nkv, page_size, hd | vd].
// tile_seq / tile_q0 list tiles of 64 queries; an entry with sequence -1 is skipped.
LLMK_EXPORT int llmk_attention_mma(void* out, long long o_stride, const void* q, long long q_stride, const void* kcache,
                                   const void* vcache, const int* block_tables, int max_blocks, const int* ctx_len, const int* cu_q,
                                   const int* tile_seq, const int* tile_q0, int n_tiles, int nq, int nkv, int hd, int vd,
                                   int page_size, int window, float scale, float softcap, int sink, const float* sink_values, const void* gate,
                                   long long gate_stride, int chunk, int gate_heads, const float* turn_cos, const float* turn_sin,
                                   const float* k_scale, void* stream) {
    if (n_tiles <= 0) return LLMK_OK;
    if (llmk_attention_mma_tile_queries(nq, nkv, hd, vd) == 0)
        LLMK_FAIL("attention_mma: not taken (heads %d/%d, key width %d and value width %d must be 64 or 128)", nq, nkv, hd, vd);
    if (q_stride % 8 != 0 || o_stride % 2 != 0 || !host_aligned16(q) || !host_aligned16(kcache) || !host_aligned16(vcache) ||
        (reinterpret_cast<uintptr_t>(out) & 3) != 0 || page_size <= 0)
        LLMK_FAIL("attention_mma: q and the cache must start on 16-byte boundaries, q's row stride a multiple of 8");
    if (nq > 65535) LLMK_FAIL("attention_mma: grid too large");
    if (k_scale && hd != vd) LLMK_FAIL("attention_mma: keys that are values have one width (%d, %d)", hd, vd);
    if (!k_scale && !vcache) LLMK_FAIL("attention_mma: no values");
    Params p;
    p.q = (const bf16*)q; p.kcache = (const bf16*)kcache; p.vcache = (const bf16*)vcache; p.out = (bf16*)out;
    p.gate = (const bf16*)gate; p.sink_values = sink_values; p.gate_heads = gate_heads ? 1 : 0;
    p.turn_cos = (turn_cos && turn_sin) ? turn_cos : nullptr; p.turn_sin = turn_sin; p.block_tables = block_tables; p.ctx_len = ctx_len; p.cu_q = cu_q;
    p.tile_seq = tile_seq; p.tile_q0 = tile_q0; p.q_stride = q_stride; p.o_stride = o_stride; p.gate_stride = gate_stride;
    p.max_blocks = max_blocks; p.nq = nq; p.nkv = nkv; p.page_size = page_size; p.window = window; p.sink = sink ? 1 : 0; p.chunk = chunk > 0 ? chunk : 0;
    p.scale = scale; p.softcap = softcap; p.k_scale = k_scale;
    dim3 grid(n_tiles, nq);
    cudaStream_t s = (cudaStream_t)stream;
    if (k_scale) return hd == 64 ? launch<64, 64, true>(p, grid, s) : launch<128, 128, true>(p, grid, s);
    if (hd == 64 && vd == 64) return launch<64, 64>(p, grid, s);
    if (hd == 64) return launch<64, 128>(p, grid, s);
    if (vd == 64) return launch<128, 64>(p, grid, s);
    return launch<128, 128>(p, grid, s);
}

// Steps of single tokens: sequence s < n_seqs owns the one query row cu_q[s] (or none), its visible keys are cut into `parts` (1 to 8)
// parts that merge inside a cluster.  Everything else as above; no gate, no turn back.
LLMK_EXPORT int llmk_attention_mma_parts(void* out, long long o_stride, const void* q, long long q_stride, const void* kcache,
                                         const void* vcache, const int* block_tables, int max_blocks, const int* ctx_len, const int* cu_q,
                                         int n_seqs, int nq, int nkv, int hd, int vd, int page_size, int window, float scale, float softcap,
                                         int sink, const float* sink_values, int chunk, const float* k_scale, int parts, void* stream) {
    if (n_seqs <= 0) return LLMK_OK;
    if (llmk_attention_mma_tile_queries(nq, nkv, hd, vd) == 0)
        LLMK_FAIL("attention_mma_parts: not taken (heads %d/%d, key width %d and value width %d must be 64 or 128)", nq, nkv, hd, vd);
    if (parts < 1 || parts > 8) LLMK_FAIL("attention_mma_parts: %d parts (1 to 8)", parts);
    if (k_scale && hd != vd) LLMK_FAIL("attention_mma_parts: keys that are values have one width (%d, %d)", hd, vd);
    if (!k_scale && !vcache) LLMK_FAIL("attention_mma_parts: no values");
    if (q_stride % 8 != 0 || !host_aligned16(q) || !host_aligned16(kcache) || !host_aligned16(vcache) || page_size <= 0)
        LLMK_FAIL("attention_mma_parts: q and the cache must start on 16-byte boundaries, q's row stride a multiple of 8");
    if ((long long)nkv * ceil_div(nq / nkv, PROWS) > 65535) LLMK_FAIL("attention_mma_parts: grid too large");
    Params p = {};
    p.q = (const bf16*)q; p.kcache = (const bf16*)kcache; p.vcache = (const bf16*)vcache; p.out = (bf16*)out;
    p.sink_values = sink_values; p.k_scale = k_scale; p.block_tables = block_tables; p.ctx_len = ctx_len; p.cu_q = cu_q;
    p.q_stride = q_stride; p.o_stride = o_stride; p.max_blocks = max_blocks; p.nq = nq; p.nkv = nkv; p.page_size = page_size;
    p.window = window; p.sink = sink ? 1 : 0; p.chunk = chunk > 0 ? chunk : 0; p.scale = scale; p.softcap = softcap;
    cudaStream_t s = (cudaStream_t)stream;
    if (k_scale) return hd == 64 ? launch_parts<64, 64, true>(p, n_seqs, parts, s) : launch_parts<128, 128, true>(p, n_seqs, parts, s);
    if (hd == 64 && vd == 64) return launch_parts<64, 64, false>(p, n_seqs, parts, s);
    if (hd == 64) return launch_parts<64, 128, false>(p, n_seqs, parts, s);
    if (vd == 64) return launch_parts<128, 64, false>(p, n_seqs, parts, s);
    return launch_parts<128, 128, false>(p, n_seqs, parts, s);
}
