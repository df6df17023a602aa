// Retention: linear attention with a constant decay per head, between its input product and its output product.
//
// Per head, with key channels d and value channels v, for the tokens of a sequence in order:
//     S[d][v] <- decay * S[d][v] + k_t[d] * v_t[v];      o_t[v] = sum_d S[d][v] * q_t[d]
// q and k are turned (rotate-half pairs over the first R channels) at the token's position and k is scaled first; every
// head's o_t is then divided by its root mean square over v and multiplied by silu(g_t).  The input is the product as
// 32-bit partial sums; a sequence's state is a 32-bit row addressed by slot.
//
//   tb_retention_step   one token per sequence: everything in one launch.  A CTA owns one head of one sequence and
//                       streams its state through registers; the first rows are fetched while the product before is
//                       still running.
//   tb_retention_chunks whole prompts in bfloat16, as matrix products over chunks of C tokens (mma.sync): with i, j
//                       places in a chunk and S the state before it,
//                           o_i = sum_{j <= i} decay^(i - j) (q_i . k_j) v_j + decay^(i + 1) S^T q_i
//                           S'  = decay^n S + sum_j decay^(n - 1 - j) k_j v_j^T           (n tokens in the chunk)
//                       in four launches: rows prepared (turned, scaled, padded, rounded once), each chunk's own sum E,
//                       the states before the chunks from the E (a scan over chunks, element by element), and the outputs
//                       with norm and gate (a cluster of CTAs owns a head, each of them 64 value channels; they
//                       exchange their sums of squares through distributed shared memory).
//   tb_retention_prep   the 32-bit rows [q | k | v | g] for the scan of gla.cu (any sizes, both dtypes)
//
// 32-bit: angles, rotation, decays, the state, o, its norm and the gate.  v is a product's output and is rounded to the
// activations' dtype, as every other mixer's values are.  In the chunk form the turned q and k are rounded once, as an
// attention kernel's are, and so are the weights (q_i . k_j) decay^(i - j) that meet v; but a token's own product q_i . k_i
// is taken in 32-bit from the unrounded numbers: where it is all there is (a sequence's first token) or nearly all (a
// fast decay), the norm leaves little of it but its sign, which rounding must not turn.  The state and the decayed keys
// that enter it are not rounded to 16 bits: they are multiplied as sums of two bfloat16 numbers (16 bits of mantissa).
#include <cooperative_groups.h>
#include "common.cuh"

namespace cg = cooperative_groups;

TB_EXPORT_ERROR()

struct RetentionArgs {
    const float* part; int n_splits; long long split_stride, row_stride;    // [splits][T] rows of q (H*D), k (H*D), v (H*V), g (H*V)
    int heads, D, V;
    int rotary_dim; const float* inv_freq;            // [rotary_dim / 2]
    float k_scale, eps;
    const float* decay;                               // [H]
    const int* positions; const int* token_seq; const int* seq_start; const int* slot_ids;
    float* state; long long state_stride;             // [slots][H*D*V]
    void* rows;                                       // prep: float [T][2 H*D + 2 H*V]; chunks: bf16 [T][H*(2 DP + VP)]
    void* out;                                        // [T][H*V]
    int batch, n_tokens;
    float* chunk_sum; bf16* chunk_hi; bf16* chunk_lo; // chunks: [batch][n_chunks][H][DP][VP] each
    int chunk_len, n_chunks, row_blocks, DP, VP;      // DP, VP: D and V padded (64, 128, 256; multiples of 64)
    float* qk;                                        // chunks: [T][H] every token's own q . k, in 32-bit
};

// The argument block's size, for the Python mirror's check.
extern "C" int tb_retention_args_bytes() { return (int)sizeof(RetentionArgs); }

// A value as the activations' dtype keeps it.
template <typename T> __device__ __forceinline__ float kept(float v) { return to_f<T>(from_f<T>(v)); }

// A launch of clusters of `cluster` CTAs along x (with the attribute that every launch of this library has).
template <typename... KArgs, typename... Args>
static inline void launch_cluster(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, int cluster, cudaStream_t stream, Args&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster; attr[1].val.clusterDim.y = 1; attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr; cfg.numAttrs = 2;
    cudaLaunchKernelEx(&cfg, kern, KArgs(args)...);
}

constexpr int VT = 64;                                // value channels per CTA

// ---------------------------------------------------------------------------
// Rows for the generic scan
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) retention_prep_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    extern __shared__ float cs[];                     // cos[half], sin[half]
    const int t = blockIdx.x;
    const int HD = a.heads * a.D, HV = a.heads * a.V, half = a.rotary_dim >> 1;
    float* sn = cs + half;
    pdl_wait();
    const int pos = a.positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf((float)pos * a.inv_freq[i], &sn[i], &cs[i]);
    __syncthreads();
    const float* src = a.part + (size_t)t * a.row_stride;
    float* dst = (float*)a.rows + (size_t)t * (2 * HD + 2 * HV);
    auto at = [&](int c) {
        float s = src[c];
        for (int sp = 1; sp < a.n_splits; sp++) s += src[(size_t)sp * a.split_stride + c];
        return s;
    };
    for (int c = threadIdx.x; c < 2 * HD; c += blockDim.x) {
        const int i = c % a.D;
        const float scale = c < HD ? 1.f : a.k_scale;
        if (i < half) {
            const float u = at(c), w = at(c + half);
            dst[c] = (u * cs[i] - w * sn[i]) * scale;
            dst[c + half] = (w * cs[i] + u * sn[i]) * scale;
        } else if (i >= 2 * half) {
            dst[c] = at(c) * scale;
        }
    }
    for (int c = 2 * HD + threadIdx.x; c < 2 * HD + 2 * HV; c += blockDim.x) {
        const float v = at(c);
        dst[c] = c < 2 * HD + HV ? kept<T>(v) : v;
    }
}

// ---------------------------------------------------------------------------
// One token per sequence
// ---------------------------------------------------------------------------
// A lane owns NC groups of four neighbouring value channels; LPR lanes (16 or 32) span a row of the state, so a warp
// takes 32 / LPR key channels at a time, with 16-byte loads and stores.

template <typename T, int NC, int LPR>
__global__ void __launch_bounds__(1024) retention_step_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[33];
    constexpr int RPW = 32 / LPR;                     // rows of the state per pass of a warp
    constexpr int STEP_ROWS = NC > 2 ? 2 : 4;         // passes whose loads are in flight together
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarp = blockDim.x >> 5;
    const int h = blockIdx.x, b = blockIdx.y;
    const int D = a.D, V = a.V, HD = a.heads * D, HV = a.heads * V, half = a.rotary_dim >> 1;
    float* raw_s = sm;                                // [2 D] q, k as the product left them
    float* q_s = raw_s + 2 * D;                       // [D]
    float* k_s = q_s + D;                             // [D]
    float* cs = k_s + D;                              // [D / 2 rounded up] each
    float* sn = cs + (D + 1) / 2;
    float* v_s = sm + (((5 * D + 2) + 3) & ~3);       // [V], 16-byte aligned
    float* g_s = v_s + V;                             // [V]
    float* part_s = g_s + V;                          // [nwarp][V]
    const int sub = lane % LPR, r_in = lane / LPR;
    // The step's integer inputs were copied before its first kernel, and this sequence's state was last written in an
    // earlier step (or zeroed when its slot was claimed): both may be read ahead of the wait.
    float* st = a.state + (size_t)a.slot_ids[b] * a.state_stride + (size_t)h * D * V;
    const int passes = (D + nwarp * RPW - 1) / (nwarp * RPW);
    float4 S[STEP_ROWS][NC];
    auto row_of = [&](int p) { return (p * nwarp + warp) * RPW + r_in; };
    auto fetch = [&](int p0) {
#pragma unroll
        for (int u = 0; u < STEP_ROWS; u++) {
            const int d = row_of(p0 + u);
#pragma unroll
            for (int c = 0; c < NC; c++) {
                const int v = (c * LPR + sub) * 4;
                S[u][c] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (p0 + u < passes && d < D && v < V) S[u][c] = *(const float4*)(st + (size_t)d * V + v);
            }
        }
    };
    fetch(0);
    const float dec = a.decay[h];
    const int pos = a.positions[b];
    for (int i = tid; i < half; i += blockDim.x) sincosf((float)pos * a.inv_freq[i], &sn[i], &cs[i]);
    pdl_wait();
    const float* src = a.part + (size_t)b * a.row_stride;
    for (int u = tid; u < 2 * D + 2 * V; u += blockDim.x) {
        const int c = u < D ? h * D + u : u < 2 * D ? HD + h * D + (u - D) : u < 2 * D + V ? 2 * HD + h * V + (u - 2 * D)
                                                                                            : 2 * HD + HV + h * V + (u - 2 * D - V);
        float s = src[c];
#pragma unroll 8
        for (int sp = 1; sp < a.n_splits; sp++) s += src[(size_t)sp * a.split_stride + c];
        if (u < 2 * D) raw_s[u] = s;
        else if (u < 2 * D + V) v_s[u - 2 * D] = kept<T>(s);
        else g_s[u - 2 * D - V] = s;
    }
    __syncthreads();
    for (int u = tid; u < 2 * D; u += blockDim.x) {
        const int w = u >= D, i = u - w * D;
        const float* x = raw_s + w * D;
        const float y = i < half ? x[i] * cs[i] - x[i + half] * sn[i]
                      : i < 2 * half ? x[i] * cs[i - half] + x[i - half] * sn[i - half] : x[i];
        if (w) k_s[i] = y * a.k_scale; else q_s[i] = y;
    }
    __syncthreads();
    float4 acc[NC];
#pragma unroll
    for (int c = 0; c < NC; c++) acc[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int p0 = 0; p0 < passes; p0 += STEP_ROWS) {
        if (p0 > 0) fetch(p0);
#pragma unroll
        for (int u = 0; u < STEP_ROWS; u++) {
            const int d = row_of(p0 + u);
            const bool in = p0 + u < passes && d < D;
            const float kk = in ? k_s[d] : 0.f, qq = in ? q_s[d] : 0.f;
#pragma unroll
            for (int c = 0; c < NC; c++) {
                const int v = (c * LPR + sub) * 4;
                if (!in || v >= V) continue;
                const float4 x = *(const float4*)(v_s + v);
                float4& s = S[u][c];
                s.x = fmaf(dec, s.x, kk * x.x); s.y = fmaf(dec, s.y, kk * x.y);
                s.z = fmaf(dec, s.z, kk * x.z); s.w = fmaf(dec, s.w, kk * x.w);
                acc[c].x = fmaf(s.x, qq, acc[c].x); acc[c].y = fmaf(s.y, qq, acc[c].y);
                acc[c].z = fmaf(s.z, qq, acc[c].z); acc[c].w = fmaf(s.w, qq, acc[c].w);
                *(float4*)(st + (size_t)d * V + v) = s;
            }
        }
    }
    if (LPR == 16) {                                  // the two rows of a pass meet
#pragma unroll
        for (int c = 0; c < NC; c++) {
            acc[c].x += __shfl_xor_sync(0xffffffffu, acc[c].x, 16); acc[c].y += __shfl_xor_sync(0xffffffffu, acc[c].y, 16);
            acc[c].z += __shfl_xor_sync(0xffffffffu, acc[c].z, 16); acc[c].w += __shfl_xor_sync(0xffffffffu, acc[c].w, 16);
        }
    }
#pragma unroll
    for (int c = 0; c < NC; c++) {
        const int v = (c * LPR + sub) * 4;
        if (r_in == 0 && v < V) *(float4*)(part_s + (size_t)warp * V + v) = acc[c];
    }
    __syncthreads();
    // a thread sums up to two channels (V is at most twice the smallest block)
    float o[2] = {0.f, 0.f};
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int v = tid + e * blockDim.x;
        if (v < V) for (int w = 0; w < nwarp; w++) o[e] += part_s[(size_t)w * V + v];
    }
    const float ss = block_sum(o[0] * o[0] + o[1] * o[1], red);
    const float r = 1.f / sqrtf(ss / (float)V + a.eps);
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int v = tid + e * blockDim.x;
        if (v >= V) continue;
        const float g = g_s[v];
        ((T*)a.out)[(size_t)b * HV + (size_t)h * V + v] = from_f<T>(o[e] * r * (g / (1.f + expf(-g))));
    }
}

// ---------------------------------------------------------------------------
// Whole prompts as products over chunks
// ---------------------------------------------------------------------------
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;                     // 0 source bytes: the 16 destination bytes become zero
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t* r) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t* r) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *(uint32_t*)&h;
}
// Two numbers as the sum of two bfloat16 pairs.
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

// Rows of bfloat16 [H][DP] q, [H][DP] k, [H][VP] v per token: q and k turned, k scaled, zeros in the padding.
// VEC: D, V and half of the rotated part are multiples of four and the partial sums 16-byte aligned.
template <bool VEC>
__global__ void __launch_bounds__(256) retention_rows_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    __shared__ __align__(16) float cs[128], sn[128];
    const int t = blockIdx.x;
    const int H = a.heads, D = a.D, V = a.V, DP = a.DP, VP = a.VP, HD = H * D, half = a.rotary_dim >> 1;
    const int pos = a.positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf((float)pos * a.inv_freq[i], &sn[i], &cs[i]);
    pdl_wait();
    __syncthreads();
    const float* src = a.part + (size_t)t * a.row_stride;
    bf16* dst = (bf16*)a.rows + (size_t)t * H * (2 * DP + VP);
    if (VEC) {
        auto at = [&](int c) {
            float4 s = *(const float4*)(src + c);
            for (int sp = 1; sp < a.n_splits; sp++) {
                const float4 x = *(const float4*)(src + (size_t)sp * a.split_stride + c);
                s.x += x.x; s.y += x.y; s.z += x.z; s.w += x.w;
            }
            return s;
        };
        const int vq = VP >> 2, lane = threadIdx.x & 31;
        // a warp makes a head's q and k together: four numbers (and their rotation partners) of both per lane
        for (int h = threadIdx.x >> 5; h < H; h += blockDim.x >> 5) {
            float dot = 0.f;
            for (int i = lane << 2; i < DP; i += 128) {
                if (i >= half && i < 2 * half) continue;                 // made together with its partner
                bf16* qd = dst + (size_t)h * DP + i;
                bf16* kd = dst + (size_t)(H + h) * DP + i;
                float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
                if (i < D) { q = at(h * D + i); k = at(HD + h * D + i); }
                if (i < half) {
                    const float4 q2 = at(h * D + i + half), k2 = at(HD + h * D + i + half);
                    const float4 c = *(const float4*)(cs + i), s = *(const float4*)(sn + i);
                    auto turn = [&](float4& x, const float4& w) {
                        const float4 lo = make_float4(x.x * c.x - w.x * s.x, x.y * c.y - w.y * s.y, x.z * c.z - w.z * s.z, x.w * c.w - w.w * s.w);
                        const float4 hi = make_float4(w.x * c.x + x.x * s.x, w.y * c.y + x.y * s.y, w.z * c.z + x.z * s.z, w.w * c.w + x.w * s.w);
                        x = lo;
                        return hi;
                    };
                    const float4 qh = turn(q, q2);
                    float4 kh = turn(k, k2);
                    kh.x *= a.k_scale; kh.y *= a.k_scale; kh.z *= a.k_scale; kh.w *= a.k_scale;
                    dot += qh.x * kh.x + qh.y * kh.y + qh.z * kh.z + qh.w * kh.w;
                    *(uint2*)(qd + half) = make_uint2(pack_bf16(qh.x, qh.y), pack_bf16(qh.z, qh.w));
                    *(uint2*)(kd + half) = make_uint2(pack_bf16(kh.x, kh.y), pack_bf16(kh.z, kh.w));
                }
                k.x *= a.k_scale; k.y *= a.k_scale; k.z *= a.k_scale; k.w *= a.k_scale;
                dot += q.x * k.x + q.y * k.y + q.z * k.z + q.w * k.w;
                *(uint2*)qd = make_uint2(pack_bf16(q.x, q.y), pack_bf16(q.z, q.w));
                *(uint2*)kd = make_uint2(pack_bf16(k.x, k.y), pack_bf16(k.z, k.w));
            }
            dot = warp_sum(dot);
            if (lane == 0) a.qk[(size_t)t * H + h] = dot;
        }
#pragma unroll 2
        for (int u = threadIdx.x; u < H * vq; u += blockDim.x) {
            const int hs = u / vq, i = (u - hs * vq) << 2;
            uint2 y = make_uint2(0u, 0u);
            if (i < V) { const float4 x = at(2 * HD + hs * V + i); y = make_uint2(pack_bf16(x.x, x.y), pack_bf16(x.z, x.w)); }
            *(uint2*)(dst + (size_t)2 * H * DP + (size_t)hs * VP + i) = y;
        }
    } else {
        auto at = [&](int c) {
            float s = src[c];
            for (int sp = 1; sp < a.n_splits; sp++) s += src[(size_t)sp * a.split_stride + c];
            return s;
        };
        const int lane = threadIdx.x & 31;
        for (int h = threadIdx.x >> 5; h < H; h += blockDim.x >> 5) {
            float dot = 0.f;
            for (int i = lane; i < DP; i += 32) {
                float y[2];
#pragma unroll
                for (int w = 0; w < 2; w++) {
                    const int c = (w * H + h) * D + i;
                    y[w] = i < half ? at(c) * cs[i] - at(c + half) * sn[i]
                         : i < 2 * half ? at(c) * cs[i - half] + at(c - half) * sn[i - half] : i < D ? at(c) : 0.f;
                    if (w) y[w] *= a.k_scale;
                    dst[(size_t)(w * H + h) * DP + i] = __float2bfloat16_rn(y[w]);
                }
                dot = fmaf(y[0], y[1], dot);
            }
            dot = warp_sum(dot);
            if (lane == 0) a.qk[(size_t)t * H + h] = dot;
        }
        for (int u = threadIdx.x; u < H * VP; u += blockDim.x) {
            const int hs = u / VP, i = u - hs * VP;
            dst[(size_t)2 * H * DP + u] = __float2bfloat16_rn(i < V ? at(2 * HD + hs * V + i) : 0.f);
        }
    }
}

constexpr int CT = 256;                               // threads of the chunk kernels: eight warps
constexpr int KB = 64;                                // tokens per tile of keys and values
constexpr int VPITCH = VT * 2 + 16;                   // bytes per shared-memory row of 64 values (ldmatrix without bank conflicts)

// ROWS token rows [row0, row0 + ROWS) of COLS bfloat16 columns into padded shared rows; rows from row_end on become zero.
template <int ROWS, int COLS>
__device__ __forceinline__ void load_rows(uint8_t* dst, const bf16* src, long long stride, int row0, int row_end) {
    constexpr int CPR = COLS / 8, PITCH = COLS * 2 + 16;
#pragma unroll 4
    for (int c = threadIdx.x; c < ROWS * CPR; c += CT) {
        const int r = c / CPR, ch = c % CPR;
        const bool valid = row0 + r < row_end;
        cp_async16(dst + r * PITCH + ch * 16, src + (size_t)(valid ? row0 + r : row0) * stride + ch * 8, valid);
    }
}

// E = sum_j decay^(n - 1 - j) k_j v_j^T of one chunk: 64 value channels of one head.
template <int DP>
__global__ void __launch_bounds__(CT) retention_sum_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    constexpr int KPITCH = DP * 2 + 16;
    constexpr int MT = DP / 16;                       // 16-channel tiles of E
    constexpr int NW = MT >= 8 ? 1 : 8 / MT;          // warps that share a tile's 64 columns
    constexpr int MPW = MT >= 8 ? MT / 8 : 1;         // tiles per warp
    constexpr int NT = 8 / NW;                        // 8-column pieces per warp
    extern __shared__ __align__(128) uint8_t smem[];
    uint8_t* sK = smem;                               // [2][KB][KPITCH]
    uint8_t* sV = sK + 2 * KB * KPITCH;               // [2][KB][VPITCH]
    float* pw = (float*)(sV + 2 * KB * VPITCH);       // [chunk_len] decay^n
    const int h = blockIdx.y, b = blockIdx.z / a.n_chunks, chunk = blockIdx.z % a.n_chunks;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int s0 = a.seq_start[b], len = a.seq_start[b + 1] - s0;
    const int c0 = chunk * a.chunk_len, n = min(a.chunk_len, len - c0);
    if (n <= 0) return;
    const float dec = a.decay[h];
    for (int i = threadIdx.x; i < a.chunk_len; i += CT) pw[i] = powf(dec, (float)i);
    const long long stride = (long long)a.heads * (2 * a.DP + a.VP);
    const bf16* kb = (const bf16*)a.rows + (size_t)(s0 + c0) * stride + (size_t)(a.heads + h) * DP;
    const bf16* vb = (const bf16*)a.rows + (size_t)(s0 + c0) * stride + (size_t)2 * a.heads * DP + (size_t)h * a.VP + blockIdx.x * VT;
    pdl_wait();
    load_rows<KB, DP>(sK, kb, stride, 0, n);
    load_rows<KB, VT>(sV, vb, stride, 0, n);
    cp_async_commit();
    const int m0 = (warp / NW) * MPW * 16, n0 = (warp % NW) * NT * 8;
    float acc[MPW][NT][4];
#pragma unroll
    for (int m = 0; m < MPW; m++)
#pragma unroll
        for (int j = 0; j < NT; j++) { acc[m][j][0] = acc[m][j][1] = acc[m][j][2] = acc[m][j][3] = 0.f; }
    const int nb = (n + KB - 1) / KB;
    for (int kb_i = 0; kb_i < nb; kb_i++) {
        const int st = kb_i & 1;
        if (kb_i + 1 < nb) {
            load_rows<KB, DP>(sK + (st ^ 1) * KB * KPITCH, kb, stride, (kb_i + 1) * KB, n);
            load_rows<KB, VT>(sV + (st ^ 1) * KB * VPITCH, vb, stride, (kb_i + 1) * KB, n);
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint8_t* ks = sK + st * KB * KPITCH;
        const uint8_t* vs = sV + st * KB * VPITCH;
#pragma unroll
        for (int kk = 0; kk < KB / 16; kk++) {
            // weights of this lane's four tokens (places in the chunk; those past its end hold zero rows)
            const int j0 = n - 1 - (kb_i * KB + kk * 16 + 2 * t);
            const float w0 = pw[max(j0, 0)], w1 = pw[max(j0 - 1, 0)], w2 = pw[max(j0 - 8, 0)], w3 = pw[max(j0 - 9, 0)];
            uint32_t vbf[NT / 2][4];
#pragma unroll
            for (int j = 0; j < NT; j += 2)
                ldsm_x4_t(smem_addr(vs + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * VPITCH + (n0 + j * 8 + (lane >> 4) * 8) * 2), vbf[j / 2]);
#pragma unroll
            for (int m = 0; m < MPW; m++) {
                uint32_t k[4], hi[4], lo[4];
                ldsm_x4_t(smem_addr(ks + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * KPITCH + (m0 + m * 16 + ((lane >> 3) & 1) * 8) * 2), k);
#pragma unroll
                for (int e = 0; e < 4; e++)
                    split_bf16(__uint_as_float(k[e] << 16) * (e < 2 ? w0 : w2), __uint_as_float(k[e] & 0xffff0000u) * (e < 2 ? w1 : w3), hi[e], lo[e]);
#pragma unroll
                for (int j = 0; j < NT; j++) {
                    mma_bf16(acc[m][j], hi, vbf[j / 2][(j & 1) * 2], vbf[j / 2][(j & 1) * 2 + 1]);
                    mma_bf16(acc[m][j], lo, vbf[j / 2][(j & 1) * 2], vbf[j / 2][(j & 1) * 2 + 1]);
                }
            }
        }
        __syncthreads();
    }
    float* E = a.chunk_sum + (((size_t)b * a.n_chunks + chunk) * a.heads + h) * DP * a.VP + blockIdx.x * VT;
#pragma unroll
    for (int m = 0; m < MPW; m++)
#pragma unroll
        for (int j = 0; j < NT; j++) {
            const int d = m0 + m * 16 + g, c = n0 + j * 8 + 2 * t;
            *(float2*)(E + (size_t)d * a.VP + c) = make_float2(acc[m][j][0], acc[m][j][1]);
            *(float2*)(E + (size_t)(d + 8) * a.VP + c) = make_float2(acc[m][j][2], acc[m][j][3]);
        }
}

// The state before every chunk, as two bfloat16 numbers, and the state after the last token.  A thread owns two elements.
__global__ void __launch_bounds__(256) retention_fold_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    const int DP = a.DP, VP = a.VP, D = a.D, V = a.V;
    const int per = DP * VP / 2;
    const int b = blockIdx.z, h = blockIdx.y;
    const int e = blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= per) return;
    const int d = e / (VP / 2), v = (e - d * (VP / 2)) * 2;
    const int len = a.seq_start[b + 1] - a.seq_start[b];
    const int n_chunks = (len + a.chunk_len - 1) / a.chunk_len;
    float* st = a.state + (size_t)a.slot_ids[b] * a.state_stride + ((size_t)h * D + d) * V + v;
    const bool ok0 = d < D && v < V, ok1 = d < D && v + 1 < V;
    const float dec = a.decay[h], full = powf(dec, (float)a.chunk_len);
    pdl_wait();
    float s0 = ok0 ? st[0] : 0.f, s1 = ok1 ? st[1] : 0.f;
    const size_t step = (size_t)a.heads * DP * VP;
    const size_t at = ((size_t)b * a.n_chunks * a.heads + h) * DP * VP + (size_t)d * VP + v;
    for (int c0 = 0; c0 < n_chunks; c0 += 8) {         // eight chunks' sums on their way together
        float2 E[8];
#pragma unroll
        for (int u = 0; u < 8; u++) if (c0 + u < n_chunks) E[u] = *(const float2*)(a.chunk_sum + at + (c0 + u) * step);
#pragma unroll
        for (int u = 0; u < 8; u++)
            if (c0 + u < n_chunks) {
                uint32_t hi, lo;
                split_bf16(s0, s1, hi, lo);
                *(uint32_t*)(a.chunk_hi + at + (c0 + u) * step) = hi;
                *(uint32_t*)(a.chunk_lo + at + (c0 + u) * step) = lo;
                const bool last = c0 + u == n_chunks - 1;
                const float p = last ? powf(dec, (float)(len - (c0 + u) * a.chunk_len)) : full;
                s0 = fmaf(p, s0, E[u].x);
                s1 = fmaf(p, s1, E[u].y);
            }
    }
    if (n_chunks > 0) {
        if (ok0) st[0] = s0;
        if (ok1) st[1] = s1;
    }
}

// Outputs of 128 tokens of one head, 64 value channels per CTA; the cluster's CTAs together hold the head.
constexpr int RB = 128;
template <int DP>
__global__ void __launch_bounds__(CT) retention_out_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    constexpr int KPITCH = DP * 2 + 16;
    constexpr int STAGE = KB * (KPITCH + VPITCH);
    constexpr int Q_BYTES = RB * KPITCH, S_BYTES = DP * VPITCH;
    extern __shared__ __align__(128) uint8_t smem[];
    uint8_t* sQ = smem;                               // [RB][KPITCH], then a tile of keys and values
    uint8_t* sHi = sQ + (Q_BYTES > STAGE ? Q_BYTES : STAGE);     // [DP][VPITCH]
    uint8_t* sLo = sHi + S_BYTES;                     // [DP][VPITCH]; both then another tile
    float* pw = (float*)(sHi + (2 * S_BYTES > STAGE ? 2 * S_BYTES : STAGE));      // [chunk_len + 1] decay^n
    float* row_ss = pw + a.chunk_len + 1;             // [RB]
    cg::cluster_group cluster = cg::this_cluster();
    const int h = blockIdx.y, b = blockIdx.z / a.row_blocks, rb = blockIdx.z % a.row_blocks;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int s0 = a.seq_start[b], len = a.seq_start[b + 1] - s0;
    const int r0 = rb * RB;
    if (r0 >= len) return;                            // the whole cluster leaves
    const int chunk = r0 / a.chunk_len, c0 = chunk * a.chunk_len;         // chunks are whole row blocks
    const float dec = a.decay[h];
    for (int i = threadIdx.x; i <= a.chunk_len; i += CT) pw[i] = powf(dec, (float)i);
    const long long stride = (long long)a.heads * (2 * a.DP + a.VP);
    const bf16* qb = (const bf16*)a.rows + (size_t)s0 * stride + (size_t)h * DP;
    const bf16* kb = qb + (size_t)a.heads * DP;
    const bf16* vb = (const bf16*)a.rows + (size_t)s0 * stride + (size_t)2 * a.heads * DP + (size_t)h * a.VP + blockIdx.x * VT;
    const size_t at = (((size_t)b * a.n_chunks + chunk) * a.heads + h) * DP * a.VP + blockIdx.x * VT;
    pdl_wait();
    load_rows<RB, DP>(sQ, qb, stride, r0, len);
    cp_async_commit();
    load_rows<DP, VT>(sHi, a.chunk_hi + at, a.VP, 0, DP);
    load_rows<DP, VT>(sLo, a.chunk_lo + at, a.VP, 0, DP);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    uint32_t q[DP / 16][4];
#pragma unroll
    for (int ks = 0; ks < DP / 16; ks++) ldsm_x4(smem_addr(sQ + (warp * 16 + (lane & 15)) * KPITCH + (ks * 16 + (lane >> 4) * 8) * 2), q[ks]);
    __syncthreads();                                  // the queries are in registers: their place takes the first tile
    const int j_end = min(len, r0 + RB);              // keys c0 .. j_end - 1
    const int nb = (j_end - c0 + KB - 1) / KB;
    auto stage_of = [&](int i) { return (i & 1) ? sHi : sQ; };
    load_rows<KB, DP>(stage_of(0), kb, stride, c0, len);
    load_rows<KB, VT>(stage_of(0) + KB * KPITCH, vb, stride, c0, len);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    // ---- what the state before the chunk gives
    float o[8][4];
#pragma unroll
    for (int j = 0; j < 8; j++) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
#pragma unroll
    for (int p = 0; p < 2; p++) {
        const uint8_t* s = p ? sLo : sHi;
#pragma unroll
        for (int ks = 0; ks < DP / 16; ks++)
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                uint32_t f[4];
                ldsm_x4_t(smem_addr(s + (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * VPITCH + (j * 8 + (lane >> 4) * 8) * 2), f);
                mma_bf16(o[j], q[ks], f[0], f[1]);
                mma_bf16(o[j + 1], q[ks], f[2], f[3]);
            }
    }
    const int row_a = r0 + warp * 16 + g - c0, row_b = row_a + 8;         // places in the chunk
    {
        const float fa = pw[row_a + 1], fb = pw[row_b + 1];
#pragma unroll
        for (int j = 0; j < 8; j++) { o[j][0] *= fa; o[j][1] *= fa; o[j][2] *= fb; o[j][3] *= fb; }
    }
    __syncthreads();                                  // the state's place takes the second tile
    const int last_row = r0 - c0 + warp * 16 + 15;    // of this warp
    const float own_a = a.qk[(size_t)min(s0 + c0 + row_a, s0 + len - 1) * a.heads + h];
    const float own_b = a.qk[(size_t)min(s0 + c0 + row_b, s0 + len - 1) * a.heads + h];
    for (int i = 0; i < nb; i++) {
        if (i + 1 < nb) {
            load_rows<KB, DP>(stage_of(i + 1), kb, stride, c0 + (i + 1) * KB, len);
            load_rows<KB, VT>(stage_of(i + 1) + KB * KPITCH, vb, stride, c0 + (i + 1) * KB, len);
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint8_t* ks_ = stage_of(i);
        const uint8_t* vs = ks_ + KB * KPITCH;
        if (i * KB <= last_row) {
            // two halves of 32 keys: weights stay in registers
#pragma unroll
            for (int hf = 0; hf < 2; hf++) {
                const int j0 = i * KB + hf * 32;
                if (j0 > last_row) break;
                float s[4][4];
#pragma unroll
                for (int n = 0; n < 4; n++) { s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f; }
#pragma unroll
                for (int ks = 0; ks < DP / 16; ks++)
#pragma unroll
                    for (int n = 0; n < 4; n += 2) {
                        uint32_t f[4];
                        ldsm_x4(smem_addr(ks_ + (hf * 32 + n * 8 + (lane >> 4) * 8 + (lane & 7)) * KPITCH + (ks * 16 + ((lane >> 3) & 1) * 8) * 2), f);
                        mma_bf16(s[n], q[ks], f[0], f[1]);
                        mma_bf16(s[n + 1], q[ks], f[2], f[3]);
                    }
                uint32_t p[2][4];
#pragma unroll
                for (int n = 0; n < 4; n++) {
                    const int j = j0 + n * 8 + 2 * t;
                    float x[4];
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int dist = ((e < 2) ? row_a : row_b) - (j + (e & 1));
                        x[e] = dist > 0 ? s[n][e] * pw[max(dist, 0)] : dist == 0 ? (e < 2 ? own_a : own_b) : 0.f;
                    }
                    p[n >> 1][(n & 1) * 2] = pack_bf16(x[0], x[1]);
                    p[n >> 1][(n & 1) * 2 + 1] = pack_bf16(x[2], x[3]);
                }
#pragma unroll
                for (int kk = 0; kk < 2; kk++)
#pragma unroll
                    for (int j = 0; j < 8; j += 2) {
                        uint32_t f[4];
                        ldsm_x4_t(smem_addr(vs + (hf * 32 + kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * VPITCH + (j * 8 + (lane >> 4) * 8) * 2), f);
                        mma_bf16(o[j], p[kk], f[0], f[1]);
                        mma_bf16(o[j + 1], p[kk], f[2], f[3]);
                    }
            }
        }
        __syncthreads();
    }
    // ---- the gate's columns, on their way while the CTAs exchange their sums
    const int HD = a.heads * a.D, HV = a.heads * a.V;
    const bool pairs = a.n_splits == 1 && (a.V & 1) == 0 && (a.row_stride & 1) == 0 && ((uintptr_t)a.part & 7) == 0;
    float2 gv[2][8];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int row = r0 + warp * 16 + g + e * 8;
        const float* gp = a.part + (size_t)(s0 + min(row, len - 1)) * a.row_stride + 2 * HD + HV + (size_t)h * a.V;
#pragma unroll
        for (int j = 0; j < 8; j++) {
            const int c = blockIdx.x * VT + j * 8 + 2 * t;
            gv[e][j] = make_float2(0.f, 0.f);
            if (pairs) {
                if (c < a.V) gv[e][j] = __ldg((const float2*)(gp + c));
            } else {
                for (int sp = 0; sp < a.n_splits; sp++) {
                    if (c < a.V) gv[e][j].x += gp[(size_t)sp * a.split_stride + c];
                    if (c + 1 < a.V) gv[e][j].y += gp[(size_t)sp * a.split_stride + c + 1];
                }
            }
        }
    }
    // ---- the head's root mean square over all its CTAs, the gate, the store
    float sa = 0.f, sb = 0.f;
#pragma unroll
    for (int j = 0; j < 8; j++) { sa += o[j][0] * o[j][0] + o[j][1] * o[j][1]; sb += o[j][2] * o[j][2] + o[j][3] * o[j][3]; }
    sa += __shfl_xor_sync(0xffffffffu, sa, 1); sa += __shfl_xor_sync(0xffffffffu, sa, 2);
    sb += __shfl_xor_sync(0xffffffffu, sb, 1); sb += __shfl_xor_sync(0xffffffffu, sb, 2);
    if (t == 0) { row_ss[warp * 16 + g] = sa; row_ss[warp * 16 + g + 8] = sb; }
    cluster.sync();
    float ra = 0.f, rbs = 0.f;
    for (unsigned r = 0; r < cluster.num_blocks(); r++) {
        const float* peer = cluster.map_shared_rank(row_ss, r);
        ra += peer[warp * 16 + g]; rbs += peer[warp * 16 + g + 8];
    }
    cluster.sync();                                   // nobody leaves while its sums may still be read
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int row = r0 + warp * 16 + g + e * 8;
        if (row >= len) continue;
        const float r = 1.f / sqrtf((e ? rbs : ra) / (float)a.V + a.eps);
        bf16* op = (bf16*)a.out + (size_t)(s0 + row) * HV + (size_t)h * a.V;
#pragma unroll
        for (int j = 0; j < 8; j++) {
            const int c = blockIdx.x * VT + j * 8 + 2 * t;
            const float y0 = o[j][e * 2] * r * (gv[e][j].x / (1.f + __expf(-gv[e][j].x)));
            const float y1 = o[j][e * 2 + 1] * r * (gv[e][j].y / (1.f + __expf(-gv[e][j].y)));
            if ((a.V & 1) == 0) { if (c < a.V) *(uint32_t*)(op + c) = pack_bf16(y0, y1); }
            else { if (c < a.V) op[c] = __float2bfloat16_rn(y0); if (c + 1 < a.V) op[c + 1] = __float2bfloat16_rn(y1); }
        }
    }
}

// ---------------------------------------------------------------------------
static int check(const RetentionArgs& a) {
    if (a.heads <= 0 || a.D <= 0 || a.V <= 0) return tb_refuse("retention: heads=%d D=%d V=%d", a.heads, a.D, a.V);
    if (a.part == nullptr || a.n_splits < 1) return tb_refuse("retention: needs the product's partial sums");
    if (a.rotary_dim < 0 || a.rotary_dim % 2 || a.rotary_dim > a.D || (a.rotary_dim > 0 && a.inv_freq == nullptr))
        return tb_refuse("retention: rotary_dim=%d must be even, at most D=%d, and come with its table", a.rotary_dim, a.D);
    if (a.heads > 65535 || a.batch > 65535) return tb_refuse("retention: %d heads x %d sequences exceed one launch", a.heads, a.batch);
    return 0;
}

// dtype: of the activations (what v is rounded to).
extern "C" int tb_retention_prep(const RetentionArgs* args, int dtype, cudaStream_t stream) {
    if (args->n_tokens <= 0) return 0;
    if (check(*args)) return -1;
    if (args->rotary_dim > 4096) return tb_refuse("retention: %d rotated channels, takes up to 4096", args->rotary_dim);
    TB_DISPATCH_1(dtype, T, tb_launch(retention_prep_kernel<T>, dim3(args->n_tokens), dim3(256), (size_t)args->rotary_dim * sizeof(float), stream, *args));
    return tb_launch_status();
}

// Whether one launch takes a step of one token per sequence.
extern "C" int tb_retention_step_takes(int D, int V) { return D >= 1 && D <= 1024 && V >= 4 && V <= 512 && V % 4 == 0; }

extern "C" int tb_retention_step(const RetentionArgs* args, int dtype, int sms, cudaStream_t stream) {
    const RetentionArgs& a = *args;
    if (a.batch <= 0) return 0;
    if (check(a)) return -1;
    if (!tb_retention_step_takes(a.D, a.V))
        return tb_refuse("retention: the one-token kernel takes D up to 1024 and V up to 512 in multiples of 4, got %d and %d", a.D, a.V);
    if (a.n_tokens != a.batch) return tb_refuse("retention: %d tokens for %d sequences in a step of one token each", a.n_tokens, a.batch);
    if (((uintptr_t)a.state & 15) || a.state_stride % 4) return tb_refuse("retention: states must be 16-byte aligned");
    // few (head, sequence) pairs: more threads for each, so that a state's rows are all in flight at once
    const long long ctas = (long long)a.heads * a.batch;
    const int threads = ctas <= sms ? 1024 : ctas <= 2LL * sms ? 512 : 256;
    const size_t smem = (size_t)((((5 * a.D + 2) + 3) & ~3) + 2 * a.V + (threads / 32) * a.V) * sizeof(float);
#define RSTEP(NC, LPR) do { \
        if (smem > 48 * 1024) { \
            cudaError_t e = cudaFuncSetAttribute(retention_step_kernel<T, NC, LPR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024); \
            if (e != cudaSuccess) return (int)e; \
        } \
        tb_launch(retention_step_kernel<T, NC, LPR>, dim3(a.heads, a.batch), dim3(threads), smem, stream, a); } while (0)
    TB_DISPATCH_1(dtype, T, if (a.V <= 64) RSTEP(1, 16); else if (a.V <= 128) RSTEP(1, 32); else if (a.V <= 256) RSTEP(2, 32); else RSTEP(4, 32));
#undef RSTEP
    return tb_launch_status();
}

// Whether the chunk form takes these sizes (bfloat16 only), and the padded sizes.
extern "C" int tb_retention_chunks_takes(int dtype, int D, int V) { return dtype == TB_BF16 && D >= 1 && D <= 256 && V >= 1 && V <= 8 * VT; }
extern "C" int tb_retention_padded_d(int D) { return D <= 64 ? 64 : D <= 128 ? 128 : 256; }
extern "C" int tb_retention_padded_v(int V) { return (V + VT - 1) / VT * VT; }

// Tokens per chunk: the longer the fewer states go through memory, the shorter the more CTAs make them; whole row blocks.
extern "C" int tb_retention_chunk_len(int heads, int V, int batch, int max_seq_len, int sms) {
    const long long per = (long long)heads * batch * ((V + VT - 1) / VT);
    for (int c = 512; c > RB; c >>= 1)
        if (max_seq_len >= 2 * c && per * ((max_seq_len + c - 1) / c) >= sms) return c;
    return RB;
}

template <int DP> static int run_chunks(const RetentionArgs& a, cudaStream_t stream) {
    constexpr int KPITCH = DP * 2 + 16, STAGE = KB * (KPITCH + VPITCH);
    constexpr int Q_BYTES = RB * KPITCH, S_BYTES = DP * VPITCH;
    const int nv = a.VP / VT;
    const size_t smem1 = (size_t)2 * STAGE + a.chunk_len * sizeof(float);
    const size_t smem2 = (size_t)(Q_BYTES > STAGE ? Q_BYTES : STAGE) + (2 * S_BYTES > STAGE ? 2 * S_BYTES : STAGE)
        + (a.chunk_len + 1 + RB) * sizeof(float);
    static bool attr_set = false;
    if (!attr_set) {
        cudaError_t e = cudaFuncSetAttribute(retention_sum_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 2 * STAGE + 2048);
        if (e == cudaSuccess)
            e = cudaFuncSetAttribute(retention_out_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                     (Q_BYTES > STAGE ? Q_BYTES : STAGE) + (2 * S_BYTES > STAGE ? 2 * S_BYTES : STAGE) + 4096);
        if (e != cudaSuccess) return (int)e;
        attr_set = true;
    }
    tb_launch(retention_sum_kernel<DP>, dim3(nv, a.heads, a.batch * a.n_chunks), dim3(CT), smem1, stream, a);
    int st = tb_launch_status();
    if (st) return st;
    tb_launch(retention_fold_kernel, dim3((DP * a.VP / 2 + 255) / 256, a.heads, a.batch), dim3(256), 0, stream, a);
    st = tb_launch_status();
    if (st) return st;
    launch_cluster(retention_out_kernel<DP>, dim3(nv, a.heads, a.batch * a.row_blocks), dim3(CT), smem2, nv, stream, a);
    return tb_launch_status();
}

extern "C" int tb_retention_chunks(const RetentionArgs* args, cudaStream_t stream) {
    const RetentionArgs& a = *args;
    if (a.n_tokens <= 0 || a.batch <= 0) return 0;
    if (check(a)) return -1;
    if (!tb_retention_chunks_takes(TB_BF16, a.D, a.V) || a.DP != tb_retention_padded_d(a.D) || a.VP != tb_retention_padded_v(a.V))
        return tb_refuse("retention: the chunk form takes D up to 256 and V up to 512 (got %d and %d, padded to %d and %d)", a.D, a.V, a.DP, a.VP);
    if (a.chunk_len < RB || a.chunk_len > 512 || a.chunk_len % RB || a.n_chunks < 1 || a.row_blocks < 1
        || (long long)a.n_chunks * a.chunk_len < (long long)a.row_blocks * RB)
        return tb_refuse("retention: %d chunks of %d tokens for %d row blocks", a.n_chunks, a.chunk_len, a.row_blocks);
    if ((long long)a.batch * a.n_chunks > 65535 || (long long)a.batch * a.row_blocks > 65535)
        return tb_refuse("retention: %d sequences of %d chunks exceed one launch", a.batch, a.n_chunks);
    if (a.rows == nullptr || a.chunk_sum == nullptr || a.chunk_hi == nullptr || a.chunk_lo == nullptr || a.qk == nullptr)
        return tb_refuse("retention: the chunk form needs its scratch");
    const int half = a.rotary_dim / 2;
    const bool vec = a.D % 4 == 0 && a.V % 4 == 0 && half % 4 == 0 && (uintptr_t)a.part % 16 == 0 && a.row_stride % 4 == 0 && a.split_stride % 4 == 0;
    if (vec) tb_launch(retention_rows_kernel<true>, dim3(a.n_tokens), dim3(256), 0, stream, a);
    else tb_launch(retention_rows_kernel<false>, dim3(a.n_tokens), dim3(256), 0, stream, a);
    const int st = tb_launch_status();
    if (st) return st;
    switch (a.DP) {
    case 64: return run_chunks<64>(a, stream);
    case 128: return run_chunks<128>(a, stream);
    default: return run_chunks<256>(a, stream);
    }
}
