// Retention: linear attention with a constant decay per head, between its input product and its output product.
//
// Per head, with key channels d and value channels v, for the tokens of a sequence in order:
//     S[d][v] <- decay * S[d][v] + k_t[d] * v_t[v];      o_t[v] = sum_d S[d][v] * q_t[d]
// q and k are turned (rotate-half pairs over the first R channels) at the token's position and k is scaled first; every
// head's o_t is then divided by its root mean square over v and multiplied by silu(g_t).
//
//   tb_retention_prep  the product's 32-bit partial sums added up, q and k turned, k scaled, all kept in 32-bit:
//                      rows [q | k | v | g] for the scan of gla.cu (any sizes, both dtypes)
//
// 32-bit: angles, the turned q and k, the state, o, its norm and the gate.  v is a product's output: it is rounded to
// the activations' dtype, as every other mixer's values are.
#include "common.cuh"

TB_EXPORT_ERROR()

struct RetentionArgs {
    const float* part; int n_splits; long long split_stride, row_stride;    // [splits][T] rows of q (H*D), k (H*D), v (H*V), g (H*V)
    int heads, D, V;
    int rotary_dim; const float* inv_freq;            // [rotary_dim / 2]
    float k_scale, eps;
    const float* decay;                               // [H]
    const int* positions; const int* token_seq; const int* seq_start; const int* slot_ids;
    float* state; long long state_stride;             // [slots][H*D*V]
    float* rows;                                      // [T][2 H*D + 2 H*V] (tb_retention_prep)
    void* out;                                        // [T][H*V]
    int batch, n_tokens;
};

// The argument block's size, for the Python mirror's check.
extern "C" int tb_retention_args_bytes() { return (int)sizeof(RetentionArgs); }

// A value as the activations' dtype keeps it.
template <typename T> __device__ __forceinline__ float kept(float v) { return to_f<T>(from_f<T>(v)); }

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
    float* dst = a.rows + (size_t)t * (2 * HD + 2 * HV);
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

static int check(const RetentionArgs& a) {
    if (a.heads <= 0 || a.D <= 0 || a.V <= 0) return tb_refuse("retention: heads=%d D=%d V=%d", a.heads, a.D, a.V);
    if (a.part == nullptr || a.n_splits < 1) return tb_refuse("retention: needs the product's partial sums");
    if (a.rotary_dim < 0 || a.rotary_dim % 2 || a.rotary_dim > a.D || (a.rotary_dim > 0 && a.inv_freq == nullptr))
        return tb_refuse("retention: rotary_dim=%d must be even, at most D=%d, and come with its table", a.rotary_dim, a.D);
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
