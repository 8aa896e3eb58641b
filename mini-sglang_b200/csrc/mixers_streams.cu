// Kernels of models that keep several copies of the residual stream and of attention whose heads are the difference of two
// softmax maps (sm_100a; plain C entry points, loaded by ops.py as the library "mixers_streams", built only for models with
// such parts):
//
//   stream_mix_norm_kernel   x_t <- sum_s mix[s][t] x_s + out[t] y for all copies at once, then u = sum_t in[t] x_t, normed:
//                            the end of one sublayer and the beginning of the next in one pass; a form with the row in
//                            registers for 1 to 4 copies (few rows: a row over a cluster of blocks), one for any number
//   map_difference_kernel    o = a_1 - lambda a_2 of a head's two maps, o / sqrt(mean(o^2) + eps) * scale
//
// All arithmetic is float32; the copies are float32, what a sublayer hands over (y) and takes (the normed u) is in the
// activation type.
#include "common.cuh"
#include <cooperative_groups.h>
#include <math.h>

namespace {
__device__ __forceinline__ void ms_load4(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void ms_load4(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
    v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
}
__device__ __forceinline__ void ms_store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void ms_store4(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}
}  // namespace

// ---------------------------------------------------------------------------------------
// One block per output row r; src = rows ? rows[r] : r.
//   x_s = x_in[src * row_stride + s * copy_stride]          (copy_stride 0: all copies are the same row)
//   with y:  x_t <- sum_s mix[s * S + t] x_s + out[t] y[src]   (else x_t = x_s);   x_out[src][t] = x_t  where x_out is given
//   u = sum_t w_in[t] x_t  (w_in null: ones)
//   o[r] = (u - mean(u)) / sqrt(mean((u - mean(u))^2) + eps) * w + b      center
//   o[r] = u / sqrt(mean(u^2) + eps) * w + b                              else;   b null: none
// x_out may be x_in (a thread reads its columns of all copies before it writes them).
// ---------------------------------------------------------------------------------------
struct StreamMixParams {
    const float* x_in; long long row_stride, copy_stride;
    float* x_out;
    const void* y;
    const float* mix; const float* w_out; const float* w_in;
    const float* w; const float* b; float eps; int center;
    const int* rows; void* o;
    int S, H;
};

// CL > 1: a row lies over a cluster of CL blocks, a quarter each (few rows would keep few SMs busy); the blocks' sums meet through
// distributed shared memory.
template <typename A, typename O, int S, int NV, int CL = 1>
__global__ void __launch_bounds__(512) stream_mix_norm_vec_kernel(const StreamMixParams p) {
    __shared__ float red[32];
    pdl_launch_dependents();
    const int r = blockIdx.x / CL, H = p.H / CL, W = p.H;              // H: the columns of this block, from c0
    const int c0 = CL > 1 ? (int)(blockIdx.x % CL) * H : 0;
    // the layer's numbers (and the row index) are nobody's output: fetched while the kernel before this one finishes
    const size_t src = p.rows ? (size_t)p.rows[r] : (size_t)r;
    const float* xi = p.x_in + src * p.row_stride + c0;
    // the sum over the row of what each thread holds of it
    __shared__ float part[2];
    auto row_sum = [&](float v, int which) -> float {
        float t = block_sum(v, red);
        if constexpr (CL > 1) {
            auto cluster = cooperative_groups::this_cluster();
            if (threadIdx.x == 0) part[which] = t;
            cluster.sync();
            t = 0.f;
#pragma unroll
            for (int i = 0; i < CL; ++i) t += cluster.map_shared_rank(part, i)[which];
        }
        return t;
    };
    float mix[S][S], w_out[S], w_in[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        w_in[s] = p.w_in ? p.w_in[s] : 1.f;
        w_out[s] = p.y ? p.w_out[s] : 0.f;
#pragma unroll
        for (int t = 0; t < S; ++t) mix[s][t] = p.y ? p.mix[s * S + t] : 0.f;
    }
    pdl_wait();
    pdl_after_wait();
    pdl_small();
    float u[NV][4];
    float sm = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        u[k][0] = u[k][1] = u[k][2] = u[k][3] = 0.f;
        if (i < H) {
            float x[S][4];
            ms_load4(xi + i, x[0]);
#pragma unroll
            for (int s = 1; s < S; ++s) {
                if (p.copy_stride) ms_load4(xi + s * p.copy_stride + i, x[s]);
                else { x[s][0] = x[0][0]; x[s][1] = x[0][1]; x[s][2] = x[0][2]; x[s][3] = x[0][3]; }
            }
            if (p.y) {
                float yv[4];
                ms_load4(reinterpret_cast<const A*>(p.y) + src * W + c0 + i, yv);
                float n[S][4];
#pragma unroll
                for (int t = 0; t < S; ++t)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        float acc = w_out[t] * yv[e];
#pragma unroll
                        for (int s = 0; s < S; ++s) acc = fmaf(mix[s][t], x[s][e], acc);
                        n[t][e] = acc;
                    }
#pragma unroll
                for (int t = 0; t < S; ++t) {
                    if (p.x_out) ms_store4(p.x_out + (src * S + t) * W + c0 + i, n[t]);
#pragma unroll
                    for (int e = 0; e < 4; ++e) x[t][e] = n[t][e];
                }
            }
#pragma unroll
            for (int t = 0; t < S; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e) u[k][e] = fmaf(w_in[t], x[t][e], u[k][e]);
#pragma unroll
            for (int e = 0; e < 4; ++e) sm += p.center ? u[k][e] : u[k][e] * u[k][e];
        }
    }
    float total = row_sum(sm, 0);
    if (p.center) {
        const float mean = total / (float)W;
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int i = (threadIdx.x + k * blockDim.x) * 4;
            if (i < H) {
#pragma unroll
                for (int e = 0; e < 4; ++e) { u[k][e] -= mean; ss = fmaf(u[k][e], u[k][e], ss); }
            }
        }
        total = row_sum(ss, 1);
    }
    const float inv = 1.f / sqrtf(total / (float)W + p.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i < H) {
            float wv[4], bv[4] = {0.f, 0.f, 0.f, 0.f}, ov[4];
            ms_load4(p.w + c0 + i, wv);
            if (p.b) ms_load4(p.b + c0 + i, bv);
#pragma unroll
            for (int e = 0; e < 4; ++e) ov[e] = fmaf(u[k][e] * inv, wv[e], bv[e]);
            ms_store4(reinterpret_cast<O*>(p.o) + (size_t)r * W + c0 + i, ov);
        }
    }
    if constexpr (CL > 1) cooperative_groups::this_cluster().sync();        // the others may still read this block's sums
}

#define MS_MAX_STREAMS 32

// any number of copies up to MS_MAX_STREAMS, any width: a thread takes one column at a time; u lies in shared memory
template <typename A, typename O>
__global__ void __launch_bounds__(256) stream_mix_norm_kernel(const StreamMixParams p) {
    extern __shared__ float us[];
    __shared__ float red[32];
    const int r = blockIdx.x, H = p.H, S = p.S;
    const size_t src = p.rows ? (size_t)p.rows[r] : (size_t)r;
    const float* xi = p.x_in + src * p.row_stride;
    float sm = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float x[MS_MAX_STREAMS];
        float u = 0.f;
        for (int s = 0; s < S; ++s) x[s] = xi[s * p.copy_stride + i];
        if (p.y) {
            const float yv = to_f32<A>(reinterpret_cast<const A*>(p.y)[src * H + i]);
            for (int t = 0; t < S; ++t) {
                float acc = p.w_out[t] * yv;
                for (int s = 0; s < S; ++s) acc = fmaf(p.mix[s * S + t], x[s], acc);
                if (p.x_out) p.x_out[(src * S + t) * H + i] = acc;
                u = fmaf(p.w_in ? p.w_in[t] : 1.f, acc, u);
            }
        } else {
            for (int t = 0; t < S; ++t) u = fmaf(p.w_in ? p.w_in[t] : 1.f, x[t], u);
        }
        us[i] = u;
        sm += p.center ? u : u * u;
    }
    float total = block_sum(sm, red), mean = 0.f;
    if (p.center) {
        mean = total / (float)H;
        float ss = 0.f;
        for (int i = threadIdx.x; i < H; i += blockDim.x) { const float c = us[i] - mean; ss = fmaf(c, c, ss); }
        total = block_sum(ss, red);
    }
    const float inv = 1.f / sqrtf(total / (float)H + p.eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x)
        reinterpret_cast<O*>(p.o)[(size_t)r * H + i] = from_f32<O>(fmaf((us[i] - mean) * inv, p.w[i], p.b ? p.b[i] : 0.f));
}

template <typename A, typename O>
static int stream_mix_norm_launch(const StreamMixParams& p, int n_rows, cudaStream_t stream) {
    const int H = p.H, S = p.S;
    const uintptr_t all = (uintptr_t)p.x_in | (uintptr_t)p.x_out | (uintptr_t)p.y | (uintptr_t)p.w | (uintptr_t)p.b | (uintptr_t)p.o;
    if (S <= 4 && H % 8 == 0 && (all & 15) == 0 && p.row_stride % 4 == 0 && p.copy_stride % 4 == 0 && H <= 4 * 4 * 512) {
        constexpr int CL = 4;
        if (n_rows <= 32 && H % (4 * CL) == 0 && H >= 1024 && H / (4 * CL) <= 512) {
            const int threads = (H / (4 * CL) + 31) / 32 * 32;
            cudaLaunchConfig_t cfg = {};
            cfg.gridDim = dim3(n_rows * CL);
            cfg.blockDim = dim3(threads);
            cfg.stream = stream;
            cudaLaunchAttribute attr[2];
            attr[0].id = cudaLaunchAttributeClusterDimension;
            attr[0].val.clusterDim.x = CL; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
            attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
            attr[1].val.programmaticStreamSerializationAllowed = 1;
            cfg.attrs = attr;
            cfg.numAttrs = msgl_pdl_enabled() ? 2 : 1;
            if (S == 1) cudaLaunchKernelEx(&cfg, stream_mix_norm_vec_kernel<A, O, 1, 1, CL>, p);
            else if (S == 2) cudaLaunchKernelEx(&cfg, stream_mix_norm_vec_kernel<A, O, 2, 1, CL>, p);
            else if (S == 3) cudaLaunchKernelEx(&cfg, stream_mix_norm_vec_kernel<A, O, 3, 1, CL>, p);
            else cudaLaunchKernelEx(&cfg, stream_mix_norm_vec_kernel<A, O, 4, 1, CL>, p);
            return msgl_check_launch();
        }
        const int n4 = H / 4;
        int nv = 1;
        while ((n4 + nv - 1) / nv > 512) nv *= 2;
        const int threads = (((n4 + nv - 1) / nv) + 31) / 32 * 32;
#define SMN(S_, NV_) msgl_launch_pdl(stream_mix_norm_vec_kernel<A, O, S_, NV_>, dim3(n_rows), dim3(threads), 0, stream, p)
#define SMN_S(S_) do { if (nv == 1) SMN(S_, 1); else if (nv == 2) SMN(S_, 2); else SMN(S_, 4); } while (0)
        if (S == 1) SMN_S(1); else if (S == 2) SMN_S(2); else if (S == 3) SMN_S(3); else SMN_S(4);
#undef SMN_S
#undef SMN
        return msgl_check_launch();
    }
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return MSGL_ERR_SIZE;
    if (smem > 47 * 1024) {          // with the reduction's own array beyond what a launch gets unasked
        static MsglOncePerDevice once;
        if (once.due()) {
            cudaFuncSetAttribute(stream_mix_norm_kernel<A, O>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
            once.mark();
        }
    }
    stream_mix_norm_kernel<A, O><<<n_rows, H >= 512 ? 256 : 128, smem, stream>>>(p);
    return msgl_check_launch();
}

MSGL_API int msgl_stream_mix_norm(const float* x_in, long long row_stride, long long copy_stride, float* x_out, const void* y, int y_is_f32,
                                  const float* mix, const float* w_out, const float* w_in, const float* w, const float* b, float eps,
                                  int center, const int* rows, void* o, int n_rows, int S, int H, int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return MSGL_OK;
    if (S < 1 || S > MS_MAX_STREAMS || H < 1 || x_in == nullptr || w == nullptr || o == nullptr || (y != nullptr && (mix == nullptr || w_out == nullptr)) ||
        (x_out != nullptr && (y == nullptr || rows != nullptr)))
        return MSGL_ERR_SIZE;
    StreamMixParams p;
    p.x_in = x_in; p.row_stride = row_stride; p.copy_stride = copy_stride; p.x_out = x_out; p.y = y; p.mix = mix; p.w_out = w_out; p.w_in = w_in;
    p.w = w; p.b = b; p.eps = eps; p.center = center; p.rows = rows; p.o = o; p.S = S; p.H = H;
    if (dtype == MSGL_F32) return stream_mix_norm_launch<float, float>(p, n_rows, stream);
    if (dtype == MSGL_BF16) return y_is_f32 ? stream_mix_norm_launch<float, __nv_bfloat16>(p, n_rows, stream)
                                            : stream_mix_norm_launch<__nv_bfloat16, __nv_bfloat16>(p, n_rows, stream);
    return MSGL_ERR_DTYPE;
}

// ---------------------------------------------------------------------------------------
// a [T][heads][2][dv] -> o [T][heads * dv]:  v = a[.., 0, :] - lam * a[.., 1, :];  o = v / sqrt(mean(v^2) + eps) * scale
// One warp per (token, head), a lane V neighbouring elements a turn, the difference in registers (dv up to 32 * V * MD_TURNS).
// ---------------------------------------------------------------------------------------
#define MD_TURNS 16
template <typename A, typename O, int V>
__global__ void __launch_bounds__(128) map_difference_kernel(const A* __restrict__ a, O* __restrict__ o, float lam, float eps, float scale,
                                                             long long n_jobs, int heads, int dv, long long o_stride) {
    const long long job = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (job >= n_jobs) return;
    const A* a1 = a + job * 2 * dv;
    const A* a2 = a1 + dv;
    float v[MD_TURNS][V];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < MD_TURNS; ++k) {
        const int i = (lane + 32 * k) * V;
        if (i < dv) {
            float x[V], y[V];
            if constexpr (V == 4) { ms_load4(a1 + i, x); ms_load4(a2 + i, y); }
            else { x[0] = to_f32<A>(a1[i]); y[0] = to_f32<A>(a2[i]); }
#pragma unroll
            for (int e = 0; e < V; ++e) { v[k][e] = fmaf(-lam, y[e], x[e]); ss = fmaf(v[k][e], v[k][e], ss); }
        }
    }
    const float f = scale / sqrtf(warp_sum(ss) / (float)dv + eps);
    const long long t = job / heads;
    O* dst = o + t * o_stride + (job - t * heads) * dv;
#pragma unroll
    for (int k = 0; k < MD_TURNS; ++k) {
        const int i = (lane + 32 * k) * V;
        if (i < dv) {
#pragma unroll
            for (int e = 0; e < V; ++e) v[k][e] *= f;
            if constexpr (V == 4) ms_store4(dst + i, v[k]);
            else dst[i] = from_f32<O>(v[k][0]);
        }
    }
}

MSGL_API int msgl_map_difference(const void* a, int a_is_f32, void* o, long long o_stride, float lam, float eps, float scale, int T_,
                                 int heads, int dv, int dtype, cudaStream_t stream) {
    if (T_ <= 0) return MSGL_OK;
    if (heads < 1 || dv < 1) return MSGL_ERR_SIZE;
    const long long n = (long long)T_ * heads;
    const unsigned blocks = (unsigned)((n + 3) / 4);
    const bool vec = dv % 4 == 0 && o_stride % 4 == 0 && (((uintptr_t)a | (uintptr_t)o) & 15) == 0;
    if (dv > 32 * MD_TURNS * (vec ? 4 : 1)) return MSGL_ERR_SIZE;
#define MD(A, O)                                                                                                             \
    do {                                                                                                                     \
        if (vec) map_difference_kernel<A, O, 4><<<blocks, 128, 0, stream>>>((const A*)a, (O*)o, lam, eps, scale, n, heads, dv, o_stride); \
        else map_difference_kernel<A, O, 1><<<blocks, 128, 0, stream>>>((const A*)a, (O*)o, lam, eps, scale, n, heads, dv, o_stride);     \
    } while (0)
    if (dtype == MSGL_F32) MD(float, float);
    else if (dtype == MSGL_BF16) { if (a_is_f32) MD(float, __nv_bfloat16); else MD(__nv_bfloat16, __nv_bfloat16); }
    else return MSGL_ERR_DTYPE;
#undef MD
    return msgl_check_launch();
}
