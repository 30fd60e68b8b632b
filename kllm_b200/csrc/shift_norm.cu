// What stands in front of a layer.
//
//   norm_shift    h = x / rms(x) * gain for every row of the float32 residual stream, and beside it the token
//                 shift hs = h + (h_prev - h) * mu, h_prev being the normed row before in the same request, or what
//                 the request's state slot keeps of the step before (zeros at the start of a request); the slot then
//                 takes the request's last normed row.  h and hs are stored in the model's element type; norm, shift
//                 and the slot's row are float32 and unrounded, so a portion's first row sees exactly what it would
//                 have seen beside its predecessor.
//   stream_entry  the input of a product over the stream and a copy of it from the start of the step, side by side:
//                 cat[t] = [x[t] | x0[t]] in the model's type; x[t] becomes a row vector that is the same for every
//                 token, to which the product's result is then added.
#include "common.cuh"

KLLM_EXPORT_LAST_ERROR(shift_norm)

namespace {

template <typename T, int V> __device__ __forceinline__ void store_row(T* p, const float (&v)[V]) {
    if constexpr (V == 1) {
        p[0] = from_f32<T>(v[0]);
    } else if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        uint2 pk;
        pk.x = *reinterpret_cast<uint32_t*>(&lo);
        pk.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = pk;
    }
}

template <int V> __device__ __forceinline__ void load_row(float (&v)[V], const float* p) {
    if constexpr (V == 1) {
        v[0] = p[0];
    } else {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
}

// A CTA takes `per` neighbouring rows and keeps the row before in registers; thread channels (i * blockDim + tid) * V.
template <typename T, int V, int NV>
__global__ void __launch_bounds__(512)
norm_shift_kernel(T* __restrict__ h_out, T* __restrict__ hs_out, const float* __restrict__ x, const float* __restrict__ gain,
                  const float* __restrict__ mu, float eps, float* __restrict__ state, int64_t state_stride,
                  const int* __restrict__ q_start, const int* __restrict__ token_req, const int* __restrict__ state_slots,
                  int n, int d, int per) {
    __shared__ float red[32];
    const int t0 = blockIdx.x * per, t1 = min(n, t0 + per);
    float gn[NV][V], m[NV][V];
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = (i * blockDim.x + threadIdx.x) * V;
        if (c < d) {
            load_row<V>(gn[i], gain + c);
            load_row<V>(m[i], mu + c);
        }
    }
    griddep_wait();
    griddep_launch();
    auto normed = [&](float (&h)[NV][V], int t) {           // the normed row t; one order of sums for every row
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int c = (i * blockDim.x + threadIdx.x) * V;
            if (c < d) {
                load_row<V>(h[i], x + (int64_t)t * d + c);
#pragma unroll
                for (int j = 0; j < V; j++) ss += h[i][j] * h[i][j];
            }
        }
        ss = block_sum(ss, red);
        const float scale = rsqrtf(ss / (float)d + eps);
#pragma unroll
        for (int i = 0; i < NV; i++)
#pragma unroll
            for (int j = 0; j < V; j++) h[i][j] = h[i][j] * scale * gn[i][j];
    };
    float prev[NV][V], cur[NV][V];
    for (int t = t0; t < t1; t++) {
        const int s = token_req[t];
        normed(cur, t);
        if (t == q_start[s]) {
            float* slot = state + (int64_t)state_slots[s] * state_stride;
            const int last = q_start[s + 1] - 1;
            float end[NV][V];
            if (last != t) normed(end, last);
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int c = (i * blockDim.x + threadIdx.x) * V;
                if (c < d) {
                    load_row<V>(prev[i], slot + c);
                    store_row<float, V>(slot + c, last != t ? end[i] : cur[i]);
                }
            }
        } else if (t == t0) {
            normed(prev, t - 1);
        }
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int c = (i * blockDim.x + threadIdx.x) * V;
            if (c < d) {
                float sh[V];
#pragma unroll
                for (int j = 0; j < V; j++) {
                    sh[j] = cur[i][j] + (prev[i][j] - cur[i][j]) * m[i][j];
                    prev[i][j] = cur[i][j];
                }
                store_row<T, V>(h_out + (int64_t)t * d + c, cur[i]);
                store_row<T, V>(hs_out + (int64_t)t * d + c, sh);
            }
        }
    }
}

template <typename T, int V>
int launch_norm_shift(T* h, T* hs, const float* x, const float* gain, const float* mu, float eps, float* state,
                      int64_t state_stride, const int* q_start, const int* token_req, const int* state_slots, int n, int d,
                      cudaStream_t s) {
    const int units = (d + V - 1) / V;
    int threads = units >= 512 ? 512 : (units + 31) / 32 * 32;
    const int nv = (units + threads - 1) / threads;
    const int per = n >= 8 * 148 ? 4 : 1;
    const dim3 grid((n + per - 1) / per);
#define KLLM_NS(NV)                                                                                                            \
    kllm_launch((norm_shift_kernel<T, V, NV>), grid, dim3(threads), 0, s, h, hs, x, gain, mu, eps, state, state_stride, q_start, \
                token_req, state_slots, n, d, per)
    if (nv <= 1) KLLM_NS(1);
    else if (nv <= 2) KLLM_NS(2);
    else if (nv <= 4) KLLM_NS(4);
    else if (nv <= 8) KLLM_NS(8);
    else KLLM_FAIL("norm shift: width %d is beyond this kernel", d);
#undef KLLM_NS
    KLLM_LAUNCH_STATUS();
}

template <typename T>
__global__ void __launch_bounds__(256)
stream_entry_kernel(T* __restrict__ cat, float* __restrict__ x, const float* __restrict__ row, int64_t total, int d, int copy_x0) {
    griddep_wait();
    griddep_launch();
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t t = i / d;
        const int c = (int)(i - t * d);
        const T v = from_f32<T>(x[i]);
        cat[t * 2 * d + c] = v;
        if (copy_x0) cat[t * 2 * d + d + c] = v;
        x[i] = row[c];
    }
}

}  // namespace

// h, hs [n][d] in the element type `dtype`; x float32 [n][d]; gain, mu float32 [d]; the row in front of request s at
// state[state_slots[s] * state_stride .. + d], float32.
extern "C" int kllm_norm_shift(void* h, void* hs, const float* x, const float* gain, const float* mu, float eps, float* state,
                               int64_t state_stride, const int* q_start, const int* token_req, const int* state_slots, int n,
                               int d, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (d <= 0 || state_stride < d) KLLM_FAIL("norm shift: width %d, state rows of %lld", d, (long long)state_stride);
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = d % 4 == 0 && state_stride % 4 == 0 &&
                     !(((uintptr_t)h | (uintptr_t)hs | (uintptr_t)x | (uintptr_t)gain | (uintptr_t)mu | (uintptr_t)state) & 15);
    if (dtype == KLLM_F32)
        return vec ? launch_norm_shift<float, 4>((float*)h, (float*)hs, x, gain, mu, eps, state, state_stride, q_start, token_req, state_slots, n, d, s)
                   : launch_norm_shift<float, 1>((float*)h, (float*)hs, x, gain, mu, eps, state, state_stride, q_start, token_req, state_slots, n, d, s);
    if (dtype == KLLM_BF16)
        return vec ? launch_norm_shift<bf16, 4>((bf16*)h, (bf16*)hs, x, gain, mu, eps, state, state_stride, q_start, token_req, state_slots, n, d, s)
                   : launch_norm_shift<bf16, 1>((bf16*)h, (bf16*)hs, x, gain, mu, eps, state, state_stride, q_start, token_req, state_slots, n, d, s);
    KLLM_FAIL("norm shift: unknown element type %d", dtype);
}

// cat [n][2 d] in `dtype`: the first half of every row from x (float32 [n][d]), the second half too when copy_x0;
// x then becomes `row` (float32 [d]) in every row.
extern "C" int kllm_stream_entry(void* cat, float* x, const float* row, int n, int d, int copy_x0, int dtype, void* stream) {
    if (n <= 0 || d <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int64_t total = (int64_t)n * d;
    int64_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == KLLM_F32)
        kllm_launch((stream_entry_kernel<float>), dim3((unsigned)blocks), dim3(256), 0, s, (float*)cat, x, row, total, d, copy_x0);
    else if (dtype == KLLM_BF16)
        kllm_launch((stream_entry_kernel<bf16>), dim3((unsigned)blocks), dim3(256), 0, s, (bf16*)cat, x, row, total, d, copy_x0);
    else
        KLLM_FAIL("stream entry: unknown element type %d", dtype);
    KLLM_LAUNCH_STATUS();
}
