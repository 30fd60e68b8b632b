// Gated activation of the feed-forward: out = act(gate) * up, act = SiLU,
// computed in float32 (reference backend/model.cu:477-483:
// g / (1 + expf(-g)) * u).  gate and up may be the two halves of one fused
// projection output: each has its own row stride.  They may be float32 beside a
// bfloat16 out, so that the activation sees the projection's unrounded result.
#include "common.cuh"

KLLM_EXPORT_LAST_ERROR(activation)

namespace {

// out = a * sigmoid(gate) * factor: a gate on a mixer's output, the logits float32 (they come unrounded from
// their product), out in the model's element type, a in it or float32.
template <typename T, typename I>
__global__ void sigmoid_gate_kernel(T* __restrict__ out, int64_t out_stride, const I* __restrict__ a, int64_t a_stride,
                                    const float* __restrict__ gate, int64_t gate_stride, int n, int f, float factor) {
    griddep_wait();
    griddep_launch();
    const int64_t total = (int64_t)n * f;
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = idx / f;
        const int c = (int)(idx - r * f);
        const float g = gate[r * gate_stride + c];
        out[r * out_stride + c] = from_f32<T>(to_f32(a[r * a_stride + c]) * factor / (1.f + expf(-g)));
    }
}

template <typename T, typename I>
__global__ void silu_mul_kernel(T* __restrict__ out, int64_t out_stride,
                                const I* __restrict__ gate, int64_t gate_stride,
                                const I* __restrict__ up, int64_t up_stride, int n, int f) {
    griddep_wait();
    griddep_launch();
    const int64_t total = (int64_t)n * f;
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = idx / f;
        const int c = (int)(idx - r * f);
        const float g = to_f32(gate[r * gate_stride + c]);
        const float u = to_f32(up[r * up_stride + c]);
        out[r * out_stride + c] = from_f32<T>((g / (1.f + expf(-g))) * u);
    }
}

// Same arithmetic on 4 consecutive elements per thread: float32 gate/up rows read as
// float4, the bfloat16 result stored as 8 bytes.  Needs f % 4 == 0 and 16-byte
// aligned float32 rows (8-byte aligned bfloat16 rows).
__global__ void silu_mul_vec4_kernel(bf16* __restrict__ out, int64_t out_stride,
                                     const float* __restrict__ gate, int64_t gate_stride,
                                     const float* __restrict__ up, int64_t up_stride, int n, int f4) {
    griddep_wait();
    griddep_launch();
    const int64_t total = (int64_t)n * f4;
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = idx / f4;
        const int c = (int)(idx - r * f4) * 4;
        const float4 g = *reinterpret_cast<const float4*>(gate + r * gate_stride + c);
        const float4 u = *reinterpret_cast<const float4*>(up + r * up_stride + c);
        __nv_bfloat162 lo = __floats2bfloat162_rn((g.x / (1.f + expf(-g.x))) * u.x, (g.y / (1.f + expf(-g.y))) * u.y);
        __nv_bfloat162 hi = __floats2bfloat162_rn((g.z / (1.f + expf(-g.z))) * u.z, (g.w / (1.f + expf(-g.w))) * u.w);
        uint2 pk;
        pk.x = *reinterpret_cast<uint32_t*>(&lo);
        pk.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(out + r * out_stride + c) = pk;
    }
}

// out = act(gate, up) in the clamped form: g = min(gate, L), u = clamp(up, -L, L),
// g * sigmoid(a g) * (u + 1); float32 gate and up rows at their strides.
template <typename T>
__global__ void clamped_glu_kernel(T* __restrict__ out, int64_t out_stride, const float* __restrict__ gate,
                                   int64_t gate_stride, const float* __restrict__ up, int64_t up_stride, int n, int f,
                                   float limit, float alpha) {
    griddep_wait();
    griddep_launch();
    const int64_t total = (int64_t)n * f;
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = idx / f;
        const int c = (int)(idx - r * f);
        const float g = fminf(gate[r * gate_stride + c], limit);
        const float u = fminf(fmaxf(up[r * up_stride + c], -limit), limit);
        out[r * out_stride + c] = from_f32<T>(g / (1.f + expf(-alpha * g)) * (u + 1.f));
    }
}

// out = act(gate + bg) * (up + bu), act SiLU or the gelu with tanh; float32 gate and up rows at their strides, float32
// biases or null.  V consecutive elements per thread (4: f and the strides in multiples of 4, 16-byte aligned rows).
__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
}

template <typename T, int V>
__global__ void biased_glu_kernel(T* __restrict__ out, int64_t out_stride, const float* __restrict__ gate, int64_t gate_stride,
                                  const float* __restrict__ up, int64_t up_stride, const float* __restrict__ bg,
                                  const float* __restrict__ bu, int n, int fv, int gelu) {
    griddep_wait();
    griddep_launch();
    const int64_t total = (int64_t)n * fv;
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = idx / fv;
        const int c = (int)(idx - r * fv) * V;
        float g[V], u[V];
        if constexpr (V == 4) {
            const float4 g4 = *reinterpret_cast<const float4*>(gate + r * gate_stride + c);
            const float4 u4 = *reinterpret_cast<const float4*>(up + r * up_stride + c);
            g[0] = g4.x; g[1] = g4.y; g[2] = g4.z; g[3] = g4.w;
            u[0] = u4.x; u[1] = u4.y; u[2] = u4.z; u[3] = u4.w;
        } else {
            g[0] = gate[r * gate_stride + c];
            u[0] = up[r * up_stride + c];
        }
        T v[V];
#pragma unroll
        for (int j = 0; j < V; j++) {
            const float z = g[j] + (bg ? bg[c + j] : 0.f), w = u[j] + (bu ? bu[c + j] : 0.f);
            v[j] = from_f32<T>((gelu ? gelu_tanh_f(z) : z / (1.f + expf(-z))) * w);
        }
        T* o = out + r * out_stride + c;
        if constexpr (V == 4 && sizeof(T) == 2)
            *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(v);
        else
#pragma unroll
            for (int j = 0; j < V; j++) o[j] = v[j];
    }
}

// acc[t, :] += row, every row of a float32 matrix with dense rows
__global__ void add_row_kernel(float* __restrict__ acc, const float* __restrict__ row, int64_t total, int d) {
    griddep_wait();
    griddep_launch();
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x)
        acc[i] += row[i % d];
}

// out = f(in) elementwise on float32 input rows: op 0 the square of relu, op 1 tanh, op 2 the value itself
// (a change of element type), op 3 the gelu with the error function, op 4 the gelu with tanh
// (0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3)))), op 5 arg * tanh(z / arg) (a soft cap at +-arg).
template <typename T>
__global__ void unary_kernel(T* __restrict__ out, int64_t out_stride, const float* __restrict__ in, int64_t in_stride,
                             int n, int f, int op, float arg) {
    griddep_wait();
    griddep_launch();
    const int64_t total = (int64_t)n * f;
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = idx / f;
        const int c = (int)(idx - r * f);
        const float z = in[r * in_stride + c];
        float v;
        if (op == 0) {
            const float p = fmaxf(z, 0.f);
            v = p * p;
        } else if (op == 1) {
            v = tanhf(z);
        } else if (op == 2) {
            v = z;
        } else if (op == 3) {
            v = 0.5f * z * (1.f + erff(z * 0.70710678118654752f));
        } else if (op == 4) {
            v = 0.5f * z * (1.f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
        } else {
            v = arg * tanhf(z / arg);
        }
        out[r * out_stride + c] = from_f32<T>(v);
    }
}

}  // namespace

// out [n][f] in the element type `dtype`, in float32 [n][f], dense rows at their strides.
extern "C" int kllm_unary(void* out, int64_t out_stride, const void* in, int64_t in_stride, int n, int f, int op,
                          float arg, int dtype, void* stream) {
    if (n <= 0 || f <= 0) return 0;
    if (op < 0 || op > 5) KLLM_FAIL("unary: unknown function %d", op);
    if (op == 5 && !(arg > 0.f)) KLLM_FAIL("unary: a soft cap must be positive");
    cudaStream_t s = (cudaStream_t)stream;
    int64_t blocks = ((int64_t)n * f + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == KLLM_F32)
        kllm_launch((unary_kernel<float>), dim3((unsigned)blocks), dim3(256), 0, s, (float*)out, out_stride,
                    (const float*)in, in_stride, n, f, op, arg);
    else if (dtype == KLLM_BF16)
        kllm_launch((unary_kernel<bf16>), dim3((unsigned)blocks), dim3(256), 0, s, (bf16*)out, out_stride,
                    (const float*)in, in_stride, n, f, op, arg);
    else
        KLLM_FAIL("unary: unknown element type %d", dtype);
    KLLM_LAUNCH_STATUS();
}

// out [n][f] in the element type `dtype` = act(gate + bg) * (up + bu); gate, up float32 [n][f] with dense rows at their
// strides; bg, bu float32 [f] or null; gelu 0: SiLU, 1: the gelu with tanh.
extern "C" int kllm_biased_glu(void* out, int64_t out_stride, const float* gate, int64_t gate_stride, const float* up,
                               int64_t up_stride, const float* bg, const float* bu, int n, int f, int gelu, int dtype,
                               void* stream) {
    if (n <= 0 || f <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = f % 4 == 0 && gate_stride % 4 == 0 && up_stride % 4 == 0 && out_stride % 4 == 0 &&
                     !(((uintptr_t)gate | (uintptr_t)up) & 15) && !((uintptr_t)out & 7);
    const int fv = vec ? f / 4 : f;
    int64_t blocks = ((int64_t)n * fv + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
#define KLLM_BGLU(T, V)                                                                                                       \
    kllm_launch((biased_glu_kernel<T, V>), dim3((unsigned)blocks), dim3(256), 0, s, (T*)out, out_stride, gate, gate_stride, up, \
                up_stride, bg, bu, n, fv, gelu)
    if (dtype == KLLM_F32) { if (vec) KLLM_BGLU(float, 4); else KLLM_BGLU(float, 1); }
    else if (dtype == KLLM_BF16) { if (vec) KLLM_BGLU(bf16, 4); else KLLM_BGLU(bf16, 1); }
    else KLLM_FAIL("biased glu: unknown element type %d", dtype);
#undef KLLM_BGLU
    KLLM_LAUNCH_STATUS();
}

// acc float32 [n][d] contiguous += row float32 [d] in every row.
extern "C" int kllm_add_row(float* acc, const float* row, int n, int d, void* stream) {
    if (n <= 0 || d <= 0) return 0;
    const int64_t total = (int64_t)n * d;
    int64_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    kllm_launch((add_row_kernel), dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, acc, row, total, d);
    KLLM_LAUNCH_STATUS();
}

// out [n][f] in the element type `dtype`; gate, up float32 [n][f]; dense rows at their strides.
extern "C" int kllm_clamped_glu(void* out, int64_t out_stride, const float* gate, int64_t gate_stride, const float* up,
                                int64_t up_stride, int n, int f, float limit, float alpha, int dtype, void* stream) {
    if (n <= 0 || f <= 0) return 0;
    if (!(limit > 0.f)) KLLM_FAIL("clamped glu: the limit must be positive");
    cudaStream_t s = (cudaStream_t)stream;
    int64_t blocks = ((int64_t)n * f + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == KLLM_F32)
        kllm_launch((clamped_glu_kernel<float>), dim3((unsigned)blocks), dim3(256), 0, s, (float*)out, out_stride, gate,
                    gate_stride, up, up_stride, n, f, limit, alpha);
    else if (dtype == KLLM_BF16)
        kllm_launch((clamped_glu_kernel<bf16>), dim3((unsigned)blocks), dim3(256), 0, s, (bf16*)out, out_stride, gate,
                    gate_stride, up, up_stride, n, f, limit, alpha);
    else
        KLLM_FAIL("clamped glu: unknown element type %d", dtype);
    KLLM_LAUNCH_STATUS();
}

// dtype: element type of out; in_dtype: element type of gate and up.
extern "C" int kllm_silu_mul(void* out, int64_t out_stride, const void* gate, int64_t gate_stride,
                             const void* up, int64_t up_stride, int n, int f, int dtype, int in_dtype,
                             void* stream) {
    if (n <= 0 || f <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int64_t total = (int64_t)n * f;
    int64_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == KLLM_F32 && in_dtype == KLLM_F32)
        kllm_launch((silu_mul_kernel<float, float>), dim3((unsigned)blocks), dim3(256), 0, s, 
            (float*)out, out_stride, (const float*)gate, gate_stride, (const float*)up, up_stride, n, f);
    else if (dtype == KLLM_BF16 && in_dtype == KLLM_BF16)
        kllm_launch((silu_mul_kernel<bf16, bf16>), dim3((unsigned)blocks), dim3(256), 0, s, 
            (bf16*)out, out_stride, (const bf16*)gate, gate_stride, (const bf16*)up, up_stride, n, f);
    else if (dtype == KLLM_BF16 && in_dtype == KLLM_F32 && f % 4 == 0 && gate_stride % 4 == 0 && up_stride % 4 == 0 &&
             out_stride % 4 == 0 && (((uintptr_t)gate | (uintptr_t)up) & 15) == 0 && ((uintptr_t)out & 7) == 0) {
        const int64_t work = (int64_t)n * (f / 4);
        int64_t b4 = (work + 255) / 256;
        if (b4 > 148 * 16) b4 = 148 * 16;
        kllm_launch((silu_mul_vec4_kernel), dim3((unsigned)b4), dim3(256), 0, s, (bf16*)out, out_stride,
                    (const float*)gate, gate_stride, (const float*)up, up_stride, n, f / 4);
    } else if (dtype == KLLM_BF16 && in_dtype == KLLM_F32)
        kllm_launch((silu_mul_kernel<bf16, float>), dim3((unsigned)blocks), dim3(256), 0, s, 
            (bf16*)out, out_stride, (const float*)gate, gate_stride, (const float*)up, up_stride, n, f);
    else
        KLLM_FAIL("silu_mul: element types %d (out) and %d (in) are not supported together", dtype, in_dtype);
    KLLM_LAUNCH_STATUS();
}

// out [n][f] = a [n][f] * sigmoid(gate [n][f]) * factor; out of element type `dtype`, a of `a_dtype` (the same or
// float32), gate float32; row strides in elements.
extern "C" int kllm_sigmoid_gate(void* out, int64_t out_stride, const void* a, int64_t a_stride, const float* gate,
                                 int64_t gate_stride, int n, int f, float factor, int dtype, int a_dtype, void* stream) {
    if (n <= 0 || f <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    int64_t blocks = ((int64_t)n * f + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == KLLM_F32 && a_dtype == KLLM_F32)
        kllm_launch((sigmoid_gate_kernel<float, float>), dim3((unsigned)blocks), dim3(256), 0, s, (float*)out, out_stride,
                    (const float*)a, a_stride, gate, gate_stride, n, f, factor);
    else if (dtype == KLLM_BF16 && a_dtype == KLLM_BF16)
        kllm_launch((sigmoid_gate_kernel<bf16, bf16>), dim3((unsigned)blocks), dim3(256), 0, s, (bf16*)out, out_stride,
                    (const bf16*)a, a_stride, gate, gate_stride, n, f, factor);
    else if (dtype == KLLM_BF16 && a_dtype == KLLM_F32)
        kllm_launch((sigmoid_gate_kernel<bf16, float>), dim3((unsigned)blocks), dim3(256), 0, s, (bf16*)out, out_stride,
                    (const float*)a, a_stride, gate, gate_stride, n, f, factor);
    else
        KLLM_FAIL("sigmoid gate: element types %d (out) and %d (in) are not supported together", dtype, a_dtype);
    KLLM_LAUNCH_STATUS();
}
