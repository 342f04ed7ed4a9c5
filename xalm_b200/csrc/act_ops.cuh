// act_ops.cuh — activations of the config.json families, as the fused epilogues of the fp32 row products (mix_ops.cuh) and of the grouped
// tensor-core GEMM (prefill.cu) apply them.  fp32, library expf / tanhf / log1pf.
#pragma once
#include <cuda_runtime.h>
#include <math.h>

namespace xalm {
namespace mix {

enum { GLU_CLAMPED = 0, GLU_SILU = 1, GLU_GELU_TANH = 2 };
enum { ACT_NONE = 0, ACT_RELU_SQUARED = 1, ACT_SIGMOID = 2, ACT_SILU = 3, ACT_GELU_TANH = 4, ACT_SIGMOID_POW = 5 };

__device__ __forceinline__ float sigmoidf_(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float glu_clamped(float g, float u, float limit, float alpha) {
	g = fminf(g, limit);
	u = fminf(fmaxf(u, -limit), limit);
	return g * sigmoidf_(alpha * g) * (u + 1.f);
}

__device__ __forceinline__ float gelu_tanhf_(float z) { return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }
__device__ __forceinline__ float log_sigmoidf_(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float act_apply(int act, float v, float p = 1.f) {
	if (act == ACT_RELU_SQUARED) { v = fmaxf(v, 0.f); return v * v; }
	if (act == ACT_SIGMOID) return sigmoidf_(v);
	if (act == ACT_SILU) return v * sigmoidf_(v);
	if (act == ACT_GELU_TANH) return gelu_tanhf_(v);
	if (act == ACT_SIGMOID_POW) return expf(p * log_sigmoidf_(v));
	return v;
}
__device__ __forceinline__ float glu_apply(int act, float g, float u, float limit, float alpha) {
	if (act == GLU_SILU) return g * sigmoidf_(g) * u;
	if (act == GLU_GELU_TANH) return gelu_tanhf_(g) * u;
	return glu_clamped(g, u, limit, alpha);
}

} // namespace mix
} // namespace xalm
