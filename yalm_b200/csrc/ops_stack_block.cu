// Row ops of parallel blocks that run as one product in and one product out (stack.cpp: stack_layer_block).  Like the other row
// ops every kernel takes n rows = n consecutive positions of one sequence (n = 1: a decode step), fp32 activations, and positions
// from the argument or the device control block; a call whose first position is 0 starts a sequence: stored state is taken
// as zero.
//
//   layer_norm_rows     h = (x - mean) / sqrt(var + eps) * w + b, to fp32 rows and / or the 16-bit operand of a tensor-core product
//   mix_rows            up to eight blends h + (h' - h) mu_s of a row with the previous position's
//   delta_in_rows       short causal convolutions + SiLU of q, k, v; q, k as unit vectors per head; one decay and one beta per head
//   wkv_decay_rows      exp(-exp(W_2 tanh(t) + w_0))
//   block_out_rows      the input of the block's output product: [per-head norm * gate, or the attention's output | act(g) u]
//   group_norm_rows     x += mult * (sublayer outputs), then an RMS norm over equal parts of the row: one launch between two layers
//   state_step          a decode row of a matrix-state mixer in one launch, one CTA per head: what feeds the recurrence
//                       (convolutions and unit norms, or the decay's second stage), one step of it, the head's norm and the gate
//   gemv_block_in       a decode row's product in: the layer norm (and the blends, by output segment) is applied while the input is staged
//   gemv_block_out      a decode row's product out: the gated activation is applied while the input is staged, x += in the epilogue
//
// State kept in rings indexed by position (short convolutions: `taps` rows, slot = position % taps; the previous h: two rows, slot =
// position & 1): a decode row writes a slot that no other thread of its launch reads.
#include "common.cuh"

#include <cuda_bf16.h>

#include <algorithm>

#include "gemv.cuh"
#include "launch.h"
#include "stack_rows.cuh"

namespace yalm {
namespace stack {

__device__ __forceinline__ float sigmoid_(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float head_decay(float z, float dt_bias, float a_log) { return expf(-expf(a_log) * softplus_(z + dt_bias)); }

__device__ __forceinline__ void put16(void *out, size_t i, float v, int bf16) {
	if (bf16) static_cast<__nv_bfloat16 *>(out)[i] = __float2bfloat16_rn(v);
	else static_cast<__half *>(out)[i] = __float2half_rn(v);
}
__device__ __forceinline__ uint2 pack4_16(float4 v, int bf16) {
	uint2 r;
	if (bf16) {
		const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
		r.x = *reinterpret_cast<const uint32_t *>(&a), r.y = *reinterpret_cast<const uint32_t *>(&b);
	} else {
		const __half2 a = __floats2half2_rn(v.x, v.y), b = __floats2half2_rn(v.z, v.w);
		r.x = *reinterpret_cast<const uint32_t *>(&a), r.y = *reinterpret_cast<const uint32_t *>(&b);
	}
	return r;
}

// ---- layer norm with a bias ------------------------------------------------------------------------------------------------
// One CTA per output row r = row rows[r] of x (rows null: r itself).  add (optional): x[m] += add[m] first, written back.  The row
// is kept in shared memory between the two passes (mean, then the mean of the squared deviations).
__global__ void __launch_bounds__(256) layer_norm_rows_kernel(float *__restrict__ out, void *__restrict__ out16, int bf16, float *x, const float *__restrict__ add,
                                                              const int *__restrict__ rows, const float *__restrict__ w, const float *__restrict__ b, float eps,
                                                              int dim) {
	extern __shared__ __align__(16) float xs[];
	__shared__ float red[33];
	const int r = blockIdx.x, m = rows ? rows[r] : r;
	float *row = x + (size_t)m * dim;
	float s = 0.f;
	const bool vec = dim % 4 == 0;
	if (vec) {
#pragma unroll 4
		for (int e = threadIdx.x * 4; e < dim; e += blockDim.x * 4) {
			float4 v = *reinterpret_cast<const float4 *>(row + e);
			if (add) {
				const float4 a = *reinterpret_cast<const float4 *>(add + (size_t)m * dim + e);
				v.x += a.x, v.y += a.y, v.z += a.z, v.w += a.w;
				*reinterpret_cast<float4 *>(row + e) = v;
			}
			*reinterpret_cast<float4 *>(xs + e) = v;
			s += (v.x + v.y) + (v.z + v.w);
		}
	} else
		for (int e = threadIdx.x; e < dim; e += blockDim.x) {
			float v = row[e];
			if (add) row[e] = v = v + add[(size_t)m * dim + e];
			xs[e] = v, s += v;
		}
	const float mean = block_sum(s, red) / dim;
	float ss = 0.f;
	if (vec)
		for (int e = threadIdx.x * 4; e < dim; e += blockDim.x * 4) {
			const float4 v = *reinterpret_cast<const float4 *>(xs + e);
			const float a = v.x - mean, c = v.y - mean, d = v.z - mean, f = v.w - mean;
			ss += (a * a + c * c) + (d * d + f * f);
		}
	else
		for (int e = threadIdx.x; e < dim; e += blockDim.x) ss += (xs[e] - mean) * (xs[e] - mean);
	const float sc = 1.0f / sqrtf(block_sum(ss, red) / dim + eps);
	if (vec) {
#pragma unroll 4
		for (int e = threadIdx.x * 4; e < dim; e += blockDim.x * 4) {
			const float4 v = *reinterpret_cast<const float4 *>(xs + e), g = *reinterpret_cast<const float4 *>(w + e);
			const float4 c = b ? *reinterpret_cast<const float4 *>(b + e) : make_float4(0.f, 0.f, 0.f, 0.f);
			const float4 o = make_float4((v.x - mean) * sc * g.x + c.x, (v.y - mean) * sc * g.y + c.y, (v.z - mean) * sc * g.z + c.z, (v.w - mean) * sc * g.w + c.w);
			if (out) *reinterpret_cast<float4 *>(out + (size_t)r * dim + e) = o;
			if (out16) *reinterpret_cast<uint2 *>(static_cast<uint16_t *>(out16) + (size_t)r * dim + e) = pack4_16(o, bf16);
		}
	} else
		for (int e = threadIdx.x; e < dim; e += blockDim.x) {
			const float o = (xs[e] - mean) * sc * w[e] + (b ? b[e] : 0.f);
			if (out) out[(size_t)r * dim + e] = o;
			if (out16) put16(out16, (size_t)r * dim + e, o, bf16);
		}
}

// ---- blends with the previous position's row -----------------------------------------------------------------------------------
// Slab s of out (nmix slabs of n x dim; fp32 or 16-bit): h + (h' - h) mu_s, mu (nmix, dim), plain[s] != 0: h itself.  h' of row 0
// is state row (p0 - 1) & 1 (zero at position 0).
struct MixMask {
	int plain; // bit s: slab s is h itself
};
__global__ void __launch_bounds__(256) mix_rows_kernel(float *__restrict__ out, void *__restrict__ out16, int bf16, const float *__restrict__ h,
                                                       const float *__restrict__ mu, int nmix, MixMask mask, const float *__restrict__ state, int n, int dim,
                                                       int pos0, const int *__restrict__ ctl) {
	const int m = blockIdx.y, p = first_pos(ctl, pos0) + m;
	const int e = blockIdx.x * blockDim.x + threadIdx.x;
	if (e >= dim) return;
	const float v = h[(size_t)m * dim + e];
	const float prev = m > 0 ? h[(size_t)(m - 1) * dim + e] : (p > 0 ? state[(size_t)((p - 1) & 1) * dim + e] : 0.f);
	for (int s = 0; s < nmix; ++s) {
		const float o = (mask.plain >> s) & 1 ? v : v + (prev - v) * mu[(size_t)s * dim + e];
		const size_t at = ((size_t)s * n + m) * dim + e;
		if (out) out[at] = o;
		if (out16) put16(out16, at, o, bf16);
	}
}
__global__ void keep_row_kernel(float *__restrict__ state, const float *__restrict__ h, int n, int dim, int pos0, const int *__restrict__ ctl) {
	const int e = blockIdx.x * blockDim.x + threadIdx.x;
	if (e < dim) state[(size_t)((first_pos(ctl, pos0) + n - 1) & 1) * dim + e] = h[(size_t)(n - 1) * dim + e];
}

// ---- short convolutions, unit vectors, decay and beta of the delta rule ----------------------------------------------------------
// Channels [0, G D) are q, [G D, 2 G D) k, the rest v (H P).  Input of position p >= p0: in[p - p0]; of earlier ones: ring slot p % taps.
__device__ __forceinline__ float ring_input(const float *in, int ldi, const float *ring, int C, int taps, int c, int row, int p0) {
	if (row >= 0) return in[(size_t)row * ldi + c];
	const int p = p0 + row;
	return p >= 0 ? ring[(size_t)(p % taps) * C + c] : 0.f;
}
__device__ __forceinline__ float conv_silu(const float *in, int ldi, const float *ring, const float *w, int C, int taps, int c, int row, int p0) {
	float acc = 0.f;
	for (int j = 0; j < taps; ++j) acc = fmaf(w[(size_t)c * taps + j], ring_input(in, ldi, ring, C, taps, c, row - (taps - 1) + j, p0), acc);
	return act_silu(acc);
}
struct DeltaInArgs {
	float *out;          // (n, C): q | k | v
	float *gates;        // (n, 2 H): decay | beta
	const float *in;     // (n, ldi): q | k | v projections
	const float *raw;    // (n, ldi): beta (H) | decay (H) projections
	int ldi;
	const float *conv_w; // (C, taps)
	float *ring;         // (taps, C)
	const float *a_log, *dt_bias;
	int n, H, G, D, P, taps;
	float unit_eps, q_scale;
	int pos0;
	const int *ctl;
};
constexpr int kDeltaMaxD = 256, kDeltaWarps = 8;
__global__ void __launch_bounds__(kDeltaWarps * 32) delta_in_rows_kernel(DeltaInArgs a) {
	const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
	const int p0 = first_pos(a.ctl, a.pos0), dk = a.G * a.D, dv = a.H * a.P, C = 2 * dk + dv;
	const int vchunks = (dv + 127) / 128, units = 2 * a.G + vchunks; // a warp takes a q / k vector or 128 channels of v
	for (int u = blockIdx.y * kDeltaWarps + warp; u < units; u += gridDim.y * kDeltaWarps) {
		if (u < 2 * a.G) {
			const int c0 = u * a.D;
			float v[kDeltaMaxD / 32], ss = 0.f;
#pragma unroll
			for (int i = 0; i < kDeltaMaxD / 32; ++i) {
				const int d = i * 32 + lane;
				v[i] = d < a.D ? conv_silu(a.in, a.ldi, a.ring, a.conv_w, C, a.taps, c0 + d, m, p0) : 0.f;
				ss += v[i] * v[i];
				if (i * 32 + 32 >= a.D) break;
			}
			ss = warp_sum(ss);
			const float r = (u < a.G ? a.q_scale : 1.f) / sqrtf(ss + a.unit_eps);
#pragma unroll
			for (int i = 0; i < kDeltaMaxD / 32; ++i) {
				const int d = i * 32 + lane;
				if (d < a.D) a.out[(size_t)m * C + c0 + d] = v[i] * r;
				if (i * 32 + 32 >= a.D) break;
			}
		} else
#pragma unroll
			for (int i = 0; i < 4; ++i) {
				const int c = 2 * dk + (u - 2 * a.G) * 128 + i * 32 + lane;
				if (c < C) a.out[(size_t)m * C + c] = conv_silu(a.in, a.ldi, a.ring, a.conv_w, C, a.taps, c, m, p0);
			}
	}
	if (blockIdx.y == 0)
		for (int h = threadIdx.x; h < a.H; h += blockDim.x) {
			const float *raw = a.raw + (size_t)m * a.ldi;
			a.gates[(size_t)m * 2 * a.H + h] = head_decay(raw[a.H + h], a.dt_bias[h], a.a_log[h]);
			a.gates[(size_t)m * 2 * a.H + a.H + h] = sigmoid_(raw[h]);
		}
}
// the call's last inputs into the ring (every slot whose position is one of the call's rows)
__global__ void conv_ring_rows_kernel(float *__restrict__ ring, const float *__restrict__ in, int ldi, int n, int C, int taps, int pos0,
                                      const int *__restrict__ ctl) {
	const int c = blockIdx.x * blockDim.x + threadIdx.x;
	if (c >= C) return;
	const int p0 = first_pos(ctl, pos0);
	for (int m = max(0, n - taps); m < n; ++m) ring[(size_t)((p0 + m) % taps) * C + c] = in[(size_t)m * ldi + c];
}

// ---- decay of the time mixing -----------------------------------------------------------------------------------------------
// out[m, c] = exp(-exp(w0[c] + sum_j w2[c, j] tanh(t[m, j]))): 16 rows and 128 channels per CTA, products in fp32.
constexpr int kDecayRows = 16;
template <int DT>
__global__ void __launch_bounds__(128) wkv_decay_rows_kernel(float *__restrict__ out, int ldo, const float *__restrict__ t, int ldt, const void *__restrict__ w2,
                                                             const float *__restrict__ w0, int n, int C, int rank, int vec) {
	extern __shared__ __align__(16) float ts[]; // kDecayRows x rank padded to 8
	const int rp = (rank + 7) & ~7, m0 = blockIdx.y * kDecayRows, rows = min(kDecayRows, n - m0);
	for (int i = threadIdx.x; i < kDecayRows * rp; i += blockDim.x) {
		const int r = i / rp, j = i % rp;
		ts[i] = r < rows && j < rank ? tanhf(t[(size_t)(m0 + r) * ldt + j]) : 0.f;
	}
	__syncthreads();
	const int c = blockIdx.x * blockDim.x + threadIdx.x;
	if (c >= C) return;
	float acc[kDecayRows];
#pragma unroll
	for (int r = 0; r < kDecayRows; ++r) acc[r] = 0.f;
	constexpr int V = Elem<DT>::VEC;
	for (int j = 0; j < rank; j += V) {
		float f[8];
		if (vec) Elem<DT>::unpack(ldg_stream(static_cast<const typename Elem<DT>::T *>(w2) + (size_t)c * rank + j), f);
		else
#pragma unroll
			for (int i = 0; i < V; ++i) f[i] = j + i < rank ? Elem<DT>::get(w2, (size_t)c * rank + j + i) : 0.f;
#pragma unroll
		for (int r = 0; r < kDecayRows; ++r)
#pragma unroll
			for (int i = 0; i < V; i += 4) {
				const float4 tv = *reinterpret_cast<const float4 *>(ts + r * rp + j + i);
				acc[r] = fmaf(f[i], tv.x, acc[r]), acc[r] = fmaf(f[i + 1], tv.y, acc[r]);
				acc[r] = fmaf(f[i + 2], tv.z, acc[r]), acc[r] = fmaf(f[i + 3], tv.w, acc[r]);
			}
	}
	const float b = w0[c];
#pragma unroll
	for (int r = 0; r < kDecayRows; ++r)
		if (r < rows) out[(size_t)(m0 + r) * ldo + c] = expf(-expf(acc[r] + b));
}

// ---- the output product's input ---------------------------------------------------------------------------------------------
// Columns [0, H P): o (norm_w null), or per head o / sqrt(mean o^2 + eps) * norm_w[h * w_stride + c] * silu(gate); columns [H P,
// H P + ff): silu-gated activation of (g | u).  fp32 rows or 16-bit rows.  A warp takes a head or 128 columns of the activation.
struct BlockOutArgs {
	float *out;
	void *out16;
	int bf16, ldo;
	const float *o;
	int ldi;
	const float *gate, *gu; // rows of stride ldp
	int ldp;
	const float *norm_w;
	int w_stride, H, P, ff, act;
	float eps;
};
__global__ void __launch_bounds__(256) block_out_rows_kernel(BlockOutArgs a) {
	const int m = blockIdx.x, lane = threadIdx.x & 31, no = a.H * a.P;
	const int units = a.H + (a.ff + 127) / 128;
	auto put = [&](int c, float v) {
		if (a.out) a.out[(size_t)m * a.ldo + c] = v;
		if (a.out16) put16(a.out16, (size_t)m * a.ldo + c, v, a.bf16);
	};
	for (int u = blockIdx.y * 8 + (threadIdx.x >> 5); u < units; u += gridDim.y * 8) {
		if (u < a.H) {
			const float *row = a.o + (size_t)m * a.ldi + (size_t)u * a.P;
			if (!a.norm_w) {
				for (int c = lane; c < a.P; c += 32) put(u * a.P + c, row[c]);
				continue;
			}
			float ss = 0.f;
			for (int c = lane; c < a.P; c += 32) ss += row[c] * row[c];
			ss = warp_sum(ss);
			const float r = 1.0f / sqrtf(ss / a.P + a.eps);
			for (int c = lane; c < a.P; c += 32)
				put(u * a.P + c, row[c] * r * a.norm_w[u * a.w_stride + c] * act_silu(a.gate[(size_t)m * a.ldp + (size_t)u * a.P + c]));
		} else {
			const float *g = a.gu + (size_t)m * a.ldp;
#pragma unroll
			for (int i = 0; i < 4; ++i) {
				const int f = (u - a.H) * 128 + i * 32 + lane;
				if (f < a.ff) put(no + f, glu_value(g[f], g[a.ff + f], a.act, 1.f, 0.f, 0.f));
			}
		}
	}
}

// ---- a decode row of a matrix-state mixer ---------------------------------------------------------------------------------------
// One CTA per head: (delta rule) convolution + SiLU + unit norms of the head's q and k and of its P channels of v, decay and beta; or
// (time mixing) the decay's second stage for the head's D channels; or (retention) the rotation of q and k, with a fixed decay.  Then one step of the recurrence with the state in the layout
// of state_scan_kernel (8 lanes per column, EPL consecutive rows each), the head's RMS norm, weight and gate.
struct StateStepArgs {
	float *out;                   // (H P)
	float *state;                 // (H, P, D)
	const float *proj;            // the row of the packed projection
	int o_q, o_k, o_v, o_gate;    // DELTA: o_q is the first channel of q | k | v; else r, k, v
	int o_beta, o_decay;          // raw beta / raw decay (DELTA), or the decay's first stage (o_decay)
	int H, G, D, P;
	const float *conv_w;
	float *ring;
	int taps;
	const float *a_log, *dt_bias; // DELTA
	float unit_eps, q_scale;
	const void *w2;               // (H D, rank)
	const float *w0, *bonus;
	int rank, vec;
	const float *norm_w;          // null: no weight
	int w_stride;
	float eps;
	int pos0;
	const int *ctl;
	const float *decay, *freq;    // retention: (H) decays; rotary frequencies (rot_dims / 2), q_scale is k's factor
	float rot_mag;
	int rot_dims, interleaved;
};
constexpr int kStepThreads = 512;
constexpr int kStepDelta = 0, kStepBonus = 1, kStepFixed = 2;
template <int EPL, int MODE, int DT>
__global__ void __launch_bounds__(kStepThreads) state_step_kernel(StateStepArgs a) {
	extern __shared__ __align__(16) float sm[];
	__shared__ float red[33], gates[2];
	const int h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
	// in shared memory a row of D channels is cut into the 8 lanes' segments, padded so that the lanes read different banks
	constexpr int SEG = EPL + (EPL >= 8 ? 4 : 0), DP = 8 * SEG;
	const int D = a.D, P = a.P;
	auto slot = [](int d) { return d / EPL * SEG + d % EPL; };
	float *qs = sm, *ks = qs + DP, *gs = ks + DP, *us = gs + DP, *vs = us + DP, *os = vs + P; // gs, us: decay and bonus per key channel
	const int p = first_pos(a.ctl, a.pos0);
	const bool fresh = p == 0;
	constexpr int COLS = kStepThreads / 8;
	const int sub = tid & 7, col0 = tid >> 3;
	// the first columns' state is on its way while the inputs are prepared
	float s[EPL];
	auto load_state = [&](int c) {
		const float *sp = a.state + ((size_t)h * P + c) * D + sub * EPL;
		if (EPL % 4 == 0 && D == 8 * EPL) {
#pragma unroll
			for (int e = 0; e < EPL; e += 4) {
				const float4 v = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4 *>(sp + e);
				s[e] = v.x;
				if constexpr (EPL >= 4) s[e + 1] = v.y, s[e + 2] = v.z, s[e + 3] = v.w;
			}
		} else
#pragma unroll
			for (int e = 0; e < EPL; ++e) s[e] = (!fresh && sub * EPL + e < D) ? sp[e] : 0.f;
	};
	if (col0 < P) load_state(col0);
	for (int i = tid; i < 4 * DP; i += kStepThreads) sm[i] = 0.f; // rows past D
	__syncthreads();
	float decay = 1.f, beta = 0.f;
	if constexpr (MODE == kStepFixed) {
		decay = a.decay[h];
		const int half = a.rot_dims / 2;
		for (int i = tid; i < D - half; i += kStepThreads) { // a rotated pair, or a channel past the rotated ones
			const int da = i >= half ? i + half : a.interleaved ? 2 * i : i, db = a.interleaved ? 2 * i + 1 : i + half;
			float q0 = a.proj[a.o_q + h * D + da], k0 = a.proj[a.o_k + h * D + da];
			if (i < half) {
				float q1 = a.proj[a.o_q + h * D + db], k1 = a.proj[a.o_k + h * D + db];
				rotate_pair(q0, q1, p, a.freq[i], a.rot_mag, &q0, &q1);
				rotate_pair(k0, k1, p, a.freq[i], a.rot_mag, &k0, &k1);
				qs[slot(db)] = q1, ks[slot(db)] = k1 * a.q_scale;
			}
			qs[slot(da)] = q0, ks[slot(da)] = k0 * a.q_scale;
		}
		for (int c = tid; c < P; c += kStepThreads) vs[c] = a.proj[a.o_v + h * P + c];
		__syncthreads();
	} else if constexpr (MODE == kStepDelta) {
		const int g = h / (a.H / a.G), dk = a.G * D, C = 2 * dk + a.H * P;
		const float *in = a.proj + a.o_q;
		for (int i = tid; i < 2 * D + P; i += kStepThreads) {
			const int c = i < D ? g * D + i : i < 2 * D ? dk + g * D + i - D : 2 * dk + h * P + i - 2 * D;
			const float v = conv_silu(in, 0, a.ring, a.conv_w, C, a.taps, c, 0, p);
			if (i < D) qs[slot(i)] = v;
			else if (i < 2 * D) ks[slot(i - D)] = v;
			else vs[i - 2 * D] = v;
			if (i >= 2 * D || h % (a.H / a.G) == 0) a.ring[(size_t)(p % a.taps) * C + c] = in[c]; // q, k: one of the heads that share them
		}
		if (tid == 0) gates[0] = head_decay(a.proj[a.o_decay + h], a.dt_bias[h], a.a_log[h]), gates[1] = sigmoid_(a.proj[a.o_beta + h]);
		__syncthreads();
		if (warp < 2) {
			float *v = warp ? ks : qs, ss = 0.f;
			for (int d = lane; d < D; d += 32) ss += v[slot(d)] * v[slot(d)];
			ss = warp_sum(ss);
			const float r = (warp ? 1.f : a.q_scale) / sqrtf(ss + a.unit_eps);
			for (int d = lane; d < D; d += 32) v[slot(d)] *= r;
		}
		__syncthreads();
		decay = gates[0], beta = gates[1];
	} else {
		float *ts = os; // rank floats; os is written only after the recurrence
		for (int j = tid; j < a.rank; j += kStepThreads) ts[j] = tanhf(a.proj[a.o_decay + j]);
		for (int d = tid; d < D; d += kStepThreads) {
			qs[slot(d)] = a.proj[a.o_q + h * D + d], ks[slot(d)] = a.proj[a.o_k + h * D + d];
			us[slot(d)] = a.bonus[h * D + d];
		}
		for (int c = tid; c < P; c += kStepThreads) vs[c] = a.proj[a.o_v + h * P + c];
		__syncthreads();
		for (int d0 = 0; d0 < D; d0 += kStepThreads / 4) { // four lanes per channel
			const int d = d0 + (tid >> 2), part = tid & 3;
			float acc = 0.f;
			if (d < D) {
				const size_t row = (size_t)(h * D + d) * a.rank;
				constexpr int V = Elem<DT>::VEC;
				if (a.vec)
					for (int j = part * V; j < a.rank; j += 4 * V) {
						float f[8];
						Elem<DT>::unpack(ldg_stream(static_cast<const typename Elem<DT>::T *>(a.w2) + row + j), f);
#pragma unroll
						for (int i = 0; i < V; ++i) acc = fmaf(f[i], ts[j + i], acc);
					}
				else
					for (int j = part; j < a.rank; j += 4) acc = fmaf(Elem<DT>::get(a.w2, row + j), ts[j], acc);
			}
			acc += __shfl_xor_sync(kFull, acc, 1), acc += __shfl_xor_sync(kFull, acc, 2);
			if (d < D && part == 0) gs[slot(d)] = expf(-expf(acc + a.w0[h * D + d]));
		}
		__syncthreads();
	}
	for (int c0 = 0; c0 < P; c0 += COLS) { // all lanes of a warp stay in step: the column groups shuffle among themselves
		const int c = c0 + col0;
		const bool live = c < P;
		if (c0 > 0 && live) load_state(c);
		const float vv = live ? vs[c] : 0.f;
		float o4[4] = {0.f, 0.f, 0.f, 0.f};
		if constexpr (MODE == kStepFixed) {
#pragma unroll
			for (int e = 0; e < EPL; ++e) {
				s[e] = fmaf(decay, s[e], ks[sub * SEG + e] * vv);
				o4[e & 3] = fmaf(s[e], qs[sub * SEG + e], o4[e & 3]);
			}
		} else if constexpr (MODE == kStepDelta) {
			float d4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
			for (int e = 0; e < EPL; ++e) {
				s[e] *= decay;
				d4[e & 3] = fmaf(s[e], ks[sub * SEG + e], d4[e & 3]);
			}
			float dot = (d4[0] + d4[1]) + (d4[2] + d4[3]);
			dot += __shfl_xor_sync(kFull, dot, 4), dot += __shfl_xor_sync(kFull, dot, 2), dot += __shfl_xor_sync(kFull, dot, 1);
			const float u = beta * (vv - dot);
#pragma unroll
			for (int e = 0; e < EPL; ++e) {
				s[e] = fmaf(ks[sub * SEG + e], u, s[e]);
				o4[e & 3] = fmaf(s[e], qs[sub * SEG + e], o4[e & 3]);
			}
		} else {
#pragma unroll
			for (int e = 0; e < EPL; ++e) {
				const int d = sub * SEG + e;
				const float kv = ks[d] * vv;
				o4[e & 3] = fmaf(fmaf(us[d], kv, s[e]), qs[d], o4[e & 3]);
				s[e] = fmaf(gs[d], s[e], kv);
			}
		}
		float o = (o4[0] + o4[1]) + (o4[2] + o4[3]);
		o += __shfl_xor_sync(kFull, o, 4), o += __shfl_xor_sync(kFull, o, 2), o += __shfl_xor_sync(kFull, o, 1);
		if (live) {
			float *sp = a.state + ((size_t)h * P + c) * D + sub * EPL;
			if (EPL % 4 == 0 && D == 8 * EPL) {
#pragma unroll
				for (int e = 0; e < EPL; e += 4)
					if constexpr (EPL >= 4) *reinterpret_cast<float4 *>(sp + e) = make_float4(s[e], s[e + 1], s[e + 2], s[e + 3]);
			} else
#pragma unroll
				for (int e = 0; e < EPL; ++e)
					if (sub * EPL + e < D) sp[e] = s[e];
			if (sub == 0) os[c] = o;
		}
	}
	__syncthreads();
	float ss = 0.f;
	for (int c = tid; c < P; c += kStepThreads) ss += os[c] * os[c];
	ss = block_sum(ss, red);
	const float r = 1.0f / sqrtf(ss / P + a.eps);
	for (int c = tid; c < P; c += kStepThreads) a.out[h * P + c] = os[c] * r * (a.norm_w ? a.norm_w[h * a.w_stride + c] : 1.f) * act_silu(a.proj[a.o_gate + h * P + c]);
}

// ---- residual add + norm in groups ----------------------------------------------------------------------------------------------
// x += mult * (a + bias + b + sum_j y_j) (whatever is given), then h = x over the root mean square of its group (the row is `groups`
// equal neighbouring parts), times w; to fp32 rows and / or a 16-bit operand (neither: only the add).  One CTA per row; a warp, or
// several for few groups, sums a group's squares.  rows: norm only, of x[rows[r]].
struct GroupNormArgs {
	float *x;
	float mult;
	const float *a, *abias, *b, *y;
	int ldy, nsum;
	float *out;
	void *out16;
	int bf16;
	const int *rows;
	const float *w;
	int groups, dim;
	float eps;
	int vec; // rows are 16-byte aligned multiples of four channels
};
__global__ void __launch_bounds__(1024) group_norm_rows_kernel(GroupNormArgs g) {
	extern __shared__ __align__(16) float gn_sm[]; // dim values, then partial sums of squares
	const int m = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, nw = nt >> 5, dim = g.dim;
	float *vals = gn_sm, *part = gn_sm + dim;
	float *xr = g.x + (size_t)(g.rows ? g.rows[m] : m) * dim;
	const bool add = g.a || g.b || g.y;
	const size_t o = (size_t)m * dim;
	if (g.vec) {
		// every operand of a piece of four channels is on its way before the first is used: one memory round trip
		constexpr int U = 4;
		const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
		auto get = [&](const float *p) { return *reinterpret_cast<const float4 *>(p); };
		auto plus = [](float4 p, float4 q) { return make_float4(p.x + q.x, p.y + q.y, p.z + q.z, p.w + q.w); };
		for (int e = tid * 4; e < dim; e += nt * 4) {
			float4 v = get(xr + e);
			if (add) {
				const float *y = g.y + (size_t)m * g.nsum * g.ldy + e;
				const float4 a = g.a ? get(g.a + o + e) : zero, c = g.abias ? get(g.abias + e) : zero, b = g.b ? get(g.b + o + e) : zero;
				float4 f[U];
#pragma unroll
				for (int j = 0; j < U; ++j) f[j] = j < g.nsum ? get(y + (size_t)j * g.ldy) : zero;
				float4 t = plus(plus(f[0], f[1]), plus(f[2], f[3]));
				for (int j = U; j < g.nsum; ++j) t = plus(t, get(y + (size_t)j * g.ldy));
				t = plus(plus(plus(a, c), b), t);
				v = make_float4(fmaf(g.mult, t.x, v.x), fmaf(g.mult, t.y, v.y), fmaf(g.mult, t.z, v.z), fmaf(g.mult, t.w, v.w));
				*reinterpret_cast<float4 *>(xr + e) = v;
			}
			*reinterpret_cast<float4 *>(vals + e) = v;
		}
	} else
		for (int e = tid; e < dim; e += nt) {
			float v = xr[e];
			if (add) {
				float s = g.a ? g.a[o + e] : 0.f, f = 0.f;
				if (g.abias) s += g.abias[e];
				if (g.b) s += g.b[o + e];
				for (int j = 0; j < g.nsum; ++j) f += g.y[((size_t)m * g.nsum + j) * g.ldy + e];
				v = fmaf(g.mult, s + f, v);
				xr[e] = v;
			}
			vals[e] = v;
		}
	if (!g.w) return;
	__syncthreads();
	const int size = dim / g.groups, wpg = max(1, nw / g.groups), slots = nw / wpg; // warps per group, groups in flight
	if (warp / wpg < slots)
		for (int k = warp / wpg; k < g.groups; k += slots) {
			float s = 0.f;
			for (int e = lane + 32 * (warp % wpg); e < size; e += 32 * wpg) s = fmaf(vals[k * size + e], vals[k * size + e], s);
			s = warp_sum(s);
			if (lane == 0) part[k * wpg + warp % wpg] = s;
		}
	__syncthreads();
	for (int k = tid; k < g.groups; k += nt) { // a thread owns its groups' partials
		float s = 0.f;
		for (int i = 0; i < wpg; ++i) s += part[k * wpg + i];
		part[g.groups * wpg + k] = 1.0f / sqrtf(s / size + g.eps);
	}
	__syncthreads();
	const float *r = part + g.groups * wpg;
	if (g.vec && size % 4 == 0) {
		for (int e = tid * 4; e < dim; e += nt * 4) {
			const float4 v = *reinterpret_cast<const float4 *>(vals + e), w = *reinterpret_cast<const float4 *>(g.w + e);
			const float k = r[e / size];
			const float4 h = make_float4(v.x * k * w.x, v.y * k * w.y, v.z * k * w.z, v.w * k * w.w);
			if (g.out) *reinterpret_cast<float4 *>(g.out + o + e) = h;
			if (g.out16) *reinterpret_cast<uint2 *>(static_cast<uint16_t *>(g.out16) + o + e) = pack4_16(h, g.bf16);
		}
		return;
	}
	for (int e = tid; e < dim; e += nt) {
		const float v = vals[e] * r[e / size] * g.w[e];
		if (g.out) g.out[o + e] = v;
		if (g.out16) put16(g.out16, o + e, v, g.bf16);
	}
}

// ---- a decode row's products ------------------------------------------------------------------------------------------------
// The streaming GEMV of gemv.cuh (a warp owns R rows, 16 / R chunks of each in flight).  IN: input = layer norm of x, per output
// segment blended with the previous position's norm output; a CTA takes a contiguous range of row groups, so that it stages one
// or two segments' inputs.  OUT: input = [x1 (n1) | silu-gated activation of (g | u)], the output rows are added to res.
constexpr int kBlockThreads = 256, kMaxSegs = 8;
struct GemvBlockArgs {
	float *out;
	const char *w;
	int n, d;
	const float *x, *nw, *nb; // IN: residual row, norm weight and bias
	float eps;
	int nseg, seg_end[kMaxSegs]; // output rows of a segment: [seg_end[s - 1], seg_end[s])
	const float *mu;             // (nseg, n); plain bit s: the norm output itself
	int plain;
	float *state;                // (2, n) or null
	const float *x1, *gu;        // OUT
	int n1, ff, act;
	float *res;
	const float *add;            // OUT: also added to res (null: nothing)
	int pos0;
	const int *ctl;
};

template <int DT, int R, bool IN>
__global__ void __launch_bounds__(kBlockThreads) gemv_block_kernel(GemvBlockArgs a) {
	extern __shared__ __align__(16) float smem[];
	float *red = smem, *xs = smem + 36;
	constexpr int EP = WTraits<DT>::EP, B = WTraits<DT>::BYTES, U = 16 / R;
	const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
	const size_t row_bytes = (size_t)a.n * B;
	auto rows = [&](int row, int end) {
		const char *ptr[R];
#pragma unroll
		for (int r = 0; r < R; ++r) ptr[r] = a.w + (size_t)min(row + r, end - 1) * row_bytes;
		float acc[R];
		warp_rows_dot<DT, R, U>(ptr, xs, a.n, acc);
#pragma unroll
		for (int r = 0; r < R; ++r)
			if (lane == r && row + r < end) {
				if (IN) a.out[row + r] = acc[r];
				else {
					float v = a.res[row + r] + acc[r];
					if (a.add) v += a.add[row + r];
					a.res[row + r] = v;
				}
			}
	};
	if constexpr (!IN) {
		const int ntasks = (a.d + R - 1) / R;
		const int first = blockIdx.x * nw + warp;
#pragma unroll 4
		for (int e = threadIdx.x * 4; e < a.n1; e += blockDim.x * 4) *reinterpret_cast<float4 *>(xs + xs_slot<EP>(e)) = *reinterpret_cast<const float4 *>(a.x1 + e);
#pragma unroll 4
		for (int e = threadIdx.x * 4; e < a.ff; e += blockDim.x * 4) {
			const float4 g = *reinterpret_cast<const float4 *>(a.gu + e), u = *reinterpret_cast<const float4 *>(a.gu + a.ff + e);
			*reinterpret_cast<float4 *>(xs + xs_slot<EP>(a.n1 + e)) =
			    make_float4(glu_value(g.x, u.x, a.act, 1.f, 0.f, 0.f), glu_value(g.y, u.y, a.act, 1.f, 0.f, 0.f), glu_value(g.z, u.z, a.act, 1.f, 0.f, 0.f),
			                glu_value(g.w, u.w, a.act, 1.f, 0.f, 0.f));
		}
		__syncthreads();
		for (int t = first; t < ntasks; t += gridDim.x * nw) rows(t * R, a.d);
	} else {
		// row groups never straddle two segments; this CTA's range [t0, t1) of all groups
		int total = 0;
		for (int g = 0, at = 0; g < a.nseg; ++g) total += (a.seg_end[g] - at + R - 1) / R, at = a.seg_end[g];
		const int t0 = (int)((long long)blockIdx.x * total / gridDim.x), t1 = (int)((long long)(blockIdx.x + 1) * total / gridDim.x);
		float s = 0.f;
#pragma unroll 4
		for (int e = threadIdx.x * 4; e < a.n; e += blockDim.x * 4) {
			const float4 v = *reinterpret_cast<const float4 *>(a.x + e);
			s += (v.x + v.y) + (v.z + v.w);
		}
		const float mean = block_sum(s, red) / a.n;
		float ss = 0.f;
#pragma unroll 4
		for (int e = threadIdx.x * 4; e < a.n; e += blockDim.x * 4) {
			const float4 v = *reinterpret_cast<const float4 *>(a.x + e);
			const float b = v.x - mean, c = v.y - mean, d = v.z - mean, f = v.w - mean;
			ss += (b * b + c * c) + (d * d + f * f);
		}
		const float sc = 1.0f / sqrtf(block_sum(ss, red) / a.n + a.eps);
		const int p = first_pos(a.ctl, a.pos0);
		const float *prev = a.state ? a.state + (size_t)((p + 1) & 1) * a.n : nullptr;
		auto stage = [&](int seg) {
			const bool mix = !((a.plain >> seg) & 1);
			float *keep = a.state && blockIdx.x == 0 ? a.state + (size_t)(p & 1) * a.n : nullptr;
#pragma unroll 2
			for (int e = threadIdx.x * 4; e < a.n; e += blockDim.x * 4) {
				const float4 v = *reinterpret_cast<const float4 *>(a.x + e), g = *reinterpret_cast<const float4 *>(a.nw + e), b = *reinterpret_cast<const float4 *>(a.nb + e);
				float4 o = make_float4((v.x - mean) * sc * g.x + b.x, (v.y - mean) * sc * g.y + b.y, (v.z - mean) * sc * g.z + b.z, (v.w - mean) * sc * g.w + b.w);
				if (keep) *reinterpret_cast<float4 *>(keep + e) = o;
				if (mix) {
					const float4 m = *reinterpret_cast<const float4 *>(a.mu + (size_t)seg * a.n + e);
					const float4 q = p > 0 ? *reinterpret_cast<const float4 *>(prev + e) : make_float4(0.f, 0.f, 0.f, 0.f);
					o.x += (q.x - o.x) * m.x, o.y += (q.y - o.y) * m.y, o.z += (q.z - o.z) * m.z, o.w += (q.w - o.w) * m.w;
				}
				*reinterpret_cast<float4 *>(xs + xs_slot<EP>(e)) = o;
			}
		};
		int base = 0, start = 0; // first group and first row of the segment
		for (int g = 0; g < a.nseg; ++g) {
			const int groups = (a.seg_end[g] - start + R - 1) / R;
			const int lo = max(t0, base), hi = min(t1, base + groups);
			if (lo < hi) {
				__syncthreads(); // the previous segment's input has been read
				stage(g);
				__syncthreads();
				for (int t = lo + warp; t < hi; t += nw) rows(start + (t - base) * R, a.seg_end[g]);
			}
			base += groups, start = a.seg_end[g];
		}
	}
}

template <bool IN>
static int launch_gemv_block(const GemvBlockArgs &a, int dtype, cudaStream_t st) {
	const int ep = dtype == YALM_F32 ? 4 : 8, ch = 32 * ep;
	const size_t smem = (36 + (size_t)((a.n + ch - 1) / ch * ch)) * sizeof(float);
	if (!a.w || a.n < 1 || a.d < 1 || a.n % ep || ((uintptr_t)a.w & 15) || (int)smem > device_info().max_smem_optin) return YALM_EINVAL;
	// Rows per warp.  IN: two (four leave every CTA fewer, longer turns behind its staging: 10 % slower per token at widths 2048 and 4096).
	// OUT stages long inputs, so fewer CTAs with two rows per warp when that still gives 12 warps per SM a task, else one.
	int R = IN || (a.d + 1) / 2 >= (long)device_info().sms * 12 ? 2 : 1;
	while (R < 4 && a.n / ch < 16 / R) R *= 2;                         // short rows: the 16 loads in flight must come from more rows
	cudaError_t err = cudaSuccess;
#define BLOCK_LAUNCH(DT_, R_)                                                                                                              \
	{                                                                                                                                      \
		const int grid = persistent_grid((const void *)gemv_block_kernel<DT_, R_, IN>, kBlockThreads, smem, (a.d + R_ - 1) / R_, &err);    \
		if (err != cudaSuccess) return (int)err;                                                                                           \
		gemv_block_kernel<DT_, R_, IN><<<grid, kBlockThreads, smem, st>>>(a);                                                              \
	}
#define BLOCK_ROWS(DT_)                       \
	{                                         \
		if (R == 4) BLOCK_LAUNCH(DT_, 4)      \
		else if (R == 2) BLOCK_LAUNCH(DT_, 2) \
		else BLOCK_LAUNCH(DT_, 1)             \
	}
	if (dtype == YALM_F32) BLOCK_ROWS(YALM_F32)
	else if (dtype == YALM_F16) BLOCK_ROWS(YALM_F16)
	else if (dtype == YALM_BF16) BLOCK_ROWS(YALM_BF16)
	else return YALM_EINVAL;
#undef BLOCK_ROWS
#undef BLOCK_LAUNCH
	return (int)cudaGetLastError();
}

} // namespace stack
} // namespace yalm

using namespace yalm;
using namespace yalm::stack;

static inline bool al16(const void *p) { return ((uintptr_t)p & 15) == 0; }

extern "C" int yalm_layer_norm_rows(float *out, void *out16, int bf16, float *x, const float *add, const int *rows, const float *w, const float *bias, float eps,
                                    int n, int dim, yalm_stream_t s) {
	if ((!out && !out16) || !x || !w || n < 1 || dim < 1 || (size_t)dim * 4 > 200 * 1024 || (dim % 4 == 0 && (!al16(x) || !al16(w) || !al16(bias) || !al16(out) || !al16(add) || ((uintptr_t)out16 & 7))))
		return YALM_EINVAL;
	const size_t smem = sizeof(float) * (size_t)dim;
	if (smem > 48 * 1024) YALM_TRY(cudaFuncSetAttribute(layer_norm_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
	layer_norm_rows_kernel<<<n, 256, smem, (cudaStream_t)s>>>(out, out16, bf16, x, add, rows, w, bias, eps, dim);
	return (int)cudaGetLastError();
}

static int launch_group_norm(GroupNormArgs g, int n, cudaStream_t st) {
	if (!g.x || n < 1 || g.dim < 1 || g.groups < 1 || g.dim % g.groups || g.nsum < 0 || (g.nsum && !g.y) || (g.w && !g.out && !g.out16)) return YALM_EINVAL;
	g.vec = g.dim % 4 == 0 && g.ldy % 4 == 0 && al16(g.x) && al16(g.a) && al16(g.abias) && al16(g.b) && al16(g.y) && al16(g.out) && al16(g.w) && ((uintptr_t)g.out16 & 7) == 0;
	const int threads = n <= 4 && g.dim > 512 ? std::min(1024, (g.vec ? g.dim / 4 + 31 : g.dim + 31) / 32 * 32) : 256;
	const size_t smem = sizeof(float) * ((size_t)g.dim + 2 * (size_t)g.groups + threads / 32);
	if ((int)smem > device_info().max_smem_optin) return YALM_EINVAL;
	if (smem > 48 * 1024) YALM_TRY(cudaFuncSetAttribute(group_norm_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
	group_norm_rows_kernel<<<n, threads, smem, st>>>(g);
	return (int)cudaGetLastError();
}

extern "C" int yalm_group_norm_rows(float *out, void *out16, int bf16, const float *x, const int *rows, const float *w, int groups, float eps, int n, int dim,
                                    yalm_stream_t s) {
	if (!w) return YALM_EINVAL;
	GroupNormArgs g{};
	g.x = const_cast<float *>(x), g.out = out, g.out16 = out16, g.bf16 = bf16, g.rows = rows, g.w = w, g.groups = groups, g.dim = dim, g.eps = eps;
	return launch_group_norm(g, n, (cudaStream_t)s);
}

extern "C" int yalm_residual_group_norm_rows(float *x, float mult, const float *a, const float *a_bias, const float *b, const float *y, int ldy, int nsum,
                                             float *out, void *out16, int bf16, const float *w, int groups, float eps, int n, int dim, yalm_stream_t s) {
	if (!a && !b && !y) return YALM_EINVAL;
	GroupNormArgs g{};
	g.x = x, g.mult = mult, g.a = a, g.abias = a_bias, g.b = b, g.y = y, g.ldy = ldy, g.nsum = nsum;
	g.out = out, g.out16 = out16, g.bf16 = bf16, g.w = w, g.groups = groups, g.dim = dim, g.eps = eps;
	return launch_group_norm(g, n, (cudaStream_t)s);
}

extern "C" int yalm_mix_rows(float *out, void *out16, int bf16, const float *h, const float *mu, int n_mixes, int plain_mask, float *state, int n, int dim, int pos0,
                             const int *ctl, yalm_stream_t s) {
	if ((!out && !out16) || !h || !mu || !state || n_mixes < 1 || n_mixes > 31 || n < 1 || dim < 1) return YALM_EINVAL;
	cudaStream_t st = (cudaStream_t)s;
	mix_rows_kernel<<<dim3((dim + 255) / 256, n), 256, 0, st>>>(out, out16, bf16, h, mu, n_mixes, MixMask{plain_mask}, state, n, dim, pos0, ctl);
	keep_row_kernel<<<(dim + 255) / 256, 256, 0, st>>>(state, h, n, dim, pos0, ctl);
	return (int)cudaGetLastError();
}

extern "C" int yalm_delta_in_rows(float *out, float *gates, const float *in, const float *raw, int ldi, const float *conv_w, float *ring, const float *a_log,
                                  const float *dt_bias, int n, int heads, int kv_heads, int dim, int vdim, int taps, float unit_eps, float q_scale, int pos0,
                                  const int *ctl, yalm_stream_t s) {
	if (!out || !gates || !in || !raw || !conv_w || !ring || !a_log || !dt_bias || n < 1 || heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 1 ||
	    dim > kDeltaMaxD || vdim < 1 || taps < 1)
		return YALM_EINVAL;
	cudaStream_t st = (cudaStream_t)s;
	const DeltaInArgs a{out, gates, in, raw, ldi, conv_w, ring, a_log, dt_bias, n, heads, kv_heads, dim, vdim, taps, unit_eps, q_scale, pos0, ctl};
	const int units = 2 * kv_heads + (heads * vdim + 127) / 128, C = 2 * kv_heads * dim + heads * vdim;
	delta_in_rows_kernel<<<dim3(n, std::max(1, std::min((units + kDeltaWarps - 1) / kDeltaWarps, n >= 64 ? 4 : 16))), kDeltaWarps * 32, 0, st>>>(a);
	conv_ring_rows_kernel<<<(C + 127) / 128, 128, 0, st>>>(ring, in, ldi, n, C, taps, pos0, ctl);
	return (int)cudaGetLastError();
}

extern "C" int yalm_wkv_decay_rows(float *out, int ldo, const float *t, int ldt, const void *w2, const float *w0, int dtype, int n, int channels, int rank,
                                   yalm_stream_t s) {
	if (!out || !t || !w2 || !w0 || n < 1 || channels < 1 || rank < 1) return YALM_EINVAL;
	const size_t smem = sizeof(float) * kDecayRows * (size_t)((rank + 7) & ~7);
	if (smem > 48 * 1024) return YALM_EINVAL;
	const dim3 grid((channels + 127) / 128, (n + kDecayRows - 1) / kDecayRows);
	cudaStream_t st = (cudaStream_t)s;
	const int vec = al16(w2) && rank % (dtype == YALM_F32 ? 4 : 8) == 0;
	if (dtype == YALM_F32) wkv_decay_rows_kernel<YALM_F32><<<grid, 128, smem, st>>>(out, ldo, t, ldt, w2, w0, n, channels, rank, vec);
	else if (dtype == YALM_F16) wkv_decay_rows_kernel<YALM_F16><<<grid, 128, smem, st>>>(out, ldo, t, ldt, w2, w0, n, channels, rank, vec);
	else if (dtype == YALM_BF16) wkv_decay_rows_kernel<YALM_BF16><<<grid, 128, smem, st>>>(out, ldo, t, ldt, w2, w0, n, channels, rank, vec);
	else return YALM_EINVAL;
	return (int)cudaGetLastError();
}

extern "C" int yalm_block_out_rows(float *out, void *out16, int bf16, int ldo, const float *o, int ldi, const float *gate, const float *gu, int ldp,
                                   const float *norm_w, int w_stride, float eps, int n, int heads, int vdim, int ff, int act, yalm_stream_t s) {
	if ((!out && !out16) || !o || n < 1 || heads < 1 || vdim < 1 || ff < 0 || (ff && !gu) || (norm_w && !gate) || ldo < heads * vdim + ff) return YALM_EINVAL;
	const BlockOutArgs a{out, out16, bf16, ldo, o, ldi, gate, gu, ldp, norm_w, w_stride, heads, vdim, ff, act, eps};
	const int units = heads + (ff + 127) / 128;
	block_out_rows_kernel<<<dim3(n, std::max(1, std::min((units + 7) / 8, n >= 64 ? 4 : 16))), 256, 0, (cudaStream_t)s>>>(a);
	return (int)cudaGetLastError();
}

template <int MODE>
static int launch_state_step(const StateStepArgs &a, int dtype, cudaStream_t st) {
	if (a.D < 1 || a.D > 256 || a.P < 1 || a.H < 1 || a.G < 1 || a.H % a.G) return YALM_EINVAL;
	const int epl = a.D <= 8 ? 1 : a.D <= 16 ? 2 : a.D <= 32 ? 4 : a.D <= 64 ? 8 : a.D <= 128 ? 16 : 32;
	const size_t smem = sizeof(float) * (4 * (size_t)8 * (epl + (epl >= 8 ? 4 : 0)) + a.P + std::max(a.P, MODE == kStepBonus ? a.rank : 0));
	if (smem > 48 * 1024) return YALM_EINVAL;
#define STEP_DT(EPL_, DT_) state_step_kernel<EPL_, MODE, DT_><<<a.H, kStepThreads, smem, st>>>(a)
#define STEP_CASE(EPL_)                                             \
	{                                                               \
		if constexpr (MODE != kStepBonus) STEP_DT(EPL_, YALM_F32);  \
		else if (dtype == YALM_F32) STEP_DT(EPL_, YALM_F32);        \
		else if (dtype == YALM_F16) STEP_DT(EPL_, YALM_F16);        \
		else if (dtype == YALM_BF16) STEP_DT(EPL_, YALM_BF16);      \
		else return YALM_EINVAL;                                    \
	}
	if (epl == 1) STEP_CASE(1)
	else if (epl == 2) STEP_CASE(2)
	else if (epl == 4) STEP_CASE(4)
	else if (epl == 8) STEP_CASE(8)
	else if (epl == 16) STEP_CASE(16)
	else STEP_CASE(32)
#undef STEP_CASE
#undef STEP_DT
	return (int)cudaGetLastError();
}

extern "C" int yalm_delta_step(float *out, float *state, const float *proj, int o_qkv, int o_gate, int o_beta, int o_decay, const float *conv_w, float *ring,
                               const float *a_log, const float *dt_bias, const float *norm_w, int heads, int kv_heads, int dim, int vdim, int taps,
                               float unit_eps, float q_scale, float eps, int pos0, const int *ctl, yalm_stream_t s) {
	if (!out || !state || !proj || !conv_w || !ring || !a_log || !dt_bias || !norm_w || taps < 1) return YALM_EINVAL;
	StateStepArgs a{};
	a.out = out, a.state = state, a.proj = proj, a.o_q = o_qkv, a.o_gate = o_gate, a.o_beta = o_beta, a.o_decay = o_decay;
	a.H = heads, a.G = kv_heads, a.D = dim, a.P = vdim, a.conv_w = conv_w, a.ring = ring, a.taps = taps, a.a_log = a_log, a.dt_bias = dt_bias;
	a.unit_eps = unit_eps, a.q_scale = q_scale, a.norm_w = norm_w, a.w_stride = 0, a.eps = eps, a.pos0 = pos0, a.ctl = ctl;
	return launch_state_step<kStepDelta>(a, YALM_F32, (cudaStream_t)s);
}

extern "C" int yalm_wkv_step(float *out, float *state, const float *proj, int o_r, int o_k, int o_v, int o_gate, int o_decay, const void *w2, const float *w0,
                             const float *bonus, const float *norm_w, int dtype, int heads, int dim, int rank, float eps, int pos0, const int *ctl,
                             yalm_stream_t s) {
	if (!out || !state || !proj || !w2 || !w0 || !bonus || !norm_w || rank < 1) return YALM_EINVAL;
	StateStepArgs a{};
	a.out = out, a.state = state, a.proj = proj, a.o_q = o_r, a.o_k = o_k, a.o_v = o_v, a.o_gate = o_gate, a.o_decay = o_decay;
	a.H = heads, a.G = heads, a.D = dim, a.P = dim, a.w2 = w2, a.w0 = w0, a.bonus = bonus, a.rank = rank;
	a.vec = al16(w2) && rank % (dtype == YALM_F32 ? 4 : 8) == 0;
	a.norm_w = norm_w, a.w_stride = dim, a.eps = eps, a.pos0 = pos0, a.ctl = ctl;
	return launch_state_step<kStepBonus>(a, dtype, (cudaStream_t)s);
}

extern "C" int yalm_retention_step(float *out, float *state, const float *proj, int o_q, int o_k, int o_v, int o_gate, const float *decay, const float *freq,
                                   float magnitude, int rot_dims, int interleaved, float k_scale, int heads, int dim, int vdim, float eps, int pos0, const int *ctl,
                                   yalm_stream_t s) {
	if (!out || !state || !proj || !decay || rot_dims < 0 || rot_dims % 2 || rot_dims > dim || (rot_dims > 0 && !freq)) return YALM_EINVAL;
	StateStepArgs a{};
	a.out = out, a.state = state, a.proj = proj, a.o_q = o_q, a.o_k = o_k, a.o_v = o_v, a.o_gate = o_gate;
	a.H = heads, a.G = heads, a.D = dim, a.P = vdim, a.q_scale = k_scale, a.eps = eps, a.pos0 = pos0, a.ctl = ctl;
	a.decay = decay, a.freq = freq, a.rot_mag = magnitude, a.rot_dims = rot_dims, a.interleaved = interleaved;
	return launch_state_step<kStepFixed>(a, YALM_F32, (cudaStream_t)s);
}

extern "C" int yalm_gemv_block_in(float *out, const float *x, const void *w, int n, int d, int dtype, const float *norm_w, const float *norm_b, float eps,
                                  int n_segments, const int *segment_end, const float *mu, int plain_mask, float *state, int pos0, const int *ctl, yalm_stream_t s) {
	if (!out || !x || !norm_w || !norm_b || !al16(x) || !al16(norm_w) || !al16(norm_b) || n_segments < 1 || n_segments > kMaxSegs || (n_segments > 1 && !segment_end) ||
	    (state && !al16(state)) || !al16(mu))
		return YALM_EINVAL;
	GemvBlockArgs a{};
	a.out = out, a.w = (const char *)w, a.n = n, a.d = d, a.x = x, a.nw = norm_w, a.nb = norm_b, a.eps = eps, a.nseg = n_segments;
	for (int i = 0, at = 0; i < n_segments; ++i) {
		a.seg_end[i] = segment_end ? segment_end[i] : d;
		if (a.seg_end[i] <= at || a.seg_end[i] > d) return YALM_EINVAL;
		at = a.seg_end[i];
		if (!((plain_mask >> i) & 1) && (!mu || !state)) return YALM_EINVAL;
	}
	if (a.seg_end[n_segments - 1] != d) return YALM_EINVAL;
	a.mu = mu, a.plain = plain_mask, a.state = state, a.pos0 = pos0, a.ctl = ctl;
	return launch_gemv_block<true>(a, dtype, (cudaStream_t)s);
}

extern "C" int yalm_gemv_block_out(float *res, const float *x1, int n1, const float *gu, int ff, int act, const void *w, int d, int dtype, const float *add,
                                   yalm_stream_t s) {
	if (!res || n1 < 0 || ff < 0 || n1 % 4 || ff % 4 || (n1 && (!x1 || !al16(x1))) || (ff && (!gu || !al16(gu)))) return YALM_EINVAL;
	GemvBlockArgs a{};
	a.w = (const char *)w, a.n = n1 + ff, a.d = d, a.x1 = x1, a.gu = gu, a.n1 = n1, a.ff = ff, a.act = act, a.res = res, a.add = add;
	return launch_gemv_block<false>(a, dtype, (cudaStream_t)s);
}
