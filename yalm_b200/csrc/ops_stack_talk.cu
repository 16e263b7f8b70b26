// Attention whose heads exchange scores before the softmax ("talking heads"), with a soft cap and a learned distance bias.
// Position i, key j, heads h:
//   z_h(j) = cap * tanh(q_h . k_g(h)(j) * scale / cap) + bias[h, min(i - j, n_bias - 1)]      (cap 0: no cap; bias null: none)
//   s_h(j) = sum_g mix[h, g] z_g(j)                                                           (mix null: s = z)
//   a_h = softmax of s_h over the visible keys,  out_h = sum_j a_h(j) v_g(h)(j)  (* sigmoid(gate[h]) with a gate)
// Keys and values are rings (kv head, slot = position % ring, channel); position i sees 0 <= i - j < window (0: all j <= i).
// A score depends on every head's query, so unlike the other attentions a CTA works on all heads at once.
//
//   attn_mixed_rows_kernel    any sizes, fp32 or bf16 rings, fp32 arithmetic: one CTA per (row, key split)
//   attn_mixed_decode_kernel  a few rows over bf16 rings: the heads of a kv head are the M tile of the tensor-core products
//   attn_mixed_mma_kernel     prompt portions over bf16 rings: 16 rows are the M tile, all heads' scores of a key tile meet in
//                             shared memory, where they are mixed in fp32
// Operands of the products are bf16 in the last two; scores, cap, bias, mixing, maxima, sums and accumulators are fp32 in all
// three.  Split keys leave unnormalised partials (accumulator, max, sum) that yalm_attn_split_merge joins in order.
#include "common.cuh"
#include "launch.h"
#include "stack_rows.cuh"

#include <cuda_bf16.h>

#include <algorithm>
#include <type_traits>

namespace yalm {
namespace stack {

struct MixedArgs {
	float *out;
	int ldo;
	const float *q;
	int ldq;
	const void *kc, *vc;
	const float *bias;
	int n_bias;
	const float *mix;
	const float *gate;
	int ldg;
	float *part;
	int n, H, G, dk, dv, ring, window;
	float scale, cap;
	int pos0;
	const int *ctl;
};

__device__ __forceinline__ void mx_ldsm_x4(uint32_t (&r)[4], const void *p) {
	asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
	             : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
	             : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void mx_ldsm_x4_t(uint32_t (&r)[4], const void *p) {
	asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
	             : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
	             : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void mx_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
	asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
	             : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
	             : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16 bytes global -> shared; valid false: zeros (the source is not read)
__device__ __forceinline__ void mx_cp16(void *smem, const void *gmem, bool valid) {
	asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ uint32_t mx_pack(float a, float b) {
	const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
	return *reinterpret_cast<const uint32_t *>(&h);
}
// cap * tanh(x / cap).  FAST: from one exponential; its error is about 1e-7 of the cap, far below a bf16 product's.
template <bool FAST>
__device__ __forceinline__ float soft_cap(float x, float cap, float inv_cap) {
	if (FAST) return cap - __fdividef(2.f * cap, 1.f + __expf(fminf(2.f * x * inv_cap, 80.f)));
	return cap * tanhf(x / cap);
}

// ---- any sizes ----------------------------------------------------------------------------------------------------------
// grid (rows, splits), 256 threads.  Key tiles of 32: warp = head, lane = key for the scores; the mixing reads them back from
// shared memory; a warp then runs a head's online softmax, and every thread adds the tile to its output channels.
constexpr int kMixTile = 32, kMixThreads = 256;
template <typename CT>
__global__ void __launch_bounds__(kMixThreads) attn_mixed_rows_kernel(MixedArgs a) {
	extern __shared__ __align__(16) float mx_sm[];
	const int H = a.H, G = a.G, R = H / G, dk = a.dk, dv = a.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = kMixThreads / 32;
	constexpr int LD = kMixTile + 1;
	float *qs = mx_sm, *z = qs + H * dk, *p = z + H * LD, *acc = p + H * LD, *ml = acc + H * dv; // ml: max, sum, correction per head
	const int m = blockIdx.x, sp = blockIdx.y, nsplit = gridDim.y;
	const int i = first_pos(a.ctl, a.pos0) + m, lo = a.window > 0 ? max(0, i - a.window + 1) : 0;
	const int tiles = (i - lo) / kMixTile + 1, per = (tiles + nsplit - 1) / nsplit, t_end = min(tiles, (sp + 1) * per);
	const CT *kc = static_cast<const CT *>(a.kc), *vc = static_cast<const CT *>(a.vc);
	for (int e = tid; e < H * dk; e += kMixThreads) qs[e] = a.q[(size_t)m * a.ldq + e];
	for (int e = tid; e < H * dv; e += kMixThreads) acc[e] = 0.f;
	for (int h = tid; h < H; h += kMixThreads) ml[h] = -INFINITY, ml[H + h] = 0.f;
	__syncthreads();
	for (int t = sp * per; t < t_end; ++t) {
		const int base = lo + t * kMixTile, j = base + lane, cnt = min(kMixTile, i - base + 1);
		for (int h = warp; h < H; h += nw) {
			float s = 0.f;
			if (lane < cnt) {
				const CT *kr = kc + ((size_t)(h / R) * a.ring + j % a.ring) * dk;
				for (int d = 0; d < dk; ++d) s = fmaf(cache_get(kr, d), qs[h * dk + d], s);
				s *= a.scale;
				if (a.cap > 0.f) s = soft_cap<false>(s, a.cap, 0.f);
				if (a.bias) s += a.bias[(size_t)h * a.n_bias + min(i - j, a.n_bias - 1)];
			}
			z[h * LD + lane] = s;
		}
		__syncthreads();
		for (int h = warp; h < H; h += nw) {
			float s = z[h * LD + lane];
			if (a.mix) {
				s = 0.f;
				for (int g = 0; g < H; ++g) s = fmaf(a.mix[h * H + g], z[g * LD + lane], s);
			}
			if (lane >= cnt) s = -INFINITY;
			const float m0 = ml[h], nm = fmaxf(m0, warp_max(s)), e = expf(s - nm); // nm is finite: a tile holds a visible key
			const float c = m0 == -INFINITY ? 0.f : expf(m0 - nm), l = warp_sum(e);
			p[h * LD + lane] = e;
			__syncwarp();
			if (lane == 0) ml[h] = nm, ml[H + h] = ml[H + h] * c + l, ml[2 * H + h] = c;
		}
		__syncthreads();
		for (int e = tid; e < H * dv; e += kMixThreads) {
			const int h = e / dv, c = e % dv;
			const CT *vb = vc + (size_t)(h / R) * a.ring * dv + c;
			float o = acc[e] * ml[2 * H + h];
			for (int k = 0; k < cnt; ++k) o = fmaf(p[h * LD + k], cache_get(vb, (size_t)((base + k) % a.ring) * dv), o);
			acc[e] = o;
		}
		__syncthreads();
	}
	for (int e = tid; e < H * dv; e += kMixThreads) {
		const int h = e / dv, c = e % dv;
		if (a.part) {
			float *pr = a.part + ((size_t)(m * H + h) * nsplit + sp) * (dv + 2);
			pr[c] = acc[e];
			if (c == 0) pr[dv] = ml[h], pr[dv + 1] = ml[H + h];
		} else {
			const float f = a.gate ? 1.f / (1.f + expf(-a.gate[(size_t)m * a.ldg + h])) : 1.f;
			a.out[(size_t)m * a.ldo + e] = acc[e] / ml[H + h] * f;
		}
	}
}

// ---- a few rows, bf16 rings ---------------------------------------------------------------------------------------------
// grid (rows, splits), 8 warps.  The up to 16 heads of a kv head are one A operand.  Per tile of TK keys: a warp takes (kv head,
// 16 keys) products for the scores of all heads, which meet in shared memory; a warp mixes and normalises one head (lane = key)
// and leaves its weights as bf16; a warp then takes (kv head, 16 value channels) products.  Keys of the next tile load while the
// weights are formed, its values behind the products that use this tile's.
constexpr int kMdWarps = 8, kMdThreads = kMdWarps * 32;
struct MixedDecodeLayout { // byte offsets in shared memory
	size_t k, v, z, p, ml, total;
};
__host__ __device__ inline MixedDecodeLayout mixed_decode_layout(int H, int G, int dk, int dv, int tk) {
	MixedDecodeLayout L;
	L.k = 2 * (size_t)G * 16 * (dk + 8);
	L.v = L.k + 2 * (size_t)G * tk * (dk + 8);
	L.p = L.v + 2 * (size_t)G * tk * (dv + 8);
	L.z = L.p + 2 * (size_t)G * 16 * (tk + 8);
	L.ml = L.z + 4 * (size_t)H * (tk + 1);
	L.total = L.ml + 4 * (size_t)3 * G * 16;
	return L;
}
template <int TK, int NU>
__global__ void __launch_bounds__(kMdThreads) attn_mixed_decode_kernel(MixedArgs a) {
	extern __shared__ __align__(16) char md_sm[];
	const int H = a.H, G = a.G, R = H / G, dk = a.dk, dv = a.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
	const int LDK = dk + 8, LDV = dv + 8;
	constexpr int LDP = TK + 8, LDZ = TK + 1;
	const MixedDecodeLayout lay = mixed_decode_layout(H, G, dk, dv, TK);
	__nv_bfloat16 *Qs = reinterpret_cast<__nv_bfloat16 *>(md_sm), *Ks = reinterpret_cast<__nv_bfloat16 *>(md_sm + lay.k),
	              *Vs = reinterpret_cast<__nv_bfloat16 *>(md_sm + lay.v), *Ps = reinterpret_cast<__nv_bfloat16 *>(md_sm + lay.p);
	float *z = reinterpret_cast<float *>(md_sm + lay.z), *ml = reinterpret_cast<float *>(md_sm + lay.ml); // per (kv head, row of 16): max, sum, correction
	const int m = blockIdx.x, sp = blockIdx.y, nsplit = gridDim.y, GR = G * 16;
	const int i = first_pos(a.ctl, a.pos0) + m, lo = a.window > 0 ? max(0, i - a.window + 1) : 0;
	const int tiles = (i - lo) / TK + 1, per = (tiles + nsplit - 1) / nsplit, t0 = sp * per, t_end = min(tiles, t0 + per);
	const __nv_bfloat16 *kc = static_cast<const __nv_bfloat16 *>(a.kc), *vc = static_cast<const __nv_bfloat16 *>(a.vc);
	const float inv_cap = a.cap > 0.f ? 1.f / a.cap : 0.f;
	auto stage = [&](__nv_bfloat16 *dst, const __nv_bfloat16 *src, int d, int ld, int t) { // rows past the position are zero-filled
		const int base = lo + t * TK, pieces = d / 8;
		for (int c = tid; c < G * TK * pieces; c += kMdThreads) {
			const int row = c / pieces, e = (c % pieces) * 8, g = row / TK, r = row % TK;
			const bool in = base + r <= i;
			mx_cp16(dst + (size_t)row * ld + e, src + ((size_t)g * a.ring + (in ? base + r : i) % a.ring) * d + e, in);
		}
		asm volatile("cp.async.commit_group;" ::: "memory");
	};
	if (t0 < t_end) stage(Ks, kc, dk, LDK, t0), stage(Vs, vc, dv, LDV, t0);
	for (int c = tid; c < GR * (dk / 4); c += kMdThreads) { // queries as bf16; rows past a kv head's heads: zeros
		const int row = c / (dk / 4), d = (c % (dk / 4)) * 4, g = row >> 4, r = row & 15;
		float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
		if (r < R) v = *reinterpret_cast<const float4 *>(a.q + (size_t)m * a.ldq + (size_t)(g * R + r) * dk + d);
		uint2 pk;
		pk.x = mx_pack(v.x, v.y), pk.y = mx_pack(v.z, v.w);
		*reinterpret_cast<uint2 *>(Qs + (size_t)row * LDK + d) = pk;
	}
	for (int c = tid; c < GR * LDP; c += kMdThreads) Ps[c] = __float2bfloat16_rn(0.f);
	for (int c = tid; c < GR; c += kMdThreads) ml[c] = -INFINITY, ml[GR + c] = 0.f, ml[2 * GR + c] = 0.f;
	float o[NU][2][4];
#pragma unroll
	for (int u = 0; u < NU; ++u)
#pragma unroll
		for (int t = 0; t < 2; ++t) o[u][t][0] = o[u][t][1] = o[u][t][2] = o[u][t][3] = 0.f;
	const int ar = (lane & 7) + ((lane >> 3) & 1) * 8, ac = (lane >> 4) * 8;  // A operand (and, transposed, values)
	const int br = (lane & 7) + (lane >> 4) * 8, bc = ((lane >> 3) & 1) * 8;  // keys
	const int vunits = G * (dv / 16), vper = dv / 16;
	for (int t = t0; t < t_end; ++t) {
		asm volatile("cp.async.wait_group 1;" ::: "memory"); // the tile's keys (its values are the group after)
		__syncthreads();
		const int base = lo + t * TK;
		// ---- scores ----
		for (int u = warp; u < G * (TK / 16); u += kMdWarps) {
			const int g = u / (TK / 16), k0 = (u % (TK / 16)) * 16;
			float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
			const __nv_bfloat16 *qp = Qs + (size_t)(g * 16 + ar) * LDK + ac, *kp = Ks + (size_t)(g * TK + k0 + br) * LDK + bc;
#pragma unroll 4
			for (int d = 0; d < dk; d += 16) {
				uint32_t A[4], B[4];
				mx_ldsm_x4(A, qp + d);
				mx_ldsm_x4(B, kp + d);
				mx_mma(s[0], A, B[0], B[1]);
				mx_mma(s[1], A, B[2], B[3]);
			}
#pragma unroll
			for (int e = 0; e < 8; ++e) {
				const int r = (lane >> 2) + ((e >> 1) & 1) * 8, key = k0 + (e >> 2) * 8 + (lane & 3) * 2 + (e & 1);
				if (r < R) {
					const int h = g * R + r;
					float v = s[e >> 2][e & 3] * a.scale;
					if (a.cap > 0.f) v = soft_cap<true>(v, a.cap, inv_cap);
					if (a.bias) v += a.bias[(size_t)h * a.n_bias + min(max(i - base - key, 0), a.n_bias - 1)];
					z[h * LDZ + key] = v;
				}
			}
		}
		__syncthreads();
		if (t + 1 < t_end) stage(Ks, kc, dk, LDK, t + 1);
		else asm volatile("cp.async.commit_group;" ::: "memory"); // an empty group keeps the count
		// ---- mixing and online softmax: warp = head, lane = key ----
		for (int h = warp; h < H; h += kMdWarps) {
			const int row = (h / R) * 16 + h % R;
			float s = -INFINITY;
			if (lane < TK) {
				s = z[h * LDZ + lane];
				if (a.mix) {
					s = 0.f;
#pragma unroll 4
					for (int g = 0; g < H; ++g) s = fmaf(__ldg(a.mix + h * H + g), z[g * LDZ + lane], s);
				}
				if (base + lane > i) s = -INFINITY;
			}
			const float m0 = ml[row], nm = fmaxf(m0, warp_max(s)), e = __expf(s - nm), c = m0 == -INFINITY ? 0.f : __expf(m0 - nm), l = warp_sum(e);
			if (lane < TK) Ps[row * LDP + lane] = __float2bfloat16_rn(e);
			__syncwarp();
			if (lane == 0) ml[row] = nm, ml[GR + row] = ml[GR + row] * c + l, ml[2 * GR + row] = c;
		}
		asm volatile("cp.async.wait_group 1;" ::: "memory"); // the tile's values
		__syncthreads();
		// ---- weighted sums ----
#pragma unroll
		for (int k = 0; k < NU; ++k) {
			const int u = warp + k * kMdWarps;
			if (u < vunits) {
				const int g = u / vper, c0 = (u % vper) * 16;
				const float ca = ml[2 * GR + g * 16 + (lane >> 2)], cb = ml[2 * GR + g * 16 + (lane >> 2) + 8];
#pragma unroll
				for (int x = 0; x < 2; ++x) o[k][x][0] *= ca, o[k][x][1] *= ca, o[k][x][2] *= cb, o[k][x][3] *= cb;
#pragma unroll
				for (int kk = 0; kk < TK / 16; ++kk) {
					uint32_t A[4], B[4];
					mx_ldsm_x4(A, Ps + (size_t)(g * 16 + ar) * LDP + kk * 16 + ac);
					mx_ldsm_x4_t(B, Vs + (size_t)(g * TK + kk * 16 + ar) * LDV + c0 + ac);
					mx_mma(o[k][0], A, B[0], B[1]);
					mx_mma(o[k][1], A, B[2], B[3]);
				}
			}
		}
		__syncthreads(); // values, weights and scores are read
		if (t + 1 < t_end) stage(Vs, vc, dv, LDV, t + 1);
	}
	asm volatile("cp.async.wait_group 0;" ::: "memory");
	__syncthreads();
#pragma unroll
	for (int k = 0; k < NU; ++k) {
		const int u = warp + k * kMdWarps;
		if (u >= vunits) continue;
		const int g = u / vper, c0 = (u % vper) * 16 + (lane & 3) * 2;
#pragma unroll
		for (int half = 0; half < 2; ++half) {
			const int r = (lane >> 2) + half * 8, h = g * R + r, row = g * 16 + r;
			if (r >= R) continue;
			float *dst;
			float f = 1.f;
			if (a.part) dst = a.part + ((size_t)(m * H + h) * nsplit + sp) * (dv + 2);
			else {
				dst = a.out + (size_t)m * a.ldo + (size_t)h * dv;
				f = 1.f / ml[GR + row];
				if (a.gate) f /= 1.f + expf(-a.gate[(size_t)m * a.ldg + h]);
			}
#pragma unroll
			for (int x = 0; x < 2; ++x) dst[c0 + x * 8] = o[k][x][half * 2] * f, dst[c0 + x * 8 + 1] = o[k][x][half * 2 + 1] * f;
			if (a.part && c0 == 0) dst[dv] = ml[row], dst[dv + 1] = ml[GR + row];
		}
	}
}

// ---- prompt portions, bf16 rings ------------------------------------------------------------------------------------------
// grid (ceil(n / 16), ceil(H / HS), splits), 16 warps; a CTA computes every head's scores for its 16 rows and the outputs of HS heads.
// Per tile of TK keys (all kv heads' keys and values at once):
//   scores   a warp takes (head, 16 keys) products; scaled, capped and biased they go to Z (head, row, key) in shared memory
//   mixing   a thread takes 8 heads x 2 keys of a row: sums over all heads' Z in registers, then back over Z's first HS planes
//   sums     16 / HS warps per head: the online softmax of the head's rows (the same in each of them), then P V for the warp's DW
//            value channels
// Keys of the next tile load from the end of the scores on, its values from the end of the sums on.
constexpr int kMmWarps = 16, kMmThreads = kMmWarps * 32, kMmRows = 16;
struct MixedMmaLayout {
	size_t k, v, z, mix, total;
};
__host__ __device__ inline MixedMmaLayout mixed_mma_layout(int H, int G, int dk, int dv, int tk, int hs) {
	MixedMmaLayout L;
	L.k = 2 * (size_t)H * 16 * (dk + 8);
	L.v = L.k + 2 * (size_t)G * tk * (dk + 8);
	L.z = L.v + 2 * (size_t)G * tk * (dv + 8);
	L.mix = L.z + 4 * (size_t)H * 16 * (tk + 8);
	L.total = L.mix + 4 * (size_t)H * (hs < 8 ? 8 : hs); // mix transposed: (g, output head)
	return L;
}
template <int TK, int DW>
__global__ void __launch_bounds__(kMmThreads) attn_mixed_mma_kernel(MixedArgs a, int HS) {
	extern __shared__ __align__(16) char mm_sm[];
	const int H = a.H, G = a.G, R = H / G, dk = a.dk, dv = a.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
	const int LDK = dk + 8, LDV = dv + 8, HP = HS < 8 ? 8 : HS;
	constexpr int LDZ = TK + 8, OT = DW / 8;
	const MixedMmaLayout lay = mixed_mma_layout(H, G, dk, dv, TK, HS);
	__nv_bfloat16 *Qs = reinterpret_cast<__nv_bfloat16 *>(mm_sm), *Ks = reinterpret_cast<__nv_bfloat16 *>(mm_sm + lay.k),
	              *Vs = reinterpret_cast<__nv_bfloat16 *>(mm_sm + lay.v);
	float *Z = reinterpret_cast<float *>(mm_sm + lay.z), *Ms = reinterpret_cast<float *>(mm_sm + lay.mix);
	const int i0 = blockIdx.x * kMmRows, h0 = blockIdx.y * HS, nh = min(HS, H - h0), sp = blockIdx.z, nsplit = gridDim.z;
	const int p0 = first_pos(a.ctl, a.pos0), last = min(i0 + kMmRows - 1, a.n - 1), i_last = p0 + last;
	const int lo_min = a.window > 0 ? max(0, p0 + i0 - a.window + 1) : 0;
	const int tiles = (i_last - lo_min) / TK + 1, per = (tiles + nsplit - 1) / nsplit, t0 = sp * per, t_end = min(tiles, t0 + per);
	const __nv_bfloat16 *kc = static_cast<const __nv_bfloat16 *>(a.kc), *vc = static_cast<const __nv_bfloat16 *>(a.vc);
	const float inv_cap = a.cap > 0.f ? 1.f / a.cap : 0.f;
	auto stage = [&](__nv_bfloat16 *dst, const __nv_bfloat16 *src, int d, int ld, int t) { // rows past the last position are zero-filled
		const int base = lo_min + t * TK, pieces = d / 8;
		for (int c = tid; c < G * TK * pieces; c += kMmThreads) {
			const int row = c / pieces, e = (c % pieces) * 8, g = row / TK, r = row % TK;
			const bool in = base + r <= i_last;
			mx_cp16(dst + (size_t)row * ld + e, src + ((size_t)g * a.ring + (in ? base + r : i_last) % a.ring) * d + e, in);
		}
		asm volatile("cp.async.commit_group;" ::: "memory");
	};
	if (t0 < t_end) stage(Ks, kc, dk, LDK, t0), stage(Vs, vc, dv, LDV, t0);
	for (int c = tid; c < H * 16 * (dk / 4); c += kMmThreads) { // (head, row, channel); rows past the last repeat it
		const int row = c / (dk / 4), d = (c % (dk / 4)) * 4, h = row >> 4, r = min(i0 + (row & 15), a.n - 1);
		const float4 v = *reinterpret_cast<const float4 *>(a.q + (size_t)r * a.ldq + (size_t)h * dk + d);
		uint2 pk;
		pk.x = mx_pack(v.x, v.y), pk.y = mx_pack(v.z, v.w);
		*reinterpret_cast<uint2 *>(Qs + (size_t)row * LDK + d) = pk;
	}
	for (int c = tid; c < H * HP; c += kMmThreads) {
		const int g = c / HP, oh = c % HP;
		Ms[c] = oh < nh ? (a.mix ? a.mix[(h0 + oh) * H + g] : (h0 + oh == g ? 1.f : 0.f)) : 0.f;
	}
	const int parts = kMmWarps / HS, hl = warp / parts, c_first = (warp % parts) * DW; // the head and value channels of this warp's sums
	const bool sums = hl < nh && c_first < dv;
	const int hg = (h0 + min(hl, nh - 1)) / R;
	float o[OT][4];
#pragma unroll
	for (int t = 0; t < OT; ++t) o[t][0] = o[t][1] = o[t][2] = o[t][3] = 0.f;
	float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f; // rows lane / 4 and lane / 4 + 8
	const int ar = (lane & 7) + ((lane >> 3) & 1) * 8, ac = (lane >> 4) * 8;
	const int br = (lane & 7) + (lane >> 4) * 8, bc = ((lane >> 3) & 1) * 8;
	for (int t = t0; t < t_end; ++t) {
		asm volatile("cp.async.wait_group 1;" ::: "memory"); // the tile's keys
		__syncthreads();
		const int base = lo_min + t * TK;
		// ---- scores ----
		auto scores = [&](int h, int k0, auto pieces) { // NP products of 16 keys that share the query fragments
			constexpr int NP = decltype(pieces)::value;
			const int g = h / R;
			float s[2 * NP][4];
#pragma unroll
			for (int x = 0; x < 2 * NP; ++x) s[x][0] = s[x][1] = s[x][2] = s[x][3] = 0.f;
			const __nv_bfloat16 *qp = Qs + (size_t)(h * 16 + ar) * LDK + ac, *kp = Ks + (size_t)(g * TK + k0 + br) * LDK + bc;
#pragma unroll 4
			for (int d = 0; d < dk; d += 16) {
				uint32_t A[4], B[NP][4];
				mx_ldsm_x4(A, qp + d);
#pragma unroll
				for (int x = 0; x < NP; ++x) mx_ldsm_x4(B[x], kp + (size_t)x * 16 * LDK + d);
#pragma unroll
				for (int x = 0; x < NP; ++x) mx_mma(s[2 * x], A, B[x][0], B[x][1]), mx_mma(s[2 * x + 1], A, B[x][2], B[x][3]);
			}
			const float *bh = a.bias ? a.bias + (size_t)h * a.n_bias : nullptr;
#pragma unroll
			for (int x = 0; x < 2 * NP; ++x)
#pragma unroll
				for (int half = 0; half < 2; ++half) {
					const int r = (lane >> 2) + half * 8, key = k0 + x * 8 + (lane & 3) * 2, dist = p0 + i0 + r - base - key; // of the first of two keys
					float2 v = make_float2(s[x][half * 2] * a.scale, s[x][half * 2 + 1] * a.scale);
					if (a.cap > 0.f) v.x = soft_cap<true>(v.x, a.cap, inv_cap), v.y = soft_cap<true>(v.y, a.cap, inv_cap);
					if (bh) v.x += __ldg(bh + min(max(dist, 0), a.n_bias - 1)), v.y += __ldg(bh + min(max(dist - 1, 0), a.n_bias - 1));
					*reinterpret_cast<float2 *>(Z + ((size_t)h * 16 + r) * LDZ + key) = v;
				}
		};
		if (H >= kMmWarps)
			for (int h = warp; h < H; h += kMmWarps) scores(h, 0, std::integral_constant<int, TK / 16>());
		else
			for (int u = warp; u < H * (TK / 16); u += kMmWarps) scores(u / (TK / 16), (u % (TK / 16)) * 16, std::integral_constant<int, 1>());
		__syncthreads();
		if (t + 1 < t_end) stage(Ks, kc, dk, LDK, t + 1);
		else asm volatile("cp.async.commit_group;" ::: "memory");
		// ---- mixing: 8 heads x 2 keys of one row per thread ----
		constexpr int PAIRS = 16 * TK / 2; // (row, 2 keys)
		const int mu = tid / PAIRS, mq = tid % PAIRS, mr = mq / (TK / 2), mk = (mq % (TK / 2)) * 2;
		const bool mixes = mu * 8 < HP;
		float acc[8][2];
		if (mixes) {
#pragma unroll
			for (int x = 0; x < 8; ++x) acc[x][0] = acc[x][1] = 0.f;
			const float *zp = Z + (size_t)mr * LDZ + mk, *mp = Ms + mu * 8;
#pragma unroll 4
			for (int g = 0; g < H; ++g) {
				const float2 v = *reinterpret_cast<const float2 *>(zp + (size_t)g * 16 * LDZ);
				const float4 wa = *reinterpret_cast<const float4 *>(mp + g * HP), wb = *reinterpret_cast<const float4 *>(mp + g * HP + 4);
				const float w[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
#pragma unroll
				for (int x = 0; x < 8; ++x) acc[x][0] = fmaf(w[x], v.x, acc[x][0]), acc[x][1] = fmaf(w[x], v.y, acc[x][1]);
			}
		}
		__syncthreads(); // every thread has its sums: the planes may be overwritten
		if (mixes) {
			const int i = p0 + min(i0 + mr, a.n - 1), lo = a.window > 0 ? max(0, i - a.window + 1) : 0, key = base + mk;
#pragma unroll
			for (int x = 0; x < 8; ++x) {
				if (mu * 8 + x >= nh) break;
				*reinterpret_cast<float2 *>(Z + ((size_t)(mu * 8 + x) * 16 + mr) * LDZ + mk) =
				    make_float2(key >= lo && key <= i ? acc[x][0] : -INFINITY, key + 1 >= lo && key + 1 <= i ? acc[x][1] : -INFINITY);
			}
		}
		asm volatile("cp.async.wait_group 1;" ::: "memory"); // the tile's values
		__syncthreads();
		// ---- online softmax of the head's rows, weighted sums ----
		if (sums) {
			float sa[TK / 8][2], sb[TK / 8][2], mxA = -INFINITY, mxB = -INFINITY;
			const float *za = Z + ((size_t)hl * 16 + (lane >> 2)) * LDZ + (lane & 3) * 2, *zb = za + 8 * LDZ;
#pragma unroll
			for (int x = 0; x < TK / 8; ++x) {
				const float2 va = *reinterpret_cast<const float2 *>(za + x * 8), vb = *reinterpret_cast<const float2 *>(zb + x * 8);
				sa[x][0] = va.x, sa[x][1] = va.y, sb[x][0] = vb.x, sb[x][1] = vb.y;
				mxA = fmaxf(mxA, fmaxf(va.x, va.y)), mxB = fmaxf(mxB, fmaxf(vb.x, vb.y));
			}
			mxA = fmaxf(mxA, __shfl_xor_sync(kFull, mxA, 1)), mxA = fmaxf(mxA, __shfl_xor_sync(kFull, mxA, 2));
			mxB = fmaxf(mxB, __shfl_xor_sync(kFull, mxB, 1)), mxB = fmaxf(mxB, __shfl_xor_sync(kFull, mxB, 2));
			const float nA = fmaxf(m0, mxA), nB = fmaxf(m1, mxB);
			const float eA = nA == -INFINITY ? 0.f : nA, eB = nB == -INFINITY ? 0.f : nB; // a row that has seen nothing yet stays empty
			const float cA = m0 == -INFINITY ? 0.f : __expf(m0 - eA), cB = m1 == -INFINITY ? 0.f : __expf(m1 - eB);
			m0 = nA, m1 = nB;
			l0 *= cA, l1 *= cB;
#pragma unroll
			for (int x = 0; x < OT; ++x) o[x][0] *= cA, o[x][1] *= cA, o[x][2] *= cB, o[x][3] *= cB;
			uint32_t pf[TK / 16][4];
#pragma unroll
			for (int x = 0; x < TK / 8; ++x) {
				const float p0v = __expf(sa[x][0] - eA), p1v = __expf(sa[x][1] - eA), p2v = __expf(sb[x][0] - eB), p3v = __expf(sb[x][1] - eB);
				l0 += p0v + p1v, l1 += p2v + p3v;
				pf[x >> 1][(x & 1) * 2] = mx_pack(p0v, p1v);
				pf[x >> 1][(x & 1) * 2 + 1] = mx_pack(p2v, p3v);
			}
#pragma unroll
			for (int kk = 0; kk < TK / 16; ++kk)
#pragma unroll
				for (int x = 0; x < OT; x += 2) {
					if (c_first + x * 8 < dv) {
						uint32_t B[4];
						mx_ldsm_x4_t(B, Vs + (size_t)(hg * TK + kk * 16 + ar) * LDV + c_first + x * 8 + ac);
						mx_mma(o[x], pf[kk], B[0], B[1]);
						mx_mma(o[x + 1], pf[kk], B[2], B[3]);
					}
				}
		}
		__syncthreads(); // values and mixed scores are read
		if (t + 1 < t_end) stage(Vs, vc, dv, LDV, t + 1);
	}
	asm volatile("cp.async.wait_group 0;" ::: "memory");
	if (!sums) return;
	l0 += __shfl_xor_sync(kFull, l0, 1), l0 += __shfl_xor_sync(kFull, l0, 2);
	l1 += __shfl_xor_sync(kFull, l1, 1), l1 += __shfl_xor_sync(kFull, l1, 2);
	const int h = h0 + hl;
#pragma unroll
	for (int half = 0; half < 2; ++half) {
		const int r = i0 + (lane >> 2) + half * 8;
		if (r >= a.n) continue;
		const float mm = half ? m1 : m0, ll = half ? l1 : l0;
		float *dst;
		float f = 1.f;
		if (a.part) dst = a.part + ((size_t)((size_t)r * H + h) * nsplit + sp) * (dv + 2);
		else {
			dst = a.out + (size_t)r * a.ldo + (size_t)h * dv;
			f = 1.f / ll;
			if (a.gate) f /= 1.f + expf(-a.gate[(size_t)r * a.ldg + h]);
		}
#pragma unroll
		for (int x = 0; x < OT; ++x) {
			const int c = c_first + x * 8 + (lane & 3) * 2;
			if (c < dv) dst[c] = o[x][half * 2] * f, dst[c + 1] = o[x][half * 2 + 1] * f;
		}
		if (a.part && c_first == 0 && (lane & 3) == 0) dst[dv] = mm, dst[dv + 1] = ll;
	}
}

} // namespace stack
} // namespace yalm

using namespace yalm;
using namespace yalm::stack;

static bool mixed_ok(const MixedArgs &a) {
	return a.out && a.q && a.kc && a.vc && a.n >= 1 && a.H >= 1 && a.G >= 1 && a.H % a.G == 0 && a.dk >= 1 && a.dv >= 1 && a.ring >= 1 && a.window >= 0 &&
	       (!a.bias || a.n_bias >= 1) && a.cap >= 0.f;
}
static int mixed_finish(const MixedArgs &a, int nsplit, cudaStream_t st) {
	if (int rc = (int)cudaGetLastError()) return rc;
	return nsplit > 1 ? yalm_attn_split_merge(a.out, a.ldo, a.part, a.n, a.H, a.dv, nsplit, nullptr, a.gate, a.ldg, st) : 0;
}
// how many CTAs share a row's (or row block's) keys: enough to fill the GPU, at most one per tile, and as the workspace allows
static int mixed_splits(const MixedArgs &a, int ctas, int tile, size_t ws_floats, int context) {
	const long most = a.window > 0 ? a.window : context > 0 ? context : a.ring;
	const long tiles = (most + tile - 1) / tile + 1, fit = (long)(ws_floats / ((size_t)a.n * a.H * (a.dv + 2)));
	return (int)std::max(1L, std::min({(long)device_info().sms / ctas, tiles, fit, 128L}));
}

// Floats of workspace the three routes below want for calls of at most `rows` rows (fewer: fewer splits; none: no splits).
extern "C" size_t yalm_attn_mixed_workspace(int rows, int heads, int dv) {
	return (size_t)std::max(16 * 160, std::min(rows, 16 * 160)) * heads * (dv + 2);
}

extern "C" int yalm_attn_mixed_rows(float *out, int ldo, const float *q, int ldq, const void *key_ring, const void *value_ring, const float *bias, int n_bias,
                                    const float *mix, const float *gate, int ldg, float *workspace, size_t workspace_floats, int n, int n_heads, int n_kv,
                                    int dk, int dv, int ring, int window, float scale, float softcap, int cache_f32, int context, int pos0, const int *ctl,
                                    yalm_stream_t s) {
	MixedArgs a{out, ldo, q, ldq, key_ring, value_ring, bias, n_bias, mix, gate, ldg, nullptr, n, n_heads, n_kv, dk, dv, ring, window, scale, softcap, pos0, ctl};
	if (!mixed_ok(a)) return YALM_EINVAL;
	const size_t smem = sizeof(float) * ((size_t)n_heads * (dk + dv + 2 * (kMixTile + 1)) + 3 * n_heads);
	if ((int)smem > device_info().max_smem_optin) return YALM_EINVAL;
	const int nsplit = workspace ? mixed_splits(a, n, kMixTile, workspace_floats, context) : 1;
	if (nsplit > 1) a.part = workspace;
	cudaStream_t st = (cudaStream_t)s;
	if (cache_f32) {
		if (smem > 48 * 1024) YALM_TRY(cudaFuncSetAttribute(attn_mixed_rows_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
		attn_mixed_rows_kernel<float><<<dim3(n, nsplit), kMixThreads, smem, st>>>(a);
	} else {
		if (smem > 48 * 1024) YALM_TRY(cudaFuncSetAttribute(attn_mixed_rows_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
		attn_mixed_rows_kernel<__nv_bfloat16><<<dim3(n, nsplit), kMixThreads, smem, st>>>(a);
	}
	return mixed_finish(a, nsplit, st);
}

// Key tile of the two tensor-core routes for these sizes (bf16 rings), 0: no kernel.
extern "C" int yalm_attn_mixed_decode_shape(int n_heads, int n_kv, int dk, int dv) {
	if (n_kv < 1 || n_heads % n_kv || n_heads / n_kv > 16 || dk < 16 || dk % 16 || dv < 16 || dv % 16 || n_kv * (dv / 16) > 16 * kMdWarps) return 0;
	for (int tk = 32; tk >= 16; tk /= 2)
		if ((int)mixed_decode_layout(n_heads, n_kv, dk, dv, tk).total <= device_info().max_smem_optin) return tk;
	return 0;
}
static int mixed_mma_heads(int n_heads) { return n_heads <= 4 ? 4 : n_heads <= 8 ? 8 : 16; }
extern "C" int yalm_attn_mixed_mma_shape(int n_heads, int n_kv, int dk, int dv) {
	if (n_kv < 1 || n_heads % n_kv || dk < 16 || dk % 16 || dv < 16 || dv % 16 || dv > 128 * (kMmWarps / mixed_mma_heads(n_heads))) return 0;
	for (int tk = 32; tk >= 16; tk /= 2)
		if ((int)mixed_mma_layout(n_heads, n_kv, dk, dv, tk, mixed_mma_heads(n_heads)).total <= device_info().max_smem_optin) return tk;
	return 0;
}

template <int TK, int NU>
static int launch_mixed_decode(const MixedArgs &a, int nsplit, cudaStream_t st) {
	const size_t smem = mixed_decode_layout(a.H, a.G, a.dk, a.dv, TK).total;
	if (smem > 48 * 1024) YALM_TRY(cudaFuncSetAttribute(attn_mixed_decode_kernel<TK, NU>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
	attn_mixed_decode_kernel<TK, NU><<<dim3(a.n, nsplit), kMdThreads, smem, st>>>(a);
	return mixed_finish(a, nsplit, st);
}

extern "C" int yalm_attn_mixed_decode(float *out, int ldo, const float *q, int ldq, const void *key_ring, const void *value_ring, const float *bias, int n_bias,
                                      const float *mix, const float *gate, int ldg, float *workspace, size_t workspace_floats, int n, int n_heads, int n_kv,
                                      int dk, int dv, int ring, int window, float scale, float softcap, int context, int pos0, const int *ctl, yalm_stream_t s) {
	MixedArgs a{out, ldo, q, ldq, key_ring, value_ring, bias, n_bias, mix, gate, ldg, nullptr, n, n_heads, n_kv, dk, dv, ring, window, scale, softcap, pos0, ctl};
	const int tk = yalm_attn_mixed_decode_shape(n_heads, n_kv, dk, dv);
	if (!mixed_ok(a) || !tk || !aligned16(key_ring) || !aligned16(value_ring) || !aligned16(q) || ldq % 4) return YALM_EINVAL;
	const int nsplit = workspace ? mixed_splits(a, n, tk, workspace_floats, context) : 1, units = (n_kv * (dv / 16) + kMdWarps - 1) / kMdWarps;
	if (nsplit > 1) a.part = workspace;
	cudaStream_t st = (cudaStream_t)s;
#define MD_CASE(TK_)                                                             \
	{                                                                            \
		if (units <= 2) return launch_mixed_decode<TK_, 2>(a, nsplit, st);       \
		if (units <= 4) return launch_mixed_decode<TK_, 4>(a, nsplit, st);       \
		if (units <= 8) return launch_mixed_decode<TK_, 8>(a, nsplit, st);       \
		return launch_mixed_decode<TK_, 16>(a, nsplit, st);                      \
	}
	if (tk == 32) MD_CASE(32)
	MD_CASE(16)
#undef MD_CASE
}

template <int TK, int DW>
static int launch_mixed_mma(const MixedArgs &a, int hs, int nsplit, cudaStream_t st) {
	const size_t smem = mixed_mma_layout(a.H, a.G, a.dk, a.dv, TK, hs).total;
	if (smem > 48 * 1024) YALM_TRY(cudaFuncSetAttribute(attn_mixed_mma_kernel<TK, DW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
	attn_mixed_mma_kernel<TK, DW><<<dim3((a.n + kMmRows - 1) / kMmRows, (a.H + hs - 1) / hs, nsplit), kMmThreads, smem, st>>>(a, hs);
	return mixed_finish(a, nsplit, st);
}

extern "C" int yalm_attn_mixed_mma(float *out, int ldo, const float *q, int ldq, const void *key_ring, const void *value_ring, const float *bias, int n_bias,
                                   const float *mix, const float *gate, int ldg, float *workspace, size_t workspace_floats, int n, int n_heads, int n_kv, int dk,
                                   int dv, int ring, int window, float scale, float softcap, int context, int pos0, const int *ctl, yalm_stream_t s) {
	MixedArgs a{out, ldo, q, ldq, key_ring, value_ring, bias, n_bias, mix, gate, ldg, nullptr, n, n_heads, n_kv, dk, dv, ring, window, scale, softcap, pos0, ctl};
	const int tk = yalm_attn_mixed_mma_shape(n_heads, n_kv, dk, dv);
	if (!mixed_ok(a) || !tk || !aligned16(key_ring) || !aligned16(value_ring) || !aligned16(q) || ldq % 4) return YALM_EINVAL;
	const int hs = mixed_mma_heads(n_heads), parts = kMmWarps / hs, ctas = (n + kMmRows - 1) / kMmRows * ((n_heads + hs - 1) / hs);
	// without a device-side position the keys of the last row are known
	const int seen = ctl ? context : pos0 + n;
	const int nsplit = workspace ? mixed_splits(a, ctas, tk, workspace_floats, seen) : 1;
	if (nsplit > 1) a.part = workspace;
	cudaStream_t st = (cudaStream_t)s;
	const int dw = (dv + parts - 1) / parts;
#define MM_CASE(TK_)                                                                 \
	{                                                                                \
		if (dw <= 16) return launch_mixed_mma<TK_, 16>(a, hs, nsplit, st);           \
		if (dw <= 32) return launch_mixed_mma<TK_, 32>(a, hs, nsplit, st);           \
		if (dw <= 64) return launch_mixed_mma<TK_, 64>(a, hs, nsplit, st);           \
		return launch_mixed_mma<TK_, 128>(a, hs, nsplit, st);                        \
	}
	if (tk == 32) MM_CASE(32)
	MM_CASE(16)
#undef MM_CASE
}
