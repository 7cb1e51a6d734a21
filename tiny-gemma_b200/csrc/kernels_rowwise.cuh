// Row-wise kernels over the tokens of one step: embedding, layer / RMS norm, norm with the input convolution (of which
// the token shift h + (h' - h) s is the two-tap case), rotation tables.
#pragma once
#include <cuda_bf16.h>

#include "tg_common.cuh"

namespace tg {

// The rows of a step. A segment is the run of consecutive tokens that one sequence brings; rows of a segment are
// consecutive. `par` selects which of a sequence's two history buffers holds what earlier steps left; a step writes
// the other one, so no row of the step can overwrite what another still has to read.
struct StepDesc {
	const int *tok;      // [R] token ids
	const int *row_seg;  // [R] segment of a row
	const int *seg_seq;  // [S] sequence slot
	const int *seg_row;  // [S] first row
	const int *seg_len;  // [S] rows
	const int *seg_pos;  // [S] position of the first row
	const int *seg_par;  // [S]
};

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float bf16_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t u) { return __uint_as_float(u & 0xFFFF0000u); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// x[r] = scale embed[tok[r]], or x[r] += that (another pass through a looped block)
static __global__ void __launch_bounds__(256) embed_rows_kernel(float *x, int ldx, const __nv_bfloat16 *embed, int lde, float scale, StepDesc d, int D, int V,
                                                                int add, int *err) {
	pdl_trigger();
	pdl_wait();
	const int r = blockIdx.x;
	int tok = d.tok[r];
	if (tok < 0 || tok >= V) {
		if (threadIdx.x == 0) *err = 1;
		tok = 0;
	}
	for (int i = threadIdx.x; i < D; i += 256) {
		const float e = scale * __bfloat162float(embed[size_t(tok) * lde + i]);
		float *p = x + size_t(r) * ldx + i;
		*p = add ? *p + e : e;
	}
}

// sum of v over a CTA of NW warps, in every thread
template <int NW> __device__ __forceinline__ float cta_sum(float v, float *red) {
	v = warp_sum(v);
	__syncthreads();
	if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
	__syncthreads();
	float t = 0.0f;
#pragma unroll
	for (int w = 0; w < NW; w++) t += red[w];
	return t;
}
template <typename T> __device__ __forceinline__ void store4(T *p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16 *p, float4 v) {
	__nv_bfloat162 q[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
	*reinterpret_cast<uint2 *>(p) = *reinterpret_cast<const uint2 *>(q);
}

// out[i] = norm(x[row(i)]) for i < n; row(i) = rows ? rows[i] : i; rms: no mean is taken off. Columns D .. ldo-1 become 0 (operand padding).
// One CTA of 128 threads per row, the row in registers while it fits (D <= 4096, D % 4 == 0; ldx, ldo multiples of 4).
template <typename OT>
__global__ void __launch_bounds__(128) row_norm_kernel(OT *out, int ldo, const float *x, int ldx, const float *w, const int *rows, int n, int D, float eps,
                                                       int rms, float *out32) {
	pdl_trigger();
	pdl_wait();
	__shared__ float red[4];
	const int i = blockIdx.x, tid = threadIdx.x;
	const float *xr = x + size_t(rows ? rows[i] : i) * ldx;
	OT *o = out + size_t(i) * ldo;
	if (D <= 4096 && D % 4 == 0) {
		float4 v[8];
		float s = 0.0f;
#pragma unroll
		for (int j = 0; j < 8; j++) {
			const int c = 4 * (tid + 128 * j);
			v[j] = c < D ? *reinterpret_cast<const float4 *>(xr + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
			s += (v[j].x + v[j].y) + (v[j].z + v[j].w);
		}
		const float mean = rms ? 0.0f : cta_sum<4>(s, red) / float(D);
		float q = 0.0f;
#pragma unroll
		for (int j = 0; j < 8; j++)
			if (4 * (tid + 128 * j) < D) {
				v[j].x -= mean; v[j].y -= mean; v[j].z -= mean; v[j].w -= mean;
				q = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, fmaf(v[j].w, v[j].w, q))));
			}
		const float f = 1.0f / sqrtf(cta_sum<4>(q, red) / float(D) + eps);
#pragma unroll
		for (int j = 0; j < 8; j++) {
			const int c = 4 * (tid + 128 * j);
			if (c < D) {
				const float4 g = *reinterpret_cast<const float4 *>(w + c);
				const float4 y = make_float4(v[j].x * f * g.x, v[j].y * f * g.y, v[j].z * f * g.z, v[j].w * f * g.w);
				store4<OT>(o + c, y);
				if (out32) *reinterpret_cast<float4 *>(out32 + size_t(i) * D + c) = y;
			} else if (c < ldo) {
				store4<OT>(o + c, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
			}
		}
		return;
	}
	float s = 0.0f, q = 0.0f;
	for (int c = tid; c < D; c += 128) s += xr[c];
	const float mean = rms ? 0.0f : cta_sum<4>(s, red) / float(D);
	for (int c = tid; c < D; c += 128) q = fmaf(xr[c] - mean, xr[c] - mean, q);
	const float f = 1.0f / sqrtf(cta_sum<4>(q, red) / float(D) + eps);
	for (int c = tid; c < ldo; c += 128) {
		const float y = c < D ? (xr[c] - mean) * f * w[c] : 0.0f;
		o[c] = from_f32<OT>(y);
		if (out32 && c < D) out32[size_t(i) * D + c] = y;
	}
}

// h = n + conv(n), n = norm(x): the causal convolution over time on each channel (taps at cw[j][D], the last one
// meets the current row). The taps - 1 normed rows before a segment come from hist[seq][par], and the segment's
// last ones (or, in a shorter segment, the older ones that still matter) are left in hist[seq][par ^ 1], oldest
// first. hist: [B][2][taps-1][D]. Rows before a sequence's start count as zero, whatever hist holds.
// Two kernels: mean (0 for an RMS norm) and 1/deviation of every row, then a walk down the rows with the window in registers, four
// channels per thread, LC_ROWS rows per CTA (the rows before them are normed again, not exchanged).
// The statistics kernel may first add what the preceding layer left to be added (`add`): the row is read here anyway.
template <typename YT> struct RowSum {
	const float *part;  // partial sums of a product whose K was shared, [n_part][rows][ldx]
	int n_part;
	size_t part_stride;
	const YT *y;        // [slots][ldy] outputs of the experts, or null
	int ldy, top;
	const int *slot;    // [R][top]
	const float *w;     // [R][top]
	int *zero;          // counters that the next layer's routing finds at zero, or null
	int n_zero;
};
__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16 *p) {
	const uint2 u = *reinterpret_cast<const uint2 *>(p);
	return make_float4(bf16_lo(u.x), bf16_hi(u.x), bf16_lo(u.y), bf16_hi(u.y));
}
template <typename YT>
__global__ void __launch_bounds__(128) row_stats_kernel(float2 *stats, float *x, int ldx, int D, float eps, int rms, RowSum<YT> add) {
	pdl_trigger();
	pdl_wait();
	__shared__ float red[4];
	const int tid = threadIdx.x;
	float *xr = x + size_t(blockIdx.x) * ldx;
	const int *slot = add.slot + size_t(blockIdx.x) * add.top;
	const float *wt = add.w + size_t(blockIdx.x) * add.top;
	if (add.zero && blockIdx.x == 0)
		for (int i = tid; i < add.n_zero; i += 128) add.zero[i] = 0;
	float mean, q = 0.0f, s = 0.0f;
	if (D <= 4096 && D % 4 == 0) {
		float4 v[8];
#pragma unroll
		for (int j = 0; j < 8; j++) {
			const int c = 4 * (tid + 128 * j);
			v[j] = c < D ? *reinterpret_cast<const float4 *>(xr + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
		}
		if (add.n_part) {
			const float *p = add.part + size_t(blockIdx.x) * ldx;
#pragma unroll
			for (int j = 0; j < 8; j++) {
				const int c = 4 * (tid + 128 * j);
				if (c < D) {
#pragma unroll 4
					for (int e = 0; e < add.n_part; e++) {
						const float4 u = *reinterpret_cast<const float4 *>(p + e * add.part_stride + c);
						v[j].x += u.x; v[j].y += u.y; v[j].z += u.z; v[j].w += u.w;
					}
				}
			}
		}
		if (add.y) {
			for (int e = 0; e < add.top; e++) {
				const YT *y = add.y + size_t(slot[e]) * add.ldy;
				const float w = wt[e];
#pragma unroll
				for (int j = 0; j < 8; j++) {
					const int c = 4 * (tid + 128 * j);
					if (c < D) {
						const float4 u = load4(y + c);
						v[j].x = fmaf(w, u.x, v[j].x); v[j].y = fmaf(w, u.y, v[j].y); v[j].z = fmaf(w, u.z, v[j].z); v[j].w = fmaf(w, u.w, v[j].w);
					}
				}
			}
		}
		if (add.y || add.n_part) {
#pragma unroll
			for (int j = 0; j < 8; j++)
				if (4 * (tid + 128 * j) < D) *reinterpret_cast<float4 *>(xr + 4 * (tid + 128 * j)) = v[j];
		}
#pragma unroll
		for (int j = 0; j < 8; j++) s += (v[j].x + v[j].y) + (v[j].z + v[j].w);
		mean = rms ? 0.0f : cta_sum<4>(s, red) / float(D);
#pragma unroll
		for (int j = 0; j < 8; j++)
			if (4 * (tid + 128 * j) < D) {
				v[j].x -= mean; v[j].y -= mean; v[j].z -= mean; v[j].w -= mean;
				q = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, fmaf(v[j].w, v[j].w, q))));
			}
	} else {
		for (int c = tid; c < D; c += 128) {
			float v = xr[c];
			for (int e = 0; e < add.n_part; e++) v += add.part[e * add.part_stride + size_t(blockIdx.x) * ldx + c];
			if (add.y)
				for (int e = 0; e < add.top; e++) v = fmaf(wt[e], to_f32(add.y[size_t(slot[e]) * add.ldy + c]), v);
			if (add.y || add.n_part) xr[c] = v;
			s += v;
		}
		mean = rms ? 0.0f : cta_sum<4>(s, red) / float(D);
		for (int c = tid; c < D; c += 128) q = fmaf(xr[c] - mean, xr[c] - mean, q);
	}
	q = cta_sum<4>(q, red);
	if (tid == 0) stats[blockIdx.x] = make_float2(mean, 1.0f / sqrtf(q / float(D) + eps));
}

// grid (ceil(R / rows), ceil(ldo / 512)); rows <= LC_ROWS; ldx and ldo multiples of 4. `plain`, if not null, gets n itself
// (for what reads the norm without the convolution), rows of ldo too.
constexpr int LC_ROWS = 16;
template <typename OT, int MT>
__global__ void __launch_bounds__(128) norm_conv_kernel(OT *out, OT *plain, int ldo, const float *x, int ldx, const float2 *stats, const float *w, const float *cw,
                                                      float *hist, StepDesc d, int R, int D, int taps, int rows) {
	pdl_trigger();
	pdl_wait();
	__shared__ float2 st[LC_ROWS + MT];
	__shared__ int seg_s[LC_ROWS];
	const int r0 = blockIdx.x * rows, nr = min(rows, R - r0), H = taps - 1, tid = threadIdx.x;
	if (tid < nr) seg_s[tid] = d.row_seg[r0 + tid];
	if (tid < nr + H && r0 - H + tid >= 0) st[tid] = stats[r0 - H + tid];
	__syncthreads();
	const int c = 4 * (blockIdx.y * 128 + tid);
	if (c >= ldo) return;
	if (c >= D) {
		for (int i = 0; i < nr; i++) {
			store4<OT>(out + size_t(r0 + i) * ldo + c, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
			if (plain) store4<OT>(plain + size_t(r0 + i) * ldo + c, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
		}
		return;
	}
	auto get = [&](const float *p) {  // four consecutive channels of an unpadded row
		return make_float4(p[0], c + 1 < D ? p[1] : 0.0f, c + 2 < D ? p[2] : 0.0f, c + 3 < D ? p[3] : 0.0f);
	};
	auto put = [&](float *p, const float4 &v) {
		p[0] = v.x;
		if (c + 1 < D) p[1] = v.y;
		if (c + 2 < D) p[2] = v.z;
		if (c + 3 < D) p[3] = v.w;
	};
	auto norm = [&](const float4 &v, const float2 &t, const float4 &g) {
		return make_float4((v.x - t.x) * t.y * g.x, (v.y - t.x) * t.y * g.y, (v.z - t.x) * t.y * g.z, (v.w - t.x) * t.y * g.w);
	};
	const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f), wc = get(w + c);
	float4 cf[MT], win[MT];  // win[MT-1] is the current row; taps are right-aligned
#pragma unroll
	for (int j = 0; j < MT; j++) cf[j] = j >= MT - taps ? get(cw + size_t(j - (MT - taps)) * D + c) : zero;
	int seg = -1, row0 = 0, len = 0;
	float *hw = nullptr;
	for (int i0 = 0; i0 < nr; i0 += 4) {
		float4 xv[4];
#pragma unroll
		for (int u = 0; u < 4; u++) xv[u] = i0 + u < nr ? *reinterpret_cast<const float4 *>(x + size_t(r0 + i0 + u) * ldx + c) : zero;
#pragma unroll
		for (int u = 0; u < 4; u++) {
			const int i = i0 + u, r = r0 + i;
			if (i >= nr) break;
			if (seg_s[i] != seg) {
				seg = seg_s[i];
				row0 = d.seg_row[seg];
				len = d.seg_len[seg];
				const int pos = d.seg_pos[seg];
				float *hb = hist + size_t(d.seg_seq[seg]) * 2 * H * D + c;
				const float *hr = hb + size_t(d.seg_par[seg]) * H * D;
				hw = hb + size_t(d.seg_par[seg] ^ 1) * H * D;
				const int t = r - row0;
#pragma unroll
				for (int j = 0; j < MT; j++) {  // slot j of the window before row t: time t - (MT - j)
					const int back = MT - j, tt = t - back;
					win[j] = zero;
					if (back <= H) {
						if (tt >= 0)
							win[j] = norm(*reinterpret_cast<const float4 *>(x + size_t(r - back) * ldx + c), st[i + H - back], wc);
						else if (pos + tt >= 0)
							win[j] = get(hr + size_t(H + tt) * D);
					}
				}
				if (t == 0)  // history rows that lie before this segment and stay relevant
					for (int q = 0; q < H; q++) {
						const int tt = len - H + q;
						if (tt < 0) put(hw + size_t(q) * D, pos + tt >= 0 ? get(hr + size_t(H + tt) * D) : zero);
					}
			}
			const float4 nv = norm(xv[u], st[i + H], wc);
			float4 y = nv;
#pragma unroll
			for (int j = 0; j < MT; j++) {
				win[j] = j + 1 < MT ? win[j + 1] : nv;
				y.x = fmaf(cf[j].x, win[j].x, y.x); y.y = fmaf(cf[j].y, win[j].y, y.y);
				y.z = fmaf(cf[j].z, win[j].z, y.z); y.w = fmaf(cf[j].w, win[j].w, y.w);
			}
			if (c + 1 >= D) y.y = 0.0f;
			if (c + 2 >= D) y.z = 0.0f;
			if (c + 3 >= D) y.w = 0.0f;
			store4<OT>(out + size_t(r) * ldo + c, y);
			if (plain) store4<OT>(plain + size_t(r) * ldo + c, make_float4(nv.x, c + 1 < D ? nv.y : 0.0f, c + 2 < D ? nv.z : 0.0f, c + 3 < D ? nv.w : 0.0f));
			const int q = (r - row0) - (len - H);
			if (q >= 0) put(hw + size_t(q) * D, nv);
		}
	}
}

// ------------------------------------------------------------------ rotation
// cs[rot][row][i] = (cos, sin) of position x frequency i, times the rotation's factor. The angle is formed and reduced
// in double, so it is exact to fp32 rounding at any position. grid (R, rotations)
struct RopeTable {
	const double *freq;   // [rotations][half]
	const float *factor;  // [rotations]
	float2 *cs;           // [rotations][rows][half]
	int rows, half;
};
static __global__ void __launch_bounds__(128) rope_table_kernel(RopeTable t, StepDesc d) {
	pdl_trigger();
	pdl_wait();
	const int r = blockIdx.x, rot = blockIdx.y, seg = d.row_seg[r];
	const double p = double(d.seg_pos[seg] + r - d.seg_row[seg]);
	const float m = t.factor[rot];
	for (int i = threadIdx.x; i < t.half; i += 128) {
		double a = p * t.freq[size_t(rot) * t.half + i];
		a -= 6.283185307179586 * rint(a * 0.15915494309189535);
		float s, c;
		sincosf(float(a), &s, &c);
		t.cs[(size_t(rot) * t.rows + r) * t.half + i] = make_float2(c * m, s * m);
	}
}

}  // namespace tg
