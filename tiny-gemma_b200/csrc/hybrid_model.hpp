// The layered decoders that are read from a model folder: what config.json says, and the packed bf16 weights. Every size
// and constant comes from config.json or from a tensor's shape. Two designs are described in the same terms:
//
//   "Nabelix"   x <- x + mixer(conv(norm1(x)));  x <- x + ff(norm2(x)).  Layer norms, a causal input convolution, and in
//               every layer windowed attention with kept first tokens beside a gated delta rule. A block of layers may run
//               several times (a loop). Tied, soft-capped output.
//   "Sominex"   x <- x + mixer(shift(h)) + ff(h), h = norm1(x).  RMS norms, a token shift before the mixer; every layer has
//               one mixer: windowed attention over tokens and pooled blocks with rotated keys, a state-space recurrence
//               (Mamba-2), or a matrix memory with exponential gates (mLSTM); the feed-forward is a clamped gated one or a
//               mixture of experts. Output matrix of its own.
#pragma once
#include <cuda_bf16.h>

#include <algorithm>
#include <cmath>
#include <cstring>
#include <limits>
#include <map>
#include <memory>

#include "kernels_delta.cuh"
#include "kernels_moe.cuh"
#include "kernels_recurrent.cuh"
#include "model_dir.hpp"
#include "tg_internal.hpp"

namespace tg {

typedef __nv_bfloat16 bf16;

inline int round_up(int x, int m) { return (x + m - 1) / m * m; }

// A linear layer: weights [N][ld] bf16 with K used columns (padded with zeros to a multiple of 8).
struct Lin {
	const bf16 *W = nullptr;
	int N = 0, K = 0, ld = 0;
	CUtensorMap map[3];  // boxes of 64, 128 and 256 rows
};

inline int make_map(CUtensorMap *out, const void *base, size_t rows, int cols, int ld, int box_rows) {
	PFN_encodeTiled enc = get_encode_fn();
	if (!enc) return fail(TG_ECUDA, "cuTensorMapEncodeTiled is not available");
	cuuint64_t dims[2] = {cuuint64_t(cols), cuuint64_t(rows)};
	cuuint64_t strides[1] = {cuuint64_t(ld) * 2};
	cuuint32_t box[2] = {64, cuuint32_t(box_rows)}, es[2] = {1, 1};
	CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
	                 CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
	if (r != CUDA_SUCCESS) return fail(TG_ECUDA, "cuTensorMapEncodeTiled failed (" + std::to_string(int(r)) + ")");
	return TG_OK;
}

// ------------------------------------------------------------------ a layer
struct AttnSpec {  // H = 0: no attention
	int H = 0, G = 0, dk = 0, dv = 0, dkp = 0, dvp = 0;
	float scale = 0.0f;
	int window = 0, keep = 0, pool = 0;
	int rot = -1, rot_dims = 0;  // which of the model's rotations
	bool vnorm = false, gated = false;
};
struct DeltaSpec {  // H = 0: no delta rule
	int H = 0, KH = 0, dk = 0, dv = 0, taps = 0, ra = 0, rg = 0;
	int channels() const { return 2 * KH * dk + H * dv; }
	int dkp() const { return dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 128 ? 128 : 256)); }
};
struct LinSpec {  // a recurrence of kernels_recurrent.cuh
	int kind = LIN_NONE, H = 0, G = 0, N = 0, vd = 0, Np = 0, vdp = 0, taps = 1, parts = 1;
	float gate_cap = 1.0f;
	int channels() const { return H * vd + 2 * G * N; }
	int xc_cols() const { return round_up(H * vdp + 2 * G * Np, 8); }
};
struct FfSpec {
	int ff = 0, ffp = 0;  // the dense feed-forward or the shared expert; 0: none
	int act = GLU_GELU;
	float limit = 0.0f;
	int experts = 0, top = 0, eff = 0, effp = 0;  // experts = 0: no mixture
	float route_scale = 1.0f;
	bool any() const { return ff > 0 || experts > 0; }
};
struct Layer {
	AttnSpec at;
	DeltaSpec de;
	LinSpec li;
	FfSpec ff;
	bool beside = false;  // the feed-forward reads norm1 and is added together with the mixer
	float left_scale = 1.0f, right_scale = 1.0f;
	// columns of a projection row; from n32 on they are kept in fp32, in a buffer of their own
	int p_q = 0, p_k = 0, p_v = 0, p_g = -1, p_a1 = 0, p_g1 = 0, p_conv = 0, p_b = 0, p_z = 0, ldp = 0, n32 = 0;
	int o_col = 0, kc = 0;  // columns of a mixed row: attention heads at 0, delta heads at o_col; kc in all
	int kcat = 0;           // kc, and the feed-forward's activations beside them
	float *norm1 = nullptr, *norm2 = nullptr, *canon = nullptr, *r1 = nullptr, *r2 = nullptr, *conv = nullptr, *A_log = nullptr, *dt_bias = nullptr, *rnorm = nullptr;
	float *conv_b = nullptr, *Dv = nullptr, *ib = nullptr, *fb = nullptr;
	// `beside`: front is [proj][gu] one after the other; out is [output projection | down] side by side
	Lin front, proj, a2, g2, out, gu, down, ex_gu, ex_down;
	int tail() const { return proj.N - n32; }
};
struct Run {
	int layer;
	bool add_embed;  // another pass through the loop begins here
};
struct Rotation {
	int dims = 0;
	double base = 0.0, factor = 0.0, fast = 0.0, slow = 0.0, original = 0.0;  // factor = 0: no scaling
	bool operator==(const Rotation &o) const {
		return dims == o.dims && base == o.base && factor == o.factor && fast == o.fast && slow == o.slow && original == o.original;
	}
	// frequencies of the pairs; returns the factor on cos and sin
	float frequencies(double *f) const {
		const double pi = 3.14159265358979323846;
		auto at = [&](double turns) { return dims * std::log(original / (2.0 * pi * turns)) / (2.0 * std::log(base)); };
		const double lo = factor > 0.0 ? std::max(std::floor(at(fast)), 0.0) : 0.0, hi = factor > 0.0 ? std::min(std::ceil(at(slow)), double(dims - 1)) : 0.0;
		for (int i = 0; i < dims / 2; i++) {
			f[i] = std::pow(base, -2.0 * i / dims);
			if (factor > 0.0) {
				const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
				f[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp);
			}
		}
		return factor > 0.0 ? float(0.1 * std::log(factor) + 1.0) : 1.0f;
	}
};

}  // namespace tg

struct HybridModel : tg_model {
	std::string architecture;
	int dtype = TG_BF16;
	int D = 0, Dp = 0, taps = 1;  // taps of the input convolution (2: token shift)
	bool has_canon = false, rms = false;
	float eps = 1e-6f, softcap = 0.0f, embed_scale = 1.0f;
	std::vector<tg::Layer> layers;
	std::vector<tg::Run> runs;
	std::vector<tg::Rotation> rots;
	int rot_half = 0;             // most pairs of a rotation, an even number
	double *rot_freq = nullptr;   // [rotations][rot_half]
	float *rot_factor = nullptr;  // [rotations]
	tg::Lin embed, head;          // head: the output matrix (the embedding's, if tied)
	float *final_norm = nullptr;
	std::vector<void *> mem;

	~HybridModel() override {
		for (void *p : mem) cudaFree(p);
	}
	const char *arch() const override { return architecture.c_str(); }
	int new_state(int batch, int max_pos, tg_state **out) override;
};

namespace tg {

// ------------------------------------------------------------------ loading
struct Loader {
	HybridModel *m;
	SafeTensors st;

	int get(const std::string &name, std::vector<long long> shape, const SafeTensors::Tensor **out) {
		auto it = st.tensors.find(name);
		if (it == st.tensors.end()) return fail(TG_EIO, "model.safetensors has no tensor " + name);
		const auto &t = it->second;
		if (t.dtype != "BF16" && t.dtype != "F32") return fail(TG_EINVAL, name + ": dtype " + t.dtype + " is not supported");
		bool ok = t.shape.size() == shape.size();
		for (size_t i = 0; ok && i < shape.size(); i++) ok = shape[i] < 0 || t.shape[i] == shape[i];
		if (!ok) {
			std::string got, want;
			for (long long d : t.shape) got += (got.empty() ? "" : ", ") + std::to_string(d);
			for (long long d : shape) want += (want.empty() ? "" : ", ") + (d < 0 ? std::string("*") : std::to_string(d));
			return fail(TG_ESHAPE, name + ": shape [" + got + "], expected [" + want + "]");
		}
		*out = &t;
		return TG_OK;
	}
	int upload(const void *host, size_t bytes, void **dev) {
		if (cudaMalloc(dev, std::max<size_t>(bytes, 16)) != cudaSuccess) {
			cudaGetLastError();
			return fail(TG_ENOMEM, "cudaMalloc(weights)");
		}
		m->mem.push_back(*dev);
		TG_CUDA(cudaMemcpy(*dev, host, bytes, cudaMemcpyHostToDevice));
		return TG_OK;
	}
	int vec(const std::string &name, int n, float **dev) {
		const SafeTensors::Tensor *t;
		TG_TRY(get(name, {n}, &t));
		std::vector<float> h(n);
		for (int i = 0; i < n; i++) h[i] = t->at(i);
		return upload(h.data(), size_t(n) * 4, reinterpret_cast<void **>(dev));
	}
	// a matrix under construction on the host
	struct Host {
		int rows, ld;
		std::vector<uint16_t> v;
		Host(int r, int l) : rows(r), ld(l), v(size_t(r) * l, 0) {}
	};
	static uint16_t to16(const SafeTensors::Tensor &t, size_t i) {
		if (t.dtype == "BF16") {
			uint16_t h;
			std::memcpy(&h, t.data + 2 * i, 2);
			return h;
		}
		uint32_t b;
		std::memcpy(&b, t.data + 4 * i, 4);
		return uint16_t((b + 0x7FFF + ((b >> 16) & 1)) >> 16);
	}
	// rows [r0, r0 + n) and columns [c0, c0 + k) of t -> dst rows d0.., columns e0..
	static void put(Host &h, int d0, int e0, const SafeTensors::Tensor &t, size_t r0, int n, size_t c0, int k) {
		const size_t cols = size_t(t.shape[1]);
		for (int i = 0; i < n; i++) {
			uint16_t *dst = h.v.data() + size_t(d0 + i) * h.ld + e0;
			const size_t src = (r0 + i) * cols + c0;
			if (t.dtype == "BF16") std::memcpy(dst, t.data + 2 * src, 2 * size_t(k));
			else
				for (int j = 0; j < k; j++) dst[j] = to16(t, src + j);
		}
	}
	int linear(const Host &h, Lin *l) {
		l->N = h.rows;
		l->K = l->ld = h.ld;
		TG_TRY(upload(h.v.data(), h.v.size() * 2, reinterpret_cast<void **>(const_cast<bf16 **>(&l->W))));
		for (int i = 0; i < 3; i++) TG_TRY(make_map(&l->map[i], l->W, l->N, l->K, l->ld, 64 << i));
		return TG_OK;
	}
	// a linear layer that is a run of another one's rows
	int rows_of(const Lin &all, int row0, int n, Lin *l) {
		l->W = all.W + size_t(row0) * all.ld;
		l->N = n;
		l->K = l->ld = all.ld;
		for (int i = 0; i < 3; i++) TG_TRY(make_map(&l->map[i], l->W, l->N, l->K, l->ld, 64 << i));
		return TG_OK;
	}
	// [taps][channels] fp32 from [channels, taps] tensors laid one after the other
	int conv(const std::vector<std::pair<std::string, int>> &parts, int taps, float **dev) {
		int n = 0, c0 = 0;
		for (const auto &p : parts) n += p.second;
		std::vector<float> h(size_t(taps) * n);
		for (const auto &p : parts) {
			const SafeTensors::Tensor *t;
			TG_TRY(get(p.first, {p.second, taps}, &t));
			for (int c = 0; c < p.second; c++)
				for (int j = 0; j < taps; j++) h[size_t(j) * n + c0 + c] = t->at(size_t(c) * taps + j);
			c0 += p.second;
		}
		return upload(h.data(), h.size() * 4, reinterpret_cast<void **>(dev));
	}
	// ---- Nabelix
	int nabelix_layer(int i) {
		Layer &L = m->layers[i];
		const int D = m->D, Dp = m->Dp;
		const std::string p = "l" + std::to_string(i) + ".", lp = p + "mix.left.", rp = p + "mix.right.";
		const AttnSpec &A = L.at;
		DeltaSpec &E = L.de;
		TG_TRY(vec(p + "norm1", D, &L.norm1));
		if (m->has_canon) {
			TG_TRY(conv({{p + "canon1", D}}, m->taps, &L.canon));
		} else {
			const std::vector<float> none(D, 0.0f);
			TG_TRY(upload(none.data(), size_t(D) * 4, reinterpret_cast<void **>(&L.canon)));
		}
		const SafeTensors::Tensor *q, *k, *v, *g, *o, *rq, *rk, *rv, *b, *a1, *a2, *g1, *g2, *ro;
		TG_TRY(get(lp + "q", {A.H * A.dk, D}, &q));
		TG_TRY(get(lp + "k", {A.G * A.dk, D}, &k));
		TG_TRY(get(lp + "v", {A.G * A.dv, D}, &v));
		TG_TRY(get(lp + "g", {A.H * A.dv, D}, &g));
		TG_TRY(get(lp + "o", {D, A.H * A.dv}, &o));
		TG_TRY(vec(lp + "r1", A.H, &L.r1));
		TG_TRY(vec(lp + "r2", A.H, &L.r2));
		TG_TRY(get(rp + "q", {E.KH * E.dk, D}, &rq));
		TG_TRY(get(rp + "k", {E.KH * E.dk, D}, &rk));
		TG_TRY(get(rp + "v", {E.H * E.dv, D}, &rv));
		TG_TRY(get(rp + "b", {E.H, D}, &b));
		TG_TRY(get(rp + "a1", {-1, D}, &a1));
		TG_TRY(get(rp + "g1", {-1, D}, &g1));
		const int ra = int(a1->shape[0]), rg = int(g1->shape[0]);
		TG_TRY(get(rp + "a2", {E.H * E.dk, ra}, &a2));
		TG_TRY(get(rp + "g2", {E.H * E.dv, rg}, &g2));
		TG_TRY(get(rp + "o", {D, E.H * E.dv}, &ro));
		TG_TRY(vec(rp + "A_log", E.H, &L.A_log));
		TG_TRY(vec(rp + "dt_bias", E.H * E.dk, &L.dt_bias));
		TG_TRY(vec(rp + "norm", E.dv, &L.rnorm));
		TG_TRY(conv({{rp + "q.conv", E.KH * E.dk}, {rp + "k.conv", E.KH * E.dk}, {rp + "v.conv", E.H * E.dv}}, E.taps, &L.conv));
		E.ra = round_up(ra, 8);
		E.rg = round_up(rg, 8);
		// the projections, one matrix: heads of the attention padded to multiples of 16 columns
		int n = 0;
		auto place = [&](int w) {
			const int at = n;
			n += w;
			return at;
		};
		L.p_q = place(A.H * A.dkp);
		L.p_k = place(A.G * A.dkp);
		L.p_v = place(A.G * A.dvp);
		L.p_g = place(A.H * A.dvp);
		L.p_a1 = place(E.ra);
		L.p_g1 = place(E.rg);
		L.p_conv = place(E.channels());
		L.p_b = place(E.H);
		L.n32 = L.ldp = round_up(n, 8);
		{
			Host h(L.ldp, Dp);
			for (int x = 0; x < A.H; x++) put(h, L.p_q + x * A.dkp, 0, *q, size_t(x) * A.dk, A.dk, 0, D);
			for (int x = 0; x < A.G; x++) put(h, L.p_k + x * A.dkp, 0, *k, size_t(x) * A.dk, A.dk, 0, D);
			for (int x = 0; x < A.G; x++) put(h, L.p_v + x * A.dvp, 0, *v, size_t(x) * A.dv, A.dv, 0, D);
			for (int x = 0; x < A.H; x++) put(h, L.p_g + x * A.dvp, 0, *g, size_t(x) * A.dv, A.dv, 0, D);
			put(h, L.p_a1, 0, *a1, 0, ra, 0, D);
			put(h, L.p_g1, 0, *g1, 0, rg, 0, D);
			put(h, L.p_conv, 0, *rq, 0, E.KH * E.dk, 0, D);
			put(h, L.p_conv + E.KH * E.dk, 0, *rk, 0, E.KH * E.dk, 0, D);
			put(h, L.p_conv + 2 * E.KH * E.dk, 0, *rv, 0, E.H * E.dv, 0, D);
			put(h, L.p_b, 0, *b, 0, E.H, 0, D);
			TG_TRY(linear(h, &L.proj));
		}
		{
			Host h(E.H * E.dk, E.ra);
			put(h, 0, 0, *a2, 0, E.H * E.dk, 0, ra);
			TG_TRY(linear(h, &L.a2));
		}
		{
			Host h(E.H * E.dv, E.rg);
			put(h, 0, 0, *g2, 0, E.H * E.dv, 0, rg);
			TG_TRY(linear(h, &L.g2));
		}
		// both output projections side by side
		L.o_col = A.H * A.dvp;
		L.kcat = L.kc = round_up(L.o_col + E.H * E.dv, 8);
		{
			Host h(D, L.kc);
			for (int x = 0; x < A.H; x++) put(h, 0, x * A.dvp, *o, 0, D, size_t(x) * A.dv, A.dv);
			put(h, 0, L.o_col, *ro, 0, D, 0, E.H * E.dv);
			TG_TRY(linear(h, &L.out));
		}
		if (L.ff.ff) {
			const SafeTensors::Tensor *ga, *up, *dn;
			TG_TRY(vec(p + "norm2", D, &L.norm2));
			TG_TRY(get(p + "mlp.gate", {L.ff.ff, D}, &ga));
			TG_TRY(get(p + "mlp.up", {L.ff.ff, D}, &up));
			TG_TRY(get(p + "mlp.down", {D, L.ff.ff}, &dn));
			{
				Host h(2 * L.ff.ffp, Dp);  // blocks of 16 gate rows, 16 up rows
				for (int x = 0; x < L.ff.ff; x += 16) {
					const int c = std::min(16, L.ff.ff - x);
					put(h, 2 * x, 0, *ga, x, c, 0, D);
					put(h, 2 * x + 16, 0, *up, x, c, 0, D);
				}
				TG_TRY(linear(h, &L.gu));
			}
			Host h(D, L.ff.ffp);
			put(h, 0, 0, *dn, 0, D, 0, L.ff.ff);
			TG_TRY(linear(h, &L.down));
		}
		return TG_OK;
	}

	// ---- Sominex: the rows of the mixer's projections, then those of the feed-forward, go into `front`
	struct Place {  // rows [r0, r0 + n) of a tensor -> rows at ..
		int at;
		const SafeTensors::Tensor *t;
		size_t r0;
		int n;
	};
	int sominex_layer(int i) {
		Layer &L = m->layers[i];
		const int D = m->D, Dp = m->Dp;
		const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.", fp = p + "mlp.";
		TG_TRY(vec(p + "norm1", D, &L.norm1));
		{  // h + (h' - h) s as a convolution beside h: taps s, -s
			const SafeTensors::Tensor *t;
			TG_TRY(get(p + "shift", {D}, &t));
			std::vector<float> h(size_t(2) * D);
			for (int c = 0; c < D; c++) {
				h[c] = t->at(c);
				h[D + c] = -h[c];
			}
			TG_TRY(upload(h.data(), h.size() * 4, reinterpret_cast<void **>(&L.canon)));
		}
		std::vector<Place> rows;
		int n = 0;
		auto heads = [&](const SafeTensors::Tensor *t, size_t r0, int count, int size, int padded) {
			const int at = n;
			for (int x = 0; x < count; x++) rows.push_back({at + x * padded, t, r0 + size_t(x) * size, size});
			n += count * padded;
			return at;
		};
		// the output projection: `count` heads of `size` columns, padded
		const SafeTensors::Tensor *o;
		int o_heads, o_size, o_pad;
		if (L.at.H) {
			const AttnSpec &A = L.at;
			const SafeTensors::Tensor *q, *k, *v;
			TG_TRY(get(mp + "q", {A.H * A.dk, D}, &q));
			TG_TRY(get(mp + "k", {A.G * A.dk, D}, &k));
			TG_TRY(get(mp + "v", {A.G * A.dv, D}, &v));
			TG_TRY(get(mp + "o", {D, A.H * A.dv}, &o));
			L.p_q = heads(q, 0, A.H, A.dk, A.dkp);
			L.p_k = heads(k, 0, A.G, A.dk, A.dkp);
			L.p_v = heads(v, 0, A.G, A.dv, A.dvp);
			L.n32 = n;
			o_heads = A.H;
			o_size = A.dv;
			o_pad = A.dvp;
		} else {
			const LinSpec &R = L.li;
			const int inner = R.H * R.vd;
			TG_TRY(vec(mp + "norm", inner, &L.rnorm));
			TG_TRY(get(mp + "o", {D, inner}, &o));
			o_heads = 1;
			o_size = o_pad = inner;
			if (R.kind == LIN_SSM) {
				const SafeTensors::Tensor *in;
				TG_TRY(get(mp + "in", {inner + R.channels() + R.H, D}, &in));
				L.p_z = heads(in, 0, 1, inner, inner);
				L.p_conv = heads(in, inner, 1, R.channels(), R.channels());
				L.n32 = n = round_up(n, 8);
				heads(in, inner + R.channels(), 1, R.H, R.H);
				TG_TRY(conv({{mp + "conv", R.channels()}}, R.taps, &L.conv));
				TG_TRY(vec(mp + "conv.b", R.channels(), &L.conv_b));
				TG_TRY(vec(mp + "dt_bias", R.H, &L.dt_bias));
				TG_TRY(vec(mp + "A_log", R.H, &L.A_log));
				TG_TRY(vec(mp + "D", R.H, &L.Dv));
			} else {
				const SafeTensors::Tensor *q, *k, *v, *g, *gi, *gf;
				TG_TRY(get(mp + "q", {R.H * R.N, D}, &q));
				TG_TRY(get(mp + "k", {R.H * R.N, D}, &k));
				TG_TRY(get(mp + "v", {inner, D}, &v));
				TG_TRY(get(mp + "g", {inner, D}, &g));
				TG_TRY(get(mp + "i", {R.H, D}, &gi));
				TG_TRY(get(mp + "f", {R.H, D}, &gf));
				L.p_q = heads(q, 0, R.H, R.N, R.Np);
				L.p_k = heads(k, 0, R.H, R.N, R.Np);
				L.p_v = heads(v, 0, R.H, R.vd, R.vdp);
				L.p_z = heads(g, 0, 1, inner, inner);
				L.n32 = n = round_up(n, 8);
				heads(gi, 0, 1, R.H, R.H);
				heads(gf, 0, 1, R.H, R.H);
				TG_TRY(vec(mp + "i.b", R.H, &L.ib));
				TG_TRY(vec(mp + "f.b", R.H, &L.fb));
			}
		}
		L.ldp = L.n32;
		const int n_proj = n = round_up(n, 8);
		const FfSpec &F = L.ff;
		const SafeTensors::Tensor *down = nullptr;
		if (F.ff) {
			const std::string q = F.experts ? fp + "shared." : fp;
			const SafeTensors::Tensor *ga, *up;
			TG_TRY(get(q + "gate", {F.ff, D}, &ga));
			TG_TRY(get(q + "up", {F.ff, D}, &up));
			TG_TRY(get(q + "down", {D, F.ff}, &down));
			for (int x = 0; x < F.ff; x += 16) {  // blocks of 16 gate rows, 16 up rows
				const int c = std::min(16, F.ff - x);
				rows.push_back({n + 2 * x, ga, size_t(x), c});
				rows.push_back({n + 2 * x + 16, up, size_t(x), c});
			}
			n += 2 * F.ffp;
		}
		if (F.experts) {
			const SafeTensors::Tensor *r;
			TG_TRY(get(fp + "router", {F.experts, D}, &r));
			heads(r, 0, 1, F.experts, round_up(F.experts, 8));
		}
		{
			Host h(n, Dp);
			for (const Place &w : rows) put(h, w.at, 0, *w.t, w.r0, w.n, 0, D);
			TG_TRY(linear(h, &L.front));
			TG_TRY(rows_of(L.front, 0, n_proj, &L.proj));
			if (n > n_proj) TG_TRY(rows_of(L.front, n_proj, n - n_proj, &L.gu));
		}
		L.kc = round_up(o_heads * o_pad, 8);
		L.kcat = L.kc + F.ffp;
		{
			Host h(D, L.kcat);
			for (int x = 0; x < o_heads; x++) put(h, 0, x * o_pad, *o, 0, D, size_t(x) * o_size, o_size);
			if (F.ff) put(h, 0, L.kc, *down, 0, D, 0, F.ff);
			TG_TRY(linear(h, &L.out));
		}
		if (F.experts) {
			Host gu(F.experts * 2 * F.effp, Dp), dn(F.experts * D, F.effp);
			for (int e = 0; e < F.experts; e++) {
				const std::string q = fp + "e" + std::to_string(e) + ".";
				const SafeTensors::Tensor *ga, *up, *d;
				TG_TRY(get(q + "gate", {F.eff, D}, &ga));
				TG_TRY(get(q + "up", {F.eff, D}, &up));
				TG_TRY(get(q + "down", {D, F.eff}, &d));
				for (int x = 0; x < F.eff; x += 16) {
					const int c = std::min(16, F.eff - x), at = e * 2 * F.effp + 2 * x;
					put(gu, at, 0, *ga, x, c, 0, D);
					put(gu, at + 16, 0, *up, x, c, 0, D);
				}
				put(dn, e * D, 0, *d, 0, D, 0, F.eff);
			}
			TG_TRY(linear(gu, &L.ex_gu));
			TG_TRY(linear(dn, &L.ex_down));
			L.ex_gu.N = 2 * F.effp;  // rows of one expert (the maps cover all of them)
			L.ex_down.N = D;
		}
		return TG_OK;
	}
};

// ------------------------------------------------------------------ config.json
struct ConfigReader {
	std::string err;
	double num(const json::Value *o, const char *key, const char *where, bool need = true, double dflt = 0.0) {
		const json::Value *v = o ? o->find(key) : nullptr;
		if (v && v->kind == json::Value::NUMBER) return v->num;
		if ((need || v) && err.empty()) err = std::string("config.json: ") + where + "." + key + " is not a number";
		return dflt;
	}
	int size(const json::Value *o, const char *key, const char *where, int lo = 1) {
		const double d = num(o, key, where);
		if (err.empty() && (d < lo || d > 1e9 || d != std::floor(d))) err = std::string("config.json: ") + where + "." + key + " is out of range";
		return err.empty() ? int(d) : lo;
	}
	const json::Value *obj(const json::Value *o, const char *key, const char *where) {
		const json::Value *v = o ? o->find(key) : nullptr;
		if ((!v || v->kind != json::Value::OBJECT) && err.empty()) err = std::string("config.json: ") + where + "." + key + " is missing";
		return v;
	}
};

// what both designs have
inline void read_model(ConfigReader &r, const json::Value &c, HybridModel *m) {
	m->D = r.size(&c, "width", "model");
	m->hidden_size = m->D;
	m->Dp = round_up(m->D, 8);
	m->n_vocab = r.size(&c, "vocab", "model");
	m->n_pos = 1 << 24;  // distances stay exact in fp32
	m->eps = float(r.num(r.obj(&c, "norm", "model"), "eps", "norm"));
}
inline int layer_list(const json::Value &c, const json::Value **ls) {
	*ls = c.find("layers");
	if (!*ls || (*ls)->kind != json::Value::ARRAY || (*ls)->items.empty()) return fail(TG_EINVAL, "config.json: no layers");
	return TG_OK;
}
inline std::string type_of(const json::Value *v) { return v ? " " + v->str : std::string(); }

inline int read_nabelix(const json::Value &c, HybridModel *m) {
	ConfigReader r;
	read_model(r, c, m);
	m->softcap = float(r.num(&c, "logit_softcap", "model", false, 0.0));
	if (const json::Value *cn = c.find("canon")) {
		m->has_canon = true;
		m->taps = r.size(cn, "taps", "canon");
	}
	const json::Value *ls;
	TG_TRY(layer_list(c, &ls));
	for (const auto &l : ls->items) {
		Layer L;
		const json::Value *ty = l.find("type");
		if (!ty || ty->str != "parallel") return fail(TG_EINVAL, "config.json: unknown layer type" + type_of(ty));
		const json::Value *mx = r.obj(&l, "mixer", "layer"), *a = r.obj(mx, "left", "mixer"), *d = r.obj(mx, "right", "mixer");
		L.left_scale = float(r.num(mx, "left_scale", "mixer"));
		L.right_scale = float(r.num(mx, "right_scale", "mixer"));
		L.at.H = r.size(a, "heads", "left");
		L.at.G = r.size(a, "kv_heads", "left");
		L.at.dk = r.size(a, "dim", "left");
		L.at.dv = r.size(a, "vdim", "left");
		L.at.scale = float(r.num(a, "scale", "left"));
		const json::Value *mk = r.obj(a, "mask", "left");
		L.at.window = r.size(mk, "size", "mask");
		if (mk && mk->find("keep_first")) L.at.keep = r.size(mk, "keep_first", "mask", 0);
		L.at.dkp = round_up(L.at.dk, 16);
		L.at.dvp = round_up(L.at.dv, 16);
		L.at.gated = true;
		L.de.H = r.size(d, "heads", "right");
		L.de.KH = r.size(d, "kv_heads", "right");
		L.de.dk = r.size(d, "dim", "right");
		L.de.dv = r.size(d, "vdim", "right");
		L.de.taps = r.size(d, "conv", "right");
		const json::Value *ff = l.find("mlp");
		if (ff) {
			const json::Value *kd = ff->find("kind");
			if (!kd || kd->str != "dense") return fail(TG_EINVAL, "config.json: unknown kind of feed-forward");
			L.ff.ff = r.size(ff, "ff", "mlp");
			L.ff.ffp = round_up(L.ff.ff, 16);
		}
		if (!r.err.empty()) return fail(TG_EINVAL, r.err);
		if (L.at.H % L.at.G || L.de.H % L.de.KH) return fail(TG_ESHAPE, "config.json: heads are not a multiple of kv_heads");
		if (L.de.dk > 256) return fail(TG_ESHAPE, "delta rule: key sizes above 256 are not supported");
		m->layers.push_back(L);
	}
	const int n = int(m->layers.size());
	int start = 0, stop = 0, times = 1;
	if (const json::Value *lp = c.find("loop")) {
		start = r.size(lp, "start", "loop", 0);
		stop = r.size(lp, "stop", "loop", 0);
		times = r.size(lp, "times", "loop", 1);
		if (r.err.empty() && (start > stop || stop > n)) return fail(TG_EINVAL, "config.json: loop lies outside the layers");
	}
	if (!r.err.empty()) return fail(TG_EINVAL, r.err);
	if (m->taps > 16) return fail(TG_ESHAPE, "input convolutions of more than 16 taps are not supported");
	for (int i = 0; i < start; i++) m->runs.push_back({i, false});
	for (int t = 0; t < times; t++)
		for (int i = start; i < stop; i++) m->runs.push_back({i, t > 0 && i == start});
	for (int i = std::max(start, stop); i < n; i++) m->runs.push_back({i, false});
	return TG_OK;
}

inline int read_sominex(const json::Value &c, HybridModel *m) {
	ConfigReader r;
	read_model(r, c, m);
	m->rms = true;
	m->has_canon = true;
	m->taps = 2;
	m->embed_scale = float(r.num(r.obj(&c, "embedding", "model"), "scale", "embedding"));
	const json::Value *ls;
	TG_TRY(layer_list(c, &ls));
	for (const auto &l : ls->items) {
		Layer L;
		L.beside = true;
		const json::Value *ty = l.find("type"), *mx = r.obj(&l, "mixer", "layer");
		const std::string type = ty ? ty->str : "";
		if (type == "attention") {
			AttnSpec &A = L.at;
			A.H = r.size(mx, "heads", "mixer");
			A.G = r.size(mx, "kv_heads", "mixer");
			A.dk = r.size(mx, "dim", "mixer");
			A.dv = r.size(mx, "vdim", "mixer");
			A.scale = float(r.num(mx, "scale", "mixer"));
			const json::Value *mk = r.obj(mx, "mask", "mixer");
			A.window = r.size(mk, "size", "mask");
			if (mk && mk->find("pool")) A.pool = r.size(mk, "pool", "mask", 0);
			A.dkp = round_up(A.dk, 16);
			A.dvp = round_up(A.dv, 16);
			A.vnorm = true;
			if (r.err.empty() && A.H % A.G) return fail(TG_ESHAPE, "config.json: heads are not a multiple of kv_heads");
			if (const json::Value *ro = mx ? mx->find("rot") : nullptr) {
				Rotation t;
				t.dims = r.size(ro, "dims", "rot", 0);
				t.base = r.num(ro, "base", "rot");
				if (const json::Value *sc = ro->find("scaling")) {
					t.factor = r.num(sc, "factor", "scaling");
					t.original = r.num(sc, "original", "scaling");
					t.fast = r.num(sc, "fast", "scaling");
					t.slow = r.num(sc, "slow", "scaling");
					if (r.err.empty() && !(t.factor > 0 && t.original > 0 && t.fast > 0 && t.slow > 0)) return fail(TG_EINVAL, "config.json: rot.scaling is out of range");
				}
				if (r.err.empty() && (t.dims % 2 || t.dims > A.dk || !(t.base > 0.0) || t.base == 1.0)) return fail(TG_ESHAPE, "config.json: rot.dims or rot.base is out of range");
				if (t.dims) {
					A.rot = int(std::find(m->rots.begin(), m->rots.end(), t) - m->rots.begin());
					if (size_t(A.rot) == m->rots.size()) m->rots.push_back(t);
					A.rot_dims = t.dims;
					m->rot_half = std::max(m->rot_half, round_up(t.dims / 2, 2));
				}
			}
		} else if (type == "mamba2" || type == "mlstm") {
			LinSpec &R = L.li;
			R.kind = type == "mamba2" ? LIN_SSM : LIN_MLSTM;
			R.H = r.size(mx, "heads", "mixer");
			R.vd = r.size(mx, "vdim", "mixer");
			if (R.kind == LIN_SSM) {
				R.N = r.size(mx, "state", "mixer");
				R.G = r.size(mx, "groups", "mixer");
				R.taps = r.size(mx, "conv", "mixer");
				R.parts = r.size(mx, "norm_groups", "mixer");
				if (r.err.empty() && R.H % R.G) return fail(TG_ESHAPE, "config.json: heads are not a multiple of groups");
				if (r.err.empty() && R.H * R.vd % R.parts) return fail(TG_ESHAPE, "config.json: norm_groups does not divide the inner size");
				if (R.taps > 16) return fail(TG_ESHAPE, "convolutions of more than 16 taps are not supported");
			} else {
				R.N = r.size(mx, "dim", "mixer");
				R.G = R.parts = R.H;
				R.gate_cap = float(r.num(mx, "gate_cap", "mixer"));
				if (r.err.empty() && !(R.gate_cap > 0.0f)) return fail(TG_EINVAL, "config.json: mixer.gate_cap is out of range");
			}
			if (R.N > 512) return fail(TG_ESHAPE, "recurrences with more than 512 key dimensions are not supported");
			R.Np = round_up(R.N, 16);
			R.vdp = round_up(R.vd, 16);
		} else {
			return fail(TG_EINVAL, "config.json: unknown layer type" + type_of(ty));
		}
		if (const json::Value *ff = l.find("mlp")) {
			const json::Value *kd = ff->find("kind");
			FfSpec &F = L.ff;
			if (kd && kd->str == "dense") {
				F.ff = r.size(ff, "ff", "mlp");
				F.act = GLU_CLAMP;
				F.limit = float(r.num(ff, "limit", "mlp"));
			} else if (kd && kd->str == "moe") {
				const json::Value *ro = r.obj(ff, "router", "mlp");
				F.act = GLU_SILU;
				F.experts = r.size(ro, "experts", "router");
				F.top = r.size(ro, "top", "router");
				F.route_scale = float(r.num(ro, "scale", "router"));
				F.eff = r.size(r.obj(ff, "expert", "mlp"), "ff", "expert");
				F.effp = round_up(F.eff, 16);
				if (const json::Value *sh = ff->find("shared")) F.ff = r.size(sh, "ff", "shared");
				if (r.err.empty() && F.top > F.experts) return fail(TG_EINVAL, "config.json: router.top exceeds router.experts");
				if (F.experts > MOE_MAX || F.top > MOE_TOP) return fail(TG_ESHAPE, "mixtures of more than 512 experts or 32 per token are not supported");
			} else {
				return fail(TG_EINVAL, "config.json: unknown kind of feed-forward" + type_of(kd));
			}
			F.ffp = round_up(F.ff, 16);
		}
		if (!r.err.empty()) return fail(TG_EINVAL, r.err);
		m->runs.push_back({int(m->layers.size()), false});
		m->layers.push_back(L);
	}
	return r.err.empty() ? TG_OK : fail(TG_EINVAL, r.err);
}

// the part of opening that needs the weights
inline int load_common(Loader &ld) {
	HybridModel *m = ld.m;
	const SafeTensors::Tensor *e;
	auto table = [&](const char *name, Lin *l) -> int {
		TG_TRY(ld.get(name, {m->n_vocab, m->D}, &e));
		Loader::Host h(m->n_vocab, m->Dp);
		Loader::put(h, 0, 0, *e, 0, m->n_vocab, 0, m->D);
		return ld.linear(h, l);
	};
	TG_TRY(table("embed", &m->embed));
	if (m->architecture == "Nabelix") m->head = m->embed;
	else TG_TRY(table("head", &m->head));
	TG_TRY(ld.vec("final.norm", m->D, &m->final_norm));
	if (!m->rots.empty()) {
		std::vector<double> f(m->rots.size() * m->rot_half, 0.0);
		std::vector<float> k(m->rots.size());
		for (size_t i = 0; i < k.size(); i++) k[i] = m->rots[i].frequencies(f.data() + i * m->rot_half);
		TG_TRY(ld.upload(f.data(), f.size() * 8, reinterpret_cast<void **>(&m->rot_freq)));
		TG_TRY(ld.upload(k.data(), k.size() * 4, reinterpret_cast<void **>(&m->rot_factor)));
	}
	return TG_OK;
}

inline int open_hybrid(const char *dir, int device, int dtype, tg_model **out) {
	json::Value cfg;
	std::string err;
	if (!json::parse_file(std::string(dir) + "/config.json", &cfg, &err)) return fail(TG_EIO, err);
	std::unique_ptr<HybridModel> m(new HybridModel());
	m->architecture = cfg.find("architecture")->str;
	m->device = device;
	m->dtype = dtype;
	const bool nabelix = m->architecture == "Nabelix";
	TG_TRY(nabelix ? read_nabelix(cfg, m.get()) : read_sominex(cfg, m.get()));
	Loader ld;
	ld.m = m.get();
	if (!ld.st.open(std::string(dir) + "/model.safetensors", &err)) return fail(TG_EIO, err);
	TG_TRY(ensure_device(device));
	TG_TRY(load_common(ld));
	for (size_t i = 0; i < m->layers.size(); i++) TG_TRY(nabelix ? ld.nabelix_layer(int(i)) : ld.sominex_layer(int(i)));
	*out = m.release();
	return TG_OK;
}

static RegisterArch reg_nabelix("Nabelix", open_hybrid), reg_sominex("Sominex", open_hybrid);

}  // namespace tg
