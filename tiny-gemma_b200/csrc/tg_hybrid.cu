// Layered decoders read from a model folder, bf16 weights: the family of "Nabelix" (config.json names the layers and
// every size and constant). A layer is
//     x <- x + mixer(conv(norm1(x)));   x <- x + ff(norm2(x))
// with layer norms, a causal input convolution, and the "parallel" mixer: windowed attention with kept first tokens
// and a distance bias beside a gated delta rule, both reading the same input. A block of layers may run several
// times in a row (a loop), every pass with a cache of its own.
//
// Two pipelines compute a step; both use the same caches and states:
//   up to 4 rows, one token per sequence: five launches per layer (kernels_gemv_bf16.cuh, hybrid_token_mix_kernel)
//   anything else: tensor-core (or fp32) matrix products over all rows of the step
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>
#include <climits>
#include <cmath>
#include <cstdio>
#include <cstring>
#include <memory>

#include "kernels_delta.cuh"
#include "kernels_gemm_bf16.cuh"
#include "kernels_gemv_bf16.cuh"
#include "kernels_rowwise.cuh"
#include "kernels_window_attn.cuh"
#include "model_dir.hpp"
#include "tg_internal.hpp"

using namespace tg;
typedef __nv_bfloat16 bf16;

namespace {

int round_up(int x, int m) { return (x + m - 1) / m * m; }

// One token per sequence: the attention of every (sequence, key/value head, run of keys) and the delta rule of every
// (sequence, head) in one launch. grid (G * nsplit + delta heads, rows)
template <typename PT, typename CT, typename OT>
__global__ void __launch_bounds__(256) hybrid_token_mix_kernel(WAttnArgs w, DeltaArgs d) {
	pdl_trigger();
	pdl_wait();
	extern __shared__ __align__(16) float mix_sm[];
	const int n_attn = w.G * w.nsplit;
	// (the delta heads are the longer chains: they start first)
	if (int(blockIdx.x) < d.H)
		delta_token_cta<PT, OT>(d, blockIdx.y, blockIdx.x, mix_sm);
	else if (int(blockIdx.x) - d.H < n_attn)
		window_attn_token_cta<PT, CT, OT>(w, blockIdx.y, (blockIdx.x - d.H) / w.nsplit, (blockIdx.x - d.H) % w.nsplit, mix_sm);
}

// positions and history parities of the lock-step decode after a token
__global__ void hybrid_advance_kernel(int *pos, int *par, int n) {
	pdl_trigger();
	pdl_wait();
	const int i = blockIdx.x * blockDim.x + threadIdx.x;
	if (i < n) {
		pos[i] += 1;
		par[i] ^= 1;
	}
}

// A linear layer: weights [N][ld] bf16 with K used columns (padded with zeros to a multiple of 8).
struct Lin {
	const bf16 *W = nullptr;
	int N = 0, K = 0, ld = 0;
	CUtensorMap map[3];  // boxes of 64, 128 and 256 rows
};

int make_map(CUtensorMap *out, const void *base, size_t rows, int cols, int ld, int box_rows) {
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

// ------------------------------------------------------------------ what config.json says
struct AttnSpec {
	int H = 0, G = 0, dk = 0, dv = 0, dkp = 0, dvp = 0;
	float scale = 0.0f;
	int window = 0, keep = 0;
};
struct DeltaSpec {
	int H = 0, KH = 0, dk = 0, dv = 0, taps = 0, ra = 0, rg = 0;
	int channels() const { return 2 * KH * dk + H * dv; }
	int dkp() const { return dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 128 ? 128 : 256)); }
};
struct Layer {
	AttnSpec at;
	DeltaSpec de;
	float left_scale = 1.0f, right_scale = 1.0f;
	int ff = 0, ffp = 0;  // 0: no feed-forward
	// columns of a projection row
	int p_q, p_k, p_v, p_g, p_a1, p_g1, p_conv, p_b, ldp;
	int o_col, kc;        // columns of a mixed row: attention heads at 0, delta heads at o_col; kc in all
	float *norm1, *norm2 = nullptr, *canon = nullptr, *r1, *r2, *conv, *A_log, *dt_bias, *rnorm;
	Lin proj, a2, g2, out, gu, down;
};
struct Run {
	int layer;
	bool add_embed;  // another pass through the loop begins here
};

}  // namespace

struct HybridModel : tg_model {
	std::string architecture;
	int dtype = TG_BF16;
	int D = 0, Dp = 0, taps = 1;  // taps of the input convolution
	bool has_canon = false;
	float eps = 1e-6f, softcap = 0.0f;
	std::vector<Layer> layers;
	std::vector<Run> runs;
	Lin embed;
	float *final_norm = nullptr;
	std::vector<void *> mem;

	~HybridModel() override {
		for (void *p : mem) cudaFree(p);
	}
	const char *arch() const override { return architecture.c_str(); }
	int new_state(int batch, int max_pos, tg_state **out) override;
};

namespace {

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

	int layer(int i) {
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
		L.ldp = round_up(n, 8);
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
		L.kc = round_up(L.o_col + E.H * E.dv, 8);
		{
			Host h(D, L.kc);
			for (int x = 0; x < A.H; x++) put(h, 0, x * A.dvp, *o, 0, D, size_t(x) * A.dv, A.dv);
			put(h, 0, L.o_col, *ro, 0, D, 0, E.H * E.dv);
			TG_TRY(linear(h, &L.out));
		}
		if (L.ff) {
			const SafeTensors::Tensor *ga, *up, *dn;
			TG_TRY(vec(p + "norm2", D, &L.norm2));
			TG_TRY(get(p + "mlp.gate", {L.ff, D}, &ga));
			TG_TRY(get(p + "mlp.up", {L.ff, D}, &up));
			TG_TRY(get(p + "mlp.down", {D, L.ff}, &dn));
			{
				Host h(2 * L.ffp, Dp);  // blocks of 16 gate rows, 16 up rows
				for (int x = 0; x < L.ff; x += 16) {
					const int c = std::min(16, L.ff - x);
					put(h, 2 * x, 0, *ga, x, c, 0, D);
					put(h, 2 * x + 16, 0, *up, x, c, 0, D);
				}
				TG_TRY(linear(h, &L.gu));
			}
			Host h(D, L.ffp);
			put(h, 0, 0, *dn, 0, D, 0, L.ff);
			TG_TRY(linear(h, &L.down));
		}
		return TG_OK;
	}
};

// config.json -> the model's layer list. Every size and constant comes from here (or from a tensor's shape).
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

int read_config(const json::Value &c, HybridModel *m) {
	ConfigReader r;
	m->D = r.size(&c, "width", "model");
	m->hidden_size = m->D;
	m->Dp = round_up(m->D, 8);
	m->n_vocab = r.size(&c, "vocab", "model");
	m->n_pos = 1 << 24;  // distances stay exact in fp32
	m->eps = float(r.num(r.obj(&c, "norm", "model"), "eps", "norm"));
	m->softcap = float(r.num(&c, "logit_softcap", "model", false, 0.0));
	if (const json::Value *cn = c.find("canon")) {
		m->has_canon = true;
		m->taps = r.size(cn, "taps", "canon");
	}
	const json::Value *ls = c.find("layers");
	if (!ls || ls->kind != json::Value::ARRAY || ls->items.empty()) return fail(TG_EINVAL, "config.json: no layers");
	for (const auto &l : ls->items) {
		Layer L;
		const json::Value *ty = l.find("type");
		if (!ty || ty->str != "parallel") return fail(TG_EINVAL, "config.json: unknown layer type" + (ty ? " " + ty->str : std::string()));
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
		L.de.H = r.size(d, "heads", "right");
		L.de.KH = r.size(d, "kv_heads", "right");
		L.de.dk = r.size(d, "dim", "right");
		L.de.dv = r.size(d, "vdim", "right");
		L.de.taps = r.size(d, "conv", "right");
		const json::Value *ff = l.find("mlp");
		if (ff) {
			const json::Value *kd = ff->find("kind");
			if (!kd || kd->str != "dense") return fail(TG_EINVAL, "config.json: unknown kind of feed-forward");
			L.ff = r.size(ff, "ff", "mlp");
			L.ffp = round_up(L.ff, 16);
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

int open_hybrid(const char *dir, int device, int dtype, tg_model **out) {
	json::Value cfg;
	std::string err;
	if (!json::parse_file(std::string(dir) + "/config.json", &cfg, &err)) return fail(TG_EIO, err);
	std::unique_ptr<HybridModel> m(new HybridModel());
	m->architecture = cfg.find("architecture")->str;
	m->device = device;
	m->dtype = dtype;
	TG_TRY(read_config(cfg, m.get()));
	Loader ld;
	ld.m = m.get();
	if (!ld.st.open(std::string(dir) + "/model.safetensors", &err)) return fail(TG_EIO, err);
	TG_TRY(ensure_device(device));
	const SafeTensors::Tensor *e;
	TG_TRY(ld.get("embed", {m->n_vocab, m->D}, &e));
	{
		Loader::Host h(m->n_vocab, m->Dp);
		Loader::put(h, 0, 0, *e, 0, m->n_vocab, 0, m->D);
		TG_TRY(ld.linear(h, &m->embed));
	}
	TG_TRY(ld.vec("final.norm", m->D, &m->final_norm));
	for (size_t i = 0; i < m->layers.size(); i++) TG_TRY(ld.layer(int(i)));
	*out = m.release();
	return TG_OK;
}

RegisterArch reg_nabelix("Nabelix", open_hybrid);

}  // namespace

// ===================================================================== state
struct HybridState : tg_state {
	HybridModel *m = nullptr;
	bool f32 = false;
	int max_rows = 0, max_seq_rows = 0;  // rows of a pass, rows one sequence brings to it
	struct RunCache {
		void *kc = nullptr, *vc = nullptr, *ks = nullptr, *vs = nullptr;
		int cap = 0, keep_rows = 0;
		float *canon = nullptr, *conv = nullptr, *S = nullptr;
		CUtensorMap kmap, vmap, ksmap, vsmap;
	};
	std::vector<RunCache> cache;
	std::vector<void *> mem;
	// activations of a pass
	float *x = nullptr;
	int ldx = 0;
	float2 *stats = nullptr;          // mean and 1/deviation of the rows
	void *h = nullptr, *P = nullptr, *O = nullptr, *act = nullptr;   // bf16, or fp32 in a 32-bit state
	float *P32 = nullptr, *O32 = nullptr, *act32 = nullptr;          // the few-row pipeline's, always fp32
	float *z = nullptr, *gz = nullptr, *o_raw = nullptr, *blk = nullptr, *bV = nullptr;
	float *part = nullptr;
	unsigned *tickets = nullptr;
	int nsplit_cap = 1;
	CUtensorMap hmap;                 // h as an operand
	std::vector<CUtensorMap> pmap, omap, amap, a1map, g1map;  // per layer
	float *wl = nullptr;              // logits of wanted rows
	int wl_rows = 0;
	void *hn = nullptr;               // their normed rows
	CUtensorMap hnmap;
	int *want_dev = nullptr;
	// descriptors: of a general pass, and of the lock-step decode (row b = sequence b)
	int *desc = nullptr, *desc_pin = nullptr;
	size_t desc_ints = 0;
	int *ls_desc = nullptr, *ls_pos = nullptr, *ls_par = nullptr;
	bool ls_dirty = true;
	std::vector<int> host_par;
	// layer trace
	bool tracing = false;
	std::vector<float> trace;
	int trace_rows = 0;

	~HybridState() override {
		for (void *p : mem) cudaFree(p);
		if (desc_pin) cudaFreeHost(desc_pin);
		free_common();
	}
	int alloc();
	int reset() override;
	int prefill(const int *ids, int S, float *logits_host) override;
	int append(const int *ids, int n, float *logits_host) override;
	int enqueue_decode_all() override;
	int enqueue_forward() override;
	int run_steps(int n_steps, float minp, float temp) override;
	int step(int n, const int *seq, const int *count, const int *ids, const int *n_want, const int *want, float *logits_host) override;
	int free_sequence(int b) override;
	int trace_enable(int on) override;
	int trace_read(float *x_host, size_t cap_floats, int *runs, int *tokens) override;

	int sync_lockstep();
	StepDesc lockstep_desc() const;
	int run_layers(const StepDesc &d, int R, int nseg, int max_len);
	int score_rows(const int *rows_dev, int n, float *out, float *norm_out);
	int gemm(int epi, const void *A, int lda, const CUtensorMap *amap_, const Lin &w, int M, void *C, int ldc, float cap = 0.0f);
	int gemv(int pro, int epi, GemvArgs g, int R);
	WAttnArgs attn_args(const StepDesc &d, int run, const void *p, int ldp, void *out, int ldo);
	DeltaArgs delta_args(const StepDesc &d, int run, const void *p, int ldp, void *out, int ldo);

	struct Entry {
		int seq, count, done;
		const int *ids;
		std::vector<int> want;  // places
		size_t out0;            // first output row
		size_t given = 0;       // wanted rows already scored
	};
	// last = true: instead of `want`, the last token of every entry is scored into `logits` (row = sequence)
	int run_entries(std::vector<Entry> &es, bool last, float *logits_host);

	template <typename T> int take(T **p, size_t n) {
		if (n == 0) n = 1;
		cudaError_t e = cudaMalloc(reinterpret_cast<void **>(p), n * sizeof(T));
		if (e != cudaSuccess) {
			cudaGetLastError();
			return fail(TG_ENOMEM, std::string("cudaMalloc(state): ") + cudaGetErrorString(e));
		}
		mem.push_back(*p);
		TG_CUDA(cudaMemsetAsync(*p, 0, n * sizeof(T), stream));
		return TG_OK;
	}
	int take_act(void **p, size_t n) {
		uint8_t *q;
		TG_TRY(take(&q, n * (f32 ? 4 : 2)));
		*p = q;
		return TG_OK;
	}
};

namespace {
constexpr int FEW_ROWS = 4;  // rows of the matrix-vector pipeline
constexpr int TOKEN_SPLITS = 32;

template <typename K> int allow_smem(K kernel, size_t bytes) {
	if (bytes <= 48 * 1024) return TG_OK;
	if (bytes > 227 * 1024) return fail(TG_ESHAPE, "a layer's sizes need more shared memory than an SM has");
	TG_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(bytes)));
	return TG_OK;
}

// columns of a tile: waves x measured time of a K-block (a tile is bound by what it reads from the L2)
int pick_bn(int m_tiles, int N) {
	static const int forced = env_int("TG_GEMM_BN", 0);
	if (forced) return forced;
	int best = 64;
	double cost = 1e30;
	for (int bn : {256, 128, 64}) {
		const int tiles = m_tiles * ((N + bn - 1) / bn);
		const double c = double((tiles + g_num_sms - 1) / g_num_sms) * (bn == 256 ? 1.0 : (bn == 128 ? 0.79 : 0.6));
		if (c < cost) {
			cost = c;
			best = bn;
		}
	}
	return best;
}

template <int BN, int EPI> int launch_gemm_tc(const CUtensorMap &am, const CUtensorMap &wm, const GemmArgs &a, cudaStream_t st) {
	static bool done[TG_MAX_DEVICES] = {};
	bool &d = done[current_device_slot()];
	if (!d) {
		TG_TRY(allow_smem(gemm_bf16_tc_kernel<BN, EPI>, GbShape<BN>::SMEM));
		d = true;
	}
	launch_k(gemm_bf16_tc_kernel<BN, EPI>, dim3(std::min(g_num_sms, a.m_tiles * a.n_tiles)), dim3(GB_THREADS), size_t(GbShape<BN>::SMEM), st, am, wm, a);
	count_launch();
	return check_launch("gemm_bf16_tc");
}
template <int EPI> int launch_gemm(const CUtensorMap &am, const Lin &w, GemmArgs a, cudaStream_t st) {
	a.m_tiles = (a.M + GB_BM - 1) / GB_BM;
	const int cols = EPI == GEMM_LOGITS ? a.ldc : a.N, bn = pick_bn(a.m_tiles, cols);
	a.n_tiles = (cols + bn - 1) / bn;
	if (bn == 256) return launch_gemm_tc<256, EPI>(am, w.map[2], a, st);
	if (bn == 128) return launch_gemm_tc<128, EPI>(am, w.map[1], a, st);
	return launch_gemm_tc<64, EPI>(am, w.map[0], a, st);
}
template <int EPI> int launch_gemm_f32(const float *A, int lda, const Lin &w, const GemmArgs &a, cudaStream_t st) {
	const int cols = EPI == GEMM_LOGITS ? a.ldc : a.N;
	launch_k(gemm_f32_kernel<EPI>, dim3((cols + GF_T - 1) / GF_T, (a.M + GF_T - 1) / GF_T), dim3(256), 0, st, A, lda, w.W, w.ld, a);
	count_launch();
	return check_launch("gemm_f32");
}

template <int R, int NR, int KS, int PRO, int EPI> int launch_gemv(const GemvArgs &g, cudaStream_t st) {
	const size_t smem = gv_smem<R, NR>(g.K, PRO);
	auto kernel = gemv_bf16_kernel<R, NR, KS, PRO, EPI>;
	TG_TRY(allow_smem(kernel, smem));
	int occ = 1;
	TG_CUDA(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&occ, kernel, GV_THREADS, smem));
	const int outs = (8 / KS) * NR / (EPI == GV_GEGLU ? 2 : 1);
	const int n_out = EPI == GV_GEGLU ? g.N / 2 : (EPI == GV_LOGITS ? g.ldo : g.N);
	const int groups = (n_out + outs - 1) / outs;
	launch_k(kernel, dim3(std::min(groups, std::max(1, occ) * g_num_sms)), dim3(GV_THREADS), smem, st, g);
	count_launch();
	return check_launch("gemv_bf16");
}
template <int R> int launch_gemv_r(int pro, int epi, const GemvArgs &g, cudaStream_t st) {
	if (pro == GV_LN_CONV && epi == GV_PROJ) return launch_gemv<R, 4, 2, GV_LN_CONV, GV_PROJ>(g, st);
	if (pro == GV_VEC && epi == GV_ADD) return launch_gemv<R, 4, 8, GV_VEC, GV_ADD>(g, st);
	if (pro == GV_LN && epi == GV_GEGLU) return launch_gemv<R, 4, 2, GV_LN, GV_GEGLU>(g, st);
	if (pro == GV_LN && epi == GV_LOGITS) return launch_gemv<R, 4, 2, GV_LN, GV_LOGITS>(g, st);
	return fail(TG_EINVAL, "gemv: no such combination");
}
}  // namespace

int HybridModel::new_state(int batch, int max_pos, tg_state **out) {
	HybridState *s = new HybridState();
	s->m = this;
	s->model = this;
	s->B = batch;
	s->max_pos_global = max_pos;
	s->f32 = dtype == TG_F32;
	const int rc = s->alloc();
	if (rc != TG_OK) {
		const std::string keep = tg_last_error();
		tg_state_free(s);
		return fail(rc, keep);
	}
	*out = s;
	return TG_OK;
}

int HybridState::alloc() {
	TG_TRY(alloc_common());
	const int D = m->D;
	const int pass = std::max(B, env_int("TG_PASS_ROWS", 4096));
	max_seq_rows = std::min(std::max(128, pass / B), max_pos_global);
	max_rows = std::min<long long>(std::max(pass, B), (long long)B * max_seq_rows);
	const int R = max_rows;
	const size_t es = f32 ? 4 : 2;
	ldx = round_up(D, 8);
	int ldp = 8, kc = 8, ffp = 16, hz = 1, hv = 1;
	size_t blkn = 1, blkV = 1, partn = 1;
	int gmax = 1;
	for (const Layer &L : m->layers) {
		ldp = std::max(ldp, L.ldp);
		kc = std::max(kc, L.kc);
		ffp = std::max(ffp, L.ffp);
		hz = std::max(hz, round_up(L.de.H * L.de.dk, 4));
		hv = std::max(hv, round_up(L.de.H * L.de.dv, 4));
		blkn = std::max(blkn, size_t(L.de.H) * delta_block_floats(L.de.dkp()));
		blkV = std::max(blkV, size_t(L.de.H) * DB * L.de.dv);
		partn = std::max(partn, size_t(L.at.H) * (L.at.dvp + 2));
		gmax = std::max(gmax, L.at.G);
	}
	TG_TRY(take(&x, size_t(R) * ldx));
	TG_TRY(take(&stats, R));
	TG_TRY(take_act(&h, size_t(R) * m->Dp));
	TG_TRY(take_act(&P, size_t(R) * ldp));
	TG_TRY(take_act(&O, size_t(R) * kc));
	TG_TRY(take_act(&act, size_t(R) * ffp));
	const int F = std::min(FEW_ROWS, B);
	TG_TRY(take(&P32, size_t(F) * ldp));
	TG_TRY(take(&O32, size_t(F) * kc));
	TG_TRY(take(&act32, size_t(F) * ffp));
	TG_TRY(take(&z, size_t(R) * hz));
	TG_TRY(take(&gz, size_t(R) * hv));
	TG_TRY(take(&o_raw, size_t(R) * hv));
	const size_t nb = size_t(R) / DB + B + 1;
	TG_TRY(take(&blk, nb * blkn));
	TG_TRY(take(&bV, nb * blkV));
	nsplit_cap = std::max(1, std::min(TOKEN_SPLITS, 2 * g_num_sms / B));
	TG_TRY(take(&part, size_t(B) * nsplit_cap * partn));
	TG_TRY(take(&tickets, size_t(B) * gmax));
	// caches
	cache.resize(m->runs.size());
	for (size_t i = 0; i < cache.size(); i++) {
		const Layer &L = m->layers[m->runs[i].layer];
		const AttnSpec &A = L.at;
		RunCache &c = cache[i];
		c.cap = round_up(int(std::min<long long>(max_pos_global, (long long)A.window + max_seq_rows)), 64);
		c.keep_rows = round_up(std::min(A.keep, max_pos_global), 64);
		uint8_t *q;
		auto rows = [&](void **p, size_t n, int w) -> int {
			TG_TRY(take(&q, size_t(B) * n * w * es));
			*p = q;
			return TG_OK;
		};
		TG_TRY(rows(&c.kc, c.cap, A.G * A.dkp));
		TG_TRY(rows(&c.vc, c.cap, A.G * A.dvp));
		TG_TRY(rows(&c.ks, c.keep_rows, A.G * A.dkp));
		TG_TRY(rows(&c.vs, c.keep_rows, A.G * A.dvp));
		TG_TRY(take(&c.canon, size_t(B) * 2 * (m->taps - 1) * D));
		TG_TRY(take(&c.conv, size_t(B) * 2 * (L.de.taps - 1) * L.de.channels()));
		TG_TRY(take(&c.S, size_t(B) * L.de.H * L.de.dk * L.de.dv));
		if (!f32) {
			TG_TRY(make_map(&c.kmap, c.kc, size_t(B) * c.cap, A.G * A.dkp, A.G * A.dkp, WT_KEYS));
			TG_TRY(make_map(&c.vmap, c.vc, size_t(B) * c.cap, A.G * A.dvp, A.G * A.dvp, WT_KEYS));
			c.ksmap = c.kmap;  // (not used without kept tokens)
			c.vsmap = c.vmap;
			if (c.keep_rows) {
				TG_TRY(make_map(&c.ksmap, c.ks, size_t(B) * c.keep_rows, A.G * A.dkp, A.G * A.dkp, WT_KEYS));
				TG_TRY(make_map(&c.vsmap, c.vs, size_t(B) * c.keep_rows, A.G * A.dvp, A.G * A.dvp, WT_KEYS));
			}
		}
	}
	// wanted rows
	wl_rows = std::max(16, std::min(1024, int((size_t(64) << 20) / ld_logits)));
	wl_rows = std::min(wl_rows, std::max(16, R));
	TG_TRY(take(&wl, size_t(wl_rows) * ld_logits));
	TG_TRY(take_act(&hn, size_t(std::max(wl_rows, B)) * m->Dp));
	TG_TRY(take(&want_dev, wl_rows));
	if (!f32) {
		TG_TRY(make_map(&hmap, h, R, m->Dp, m->Dp, GB_BM));
		TG_TRY(make_map(&hnmap, hn, std::max(wl_rows, B), m->Dp, m->Dp, GB_BM));
		const size_t n = m->layers.size();
		for (auto *v : {&pmap, &omap, &amap, &a1map, &g1map}) v->resize(n);
		for (size_t i = 0; i < n; i++) {
			const Layer &L = m->layers[i];
			const bf16 *p = static_cast<const bf16 *>(P);
			TG_TRY(make_map(&pmap[i], P, R, L.ldp, L.ldp, 128));
			TG_TRY(make_map(&omap[i], O, R, L.kc, L.kc, GB_BM));
			if (L.ff) TG_TRY(make_map(&amap[i], act, R, L.ffp, L.ffp, GB_BM));
			TG_TRY(make_map(&a1map[i], p + L.p_a1, R, L.de.ra, L.ldp, GB_BM));
			TG_TRY(make_map(&g1map[i], p + L.p_g1, R, L.de.rg, L.ldp, GB_BM));
		}
	}
	// descriptors
	desc_ints = size_t(2) * R + 5 * size_t(B);
	TG_TRY(take(&desc, desc_ints));
	TG_CUDA(cudaMallocHost(&desc_pin, desc_ints * 4));
	TG_TRY(take(&ls_desc, size_t(5) * B));
	ls_pos = ls_desc + 3 * B;
	ls_par = ls_desc + 4 * B;
	std::vector<int> init(size_t(5) * B, 0);
	for (int b = 0; b < B; b++) {
		init[b] = b;          // row -> segment, segment -> sequence, segment -> first row
		init[B + b] = 1;      // length
	}
	TG_CUDA(cudaMemcpyAsync(ls_desc, init.data(), init.size() * 4, cudaMemcpyHostToDevice, stream));
	host_par.assign(B, 0);
	TG_CUDA(cudaStreamSynchronize(stream));
	return TG_OK;
}

StepDesc HybridState::lockstep_desc() const {
	StepDesc d;
	d.tok = tok;
	d.row_seg = d.seg_seq = d.seg_row = ls_desc;
	d.seg_len = ls_desc + B;
	d.seg_pos = ls_pos;
	d.seg_par = ls_par;
	return d;
}

// the device's positions and parities of the lock-step decode follow the host's after anything else has run
int HybridState::sync_lockstep() {
	if (!ls_dirty) return TG_OK;
	TG_CUDA(cudaStreamSynchronize(stream));  // (desc_pin may still be read by an earlier copy)
	for (int b = 0; b < B; b++) {
		desc_pin[b] = host_pos[b];
		desc_pin[B + b] = host_par[b];
	}
	TG_CUDA(cudaMemcpyAsync(ls_pos, desc_pin, size_t(2) * B * 4, cudaMemcpyHostToDevice, stream));
	ls_dirty = false;
	return TG_OK;
}

int HybridState::reset() {
	// What caches and histories hold is never read before it has been written again: rows at negative positions count
	// as zero, and a state matrix is read from position 1 on.
	host_par.assign(B, 0);
	ls_dirty = true;
	return TG_OK;
}

int HybridState::free_sequence(int b) {
	TG_CUDA(cudaStreamSynchronize(stream));
	host_pos[b] = 0;
	host_par[b] = 0;
	ls_dirty = true;
	return TG_OK;
}

int HybridState::trace_enable(int on) {
	tracing = on != 0;
	trace.clear();
	trace_rows = 0;
	return TG_OK;
}

int HybridState::trace_read(float *x_host, size_t cap_floats, int *runs, int *tokens) {
	*runs = trace_rows ? int(m->runs.size()) : 0;
	*tokens = trace_rows;
	if (!x_host) return TG_OK;
	if (cap_floats < trace.size()) return fail(TG_EINVAL, "buffer too small for the trace");
	std::memcpy(x_host, trace.data(), trace.size() * 4);
	return TG_OK;
}

// ------------------------------------------------------------------ pieces of a step
int HybridState::gemm(int epi, const void *A, int lda, const CUtensorMap *am, const Lin &w, int M, void *C, int ldc, float cap) {
	GemmArgs a{};
	a.M = M;
	a.N = w.N;
	a.K = w.K;
	a.C = C;
	a.ldc = ldc;
	a.cap = cap;
	a.err = err_flag;
	if (f32) {
		const float *Af = static_cast<const float *>(A);
		switch (epi) {
			case GEMM_ADD: return launch_gemm_f32<GEMM_ADD>(Af, lda, w, a, stream);
			case GEMM_GEGLU: return launch_gemm_f32<GEMM_GEGLU>(Af, lda, w, a, stream);
			case GEMM_LOGITS: return launch_gemm_f32<GEMM_LOGITS>(Af, lda, w, a, stream);
			default: return launch_gemm_f32<GEMM_STORE>(Af, lda, w, a, stream);
		}
	}
	switch (epi) {
		case GEMM_STORE: return launch_gemm<GEMM_STORE>(*am, w, a, stream);
		case GEMM_STORE32: return launch_gemm<GEMM_STORE32>(*am, w, a, stream);
		case GEMM_ADD: return launch_gemm<GEMM_ADD>(*am, w, a, stream);
		case GEMM_GEGLU: return launch_gemm<GEMM_GEGLU>(*am, w, a, stream);
		default: return launch_gemm<GEMM_LOGITS>(*am, w, a, stream);
	}
}

int HybridState::gemv(int pro, int epi, GemvArgs g, int R) {
	g.err = err_flag;
	// (rows whose activations do not fit shared memory together go in smaller groups)
	int most = R >= 4 ? 4 : (R >= 2 ? 2 : 1);
	while (most > 1 && size_t(most) * 8 * gv_k8(g.K) * 4 > 160 * 1024) most /= 2;
	for (int r = 0; r < R;) {
		int n = most;
		while (n > R - r) n /= 2;
		GemvArgs s = g;
		s.d.tok += r;
		s.d.row_seg += r;
		if (s.vec) s.vec += size_t(r) * g.ldv;
		if (s.x) s.x += size_t(r) * g.ldx;
		s.out += size_t(r) * g.ldo;
		if (s.norm_out) s.norm_out += size_t(r) * g.D;
		TG_TRY(n == 4 ? launch_gemv_r<4>(pro, epi, s, stream) : (n == 2 ? launch_gemv_r<2>(pro, epi, s, stream) : launch_gemv_r<1>(pro, epi, s, stream)));
		r += n;
	}
	return TG_OK;
}

WAttnArgs HybridState::attn_args(const StepDesc &d, int run, const void *p, int ldp, void *out, int ldo) {
	const Layer &L = m->layers[m->runs[run].layer];
	const RunCache &c = cache[run];
	WAttnArgs a{};
	a.d = d;
	a.H = L.at.H;
	a.G = L.at.G;
	a.dk = L.at.dk;
	a.dv = L.at.dv;
	a.dkp = L.at.dkp;
	a.dvp = L.at.dvp;
	a.scale = L.at.scale;
	a.window = L.at.window;
	a.keep = std::min(L.at.keep, c.keep_rows);
	a.r1 = L.r1;
	a.r2 = L.r2;
	a.p = p;
	a.ldp = ldp;
	a.p_q = L.p_q;
	a.p_k = L.p_k;
	a.p_v = L.p_v;
	a.p_g = L.p_g;
	a.kc = c.kc;
	a.vc = c.vc;
	a.ks = c.ks;
	a.vs = c.vs;
	a.cap = c.cap;
	a.keep_rows = c.keep_rows;
	a.out = out;
	a.ldo = ldo;
	a.out_scale = L.left_scale;
	a.part = part;
	a.tickets = tickets;
	a.nsplit = 1;
	a.err = err_flag;
	return a;
}

DeltaArgs HybridState::delta_args(const StepDesc &d, int run, const void *p, int ldp, void *out, int ldo) {
	const Layer &L = m->layers[m->runs[run].layer];
	const RunCache &c = cache[run];
	DeltaArgs a{};
	a.d = d;
	a.H = L.de.H;
	a.KH = L.de.KH;
	a.dk = L.de.dk;
	a.dv = L.de.dv;
	a.taps = L.de.taps;
	a.p = p;
	a.ldp = ldp;
	a.p_conv = L.p_conv;
	a.p_b = L.p_b;
	a.cw = L.conv;
	a.hist = c.conv;
	a.A_log = L.A_log;
	a.dt_bias = L.dt_bias;
	a.z = z;
	a.gz = gz;
	a.ldz = round_up(L.de.H * L.de.dk, 4);
	a.ldgz = round_up(L.de.H * L.de.dv, 4);
	a.S = c.S;
	a.norm = L.rnorm;
	a.eps = m->eps;
	a.out_scale = L.right_scale;
	a.out = out;
	a.ldo = ldo;
	a.o_col = L.o_col;
	a.ra = L.de.ra;
	a.rg = L.de.rg;
	a.p_a1 = L.p_a1;
	a.p_g1 = L.p_g1;
	a.a2 = L.a2.W;
	a.g2 = L.g2.W;
	a.lda2 = L.a2.ld;
	a.ldg2 = L.g2.ld;
	a.dkp = L.de.dkp();
	a.blk = blk;
	a.bV = bV;
	a.err = err_flag;
	a.o = o_raw;
	return a;
}

namespace {
template <typename PT, typename CT, typename OT> int launch_token_mix(const WAttnArgs &w, const DeltaArgs &d, int R, cudaStream_t st) {
	const size_t smem = std::max(wattn_token_smem(w.H / w.G, w.dkp, w.dvp), delta_token_smem(d.dk, d.dv, d.ra, d.rg));
	auto kernel = hybrid_token_mix_kernel<PT, CT, OT>;
	TG_TRY(allow_smem(kernel, smem));
	launch_k(kernel, dim3(w.G * w.nsplit + d.H, R), dim3(256), smem, st, w, d);
	count_launch();
	return check_launch("hybrid_token_mix");
}
template <int RPL, int NW, int NC> int launch_scan_nc(const DeltaArgs &a, int nseg, cudaStream_t st) {
	const int groups = (a.dv + 4 * NC - 1) / (4 * NC);
	// few CTAs: deep prefetch; many: more of them per SM
	int stages = (long long)groups * a.H * nseg <= 2 * g_num_sms ? 4 : 2;
	while (stages > 2 && delta_scan_smem<RPL, NW, NC>(stages) > 200 * 1024) stages--;
	const size_t smem = delta_scan_smem<RPL, NW, NC>(stages);
	auto kernel = delta_scan_kernel<RPL, NW, NC>;
	TG_TRY(allow_smem(kernel, smem));
	launch_k(kernel, dim3(groups, a.H, nseg), dim3(32 * NW), smem, st, a, stages);
	count_launch();
	return check_launch("delta_scan");
}
// columns per lane: one while every SM gets at most one CTA, more (fewer shared-memory reads per column) beyond
template <int RPL, int NW> int launch_scan(const DeltaArgs &a, int nseg, cudaStream_t st) {
	static const int forced = env_int("TG_SCAN_COLS", 0);
	const long long cols = (long long)a.dv * a.H * nseg;
	const int nc = forced ? forced : (cols <= 4 * g_num_sms ? 1 : (cols <= 40 * g_num_sms ? 2 : 4));
	if (nc == 1) return launch_scan_nc<RPL, NW, 1>(a, nseg, st);
	if (nc == 2) return launch_scan_nc<RPL, NW, 2>(a, nseg, st);
	return launch_scan_nc<RPL, NW, 4>(a, nseg, st);
}
template <typename PT> int launch_delta(const DeltaArgs &a, int R, int nseg, int max_len, cudaStream_t st) {
	const size_t smem = delta_block_smem(a.dkp, a.dv);
	TG_TRY(allow_smem(delta_block_kernel<PT>, smem));
	launch_k(delta_block_kernel<PT>, dim3((max_len + DB - 1) / DB, a.H, nseg), dim3(256), smem, st, a);
	count_launch();
	TG_TRY(check_launch("delta_block"));
	switch (a.dkp) {
		case 32: TG_TRY((launch_scan<4, 1>(a, nseg, st))); break;
		case 64: TG_TRY((launch_scan<4, 2>(a, nseg, st))); break;
		case 128: TG_TRY((launch_scan<4, 4>(a, nseg, st))); break;
		default: TG_TRY((launch_scan<8, 4>(a, nseg, st))); break;
	}
	launch_k(delta_out_kernel<PT>, dim3((R * a.H + 7) / 8), dim3(256), 0, st, a, R);
	count_launch();
	return check_launch("delta_out");
}
template <typename PT> int launch_ln_conv(void *out, int ldo, const float *x, int ldx, float2 *stats, const float *w, const float *cw, float *hist,
                                          const StepDesc &d, int R, int D, int taps, float eps, cudaStream_t st) {
	launch_k(ln_stats_kernel, dim3(R), dim3(128), 0, st, stats, x, ldx, D, eps);
	count_launch();
	TG_TRY(check_launch("ln_stats"));
	const int cols = (ldo + 511) / 512;
	int rows = LC_ROWS;
	while (rows > 1 && (R + rows - 1) / rows * cols < 4 * g_num_sms) rows /= 2;
	const dim3 grid((R + rows - 1) / rows, cols);
	if (taps <= 4) launch_k(ln_conv_kernel<PT, 4>, grid, dim3(128), 0, st, static_cast<PT *>(out), ldo, x, ldx, stats, w, cw, hist, d, R, D, taps, rows);
	else launch_k(ln_conv_kernel<PT, 16>, grid, dim3(128), 0, st, static_cast<PT *>(out), ldo, x, ldx, stats, w, cw, hist, d, R, D, taps, rows);
	count_launch();
	return check_launch("ln_conv");
}
template <typename PT> int launch_ln(void *out, int ldo, const float *x, int ldx, const float *w, const int *rows, int n, int D, float eps, float *out32,
                                     cudaStream_t st) {
	launch_k(layer_norm_kernel<PT>, dim3(n), dim3(128), 0, st, static_cast<PT *>(out), ldo, x, ldx, w, rows, n, D, eps, out32);
	count_launch();
	return check_launch("layer_norm");
}
// portions on CUDA cores
template <typename PT> int launch_attn_simt(const WAttnArgs &a, int R, cudaStream_t st) {
	const size_t smem = size_t(4) * (a.dkp + a.dvp) * 4;
	TG_TRY(allow_smem(window_attn_kernel<PT, PT>, smem));
	launch_k(window_attn_kernel<PT, PT>, dim3((R * a.H + 3) / 4), dim3(128), smem, st, a, R);
	count_launch();
	return check_launch("window_attn");
}
}  // namespace

// All layers for R rows in nseg segments (the longest: max_len), leaving the residual stream in x.
int HybridState::run_layers(const StepDesc &d, int R, int nseg, int max_len) {
	const bool single = max_len == 1, few = single && R <= FEW_ROWS;
	const int D = m->D;
	auto embed_rows = [&](int add) -> int {
		launch_k(embed_rows_kernel, dim3(R), dim3(256), 0, stream, x, ldx, m->embed.W, m->embed.ld, d, D, m->n_vocab, add, err_flag);
		count_launch();
		return check_launch("embed_rows");
	};
	if (!few) TG_TRY(embed_rows(0));
	for (size_t run = 0; run < m->runs.size(); run++) {
		const Layer &L = m->layers[m->runs[run].layer];
		const int li = m->runs[run].layer;
		const RunCache &c = cache[run];
		if (few) {
			GemvArgs g{};
			g.d = d;
			g.x = x;
			g.ldx = ldx;
			g.D = D;
			g.embed = m->embed.W;
			g.lde = m->embed.ld;
			g.V = m->n_vocab;
			g.eps = m->eps;
			g.cw = L.canon;
			g.hist = c.canon;
			g.taps = m->taps;
			const int embed_mode = run == 0 ? 1 : (m->runs[run].add_embed ? 2 : 0);
			auto product = [&](int pro, int epi, const Lin &w, const float *norm, const float *vec, int ldv, float *out, int ldo, int em) -> int {
				GemvArgs s = g;
				s.W = w.W;
				s.ldw = w.ld;
				s.N = w.N;
				s.K = w.K;
				s.w = norm;
				s.vec = vec;
				s.ldv = ldv;
				s.out = out;
				s.ldo = ldo;
				s.embed_mode = em;
				if (epi == GV_PROJ) {
					s.p_k = L.p_k;
					s.n_k = L.at.G * L.at.dkp;
					s.p_v = L.p_v;
					s.n_v = L.at.G * L.at.dvp;
					s.kc = c.kc;
					s.vc = c.vc;
					s.ks = c.ks;
					s.vs = c.vs;
					s.cap_rows = c.cap;
					s.keep = std::min(L.at.keep, c.keep_rows);
					s.keep_rows = c.keep_rows;
					s.cache_f32 = f32;
				}
				return gemv(pro, epi, s, R);
			};
			TG_TRY(product(GV_LN_CONV, GV_PROJ, L.proj, L.norm1, nullptr, 0, P32, L.ldp, embed_mode));
			WAttnArgs wa = attn_args(d, int(run), P32, L.ldp, O32, L.kc);
			const DeltaArgs da = delta_args(d, int(run), P32, L.ldp, O32, L.kc);
			const long long keys = std::min<long long>((long long)wa.window + wa.keep, max_pos_global);
			wa.nsplit = int(std::max<long long>(1, std::min<long long>(nsplit_cap, (keys + WK_KEYS - 1) / WK_KEYS)));
			if (f32) TG_TRY((launch_token_mix<float, float, float>(wa, da, R, stream)));
			else TG_TRY((launch_token_mix<float, bf16, float>(wa, da, R, stream)));
			TG_TRY(product(GV_VEC, GV_ADD, L.out, nullptr, O32, L.kc, x, ldx, embed_mode));
			if (L.ff) {
				TG_TRY(product(GV_LN, GV_GEGLU, L.gu, L.norm2, nullptr, 0, act32, L.ffp, 0));
				TG_TRY(product(GV_VEC, GV_ADD, L.down, nullptr, act32, L.ffp, x, ldx, 0));
			}
		} else {
			if (m->runs[run].add_embed) TG_TRY(embed_rows(1));
			if (f32) TG_TRY(launch_ln_conv<float>(h, m->Dp, x, ldx, stats, L.norm1, L.canon, c.canon, d, R, D, m->taps, m->eps, stream));
			else TG_TRY(launch_ln_conv<bf16>(h, m->Dp, x, ldx, stats, L.norm1, L.canon, c.canon, d, R, D, m->taps, m->eps, stream));
			TG_TRY(gemm(GEMM_STORE, h, m->Dp, &hmap, L.proj, R, P, L.ldp));
			WAttnArgs wa = attn_args(d, int(run), P, L.ldp, O, L.kc);
			const DeltaArgs da = delta_args(d, int(run), P, L.ldp, O, L.kc);
			if (f32) launch_k(kv_append_kernel<float, float>, dim3(R), dim3(256), 0, stream, wa);
			else launch_k(kv_append_kernel<bf16, bf16>, dim3(R), dim3(256), 0, stream, wa);
			count_launch();
			TG_TRY(check_launch("kv_append"));
			if (single) {
				const long long keys = std::min<long long>((long long)wa.window + wa.keep, max_pos_global);
				const int fill = std::max(1, 2 * g_num_sms / std::max(1, R * wa.G));
				wa.nsplit = int(std::max<long long>(1, std::min<long long>(std::min(nsplit_cap, fill), (keys + WK_KEYS - 1) / WK_KEYS)));
				if (f32) TG_TRY((launch_token_mix<float, float, float>(wa, da, R, stream)));
				else TG_TRY((launch_token_mix<bf16, bf16, bf16>(wa, da, R, stream)));
			} else {
				static const int use_tc = env_int("TG_WATTN_TC", 1);
				if (!f32 && use_tc && wa.dkp <= 256 && wa.dvp <= 256) {
					const WtShape sh = wt_shape(wa.dkp, wa.dvp, wa.window);
					TG_TRY(allow_smem(window_attn_tc_kernel, sh.total));
					launch_k(window_attn_tc_kernel, dim3((max_len + 127) / 128, wa.H, nseg), dim3(WT_THREADS), size_t(sh.total), stream, pmap[li], c.kmap, c.vmap,
					         c.ksmap, c.vsmap, wa);
					count_launch();
					TG_TRY(check_launch("window_attn_tc"));
				} else {
					if (f32) TG_TRY(launch_attn_simt<float>(wa, R, stream));
					else TG_TRY(launch_attn_simt<bf16>(wa, R, stream));
				}
				const size_t esz = f32 ? 4 : 2;
				const uint8_t *pb = static_cast<const uint8_t *>(P);
				TG_TRY(gemm(GEMM_STORE32, pb + size_t(L.p_a1) * esz, L.ldp, f32 ? nullptr : &a1map[li], L.a2, R, z, da.ldz));
				TG_TRY(gemm(GEMM_STORE32, pb + size_t(L.p_g1) * esz, L.ldp, f32 ? nullptr : &g1map[li], L.g2, R, gz, da.ldgz));
				if (f32) TG_TRY(launch_delta<float>(da, R, nseg, max_len, stream));
				else TG_TRY(launch_delta<bf16>(da, R, nseg, max_len, stream));
			}
			TG_TRY(gemm(GEMM_ADD, O, L.kc, f32 ? nullptr : &omap[li], L.out, R, x, ldx));
			if (L.ff) {
				if (f32) TG_TRY(launch_ln<float>(h, m->Dp, x, ldx, L.norm2, nullptr, R, D, m->eps, nullptr, stream));
				else TG_TRY(launch_ln<bf16>(h, m->Dp, x, ldx, L.norm2, nullptr, R, D, m->eps, nullptr, stream));
				TG_TRY(gemm(GEMM_GEGLU, h, m->Dp, &hmap, L.gu, R, act, L.ffp));
				TG_TRY(gemm(GEMM_ADD, act, L.ffp, f32 ? nullptr : &amap[li], L.down, R, x, ldx));
			}
		}
		if (tracing) {
			const size_t at = trace.size();
			trace.resize(at + size_t(R) * D);
			TG_CUDA(cudaMemcpy2DAsync(trace.data() + at, size_t(D) * 4, x, size_t(ldx) * 4, size_t(D) * 4, R, cudaMemcpyDeviceToHost, stream));
			TG_CUDA(cudaStreamSynchronize(stream));
		}
	}
	return TG_OK;
}

// logits of n rows of x (rows_dev: which; null: 0 .. n-1) -> out [n][ld_logits]
int HybridState::score_rows(const int *rows_dev, int n, float *out, float *norm_out) {
	if (f32) TG_TRY(launch_ln<float>(hn, m->Dp, x, ldx, m->final_norm, rows_dev, n, m->D, m->eps, norm_out, stream));
	else TG_TRY(launch_ln<bf16>(hn, m->Dp, x, ldx, m->final_norm, rows_dev, n, m->D, m->eps, norm_out, stream));
	return gemm(GEMM_LOGITS, hn, m->Dp, &hnmap, m->embed, n, out, ld_logits, m->softcap);
}

// ------------------------------------------------------------------ lock-step decoding
int HybridState::enqueue_decode_all() {
	const StepDesc d = lockstep_desc();
	TG_TRY(run_layers(d, B, B, 1));
	if (B <= FEW_ROWS) {
		GemvArgs g{};
		g.d = d;
		g.x = x;
		g.ldx = ldx;
		g.D = m->D;
		g.W = m->embed.W;
		g.ldw = m->embed.ld;
		g.N = m->embed.N;
		g.K = m->embed.K;
		g.w = m->final_norm;
		g.eps = m->eps;
		g.taps = 1;
		g.out = logits;
		g.ldo = ld_logits;
		g.norm_out = xnorm;
		g.cap = m->softcap;
		TG_TRY(gemv(GV_LN, GV_LOGITS, g, B));
	} else {
		TG_TRY(score_rows(nullptr, B, logits, xnorm));
	}
	launch_k(hybrid_advance_kernel, dim3((B + 255) / 256), dim3(256), 0, stream, ls_pos, ls_par, B);
	count_launch();
	return check_launch("hybrid_advance");
}

int HybridState::enqueue_forward() {
	TG_TRY(sync_lockstep());
	if (tracing) {
		trace.clear();
		trace_rows = B;
		TG_TRY(enqueue_decode_all());
	} else {
		TG_TRY(enqueue_decode_step());
	}
	for (int &p : host_par) p ^= 1;
	return TG_OK;
}

int HybridState::run_steps(int n_steps, float minp, float temp) {
	TG_TRY(sync_lockstep());
	TG_TRY(tg_state::run_steps(n_steps, minp, temp));
	if (n_steps & 1)
		for (int &p : host_par) p ^= 1;
	return TG_OK;
}

// ------------------------------------------------------------------ portions
int HybridState::run_entries(std::vector<Entry> &es, bool last, float *logits_host) {
	TG_CUDA(cudaStreamSynchronize(stream));
	staging_busy = false;
	trace.clear();
	trace_rows = 0;
	ls_dirty = true;
	for (;;) {
		// a pass: what fits of every entry that has tokens left
		int R = 0, nseg = 0, max_len = 0;
		int *tk = desc_pin, *rs = tk + max_rows, *sg = rs + max_rows;
		struct Out {
			size_t entry;
			int row;
			size_t out;
		};
		std::vector<Out> outs;
		for (size_t e = 0; e < es.size(); e++) {
			Entry &E = es[e];
			const int n = std::min(std::min(E.count - E.done, max_seq_rows), max_rows - R);
			if (n <= 0) continue;
			for (int i = 0; i < n; i++) {
				tk[R + i] = E.ids[E.done + i];
				rs[R + i] = nseg;
			}
			sg[nseg] = E.seq;
			sg[B + nseg] = R;
			sg[2 * B + nseg] = n;
			sg[3 * B + nseg] = host_pos[E.seq];
			sg[4 * B + nseg] = host_par[E.seq];
			if (last) {
				if (E.done + n == E.count) outs.push_back({e, R + n - 1, size_t(E.seq)});
			} else {
				for (size_t w = 0; w < E.want.size(); w++)
					if (E.want[w] >= E.done && E.want[w] < E.done + n) outs.push_back({e, R + E.want[w] - E.done, E.out0 + w});
			}
			host_pos[E.seq] += n;
			host_par[E.seq] ^= 1;
			E.done += n;
			R += n;
			nseg++;
			max_len = std::max(max_len, n);
		}
		if (R == 0) break;
		TG_CUDA(cudaMemcpyAsync(desc, desc_pin, desc_ints * 4, cudaMemcpyHostToDevice, stream));
		StepDesc d;
		d.tok = desc;
		d.row_seg = desc + max_rows;
		d.seg_seq = desc + 2 * size_t(max_rows);
		d.seg_row = d.seg_seq + B;
		d.seg_len = d.seg_seq + 2 * B;
		d.seg_pos = d.seg_seq + 3 * B;
		d.seg_par = d.seg_seq + 4 * B;
		trace_rows += R;
		TG_TRY(run_layers(d, R, nseg, max_len));
		for (size_t i = 0; i < outs.size();) {
			// a run of consecutive output rows
			std::vector<int> rows{outs[i].row};
			while (i + rows.size() < outs.size() && rows.size() < size_t(wl_rows) && outs[i + rows.size()].out == outs[i].out + rows.size())
				rows.push_back(outs[i + rows.size()].row);
			const int n = int(rows.size());
			TG_CUDA(cudaMemcpyAsync(want_dev, rows.data(), size_t(n) * 4, cudaMemcpyHostToDevice, stream));
			if (last) {
				TG_TRY(score_rows(want_dev, n, logits + outs[i].out * ld_logits, xnorm + outs[i].out * m->D));
			} else {
				TG_TRY(score_rows(want_dev, n, wl, nullptr));
				const size_t row = size_t(m->n_vocab) * 4;
				TG_CUDA(cudaMemcpy2DAsync(logits_host + outs[i].out * m->n_vocab, row, wl, size_t(ld_logits) * 4, row, n, cudaMemcpyDeviceToHost, stream));
			}
			i += size_t(n);
		}
		TG_TRY(check_err_flag());  // synchronises: the pinned descriptors may be rewritten
	}
	if (last && logits_host) {
		TG_TRY(read_logits(logits_host));
		TG_CUDA(cudaStreamSynchronize(stream));
	}
	return TG_OK;
}

int HybridState::prefill(const int *ids, int S, float *logits_host) {
	for (long long i = 0; i < (long long)B * S; i++)
		if (ids[i] < 0 || ids[i] >= m->n_vocab) return fail(TG_EINVAL, "token id out of range");
	std::vector<Entry> es(B);
	for (int b = 0; b < B; b++) {
		es[b].seq = b;
		es[b].count = S;
		es[b].done = 0;
		es[b].ids = ids + size_t(b) * S;
		es[b].out0 = 0;
	}
	return run_entries(es, true, logits_host);
}

int HybridState::append(const int *ids, int n, float *logits_host) {
	std::vector<Entry> es(1);
	es[0].seq = 0;
	es[0].count = n;
	es[0].done = 0;
	es[0].ids = ids;
	es[0].out0 = 0;
	return run_entries(es, true, logits_host);
}

int HybridState::step(int n, const int *seq, const int *count, const int *ids, const int *n_want, const int *want, float *logits_host) {
	std::vector<Entry> es(n);
	std::vector<char> used(B, 0);
	size_t at = 0, out = 0;
	bool in_order = n == B;
	for (int e = 0; e < n; e++) {
		Entry &E = es[e];
		if (seq[e] < 0 || seq[e] >= B || used[seq[e]]) return fail(TG_EINVAL, "tg_step: bad or repeated sequence");
		if (count[e] < 1) return fail(TG_EINVAL, "tg_step: an entry without tokens");
		used[seq[e]] = 1;
		if (count[e] > max_pos_global - host_pos[seq[e]]) return fail(TG_ESTATE, "cache full (max_pos_global reached)");
		E.seq = seq[e];
		E.count = count[e];
		E.done = 0;
		E.ids = ids + at;
		for (int i = 0; i < count[e]; i++)
			if (E.ids[i] < 0 || E.ids[i] >= m->n_vocab) return fail(TG_EINVAL, "token id out of range");
		E.out0 = out;
		for (int w = 0; n_want && w < n_want[e]; w++) {
			const int p = want[out + w];
			if (p < 0 || p >= count[e]) return fail(TG_EINVAL, "tg_step: a wanted place outside the entry");
			E.want.push_back(p);
		}
		at += count[e];
		out += E.want.size();
		in_order = in_order && seq[e] == e && count[e] == 1;
	}
	if (out && !logits_host) return fail(TG_EINVAL, "tg_step: no buffer for the logits");
	if (!in_order) return run_entries(es, false, logits_host);
	// one token for every sequence: the decode step of the generation loop
	TG_TRY(staging_acquire());
	std::memcpy(host_pin, ids, 4 * size_t(B));
	TG_CUDA(cudaMemcpyAsync(tok, host_pin, 4 * size_t(B), cudaMemcpyHostToDevice, stream));
	TG_TRY(enqueue_forward());
	for (int b = 0; b < B; b++) {
		host_pos[b] += 1;
		for (size_t w = 0; w < es[b].want.size(); w++)
			TG_CUDA(cudaMemcpyAsync(logits_host + (es[b].out0 + w) * m->n_vocab, logits + size_t(b) * ld_logits, size_t(m->n_vocab) * 4, cudaMemcpyDeviceToHost, stream));
	}
	return check_err_flag();
}
