// pavitar.cu — the Pavitar family of the model registry (family.h): a pre-norm decoder described by a config.json whose layers each carry one
// softmax mixer that forgets — latent attention in a sliding window, or grouped-query attention inside fixed chunks of positions — and a mixture
// of experts, and which runs a stretch of its layers several times with the same weights.
//
//   embedding                 token row x_0
//   layer                     x <- x + mixer(n1(x)), x <- x + mixture(n2(x)), n(x) = x / rms(x) (1 + w)
//   mixer "latent_attention"  c = rmsnorm(W_dkv h) is all the cache keeps; k_h = W_uk,h c, v_h = W_uv,h c; q = W_uq rmsnorm(W_dq h); no positions;
//                             position i sees the `mask.size` positions up to itself; one sigmoid gate per head; W_o
//   mixer "attention"         H query heads over G key/value heads; RMS norm of the whole q row and the whole k row, then rotary positions on
//                             neighbouring entries (2i, 2i + 1) of the first `rot.dims` of every head; position i sees the positions up to itself that
//                             lie in its own run of `mask.size`, counted from position 0; W_o
//   mixture                   the `top` largest logits W_router h + b are chosen and weighted by the softmax over the chosen; an expert is
//                             W_down (silu(W_gate h) . W_up h); a shared expert runs for every token, times sigmoid(w_sg h)
//   loop                      layers start .. stop - 1 run `times` times, every pass with a cache of its own, and every pass but the first begins
//                             with x <- x + x_0
//   output                    norm, logits = cap tanh((embedding table . row) / cap)
//
// The step function, graph replay of one-token steps, uploads, release and the C entry points are the shared sequence engine's (seq_family.cuh),
// the latent mixer's kernels in order are seq_latent.cuh's, the mixture's seq_moe.cuh's.  Per pass and layer run here:
//     norm (with x_0 added first where a pass over the loop begins: one kernel)
//     latent:     rows product [dq | dkv | g] -> latent_attention (absorbed form, window ring, head gate fused)
//     attention:  rows product [q | k | v] -> qkv_rows_post (row norms, rotation, cache rows) -> swa_attn / swa_tile with the chunk mask
//     rows product [o] with the residual add fused
//     norm -> router (with the shared expert's gate) and sort on the side stream beside the shared expert on the main one -> experts ->
//     moe_combine (+ gated shared row + residual)
//
// Cache / state manager: per layer RUN a ring of mask.size - 1 + seq_chunk rows (at most max_tokens): latents, or normed and turned keys and
// values.  Rows need no clearing: a sequence only reads positions it wrote.
//
// Precision: the residual stream, norms, angles, scores, softmax, router, gates and every sum are fp32 in both modes.  XALM_PRECISION_BF16 keeps
// matrices and caches in bf16 and sends dense products of long passes through the tcgen05 GEMM (fp16 operands, fp32 accumulation);
// XALM_PRECISION_F32 widens both and uses the fp32 FMA kernels only.
#include "seq_family.cuh"

#include "seq_latent.cuh"
#include "seq_moe.cuh"

namespace xalm {
namespace {

using namespace mix;
using namespace seq;

struct Layer { // weights and sizes; what a sequence holds lives in Run
	bool latent = false;
	LatentWeights lat;
	// attention
	int H = 0, G = 0, d = 0, dv = 0, rot_dims = 0;
	int reach = 0x7fffffff; // mask.size: the latent window, or the chunk of the attention; 0x7fffffff: everything before
	float scale = 1.f;
	std::vector<float> freq_host;
	float *freq = nullptr, *q_norm = nullptr, *k_norm = nullptr;
	int off_k = 0, off_v = 0, n_in = 0; // columns of the stacked projection [q | k | v]
	void *w_in = nullptr, *w_o = nullptr;
	WMat m_in, m_o;
	TcWeight t_in, t_o;
	float *norm1 = nullptr, *norm2 = nullptr;
	bool has_moe = false;
	MoeWeights moe;
	long long bytes = 0, expert_bytes = 0; // what one run of the layer reads of its matrices; of that, one expert's share
	int chunk() const { return reach < 0x7fffffff ? reach : 0; }
};

struct Run { // one execution of a layer within a pass: the sequence's cache there
	int layer = 0;
	bool again = false; // begins a pass over the loop other than the first
	LatentCache lat;
	void *kc = nullptr, *vc = nullptr; // (ring, G * d) finished keys, (ring, G * dv) values
	int ring = 0;
};

struct PavitarModel : SeqModel {
	float logit_cap = 0.f;
	bool loops = false;
	std::vector<Layer> layers;
	std::vector<Run> runs;
	// one pass: the residual stream before and behind the embedded rows, so that either neighbour and x_0 are two "streams" of one norm
	float *x = nullptr, *x0 = nullptr, *x2 = nullptr, *hn = nullptr, *proj = nullptr, *q = nullptr, *att = nullptr;
	int proj_ld = 4;
	LatentBuffers lat;
	AttnParts parts;
	MoeBuffers moe;
};
typedef PavitarModel Pv;

// ---- config.json ------------------------------------------------------------------------------------------------------------------
int parse_mixer(Pv* m, size_t li, const std::string& p, const std::string& type, const xjson::Value& mx, Layer* L) {
	const int W = m->width;
	L->H = geti(mx, "heads");
	L->d = geti(mx, "dim");
	L->dv = mx.contains("vdim") ? geti(mx, "vdim") : L->d;
	if (L->H <= 0 || L->d <= 0 || L->dv <= 0) return set_error(XALM_ERR_INVALID, "config: layer %zu: %d heads of %d and %d", li, L->H, L->d, L->dv);
	L->scale = mx.contains("scale") ? (float) getf(mx, "scale") : 1.f / sqrtf((float) L->d);
	if (const xjson::Value* mk = object_or_null(mx, "mask")) {
		L->reach = geti(*mk, "size");
		if (L->reach <= 0) return set_error(XALM_ERR_INVALID, "config: layer %zu: mask of %d positions", li, L->reach);
	}
	if (type == "latent_attention") {
		L->latent = true;
		LatentWeights& A = L->lat;
		A.H = L->H; A.d = L->d; A.dv = L->dv;
		A.R = geti(mx, "kv_rank");
		A.Rq = geti(mx, "q_rank");
		if (A.R <= 0 || A.Rq <= 0) return set_error(XALM_ERR_INVALID, "config: layer %zu: latent sizes %d and %d", li, A.R, A.Rq);
		A.gate = LATENT_GATE_HEADS;
		A.window = L->reach;
		A.scale = L->scale;
		latent_expect(m, p + "mix.", A);
	} else if (type == "attention") {
		L->G = mx.contains("kv_heads") ? geti(mx, "kv_heads") : L->H;
		if (L->G <= 0 || L->H % L->G) return set_error(XALM_ERR_INVALID, "config: layer %zu: %d query heads over %d key/value heads", li, L->H, L->G);
		if (const xjson::Value* rt = object_or_null(mx, "rot")) {
			L->rot_dims = geti(*rt, "dims");
			if (L->rot_dims < 0 || L->rot_dims > L->d || L->rot_dims % 2) return set_error(XALM_ERR_INVALID, "config: layer %zu: %d rotary dimensions in a head of %d", li, L->rot_dims, L->d);
			if (L->rot_dims) L->freq_host = rotary_frequencies(getf(*rt, "base"), L->rot_dims);
		}
		expect(m, p + "mix.q", {L->H * L->d, W}, true);
		expect(m, p + "mix.k", {L->G * L->d, W}, true);
		expect(m, p + "mix.v", {L->G * L->dv, W}, true);
		expect(m, p + "mix.q.norm", {L->H * L->d}, false);
		expect(m, p + "mix.k.norm", {L->G * L->d}, false);
	} else return set_error(XALM_ERR_UNSUPPORTED, "config: layer %zu has mixer type '%s' (this family runs 'latent_attention' and 'attention')", li, type.c_str());
	expect(m, p + "mix.o", {W, L->H * L->dv}, true);
	return XALM_OK;
}

int parse_mixture(Pv* m, size_t li, const std::string& p, const xjson::Value& mlp, Layer* L) {
	const std::string kind = mlp.contains("kind") ? mlp.at("kind").str : "moe";
	if (kind != "moe") return set_error(XALM_ERR_UNSUPPORTED, "config: layer %zu has feed-forward kind '%s' (this family runs 'moe')", li, kind.c_str());
	L->has_moe = true;
	MoeWeights& e = L->moe;
	const xjson::Value& r = mlp.at("router");
	e.ff = geti(mlp.at("expert"), "ff");
	e.E = geti(r, "experts");
	e.top = geti(r, "top");
	if (e.ff <= 0 || e.E <= 0 || e.top <= 0 || e.top > e.E) return set_error(XALM_ERR_INVALID, "config: layer %zu: %d of %d experts of %d", li, e.top, e.E, e.ff);
	expect(m, p + "norm2", {m->width}, false);
	moe_expect(m, p + "mlp.", e.E, e.ff, true);
	expect(m, p + "mlp.router", {e.E, m->width}, true);
	expect(m, p + "mlp.router.b", {e.E}, false);
	if (const xjson::Value* sh = object_or_null(mlp, "shared")) {
		const int sff = geti(*sh, "ff");
		if (sff <= 0) return set_error(XALM_ERR_INVALID, "config: layer %zu: shared expert of %d", li, sff);
		moe_expect_shared(m, p + "mlp.shared.", &e, sff, true);
	}
	return XALM_OK;
}

int parse_config(SeqModel* sm, const char* json) {
	Pv* m = static_cast<Pv*>(sm);
	try {
		const xjson::Value c = xjson::Parser::parse(json, strlen(json));
		m->vocab = geti(c, "vocab");
		m->width = geti(c, "width");
		if (m->vocab <= 0 || m->width <= 0) return set_error(XALM_ERR_INVALID, "config: vocab / width must be positive");
		if (const xjson::Value* nv = object_or_null(c, "norm"); nv && nv->contains("eps")) m->eps = (float) getf(*nv, "eps");
		if (const xjson::Value* lc = c.find("logit_softcap"); lc && lc->kind == xjson::Value::Number) m->logit_cap = (float) lc->num;
		expect(m, "embed", {m->vocab, m->width}, true);
		const xjson::Value& layers = c.at("layers");
		if (layers.kind != xjson::Value::Array || layers.arr.empty()) return set_error(XALM_ERR_INVALID, "config: no layers");
		for (size_t li = 0; li < layers.arr.size(); li++) {
			const xjson::Value& lv = layers.arr[li];
			const std::string p = "l" + std::to_string(li) + ".";
			Layer L;
			expect(m, p + "norm1", {m->width}, false);
			XALM_TRY(parse_mixer(m, li, p, lv.at("type").str, lv.at("mixer"), &L));
			if (const xjson::Value* mlp = object_or_null(lv, "mlp")) XALM_TRY(parse_mixture(m, li, p, *mlp, &L));
			m->layers.push_back(std::move(L));
		}
		std::vector<LayerRun> order;
		XALM_TRY(layer_order(c, (int) m->layers.size(), &order));
		for (const LayerRun& r : order) {
			Run R;
			R.layer = r.layer;
			R.again = r.pass > 1;
			m->loops = m->loops || R.again;
			m->runs.push_back(R);
		}
		m->n_layers = (int) m->runs.size(); // what read_state counts: layer runs
		expect(m, "final.norm", {m->width}, false);
	} catch (const std::exception& e) {
		return set_error(XALM_ERR_INVALID, "config.json: %s", e.what());
	}
	return XALM_OK;
}

// ---- the kernels of one pass ----------------------------------------------------------------------------------------------------------
// row norms, rotation, cache rows, attention: proj -> att
int enqueue_attention(Pv* m, const Layer& L, const Run& R, int n, int* nl) {
	const bool f32 = m->precision == XALM_PRECISION_F32;
	cudaStream_t s = m->stream;
	QkvPostArgs qa = {};
	qa.proj = m->proj; qa.ld = m->proj_ld; qa.q_off = 0; qa.k_off = L.off_k; qa.v_off = L.off_v;
	qa.H = L.H; qa.G = L.G; qa.d = L.d; qa.dv = L.dv;
	qa.freq = L.freq; qa.rot_half = L.rot_dims / 2; qa.rot_neighbours = 1;
	qa.norm_rows = 1; qa.q_norm_w = L.q_norm; qa.k_norm_w = L.k_norm; qa.eps = m->eps;
	qa.q_out = m->q; qa.ldq_out = L.H * L.d;
	qa.kc = R.kc; qa.vc = R.vc; qa.cache_f32 = f32; qa.keep_first = 0; qa.ring = R.ring;
	qa.step = m->d_step;
	XALM_TRY(launch_qkv_post(qa, n, s));
	(*nl)++;
	SwaArgs sa = {};
	sa.q = m->q; sa.ldq = L.H * L.d; sa.q_off = 0;
	sa.kc = R.kc; sa.vc = R.vc; sa.ring = R.ring; sa.keep_first = 0;
	sa.H = L.H; sa.G = L.G; sa.d = L.d; sa.dv = L.dv;
	sa.window = 0x7fffffff; sa.mask_chunk = L.chunk(); sa.scale = L.scale;
	sa.step = m->d_step; sa.out = m->att;
	m->parts.use(&sa);
	int launches = 1;
	XALM_TRY(launch_swa(sa, n, f32, s, &launches));
	*nl += launches;
	return XALM_OK;
}

int enqueue_pass(SeqModel* sm, int n, int want, int* nl) {
	Pv* m = static_cast<Pv*>(sm);
	cudaStream_t s = m->stream;
	const int W = m->width;
	const size_t hs = (size_t) m->chunk * W;
	float* x = m->x;
	const int copies = m->loops ? 2 : 1; // the residual stream, and x_0 for the passes to come
	if (m->w_bf16) embed_streams_kernel<__nv_bfloat16><<<n, norm_threads(W), 0, s>>>((const __nv_bfloat16*) m->embed, m->d_tokens, W, copies, hs, x);
	else embed_streams_kernel<float><<<n, norm_threads(W), 0, s>>>((const float*) m->embed, m->d_tokens, W, copies, hs, x);
	XALM_SEQ_LAUNCH_CHECK("embed");
	for (size_t ri = 0; ri < m->runs.size(); ri++) {
		const Run& R = m->runs[ri];
		const Layer& L = m->layers[(size_t) R.layer];
		if (R.again) { // x <- x + x_0, into the buffer on the other side of x_0, and its norm
			float* to = x == m->x ? m->x2 : m->x;
			XALM_TRY(launch_hc_norm(std::min(x, m->x0), 2, hs, nullptr, L.norm1, 1, m->eps, W, m->hn, to, n, s));
			x = to;
		} else XALM_TRY(launch_hc_norm(x, 1, hs, nullptr, L.norm1, 1, m->eps, W, m->hn, nullptr, n, s));
		(*nl)++;
		RowsEpi est;
		est.kind = EPI_STORE; est.out = m->proj; est.ldo = m->proj_ld;
		if (L.latent) {
			XALM_TRY(rows_product(m, m->hn, W, L.lat.w_in, &L.lat.t_in, n, L.lat.n_in, W, est, nl));
			XALM_TRY(latent_attention(m, L.lat, R.lat, m->lat, m->parts, m->proj, m->proj_ld, m->att, n, nl));
		} else {
			XALM_TRY(rows_product(m, m->hn, W, L.w_in, &L.t_in, n, L.n_in, W, est, nl));
			XALM_TRY(enqueue_attention(m, L, R, n, nl));
		}
		RowsEpi eo; // x <- x + product
		eo.kind = EPI_HC; eo.xs = x; eo.S = 1; eo.stream_stride = hs;
		XALM_TRY(rows_product(m, m->att, L.H * L.dv, L.w_o, &L.t_o, n, W, L.H * L.dv, eo, nl));
		if (L.has_moe) {
			XALM_TRY(launch_hc_norm(x, 1, hs, nullptr, L.norm2, 1, m->eps, W, m->hn, nullptr, n, s));
			MoeRouteArgs ra = {};
			ra.score_kind = MOE_SCORE_CHOSEN;
			RowsEpi eg;
			eg.kind = EPI_GLU; eg.glu_act = GLU_SILU;
			MoeCombineArgs ca = {};
			ca.x_in = x; ca.x_out = x;
			XALM_TRY(moe_experts(m, L.moe, m->moe, m->hn, n, ra, eg, &ca, nl, tune("seq_overlap") != 0));
			XALM_TRY(launch_moe_combine(ca, n, s));
			*nl += 2;
		}
		if (m->keep_layers) XALM_CUDA_CHECK(cudaMemcpyAsync(m->layer_sums + ri * hs, x, (size_t) n * W * 4, cudaMemcpyDeviceToDevice, s));
	}
	if (want) {
		const int rows = want == 2 ? n : 1, first = want == 2 ? 0 : n - 1;
		XALM_TRY(launch_hc_norm(x + (size_t) first * W, 1, hs, nullptr, m->final_norm, 1, m->eps, W, m->hn, nullptr, rows, s));
		(*nl)++;
		RowsEpi eh;
		eh.kind = EPI_STORE; eh.out = m->logits; eh.ldo = m->vocab; eh.cap = m->logit_cap;
		XALM_TRY(rows_product(m, m->hn, W, m->w_head, &m->t_head, rows, m->vocab, W, eh, nl));
	}
	return XALM_OK;
}

// ---- device layouts, cache, pass buffers ---------------------------------------------------------------------------------------------
int finalize(SeqModel* sm) {
	Pv* m = static_cast<Pv*>(sm);
	const int W = m->width;
	const size_t C = (size_t) m->chunk, kelem = m->precision == XALM_PRECISION_F32 ? 4 : 2;
	auto T = [&](const std::string& n) { return tensor_or_null(m, n); };
	size_t max_in = 4, max_q = 1, max_att = 1;
	for (size_t li = 0; li < m->layers.size(); li++) {
		Layer& L = m->layers[li];
		const std::string p = "l" + std::to_string(li) + ".";
		const int H = L.H, G = L.G, d = L.d, dv = L.dv;
		const long long bytes0 = m->weight_bytes;
		XALM_TRY(upload_vec(m, p + "norm1", &L.norm1));
		if (L.latent) {
			XALM_TRY(latent_upload(m, p + "mix.", li, &L.lat, &m->lat, &m->parts));
			max_in = std::max(max_in, (size_t) L.lat.n_in);
		} else {
			L.off_k = H * d; L.off_v = L.off_k + G * d;
			const int used = L.off_v + G * dv;
			L.n_in = (used + 3) / 4 * 4; // rows of zeros round the stack up to what the tensor-core GEMM takes
			HostTensor zeros;
			zeros.shape = {L.n_in - used, W};
			zeros.v.assign((size_t) zeros.shape[0] * W, 0.f);
			XALM_TRY(upload_rows(m, {T(p + "mix.q"), T(p + "mix.k"), T(p + "mix.v"), &zeros}, W, false, &L.w_in, &L.m_in));
			XALM_TRY(upload_vec(m, p + "mix.q.norm", &L.q_norm));
			XALM_TRY(upload_vec(m, p + "mix.k.norm", &L.k_norm));
			if (!L.freq_host.empty()) XALM_TRY(upload_floats(m, L.freq_host.data(), L.freq_host.size(), &L.freq));
			if (!swa_pick_tq(H, G, d, dv, m->chunk) && swa_smem_bytes(H, d, dv) > 200 * 1024)
				return set_error(XALM_ERR_UNSUPPORTED, "layer %zu: attention heads need %zu bytes of shared memory", li, swa_smem_bytes(H, d, dv));
			XALM_TRY(swa_prepare(H, d, dv));
			m->parts.need((size_t) H * dv, (size_t) H);
			max_in = std::max(max_in, (size_t) L.n_in);
			max_q = std::max(max_q, (size_t) H * d);
		}
		XALM_TRY(upload_rows(m, {T(p + "mix.o")}, H * dv, false, &L.w_o, &L.m_o));
		max_att = std::max(max_att, (size_t) H * dv);
		if (L.has_moe) {
			XALM_TRY(upload_vec(m, p + "norm2", &L.norm2));
			XALM_TRY(upload_vec(m, p + "mlp.router.b", &L.moe.bias));
			XALM_TRY(moe_upload(m, p + "mlp.", true, &L.moe, &m->moe));
			L.expert_bytes = 3ll * L.moe.ff * W * (m->w_bf16 ? 2 : 4);
		}
		L.bytes = m->weight_bytes - bytes0;
	}
	XALM_TRY(hc_norm_prepare(W));
	for (Layer& L : m->layers) {
		XALM_TRY(L.latent ? latent_tc_register(m, &L.lat) : tc_register(m, L.m_in, &L.t_in));
		XALM_TRY(tc_register(m, L.m_o, &L.t_o));
		if (L.has_moe) XALM_TRY(moe_tc_register(m, &L.moe, &m->moe));
	}
	for (Run& R : m->runs) { // what the sequence holds, per layer run
		const Layer& L = m->layers[(size_t) R.layer];
		if (L.latent) {
			XALM_TRY(latent_cache_alloc(m, L.lat, &R.lat));
			continue;
		}
		R.ring = ring_slots(m, L.reach);
		uint8_t *kc = nullptr, *vc = nullptr;
		XALM_TRY(dev_alloc(m, &kc, (size_t) R.ring * L.G * L.d * kelem, true));
		XALM_TRY(dev_alloc(m, &vc, (size_t) R.ring * L.G * L.dv * kelem, true));
		R.kc = kc; R.vc = vc;
	}
	m->proj_ld = (int) ((max_in + 3) / 4 * 4);
	XALM_TRY(dev_alloc(m, &m->x, (m->loops ? 3 : 1) * C * W));
	m->x0 = m->x + C * W;
	m->x2 = m->x0 + C * W;
	XALM_TRY(dev_alloc(m, &m->hn, C * W));
	XALM_TRY(dev_alloc(m, &m->proj, C * m->proj_ld));
	XALM_TRY(dev_alloc(m, &m->q, C * max_q));
	XALM_TRY(dev_alloc(m, &m->att, C * max_att));
	XALM_TRY(latent_alloc(m, &m->lat));
	XALM_TRY(attn_parts_alloc(m, &m->parts));
	return moe_alloc(m, &m->moe);
}

int release(SeqModel*) { return XALM_OK; } // nothing but cache rows, and a sequence only reads positions it wrote

// beyond one reading of every matrix: repeated layers read theirs again, a mixture reads only the chosen experts; the visible cache rows
long long active_bytes(SeqModel* sm, long long pos) {
	Pv* m = static_cast<Pv*>(sm);
	const long long W = m->width, kelem = m->precision == XALM_PRECISION_F32 ? 4 : 2, welem = m->w_bf16 ? 2 : 4;
	long long b = (m->vocab - 1) * W * welem; // the embedding table is read once more, whole, as the head matrix
	std::vector<int> seen(m->layers.size(), 0);
	for (const Run& R : m->runs) {
		const Layer& L = m->layers[(size_t) R.layer];
		const long long live = L.bytes - (L.has_moe ? L.moe.E - L.moe.top : 0) * L.expert_bytes;
		b += seen[(size_t) R.layer]++ ? live : live - L.bytes;
		if (L.latent) b += std::min<long long>(pos + 1, L.reach) * L.lat.R * kelem;
		else b += (L.chunk() ? pos % L.chunk() + 1 : pos + 1) * L.G * (L.d + L.dv) * kelem;
	}
	return b;
}

bool state_buffer(SeqModel*, int, const float**, size_t*) { return false; }

void destroy(SeqModel* sm) {
	Pv* m = static_cast<Pv*>(sm);
	for (Layer& L : m->layers) {
		for (TcWeight* t : {&L.t_in, &L.t_o}) tc_weight_free(t);
		latent_free(&L.lat);
		moe_free(&L.moe);
	}
	delete m;
}

const SeqHooks pavitar_hooks = {parse_config, finalize, enqueue_pass, release, active_bytes, state_buffer, destroy};
extern const ModelFamily pavitar_family;
int create(const char* json, int device, int max_tokens, int precision, xalm_cuda_model** out) {
	return seq_create<Pv>(&pavitar_family, &pavitar_hooks, json, device, max_tokens, precision, out);
}
const ModelFamily pavitar_family = seq_family_table("Pavitar", create);
const FamilyRegistrar pavitar_registrar(&pavitar_family);

} // namespace
} // namespace xalm
