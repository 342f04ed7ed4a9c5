// seq_latent.cuh — latent attention as a mixer of the config.json families: the tensors of one layer, their device layouts, and the kernels in
// order.
//
//   [rows product of the stacked down projections dq | dkv | g] -> latent_post (latent norms, rotated shared key, cache row) -> rows product [uq] ->
//   batched per-head product with uk^T (queries into the latent) (+ rope_heads for a rotated query part) -> swa_attn / swa_tile with ONE key/value
//   head that reads the cache rows in place -> batched per-head product with uv.  No per-head key or value is ever written to memory.
//
// A design says what it has: a rotated part or none, a window or the whole past, no output gate, one value per output column, or one per head.
// The gate per head multiplies the attention's result in the latent (the value expansion is linear), the one per column the expansion's output.
// What a sequence keeps is a LatentCache of the caller's: one row of kv_rank + rot elements per position, in a ring when there is a window.
#pragma once
#include "latent_ops.cuh"
#include "seq_family.cuh"

namespace xalm {
namespace seq {
namespace {

enum { LATENT_GATE_NONE = 0, LATENT_GATE_COLUMNS = 1, LATENT_GATE_HEADS = 2 };

struct LatentWeights {
	int H = 0, d = 0, dv = 0; // heads; plain query/key and value entries per head
	int r = 0, R = 0, Rq = 0; // rotated entries per head; latent sizes of keys and values, of queries
	int window = 0x7fffffff, gate = LATENT_GATE_NONE;
	bool own_cache = true;    // false: the rows are another layer's, and there is no dkv
	float scale = 1.f;
	std::vector<float> freq_host;
	float *freq = nullptr, *dq_norm = nullptr, *dkv_norm = nullptr;
	int off_kv = 0, off_g = 0, n_in = 0; // columns of the stacked projection
	void *w_in = nullptr, *w_uq = nullptr, *w_ukT = nullptr, *w_uv = nullptr;
	WMat m_in, m_uq;
	TcWeight t_in, t_uq;
	int gate_rows() const { return gate == LATENT_GATE_COLUMNS ? H * dv : gate == LATENT_GATE_HEADS ? H : 0; }
};

struct LatentCache { // what one sequence holds in one run of the layer
	void* rows = nullptr; // (ring, ld)
	int ld = 0, ring = 0;
};

struct LatentBuffers { // of one pass, sized for the largest layer of the model
	size_t max_cq = 0, max_q = 0, max_qabs = 0, max_olat = 0;
	float *cq = nullptr, *q = nullptr, *qabs = nullptr, *olat = nullptr;
};

// partial results of attention whose keys are split over CTAs, shared by every softmax mixer of a model
struct AttnParts {
	size_t max_row = 1, max_h = 1; // result entries of a token, heads
	float *o = nullptr, *ml = nullptr;
	unsigned* tickets = nullptr;
	int cap = 0;
	void need(size_t row, size_t heads) {
		max_row = std::max(max_row, row);
		max_h = std::max(max_h, heads);
	}
	void use(SwaArgs* a) const {
		a->part_o = o; a->part_ml = ml; a->part_cap = cap; a->tickets = tickets;
		a->n_splits = 0;
	}
};
int attn_parts_alloc(SeqModel* m, AttnParts* p) {
	p->cap = std::max(4 * 64, 4 * m->chunk); // one-token steps: up to 64 key splits; passes of a prompt: up to 4 per token
	XALM_TRY(dev_alloc(m, &p->o, (size_t) p->cap * p->max_row));
	XALM_TRY(dev_alloc(m, &p->ml, (size_t) p->cap * 2 * p->max_h));
	return dev_alloc(m, &p->tickets, 8 * (size_t) m->chunk, true); // the heads of a layer may run in up to 8 launches, each with counters of its own
}

// slots of a cache of which a query sees the last `reach` positions: one pass is written before its first query reads (reach 0x7fffffff: all)
inline int ring_slots(const SeqModel* m, int reach) {
	return reach < 0x7fffffff ? (int) std::min<long long>(m->max_tokens, (long long) reach - 1 + m->chunk) : m->max_tokens;
}

// tensors of the mixer under prefix p ("l0.mix.")
void latent_expect(SeqModel* m, const std::string& p, const LatentWeights& L) {
	expect(m, p + "dq", {L.Rq, m->width}, true);
	expect(m, p + "dq.norm", {L.Rq}, false);
	expect(m, p + "uq", {L.H * (L.d + L.r), L.Rq}, true);
	if (L.own_cache) {
		expect(m, p + "dkv", {L.R + L.r, m->width}, true);
		expect(m, p + "dkv.norm", {L.R}, false);
	}
	expect(m, p + "uk", {L.H * L.d, L.R}, true);
	expect(m, p + "uv", {L.H * L.dv, L.R}, true);
	if (L.gate) expect(m, p + "g", {L.gate_rows(), m->width}, true);
}

// uk (H * d, R) as H matrices (R, d): row j of head h holds column j of that head's rows, so that q_h -> uk_h^T q_h is a rows product
int upload_transposed_heads(SeqModel* m, const HostTensor* uk, int H, int d, int R, void** dst) {
	HostTensor t;
	t.shape = {H * R, d};
	t.v.resize((size_t) H * R * d);
	for (int h = 0; h < H; h++)
		for (int i = 0; i < d; i++)
			for (int j = 0; j < R; j++) t.v[((size_t) h * R + j) * d + i] = uk->v[((size_t) h * d + i) * R + j];
	return upload_rows(m, {&t}, d, false, dst, nullptr);
}

// device layouts; what the pass buffers must hold.  `li`: the layer's number, for messages
int latent_upload(SeqModel* m, const std::string& p, size_t li, LatentWeights* L, LatentBuffers* b, AttnParts* parts) {
	const int H = L->H, d = L->d, r = L->r, R = L->R, Rq = L->Rq, W = m->width;
	auto T = [&](const char* n) { return tensor_or_null(m, p + n); };
	if (!L->freq_host.empty()) XALM_TRY(upload_floats(m, L->freq_host.data(), L->freq_host.size(), &L->freq));
	L->off_kv = Rq;
	L->off_g = Rq + (L->own_cache ? R + r : 0);
	const int used = L->off_g + L->gate_rows();
	L->n_in = (used + 3) / 4 * 4; // rows of zeros round the stack up to what the tensor-core GEMM takes
	HostTensor zeros;
	zeros.shape = {L->n_in - used, W};
	zeros.v.assign((size_t) zeros.shape[0] * W, 0.f);
	XALM_TRY(upload_rows(m, {T("dq"), L->own_cache ? T("dkv") : nullptr, L->gate ? T("g") : nullptr, &zeros}, W, false, &L->w_in, &L->m_in));
	XALM_TRY(upload_vec(m, p + "dq.norm", &L->dq_norm));
	XALM_TRY(upload_rows(m, {T("uq")}, Rq, false, &L->w_uq, &L->m_uq));
	XALM_TRY(upload_transposed_heads(m, T("uk"), H, d, R, &L->w_ukT));
	XALM_TRY(upload_rows(m, {T("uv")}, R, false, &L->w_uv, nullptr));
	if (L->own_cache) XALM_TRY(upload_vec(m, p + "dkv.norm", &L->dkv_norm));
	// the attention sees one key/value head of R + r (values: R)
	if (!swa_pick_tq(H, 1, R + r, R, m->chunk) && swa_smem_bytes(H, R + r, R) > 200 * 1024)
		return set_error(XALM_ERR_UNSUPPORTED, "layer %zu: %d heads over a latent of %d + %d need %zu bytes of shared memory", li, H, R, r, swa_smem_bytes(H, R + r, R));
	XALM_TRY(swa_prepare(H, R + r, R));
	b->max_cq = std::max(b->max_cq, (size_t) Rq);
	b->max_q = std::max(b->max_q, (size_t) H * (d + r));
	b->max_qabs = std::max(b->max_qabs, (size_t) H * (R + r));
	b->max_olat = std::max(b->max_olat, (size_t) H * R);
	parts->need((size_t) H * R, (size_t) H);
	return XALM_OK;
}
int latent_tc_register(SeqModel* m, LatentWeights* L) {
	XALM_TRY(tc_register(m, L->m_in, &L->t_in));
	return tc_register(m, L->m_uq, &L->t_uq);
}
int latent_alloc(SeqModel* m, LatentBuffers* b) {
	const size_t C = (size_t) m->chunk;
	XALM_TRY(dev_alloc(m, &b->cq, C * b->max_cq));
	XALM_TRY(dev_alloc(m, &b->q, C * b->max_q));
	XALM_TRY(dev_alloc(m, &b->qabs, C * b->max_qabs));
	return dev_alloc(m, &b->olat, C * b->max_olat);
}
int latent_cache_alloc(SeqModel* m, const LatentWeights& L, LatentCache* c) {
	c->ld = L.R + L.r;
	c->ring = ring_slots(m, L.window);
	uint8_t* rows = nullptr;
	XALM_TRY(dev_alloc(m, &rows, (size_t) c->ring * c->ld * (m->precision == XALM_PRECISION_F32 ? 4 : 2), true));
	c->rows = rows;
	return XALM_OK;
}
void latent_free(LatentWeights* L) {
	tc_weight_free(&L->t_in);
	tc_weight_free(&L->t_uq);
}

// Everything between the stacked projection (proj, (n, ld)) and the output projection: att (n, H * dv).
int latent_attention(SeqModel* m, const LatentWeights& L, const LatentCache& c, const LatentBuffers& b, const AttnParts& parts, const float* proj, int ld, float* att,
                     int n, int* nl) {
	cudaStream_t s = m->stream;
	const int H = L.H, d = L.d, r = L.r, dv = L.dv, R = L.R, Rq = L.Rq;
	const bool f32 = m->precision == XALM_PRECISION_F32;
	LatentPostArgs pa = {};
	pa.proj = proj; pa.ld = ld;
	pa.q_off = 0; pa.q_rank = Rq; pa.q_norm = L.dq_norm; pa.cq = b.cq; pa.ldc = Rq;
	pa.kv_off = L.off_kv; pa.kv_rank = L.own_cache ? R : 0; pa.rot = r; pa.kv_norm = L.dkv_norm; pa.freq = L.freq;
	pa.eps = m->eps; pa.cache = c.rows; pa.cache_f32 = f32; pa.ring = c.ring; pa.step = m->d_step;
	XALM_TRY(launch_latent_post(pa, n, s));
	(*nl)++;
	RowsEpi est;
	est.kind = EPI_STORE; est.out = b.q; est.ldo = H * (d + r);
	XALM_TRY(rows_product(m, b.cq, Rq, L.w_uq, &L.t_uq, n, H * (d + r), Rq, est, nl));
	// queries into the latent, head by head: qabs[h] = [uk_h^T q_h | rotated q_h]
	RowsEpi eb;
	eb.kind = EPI_STORE; eb.out = b.qabs; eb.ldo = H * (R + r);
	eb.batch_a = d + r; eb.batch_w = (size_t) R * d; eb.batch_o = R + r;
	XALM_TRY(launch_rows(b.q, H * (d + r), L.w_ukT, m->w_bf16, n, R, d, eb, s, H));
	(*nl)++;
	if (r) {
		RopeHeadsArgs ra = {};
		ra.src = b.q; ra.lds = H * (d + r); ra.src_off = d; ra.src_stride = d + r;
		ra.dst = b.qabs; ra.ldd = H * (R + r); ra.dst_off = R; ra.dst_stride = R + r;
		ra.heads = H; ra.n = r; ra.rot_half = r / 2; ra.freq = L.freq; ra.step = m->d_step;
		XALM_TRY(launch_rope_heads(ra, n, s));
		(*nl)++;
	}
	SwaArgs sa = {};
	sa.q = b.qabs; sa.ldq = H * (R + r); sa.q_off = 0;
	sa.kc = c.rows; sa.vc = c.rows; sa.ldk = c.ld; sa.ldv = c.ld;
	sa.ring = c.ring; sa.keep_first = 0;
	sa.H = H; sa.G = 1; sa.d = R + r; sa.dv = R;
	sa.window = L.window; sa.scale = L.scale;
	if (L.gate == LATENT_GATE_HEADS) { sa.gate = proj; sa.ldg = ld; sa.g_off = L.off_g; sa.gate_per_head = 1; }
	sa.step = m->d_step; sa.out = b.olat;
	parts.use(&sa);
	int launches = 1;
	XALM_TRY(launch_swa(sa, n, f32, s, &launches));
	*nl += launches;
	// values out of the latent, head by head
	RowsEpi ev;
	ev.kind = EPI_STORE; ev.out = att; ev.ldo = H * dv;
	ev.batch_a = R; ev.batch_w = (size_t) dv * R; ev.batch_o = dv;
	if (L.gate == LATENT_GATE_COLUMNS) { ev.mul = proj + L.off_g; ev.ldm = ld; ev.mul_act = ACT_SIGMOID; }
	XALM_TRY(launch_rows(b.olat, H * R, L.w_uv, m->w_bf16, n, dv, R, ev, s, H));
	(*nl)++;
	return XALM_OK;
}

} // namespace
} // namespace seq
} // namespace xalm
