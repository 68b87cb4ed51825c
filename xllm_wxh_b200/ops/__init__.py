"""Hot ops.  A CUDA tensor runs the hand-written sm_100a kernel from `libxllm_kernels.so`
(loaded by `cuda_ops`; missing library on a CUDA device is an error, never a silent fallback);
a CPU tensor runs the PyTorch statement of the same op from `reference`, which is also the oracle
the kernels are tested against."""
from __future__ import annotations

from . import reference as ref


def _cuda():
    from . import cuda_ops
    return cuda_ops


def rms_norm(x, w, eps):
    return _cuda().rms_norm(x, w, eps) if x.is_cuda else ref.rms_norm(x, w, eps)


def add_rms_norm(x, residual, w, eps):
    return _cuda().add_rms_norm(x, residual, w, eps) if x.is_cuda else ref.add_rms_norm(x, residual, w, eps)


def linear(x, w, bias=None):
    return _cuda().linear(x, w, bias) if x.is_cuda else ref.linear(x, w, bias)


def silu_and_mul(x):
    return _cuda().silu_and_mul(x) if x.is_cuda else ref.silu_and_mul(x)


def embedding(ids, table):
    return _cuda().embedding(ids, table) if table.is_cuda else ref.embedding(ids, table)


def rope_qknorm_kvwrite(qkv, positions, slots, cos_sin, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, head_dim):
    f = _cuda().rope_qknorm_kvwrite if qkv.is_cuda else ref.rope_qknorm_kvwrite
    return f(qkv, positions, slots, cos_sin, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, head_dim)


def paged_attention(q, k_cache, v_cache, inp, scale, sliding_window=-1):
    """q [T, Hq, D]; `inp` is a StepInput (q_cu, kv_lens, block_tables, n_seqs, n_decode ...)."""
    if q.is_cuda:
        return _cuda().paged_attention(q, k_cache, v_cache, inp, scale, sliding_window)
    return ref.paged_attention(q, k_cache, v_cache, inp.q_cu, inp.kv_lens, inp.block_tables, inp.n_seqs, scale,
                               sliding_window)


def paged_attention_ext(q, k_cache, v_cache, inp, scale, window=-1, chunk=0, slopes=None, sinks=None, keep_first=0, softcap=0.0, mix=None,
                        bound=0.0):
    """Paged attention with a per-head linear distance bias (`slopes` [Hq] fp32), a per-head sink score in the softmax
    denominator (`sinks` [Hq] fp32), keys limited to the query's chunk of `chunk` positions, first positions that stay
    visible behind the window (`keep_first`), scores bounded by `softcap` * tanh(score / softcap), and a value head dimension of
    its own.  q [T, Hq, dk] -> [T, Hq * dv].
    `mix` = (factor fp32 [1], mult, eps): differential attention.  Query and key heads are pairs of two maps, every pair of query
    heads has one value head's values, and its output is rms(first - factor * second) * mult: [T, Hq / 2 * dv].
    `bound` > 0 promises |q . k| <= bound (normed queries and keys), which saves the kernels a check of bounded scores.
    k_cache may have one key head beside several value heads: all query heads then share it (queries of `mix_query_heads`)."""
    if q.is_cuda:
        return _cuda().paged_attention_ext(q, k_cache, v_cache, inp, scale, window, chunk, slopes, sinks, keep_first, softcap, mix, bound)
    return ref.paged_attention(q, k_cache, v_cache, inp.q_cu, inp.kv_lens, inp.block_tables, inp.n_seqs, scale, window, chunk,
                               slopes, sinks, keep_first, softcap, mix)


def sample(logits, inp):
    """Penalties -> temperature -> top-k/top-p -> sample/argmax (+logprobs).  Returns
    (tokens int32 [S], logprobs | None, top_vals | None, top_ids | None)."""
    if logits.is_cuda:
        return _cuda().sample(logits, inp)
    lg = logits.float()
    S = lg.shape[0]
    if inp.any_penalty:
        ref.apply_penalties(lg, inp.pen_cu[:S + 1], inp.pen_ids, inp.pen_counts, inp.rep_pen[:S], inp.freq_pen[:S],
                            inp.pres_pen[:S])
    return ref.sample(lg, inp.temperature[:S], inp.top_k[:S], inp.top_p[:S], inp.seed_lo[:S], inp.seed_hi[:S],
                      inp.any_logprobs, inp.max_top_logprobs)


def topk_candidates(logits, inp, id_offset: int, width: int):
    """Candidates of one vocabulary slice for vocabulary-parallel sampling (values, global ids, overflow flag)."""
    if logits.is_cuda:
        return _cuda().topk_candidates(logits, inp, id_offset, width)
    S = logits.shape[0]
    return ref.topk_candidates(logits, inp.temperature[:S], inp.top_k[:S], id_offset, width)


def moe_router(logits, top_k, scoring="softmax", renorm=True, bias=None, n_group=1, topk_group=1, route_scale=1.0, group_score=None):
    """`group_score`: how a group of experts is ranked, "max" or "top2" (sum of its two best); None: top2 with a bias, else max.
    scoring "softmax_chosen": the bias is part of the logits, the weights are the softmax over the chosen ones."""
    f = _cuda().moe_router if logits.is_cuda else ref.moe_router
    extra = {} if group_score is None else {"group_score": group_score}
    return f(logits, top_k, scoring, renorm, bias, n_group, topk_group, route_scale, **extra)


def moe_experts(x, w13, w2, weights, ids, expert_offset=0, interleaved=False):
    """`interleaved`: w13 rows were re-ordered by `finalize_weights` for the fused SwiGLU epilogue (CUDA only)."""
    if x.is_cuda:
        return _cuda().moe_experts(x, w13, w2, weights, ids, expert_offset, interleaved)
    assert not interleaved
    return ref.moe_experts(x, w13, w2, weights, ids, expert_offset)


def gate_up_swiglu(x, w, interleaved=False):
    """silu(x Wg^T) * (x Wu^T) with W = [gate rows; up rows] (or the interleaved layout on CUDA: one fused kernel)."""
    if x.is_cuda and interleaved:
        return _cuda().linear_swiglu(x, w)
    assert not interleaved
    return silu_and_mul(linear(x, w))


# ----------------------------------------------------------------------------- sublayers normed before and after, fp32 residual
def embed_rms_norm(ids, table, scale, w_next, eps, positions=None, pos_table=None, w_offset=0.0, w_rows=None):
    """(fp32 residual x = table[ids] * scale (+ pos_table[positions]), rms(x) * (w_next + w_offset) in the table's dtype).
    With `w_rows` the embedding is normed itself: x = rms(row) * w_rows."""
    return (_cuda() if table.is_cuda else ref).embed_rms_norm(ids, table, scale, w_next, eps, positions, pos_table, w_offset, w_rows)


def post_norm_add_norm(y, x, w_post, w_next, eps):
    """x += rms(y) * w_post (x fp32, in place); returns rms(x) * w_next."""
    return (_cuda() if y.is_cuda else ref).post_norm_add_norm(y, x, w_post, w_next, eps)


def branches_post_norm_add_norm(ya, yb, w_a, w_b, scale, x, w_post, w_next, eps):
    """y = scale * (rms(ya) * w_a + rms(yb) * w_b); x += rms(y) * w_post (x fp32, in place); returns rms(x) * w_next."""
    return (_cuda() if ya.is_cuda else ref).branches_post_norm_add_norm(ya, yb, w_a, w_b, scale, x, w_post, w_next, eps)


def qknorm_kvwrite(qkv, slots, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, rot=None):
    """Per-head RMSNorm of q and k, then the rotation `rot` = (table of `ref.rotary_table`, positions, interleaved) if there is one;
    k and v into the paged caches (n_kv key heads, as many value heads as v_cache has).  Returns q [T, n_q * dk]."""
    return (_cuda() if qkv.is_cuda else ref).qknorm_kvwrite(qkv, slots, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, rot)


def linear_f32(x, w):
    """x w^T in fp32 (router logits)."""
    return (_cuda() if x.is_cuda else ref).linear_f32(x, w)


def gated_linear(x, w, act="silu", interleaved=False, limit=0.0):
    """act(x Wg^T) * (x Wu^T) with W = [gate rows; up rows], or the interleaved layout on CUDA (applied in the GEMM epilogue).
    act: "silu" | "gelu_tanh" | "clamped" (g sigmoid(1.702 g) (u + 1), g at most `limit`, u within +- limit)."""
    if not x.is_cuda:
        return ref.gated_act(linear(x, w), act, limit)
    return _cuda().linear_gated(x, w, act, limit) if interleaved else _cuda().gated_act(linear(x, w), act, limit)


def linear_softcap(x, w, cap):
    """cap * tanh(x w^T / cap), applied to the fp32 sums (logits)."""
    return (_cuda() if x.is_cuda else ref).linear_softcap(x, w, cap)


def moe_post_norm_add_norm(h_in, w13, w2, weights, ids, shared, first_identity, x, w_post, w_next, eps, act="silu", interleaved=False):
    """Mixture sublayer from its routing to the next sublayer's input: y = sum_j weights_j expert_j(h_in) (ids from
    `first_identity` on are identity experts: weight times h_in) + shared (or None); x += rms(y) * w_post (fp32, in place);
    returns rms(x) * w_next.  act "relu2": experts without a gate, w13 [experts, ff, H]."""
    if h_in.is_cuda:
        from . import moe_cuda
        y, dst_of = moe_cuda.expert_rows(h_in, w13, w2, ids, act, interleaved)
        return moe_cuda.combine_post_norm_add_norm(y, dst_of, ids, weights, h_in, shared, first_identity, x, w_post, w_next, eps)
    y = ref.moe_mixture(h_in, w13, w2, weights, ids, shared, first_identity, act)
    return ref.post_norm_add_norm(y, x, w_post, w_next, eps)


# ----------------------------------------------------------------------------- sublayers normed before only, fp32 residual
def add_norm(y, x, mult, w_next, eps, vec=None, w_offset=0.0, lead=None):
    """x += mult * y, or vec * y element by element (x fp32, in place); returns rms(x) * (w_next + w_offset).
    `lead` = (ids, table, scale, positions, pos_table): rows of the embedding that are added to x before the norm."""
    return (_cuda() if y.is_cuda else ref).add_norm(y, x, mult, w_next, eps, vec, w_offset, lead)


def lead_norm(lead, x, w_next, eps, w_offset=0.0):
    """x += embedding rows (`lead` as in `add_norm`); returns rms(x) * (w_next + w_offset)."""
    return (_cuda() if x.is_cuda else ref).lead_norm(lead, x, w_next, eps, w_offset)


def moe_add_norm(h_in, w13, w2, weights, ids, vec, x, w_next, eps, act="silu", interleaved=False, limit=0.0, w_offset=0.0, lead=None):
    """Mixture sublayer from its routing to the next sublayer's input: x += vec * sum_j weights_j expert_j(h_in) (x fp32, in
    place), then as `add_norm`."""
    if h_in.is_cuda:
        from . import moe_cuda
        y, dst_of = moe_cuda.expert_rows(h_in, w13, w2, ids, act, interleaved, limit)
        return moe_cuda.combine_add_norm(y, dst_of, weights, vec, x, w_next, eps, w_offset, lead)
    y = ref.moe_mixture(h_in, w13, w2, weights, ids, None, w13.shape[0], act, limit)
    return ref.add_norm(y, x, 1.0, w_next, eps, vec, w_offset, lead)


def replace_norm(y, vec, x, w_next, eps):
    """x = y + vec (y, x fp32; vec one row); returns rms(x) * w_next."""
    return (_cuda() if y.is_cuda else ref).replace_norm(y, vec, x, w_next, eps)


def split_rows(x, ids, table, scale):
    """Rows [x, x0] for a product with `split_columns` of its weight, x0 = table[ids] * scale.  In a bf16 model the fp32 x
    enters as two bf16 parts (its rounded value and the rest), so that a product of the residual stream does not round it to
    8 bits."""
    return (_cuda() if x.is_cuda else ref).split_rows(x, ids, table, scale)


def split_columns(w, width):
    """Weight [N, 2 width] of a product of [x, x0] in the column layout of `split_rows`."""
    import torch
    return w if w.dtype == torch.float32 else torch.cat([w[:, :width], w], 1).contiguous()


def act_linear(x, w, act):
    """act(x w^T), applied to the fp32 sums: "relu2" (squared relu) | "tanh"."""
    return (_cuda() if x.is_cuda else ref).act_linear(x, w, act)


def qknorm_all_kvwrite(qkv, slots, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, rot=None, mix=None):
    """RMSNorm over the whole query and the whole key projection, then the rotation `rot` (as in `qknorm_kvwrite`) if there is one;
    k and v into the paged caches.  Rows of qkv may be longer than q, k and v.  Returns q [T, n_q * dk], or with `mix` (fp32
    [n_q, n_q]) the queries [T, n_q * n_kv * dk] of attention whose scores are mixed over the heads: the product of row h and a
    token's keys of all key heads side by side is sum_g mix[h, g] q_g . k_(g's key head)."""
    return (_cuda() if qkv.is_cuda else ref).qknorm_all_kvwrite(qkv, slots, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, rot, mix)


def gate_into(o, gate, scale, out):
    """out = o * sigmoid(gate) * scale (gate and out may be strided views)."""
    (_cuda() if o.is_cuda else ref).gate_into(o, gate, scale, out)


# ----------------------------------------------------------------------------- recurrent layers
# State tensors hold one record per state slot; `inp.state_slots` names each sequence's, and it is updated in place.
def _seqs(inp):
    return inp.q_cu, inp.kv_lens, inp.state_slots, inp.n_seqs


def token_shift(h, mu, last, inp):
    """[n, T, W]: every row of h blended with its predecessor by each of the n rows of mu; `last` [slots, W] is the state."""
    return _cuda().token_shift(h, mu, last, inp) if h.is_cuda else ref.token_shift(h, mu, last, *_seqs(inp))


def time_mix(r, k, v, z, w0, u, gate, norm_w, scale, eps, state, inp, out):
    """Matrix-state recurrence with a decay exp(-exp(z + w0)) per key channel and the bonus u for the current token; per-head
    RMS, weight, silu gate and `scale` on its output, which goes to `out` (may be a strided view)."""
    if r.is_cuda:
        _cuda().time_mix(r, k, v, z, w0, u, gate, norm_w, scale, eps, state, inp, out)
    else:
        ref.time_mix(r, k, v, z, w0, u, gate, norm_w, scale, eps, state, *_seqs(inp), out)


def conv_silu(x, w, b, state, inp):
    """silu of a causal convolution per channel over each sequence; w [taps, C]; x may be a strided view; state
    [slots, taps - 1, C]."""
    return causal_conv(x, w, b, state, inp, act="silu")


def causal_conv(x, w, b, state, inp, act="none", residual=False):
    """act(b + causal convolution per channel over each sequence) (+ x with `residual`); layouts as `conv_silu`; b may be None."""
    if x.is_cuda:
        return _cuda().causal_conv(x, w, b, state, inp, act, residual)
    return ref.causal_conv(x, w, b, state, *_seqs(inp), act, residual)


def gated_memory(q, k, v, z, bias, inv_tau, gate, norm_w, eps, state, inp):
    """Matrix-state recurrence S = diag(sigmoid(z + bias)^inv_tau) S + k v^T per head, o = S^T q / sqrt(dim); RMS per head with the
    weight norm_w [vdim], silu gate.  q, k [T, heads * dim], v, gate [T, heads * vdim] may be strided views, z fp32; state
    [slots, heads, dim, vdim] fp32.  Returns [T, heads * vdim]."""
    if q.is_cuda:
        return _cuda().gated_memory(q, k, v, z, bias, inv_tau, gate, norm_w, eps, state, inp)
    return ref.gated_memory(q, k, v, z, bias, inv_tau, gate, norm_w, eps, state, *_seqs(inp))


def matrix_memory(q, k, v, gates, bias, cap, gate, norm_w, eps, state, top, inp):
    """Matrix memory with exponential gates: per head i = cap tanh((gates_i + bias_i) / cap), f = log sigmoid of the same of gates_f,
    S = e^f S + e^i k v^T and n = e^f n + e^i k, both relative to e^m of a running maximum m; o = S^T q / max(|n q|, e^-m) with q
    over sqrt(dim); RMS per head, weight norm_w [heads * vdim], sigmoid gate.  gates fp32 [T, 2 heads] (i, then f), bias fp32
    [2 heads]; state [slots, heads, dim * vdim + dim] fp32 (S, then n), top [slots, heads] fp32 (m).  Returns [T, heads * vdim]."""
    if q.is_cuda:
        return _cuda().matrix_memory(q, k, v, gates, bias, cap, gate, norm_w, eps, state, top, inp)
    return ref.matrix_memory(q, k, v, gates, bias, cap, gate, norm_w, eps, state, top, *_seqs(inp))


def selective_scan(x, dt, dt_bias, A, B, C, D, z, state, inp):
    """Diagonal state space recurrence with data-dependent steps softplus(dt + dt_bias); returns (scan + D x) silu(z)."""
    if x.is_cuda:
        return _cuda().selective_scan(x, dt, dt_bias, A, B, C, D, z, state, inp)
    return ref.selective_scan(x, dt, dt_bias, A, B, C, D, z, state, *_seqs(inp))


# ----------------------------------------------------------------------------- latent attention of any size
def latent_down(low, q_rank, kv_rank, q_w, kv_w, eps, rot, slots, cache):
    """Rows [query latent | key/value latent | key part]: both latents normed, the key part rotated (`rot` as in
    `qknorm_kvwrite`); [latent | key part] into the cache [blocks, block, kv_rank + rot_dim].  Returns the query latent."""
    return (_cuda() if low.is_cuda else ref).latent_down(low, q_rank, kv_rank, q_w, kv_w, eps, rot, slots, cache)


def latent_attention(q, w_uk, w_uv, cache, inp, rot, scale, dim):
    """Attention over cached latents in absorbed form.  q [T, H, dim + rot_dim] (unrotated part first), w_uk [H, kv_rank, dim],
    w_uv [H, vdim, kv_rank], cache of `latent_down`.  Returns [T, H * vdim]."""
    import torch
    T, H, _ = q.shape
    C, row = w_uk.shape[1], cache.shape[-1]
    if q.is_cuda and _cuda().mla_serves(H, C, row - C, q.dtype):
        return _cuda().latent_attention_mla(q, w_uk, w_uv, cache, inp, rot, scale, dim)
    lat = torch.empty((T, H, row), dtype=q.dtype, device=q.device)
    heads_linear(q[..., :dim].transpose(0, 1), w_uk, lat[..., :C].transpose(0, 1))
    rotate_into(q[..., dim:], rot, lat[..., C:])
    # one key / value head whose values are the first columns of its keys
    keys = cache.unsqueeze(2)
    o = paged_attention_ext(lat, keys, keys[..., :C], inp, scale)
    out = torch.empty((T, H, w_uv.shape[1]), dtype=q.dtype, device=q.device)
    heads_linear(o.view(T, H, C).transpose(0, 1), w_uv, out.transpose(0, 1))
    return out.flatten(1)


def heads_linear(x, w, out):
    """out[h] = x[h] w[h]^T for every head: x [H, T, K], w [H, N, K], out [H, T, N]; x and out may be views of token-major tensors."""
    return (_cuda() if x.is_cuda else ref).heads_linear(x, w, out)


def rotate_into(x, rot, out):
    """out = x rotated (x, out [T, H, d], may be strided views)."""
    (_cuda() if x.is_cuda else ref).rotate_into(x, rot, out)


# ----------------------------------------------------------------------------- MLA (DeepSeek)
def mla_prepare(q, kv_a, positions, slots, cos_sin, kv_norm_w, eps, cache, w_kc, nope, rope, kv_lora):
    """Latent RMSNorm + interleaved RoPE of k_pe -> one [kv_lora + rope] cache row per token; RoPE of q_pe; q_nope absorbed
    into the latent space with W_kc.  Returns (q_lat [T, Hh, kv_lora], q_pe [T, Hh, rope])."""
    if q.is_cuda:
        return _cuda().mla_prepare(q, kv_a, positions, slots, cos_sin, kv_norm_w, eps, cache, w_kc, nope, rope, kv_lora)
    import torch
    T = q.shape[0]
    cs = cos_sin.index_select(0, positions.long())
    cos, sin = cs[:, :rope // 2], cs[:, rope // 2:]
    latent = ref.rms_norm(kv_a[:, :kv_lora], kv_norm_w, eps)
    k_pe = ref.apply_rope_interleaved(kv_a[:, None, kv_lora:], cos, sin)[:, 0]
    cache.view(-1, kv_lora + rope).index_copy_(0, slots.long(), torch.cat([latent, k_pe], -1).to(cache.dtype))
    q_pe = ref.apply_rope_interleaved(q[..., nope:], cos, sin)
    q_lat = torch.einsum("thn,hnc->thc", q[..., :nope].float(), w_kc.float()).to(q.dtype)
    return q_lat, q_pe


def mla_attention(q_lat, q_pe, cache, inp, scale, kv_lora):
    if q_lat.is_cuda:
        return _cuda().mla_attention(q_lat, q_pe, cache, inp, scale, kv_lora)
    return ref.mla_attention(q_lat, q_pe, cache, inp.q_cu, inp.kv_lens, inp.block_tables, inp.n_seqs, scale, kv_lora)


def mla_attention_sparse(q_lat, q_pe, cache, sel, sel_len, scale, kv_lora):
    """MLA attention in which query token t reads only the cache slots `sel[t, :sel_len[t]]` (what a lightning indexer
    kept for it; the selection is causal already, so no mask applies).  Layouts as `mla_attention`."""
    if q_lat.is_cuda:
        return _cuda().mla_attention_sparse(q_lat, q_pe, cache, sel, sel_len, scale, kv_lora)
    return ref.mla_attention_sparse(q_lat, q_pe, cache, sel, sel_len, scale, kv_lora)


def mla_v_up(o_lat, w_vc):
    """[T, Hh, kv_lora] x W_vc [Hh, v, kv_lora] -> [T, Hh * v]."""
    if o_lat.is_cuda:
        return _cuda().mla_v_up(o_lat, w_vc)
    import torch
    return torch.einsum("thc,hvc->thv", o_lat.float(), w_vc.float()).to(o_lat.dtype).reshape(o_lat.shape[0], -1)


def linear_fp8_block(x, wq, wscale):
    """Block-scaled fp8 linear: dynamic 1x128 activation scales, 128x128 weight scales."""
    if x.is_cuda:
        return _cuda().linear_fp8_block(x, wq, wscale)
    return ref.linear_fp8_block(x, wq, wscale, x.dtype)


def moe_experts_q(x, layer, weights, ids, expert_offset=0):
    """Routed experts of a layer object carrying `w13`, `w2` and optional fp8 block scales `w13_scale`, `w2_scale`."""
    if layer.w13_scale is None:
        return moe_experts(x, layer.w13, layer.w2, weights, ids, expert_offset, layer.interleaved)
    if x.is_cuda:
        return _cuda().moe_experts_fp8(x, layer.w13, layer.w13_scale, layer.w2, layer.w2_scale, weights, ids, expert_offset)
    import torch
    w13 = torch.stack([ref.dequant_weight_128x128(layer.w13[e], layer.w13_scale[e]) for e in range(layer.w13.shape[0])]).to(x.dtype)
    w2 = torch.stack([ref.dequant_weight_128x128(layer.w2[e], layer.w2_scale[e]) for e in range(layer.w2.shape[0])]).to(x.dtype)
    # activations go through the same 1x128 quantisation as on the GPU path
    return ref.moe_experts_fp8(x, w13, w2, weights, ids, expert_offset)


# ----------------------------------------------------------------------------- fp8 with per-row activation / per-channel weight scales
def quant_rows_fp8(x):
    return _cuda().quant_rows_fp8(x) if x.is_cuda else ref.quant_rows_fp8(x)


def rms_norm_quant_fp8(x, w, eps):
    """(e4m3 RMSNorm(x) * w, row scales)."""
    if x.is_cuda:
        return _cuda().rms_norm_quant_fp8(x, w, eps)
    return ref.quant_rows_fp8(ref.rms_norm(x, w, eps))


def add_rms_norm_quant_fp8(x, residual, w, eps):
    """(e4m3 RMSNorm(x + residual) * w, row scales, x + residual)."""
    if x.is_cuda:
        return _cuda().add_rms_norm_quant_fp8(x, residual, w, eps)
    h, res = ref.add_rms_norm(x, residual, w, eps)
    q, s = ref.quant_rows_fp8(h)
    return q, s, res


def linear_fp8_scaled(xq, xs, wq, col_scale=None, tensor_scale=1.0, bias=None, swiglu=False, cpu_dtype=None):
    """(xq wq^T) * xs[m] * tensor_scale * col_scale[n] (+ bias).  `swiglu`: silu(gate) * up of the result (on CUDA `wq` then
    holds the interleaved gate / up rows and the GEMM epilogue applies it; on the CPU the plain [gate; up] rows)."""
    if xq.is_cuda:
        return _cuda().linear_fp8_scaled(xq, xs, wq, col_scale, tensor_scale, bias, swiglu)
    import torch
    y = ref.linear_fp8_scaled(xq, xs, wq, col_scale, tensor_scale, bias, out_dtype=cpu_dtype or torch.float32)
    return silu_and_mul(y) if swiglu else y
