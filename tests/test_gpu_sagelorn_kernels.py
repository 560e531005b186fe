"""The kernels behind the Sagelorn parts, each alone, against the plain functions of tests/plain/sagelorn.py (float64): the pair
embedding with its last tokens, attention with sinks inside a window (general and tensor-core forms, one key made to stand
out at the window's edge and at page borders, sinks far above and below the scores), the preparation with whole-projection
norms and stored heads wider than the heads, the recurrence with a fixed decay (token form and chunk form), the per-head
products with a gate a value, row norms, and the squared-relu experts with weights on their inputs in every product form."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from plain import sagelorn as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64
EPS = 1e-5


def i32(v):
    return torch.tensor(np.asarray(v), dtype=torch.int32, device=DEV)


def t32(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)


def rel(ref, got):
    ref, got = np.asarray(ref, dtype=np.float64), np.asarray(got, dtype=np.float64)
    return float(np.abs(ref - got).max() / max(np.abs(ref).max(), 1e-30))


def step_ctx(q_lens, starts):
    """A step's context and page lists in no order: sequence b brings q_lens[b] tokens behind starts[b]."""
    from mynah_slm_b200.ops import kernels
    tok_seq, tok_pos, cu, kv_len, indptr, ids = [], [], [0], [], [0], []
    total = sum((s + n + PAGE - 1) // PAGE for n, s in zip(q_lens, starts))
    pool = list(np.random.default_rng(total).permutation(total + 3))
    for b, (n, s) in enumerate(zip(q_lens, starts)):
        tok_seq += [b] * n
        tok_pos += list(range(s, s + n))
        cu.append(cu[-1] + n)
        kv_len.append(s + n)
        ids += [int(pool.pop()) for _ in range((s + n + PAGE - 1) // PAGE)]
        indptr.append(len(ids))
    B = len(q_lens)
    pages = kernels.PageTableView(i32(indptr), i32(ids), i32([0] * B), total + 3)
    ctx = SimpleNamespace(tok_seq=i32(tok_seq), tok_pos=i32(tok_pos), cu_q=i32(cu), kv_len=i32(kv_len), B=B, T=len(tok_seq),
                          status=torch.zeros((1,), dtype=torch.int32, device=DEV), is_decode=all(n == 1 for n in q_lens),
                          max_q_len=max(q_lens), decode_splits=max((k + PAGE - 1) // PAGE for k in kv_len))
    return ctx, pages, total + 3


# ------------------------------------------------------------------ embedding
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("V,D,buckets,mul_prev,mul_cur", [(50, 24, 31, 7, 3), (300, 257, 1, 0, 1), (1000, 64, 100003, 2147483646, 99991)])
def test_pair_embedding_over_steps(dtype, V, D, buckets, mul_prev, mul_cur):
    """Four sequences whose pieces come in several steps, single tokens and padding rows among them; the last tokens of slots that
    a step does not have stay what they are."""
    from mynah_slm_b200.ops import kernels
    rng = np.random.default_rng(V)
    table, pairs = (torch.tensor(rng.normal(size=(n, D)), dtype=dtype, device=DEV) for n in (V, buckets + 1))
    lens, slots = [40, 7, 1, 90], [3, 0, 4, 1]
    seqs = [rng.integers(0, V, n).tolist() for n in lens]
    big = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    want = [table.double().cpu().numpy()[s] + pairs.double().cpu().numpy()[plain.pair_rows(s, big)] for s in seqs]
    cuts = [[0, 1, 3, 39, 40], [0, 5, 6, 7, 7], [0, 0, 0, 1, 1], [0, 64, 65, 67, 90]]
    last = torch.full((6,), -77, dtype=torch.int32, device=DEV)          # what a slot's former user left, far outside the vocabulary
    got = [[] for _ in seqs]
    for i in range(4):
        live = [b for b in (2, 0, 3, 1) if cuts[b][i + 1] > cuts[b][i]]
        toks, seq, pos, cu = [], [], [], [0]
        for n, b in enumerate(live):
            lo, hi = cuts[b][i], cuts[b][i + 1]
            toks, seq, pos = toks + seqs[b][lo:hi], seq + [n] * (hi - lo), pos + list(range(lo, hi))
            cu.append(len(toks))
        ctx = SimpleNamespace(tokens=i32(toks + [0, 0]), tok_seq=i32(seq + [-1, -1]), tok_pos=i32(pos + [0, 0]), cu_q=i32(cu + [cu[-1]]),
                              slots=i32([slots[b] for b in live] + [-1]), status=torch.zeros((1,), dtype=torch.int32, device=DEV))
        before = last.cpu().numpy().copy()
        x = kernels.embed_pairs(table, pairs, last, ctx, mul_prev % buckets, mul_cur % buckets).double().cpu().numpy()
        assert int(ctx.status.item()) == 0 and np.all(x[len(toks):] == 0)
        for n, b in enumerate(live):
            got[b].append(x[cu[n]:cu[n + 1]])
        after = last.cpu().numpy()
        for s in range(6):
            b = [b for b in live if slots[b] == s]
            assert after[s] == (seqs[b[0]][cuts[b[0]][i + 1] - 1] if b else before[s])
    for w, g in zip(want, got):
        assert rel(w, np.concatenate(g)) < 1e-6


# ------------------------------------------------------------------ attention with sinks
def run_sink(dtype, H, KV, d, vd, dp, vdp, q_lens, starts, window, scale, sinks, seed, tc=True, sharp=None, shift=0.0):
    """Attention through the dispatch on heads stored `dp` / `vdp` wide; the reference on the heads that exist. `shift` is
    added to every score by a constant channel; `sharp` makes one key of sequence 0 stand out."""
    from mynah_slm_b200.ops import attention_dispatch
    rng = np.random.default_rng(seed)
    ctx, pages, n_pages = step_ctx(q_lens, starts)
    ids, indptr = pages.ids.cpu().numpy(), pages.indptr.cpu().numpy()
    T = sum(q_lens)
    hold = lambda x: torch.tensor(x, dtype=dtype).double().numpy()
    rnd = lambda *shape: hold(rng.normal(size=shape))
    q, k, v = rnd(T, H, d), [rnd(s + n, KV, d) for n, s in zip(q_lens, starts)], [rnd(s + n, KV, vd) for n, s in zip(q_lens, starts)]
    if shift:
        q[..., 1] = 1.0
        for kb in k:
            kb[..., 1] = hold(np.full(kb.shape[:-1], shift / scale))
    if sharp is not None:
        q[..., 0] = 12.0
        for kb in k:
            kb[..., 0] = 0.0
        k[0][sharp, :, 0] = 12.0
    k_cache, v_cache = torch.zeros((n_pages, KV, PAGE, dp), dtype=dtype, device=DEV), torch.zeros((n_pages, KV, PAGE, vdp), dtype=dtype, device=DEV)
    for b in range(len(q_lens)):
        for p in range(k[b].shape[0]):
            page = ids[indptr[b] + p // PAGE]
            k_cache[page, :, p % PAGE, :d] = torch.tensor(k[b][p], dtype=dtype, device=DEV)
            v_cache[page, :, p % PAGE, :vd] = torch.tensor(v[b][p], dtype=dtype, device=DEV)
    qt = torch.zeros((T, H, dp), dtype=dtype, device=DEV)
    qt[..., :d] = torch.tensor(q, dtype=dtype, device=DEV)
    vdo = (vd + 7) // 8 * 8
    out = torch.full((T, H * vdo), 9.0, dtype=dtype, device=DEV)
    st = None if sinks is None else t32(sinks)
    before = attention_dispatch.USE_TC_MASKED
    attention_dispatch.USE_TC_MASKED = tc
    try:
        if ctx.is_decode:
            scratch = torch.empty((ctx.B * H * ctx.decode_splits * (max(dp, vdp) + 2),), dtype=torch.float32, device=DEV)
            attention_dispatch.decode_capped(qt.view(T, -1), out, ctx, H, KV, dp, vdp, k_cache, v_cache, pages, window or 0, scale, 0.0, 0, 1,
                                             scratch, vdo=vdo, sink=st)
        else:
            attention_dispatch.prefill_capped(qt.view(T, -1), out, ctx, H, KV, dp, vdp, k_cache, v_cache, pages, window or 0, scale, 0.0, 0, 1,
                                              vdo=vdo, sink=st)
    finally:
        attention_dispatch.USE_TC_MASKED = before
    assert int(ctx.status.item()) == 0
    got = out.double().cpu().numpy().reshape(T, H, vdo)
    assert np.all(got[..., vd:] == 0)
    ref, at = np.zeros((T, H, vd)), 0
    for b, (n, s) in enumerate(zip(q_lens, starts)):
        see = plain.visible(s + n, {"size": window} if window else None)[s:]
        for h in range(H):
            sc = q[at:at + n, h] @ k[b][:, h // (H // KV)].T * scale
            ref[at:at + n, h] = plain.softmax_rows(sc, see, None if sinks is None else float(np.float32(sinks[h]))) @ v[b][:, h // (H // KV)]
        at += n
    return ref, got[..., :vd], v


STEPS = (([150], [0]), ([1, 70, 33], [0, 0, 0]), ([40, 2], [100, 63]), ([1, 1, 1], [0, 200, 64]), ([300, 129], [0, 7]))


@pytest.mark.parametrize("window", [None, 1, 63, 64, 65, 100])
@pytest.mark.parametrize("H,KV,d,vd", [(4, 2, 16, 24), (3, 1, 10, 7), (2, 2, 200, 256), (6, 2, 64, 40)])
def test_general_attention_with_sinks(H, KV, d, vd, window):
    p8 = lambda n: (n + 7) // 8 * 8
    sinks = np.linspace(-1.0, 4.0, H)
    for q_lens, starts in STEPS:
        ref, got, _ = run_sink(torch.float32, H, KV, d, vd, p8(d), p8(vd), q_lens, starts, window, 0.3, sinks, H + d, tc=False)
        assert rel(ref, got) < 2e-5, (q_lens, starts)


@pytest.mark.parametrize("window", [None, 1, 64, 75, 129])
@pytest.mark.parametrize("H,KV,d,vd,dp,vdp", [(4, 2, 64, 64, 64, 64), (4, 2, 128, 64, 128, 64), (4, 1, 64, 128, 64, 128), (2, 2, 128, 128, 128, 128),
                                              (6, 2, 40, 72, 64, 128), (6, 3, 64, 56, 64, 64), (16, 1, 48, 88, 64, 128)])
def test_tensor_core_attention_with_sinks(H, KV, d, vd, dp, vdp, window):
    """bfloat16: every pair of stored widths, heads narrower than stored, against the reference and the general kernels."""
    sinks = np.linspace(-2.0, 3.0, H)
    for q_lens, starts in STEPS:
        args = (torch.bfloat16, H, KV, d, vd, dp, vdp, q_lens, starts, window, d ** -0.5, sinks, d + H)
        ref, tc, _ = run_sink(*args)
        _, gen, _ = run_sink(*args, tc=False)
        assert rel(ref, tc) < 2e-2 and rel(ref, gen) < 2e-2 and rel(gen, tc) < 2e-2, (q_lens, starts)


@pytest.mark.parametrize("dtype,d", [(torch.float32, 16), (torch.bfloat16, 64)])
@pytest.mark.parametrize("shift,sink", [(-200.0, 0.0), (0.0, 200.0), (-6.0, -4.0), (6.0, 5.0), (100.0, 1.0), (0.0, -300.0), (90.0, 95.0)])
def test_sinks_far_above_and_below_the_scores(dtype, d, shift, sink):
    for q_lens, starts in (([130], [0]), ([1, 1], [140, 3])):
        ref, got, v = run_sink(dtype, 2, 1, d, d, d, d, q_lens, starts, 40, 0.25, [sink, sink + 0.5], 3, shift=shift)
        assert np.all(np.isfinite(got))
        tol = 2e-4 if dtype == torch.float32 else 3e-2
        assert np.abs(ref - got).max() < tol * max(np.abs(ref).max(), 1e-6), (shift, sink, q_lens)
        if sink - shift >= 200.0:
            assert np.abs(got).max() < 1e-20
        if shift - sink > 50.0:
            assert rel(run_sink(dtype, 2, 1, d, d, d, d, q_lens, starts, 40, 0.25, None, 3, shift=shift)[1], got) < 1e-3


@pytest.mark.parametrize("dtype,d,vd,dp,vdp", [(torch.float32, 16, 24, 16, 24), (torch.bfloat16, 48, 80, 64, 128), (torch.bfloat16, 64, 56, 64, 64)])
@pytest.mark.parametrize("window", [30, 64, 127])
def test_one_key_stands_out_inside_the_window_only(dtype, d, vd, dp, vdp, window):
    """ONE key of hundreds is large along the direction every query looks in: the queries from it to the last that the window
    reaches return its value, no other one does, in a prompt, in a later piece and for single queries at the window's edge."""
    n = 345
    for key in (0, 1, 63, 64, 65, 127, 128, 200):
        edge = key + window - 1
        for q_lens, starts in (([n], [0]), ([n - 190], [190]), ([1], [edge]), ([1], [edge + 1]), ([1], [key])):
            ref, got, v = run_sink(dtype, 2, 2, d, vd, dp, vdp, q_lens, starts, window, 1.0, [0.5, 3.0], key, sharp=key)
            assert rel(ref, got) < (1e-4 if dtype == torch.float32 else 3e-2), (key, q_lens, starts)
            for r, p in enumerate(range(starts[0], starts[0] + q_lens[0])):
                assert (rel(v[0][key], got[r]) < 0.05) == (key <= p <= edge), (key, p)


# ------------------------------------------------------------------ preparation, row norms
@pytest.mark.parametrize("writes", [True, False])
@pytest.mark.parametrize("vnorm", [True, False])
@pytest.mark.parametrize("H,G,dim,vd,rot,dimp,vdp", [(4, 2, 16, 24, 12, 64, 64), (3, 1, 10, 7, 6, 16, 8), (6, 3, 48, 80, 48, 64, 128), (4, 2, 64, 128, 32, 64, 128),
                                                     (2, 1, 128, 64, 0, 128, 64), (6, 3, 64, 56, 16, 64, 64), (16, 8, 128, 128, 32, 128, 128), (2, 2, 40, 24, 16, 64, 64)])
def test_preparation_with_whole_projection_norms(H, G, dim, vd, rot, dimp, vdp, vnorm, writes):
    from mynah_slm_b200.ops import kernels
    from mynah_slm_b200.parts.position import rotary_frequencies
    rng = np.random.default_rng(H * 10 + dim)
    T, nq, nk, nv = 130, H * dim, G * dim, G * vd
    x = rng.normal(size=(T, nq + ((nk + nv) if writes else 0)))
    gq, gk = 1.0 + 0.2 * rng.normal(size=nq), 1.0 + 0.2 * rng.normal(size=nk)
    ctx, pages, n_pages = step_ctx([T], [0])
    cos = sin = None
    r = {"dims": rot, "base": 300.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100}}
    if rot:
        cos, sin = kernels.rope_table_freqs(256, *rotary_frequencies(rot, 300.0, {"kind": "wavelength", **r["scaling"]}), DEV)
    k_cache = torch.full((n_pages, G, PAGE, dimp), 9.0, dtype=torch.float32, device=DEV)
    v_cache = torch.full((n_pages, G, PAGE, vdp), 9.0, dtype=torch.float32, device=DEV)
    q_out = torch.full((T, H * dimp), 9.0, dtype=torch.float32, device=DEV)
    kernels.attn_prep(t32(x), q_out, H, G, dim, vd, dimp, vdp, t32(gq), t32(gk) if writes else t32(gq), EPS, cos, sin, rot, ctx, pages,
                      k_cache if writes else None, v_cache if writes else None, None, None, 0, vnorm)
    assert int(ctx.status.item()) == 0
    turn = (lambda y: plain.turn(y, r, False)) if rot else (lambda y: y)
    q = turn((plain.rms_unit(x[:, :nq], EPS) * gq).reshape(T, H, dim))
    got_q = q_out.view(T, H, dimp).cpu().numpy()
    assert rel(q, got_q[..., :dim]) < 1e-5 and np.all(got_q[..., dim:] == 0)
    if not writes:
        return
    k, v = turn((plain.rms_unit(x[:, nq:nq + nk], EPS) * gk).reshape(T, G, dim)), x[:, nq + nk:].reshape(T, G, vd)
    ids = pages.ids.cpu().numpy()
    got_k = torch.stack([k_cache[ids[p // PAGE], :, p % PAGE] for p in range(T)]).cpu().numpy()
    got_v = torch.stack([v_cache[ids[p // PAGE], :, p % PAGE] for p in range(T)]).cpu().numpy()
    for ref, got, n in ((k, got_k, dim), (plain.rms_unit(v, EPS) if vnorm else v, got_v, vd)):
        assert rel(ref, got[..., :n]) < 1e-5 and np.all(got[..., n:] == 0)
    untouched = [p for p in range(n_pages) if p not in set(ids.tolist())]
    assert float(k_cache[untouched].min()) == 9.0 and float(v_cache[untouched].min()) == 9.0


@pytest.mark.parametrize("n", [5, 80, 128, 1000, 1600])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_row_norms_of_a_column_slice(n, dtype):
    from mynah_slm_b200.ops import kernels
    rng = np.random.default_rng(n)
    wide = torch.tensor(rng.normal(size=(7, n + 24)), dtype=dtype, device=DEV)
    g = 1.0 + 0.3 * rng.normal(size=n)
    got = kernels.rms_rows(wide, n, t32(g), 1e-3).double().cpu().numpy()
    ref = plain.rms_unit(wide[:, :n].double().cpu().numpy(), 1e-3) * np.float32(g)
    assert rel(ref, got) < (1e-6 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("D", [44, 64, 131, 1024, 4100])
def test_norm_behind_a_sublayer_leaves_a_rounded_copy(D):
    from mynah_slm_b200.ops import kernels
    rng = np.random.default_rng(D)
    x, y, g = rng.normal(size=(9, D)), 5.0 * rng.normal(size=(9, D)), rng.normal(size=D)
    xt, copy = t32(x), torch.empty((9, D), dtype=torch.bfloat16, device=DEV)
    assert kernels.rmsnorm_add(xt, t32(y), t32(g), 1e-3, copy=copy) is None
    assert rel(x + plain.rms_unit(y, 1e-3) * g, xt.cpu().numpy()) < 1e-6
    assert torch.equal(copy, xt.to(torch.bfloat16))


# ------------------------------------------------------------------ recurrence with a fixed decay
def fixed_case(dtype, H, dim, vd, lens, decay, seed):
    rng = np.random.default_rng(seed)
    T = sum(lens)
    hold = lambda x: torch.tensor(x, dtype=dtype).double().numpy()
    parts = {"q": hold(rng.normal(size=(T, H, dim))), "k": hold(rng.normal(size=(T, H, dim))),
             "v": hold(rng.normal(size=(T, H, vd))), "g": hold(1.5 * rng.normal(size=(T, H, vd)))}
    rows, at, col = [], {}, 0
    for name, x in parts.items():
        x = x.reshape(T, -1)
        at[name] = col
        rows.append(np.pad(x, ((0, 0), (0, -x.shape[1] % 8))))
        col += rows[-1].shape[1]
    refs, lo = [], 0
    for n in lens:
        s = slice(lo, lo + n)
        o = plain.retention_heads(parts["q"][s], parts["k"][s] * dim ** -0.5, parts["v"][s], np.asarray(decay, dtype=np.float64))
        refs.append(plain.rms_unit(o, EPS).reshape(n, -1) * plain.silu(parts["g"][s].reshape(n, -1)))
        lo += n
    logs = [np.log2(x) if x > 0 else -1e30 for x in decay]
    return SimpleNamespace(H=H, dim=dim, vd=vd, lens=lens, at=at, refs=refs, dtype=dtype, bias=t32(list(decay) + logs),
                           p=torch.tensor(np.concatenate(rows, 1), dtype=dtype, device=DEV))


def run_fixed(case, cuts, slots, S, chunk_min=None):
    from mynah_slm_b200.ops import kernels
    starts, got, width = np.cumsum([0] + case.lens), [[] for _ in case.lens], case.H * case.vd
    before = kernels.gated_memory_chunk_min(chunk_min) if chunk_min is not None else None
    try:
        for i in range(len(cuts[0]) - 1):
            pieces = [case.p[starts[b] + c[i]: starts[b] + c[i + 1]] for b, c in enumerate(cuts)]
            cu = np.cumsum([0] + [len(x) for x in pieces])
            ctx = SimpleNamespace(cu_q=i32(cu), slots=i32(slots), B=len(slots), max_q_len=int(np.diff(cu).max()), is_decode=bool(np.diff(cu).max() == 1))
            p = torch.cat(pieces, 0).contiguous()
            out = torch.full((p.shape[0], width), 9.0, dtype=case.dtype, device=DEV)
            kernels.gated_memory("fixed", p, case.at, None, case.bias, torch.ones((width,), device=DEV), case.dim ** -0.5, {"S": S}, out, ctx,
                                 case.H, case.dim, case.vd, EPS)
            for b in range(len(slots)):
                got[b].append(out[cu[b]:cu[b + 1]].double().cpu().numpy())
    finally:
        if before is not None:
            kernels.gated_memory_chunk_min(before)
    return [np.concatenate(g, 0) for g in got]


DECAYS = {1: [0.97], 2: [1.0, 0.9], 3: [0.99, 0.0, 0.999], 4: [0.5, 0.97, 0.999, 1.0], 5: [0.9, 0.8, 0.7, 0.95, 0.999]}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dim,vd", [(3, 24, 16), (1, 5, 7), (2, 128, 128), (4, 64, 24), (1, 256, 160), (5, 11, 3), (2, 40, 256), (2, 16, 72)])
def test_fixed_decay_in_steps(dtype, H, dim, vd):
    """Four sequences: whole; in pieces around the chunk's edges down to single tokens; token by token. States go from step
    to step, slots that no sequence of the step has keep what they hold."""
    lens, slots = [150, 1, 66, 2], [4, 0, 2, 3]
    case = fixed_case(dtype, H, dim, vd, lens, DECAYS[H], H + dim)
    pieces = [[0, 3, 67, 131, 150], [0, 1, 1, 1, 1], [0, 2, 3, 65, 66], [0, 0, 1, 2, 2]]
    for cuts in ([[0, n] for n in lens], pieces, [[min(i, n) for i in range(151)] for n in lens]):
        S = torch.full((7, H, dim, vd), 7.0, dtype=torch.float32, device=DEV)
        S[slots] = 0.0
        for ref, g in zip(case.refs, run_fixed(case, cuts, slots, S)):
            # a small q . k leaves the first rows of a sequence to rounding in any form: every row is held by its own size
            assert rel(ref, g) < (2e-5 if dtype == torch.float32 else 1.5e-2), (cuts[0][:5], rel(ref, g))
        assert float(S[[1, 5, 6]].min()) == 7.0 and float(S[[1, 5, 6]].max()) == 7.0


@pytest.mark.parametrize("H,dim,vd", [(2, 128, 128), (3, 64, 128), (1, 256, 256), (4, 16, 40)])
def test_fixed_decay_chunk_form_against_token_form(H, dim, vd):
    lens = [300, 64, 65, 17]
    case = fixed_case(torch.bfloat16, H, dim, vd, lens, DECAYS[H], 5 * H + dim)
    runs = []
    for chunk_min in (0, 2):
        S = torch.zeros((5, H, dim, vd), dtype=torch.float32, device=DEV)
        runs.append((run_fixed(case, [[0, n] for n in lens], [3, 1, 0, 2], S, chunk_min), S[:4].double().cpu().numpy()))
    for ref, a, b in zip(case.refs, runs[0][0], runs[1][0]):
        assert rel(ref, a) < 1e-2 and rel(ref, b) < 1e-2 and rel(a, b) < 1e-2
    assert rel(runs[0][1], runs[1][1]) < 1e-4                             # fp32 states: the operands' two summands carry them


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_early_token_is_remembered(dtype):
    """A key that one late query alone looks for, 400 tokens back: its value comes out, decayed, and only for that query."""
    H, dim, vd, n = 1, 32, 16, 420
    case = fixed_case(dtype, H, dim, vd, [n], [0.999], 3)
    p = case.p.clone()
    q, k, v = (case.at[x] for x in "qkv")
    p[:, q] = 0.0
    p[:, k] = 0.0
    p[5, k], p[405, q] = 64.0, 64.0
    case.p = p
    S = torch.zeros((2, H, dim, vd), dtype=torch.float32, device=DEV)
    out = run_fixed(case, [[0, n]], [0], S)[0]
    g = case.at["g"]
    gate = plain.silu(p[:, g:g + vd].double().cpu().numpy())
    unit = lambda t: plain.rms_unit(p[t:t + 1, v:v + vd].double().cpu().numpy(), EPS)[0]
    assert rel(unit(5), out[405] / gate[405]) < 0.15 and rel(unit(5), out[404] / gate[404]) > 0.3


# ------------------------------------------------------------------ per-head products with a gate a value
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,n_in,n_out", [(5, 64, 40), (3, 20, 20), (2, 128, 72), (5, 7, 9)])
def test_head_products_with_a_gate_a_value(dtype, H, n_in, n_out):
    from mynah_slm_b200.ops import kernels
    rng = np.random.default_rng(H * n_in)
    for T in (1, 3, 70):
        hold = lambda *s: torch.tensor(rng.normal(size=s), dtype=dtype, device=DEV)
        pad = (n_in + 7) // 8 * 8
        x, W, gate = hold(T, H * pad), hold(H, n_out, n_in), hold(T, 5 + H * n_out)
        out = torch.full((T, H * n_out), 9.0, dtype=dtype, device=DEV)
        kernels.head_linear(x, pad, 0, W, out, n_out, 0, gate=gate[:, 5:], gate_cols=True)
        xr = x.double().cpu().numpy().reshape(T, H, pad)[..., :n_in]
        ref = np.einsum("thi,hji->thj", xr, W.double().cpu().numpy()).reshape(T, -1) * plain.sigmoid(gate[:, 5:].double().cpu().numpy())
        assert rel(ref, out.double().cpu().numpy()) < (1e-5 if dtype == torch.float32 else 1e-2)


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("D,F,E,top,FS", [(48, 24, 10, 3, 40), (64, 40, 12, 1, 40), (44, 12, 1, 1, 9), (40, 10, 7, 7, 10), (48, 16, 6, 2, 16),
                                          (96, 200, 72, 4, 56), (52, 18, 9, 2, 0), (264, 104, 11, 1, 104)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_squared_relu_experts_with_weights_on_their_inputs(dtype, D, F, E, top, FS):
    """Through the part: scores, choices, weights on the inputs, the shared expert as an expert of the stack or with products of
    its own; padding rows stay out. bfloat16: tiles on tensor cores, the plain tiles, and the grouped tcgen05 form."""
    from mynah_slm_b200.config.spec import PartSpec
    from mynah_slm_b200.ops import kernels
    from mynah_slm_b200.parts.feedforward_routed import GroupRouterExperts
    rng = np.random.default_rng(D + E)
    W = {"router": 2.0 * rng.normal(size=(E, D)) / np.sqrt(D)}
    for e in [f"e{e}" for e in range(E)] + (["shared"] if FS else []):
        f = FS if e == "shared" else F
        W[f"{e}.up"], W[f"{e}.down"] = 2 * rng.normal(size=(f, D)) / np.sqrt(D), rng.normal(size=(D, f)) / np.sqrt(f)
    dev = {k: torch.tensor(v, dtype=dtype, device=DEV) for k, v in W.items()}
    W = {k: v.double().cpu().numpy() for k, v in dev.items()}
    part = GroupRouterExperts(PartSpec("group_router_experts", {
        "hidden_size": D, "intermediate_size": F, "experts": E, "top": top, "activation": "relu2", "weights_on": "input", "output": "fp32",
        "router": "router", "expert_prefix": "e", "shared": FS or None, "shared_prefix": "shared."}))
    part.bind(dev, None)
    assert part.shared_in_stack == (FS == F)
    mlp = {"router": {"experts": E, "top": top}, "shared": {"ff": FS} if FS else None}
    for T in (1, 5, 90, 700):
        hp = torch.cat([torch.tensor(rng.normal(size=(T, D)), dtype=dtype), torch.full((1, D), 100.0, dtype=dtype)], 0).to(DEV).contiguous()
        margins = []
        ref = plain.routed_ff(hp[:T].double().cpu().numpy(), W, "", mlp, margins)
        steady = margins[0] > (1e-4 if dtype == torch.float32 else 1e-3)
        ctx = SimpleNamespace(tok_seq=i32([0] * T + [-1]), status=torch.zeros((1,), dtype=torch.int32, device=DEV))
        for form in ("tiles",) if dtype == torch.float32 else ("tiles", "plain", "grouped"):
            before = kernels.moe_plain(form == "plain"), kernels.moe_grouped_min(2 if form == "grouped" else 0)
            try:
                got = part.forward(hp, ctx)[:T]
            finally:
                kernels.moe_plain(before[0]), kernels.moe_grouped_min(before[1])
            assert int(ctx.status.item()) == 0 and got.dtype == torch.float32
            err = rel(ref[steady], got.double().cpu().numpy()[steady])
            assert steady.mean() > 0.9 and err < (2e-5 if dtype == torch.float32 else 2e-2), (T, form, err)


def test_scores_that_round_to_one_still_choose_by_their_order():
    """Logits beyond what a 32-bit sigmoid tells apart: the larger one is chosen although it stands behind."""
    from mynah_slm_b200.ops import kernels
    E, D = 6, 16
    W = torch.zeros((E, D), device=DEV)
    W[:, 0] = torch.tensor([30.0, -5.0, 41.0, 40.0, 2.0, 45.0], device=DEV)
    h = torch.zeros((1, D), device=DEV)
    h[0, 0] = h[0, 1] = 1.0
    up = torch.zeros((E, 4, D), device=DEV)
    up[:, :, 1] = 1.0
    down = (10.0 ** torch.arange(E, device=DEV)).view(E, 1, 1).expand(E, D, 4).contiguous()
    ctx = SimpleNamespace(tok_seq=i32([0]), status=torch.zeros((1,), dtype=torch.int32, device=DEV))
    out = kernels.moe_group_router_ffn(h, W, None, up, down, ctx, 2, 1, 1, 1.0, None, 1.0, activation="relu2", weights_on="input")
    assert abs(float(out[0, 0]) - 4 * (1e5 + 1e2)) < 1.0 and int(ctx.status.item()) == 0


@pytest.mark.parametrize("M", [1, 8, 100, 129, 600, 2048])
def test_product_with_a_squared_relu(M):
    from mynah_slm_b200.ops import kernels
    rng = np.random.default_rng(M)
    x, w = (torch.tensor(rng.normal(size=s), dtype=torch.bfloat16, device=DEV) for s in ((M, 264), (520, 264)))
    ref = np.maximum(x.double().cpu().numpy() @ w.double().cpu().numpy().T, 0.0) ** 2
    assert rel(ref, kernels.linear_relu2(x, w).double().cpu().numpy()) < 1e-2
    xf, wf = x.float(), w.float()
    assert rel(ref, kernels.linear_relu2(xf, wf).double().cpu().numpy()) < 1e-5
