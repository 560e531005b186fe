"""The kernels behind the Buludra parts, each alone, against the plain functions of tests/plain/buludra.py (float64): the
recurrences with learned decays (token form and chunk form, several sequences, states handed over between steps, decays
and gates at their extremes), attention with a null key, an output factor and heads of two widths (general and tensor-core
forms, one key made to stand out far back and at page borders), the preparation with unit norms and query factors, softmax
routing with groups by their largest score and a shared expert, and capped logits."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from plain import buludra as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64


def i32(v):
    return torch.tensor(np.asarray(v), dtype=torch.int32, device=DEV)


def t32(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)


def rel(ref, got):
    ref, got = np.asarray(ref, dtype=np.float64), np.asarray(got, dtype=np.float64)
    return float(np.abs(ref - got).max() / max(np.abs(ref).max(), 1e-30))


# ------------------------------------------------------------------ recurrences
EPS = 1e-5


def memory_case(kind, dtype, H, dim, vd, rank, lens, seed, z_mean=1.0, z_std=1.0, gate_std=1.0, cap=15.0, tau=16.0):
    """Random rows of a stacked projection for sequences of `lens` tokens, what the kernel takes beside them, and the plain
    outputs of every sequence (norm and gate included)."""
    rng = np.random.default_rng(seed)
    T = sum(lens)
    hold = lambda x: torch.tensor(x, dtype=dtype).double().numpy()       # values the type holds
    q, k = hold(rng.normal(size=(T, H, dim))), hold(rng.normal(size=(T, H, dim)))
    v, g = hold(rng.normal(size=(T, H, vd))), hold(1.5 * rng.normal(size=(T, H, vd)))
    pieces, at, col = [], {}, 0

    def put(name, x):
        nonlocal col
        x = x.reshape(T, -1)
        pad = -x.shape[1] % 8
        at[name] = col
        pieces.append(np.pad(x, ((0, 0), (0, pad))))
        col += x.shape[1] + pad
    for name, x in (("q", q), ("k", k), ("v", v), ("g", g)):
        put(name, x)
    case = SimpleNamespace(kind=kind, dtype=dtype, H=H, dim=dim, vd=vd, lens=lens, at=at, tau=tau, cap=cap, w2=None)
    if kind == "gla":
        r, w2 = hold(rng.normal(size=(T, rank))), hold(z_std * rng.normal(size=(H * dim, rank)) / np.sqrt(rank))
        b = np.float32(z_mean + 0.5 * rng.normal(size=(H * dim,))).astype(np.float64)
        put("a", r)
        log_a = (plain.log_sigmoid(r @ w2.T + b) / tau).reshape(T, H, dim)
        w = np.float32(np.tile(1.0 + 0.1 * rng.normal(size=(vd,)), H)).astype(np.float64)
        case.w2, case.bias = torch.tensor(w2, dtype=dtype, device=DEV), t32(b)
        run = lambda s: plain.gated_linear_heads(q[s] * dim ** -0.5, k[s], v[s], log_a[s])
        act = plain.silu
    else:
        pi, pf = hold(gate_std * rng.normal(size=(T, H))), hold(z_mean + gate_std * rng.normal(size=(T, H)))
        b = np.float32(0.5 * rng.normal(size=(2 * H,))).astype(np.float64)
        put("i", pi)
        put("f", pf)
        log_i, log_f = cap * np.tanh((pi + b[:H]) / cap), plain.log_sigmoid(cap * np.tanh((pf + b[H:]) / cap))
        w = np.float32(1.0 + 0.1 * rng.normal(size=(H * vd,))).astype(np.float64)
        case.bias = t32(b)
        run = lambda s: plain.matrix_memory_heads(q[s] * dim ** -0.5, k[s], v[s], log_i[s], log_f[s])
        act = plain.sigmoid
    case.w_norm = t32(w)
    case.p = torch.tensor(np.concatenate(pieces, 1), dtype=dtype, device=DEV)
    refs, lo = [], 0
    for n in lens:
        s = slice(lo, lo + n)
        o = plain.rms_unit(run(s), EPS).reshape(n, -1) * w * act(g[s].reshape(n, -1))
        refs.append(o)
        lo += n
    case.refs = refs
    return case


def fresh_state(case, n_slots):
    z = lambda *shape: torch.full((n_slots + 1, *shape), 7.0, dtype=torch.float32, device=DEV)
    s = {"S": z(case.H, case.dim, case.vd)}
    if case.kind == "mlstm":
        s.update(n=z(case.H, case.dim), m=z(case.H))
    return s


def run_memory(case, cuts, slots, state, chunk_min=None):
    """The case's sequences in steps: step i brings tokens [cuts[b][i], cuts[b][i + 1]) of every sequence b."""
    from mynah_slm_b200.ops import kernels
    starts = np.cumsum([0] + case.lens)
    got = [[] for _ in case.lens]
    width = case.H * case.vd
    before = kernels.gated_memory_chunk_min(chunk_min) if chunk_min is not None else None
    try:
        for i in range(len(cuts[0]) - 1):
            rows, cu, sl = [], [0], []
            for b in range(len(case.lens)):
                lo, hi = cuts[b][i], cuts[b][i + 1]
                rows.append(case.p[starts[b] + lo: starts[b] + hi])
                cu.append(cu[-1] + hi - lo)
                sl.append(slots[b])
            p = torch.cat(rows, 0).contiguous()
            q_lens = np.diff(cu)
            ctx = SimpleNamespace(cu_q=i32(cu), slots=i32(sl), B=len(sl), max_q_len=int(q_lens.max()), is_decode=bool(q_lens.max() == 1))
            out = torch.full((p.shape[0], width + 8), 9.0, dtype=case.dtype, device=DEV)
            kernels.gated_memory(case.kind, p, case.at, case.w2, case.bias, case.w_norm, case.dim ** -0.5, state, out[:, :width],
                                 ctx, case.H, case.dim, case.vd, EPS, case.tau, case.cap)
            assert float(out[:, width:].float().min()) == 9.0            # the columns behind are another branch's
            for b in range(len(sl)):
                got[b].append(out[cu[b]:cu[b + 1], :width].double().cpu().numpy())
    finally:
        if before is not None:
            kernels.gated_memory_chunk_min(before)
    return [np.concatenate(g, 0) for g in got]


def zero_slots(state, slots):
    for t in state.values():
        t[slots] = 0.0


SIZES = [(3, 24, 16, 6), (1, 5, 7, 3), (2, 128, 128, 16), (4, 64, 24, 20), (1, 256, 160, 40), (5, 11, 3, 1), (2, 40, 256, 8), (2, 16, 72, 64)]


@pytest.mark.parametrize("kind", ["gla", "mlstm"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dim,vd,rank", SIZES)
def test_recurrence_in_steps(kind, dtype, H, dim, vd, rank):
    """Four sequences: whole; in pieces around the chunk's edges down to single tokens; token by token. States go from step
    to step, slots that no sequence of the step has keep what they hold."""
    lens = [150, 1, 66, 2]
    case = memory_case(kind, dtype, H, dim, vd, rank, lens, H + dim)
    slots, tol = [4, 0, 2, 3], (2e-5 if dtype == torch.float32 else 1.5e-2)
    whole = [[0, n] for n in lens]
    pieces = [[0, 3, 67, 131, 150], [0, 1, 1, 1, 1], [0, 2, 3, 65, 66], [0, 0, 1, 2, 2]]
    singles = [[min(i, n) for i in range(151)] for n in lens]
    for cuts in (whole, pieces, singles):
        state = fresh_state(case, 6)
        zero_slots(state, slots)
        got = run_memory(case, cuts, slots, state)
        for ref, g in zip(case.refs, got):
            assert rel(ref, g) < tol, (kind, dtype, cuts[0][:5], rel(ref, g))
        for t in state.values():                                         # slots 1 and 5 and the spare row: untouched
            assert float(t[[1, 5, 6]].min()) == 7.0 and float(t[[1, 5, 6]].max()) == 7.0


@pytest.mark.parametrize("kind", ["gla", "mlstm"])
@pytest.mark.parametrize("H,dim,vd", [(2, 128, 128), (3, 64, 128), (1, 256, 256), (2, 16, 40)])
def test_chunk_form_against_token_form(kind, H, dim, vd):
    """The same bfloat16 rows through both forms, and the states they leave."""
    lens = [300, 64, 65, 17]
    case = memory_case(kind, torch.bfloat16, H, dim, vd, 16, lens, 5 * H + dim)
    runs = []
    for chunk_min in (0, 2):
        state = fresh_state(case, 4)
        zero_slots(state, [0, 1, 2, 3])
        got = run_memory(case, [[0, n] for n in lens], [3, 1, 0, 2], state, chunk_min)
        runs.append((got, {k: t[:4].double().cpu().numpy() for k, t in state.items()}))
    for ref, a, b in zip(case.refs, runs[0][0], runs[1][0]):
        assert rel(ref, a) < 1e-2 and rel(ref, b) < 1e-2 and rel(a, b) < 1e-2
    for k in runs[0][1]:
        assert rel(runs[0][1][k], runs[1][1][k]) < 1e-4, k               # fp32 states: the operands' two summands carry them


@pytest.mark.parametrize("what", ["vanishing", "mixed", "slow", "capped", "closed", "rising"])
def test_extreme_decays_and_gates(what):
    """Decays that vanish within a token (a chunk's exponents then go far beyond what factors of both operands could hold),
    decays next to one, gates at their caps, input gates that rise through a chunk."""
    for dtype in (torch.float32, torch.bfloat16):
        tol = 5e-5 if dtype == torch.float32 else 2e-2
        lens = [200, 70]
        if what in ("vanishing", "mixed", "slow"):
            z = {"vanishing": dict(z_mean=-20.0, z_std=5.0, tau=1.0), "mixed": dict(z_mean=-2.0, z_std=8.0, tau=1.0),
                 "slow": dict(z_mean=9.0, z_std=0.5, tau=32.0)}[what]
            case = memory_case("gla", dtype, 2, 32, 24, 8, lens, 3, **z)
        else:
            z = {"capped": dict(gate_std=40.0, cap=15.0), "closed": dict(z_mean=-30.0, gate_std=1.0, cap=20.0),
                 "rising": dict(z_mean=6.0, gate_std=12.0, cap=30.0)}[what]
            case = memory_case("mlstm", dtype, 2, 32, 24, 8, lens, 4, **z)
        for cuts in ([[0, 200], [0, 70]], [[0, 64, 128, 131, 200], [0, 1, 2, 65, 70]]):
            state = fresh_state(case, 2)
            zero_slots(state, [0, 1])
            for ref, g in zip(case.refs, run_memory(case, cuts, [0, 1], state)):
                assert rel(ref, g) < tol, (what, dtype, rel(ref, g))


@pytest.mark.parametrize("kind", ["gla", "mlstm"])
def test_one_far_token_is_remembered(kind):
    """ONE early token's key is large in a direction that every later query looks in and no other key has: the outputs far
    behind it, in other chunks and in single steps, are its value; where the state is not handed on they are not."""
    for dtype in (torch.float32, torch.bfloat16):
        H, dim, vd, n, far = 2, 32, 32, 400, 5
        case = memory_case(kind, dtype, H, dim, vd, 4, [n], 9, z_mean=14.0, z_std=0.1, gate_std=0.1, tau=32.0)
        p = case.p.double().cpu().numpy()
        q, k = p[:, case.at["q"]:case.at["q"] + H * dim].reshape(n, H, dim), p[:, case.at["k"]:case.at["k"] + H * dim].reshape(n, H, dim)
        q[:] *= 0.01
        q[:, :, 0] = 8.0
        k[:, :, 0] = 0.0
        k[far, :, 0] = 8.0
        case.p = torch.tensor(p, dtype=dtype, device=DEV)
        v = case.p.double().cpu().numpy()[:, case.at["v"]:case.at["v"] + H * vd].reshape(n, H, vd)
        g = case.p.double().cpu().numpy()[:, case.at["g"]:case.at["g"] + H * vd]
        want = plain.rms_unit(v[far], EPS).reshape(-1) * case.w_norm.double().cpu().numpy()
        for cuts in ([0, n], [0, 64, 65, 128, 129, 390] + list(range(391, n + 1))):
            state = fresh_state(case, 1)
            zero_slots(state, [0])
            got = run_memory(case, [cuts], [0], state)[0]
            for t in (far, 63, 64, 65, 200, 399):
                gate = plain.silu(g[t]) if kind == "gla" else plain.sigmoid(g[t])
                assert rel(want * gate, got[t]) < 0.08, (kind, dtype, t)
            gate = plain.silu(g[far - 1]) if kind == "gla" else plain.sigmoid(g[far - 1])
            assert rel(want * gate, got[far - 1]) > 0.3


# ------------------------------------------------------------------ attention with a null key
def step_ctx(q_lens, starts):
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


def run_null(dtype, H, KV, d, vd, dp, vdp, q_lens, starts, scale, null, out_scale, seed, tc=True, sharp=None, shift=0.0):
    """Attention through the dispatch on heads stored `dp` / `vdp` wide; the reference on the heads that exist. `shift` is
    added to every score by a constant channel; `sharp` makes one key of sequence 0 stand out."""
    from mynah_slm_b200.ops import attention_dispatch
    rng = np.random.default_rng(seed)
    ctx, pages, n_pages = step_ctx(q_lens, starts)
    ids, indptr = pages.ids.cpu().numpy(), pages.indptr.cpu().numpy()
    T = sum(q_lens)
    rnd = lambda *shape: torch.tensor(rng.normal(size=shape), dtype=dtype).double().numpy()
    q, k, v = rnd(T, H, d), [rnd(s + n, KV, d) for n, s in zip(q_lens, starts)], [rnd(s + n, KV, vd) for n, s in zip(q_lens, starts)]
    if shift:
        q[..., 1] = 1.0
        for kb in k:
            kb[..., 1] = shift / scale
        k = [torch.tensor(kb, dtype=dtype).double().numpy() for kb in k]
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
    wide = torch.full((T, H * vdo + 16), 9.0, dtype=dtype, device=DEV)    # the heads' columns stand in wider rows
    out = wide[:, 8:8 + H * vdo]
    before = attention_dispatch.USE_TC_MASKED
    attention_dispatch.USE_TC_MASKED = tc
    try:
        if ctx.is_decode:
            scratch = torch.empty((ctx.B * H * ctx.decode_splits * (max(dp, vdp) + 2),), dtype=torch.float32, device=DEV)
            attention_dispatch.decode_capped(qt.view(T, -1), out, ctx, H, KV, dp, vdp, k_cache, v_cache, pages, 0, scale, 0.0, 0, 1,
                                             scratch, null, out_scale, vdo)
        else:
            attention_dispatch.prefill_capped(qt.view(T, -1), out, ctx, H, KV, dp, vdp, k_cache, v_cache, pages, 0, scale, 0.0, 0, 1,
                                              null, out_scale, vdo)
    finally:
        attention_dispatch.USE_TC_MASKED = before
    assert int(ctx.status.item()) == 0
    assert float(wide[:, :8].float().min()) == 9.0 and float(wide[:, 8 + H * vdo:].float().min()) == 9.0
    got = out.double().cpu().numpy().reshape(T, H, vdo)
    assert np.all(got[..., vd:] == 0)
    ref, at = [], 0
    for b, (n, s) in enumerate(zip(q_lens, starts)):
        full = np.zeros((s + n, H, d))
        full[s:] = q[at:at + n]
        ref.append(plain.grouped_heads(full, k[b], v[b], scale, null)[s:].reshape(n, H, vd))
        at += n
    return out_scale * np.concatenate(ref, 0), got[..., :vd], v


STEPS = (([150], [0]), ([1, 70, 33], [0, 0, 0]), ([40, 2], [100, 63]), ([1, 1, 1], [0, 200, 64]), ([300, 129], [0, 7]))


@pytest.mark.parametrize("null,out_scale", [(True, 1.0), (True, -0.7), (False, 1.3)])
@pytest.mark.parametrize("H,KV,d,vd", [(4, 2, 16, 24), (3, 1, 10, 7), (2, 2, 200, 256), (6, 2, 64, 40)])
def test_general_attention_with_a_null_key(H, KV, d, vd, null, out_scale):
    p8 = lambda n: (n + 7) // 8 * 8
    for q_lens, starts in STEPS:
        ref, got, _ = run_null(torch.float32, H, KV, d, vd, p8(d), p8(vd), q_lens, starts, 0.3, null, out_scale, H + d, tc=False)
        assert rel(ref, got) < 2e-5, (q_lens, starts)


@pytest.mark.parametrize("H,KV,d,vd,dp,vdp", [(4, 2, 64, 64, 64, 64), (4, 2, 128, 64, 128, 64), (4, 1, 64, 128, 64, 128), (2, 2, 128, 128, 128, 128),
                                              (6, 2, 40, 72, 64, 128), (3, 3, 100, 20, 128, 64), (16, 1, 48, 88, 64, 128)])
def test_tensor_core_attention_with_a_null_key(H, KV, d, vd, dp, vdp):
    """bfloat16: every pair of stored widths, heads narrower than stored, against the reference and the general kernels."""
    for q_lens, starts in STEPS:
        for null, out_scale in ((True, 0.8), (False, 1.0)):
            args = (torch.bfloat16, H, KV, d, vd, dp, vdp, q_lens, starts, d ** -0.5, null, out_scale, d + H)
            ref, tc, _ = run_null(*args)
            _, gen, _ = run_null(*args, tc=False)
            assert rel(ref, tc) < 2e-2 and rel(ref, gen) < 2e-2 and rel(gen, tc) < 2e-2, (q_lens, starts)


@pytest.mark.parametrize("dtype,d", [(torch.float32, 16), (torch.bfloat16, 64)])
@pytest.mark.parametrize("shift", [-200.0, -6.0, 6.0, 100.0])
def test_the_null_key_against_low_and_high_scores(dtype, d, shift):
    """All scores moved by a constant: far below the null key's the output vanishes (also where exp overflows), far above it
    the null key does."""
    for q_lens, starts in (([130], [0]), ([1, 1], [140, 3])):
        ref, got, v = run_null(dtype, 2, 1, d, d, d, d, q_lens, starts, 0.25, True, 1.0, 3, shift=shift)
        assert np.all(np.isfinite(got))
        tol = 2e-4 if dtype == torch.float32 else 3e-2
        assert np.abs(ref - got).max() < tol * max(np.abs(ref).max(), 1e-6), (shift, q_lens)
        if shift == -200.0:
            assert np.abs(got).max() < 1e-20
        if shift == 100.0:
            with_null, without = got, run_null(dtype, 2, 1, d, d, d, d, q_lens, starts, 0.25, False, 1.0, 3, shift=shift)[1]
            assert rel(without, with_null) < 1e-3


@pytest.mark.parametrize("dtype,d,vd,dp,vdp", [(torch.float32, 16, 24, 16, 24), (torch.bfloat16, 48, 80, 64, 128), (torch.bfloat16, 128, 64, 128, 64)])
def test_one_far_key_stands_out(dtype, d, vd, dp, vdp):
    """ONE key of hundreds is large along the direction every query looks in: every later query returns its value, no
    earlier one does; the key sits at the start, at page borders and far back."""
    n = 345
    for key in (0, 1, 63, 64, 65, 127, 128, 300):
        for q_lens, starts in (([n], [0]), ([n - 250], [250]), ([1], [key]), ([1], [344])):
            ref, got, v = run_null(dtype, 2, 2, d, vd, dp, vdp, q_lens, starts, 1.0, True, 1.0, key, sharp=key)
            assert rel(ref, got) < (1e-4 if dtype == torch.float32 else 3e-2), (key, q_lens, starts)
            for r, p in enumerate(range(starts[0], starts[0] + q_lens[0])):
                assert (rel(v[0][key], got[r]) < 0.05) == (key <= p), (key, p)


# ------------------------------------------------------------------ preparation
@pytest.mark.parametrize("H,G,dim,vd,rot,dimp,vdp", [(4, 2, 16, 24, 12, 64, 64), (3, 1, 10, 7, 6, 16, 8), (6, 3, 48, 80, 48, 64, 128), (4, 2, 64, 128, 32, 64, 128),
                                                     (2, 1, 128, 64, 0, 128, 64)])
def test_preparation_with_unit_norms_and_query_factors(H, G, dim, vd, rot, dimp, vdp):
    """The rotation, then the unit RMS norm (the kernel norms first), then the query's factor by position."""
    from mynah_slm_b200.ops import kernels
    from mynah_slm_b200.parts.attention_capped import query_temperatures
    from mynah_slm_b200.parts.position import rotary_frequencies
    rng = np.random.default_rng(H * 10 + dim)
    T, nq, nk, nv = 130, H * dim, G * dim, G * vd
    x = rng.normal(size=(T, nq + nk + nv))
    ctx, pages, n_pages = step_ctx([T], [0])
    cos = sin = None
    if rot:
        cos, sin = kernels.rope_table_freqs(256, *rotary_frequencies(rot, 300.0, None), DEV)
    temp = {"coef": 0.7, "every": 9}
    k_cache = torch.full((n_pages, G, PAGE, dimp), 9.0, dtype=torch.float32, device=DEV)
    v_cache = torch.full((n_pages, G, PAGE, vdp), 9.0, dtype=torch.float32, device=DEV)
    q_out = torch.full((T, H * dimp), 9.0, dtype=torch.float32, device=DEV)
    ones = torch.ones((dim,), dtype=torch.float32, device=DEV)
    kernels.capped_attn_prep(t32(x), q_out, H, G, G, dim, vd, dimp, vdp, 1, H // G, None, ones, ones, 1e-2, cos, sin, rot, False, ctx, pages,
                             k_cache, v_cache, query_temperatures(200, temp["coef"], temp["every"], DEV))
    assert int(ctx.status.item()) == 0
    turn = (lambda y: plain.turn_halves(y, {"dims": rot, "base": 300.0})) if rot else (lambda y: y)
    q = plain.rms_unit(turn(x[:, :nq].reshape(T, H, dim)), 1e-2) * plain.query_temperature(T, temp)[:, None, None]
    k, v = plain.rms_unit(turn(x[:, nq:nq + nk].reshape(T, G, dim)), 1e-2), x[:, nq + nk:].reshape(T, G, vd)
    ids = pages.ids.cpu().numpy()
    got_k = torch.stack([k_cache[ids[p // PAGE], :, p % PAGE] for p in range(T)]).cpu().numpy()
    got_v = torch.stack([v_cache[ids[p // PAGE], :, p % PAGE] for p in range(T)]).cpu().numpy()
    got_q = q_out.view(T, H, dimp).cpu().numpy()
    for ref, got, n in ((q, got_q, dim), (k, got_k, dim), (v, got_v, vd)):
        assert rel(ref, got[..., :n]) < 1e-5 and np.all(got[..., n:] == 0)
    # a position beyond the factors' table is refused, not read
    kernels.capped_attn_prep(t32(x), q_out, H, G, G, dim, vd, dimp, vdp, 1, H // G, None, ones, ones, 1e-2, cos, sin, rot, False, ctx, pages,
                             k_cache, v_cache, query_temperatures(100, 0.1, 5, DEV))
    assert int(ctx.status.item()) == kernels.ST_POS_RANGE


# ------------------------------------------------------------------ router, experts, shared expert; capped logits
@pytest.mark.parametrize("D,F,E,top,groups,keep,FS", [(48, 24, 10, 3, 2, 1, 40), (64, 40, 12, 3, 4, 2, 0), (44, 12, 1, 1, 1, 1, 9), (40, 10, 7, 7, 7, 7, 10),
                                                      (48, 16, 6, 2, 3, 3, 16), (96, 200, 72, 4, 12, 5, 56), (52, 18, 9, 2, 3, 1, 0), (64, 64, 16, 2, 16, 4, 64)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_softmax_router_experts_and_shared_expert(dtype, D, F, E, top, groups, keep, FS):
    """Choices inside the kept groups, weights over all experts, silu-gated experts, the shared expert behind its gate;
    padding rows stay out. bfloat16: the tile form and, in long steps, the grouped tcgen05 form."""
    from mynah_slm_b200.ops import kernels
    rng = np.random.default_rng(D + E)
    hold = lambda x: torch.tensor(x, dtype=dtype).double().numpy()
    dev = lambda x: torch.tensor(x, dtype=dtype, device=DEV)
    for T in (1, 5, 90, 700):
        W = {"router": hold(rng.normal(size=(E, D)) / np.sqrt(D) * 3.0), "shared.sg": hold(rng.normal(size=(1, D)) / np.sqrt(D) * 2.0)}
        for e in [f"e{e}" for e in range(E)] + (["shared"] if FS else []):
            f = FS if e == "shared" else F
            W[f"{e}.gate"], W[f"{e}.up"] = hold(rng.normal(size=(f, D)) / np.sqrt(D) * 2), hold(rng.normal(size=(f, D)) / np.sqrt(D) * 2)
            W[f"{e}.down"] = hold(rng.normal(size=(D, f)) / np.sqrt(f))
        mlp = {"expert": {"ff": F}, "router": {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}, "shared": {"ff": FS} if FS else None}
        h = hold(rng.normal(size=(T, D)))
        margins = []
        ref = plain.routed_ff(h, W, "", mlp, margins)
        steady = margins[0] > (1e-4 if dtype == torch.float32 else 1e-3)
        ctx = SimpleNamespace(tok_seq=i32([0] * T + [-1]), status=torch.zeros((1,), dtype=torch.int32, device=DEV))
        w_gu = torch.stack([torch.stack([dev(W[f"e{e}.gate"]), dev(W[f"e{e}.up"])]) for e in range(E)]).contiguous()
        w_down = torch.stack([dev(W[f"e{e}.down"]) for e in range(E)]).contiguous()
        hp = torch.cat([dev(h), torch.full((1, D), 1e4, dtype=dtype, device=DEV)], 0).contiguous()       # a padding row of large values
        router, shared = dev(W["router"]), None
        if FS:
            router = torch.cat([router, dev(W["shared.sg"])], 0).contiguous()
            gu = torch.cat([dev(W["shared.gate"]), dev(W["shared.up"])], 0).contiguous()
            shared = kernels.linear(kernels.linear_swiglu(hp, gu), dev(W["shared.down"]), out_dtype=torch.float32)
        out = kernels.moe_group_router_ffn(hp, router, None, w_gu, w_down, ctx, top, groups, keep, 1.0, None, 1.0, "softmax", "max", shared)
        assert int(ctx.status.item()) == 0
        got = out[:T].double().cpu().numpy()
        assert steady.mean() > 0.9 and rel(ref[steady], got[steady]) < (2e-5 if dtype == torch.float32 else 2e-2), (T, rel(ref[steady], got[steady]))


def test_softmax_scores_that_underflow_still_choose_by_their_order():
    """Logits hundreds apart: all but one score round to zero; the second choice still goes to the second largest logit."""
    from mynah_slm_b200.ops import kernels
    E, D = 8, 16
    W = torch.zeros((E, D), device=DEV)
    W[:, 0] = torch.tensor([0.0, -900.0, -300.0, -200.0, -500.0, -400.0, -600.0, -700.0], device=DEV)
    h = torch.zeros((1, D), device=DEV)
    h[0, 0] = 1.0
    h[0, 1] = 1.0
    w_gu = torch.zeros((E, 2, 4, D), device=DEV)
    w_gu[:, :, :, 1] = 1.0
    w_down = torch.arange(1.0, E + 1, device=DEV).view(E, 1, 1).expand(E, D, 4).contiguous()
    ctx = SimpleNamespace(tok_seq=i32([0]), status=torch.zeros((1,), dtype=torch.int32, device=DEV))
    out = kernels.moe_group_router_ffn(h, W, None, w_gu, w_down, ctx, 2, 1, 1, 1.0, None, 1.0, "softmax", "max")
    y = float(torch.nn.functional.silu(torch.tensor(1.0)))
    assert abs(float(out[0, 0]) - 4 * y) < 1e-5 and int(ctx.status.item()) == 0


def test_capped_logits():
    from mynah_slm_b200.ops import kernels
    rng = np.random.default_rng(1)
    for n in (1, 3, 4, 1001, 70000):
        x = 40.0 * rng.normal(size=(1, n))
        got = kernels.softcap_(t32(x), 15.0).cpu().numpy()
        assert np.abs(15.0 * np.tanh(np.float32(x).astype(np.float64) / 15.0) - got).max() < 1e-5
