"""The Guvolix design on the engine against the plain implementation in ``plain_guvolix.py``: every mechanism alone
(kernels against one plain function each), then whole models of configurations that share no size, fed whole, with a
decoded tail, in portions down to two tokens, token by token, in mixed batches over pools that force pages and slots to
be used again, through ``bin/trace_run`` and through the scheduler."""
from __future__ import annotations

import math
import tempfile
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import helpers as H
import plain_guvolix as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
TYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64


def _left(heads, kv_heads, dim, vdim, scale, window=None, keep=0, base=1e4, dims=None, scaling=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if window:
        m["mask"] = dict(size=window)
        if keep:
            m["mask"]["keep_first"] = keep
    if dims != 0:
        m["rot"] = dict(base=base, dims=dims or dim)
        if scaling:
            m["rot"]["scaling"] = scaling if isinstance(scaling, dict) else dict(factor=scaling)
    return m


def _ssd(left, heads, vdim, state, groups, conv, norm_groups, mlp=None):
    right = dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)
    return dict(type="parallel", mixer=dict(left=left, right=right), mlp=mlp)


def _mem(left, heads, dim, vdim, cap, scales, mlp=None):
    return dict(type="parallel_2", mlp=mlp, mixer=dict(left=left, right=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap),
                                                       left_scale=scales[0], right_scale=scales[1]))


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(ff, experts, top, identity=0, shared=0):
    f = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if identity:
        f["router"]["identity"] = identity
    if shared:
        f["shared"] = dict(ff=shared)
    return f


def _config(vocab, width, eps, scale, layers):
    return dict(architecture="Guvolix", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)


LLAMA3 = dict(factor=4.0, low=1.0, high=4.0, original=64)
# Configurations that share no size.  A: windows and kept tokens that are no multiple of the page, both mixers with every
# feed-forward.  B: values that are 1 (groups, taps, norm groups, heads, value and key sizes, a window of one), more kept
# tokens than the window, an odd width, no rotation, no scaling, no shared and no identity experts.  C: sizes at which the
# tensor-core kernels run in bfloat16; kept tokens over one tile of keys and several pages.  EDGE / EDGE_2: one layer each.
CFG_A = _config(200, 48, 1e-5, 0.7, [
    _ssd(_left(4, 2, 12, 20, 0.25, 10, 3, 500.0, 6, 2.0), 6, 5, 8, 3, 3, 2, _dense(40)),
    _mem(_left(3, 1, 8, 12, 0.4, 14, 5, 40.0, 8, LLAMA3), 3, 10, 6, 4.0, (0.8, 1.3), _moe(16, 6, 3, 2, 24)),
    _ssd(_left(6, 3, 10, 6, 0.3, 7, 9, 900.0, 10, 3.0), 4, 12, 20, 2, 5, 4),
    _mem(_left(2, 2, 16, 9, 0.5, 9), 2, 7, 11, 9.0, (1.1, 0.6), _dense(36))])
CFG_B = _config(513, 102, 1e-6, 1.0, [
    _mem(_left(1, 1, 6, 1, 0.4, 5, 8, dims=0), 1, 1, 14, 3.0, (1.0, 1.0), _moe(36, 1, 1)),
    _ssd(_left(5, 1, 7, 3, 0.3, 1, 1, 30.0, 2), 5, 1, 9, 1, 1, 1, _moe(18, 5, 2, 4)),
    _ssd(_left(6, 2, 16, 11, 0.2, None, 0, 1e3, 8, 1.0), 1, 24, 1, 1, 2, 3, _moe(10, 3, 3, 0, 30)),
    _mem(_left(2, 1, 9, 8, 0.35, 33, dims=8), 7, 5, 1, 20.0, (0.5, -0.7))])
CFG_C = _config(640, 320, 1e-5, 1.5, [
    _ssd(_left(8, 2, 64, 64, 0.125, 80, 5, 1e5, 32, 8.0), 6, 64, 32, 2, 4, 3, _moe(64, 8, 2, 3, 96)),
    _mem(_left(8, 2, 128, 128, 0.09, 70, 18, 1e4, 128, LLAMA3), 4, 64, 96, 12.0, (0.9, 1.2), _dense(160)),
    _ssd(_left(4, 4, 64, 64, 0.15, 33, 70, 5e3, 64), 3, 96, 128, 1, 2, 1, _moe(96, 4, 2, 2, 128)),
    _mem(_left(8, 1, 128, 128, 0.1, 100, 1, 1e6, 64, 2.0), 2, 160, 32, 15.0, (1.0, 0.5), _moe(128, 6, 3, 1, 64))])
CFG_EDGE = _config(150, 32, 1e-5, 1.0, [_ssd(_left(2, 1, 8, 12, 0.7, 12, 3, 100.0, 8, 2.0), 2, 6, 4, 1, 3, 1, _moe(8, 4, 2, 2, 8))])
CFG_EDGE_2 = _config(150, 36, 1e-5, 1.0, [_mem(_left(2, 1, 8, 8, 0.5, 9), 2, 6, 4, 5.0, (1.0, 0.0), _dense(24))])
CONFIGS = {"A": (CFG_A, 11, 4), "B": (CFG_B, 12, 8), "C": (CFG_C, 13, 16), "EDGE": (CFG_EDGE, 14, 4), "EDGE_2": (CFG_EDGE_2, 15, 8)}
LENGTHS = {"A": [1, 6, 23, 90], "B": [2, 9, 41, 130], "C": [3, 64, 150, 400]}


def _live(name, t, gen):
    """Tensors whose plain draw would hide a mechanism: memories from a few to some thousand tokens, sinks that matter,
    corrections that change the choice; and routers whose choices are seldom close (in bfloat16 a close one may fall
    either way, and what it changes stays in the states)."""
    u = lambda lo, hi: lo + (hi - lo) * torch.rand(t.shape, generator=gen)
    for end, lo, hi in ((".A_log", -4.5, 0.5), (".dt_bias", -4.0, -0.5), (".f.b", 1.0, 7.0), (".i.b", -1.5, 1.0),
                        (".sink", -1.0, 3.0), (".correction", 0.0, 0.4)):
        if name.endswith(end):
            return u(lo, hi)
    if name.endswith(".router"):
        return 4.0 * t
    return t


def _make(path, cfg, seed, stored, std=0.08, fixed_choice=False):
    """``fixed_choice``: corrections so far apart that they alone choose (the same experts for every token)."""
    from batchspec_b200.weights import write_safetensors
    folder = H.make_folder(path, cfg, seed, dtype=torch.float32, std=std)
    gen = torch.Generator().manual_seed(seed)
    tensors = {k: _live(k, v, gen) for k, v in P.read_tensors(folder / "model.safetensors").items()}
    if fixed_choice:
        tensors = {k: v * (200.0 if k.endswith(".correction") else 0.25 if k.endswith(".router") else 1.0) for k, v in tensors.items()}
    write_safetensors(folder / "model.safetensors", ((k, v.to(stored)) for k, v in tensors.items()))
    return folder


def _folder(tmp_path, name, dtype, std=0.08):
    cfg, seed, _ = CONFIGS[name]
    return _make(tmp_path / f"f{name}_{dtype}", cfg, seed, torch.float32 if dtype == "float32" else torch.bfloat16, std,
                 fixed_choice=name == "C" and dtype == "bfloat16")


def _engine(folder, dtype, page_size, num_pages, max_requests=8):
    from batchspec_b200.engine import Engine
    eng = Engine(dtype=dtype, device=DEV)
    eng.load_model(model_dir=folder)
    eng.setup_caches(max_batch_size=max_requests, page_size=page_size, num_pages=num_pages)
    return eng


_ORACLE = {}


def _oracle(folder, tokens):
    key = (str(folder), tuple(tokens))
    if key not in _ORACLE:
        cfg, w = P.read_model_folder(folder)
        _ORACLE[key] = P.forward(cfg, w, tokens).numpy()
    return _ORACLE[key]


def _compare(got, folder, reqs, dtype):
    """Every row against the oracle.  float32: no row beyond the tolerance.  bfloat16: five rows in a hundred, or one, may
    be (a router's choice between two experts whose scores differ by less than the rounding falls either way, and a
    later layer sees the row)."""
    bf = dtype == "bfloat16"
    return H.compare_with_oracle(got, folder, reqs, dtype, oracle=_oracle, allow_over=0.05 if bf else 0.0,
                                 allow_rows=1 if bf else 0)


def _requests(name):
    cfg, seed, _ = CONFIGS[name]
    return {f"r{i}": H.random_tokens(n, cfg["vocab"], 100 * seed + i) for i, n in enumerate(LENGTHS[name])}


def _rows_agree(a, b, dtype, share=0.05):
    bad = [k for k in a if np.abs(a[k] - b[k]).max() > H.TOL[dtype] * np.abs(a[k]).max()]
    assert len(bad) <= (max(1, share * len(a)) if dtype == "bfloat16" else 0), bad[:5]


@pytest.fixture(scope="module")
def ops():
    from batchspec_b200.kernels import ops as o
    o.load_library()
    return o


def _gen(seed):
    return torch.Generator(device=DEV).manual_seed(seed)


def _step_ctx(lens, slots, starts):
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32, device=DEV)
    pos = torch.cat([torch.arange(s, s + k) for s, k in zip(starts, lens)])
    return SimpleNamespace(qo_indptr=i32([0] + list(np.cumsum(lens))), state_slots=i32(slots), positions=i32(pos),
                           tok_entry=i32(np.repeat(np.arange(len(lens)), lens)), n_entries=len(lens), n_tokens=sum(lens),
                           max_q_len=max(lens))


# ---------------------------------------------------------------------------- both sublayers join together

@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n,d", [(3, 96), (5, 50), (2, 4096), (4, 7), (600, 640), (2, 20000), (3, 1)])
@pytest.mark.parametrize("pair", [False, True])
def test_two_branches_join_the_residual_and_are_normed(ops, dtype, n, d, pair):
    g = _gen(n + d)
    rnd = lambda *s: torch.randn(*s, device=DEV, generator=g)
    src, a, b, c = rnd(n, d), rnd(n, d).to(dtype), (3 * rnd(n, d)).to(dtype), (2 * rnd(n, d)).to(dtype)
    wa, wb, wn = (1 + 0.3 * rnd(d) for _ in range(3))
    eps = 1e-5
    y = P.rms_norm(a.double(), wa, eps) + P.rms_norm(b.double(), wb, eps) if pair else a.double()
    want = src.double() + y + c.double()
    delta = ops.BranchSum(ops.NormedPair(a, b, wa, wb, eps) if pair else a, c)
    near = lambda got, ref, t=2e-5: (got.double() - ref).abs().max() <= t * (1 + ref.abs().max())
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    x, out = src.clone(), torch.empty(n, d, device=DEV, dtype=dtype)
    ops.branch_join(x, delta, dst=x, out=out, norm_w=wn, eps=eps)
    assert near(x, want) and near(out, P.rms_norm(want, wn, eps), tol)
    rows = torch.tensor([n - 1, 0, n // 2], dtype=torch.int32, device=DEV)
    picked = torch.empty(3, d, device=DEV, dtype=dtype)
    ops.branch_join(src, delta, out=picked, norm_w=wn, eps=eps, rows=rows)
    assert near(picked, P.rms_norm(want, wn, eps)[rows.long()], tol)


# ---------------------------------------------------------------------------- attention: first tokens that stay visible

def _attention_case(ops, dtype, Hq, G, hd, vd, ps, q_lens, kv_lens, window, keep, sink=True, scale=None, change=None, seed=0,
                    generic=False, want_plain=True):
    """Random queries over cached rows whose pages lie in scrambled order; the table entries of the pages between the kept
    tokens' and the window's are -1.  ``change(q, rows, starts)`` edits the inputs.  Returns (got, want) [n, Hq, vd]."""
    g = _gen(seed)
    n, qo = sum(q_lens), [0] + list(np.cumsum(q_lens))
    q = torch.randn(n, Hq, hd, device=DEV, generator=g)
    rows = [torch.randn(L, G, hd + vd, device=DEV, generator=g) for L in kv_lens]
    if change is not None:
        change(q, rows, qo)
    q, rows = q.to(dtype), [r.to(dtype) for r in rows]
    scale = scale or 1.0 / math.sqrt(hd)
    at = [0] + list(np.cumsum([-(-L // ps) for L in kv_lens]))
    perm = torch.randperm(at[-1] + 2, generator=torch.Generator().manual_seed(seed + 1))
    pages = torch.randn(at[-1] + 2, 1, ps * G * (hd + vd), device=DEV, generator=g).to(dtype)
    for e, r in enumerate(rows):
        for p0 in range(0, r.shape[0], ps):
            k = min(ps, r.shape[0] - p0)
            page = pages[int(perm[at[e] + p0 // ps])].reshape(-1)
            page[:G * ps * hd].view(G, ps, hd)[:, :k] = r[p0:p0 + k, :, :hd].transpose(0, 1)
            page[G * ps * hd:].view(G, ps, vd)[:, :k] = r[p0:p0 + k, :, hd:].transpose(0, 1)
    table = perm.clone()
    for e, L in enumerate(kv_lens):
        dead, stay = max(0, L - q_lens[e] - window + 1) // ps, -(-keep // ps)
        table[at[e] + stay:at[e] + max(dead, stay)] = -1
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32, device=DEV)
    tables = SimpleNamespace(kv_indptr=i32(at), kv_indices=i32(table), page_size=ps)
    pos = torch.cat([torch.arange(L - k, L) for k, L in zip(q_lens, kv_lens)])
    ctx = SimpleNamespace(qo_indptr=i32(qo), positions=i32(pos), n_entries=len(q_lens), n_tokens=n, max_q_len=max(q_lens),
                          tok_entry=i32(np.repeat(np.arange(len(q_lens)), q_lens)), max_kv_len=max(kv_lens), kv_len=i32(kv_lens),
                          extras={"min_q_len": min(q_lens)})
    sinks = torch.linspace(-1.0, 4.0, Hq, device=DEV) if sink else None
    out = torch.full((n, Hq * vd), float("nan"), device=DEV, dtype=dtype)
    before = (-keep, pages, tables)
    if hd == vd:
        ops.FORCE_GENERIC_ATTENTION = generic
        try:
            ops.paged_attention(q.reshape(n, -1), out, pages, ctx, tables, Hq, G, hd, scale, window, sink=sinks,
                                sink_l2=ops.sink_table(sinks) if sink else None, pooled=before)
        finally:
            ops.FORCE_GENERIC_ATTENTION = False
    else:
        ops.masked_attention(q.reshape(n, -1), out, pages, ctx, tables, Hq, G, hd, vd, scale, window, sink=sinks, pooled=before)
    torch.cuda.synchronize()
    ops.check_status()
    got = out.double().cpu().view(n, Hq, vd)
    if not want_plain:
        return got, None
    want = torch.empty(n, Hq, vd, dtype=F64)
    for e, (k, L) in enumerate(zip(q_lens, kv_lens)):
        x = rows[e].double().cpu()
        full_q = torch.zeros(L, Hq, hd, dtype=F64)
        full_q[L - k:] = q[qo[e]:qo[e + 1]].double().cpu()
        o = P.attend(full_q, x[:, :, :hd], x[:, :, hd:], scale, window, keep, sinks.cpu() if sink else None)
        want[qo[e]:qo[e + 1]] = o[L - k:]
    return got, want


KEEP_SHAPES = [
    # Hq, G, hd, vd, page, q_lens, kv_lens, window, keep
    (3, 3, 16, 16, 4, [5, 1, 2], [5, 9, 30], 7, 3),
    (4, 1, 20, 36, 5, [3, 11], [17, 60], 9, 6),
    (2, 1, 24, 24, 4, [7, 1, 20], [60, 50, 90], 1, 1),
    (8, 2, 64, 64, 16, [1, 1, 1, 1], [300, 17, 64, 129], 64, 4),
    (8, 2, 64, 64, 16, [70, 2, 1], [200, 5, 333], 33, 17),
    (16, 2, 128, 128, 16, [130, 1, 3, 64], [130, 555, 40, 600], 96, 5),
    (6, 3, 128, 128, 8, [1, 1], [1300, 31], 1000, 8),
    (4, 1, 128, 128, 32, [300], [900], 64, 70),                       # kept tokens over two tiles of keys
    (4, 4, 128, 128, 64, [260, 1, 4], [520, 2000, 700], 16, 200),     # many more kept tokens than the window
    (4, 2, 256, 256, 16, [40, 1], [90, 200], 50, 4),
    (8, 8, 128, 128, 5, [20, 1], [90, 200], 50, 7),                   # a page size that TMA does not take
    (12, 4, 64, 64, 64, [2, 5, 9], [2, 700, 90], 40, 65),
    (2, 2, 128, 128, 16, [16, 9], [40, 9], 2, 12),                    # kept tokens of the step itself
    (2, 1, 64, 64, 8, [1, 400], [4000, 400], 24, 1)]


@pytest.mark.parametrize("generic", [False, True])
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shape", KEEP_SHAPES, ids=lambda s: f"H{s[0]}d{s[2]}v{s[3]}ps{s[4]}w{s[7]}k{s[8]}")
def test_attention_with_first_tokens_kept_behind_the_window(ops, dtype, shape, generic):
    if generic and (dtype == torch.float32 or shape[2] != shape[3]):
        pytest.skip("these run the generic kernel anyway")
    got, want = _attention_case(ops, dtype, *shape, generic=generic)
    assert (got - want).abs().max() <= (2e-5 if dtype == torch.float32 else 2.5e-2)


@pytest.mark.parametrize("dtype,hd", [(torch.float32, 32), (torch.bfloat16, 32), (torch.bfloat16, 64), (torch.bfloat16, 128)])
@pytest.mark.parametrize("q_lens", [[1, 1], [3, 70], [1, 300]])
def test_one_key_decides_in_the_window_and_among_the_kept_tokens_only(ops, dtype, hd, q_lens):
    """One query's score with one token stands out.  It takes the softmax up to 39 positions back (a window of 40) and among
    the first 18; anywhere between it leaves no trace, bit for bit."""
    L, window, keep, Hq = 640, 40, 18, 4
    t = sum(q_lens) - 1
    tol = 1e-4 if dtype == torch.float32 else 4e-2
    for where in (639, 638, 624, 623, 601, 600, 599, 598, 592, 300, 33, 32, 31, 19, 18, 17, 16, 15, 1, 0):
        def quiet(q, rows, qo):
            q[t, 2] = 0
            q[t, 2, hd - 1] = 8.0
            rows[1][:, :, hd - 1] = rows[1][:, :, hd - 1].clamp(-1, 1) * 0.1

        def stand_out(q, rows, qo):
            quiet(q, rows, qo)
            rows[1][where, :, hd - 1] = 40.0
        args = (ops, dtype, Hq, 2, hd, hd, 16, q_lens, [90, L], window, keep)
        got, want = _attention_case(*args, change=stand_out, seed=where, scale=0.5)
        assert (got - want).abs().max() <= tol, where
        got0, _ = _attention_case(*args, change=quiet, seed=where, scale=0.5, want_plain=False)
        seen = where >= L - window or where < keep
        assert bool((got[t, 2] != got0[t, 2]).any()) == seen, where


@pytest.mark.parametrize("dtype,hd", [(torch.float32, 32), (torch.bfloat16, 64), (torch.bfloat16, 128)])
def test_kept_tokens_inside_the_window_count_once(ops, dtype, hd):
    """Equal scores and values of one for the kept tokens: the output is the kept tokens' share, at lengths around the point
    where the window passes them."""
    window, keep = 20, 6
    for L in (1, 5, 6, 7, 19, 20, 21, 23, 25, 26, 27, 60):
        for k in sorted({1, min(L, 3), L}):
            def same(q, rows, qo):
                q.zero_()
                rows[0][:, :, hd:] = 0.0
                rows[0][:keep, :, hd:] = 1.0
            got, want = _attention_case(ops, dtype, 4, 2, hd, hd, 8, [k], [L], window, keep, sink=False, change=same)
            share = min(L, keep) / (min(L, window) + min(keep, max(0, L - window)))
            assert (want[-1] - share).abs().max() < 1e-9 and (got - want).abs().max() <= (1e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("scaling", [None, dict(rope_type="linear", factor=3.0),
                                     dict(rope_type="llama3", factor=6.0, low_freq_factor=1.5, high_freq_factor=5.0,
                                          original_max_position_embeddings=300)])
def test_rotation_rates_at_far_positions(scaling):
    """The frequency table against the plain rates, and one head turned at positions up to 60,000."""
    from batchspec_b200.parts.rope import RotaryEmbedding
    from batchspec_b200.parts.base import Runtime
    hd, dims, base = 40, 24, 3e4
    part = RotaryEmbedding(Runtime(torch.float32, torch.device(DEV)), hd, base, scaling, rotary_dim=dims, interleaved=False)
    rot = dict(base=base, dims=dims)
    if scaling and scaling["rope_type"] == "linear":
        rot["scaling"] = dict(factor=3.0)
    elif scaling:
        rot["scaling"] = dict(factor=6.0, low=1.5, high=5.0, original=300)
    rates = torch.tensor(P.angle_rates(rot), dtype=F64)
    assert torch.allclose(part.frequencies, rates, rtol=1e-12, atol=0)
    pos = torch.tensor([0, 1, 77, 5000, 60000], dtype=torch.int32, device=DEV)
    x = torch.randn(5, 2, hd, device=DEV, generator=_gen(3))
    want = x.double().cpu()
    a = pos.double().cpu()[:, None] * rates
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = want[..., :dims // 2].clone(), want[..., dims // 2:dims].clone()
    want[..., :dims // 2], want[..., dims // 2:dims] = u * c - v * s, v * c + u * s
    part.apply(x, None, SimpleNamespace(positions=pos))
    assert (x.double().cpu() - want).abs().max() < 5e-6


# ---------------------------------------------------------------------------- recurrences

STEPS = [dict(a=5, b=1, c=2), dict(a=1, c=1), dict(b=11, a=2, c=1), dict(c=1), dict(c=39, a=1), dict(b=2, c=37), dict(a=1, b=1)]


def _mixer_over_steps(part, dtype, d, plain, seed, w):
    """Three requests in portions of unequal sizes (one left out of some steps) against the plain mixer over each whole
    sequence; then a cleared slot again."""
    g = _gen(seed)
    part.bind({k: v.to(DEV) for k, v in w.items()})
    state = torch.zeros(5, *part.state_spec().shape, device=DEV)
    slots, at = {"a": 2, "b": 0, "c": 4}, {r: 0 for r in "abc"}
    xs = {r: torch.randn(sum(s.get(r, 0) for s in STEPS), d, device=DEV, generator=g).to(dtype) for r in slots}
    got = {r: [] for r in slots}
    for step in STEPS:
        x = torch.cat([xs[r][at[r]:at[r] + k] for r, k in step.items()]).contiguous()
        y = part.forward(x, _step_ctx(list(step.values()), [slots[r] for r in step], [at[r] for r in step]), SimpleNamespace(state=state))
        o = 0
        for r, k in step.items():
            got[r].append(y[o:o + k])
            at[r] += k
            o += k
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    for r in slots:
        want = plain(xs[r].double().cpu())
        assert (torch.cat(got[r]).double().cpu() - want).abs().max() <= tol * (1 + want.abs().max()), r
    assert not state[1].any() and not state[3].any()             # the slots of no request were never written
    state[2].zero_()
    again = part.forward(xs["c"][:7].contiguous(), _step_ctx([7], [2], [0]), SimpleNamespace(state=state))
    want = plain(xs["c"][:7].double().cpu())
    assert (again.double().cpu() - want).abs().max() <= tol * (1 + want.abs().max())
    # into the columns of wider rows, with a factor
    wide = torch.full((7, part.out_width + 9), 7.0, device=DEV, dtype=dtype)
    state[2].zero_()
    part.pre_projection(xs["c"][:7].contiguous(), _step_ctx([7], [2], [0]), SimpleNamespace(state=state), wide[:, 5:-4], -0.75)
    state[2].zero_()
    one = part.pre_projection(xs["c"][:7].contiguous(), _step_ctx([7], [2], [0]), SimpleNamespace(state=state))
    assert (wide[:, 5:-4].double() + 0.75 * one.double()).abs().max() <= (1e-6 if dtype == torch.float32 else 2e-2) * (1 + one.abs().max())
    assert (wide[:, :5] == 7).all() and (wide[:, -4:] == 7).all()


def _mixer(kind, params, dtype, seed, names, std=0.25):
    from batchspec_b200.parts.base import MIXERS, PartSpec, Runtime, build_part
    part = build_part(MIXERS, PartSpec(kind, params), Runtime(dtype, torch.device(DEV)))
    gen = torch.Generator().manual_seed(seed)
    w = {k: _live("." + names[k], torch.randn(*ps.shape, generator=gen) * std + (ps.init == "ones_normal"), gen).to(dtype)
         for k, ps in part.param_specs().items()}
    return part, w, {names[k]: v for k, v in w.items()}


SSD_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D", "norm": "norm", "o": "o"}
MEM_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "i": "i", "f": "f", "i_bias": "i.b", "f_bias": "f.b", "norm": "norm", "o": "o"}


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("Hh,V,N,G,taps,ng", [(6, 5, 8, 3, 3, 2), (1, 24, 1, 1, 1, 3), (4, 16, 33, 1, 2, 1), (8, 64, 64, 2, 4, 8),
                                              (2, 128, 128, 2, 4, 2), (3, 9, 256, 3, 6, 27), (5, 1, 6, 5, 5, 1), (10, 64, 100, 2, 4, 1)])
def test_state_space_over_portions_and_reused_slots(ops, dtype, Hh, V, N, G, taps, ng):
    d, eps = 64, 1e-5
    part, w, named = _mixer("state_space", dict(dim=d, n_heads=Hh, v_dim=V, n_state=N, n_groups=G, taps=taps, norm_groups=ng, eps=eps),
                            dtype, V + N, SSD_NAMES)
    m = dict(heads=Hh, vdim=V, state=N, groups=G, conv=taps, norm_groups=ng)
    _mixer_over_steps(part, dtype, d, lambda h: P.state_space_dual(h, named, m, eps), N, w)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("Hh,dk,dv,cap", [(3, 10, 6, 4.0), (1, 1, 14, 3.0), (7, 5, 1, 20.0), (2, 64, 48, 9.0), (4, 128, 128, 15.0),
                                          (1, 256, 31, 12.0), (8, 33, 16, 0.5), (16, 64, 15, 12.0)])
def test_matrix_memory_over_portions_and_reused_slots(ops, dtype, Hh, dk, dv, cap):
    d, eps = 64, 1e-5
    part, w, named = _mixer("matrix_memory", dict(dim=d, n_heads=Hh, head_dim=dk, v_dim=dv, gate_cap=cap, eps=eps), dtype, dk + dv,
                            MEM_NAMES)
    m = dict(heads=Hh, dim=dk, vdim=dv, gate_cap=cap)
    _mixer_over_steps(part, dtype, d, lambda h: P.mlstm(h, named, m, eps), dk, w)


@pytest.mark.parametrize("run", [None, torch.bfloat16])
@pytest.mark.parametrize("lens,C,taps", [([1, 2, 3, 4, 70, 1, 5, 30], 96, 4), ([1, 2, 3, 4, 700, 1, 5, 600], 4096, 4), ([7, 1, 2], 30, 4),
                                         ([9, 1], 64, 1), ([2, 1, 12], 64, 6)])
def test_short_convolution_of_unequal_portions(ops, run, lens, C, taps):
    """Portions shorter and longer than the taps, each after inputs of its own in a scrambled slot, in rows wider than the
    channels; the form with eight tokens per thread gives what the plain one gives."""
    g, n = _gen(C), sum(lens)
    xz = torch.randn(n, C + 8, device=DEV, generator=g)
    w, b = torch.randn(C, taps, device=DEV, generator=g), torch.randn(C, device=DEV, generator=g)
    state = torch.randn(9, 4 + taps * C, device=DEV, generator=g)
    slots = torch.randperm(9, generator=torch.Generator().manual_seed(1))[:len(lens)].tolist()
    got, got_run = ops.scan_conv(xz[:, 4:4 + C], w, b, state, 4, _step_ctx(lens, slots, [0] * len(lens)), C, taps, run)
    at = 0
    for k, slot in zip(lens, slots):
        before = state[slot, 4:4 + (taps - 1) * C].view(taps - 1, C)
        x = torch.cat([before, xz[at:at + k, 4:4 + C]]).double().cpu()
        want = P.silu(P.causal_conv(x, w.cpu(), b.cpu())[taps - 1:])
        assert (got[at:at + k].double().cpu() - want).abs().max() <= 1e-5 * (1 + want.abs().max())
        at += k
    assert got_run is got if run is None else torch.equal(got_run, got.to(run))


def test_state_space_keeps_its_digits_over_a_long_prompt(ops):
    """3,000 tokens with decays from 1 - 1e-5 to 0.2 per step, in portions and then one by one, against the plain one."""
    g = _gen(1)
    Hh, V, N, G, taps, T = 4, 6, 16, 2, 3, 3000
    C = Hh * V + 2 * G * N
    proj = torch.randn(T, C + Hh, device=DEV, generator=g)
    proj[:, C:] = proj[:, C:] * 0.5 - 3.0
    a_log = torch.tensor([-8.0, -5.0, -2.0, 3.0], device=DEV)
    conv = torch.randn(C, taps, device=DEV, generator=g)
    bias, skip = 0.1 * torch.randn(C, device=DEV, generator=g), torch.randn(Hh, device=DEV, generator=g)
    dt_bias = torch.tensor([0.0, 1.0, -1.0, 2.0], device=DEV)
    tail = Hh * V * N
    state = torch.zeros(1, tail + (taps - 1) * C, device=DEV)
    got, at = [], 0
    for k in [1500, 700, 777] + [1] * 23:
        x, ctx = proj[at:at + k], _step_ctx([k], [0], [at])
        xc, _ = ops.scan_conv(x[:, :C], conv, bias, state, tail, ctx, C, taps)
        got.append(ops.state_space(xc, x[:, :C], x[:, C:], dt_bias, torch.exp(a_log), skip, state, tail, ctx, Hh, G, N, V, taps))
        at += k
    p = proj.double().cpu()
    xbc = P.silu(P.causal_conv(p[:, :C], conv.cpu(), bias.cpu()))
    want = P.scalar_decay_state(xbc[:, :Hh * V].reshape(T, Hh, V), xbc[:, Hh * V:Hh * V + G * N].reshape(T, G, N),
                                xbc[:, Hh * V + G * N:].reshape(T, G, N), P.softplus(p[:, C:] + dt_bias.double().cpu()),
                                a_log.double().cpu(), skip.double().cpu()).reshape(T, -1)
    assert (torch.cat(got).double().cpu() - want).abs().max() <= 2e-5 * want.abs().max()


@pytest.mark.parametrize("i_shift,f_shift", [(0.0, 12.0), (-40.0, 4.0), (30.0, -3.0), (0.0, 2.0)])
def test_matrix_memory_keeps_its_digits_and_its_maximum(ops, i_shift, f_shift):
    """2,500 tokens with forget gates from nearly one (logs of some 1e-6, added one by one to the maximum) down, and input
    gates far below or above the maximum, in portions and then one by one, against the plain one; the normed read-out."""
    g = _gen(2)
    Hh, dk, dv, T, cap = 2, 8, 6, 2500, 40.0
    ld = Hh * (2 * dk + dv + 2)
    proj = torch.randn(T, ld, device=DEV, generator=g)
    i_off, f_off = ld - 2 * Hh, ld - Hh
    i_bias, f_bias = torch.tensor([i_shift, i_shift + 1.0], device=DEV), torch.tensor([f_shift, f_shift + 1.0], device=DEV)
    m_off = Hh * (dv + 1) * dk
    state = torch.zeros(1, m_off + ops.MATRIX_MEMORY_RECORD * Hh, device=DEV)
    got, at = [], 0
    for k in [1500, 700, 277] + [1] * 23:
        o, den = ops.matrix_memory(proj[at:at + k], 0, Hh * dk, 2 * Hh * dk, i_off, f_off, i_bias, f_bias, cap, dk ** -0.5, state, m_off,
                                   _step_ctx([k], [0], [at]), Hh, dk, dv)
        got.append((o.view(k, Hh, dv) / den[:, :, None]).double().cpu())
        at += k
    p = proj.double().cpu()
    i_log = cap * torch.tanh((p[:, i_off:f_off] + i_bias.double().cpu()) / cap)
    f_log = -P.softplus(-cap * torch.tanh((p[:, f_off:] + f_bias.double().cpu()) / cap))
    want = P.matrix_memory(p[:, :Hh * dk].view(T, Hh, dk) * dk ** -0.5, p[:, Hh * dk:2 * Hh * dk].view(T, Hh, dk),
                           p[:, 2 * Hh * dk:i_off].reshape(T, Hh, dv), i_log, f_log)
    got = torch.cat(got)
    assert torch.isfinite(got).all()
    err = (got - want).abs() / (1e-3 * want.abs().max() + want.abs().amax(dim=-1, keepdim=True))
    assert err.median() <= 2e-6 and err.max() <= 2e-3          # (where n . q passes zero, the quotient loses digits)


# ---------------------------------------------------------------------------- feed-forward

@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n,d,ff", [(1, 64, 160), (3, 320, 96), (8, 256, 512), (40, 48, 36), (5, 102, 18)])
def test_two_matrices_around_an_exact_gelu(ops, dtype, n, d, ff):
    from batchspec_b200.parts.base import FEED_FORWARDS, PartSpec, Runtime, build_part
    g = _gen(n + ff)
    part = build_part(FEED_FORWARDS, PartSpec("mlp", dict(dim=d, intermediate=ff, activation="gelu")), Runtime(dtype, torch.device(DEV)))
    w = {k: (torch.randn(*ps.shape, device=DEV, generator=g) * (3 / math.sqrt(d))).to(dtype) for k, ps in part.param_specs().items()}
    part.bind(w)
    x = torch.randn(n, d, device=DEV, generator=g).to(dtype)
    u = ops.linear_act(x, w["up"], "gelu").double()
    want = P.gelu(x.double() @ w["up"].double().T)
    assert (u - want).abs().max() <= (2e-5 if dtype == torch.float32 else 2e-2) * (1 + want.abs().max())
    want = P.dense_ff(x.double().cpu(), {k: v.cpu() for k, v in w.items()})
    assert (part.forward(x, None).double().cpu() - want).abs().max() <= (2e-5 if dtype == torch.float32 else 2e-2) * want.abs().max()
    ops.check_status()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n,d,ff,E,top,identity,shared", [
    (7, 48, 16, 6, 2, 3, 24), (1, 100, 20, 7, 7, 0, 0), (40, 64, 32, 1, 1, 1, 8), (300, 320, 96, 12, 3, 4, 64), (3, 320, 64, 8, 2, 8, 96),
    (70, 64, 128, 16, 3, 1, 200), (600, 96, 40, 9, 2, 5, 20), (9, 256, 96, 4, 6, 2, 0), (2000, 128, 64, 8, 4, 4, 128),
    (2500, 64, 32, 2, 1, 30, 0), (5, 102, 18, 6, 1, 2, 30)])
def test_corrected_router_identity_experts_and_a_gated_shared_expert(ops, dtype, n, d, ff, E, top, identity, shared):
    """The chosen numbers, their weights and the summed outputs, on rows whose choices are not close (spread logits)."""
    from batchspec_b200.parts.base import FEED_FORWARDS, PartSpec, Runtime, build_part
    g = _gen(n + E)
    part = build_part(FEED_FORWARDS, PartSpec("routed_glu", dict(
        dim=d, intermediate=ff, n_experts=E, top=top, bias=False, scores="softmax", correction=True, identity=identity, shared=shared,
        shared_gate=bool(shared))), Runtime(dtype, torch.device(DEV)))
    w = {}
    for name, ps in part.param_specs().items():
        std = 1.5 / math.sqrt(d) if name in ("router", "shared_gate") else 0.3
        w[name] = (torch.randn(*ps.shape, device=DEV, generator=g) * std).to(dtype)
    part.bind(w)
    x = torch.randn(n, d, device=DEV, generator=g).to(dtype)
    ids, wts, *gate = ops.moe_route(x, part.w_router, part.b_correction, 1, 1, top, 1.0, softmax=True, group_max=True, renormalise=True,
                                    extra_rows=int(bool(shared)))
    xd, router, corr = x.double().cpu(), w["router"].cpu(), w["correction"].cpu()
    idx, wt = P.route(xd, router, corr, top)
    choice = torch.sort(torch.softmax(xd @ router.double().T, -1) + corr.double(), dim=-1, descending=True).values
    clear = choice[:, top - 1] - choice[:, top] > 0.01 if top < E + identity else torch.ones(n, dtype=torch.bool)
    assert clear.float().mean() > 0.5
    assert torch.equal(torch.sort(ids.cpu().long()[clear], dim=-1).values, torch.sort(idx[clear], dim=-1).values)
    order, mine = torch.argsort(ids.cpu().long(), dim=-1), torch.argsort(idx, dim=-1)
    assert (wts.double().cpu().gather(1, order) - wt.gather(1, mine))[clear].abs().max() <= (1e-5 if dtype == torch.float32 else 1e-2)
    if identity > 2 and n > 30:
        assert (idx >= E).any(), "no identity expert was chosen"
    named = {"router": router, "correction": corr}
    for e in range(E):
        named.update({f"e{e}.{k}": w[f"{k}{e}"].cpu() for k in ("gate", "up", "down")})
    if shared:
        named.update({f"shared.{k}": w[f"shared.{k}"].cpu() for k in ("gate", "up", "down")})
        named["shared.sg"] = w["shared_gate"].cpu()
        assert (gate[0].double().cpu() - xd @ named["shared.sg"].double().T).abs().max() <= (1e-5 if dtype == torch.float32 else 1e-2) * 10
    want = P.routed_ff(xd, named, dict(router=dict(experts=E, top=top), shared=dict(ff=shared) if shared else None))
    err = (part.forward(x, None).double().cpu() - want).abs().amax(dim=-1) / want.abs().max()
    assert err[clear].max() <= (2e-5 if dtype == torch.float32 else 3e-2)


def test_rows_that_only_identity_experts_take(ops):
    """Every token's choices are identity experts: no expert has a row, and the output is the input."""
    from batchspec_b200.parts.base import FEED_FORWARDS, PartSpec, Runtime, build_part
    for dtype in TYPES:
        for n in (1, 9, 1500):
            part = build_part(FEED_FORWARDS, PartSpec("routed_glu", dict(dim=64, intermediate=32, n_experts=3, top=2, bias=False,
                              scores="softmax", correction=True, identity=4)), Runtime(dtype, torch.device(DEV)))
            w = {k: torch.randn(*ps.shape, device=DEV, generator=_gen(1)).to(dtype) for k, ps in part.param_specs().items()}
            w["router"] *= 0.1
            w["correction"] = torch.tensor([0., 0., 0., 5., 5., 5., 5.], device=DEV)
            part.bind(w)
            x = torch.randn(n, 64, device=DEV, generator=_gen(2)).to(dtype)
            assert (part.forward(x, None).double() - x.double()).abs().max() <= (1e-6 if dtype == torch.float32 else 3e-2)


# ---------------------------------------------------------------------------- whole mixers

def _one_mixer_against_plain(cfg, dtype, page, plain, lens):
    """Build the model's only mixer with random tensors and run it through the step context of a real engine: a prompt
    and then five tokens one by one."""
    from batchspec_b200.engine import StepEntry
    from batchspec_b200.kernels import ops
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    with tempfile.TemporaryDirectory() as tmp:
        folder = _make(tmp, cfg, 5, stored, std=0.25)
        _, w = P.read_model_folder(folder)
        eng = _engine(folder, dtype, page, 120, max_requests=2)
        block = eng.model.blocks[0]
        seen = {"x": [], "y": []}

        class Spy:
            def __init__(self, mixer):
                self.mixer = mixer

            def forward(self, x, ctx, cache):
                seen["x"].append(x.detach().double().cpu())
                y = self.mixer.forward(x, ctx, cache)
                seen["y"].append(y.detach().double().cpu())
                return y
        block.mixer = Spy(block.mixer)
        for rid, n in zip("ab", lens):
            toks = H.random_tokens(n, cfg["vocab"], n)
            eng.admit(rid)
            eng.step([StepEntry(rid, toks[:n - 5], [])])
            for tok in toks[n - 5:]:
                eng.step([StepEntry(rid, [tok], [])])
            xs, ys = torch.cat(seen["x"]), torch.cat(seen["y"])
            seen["x"].clear(), seen["y"].clear()
            sub = {k[len("l0.mix."):]: v for k, v in w.items() if k.startswith("l0.mix.")}
            want = plain(xs, sub, cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
            assert (ys - want).abs().max() <= (5e-5 if dtype == "float32" else 4e-2) * want.abs().max()
        ops.check_status()


SMALL, WIDE = _left(4, 2, 12, 20, 0.3, 9, 3, 777.0, 8, 2.0), _left(8, 1, 64, 64, 0.125, 40, 7, 1e4, 32, LLAMA3)
WIDER, PLAIN = _left(8, 2, 128, 128, 0.09, 30, 20, 1e5, 128, 4.0), _left(3, 3, 10, 4, 0.4, None, 0, dims=0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("left,right", [(SMALL, (3, 8, 12, 1, 4, 2)), (WIDE, (2, 32, 16, 2, 2, 1)), (WIDER, (4, 64, 128, 1, 4, 4)),
                                        (PLAIN, (6, 5, 3, 3, 1, 5))], ids=["small", "d64", "d128", "full"])
def test_attention_beside_a_state_space(ops, dtype, left, right):
    _one_mixer_against_plain(_config(50, 96, 1e-5, 1.0, [_ssd(left, *right)]), dtype, 8, P.mix_normed, lens=(33, 150))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("left,right", [(SMALL, (3, 8, 12, 5.0)), (WIDE, (2, 32, 16, 12.0)), (WIDER, (4, 64, 128, 15.0)),
                                        (PLAIN, (5, 3, 7, 2.0))], ids=["small", "d64", "d128", "full"])
def test_attention_beside_a_matrix_memory(ops, dtype, left, right):
    cfg = _config(50, 96, 1e-5, 1.0, [_mem(left, *right, (1.3, 0.6))])
    _one_mixer_against_plain(cfg, dtype, 8, P.mix_scaled, lens=(33, 150))


def test_a_sharp_softmax_over_hundreds_of_keys(ops):
    """A scale far above 1 / sqrt(size): nearly every softmax is decided by one key, which a kernel that skipped or
    misplaced it would lose.  float32, prompt and decoding."""
    cfg = _config(50, 96, 1e-5, 1.0, [_ssd(_left(8, 2, 32, 24, 6.0, 120, 60, 500.0, 16, 2.0), 1, 8, 8, 1, 2, 1)])
    _one_mixer_against_plain(cfg, "float32", 8, P.mix_normed, lens=(9, 400))


# ---------------------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_tail_portions(tmp_path, name, dtype):
    cfg, seed, page = CONFIGS[name]
    folder = _folder(tmp_path, name, dtype)
    reqs = _requests(name)
    longest = max(len(t) for t in reqs.values())
    eng = _engine(folder, dtype, page, -(-longest // page) + 1)
    for rid, toks in reqs.items():
        one = {rid: toks}
        got = H.run_steps_in_process(eng, H.whole(rid, toks))
        _compare(got, folder, one, dtype)
        got_tail = H.run_steps_in_process(eng, H.tail_decoded(rid, toks, tail=40))
        _compare(got_tail, folder, one, dtype)
        got_port = H.run_steps_in_process(eng, H.portions(rid, toks, [7, 2, 16, 3, 2, 5, 2, 31]))
        _compare(got_port, folder, one, dtype)
        _rows_agree(got, got_tail, dtype)
        _rows_agree(got, got_port, dtype)
    assert all(g.pool.num_held == 0 for g in eng.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_token_by_token_from_the_first_token(tmp_path, name, dtype):
    """A whole request decoded one token at a time (the first tokens of a sequence, every page border, window edge and
    block end, long decoding) against the oracle."""
    cfg, seed, page = CONFIGS[name]
    folder = _folder(tmp_path, name, dtype)
    toks = H.random_tokens(170, cfg["vocab"], 4)
    eng = _engine(folder, dtype, page, 44)
    got = H.run_steps_in_process(eng, H.portions("t", toks, [1]))
    _compare(got, folder, {"t": toks}, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_mixed_requests_reuse_pages_and_slots(tmp_path, name, dtype):
    cfg, seed, page = CONFIGS[name]
    folder = _folder(tmp_path, name, dtype)
    base = _requests(name)
    reqs = dict(base)
    for i, (rid, toks) in enumerate(base.items()):          # twice as many requests as may be live
        reqs[f"s{i}"] = H.random_tokens(max(2, len(toks) // 2 + 3), cfg["vocab"], 999 + i)
    steps = H.mixed(reqs, seed=seed + 7, max_live=4)
    max_tokens = H.max_live_tokens(steps, round_to=page)
    eng = _engine(folder, dtype, page, max_tokens // page, max_requests=4)
    got = H.run_steps_in_process(eng, steps)
    _compare(got, folder, reqs, dtype)
    alone = _engine(folder, dtype, page, -(-max(len(t) for t in reqs.values()) // page) + 1)
    for rid in ("r2", "r3"):                                # every request alone gives the same rows as in the batch
        one = H.run_steps_in_process(alone, H.whole(rid, reqs[rid]))
        _rows_agree(one, {k: got[k] for k in one}, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run_program(tmp_path, dtype):
    folder = _folder(tmp_path, "A", dtype)
    reqs = _requests("A")
    steps = H.mixed(reqs, seed=3, max_live=4)
    got = H.run_trace_subprocess(folder, dtype, steps, tmp_path / "out", H.max_live_tokens(steps, round_to=64))
    _compare(got, folder, reqs, dtype)


MAKERS = [lambda t: H.whole("e", t), lambda t: H.portions("e", t, [1]), lambda t: H.portions("e", t, [10, 3, 2, 9])]


EDGE_STEPS = [lambda t: H.whole("e", t), lambda t: H.portions("e", t, [1]), lambda t: H.portions("e", t, [10, 3, 2, 9])]


def _silence_right(eng):
    """Only the attention of the model's one mixer is left."""
    mixer = eng.model.blocks[0].mixer
    if mixer.out_norm_eps is not None:
        mixer.w_right.zero_()
    else:
        mixer.wo[:, mixer.left.out_width:].zero_()


@pytest.mark.parametrize("make", range(3))
@pytest.mark.parametrize("name,window,keep", [("EDGE", 12, 3), ("EDGE_2", 9, 0)])
def test_exactly_the_positions_that_see_a_token_move_with_it(tmp_path, make, name, window, keep):
    """One attention layer (the recurrence beside it silenced): after a change of one token, the positions that have it in
    their window, or all later ones for a kept token, have other logits, and the others the same ones bit for bit."""
    cfg, seed, page = CONFIGS[name]
    folder = _folder(tmp_path, name, "float32", std=0.3)
    base = H.random_tokens(48, cfg["vocab"], 2)
    eng = _engine(folder, "float32", page, -(-48 // page))
    _silence_right(eng)
    ref = H.run_steps_in_process(eng, EDGE_STEPS[make](base))
    for where in (0, 1, 2, 3, 4, 7, 8, 15, 16, 30):
        toks = list(base)
        toks[where] = (toks[where] + 1) % cfg["vocab"]
        got = H.run_steps_in_process(eng, EDGE_STEPS[make](toks))
        for p in range(48):
            sees = p >= where and (p - where < window or where < keep)
            assert np.array_equal(got[("e", p)], ref[("e", p)]) == (not sees), (where, p)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_moves_the_logits_through_kept_tokens_and_states(tmp_path, dtype):
    """Changing ONE token far back changes the last position's logits in the oracle although every window has passed it.
    The engine follows, decoded alone and as the end of a portion."""
    cfg, seed, page = CONFIGS["A"]
    folder = _make(tmp_path / "far", cfg, 21, torch.float32 if dtype == "float32" else torch.bfloat16, std=0.15)
    base = H.random_tokens(260, cfg["vocab"], 8)
    eng = _engine(folder, dtype, page, 70)
    ref0 = _oracle(folder, base)[-1]
    moved, over = [], 0
    for where in (0, 2, 4, 127, 128, 200):
        toks = list(base)
        toks[where] = (toks[where] + 17) % cfg["vocab"]
        ref = _oracle(folder, toks)
        moved.append(np.abs(ref[-1] - ref0).max() / np.abs(ref0).max())
        for steps in (H.tail_decoded("f", toks, tail=3), H.portions("f", toks, [250, 10])):
            got = H.run_steps_in_process(eng, steps)
            err = np.abs(got[("f", len(toks) - 1)] - ref[-1]).max() / np.abs(ref).max()
            over += err > H.TOL[dtype] * (1 if dtype == "float32" else 2)
    assert over <= (0 if dtype == "float32" else 1)
    assert max(moved) > 1e-3, "no far token moved the last logits: the weights hide what this test is for"


def test_generation_through_the_scheduler(tmp_path):
    """Greedy generation through Engine.generate (scheduler, portions, captured decode steps) gives the tokens that the
    oracle's argmax gives, token by token, for requests of unequal length under page pressure."""
    from batchspec_b200.engine import Engine
    from batchspec_b200.engine.sequence import Sequence
    cfg, seed, page = CONFIGS["A"]
    folder = _make(tmp_path / "gen", cfg, 31, torch.float32, std=0.2)
    prompts = [H.random_tokens(n, cfg["vocab"], 50 + n) for n in (3, 19, 42, 7, 64)]
    outputs = []
    for graphs in (True, False):
        eng = Engine(dtype="float32", device=DEV)
        eng.load_model(model_dir=folder)
        eng.use_cuda_graphs = graphs
        eng.setup_caches(max_batch_size=3, max_seq_length=96, page_size=page, prefill_chunk_size=16, num_pages=26)
        eng.setup_sampling_params(temperature=0.0)
        done = {s.seq_id: s for s in eng.generate([Sequence(i, list(p), max_new_tokens=25) for i, p in enumerate(prompts)])}
        outputs.append([done[i].output_ids for i in range(len(prompts))])
        for i, p in enumerate(prompts):
            toks = list(p) + list(done[i].output_ids)
            assert len(done[i].output_ids) == 25
            ref = _oracle(folder, toks)
            for k in range(25):
                row = ref[len(p) + k - 1]
                top2 = np.sort(row)[-2:]
                if top2[1] - top2[0] > 1e-3 * np.abs(row).max():
                    assert toks[len(p) + k] == int(row.argmax()), (graphs, i, k)
        assert all(g.pool.num_held == 0 for g in eng.cache.groups)
    assert outputs[0] == outputs[1]


@pytest.mark.parametrize("batch", [1, 3])
def test_captured_decode_steps_at_tensor_core_sizes(tmp_path, batch):
    """bfloat16 at sizes that run the tensor-core kernels: tokens from captured decode steps (padded to the bucket) equal
    those of steps launched kernel by kernel, over window edges and page borders."""
    from batchspec_b200.engine import Engine
    from batchspec_b200.engine.sequence import Sequence
    folder = _folder(tmp_path, "C", "bfloat16", std=0.05)
    prompts = [H.random_tokens(n, CFG_C["vocab"], 70 + n) for n in (150, 33, 90)[:batch]]
    out = []
    for graphs in (True, False):
        eng = Engine(dtype="bfloat16", device=DEV)
        eng.load_model(model_dir=folder)
        eng.use_cuda_graphs = graphs
        eng.setup_caches(max_batch_size=4, max_seq_length=256, page_size=16, prefill_chunk_size=64)
        eng.setup_sampling_params(temperature=0.0)
        done = {s.seq_id: s for s in eng.generate([Sequence(i, list(p), max_new_tokens=40) for i, p in enumerate(prompts)])}
        out.append([done[i].output_ids for i in range(batch)])
    assert out[0] == out[1]
