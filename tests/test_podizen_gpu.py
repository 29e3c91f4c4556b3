"""The Podizen design on the engine against the plain implementation in ``plain_podizen.py``: every mechanism alone
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
import plain_podizen as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
TYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64


def _attn(heads, kv_heads, dim, vdim, scale, window=None, mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if window:
        m["mask"] = dict(size=window)
    return dict(type="attention", mixer=m, mlp=mlp)


def _par(left, right, mlp=None):
    heads, kv_heads, dim, vdim, scale, window, pool, base, dims = left
    a = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=window),
             rot=dict(base=base, dims=dims))
    if pool:
        a["mask"]["pool"] = pool
    heads, dim, vdim, decay, base, dims = right
    b = dict(heads=heads, dim=dim, vdim=vdim, decay=decay, rot=dict(base=base, dims=dims))
    return dict(type="parallel", mixer=dict(left=a, right=b), mlp=mlp)


def _moe(ff, experts, top, groups=None, shared=0):
    f = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if groups:
        f["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if shared:
        f["shared"] = dict(ff=shared)
    return f


def _config(vocab, width, eps, layers):
    return dict(architecture="Podizen", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


# Configurations that share no size.  A: windows that are no multiple of the page or of the blocks, a part of the head
# rotated, a layer without a feed-forward.  B: a width that is no multiple of 4, blocks of ONE token, a window SHORTER than
# its blocks, one expert, all groups kept, no shared expert, a whole head rotated, an odd head.  C: sizes at which the
# tensor-core kernels run in bfloat16 (heads of 64 and 128 with values as wide), many blocks.  SEEN: one pooled attention
# layer (the retention beside it is silenced), WINDOW: one attention layer with a distance bias.
CFG_A = _config(200, 48, 1e-5, [
    _attn(4, 2, 12, 20, 0.25, 10, _moe(16, 6, 3, (3, 2), 24)),
    _par((4, 2, 10, 6, 0.3, 9, 4, 500.0, 6), (3, 8, 12, [0.5, 0.9, 0.99], 900.0, 4)),
    _par((3, 1, 8, 12, 0.4, 14, 5, 40.0, 8), (1, 4, 20, [0.999], 30.0, 4), _moe(20, 8, 2, (4, 1), 12)),
    _attn(6, 3, 6, 9, 0.5, 7, _moe(12, 5, 2, None, 8))])
CFG_B = _config(513, 102, 1e-6, [
    _par((2, 2, 6, 6, 0.4, 5, 1, 1e4, 6), (2, 10, 14, [0.97, 0.3], 77.0, 10), _moe(36, 1, 1)),
    _attn(5, 1, 7, 3, 0.3, 1, _moe(18, 4, 4, (2, 2))),
    _par((6, 1, 16, 11, 0.2, 3, 8, 1e3, 2), (5, 6, 5, [0.8, 0.85, 0.9, 0.95, 1.0], 10.0, 6), _moe(10, 9, 1, (3, 1), 30))])
CFG_C = _config(640, 320, 1e-5, [
    _attn(8, 2, 64, 64, 0.125, 80, _moe(64, 8, 2, (4, 2), 96)),
    _par((8, 2, 128, 128, 0.09, 70, 4, 1e5, 64), (4, 64, 64, [0.9, 0.97, 0.99, 0.998], 1e4, 32), _moe(96, 4, 2, (2, 1), 128)),
    _par((4, 4, 64, 64, 0.15, 33, 3, 5e3, 64), (2, 32, 96, [0.96, 0.995], 1e3, 32)),
    _attn(8, 1, 128, 128, 0.1, 100, _moe(128, 6, 3, None, 64))])
CFG_SEEN = _config(150, 32, 1e-5, [_par((2, 1, 8, 12, 0.7, 9, 4, 100.0, 8), (2, 4, 4, [0.9, 0.5], 50.0, 4), _moe(8, 4, 2, (2, 1), 8))])
CFG_WINDOW = _config(150, 32, 1e-5, [_attn(2, 1, 8, 8, 0.5, 12, _moe(8, 4, 2, (2, 1), 8))])
CONFIGS = {"A": (CFG_A, 11, 4), "B": (CFG_B, 12, 8), "C": (CFG_C, 13, 16), "SEEN": (CFG_SEEN, 14, 4),
           "WINDOW": (CFG_WINDOW, 15, 8)}
LENGTHS = {"A": [1, 6, 23, 90], "B": [2, 9, 41, 130], "C": [3, 64, 150, 400]}


def _folder(tmp_path, name, dtype, std=0.08):
    cfg, seed, _ = CONFIGS[name]
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    return H.make_folder(tmp_path / f"f{name}_{dtype}", cfg, seed, dtype=stored, std=std)


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
    """Every row against the oracle.  float32: no row beyond the tolerance.  bfloat16: three rows in a hundred, or one,
    may be (a router's choice between two experts or groups whose scores differ by less than the rounding falls either
    way, and a later layer sees the row)."""
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


# ---------------------------------------------------------------------------- branches that are normed before they join

@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n,d", [(3, 96), (5, 50), (2, 4096), (4, 7), (1, 8192), (600, 640), (2, 20000), (3, 1)])
@pytest.mark.parametrize("pair", [False, True])
def test_branch_join_norms_adds_averages_and_norms(ops, dtype, n, d, pair):
    """x = src + rms(y) post (y one branch, or a pair normed each by itself), kept in the history, averaged over depth,
    written back and normed; every part on its own is the same kernel."""
    g = _gen(n + d)
    rnd = lambda *s: torch.randn(*s, device=DEV, generator=g)
    src, a, b = rnd(n, d), rnd(n, d).to(dtype), (3 * rnd(n, d)).to(dtype)
    w = [(1 + 0.3 * rnd(d)) for _ in range(4)]
    eps, slot = 1e-5, 3
    hist = rnd(slot + 2, n, d)
    coef = rnd(slot + 1)
    y = (P.rms_norm(a.double(), w[0], eps) + P.rms_norm(b.double(), w[1], eps)) if pair else a.double()
    delta = ops.NormedPair(a, b, w[0], w[1], eps) if pair else a
    own = src.double() + P.rms_norm(y, w[2], eps)
    want = P.depth_average([hist[j].double() for j in range(slot)] + [own], coef.cpu())
    tol = (2e-5 if dtype == torch.float32 else 2e-2)
    near = lambda got, ref, t=2e-5: (got.double() - ref).abs().max() <= t * (1 + ref.abs().max())
    # the rows that go to the head: nothing is written back
    rows = torch.tensor([n - 1, 0, n // 2], dtype=torch.int32, device=DEV)
    picked, h0, s0 = torch.empty(3, d, device=DEV, dtype=dtype), hist.clone(), src.clone()
    ops.branch_join(src, delta, out=picked, post=w[2], branch_eps=eps, norm_w=w[3], eps=eps, hist=hist, slot=slot, coef=coef,
                    rows=rows)
    assert near(picked, P.rms_norm(want, w[3], eps)[rows.long()], tol) and torch.equal(hist, h0) and torch.equal(src, s0)
    # everything at once
    x, out = src.clone(), torch.empty(n, d, device=DEV, dtype=dtype)
    ops.branch_join(x, delta, dst=x, out=out, post=w[2], branch_eps=eps, norm_w=w[3], eps=eps, hist=hist, slot=slot,
                    store=True, coef=coef)
    assert near(x, want) and near(out, P.rms_norm(want, w[3], eps), tol)
    h0[slot] = hist[slot]
    assert near(hist[slot], own) and torch.equal(hist, h0)
    # no weight on the branch, no average, no history
    x2 = src.clone()
    ops.branch_join(x2, delta, dst=x2, out=out, norm_w=w[3], eps=eps)
    assert near(x2, src.double() + y) and near(out, P.rms_norm(src.double() + y, w[3], eps), tol)
    # a step's first norm: the embedding is kept and normed
    ops.branch_join(src, None, out=out, norm_w=w[3], eps=eps, hist=hist, slot=0, store=True)
    assert torch.equal(hist[0], src) and near(out, P.rms_norm(src.double(), w[3], eps), tol)
    if pair:                                                      # the pair alone, as a mixer returns it
        ops.branch_join(None, delta, out=out)
        assert near(out, y, tol)


# ---------------------------------------------------------------------------- attention: distance bias, pooled blocks

def _paged(rows, ps, perm, at, G, hd, vd, pages):
    """Write rows [L, G, hd + vd] into the pages perm[at], perm[at + 1] ... in the layout [k | v]."""
    for p in range(rows.shape[0]):
        page = pages[int(perm[at + p // ps])].reshape(-1)
        page[:G * ps * hd].view(G, ps, hd)[:, p % ps] = rows[p, :, :hd]
        page[G * ps * hd:].view(G, ps, vd)[:, p % ps] = rows[p, :, hd:]


def _attention_case(ops, dtype, Hq, G, hd, vd, ps, q_lens, kv_lens, window, pool=None, biased=False, scale=None, change=None,
                    seed=0, gate=False, generic=False, want_plain=True):
    """Random queries over cached rows whose pages lie in scrambled order; the table entries of pages that the window
    (and the block that is not yet whole) has passed are -1.  The pooled pages are filled by the kernels: ``pool_append``
    over portions that end where the step begins, then over the step's own.  ``change(q, rows, e)`` edits the inputs.
    Returns (got, want) [n, Hq, vd]."""
    g = _gen(seed)
    n = sum(q_lens)
    qo = [0] + list(np.cumsum(q_lens))
    q = torch.randn(n, Hq, hd, device=DEV, generator=g)
    rows = [torch.randn(L, G, hd + vd, device=DEV, generator=g) for L in kv_lens]
    if change is not None:
        change(q, rows, qo)
    q, rows = q.to(dtype), [r.to(dtype) for r in rows]
    scale = scale or 1.0 / math.sqrt(hd)
    per = [-(-L // ps) for L in kv_lens]
    at = [0] + list(np.cumsum(per))
    perm = torch.randperm(at[-1] + 2, generator=torch.Generator().manual_seed(seed + 1))
    pages = torch.randn(at[-1] + 2, 1, ps * G * (hd + vd), device=DEV, generator=g).to(dtype)
    for e, r in enumerate(rows):
        _paged(r, ps, perm, at[e], G, hd, vd, pages)
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32, device=DEV)
    tables = SimpleNamespace(kv_indptr=i32(at), kv_indices=i32(perm), page_size=ps)
    pooled = None
    if pool:
        pper = [-(-(L // pool) // ps) for L in kv_lens]
        pat = [0] + list(np.cumsum(pper))
        pperm = torch.randperm(pat[-1] + 1, generator=torch.Generator().manual_seed(seed + 2))
        pooled_pages = torch.zeros(pat[-1] + 1, 1, ps * G * (hd + vd), device=DEV, dtype=dtype)
        pooled = (pool, pooled_pages, SimpleNamespace(kv_indptr=i32(pat), kv_indices=i32(pperm), page_size=ps))
        for lens, ends in (([L - k for L, k in zip(kv_lens, q_lens)], [L - k for L, k in zip(kv_lens, q_lens)]), (q_lens, kv_lens)):
            live = [e for e in range(len(lens)) if lens[e] > 0]
            if not live:
                continue
            starts = torch.cat([torch.arange(ends[e] - lens[e], ends[e]) for e in range(len(lens))])
            c = SimpleNamespace(qo_indptr=i32([0] + list(np.cumsum(lens))), positions=i32(starts), n_entries=len(lens),
                                max_q_len=max(lens))
            ops.pool_append(pages, c, tables, pooled, G, hd, vd)
        for e, L in enumerate(kv_lens):                           # entries are block means, in their pages
            for b in (0, L // pool // 2, L // pool - 1):
                if L < pool:
                    continue
                page = pooled_pages[int(pperm[pat[e] + b // ps])].reshape(-1)
                ref = rows[e][b * pool:(b + 1) * pool].double().mean(0)
                tol = 1e-6 if dtype == torch.float32 else 1e-2
                assert (page[:G * ps * hd].view(G, ps, hd)[:, b % ps].double() - ref[:, :hd]).abs().max() <= tol * 4
                assert (page[G * ps * hd:].view(G, ps, vd)[:, b % ps].double() - ref[:, hd:]).abs().max() <= tol * 4
    table = perm.clone()
    for e, L in enumerate(kv_lens):
        before = L - q_lens[e]
        need = max(0, before - window + 1) if window else 0
        if pool:
            need = min(need, before // pool * pool)
        table[at[e]:at[e] + need // ps] = -1
    tables = SimpleNamespace(kv_indptr=i32(at), kv_indices=i32(table), page_size=ps)
    pos = torch.cat([torch.arange(L - k, L) for k, L in zip(q_lens, kv_lens)])
    ctx = SimpleNamespace(qo_indptr=i32(qo), positions=i32(pos), n_entries=len(q_lens), n_tokens=n, max_q_len=max(q_lens),
                          tok_entry=i32(np.repeat(np.arange(len(q_lens)), q_lens)), max_kv_len=max(kv_lens), kv_len=i32(kv_lens),
                          extras={"min_q_len": min(q_lens)})
    slopes = torch.tensor(P.bias_slopes(Hq), device=DEV, dtype=torch.float32) if biased else None
    out = torch.full((n, Hq * vd), float("nan"), device=DEV, dtype=dtype)
    gates = torch.randn(n, Hq * vd, device=DEV, generator=g) if gate else None
    if hd == vd and not gate:
        ops.FORCE_GENERIC_ATTENTION = generic
        try:
            ops.paged_attention(q.reshape(n, -1), out, pages, ctx, tables, Hq, G, hd, scale, window or 0, slopes=slopes,
                                slopes_l2=ops.sink_table(slopes) if biased else None, pooled=pooled)
        finally:
            ops.FORCE_GENERIC_ATTENTION = False
    else:
        ops.masked_attention(q.reshape(n, -1), out, pages, ctx, tables, Hq, G, hd, vd, scale, window or 0, slopes=slopes,
                             pooled=pooled, gate=gates)
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
        o = P.attend(full_q, x[:, :, :hd], x[:, :, hd:], scale, window, pool, P.bias_slopes(Hq) if biased else None)
        want[qo[e]:qo[e + 1]] = o[L - k:]
    if gate:
        want *= torch.sigmoid(gates.double().cpu()).view(n, Hq, vd)
    return got, want


BIAS_SHAPES = [
    # Hq, G, hd, vd, page, q_lens, kv_lens, window
    (3, 3, 16, 16, 4, [5, 1, 2], [5, 9, 30], 7),
    (4, 1, 20, 36, 5, [3, 11], [17, 11], None),
    (8, 2, 64, 64, 16, [1, 1, 1, 1], [300, 17, 64, 129], 64),
    (8, 2, 64, 64, 16, [70, 2, 1], [200, 5, 333], 33),
    (16, 2, 128, 128, 16, [130, 1, 3, 64], [130, 555, 40, 600], 96),
    (6, 3, 128, 128, 8, [1, 1], [1300, 31], 1000),
    (4, 1, 128, 128, 32, [300], [700], None),
    (4, 2, 256, 256, 16, [40, 1], [90, 200], 50),
    (8, 8, 128, 128, 5, [20, 1], [90, 200], 50),       # a page size that TMA does not take
    (12, 4, 64, 64, 64, [2, 5, 9], [2, 700, 90], 128),
]


@pytest.mark.parametrize("generic", [False, True])
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shape", BIAS_SHAPES, ids=lambda s: f"H{s[0]}d{s[2]}v{s[3]}ps{s[4]}w{s[7]}")
def test_attention_with_a_distance_bias(ops, dtype, shape, generic):
    if generic and (dtype == torch.float32 or shape[2] != shape[3]):
        pytest.skip("these run the generic kernel anyway")
    Hq, G, hd, vd, ps, q_lens, kv_lens, window = shape
    got, want = _attention_case(ops, dtype, Hq, G, hd, vd, ps, q_lens, kv_lens, window, biased=True, generic=generic,
                                gate=hd != vd)
    assert (got - want).abs().max() <= (2e-5 if dtype == torch.float32 else 2.5e-2)


POOL_SHAPES = [
    # Hq, G, hd, vd, page, q_lens, kv_lens, window, pool
    (3, 3, 16, 16, 4, [5, 1, 2], [5, 9, 30], 7, 2),
    (4, 2, 20, 36, 5, [3, 11, 1], [17, 60, 64], 9, 4),
    (2, 1, 24, 24, 4, [7, 1, 20], [60, 50, 90], 3, 8),                # a window shorter than its blocks
    (8, 2, 64, 64, 16, [1, 1, 1, 1], [300, 17, 64, 129], 64, 1),
    (8, 2, 64, 64, 16, [70, 2, 1], [200, 5, 333], 33, 3),
    (16, 2, 128, 128, 16, [130, 1, 3, 64], [130, 555, 40, 600], 96, 16),
    (6, 3, 128, 128, 8, [1, 1], [1300, 31], 100, 5),
    (4, 1, 128, 128, 32, [300], [900], 64, 4),
    (4, 4, 128, 128, 64, [260, 1, 4], [520, 2000, 700], 16, 2),       # many more blocks than tokens
    (4, 2, 256, 256, 16, [40, 1], [90, 200], 50, 4),
    (8, 8, 128, 128, 5, [20, 1], [90, 200], 50, 4),
    (12, 4, 64, 64, 64, [2, 5, 9], [2, 700, 90], 40, 7),
    (2, 2, 128, 128, 16, [16, 9], [40, 33], 2, 1),                    # blocks of the step itself are seen by its tokens
]


@pytest.mark.parametrize("generic", [False, True])
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("shape", POOL_SHAPES, ids=lambda s: f"H{s[0]}d{s[2]}v{s[3]}ps{s[4]}w{s[7]}p{s[8]}")
def test_attention_with_pooled_blocks_before_the_window(ops, dtype, shape, generic):
    if generic and (dtype == torch.float32 or shape[2] != shape[3]):
        pytest.skip("these run the generic kernel anyway")
    Hq, G, hd, vd, ps, q_lens, kv_lens, window, pool = shape
    got, want = _attention_case(ops, dtype, Hq, G, hd, vd, ps, q_lens, kv_lens, window, pool=pool, generic=generic)
    assert (got - want).abs().max() <= (2e-5 if dtype == torch.float32 else 2.5e-2)


@pytest.mark.parametrize("dtype,hd", [(torch.float32, 32), (torch.bfloat16, 32), (torch.bfloat16, 64), (torch.bfloat16, 128)])
@pytest.mark.parametrize("q_lens", [[1, 1], [3, 70], [1, 300]])
def test_one_key_decides_inside_the_window_and_through_its_block_only_once_that_is_seen(ops, dtype, hd, q_lens):
    """One query's score with one token (or with a whole block of 8) stands out.  In a window of 40, the token takes the
    softmax up to 39 positions back; from 40 back it leaves no trace until its block lies wholly before the window, and
    then the block's mean takes it."""
    L, window, pool, Hq = 640, 40, 8, 4
    t = sum(q_lens) - 1
    tol = 1e-4 if dtype == torch.float32 else 4e-2
    for back in (0, 1, 15, 16, 38, 39, 40, 41, 46, 47, 48, 55, 56, 200, 639):
        def stand_out(q, rows, qo):
            q[t, 2] = 0
            q[t, 2, hd - 1] = 8.0
            rows[1][:, :, hd - 1] = rows[1][:, :, hd - 1].clamp(-1, 1) * 0.1
            where = L - 1 - back
            lo = where // pool * pool
            seen_as_block = lo + pool - 1 <= L - 1 - window
            hit = slice(lo, lo + pool) if seen_as_block else slice(where, where + 1)
            rows[1][hit, :, hd - 1] = 40.0
        got, want = _attention_case(ops, dtype, Hq, 2, hd, hd, 16, q_lens, [90, L], window, pool=pool, change=stand_out,
                                    seed=back, scale=0.5)
        assert (got - want).abs().max() <= tol, back
        got0, _ = _attention_case(ops, dtype, Hq, 2, hd, hd, 16, q_lens, [90, L], window, pool=pool, seed=back, scale=0.5,
                                  want_plain=False, change=lambda q, r, qo: stand_out(q, [r[0], r[1].clone()], qo) or
                                  r[1][:, :, hd - 1].clamp_(-1, 1).mul_(0.1))
        gap = (L - 1 - back) // pool * pool + pool - 1 > L - 1 - window      # its block is not seen yet
        moved = (got[t, 2] - got0[t, 2]).abs().max()
        assert (moved == 0) == (back >= window and gap), (back, float(moved))


@pytest.mark.parametrize("dtype,hd", [(torch.float32, 32), (torch.bfloat16, 64), (torch.bfloat16, 128)])
def test_the_bias_decides_between_equal_keys(ops, dtype, hd):
    """With equal scores the weights are those of the distances alone: for the head of slope 1/2 half a unit per position;
    and a key far back whose score outweighs its distance takes the softmax."""
    L = 500
    for q_lens in ([1], [2], [40]):
        for back, lift in ((3, 0.0), (400, 0.0), (400, 230.0), (499, 300.0)):
            def same(q, rows, qo):
                q[-1] = 0
                q[-1, :, 0] = 1.0
                rows[0][:, :, 0] = 0
                rows[0][L - 1 - back, :, 0] = lift
            got, want = _attention_case(ops, dtype, 16, 2, hd, hd, 16, q_lens, [L], None, biased=True, scale=1.0, change=same,
                                        seed=back)
            assert (got - want).abs().max() <= (1e-4 if dtype == torch.float32 else 4e-2), (q_lens, back, lift)


# ---------------------------------------------------------------------------- retention

def _step_ctx(lens, slots, starts):
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32, device=DEV)
    pos = torch.cat([torch.arange(s, s + k) for s, k in zip(starts, lens)])
    return SimpleNamespace(qo_indptr=i32([0] + list(np.cumsum(lens))), state_slots=i32(slots), positions=i32(pos),
                           n_entries=len(lens), n_tokens=sum(lens), max_q_len=max(lens))


STEPS = [dict(a=5, b=1, c=2), dict(a=1, c=1), dict(b=11, a=2, c=1), dict(c=1), dict(c=9, a=1), dict(b=2, c=37), dict(a=1, b=1)]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("Hh,dk,dv,rot", [(3, 8, 12, 8), (2, 20, 7, 6), (1, 6, 40, 2), (4, 64, 64, 64), (2, 128, 33, 32), (1, 256, 16, 0),
                                          (8, 32, 128, 32)])
def test_retention_over_portions_and_reused_slots(ops, dtype, Hh, dk, dv, rot):
    """Three requests in portions of unequal sizes (one left out of some steps, some steps of one token each, where the
    rotation runs inside the recurrence) against the plain mixer over each whole sequence; then a cleared slot again."""
    from batchspec_b200.parts.base import MIXERS, PartSpec, Runtime, build_part
    g = _gen(dk + dv)
    d, eps = 64, 1e-5
    decay = [0.5, 0.9, 0.99, 1.0, 0.999, 0.7, 0.8, 0.95][:Hh]
    pos = PartSpec("rope", dict(head_dim=dk, theta=77.0, rotary_dim=rot, interleaved=False)) if rot else PartSpec("none")
    part = build_part(MIXERS, PartSpec("retention", dict(dim=d, n_heads=Hh, head_dim=dk, v_dim=dv, decay=decay, position=pos, eps=eps)),
                      Runtime(dtype, torch.device(DEV)))
    w = {k: (torch.randn(*ps.shape, device=DEV, generator=g) * 0.25).to(dtype) for k, ps in part.param_specs().items()}
    part.bind(w)
    m = dict(heads=Hh, dim=dk, vdim=dv, decay=decay, rot=dict(base=77.0, dims=rot))
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
    cpu = {k: v.cpu() for k, v in w.items()}
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    for r in slots:
        want = P.retention(xs[r].double().cpu(), cpu, m, eps)
        assert (torch.cat(got[r]).double().cpu() - want).abs().max() <= tol * (1 + want.abs().max()), r
    assert not state[1].any() and not state[3].any()             # the slots of no request were never written
    state[2].zero_()
    again = part.forward(xs["c"][:7].contiguous(), _step_ctx([7], [2], [0]), SimpleNamespace(state=state))
    want = P.retention(xs["c"][:7].double().cpu(), cpu, m, eps)
    assert (again.double().cpu() - want).abs().max() <= tol * (1 + want.abs().max())


def test_retention_keeps_its_digits_over_a_long_prompt(ops):
    """3,000 tokens with decays close to one (numbers that float32 holds exactly), in portions and then one by one,
    against the plain recurrence."""
    g = _gen(1)
    Hh, dk, dv, T = 2, 16, 8, 3000
    decays = [1 - 2.0 ** -12, 1 - 2.0 ** -11]
    decay = torch.tensor(decays, device=DEV)
    proj = torch.randn(T, Hh * (2 * dk + dv), device=DEV, generator=g)
    state = torch.zeros(1, Hh * dk * dv, device=DEV)
    got, at = [], 0
    for k in [1500, 700, 777] + [1] * 23:
        got.append(ops.lightning_recurrence(proj[at:at + k], 0, Hh * dk, 2 * Hh * dk, decay, state, _step_ctx([k], [0], [at]), Hh, dk, dv,
                                            activation=None, k_scale=dk ** -0.5))
        at += k
    x = proj.double().cpu()
    want = P.decaying_state(x[:, :Hh * dk].view(T, Hh, dk), x[:, Hh * dk:2 * Hh * dk].view(T, Hh, dk) * dk ** -0.5,
                            x[:, 2 * Hh * dk:].view(T, Hh, dv), decays).reshape(T, -1)
    assert (torch.cat(got).double().cpu() - want).abs().max() <= 2e-5 * want.abs().max()


# ---------------------------------------------------------------------------- routed experts

@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n,d,ff,E,top,groups,shared", [
    (7, 48, 16, 6, 2, (3, 2), 24), (1, 100, 20, 7, 7, (1, 1), 0), (40, 64, 32, 1, 1, (1, 1), 8), (300, 320, 96, 12, 3, (4, 1), 64),
    (3, 320, 64, 8, 2, (2, 1), 96), (70, 64, 128, 16, 3, (8, 2), 200), (600, 96, 40, 9, 2, (3, 3), 20), (9, 256, 96, 4, 4, (2, 2), 0),
    (2000, 128, 64, 8, 4, (2, 1), 128), (5, 102, 18, 6, 1, (6, 1), 30)])
def test_softmax_router_with_groups_and_a_shared_expert(ops, dtype, n, d, ff, E, top, groups, shared):
    """The chosen experts, their weights and the summed outputs, on rows whose choices are not close (spread logits)."""
    from batchspec_b200.parts.base import FEED_FORWARDS, PartSpec, Runtime, build_part
    g = _gen(n + E)
    part = build_part(FEED_FORWARDS, PartSpec("routed_glu", dict(
        dim=d, intermediate=ff, n_experts=E, top=top, bias=False, scores="softmax", n_groups=groups[0], keep_groups=groups[1],
        shared=shared)), Runtime(dtype, torch.device(DEV)))
    w = {}
    for name, ps in part.param_specs().items():
        w[name] = (torch.randn(*ps.shape, device=DEV, generator=g) * (1.5 / math.sqrt(d) if name == "router" else 0.3)).to(dtype)
    part.bind(w)
    x = torch.randn(n, d, device=DEV, generator=g).to(dtype)
    ids, wts = ops.moe_route(x, part.w_router, None, groups[0], groups[1], top, 1.0, softmax=True, group_max=True, renormalise=True)
    xd, router = x.double().cpu(), w["router"].cpu()
    idx, wt = P.route(xd, router, top, *groups)
    z = xd @ router.double().T
    # rows whose groups and chosen experts are clear of the next ones
    gz = torch.sort(z.view(n, groups[0], -1).amax(-1), dim=-1, descending=True).values
    clear = torch.ones(n, dtype=torch.bool) if groups[1] == groups[0] else gz[:, groups[1] - 1] - gz[:, groups[1]] > 0.05
    pool_size = groups[1] * (E // groups[0])
    for t in range(n):
        kept = {e // (E // groups[0]) for e in idx[t].tolist()}
        if top < pool_size:
            best = torch.argsort(z[t].view(groups[0], -1).amax(-1), descending=True)[:groups[1]].tolist()
            inside = torch.sort(z[t].view(groups[0], -1)[best].flatten(), descending=True).values
            clear[t] &= bool(inside[top - 1] - inside[top] > 0.05)
        assert len(kept) <= groups[1]
    assert clear.float().mean() > 0.5
    assert torch.equal(torch.sort(ids.cpu().long()[clear], dim=-1).values, torch.sort(idx[clear], dim=-1).values)
    assert (wts.sum(-1) - 1).abs().max() <= 1e-5
    order, mine = torch.argsort(ids.cpu().long(), dim=-1), torch.argsort(idx, dim=-1)
    assert (wts.double().cpu().gather(1, order) - wt.gather(1, mine))[clear].abs().max() <= (1e-5 if dtype == torch.float32 else 1e-2)
    named = {"router": router}
    for e in range(E):
        named.update({f"e{e}.{k}": w[f"{k}{e}"].cpu() for k in ("gate", "up", "down")})
    if shared:
        named.update({f"shared.{k}": w[f"shared.{k}"].cpu() for k in ("gate", "up", "down")})
    f = dict(router=dict(experts=E, top=top, groups=dict(count=groups[0], keep=groups[1])), shared=dict(ff=shared) if shared else None)
    want = P.routed_ff(xd, named, f)
    err = (part.forward(x, None).double().cpu() - want).abs().amax(dim=-1) / want.abs().max()
    assert err[clear].max() <= (2e-5 if dtype == torch.float32 else 3e-2)


# ---------------------------------------------------------------------------- whole mixers

def _one_mixer_against_plain(cfg, dtype, page, plain, lens):
    """Build the model's only mixer with random tensors and run it through the step context of a real engine: a prompt
    and then five tokens one by one."""
    from batchspec_b200.engine import StepEntry
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    with tempfile.TemporaryDirectory() as tmp:
        folder = H.make_folder(tmp, cfg, 5, dtype=stored, std=0.25)
        _, w = P.read_model_folder(folder)
        eng = _engine(folder, dtype, page, 96, max_requests=2)
        mixer = eng.model.blocks[0].mixer
        seen = {"x": [], "y": []}
        branches, forward = getattr(mixer, "forward_branches", None), mixer.forward

        def spy(x, ctx, cache):
            seen["x"].append(x.detach().double().cpu())
            if branches is not None:                       # the pair, and its sum as the mixer itself forms it
                pair = branches(x, ctx, cache)
                y = torch.empty_like(x)
                from batchspec_b200.kernels import ops
                ops.branch_join(None, pair, out=y)
                seen["y"].append(y.double().cpu())
                return pair
            y = forward(x, ctx, cache)
            seen["y"].append(y.detach().double().cpu())
            return y
        if branches is not None:
            type(mixer).forward_branches, keep = property(lambda self: spy if self is mixer else self._normed_pair), type(mixer).forward_branches
        else:
            mixer.forward = spy
        try:
            for rid, n in zip("ab", lens):
                toks = H.random_tokens(n, cfg["vocab"], n)
                eng.admit(rid)
                eng.step([StepEntry(rid, toks[:n - 5], [])])
                for tok in toks[n - 5:]:
                    eng.step([StepEntry(rid, [tok], [])])
                xs, ys = torch.cat(seen["x"]), torch.cat(seen["y"])
                seen["x"].clear(), seen["y"].clear()
                sub = {k[len("l0.mix."):]: v for k, v in w.items() if k.startswith("l0.mix.")}
                want = plain(xs, sub, cfg["layers"][0]["mixer"])
                assert (ys - want).abs().max() <= (5e-5 if dtype == "float32" else 4e-2) * want.abs().max()
        finally:
            if branches is not None:
                type(mixer).forward_branches = keep


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 2, 12, 20, 10), (8, 1, 64, 64, 40), (3, 3, 10, 4, 1), (8, 2, 128, 128, 70)],
                         ids=lambda s: f"H{s[0]}G{s[1]}d{s[2]}v{s[3]}w{s[4]}")
def test_attention_mixer_with_bias_window_and_gate(ops, dtype, sizes):
    Hq, G, hd, vd, window = sizes
    cfg = _config(50, 96, 1e-5, [_attn(Hq, G, hd, vd, 1.0 / math.sqrt(hd), window)])
    _one_mixer_against_plain(cfg, dtype, 8, P.biased_attention, lens=(37, 150))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("left,right", [
    ((4, 2, 12, 20, 0.3, 9, 4, 777.0, 8), (3, 8, 12, [0.5, 0.9, 0.99], 50.0, 8)),
    ((8, 1, 64, 64, 0.125, 40, 3, 1e4, 32), (2, 32, 16, [0.97, 0.9], 1e3, 16)),
    ((8, 2, 128, 128, 0.09, 30, 2, 1e5, 128), (4, 64, 32, [0.8, 0.9, 0.95, 0.999], 1e4, 64)),
    ((3, 3, 10, 4, 0.4, 6, None, 20.0, 10), (1, 6, 5, [0.4], 20.0, 2))], ids=["small", "d64", "d128", "no_pool"])
def test_parallel_mixer_with_a_norm_on_each_output(ops, dtype, left, right):
    cfg = _config(50, 96, 1e-5, [_par(left, right)])
    _one_mixer_against_plain(cfg, dtype, 8, lambda h, w, m: P.parallel_mixer(h, w, m, 1e-5), lens=(33, 150))


@pytest.mark.parametrize("kind", ["bias", "pool"])
def test_a_sharp_softmax_over_hundreds_of_keys(ops, kind):
    """A scale far above 1 / sqrt(size): nearly every softmax is decided by one key or block, which a kernel that skipped
    or misplaced it would lose.  float32, prompt and decoding."""
    if kind == "bias":
        cfg = _config(50, 96, 1e-5, [_attn(8, 2, 32, 24, 6.0, 250)])
        _one_mixer_against_plain(cfg, "float32", 8, P.biased_attention, lens=(9, 400))
    else:
        cfg = _config(50, 96, 1e-5, [_par((4, 2, 32, 24, 4.0, 30, 2, 500.0, 16), (1, 8, 8, [0.9], 50.0, 8))])
        _one_mixer_against_plain(cfg, "float32", 8, lambda h, w, m: P.parallel_mixer(h, w, m, 1e-5), lens=(9, 400))


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


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_token_outside_the_window_is_unseen_and_the_first_inside_is_seen(tmp_path, dtype):
    """One attention layer, a window of 12: changing a token that the window hides from the positions 36..47 changes none
    of their logits, bit for bit; changing the first token they see changes them."""
    cfg, seed, page = CONFIGS["WINDOW"]
    folder = _folder(tmp_path, "WINDOW", dtype, std=0.3)
    base = H.random_tokens(48, cfg["vocab"], 2)
    eng = _engine(folder, dtype, page, 12)
    cases = ((24, [], range(36, 48)), (25, [36], range(37, 48)), (35, range(36, 47), [47]), (0, [], range(36, 48)))
    for make in MAKERS:
        ref = H.run_steps_in_process(eng, make(base))
        _compare(ref, folder, {"e": base}, dtype)
        for where, moved, same in cases:
            toks = list(base)
            toks[where] = (toks[where] + 1) % cfg["vocab"]
            got = H.run_steps_in_process(eng, make(toks))
            assert all(np.array_equal(got[("e", p)], ref[("e", p)]) for p in same), where
            # (a bfloat16 logit may stay the same when a far key's weight is small: the sum over the edge has to move)
            assert all(not np.array_equal(got[("e", p)], ref[("e", p)]) for p in list(moved)[:1] or ()), where


@pytest.mark.parametrize("make", range(3))
def test_a_block_is_unseen_until_the_window_has_passed_it_wholly(tmp_path, make):
    """One pooled attention layer (window 9, blocks of 4; the retention beside it silenced): after a change of one token,
    exactly the positions that see it (in the window, or through its block) have other logits, in every schedule."""
    cfg, seed, page = CONFIGS["SEEN"]
    folder = _folder(tmp_path, "SEEN", "float32", std=0.3)
    base = H.random_tokens(48, cfg["vocab"], 2)
    eng = _engine(folder, "float32", page, 16)
    eng.model.blocks[0].mixer.w_right.zero_()
    ref = H.run_steps_in_process(eng, MAKERS[make](base))
    for where in (0, 1, 3, 4, 7, 8, 14, 15, 16, 30):
        toks = list(base)
        toks[where] = (toks[where] + 1) % cfg["vocab"]
        got = H.run_steps_in_process(eng, MAKERS[make](toks))
        last = where // 4 * 4 + 3
        for p in range(48):
            sees = 0 <= p - where < 9 or last <= p - 9
            assert np.array_equal(got[("e", p)], ref[("e", p)]) == (not sees), (where, p)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_moves_the_logits_through_blocks_and_state(tmp_path, dtype):
    """Changing ONE token far back changes the last position's logits in the oracle although every window has passed it.
    The engine follows, decoded alone and as the end of a portion."""
    cfg, seed, page = CONFIGS["A"]
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    folder = H.make_folder(tmp_path / "far", cfg, 21, dtype=stored, std=0.15)
    base = H.random_tokens(260, cfg["vocab"], 8)
    eng = _engine(folder, dtype, page, 70)
    ref0 = _oracle(folder, base)[-1]
    moved, over = [], 0
    for where in (0, 3, 4, 127, 128, 200):
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
    folder = H.make_folder(tmp_path / "gen", cfg, 31, dtype=torch.float32, std=0.2)
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
    those of steps launched kernel by kernel, over block ends and window edges."""
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
