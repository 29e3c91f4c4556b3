"""The Podizen design without a GPU: its configuration reader, its model description against the tensors a folder holds,
what its runs ask of the cache manager, the manager's groups of pooled blocks, and the plain implementation's own
mechanisms against closed forms."""
import math

import pytest
import torch

import plain_podizen as P
from batchspec_b200.cache.manager import CacheManager, OutOfPages
from batchspec_b200.config import ConfigError, config_from_json_dict
from batchspec_b200.models import get_model
from batchspec_b200.models.decoder import CacheNeed
from batchspec_b200.parts.base import CacheSpec, Runtime


def moe(ff=16, experts=6, top=2, count=3, keep=2, shared=24):
    f = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if count:
        f["router"]["groups"] = dict(count=count, keep=keep)
    if shared:
        f["shared"] = dict(ff=shared)
    return f


def attention(mlp=None, window=10):
    return dict(type="attention", mixer=dict(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.25, mask=dict(size=window)), mlp=mlp)


def parallel(mlp=None, window=9, pool=4):
    left = dict(heads=4, kv_heads=2, dim=10, vdim=6, scale=0.3, mask=dict(size=window, pool=pool), rot=dict(base=500.0, dims=6))
    right = dict(heads=3, dim=8, vdim=12, decay=[0.5, 0.9, 0.99], rot=dict(base=900.0, dims=4))
    return dict(type="parallel", mixer=dict(left=left, right=right), mlp=mlp)


def config(layers, **kw):
    d = dict(architecture="Podizen", vocab=200, width=48, norm=dict(eps=1e-5), layers=layers)
    d.update(kw)
    return d


def model(d):
    return get_model(config_from_json_dict(d), Runtime(torch.float32, torch.device("cpu")))


def test_reader_takes_every_size_from_the_file_and_round_trips():
    d = config([attention(moe()), parallel(moe(count=0, shared=0)), attention()])
    cfg = config_from_json_dict(d)
    assert (cfg.vocab_size, cfg.width, cfg.norm_eps, len(cfg.layers)) == (200, 48, 1e-5, 3) and not cfg.unread_keys
    assert config_from_json_dict(cfg.to_json_dict()) == cfg
    d2 = config([parallel(moe())], foo=1)
    d2["layers"][0]["mixer"]["left"]["mask"]["bar"] = 2
    d2["layers"][0]["mlp"]["shared"]["baz"] = 2
    assert set(config_from_json_dict(d2).unread_keys) == {"foo", "layers[0].mixer.left.mask.bar", "layers[0].mlp.shared.baz"}


@pytest.mark.parametrize("break_it", [
    lambda d: d["layers"][0].update(type="conv"), lambda d: d["layers"][0]["mixer"]["mask"].update(size=0),
    lambda d: d["layers"][0]["mixer"].update(heads=4, kv_heads=3), lambda d: d["layers"][1]["mixer"]["left"]["mask"].update(pool=0),
    lambda d: d["layers"][1]["mixer"]["left"]["rot"].update(dims=5), lambda d: d["layers"][1]["mixer"]["right"]["rot"].update(dims=10),
    lambda d: d["layers"][1]["mixer"]["right"].update(decay=[0.5]), lambda d: d["layers"][0]["mlp"].update(kind="dense"),
    lambda d: d["layers"][0]["mlp"]["router"].update(top=5), lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4),
    lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4), lambda d: d["layers"][0]["mlp"]["shared"].update(ff=0),
    lambda d: d["norm"].update(eps=0.0), lambda d: d.update(layers=[]), lambda d: d["layers"][1]["mixer"].pop("right"),
])
def test_reader_refuses_what_cannot_be_run(break_it):
    d = config([attention(moe()), parallel(moe())])
    config_from_json_dict(d)
    break_it(d)
    with pytest.raises(ConfigError):
        config_from_json_dict(d)


def test_tensor_names_block_kinds_and_needs():
    m = model(config([attention(moe()), parallel(), parallel(moe(count=0, shared=0), pool=None)]))
    specs = m.param_specs()
    assert {"embed", "final.norm", "l0.norm1b", "l0.norm2b", "l0.dwa", "l0.mix.g", "l0.mlp.e5.down", "l0.mlp.shared.up",
            "l1.mix.left.q.norm", "l1.mix.left.out", "l1.mix.right.out", "l1.mix.right.g", "l2.mlp.router"} <= set(specs)
    assert not any(n.startswith("l1.mlp") or n.startswith("l1.norm2") or n.startswith("l2.mlp.shared") or n == "head" for n in specs)
    assert [specs[f"l{i}.dwa"].shape for i in range(3)] == [(2,), (3,), (4,)]
    assert specs["l0.mix.g"].shape == (80, 48) and specs["l1.mix.right.g"].shape == (36, 48)
    assert [b.kind for b in m.blocks] == ["sandwich_averaged", "sandwich_mixer_averaged", "sandwich_averaged"]
    assert m.spec.depth_average and m.spec.lm_head_name is None and {"l1.norm2", "l1.norm2b"} == set(m.spec.ignore_names)
    needs = m.cache_needs()
    assert [(n.cache.policy, n.cache.window, n.cache.pool) for n in needs] == [("window", 10, 0), ("window", 9, 4), ("window", 9, 0)]
    assert [None if n.state is None else n.state.shape for n in needs] == [None, (288,), (288,)]
    cache = CacheManager(needs, 4, 20, 3, torch.float32, "cpu")
    assert [(g.spec.policy, g.stride) for g in cache.groups] == [("window", 1), ("window", 1), ("full", 4), ("window", 1)]
    assert cache.layer_caches[1].pooled_group == 2 and cache.layer_caches[1].pooled.shape[1:] == cache.layer_caches[1].kv.shape[1:]
    assert cache.layer_caches[0].pooled is None and cache.groups[2].pool.num_pages == 5 + 3


def test_presets_by_name_build():
    from batchspec_b200.config import get_config
    for name in ("tiny-podizen", "podizen-w2048"):
        cfg = get_config(name)
        m = get_model(cfg, Runtime(torch.bfloat16, torch.device("cpu")))
        assert cfg.architecture == "Podizen" and len(m.blocks) == len(cfg.layers)


# ---------------------------------------------------------------------------------- pooled blocks in the cache manager

def pooled_manager(window, pool, page=4, pages=40, requests=3):
    return CacheManager([CacheNeed(CacheSpec("window", (2,), window, pool=pool), None, None)], page, pages, requests,
                        torch.float32, "cpu", allocate=False)


@pytest.mark.parametrize("window,pool", [(9, 4), (16, 16), (3, 8), (5, 1), (1, 7)])
def test_tables_and_release_follow_the_length(window, pool):
    """After every commit a request has one entry per whole block, and the tokens it still holds are the window of the
    next position and the block that is not yet whole, to whole pages."""
    m = pooled_manager(window, pool)
    m.admit("a")
    for n in [1, 2, 5, 1, 1, 7, 3, 1, 16, 2, 1, 1, 1, 30]:
        need = m.pages_needed(m.length("a"), n)
        assert need == m.pages_missing("a", n)
        m.reserve("a", n)
        m.commit("a", n)
        L, rc = m.length("a"), m.requests["a"]
        assert len(rc.tables[0]) == -(-L // 4) and len(rc.tables[1]) == -(-(L // pool) // 4)
        keep = min(max(0, L - window + 1), L // pool * pool)
        assert rc.dead[0] == keep // 4 and rc.dead[1] == 0
        m.check_invariants()
    m.release("a")
    assert all(g.pool.num_held == 0 for g in m.groups)


@pytest.mark.parametrize("pool", [1, 3, 16])
def test_room_for_is_exact(pool):
    m = pooled_manager(6, pool)
    for length in (0, 1, 5, 16, 47, 48, 49):
        for free in ([3, 1], [10, 0], [10, 2], [0, 5]):
            n = m.room_for(length, free)
            fits = lambda k: all(a <= b for a, b in zip(m.pages_needed(length, k), free))
            assert n >= 0 and (n == 0 or fits(n)) and not fits(n + 1)


def test_pool_sizes_hold_the_tokens_asked_for():
    """Requests whose tokens, rounded up to 64, fill the pool exactly never run out of entries of pooled blocks."""
    for pool in (1, 4, 16, 100):
        m = CacheManager([CacheNeed(CacheSpec("window", (2,), 10, pool=pool), None, None)], 16, 256 // 16, 4, torch.float32,
                         "cpu", allocate=False)
        for rid, n in (("a", 64), ("b", 63), ("c", 64), ("d", 64)):
            m.admit(rid)
            m.reserve(rid, n)
            m.commit(rid, n)
        m.check_invariants()
    with pytest.raises(OutOfPages):
        m.reserve("a", 16 * 16 + 1)


def test_a_long_request_needs_few_pages_at_a_time():
    """Fed in portions of 4 tokens, a request never holds more pages of its window's group than ``peak_pages`` says."""
    for window, pool in ((9, 16), (16, 9), (1, 1)):
        peak = pooled_manager(window, pool).peak_pages(1000, 4)
        m = pooled_manager(window, pool, pages=peak)
        m.admit("a")
        for _ in range(250):
            m.reserve("a", 4)
            m.commit("a", 4)
        assert m.groups[1].pool.num_held == peak[1] == -(-(1000 // pool) // 4)


# ---------------------------------------------------------------------------------- the plain mechanisms

def test_plain_bias_window_and_slopes():
    assert P.bias_slopes(8)[:2] == [0.5, 0.25] and P.bias_slopes(3)[2] == 2.0 ** -8
    z = torch.zeros(4, 1, 2, dtype=P.F)
    v = torch.arange(4, dtype=P.F).reshape(4, 1, 1)
    out = P.attend(z, z, v, 1.0, window=2, slopes=[math.log(3.0)]).flatten()
    assert torch.allclose(out, torch.tensor([0.0, 0.75, 1.75, 2.75], dtype=P.F))        # weights 3/4 and 1/4


def test_plain_pooled_blocks_join_the_softmax_when_the_window_has_passed_them():
    T = 8
    z = torch.zeros(T, 1, 2, dtype=P.F)
    v = torch.arange(T, dtype=P.F).reshape(T, 1, 1)
    out = P.attend(z, z, v, 1.0, window=3, pool=2).flatten()
    # position 3: tokens 1..3 only (block 0 ends at 1 > 3 - 3); position 4: tokens 2..4 and block 0 (mean 0.5);
    # position 5: tokens 3..5 and block 0, token 2 is in neither; position 7: tokens 5..7, blocks 0 and 1
    assert torch.allclose(out[3:], torch.tensor([2.0, 9.5 / 4, 12.5 / 4, 18.0 / 5, 21.0 / 5], dtype=P.F))


def test_plain_retention_state_and_depth_average():
    q = k = torch.ones(3, 1, 1, dtype=P.F)
    v = torch.tensor([1.0, 10.0, 100.0], dtype=P.F).reshape(3, 1, 1)
    assert P.decaying_state(q, k, v, [0.5]).flatten().tolist() == [1.0, 10.5, 105.25]
    xs = [torch.full((2, 3), float(c), dtype=P.F) for c in (1, 10, 100)]
    assert P.depth_average(xs, torch.tensor([1.0, 0.5, -1.0])).unique().tolist() == [-94.0]


def test_plain_routing_keeps_groups_and_renormalises():
    h = torch.eye(1, dtype=P.F)
    router = torch.log(torch.tensor([[6.0], [1.0], [5.0], [4.0], [3.0], [3.5]]))       # softmax scores 6 : 1 : 5 : 4 : 3 : 3.5
    ids, wts = P.route(h, router, 2, 3, 2)
    assert ids[0].tolist() == [0, 2] and torch.allclose(wts[0], torch.tensor([6.0, 5.0], dtype=P.F) / 11)
    ids, wts = P.route(h, router, 2, 3, 1)            # one group of (6, 1): expert 1 is taken before 2
    assert ids[0].tolist() == [0, 1] and torch.allclose(wts[0], torch.tensor([6.0, 1.0], dtype=P.F) / 7)


def test_plain_norms_around_branches_reduce_to_their_parts():
    """Without a feed-forward and with an average that takes only the layer's own result, the model is embedding +
    norm(mixer(norm(embedding)))."""
    torch.manual_seed(0)
    d = config([attention()])
    w = {n: 0.3 * torch.randn(ps.shape) for n, ps in model(d).param_specs().items()}
    w["l0.dwa"] = torch.tensor([0.0, 1.0])
    toks = [3, 9, 150, 7, 7, 21]
    _, layers = P.forward(d, w, toks, True)
    x = P.f64(w["embed"])[toks]
    sub = {k[len("l0.mix."):]: v for k, v in w.items() if k.startswith("l0.mix.")}
    y = P.biased_attention(P.rms_norm(x, w["l0.norm1"], 1e-5), sub, d["layers"][0]["mixer"])
    assert torch.allclose(layers[0], x + P.rms_norm(y, w["l0.norm1b"], 1e-5))
