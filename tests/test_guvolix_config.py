"""The Guvolix design without a GPU: its configuration reader, its model description against the tensors a folder holds,
what its runs ask of the cache manager, the manager's pages of first tokens that stay, and the plain implementation's own
mechanisms against closed forms."""
import math

import pytest
import torch

import plain_guvolix as P
from batchspec_b200.cache.manager import CacheManager, OutOfPages
from batchspec_b200.config import ConfigError, config_from_json_dict
from batchspec_b200.models import get_model
from batchspec_b200.models.decoder import CacheNeed
from batchspec_b200.parts.base import CacheSpec, Runtime


def moe(experts=6, top=2, identity=3, shared=24):
    f = dict(kind="moe", expert=dict(ff=16), router=dict(experts=experts, top=top))
    if identity:
        f["router"]["identity"] = identity
    if shared:
        f["shared"] = dict(ff=shared)
    return f


def left(window=10, keep=3, scaling=None):
    return dict(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.25, mask=dict(size=window, keep_first=keep),
                rot=dict(base=500.0, dims=6, scaling=scaling or dict(factor=2.0)))


def ssd(mlp=None, **kw):
    return dict(type="parallel", mixer=dict(left=left(**kw), right=dict(heads=6, vdim=5, state=8, groups=3, conv=3, norm_groups=2)),
                mlp=mlp)


def mem(mlp=None, **kw):
    return dict(type="parallel_2", mlp=mlp, mixer=dict(left=left(**kw), right=dict(heads=3, dim=10, vdim=6, gate_cap=4.0),
                                                       left_scale=0.8, right_scale=1.3))


LLAMA3 = dict(factor=4.0, low=1.0, high=4.0, original=64)


def config(layers, **kw):
    d = dict(architecture="Guvolix", vocab=200, width=48, norm=dict(eps=1e-5), embedding=dict(scale=0.7), layers=layers)
    d.update(kw)
    return d


def model(d):
    return get_model(config_from_json_dict(d), Runtime(torch.float32, torch.device("cpu")))


def test_reader_takes_every_size_from_the_file_and_round_trips():
    d = config([ssd(moe()), mem(dict(kind="dense", ff=40), scaling=LLAMA3), ssd()])
    cfg = config_from_json_dict(d)
    assert (cfg.vocab_size, cfg.width, cfg.norm_eps, cfg.embed_scale, len(cfg.layers)) == (200, 48, 1e-5, 0.7, 3)
    assert not cfg.unread_keys and config_from_json_dict(cfg.to_json_dict()) == cfg
    d2 = config([ssd(moe()), mem()], foo=1)
    d2["layers"][0]["mixer"]["left"]["mask"]["bar"] = 2
    d2["layers"][0]["mixer"]["right"]["baz"] = 2
    d2["layers"][1]["mixer"]["left"]["rot"]["scaling"]["qux"] = 2
    assert set(config_from_json_dict(d2).unread_keys) == {"foo", "layers[0].mixer.left.mask.bar", "layers[0].mixer.right.baz",
                                                          "layers[1].mixer.left.rot.scaling.qux"}


@pytest.mark.parametrize("break_it", [
    lambda d: d["layers"][0].update(type="attention"), lambda d: d["layers"][0]["mixer"]["left"]["mask"].update(size=0),
    lambda d: d["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3),
    lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=5), lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=14),
    lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0), lambda d: d["layers"][0]["mixer"]["right"].update(groups=4),
    lambda d: d["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(low=4.0), lambda d: d["layers"][0]["mixer"]["right"].update(norm_groups=7),
    lambda d: d["layers"][1]["mixer"]["right"].update(gate_cap=0.0), lambda d: d["layers"][1]["mixer"].pop("left_scale"),
    lambda d: d["layers"][0]["mlp"].update(kind="glu"), lambda d: d["layers"][0]["mlp"]["router"].update(top=10),
    lambda d: d["layers"][0]["mlp"]["router"].update(identity=-1), lambda d: d["layers"][0]["mlp"]["shared"].update(ff=0),
    lambda d: d["norm"].update(eps=0.0), lambda d: d.update(layers=[]), lambda d: d["layers"][1]["mixer"].pop("right"),
])
def test_reader_refuses_what_cannot_be_run(break_it):
    d = config([ssd(moe()), mem(scaling=dict(LLAMA3))])
    config_from_json_dict(d)
    break_it(d)
    with pytest.raises(ConfigError):
        config_from_json_dict(d)


def test_tensor_names_block_kinds_and_needs():
    m = model(config([ssd(moe()), mem(dict(kind="dense", ff=40), keep=0), ssd(), mem(moe(identity=0, shared=0), window=9)]))
    specs = m.param_specs()
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.mix.left.sink", "l0.mix.left.out", "l0.mix.right.out", "l0.mix.right.conv.b",
            "l0.mlp.e5.down", "l0.mlp.shared.sg", "l1.mix.right.i.b", "l1.mix.right.norm", "l1.mlp.up", "l3.mlp.correction"} <= set(specs)
    assert not any(n.endswith("norm2") or n.startswith("l2.mlp") or n.startswith("l3.mlp.shared") or n.startswith("l1.mix.left.out")
                   for n in specs)
    shape = lambda n: tuple(specs[n].shape)
    assert shape("l0.mlp.router") == (9, 48) and shape("l0.mlp.correction") == (9,) and shape("l3.mlp.router") == (6, 48)
    assert shape("l0.mix.right.in") == (2 * 30 + 2 * 3 * 8 + 6, 48) and shape("l0.mix.right.conv") == (78, 3)
    assert shape("l0.mlp.shared.sg") == (1, 48) and shape("l1.mix.right.norm") == (18,) and shape("l1.mix.left.g") == (80, 48)
    assert [b.kind for b in m.blocks] == ["parallel_prenorm", "parallel_prenorm", "parallel_prenorm_mixer", "parallel_prenorm"]
    assert m.spec.lm_head_name == "head" and m.spec.embed_scale == 0.7 and m.graph_safe
    needs = m.cache_needs()
    assert [(n.cache.policy, n.cache.window, n.cache.keep) for n in needs] == [("window", 10, 3), ("window", 10, 0), ("window", 10, 3),
                                                                               ("window", 9, 3)]
    up4 = lambda n: -(-n // 4) * 4
    assert [n.state.shape for n in needs] == [(up4(240 + 2 * 78),), (up4(3 * 7 * 10 + 18),)] * 2
    assert len(CacheManager(needs, 4, 20, 3, torch.float32, "cpu").groups) == 3


def test_pages_of_kept_first_tokens_stay_and_the_window_moves_on():
    need = CacheNeed(CacheSpec("window", (2, 4), 10, keep=6), None, None)
    c = CacheManager([need], 4, 9, 2, torch.float32, "cpu", allocate=False)
    assert c.groups[0].kept_pages == 2
    c.admit("a")
    for k in [3, 1, 5, 7, 1, 1, 2, 30 - 20]:
        c.reserve("a", k)
        c.commit("a", k)
        c.check_invariants()
        rc = c.requests["a"]
        first = max(0, rc.length - 10 + 1) // 4
        assert [p >= 0 for p in rc.tables[0]] == [i < 2 or i >= first for i in range(len(rc.tables[0]))]
    assert c.groups[0].pool.num_held == 2 + 3 and c.peak_pages(400, 1) == [2 + 4]
    c.admit("b")
    c.reserve("b", 16)
    with pytest.raises(OutOfPages):
        c.reserve("a", 8)
    c.release("a")
    c.release("b")
    c.check_invariants()
    assert c.groups[0].pool.num_free == 9


def test_peak_pages_bound_what_a_request_holds():
    for ps, window, keep in ((4, 10, 6), (16, 7, 1), (1, 3, 5), (8, 30, 0), (5, 12, 40)):
        for portion in (1, 3, 17):
            c = CacheManager([CacheNeed(CacheSpec("window", (1, 4), window, keep=keep), None, None)], ps, 200, 1, torch.float32, "cpu",
                             allocate=False)
            c.admit("a")
            worst = 0
            for n in range(0, 150, portion):
                c.reserve("a", portion)
                worst = max(worst, c.groups[0].pool.num_held)
                c.commit("a", portion)
            assert worst <= c.peak_pages(n + portion, portion)[0]


def test_plain_mechanisms_against_closed_forms():
    see = P.visible(9, 3, 2)
    assert see[8].tolist() == [True, True] + [False] * 4 + [True] * 3 and see[2].tolist() == [True] * 3 + [False] * 6
    # equal scores of zero and a sink of log 2: the denominator is the number of visible keys plus two
    q, k, v = torch.zeros(4, 2, 3).double(), torch.zeros(4, 1, 3).double(), torch.ones(4, 1, 5).double()
    out = P.attend(q, k, v, 1.0, 3, 0, torch.tensor([math.log(2.0), -1e9]))
    assert torch.allclose(out[:, 0, 0], torch.tensor([1 / 3, 2 / 4, 3 / 5, 3 / 5], dtype=P.F)) and torch.allclose(out[:, 1], torch.ones(4, 5).double())
    # rates: short waves keep theirs, long ones are divided
    rot = dict(base=1e4, dims=8, scaling=dict(LLAMA3))
    plain = [1e4 ** (-2 * i / 8) for i in range(4)]
    assert P.angle_rates(rot)[0] == plain[0] and P.angle_rates(rot)[3] == plain[3] / 4.0
    assert P.angle_rates(dict(rot, scaling=dict(factor=2.0))) == [f / 2.0 for f in plain]
    # a constant input through the scalar decay: a geometric sum
    one = torch.ones(5, 1, 1).double()
    y = P.scalar_decay_state(one, one, one, one[:, :, 0], torch.tensor([0.0]), torch.tensor([2.0]))[:, 0, 0]
    assert torch.allclose(y, torch.tensor([2.0 + sum(math.exp(-j) for j in range(t + 1)) for t in range(5)], dtype=P.F))
    # gates that never forget and never exceed the first maximum: sums, divided by n . q
    z = torch.zeros(4, 1).double()
    o = P.matrix_memory(one[:4], one[:4], torch.arange(4).double().view(4, 1, 1), z, z)[:, 0, 0]
    assert torch.allclose(o, torch.tensor([0.0, 0.5, 1.0, 1.5], dtype=P.F), atol=1e-5)
    # an identity expert's row is the input
    h, f = torch.randn(3, 4).double(), dict(router=dict(experts=1, top=1))
    w = {"router": torch.zeros(2, 4), "correction": torch.tensor([0.0, 9.0])}
    assert torch.allclose(P.routed_ff(h, w, f), h)
    x = torch.arange(6).double().view(6, 1)
    assert P.causal_conv(x, torch.tensor([[1.0, 10.0]]), torch.tensor([0.5])).flatten().tolist() == [0.5, 10.5, 21.5, 32.5, 43.5, 54.5]
