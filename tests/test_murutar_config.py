"""Murutar on the host: configuration, registry, the model as data, cache groups, tensor names, stacked
inputs, and the plain implementation's own window, sink, routing and recurrence."""

import json

import numpy as np
import pytest
import torch

import plain_murutar as plain

_MOE = {"kind": "moe", "router": {"experts": 8, "top": 2, "groups": {"count": 4, "keep": 2}}, "expert": {"ff": 24}}
_ATT = {"type": "attention", "mlp": {"kind": "dense", "ff": 56, "limit": 2.5},
        "mixer": {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 20, "scale": 0.3, "v_mix": True, "mask": {"size": 21},
                  "rot": {"base": 5000.0, "dims": 6}}}
_PLAIN = {"type": "attention", "mlp": None, "mixer": dict(_ATT["mixer"], v_mix=False, kv_heads=6, vdim=8)}
_LIGHT = {"type": "lightning", "mlp": _MOE, "mixer": {"heads": 3, "dim": 10, "vdim": 14, "decay": [0.5, 0.9, 0.99]}}
BASE = {"architecture": "Murutar", "vocab": 97, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
        "token_side": {"dim": 10}, "logit_softcap": 9.0, "layers": [_LIGHT, _PLAIN, _ATT, _ATT, _LIGHT]}


def build(document, dtype=torch.bfloat16):
    from ayaka_py_b200 import models, parts  # noqa: F401
    from ayaka_py_b200.models.model import Model
    from ayaka_py_b200.registry import architecture_for
    arch = architecture_for(document)
    config = arch.config_class.from_dict(document)
    return arch, config, Model(arch.build_spec(config), dtype, "meta")


def test_registry_and_round_trip():
    arch, config, _ = build(BASE)
    assert arch.name == "Murutar"
    again = arch.config_class.from_dict(config.to_dict())
    assert again.to_dict() == config.to_dict() and again.to_dict()["architecture"] == "Murutar"


def test_tensor_names_and_shapes():
    arch, config, model = build(BASE)
    rows = {r.source.name: tuple(r.decl.shape) for r in model.tensor_rows()}
    assert rows == plain.tensor_shapes(BASE)
    # the head is the embedding table itself; every layer reads the one side table
    assert [r.source.name for r in model.tensor_rows() if r.part is model.head] == ["embed"]
    assert sum(r.source.name == "side.embed" for r in model.tensor_rows()) == 5
    assert [b.side.col0 for b in model.blocks] == [0, 10, 20, 30, 40]
    # a layer without feed-forward has neither its tensors nor its norm and gate, and passes them over in a checkpoint
    assert "l1.norm2" not in rows and "l1.rg2.b" not in rows and "l2.rg2.b" in rows
    for name in ("l1.norm2", "l1.ls2", "l1.rg2", "l1.rg2.b", "l1.mlp.up"):
        assert arch.normalize_name(name, config) is None
    assert arch.normalize_name("l2.ls2", config) == "l2.ls2" and arch.normalize_name("l1.side.proj", config) == "l1.side.proj"


def test_cache_groups_and_constants():
    from ayaka_py_b200.parts import KVNeed, StateNeed
    _, _, model = build(BASE)
    assert {b.KIND for b in model.blocks} == {"gated_pre_norm"}
    needs = {g.need: g.layers for g in model.groups}
    assert needs == {StateNeed((3, 10, 14)): 2, KVNeed(kv_heads=6, head_dim=12, window=21, value_heads=6, value_dim=8): 1,
                     KVNeed(kv_heads=3, head_dim=12, window=21, value_heads=3, value_dim=20): 2}
    light, other, first, later = (model.blocks[i].mixer for i in range(4))
    assert (light.KIND, light.decay, light.eps, light.heads, light.dim, light.vdim) == ("lightning", [0.5, 0.9, 0.99], 1e-5, 3, 10, 14)
    assert (first.KIND, first.window, first.sink, first.scale, first.rotary.dims, first.rotary.base, first.rotary.halves) == \
        ("rotary_attention", 21, 0.0, 0.3, 6, 5000.0, True)
    # the first layer that mixes values is the first of those that say so, not the first attention
    assert [m.value_mix for m in (other, first, later)] == [None, "first", "blend"]
    moe, dense = model.blocks[0].ffn, model.blocks[2].ffn
    assert (moe.router, moe.groups, moe.keep, moe.top, moe.activation, moe.shared_inner, moe.route_scale) == ("softmax_groups", 4, 2, 2, "relu2", 0, 1.0)
    assert (dense.activation, dense.limit, dense.slope, dense.plus, dense.inner) == ("limited_glu", 2.5, 1.702, 1.0, 56)
    assert model.embedding.scale == 3.0 and model.head.scale == 1.0 and model.head.softcap == 9.0
    assert model.final_norm.KIND == "layernorm" and not model.final_norm.has_bias and not model.blocks[0].norm1.has_bias
    # no mask: every earlier key; no groups: one; no layer that mixes values
    doc = json.loads(json.dumps(BASE))
    for i in (2, 3):
        del doc["layers"][i]["mixer"]["mask"]
        del doc["layers"][i]["mixer"]["v_mix"]
    del doc["layers"][0]["mlp"]["router"]["groups"]
    _, _, again = build(doc)
    assert again.blocks[2].mixer.window is None and again.blocks[2].mixer.value_mix is None and again.blocks[0].ffn.groups == 1
    assert "l2.mix.vmix" not in {r.source.name for r in again.tensor_rows()}


@pytest.mark.parametrize("path,value", [(("layers", 2, "type"), "mlstm"), (("layers", 2, "mixer", "kv_heads"), 4),
                                        (("layers", 2, "mixer", "rot", "dims"), 5), (("layers", 2, "mixer", "rot", "dims"), 14),
                                        (("layers", 2, "mixer", "rot"), None), (("layers", 2, "mixer", "mask", "size"), 0),
                                        (("layers", 2, "mixer", "v_mix"), 1), (("layers", 3, "mixer", "vdim"), 16),
                                        (("layers", 2, "mlp", "kind"), "gated"), (("layers", 2, "mlp", "limit"), 0),
                                        (("layers", 0, "mixer", "decay"), [0.5, 0.9]), (("layers", 0, "mixer", "decay"), [0.5, 0.9, 1.5]),
                                        (("layers", 0, "mlp", "router", "top"), 9), (("layers", 0, "mlp", "router", "groups", "count"), 3),
                                        (("layers", 0, "mlp", "router", "groups", "keep"), 5), (("layers", 0, "mlp", "expert", "ff"), 0),
                                        (("token_side",), {}), (("logit_softcap",), 0), (("embedding", "scale"), "big"), (("width",), 0)])
def test_bad_values_are_refused(path, value):
    from ayaka_py_b200.config.model import ConfigError, MurutarConfig
    doc = json.loads(json.dumps(BASE))
    at = doc
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        MurutarConfig.from_dict(doc)


def test_arrangement_takes_its_feed_forward_whole_or_not_at_all():
    from ayaka_py_b200.parts import make_block
    parts = dict.fromkeys(("norm1", "mixer", "gate1"))
    make_block("gated_pre_norm", parts)
    make_block("gated_pre_norm", dict(parts, norm2=None, ffn=None, gate2=None, side=None))
    for wrong in (dict(parts, ffn=None), dict(parts, norm2=None, ffn=None), dict(parts, extra=None), {"norm1": None, "mixer": None}):
        with pytest.raises(ValueError):
            make_block("gated_pre_norm", wrong)


def test_stacked_inputs():
    """Matrices of a group lie one under the other, groups start at multiples of 8 rows, joined ones bring biases."""
    from ayaka_py_b200.parts.stacked import StackedInput
    gen = torch.Generator().manual_seed(0)
    a, b, c, d = (torch.randn((n, 6), generator=gen) for n in (5, 4, 3, 10))
    stack = StackedInput(6, [[a, b], [c]])
    assert stack.starts == [0, 16] and stack.weight.shape == (24, 6) and stack.bias is None
    bias = torch.arange(10, dtype=torch.float32)
    assert stack.join(d, bias) == 24 and stack.weight.shape == (40, 6)
    for view, want in zip(stack.views, (a, b, c, d)):
        assert torch.equal(view, want) and view.untyped_storage().data_ptr() == stack.weight.untyped_storage().data_ptr()
    assert torch.equal(stack.weight[5:9], b) and stack.weight[9:16].abs().max() == 0
    assert torch.equal(stack.bias[24:34], bias) and stack.bias[:24].abs().max() == 0


def test_pages_behind_the_window_of_the_next_position_come_back():
    """Page size 4, a window of 10: after every step the request holds exactly the pages from the one with the first key
    of the next token's window on."""
    from ayaka_py_b200.cache import CacheGroupSpec, CacheManager
    from ayaka_py_b200.parts.base import KVNeed
    m = CacheManager([CacheGroupSpec("w", KVNeed(2, 8, window=10, value_heads=2, value_dim=6), 1)], kv_pages=9, page_size=4, max_requests=2,
                     max_len=64, device=None)
    a, n = m.open("a"), 0
    for step in (3, 2, 7, 1, 1, 9, 1, 6, 1, 5, 1, 3):
        m.commit(m.reserve([(a, n, step)]))
        n += step
        m.check_invariants()
        held = [p for p in range(-(-n // 4)) if m.tables[0][a, p] > 0]
        assert held == list(range(max(0, n - 9) // 4, -(-n // 4))), (n, held)
    m.close(a)
    m.assert_clean()


def test_routing_of_the_plain_model():
    """A group counts by its best expert alone, groups shut experts out altogether, the weights are the scores over all
    experts as they are."""
    z = np.array([2.0, 2.0, 2.0, 3.0, -5.0, -5.0, 1.0, 0.5])
    chosen, w = plain.route(z, 3, 4, 2)                  # groups of two by their best: 2, 3, -5, 1 -> groups 1 and 0
    assert chosen == [3, 0, 1]
    s = np.exp(z) / np.exp(z).sum()
    assert np.allclose(w, s[[3, 0, 1]]) and w.sum() < 1
    chosen, _ = plain.route(np.array([1.0, 1.0, 1.0, 4.0, -9.0, -9.0]), 2, 2, 1)
    assert chosen == [3, 4]                              # a dropped group's experts score more than the kept group's second
    chosen, _ = plain.route(np.array([0.1, 0.4, 0.3, 0.4]), 2, 1, 1)
    assert chosen == [1, 3]


def test_sink_softmax_of_the_plain_model():
    s = np.array([[0.3, -1.0, 2.0]])
    seen = np.array([[True, False, True]])
    want = np.exp(s) * seen / (1 + (np.exp(s) * seen).sum())
    assert np.allclose(plain.sink_softmax(s, seen), want)
    assert np.allclose(plain.sink_softmax(s - 1000, seen), 0) and np.allclose(plain.sink_softmax(s + 1000, seen).sum(), 1)


def test_the_recurrence_of_the_plain_model_against_its_closed_form():
    rs = np.random.RandomState(5)
    T, H, D, Dv = 12, 2, 6, 5
    q, k, v, decay = rs.randn(T, H, D), rs.randn(T, H, D), rs.randn(T, H, Dv), (0.7, 1.0)
    got = plain.decayed_recurrence(q, k, v, decay)
    for t in range(T):
        for h in range(H):
            want = sum(decay[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert np.allclose(got[t, h], want, rtol=1e-9, atol=1e-12)


def test_plain_model_is_causal_and_respects_its_windows():
    """Changing a token moves the logits of later positions only, and with two layers of windowed attention only those
    that two windows reach; the recurrence carries it on."""
    att = {"type": "attention", "mlp": {"kind": "dense", "ff": 16, "limit": 3.0},
           "mixer": {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 8, "scale": 0.4, "v_mix": True, "mask": {"size": 5}, "rot": {"base": 100.0, "dims": 4}}}
    cfg = {"architecture": "Murutar", "vocab": 50, "width": 24, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
           "token_side": {"dim": 3}, "logit_softcap": 10.0, "layers": [att, att]}
    t = {k: v.astype(np.float64) for k, v in plain.random_tensors(cfg, 3).items()}
    toks = np.random.RandomState(0).randint(0, 50, 30).tolist()
    base = plain.forward(cfg, t, toks)
    other = list(toks)
    other[9] = (other[9] + 1) % 50
    moved = np.abs(plain.forward(cfg, t, other) - base).max(axis=1)
    assert (moved[:9] == 0).all() and (moved[9:18] > 0).all() and (moved[18:] == 0).all()
    cfg2 = dict(cfg, layers=[att, {"type": "lightning", "mlp": None, "mixer": {"heads": 2, "dim": 4, "vdim": 6, "decay": [0.8, 0.99]}}])
    t2 = {k: v.astype(np.float64) for k, v in plain.random_tensors(cfg2, 4).items()}
    moved = np.abs(plain.forward(cfg2, t2, other) - plain.forward(cfg2, t2, toks)).max(axis=1)
    assert (moved[:9] == 0).all() and (moved[9:] > 0).all()
