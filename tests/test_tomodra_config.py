"""Tomodra on the host: configuration, registry, the model as data, caches that several run steps read, tensor names,
and the plain implementation's own masks, sink, rotation and routing."""

import json

import numpy as np
import pytest
import torch

import plain_tomodra as plain

_MOE = {"kind": "moe", "router": {"experts": 6, "top": 2}, "expert": {"ff": 20}, "shared": {"ff": 28}}
_ATT = {"type": "attention", "mlp": _MOE,
        "mixer": {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 20, "scale": 0.3, "mask": {"size": 21},
                  "rot": {"base": 5000.0, "dims": 6, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 2.0}}}}
_LAT = {"type": "latent_attention", "mlp": _MOE,
        "mixer": {"heads": 3, "dim": 10, "rot_dim": 4, "vdim": 14, "kv_rank": 18, "scale": 0.25, "mask": {"size": 9}, "rot": {"base": 100.0, "dims": 4}}}


def reader(of, **changes):
    return {"type": "latent_attention", "mlp": None, "mixer": dict(_LAT["mixer"], kv_from=of, **changes)}


BASE = {"architecture": "Tomodra", "vocab": 97, "width": 48, "norm": {"eps": 1e-5}, "postln_alpha": 1.75,
        "layers": [_LAT, _ATT, reader(0, heads=5, mask={"size": 30}), dict(_LAT, mlp=None), reader(3, dim=7, mask={"size": 4}), _ATT]}


def build(document, dtype=torch.bfloat16):
    from ayaka_py_b200 import models, parts  # noqa: F401
    from ayaka_py_b200.models.model import Model
    from ayaka_py_b200.registry import architecture_for
    arch = architecture_for(document)
    config = arch.config_class.from_dict(document)
    return arch, config, Model(arch.build_spec(config), dtype, "meta")


def test_registry_and_round_trip():
    arch, config, _ = build(BASE)
    assert arch.name == "Tomodra"
    again = arch.config_class.from_dict(config.to_dict())
    assert again.to_dict() == config.to_dict() and again.to_dict()["architecture"] == "Tomodra"


def test_tensor_names_and_shapes():
    arch, config, model = build(BASE)
    rows = {r.source.name: tuple(r.decl.shape) for r in model.tensor_rows()}
    assert rows == plain.tensor_shapes(BASE)
    assert "l0.mix.dkv" in rows and "l2.mix.dkv" not in rows and "l2.mix.dkv.norm" not in rows and "l2.mix.uk" in rows
    # a layer without feed-forward has neither its tensors nor its norm, and passes them over in a checkpoint
    assert "l2.norm2" not in rows and "l2.norm1" in rows and "l0.norm2" in rows
    assert arch.normalize_name("l2.norm2", config) is None and arch.normalize_name("l2.mlp.e0.up", config) is None
    assert arch.normalize_name("l0.norm2", config) == "l0.norm2" and arch.normalize_name("l2.norm1", config) == "l2.norm1"


def test_cache_groups_and_constants():
    from ayaka_py_b200.parts import KVNeed
    _, _, model = build(BASE)
    assert {b.KIND for b in model.blocks} == {"normed_sum"}
    latent = dict(kv_heads=1, head_dim=4, value_heads=1, value_dim=18)
    needs = {g.need: g.layers for g in model.groups}
    # layer 0's cache serves a reader with a longer window and keeps that much; layer 3's reader has a shorter one
    assert needs == {KVNeed(window=30, **latent): 1, KVNeed(window=9, **latent): 1,
                     KVNeed(kv_heads=3, head_dim=12, value_heads=3, value_dim=20, chunk=21): 2}
    own, attn, read, own2, read2, attn2 = (b["mixer"] for b in model.bindings)
    assert (read.group, read.layer, read.writes) == (own.group, own.layer, False) and own.writes
    assert (read2.group, read2.layer, read2.writes) == (own2.group, own2.layer, False) and own2.group != own.group
    assert (attn2.group, attn2.layer) == (attn.group, 1)
    first, att, second = (model.blocks[i].mixer for i in (0, 1, 2))
    assert (first.window, first.own_latent, first.gate_width, first.rotary.halves, first.rotary.dims) == (9, True, 0, True, 4)
    assert (second.window, second.own_latent, second.heads, second.down_width) == (30, False, 5, 0)
    assert (att.chunk, att.window, att.learned_sink, att.qk_norm_eps, att.scale) == (21, None, True, 1e-5, 0.3)
    assert not att.rotary.halves and att.rotary.scaling["factor"] == 3.0 and att.rotary.gain == pytest.approx(0.1 * np.log(3.0) + 1)
    moe = model.blocks[0].ffn
    assert (moe.router, moe.top, moe.weigh, moe.slope, moe.plus, moe.limit, moe.shared_gated, moe.shared_inner) == \
        ("sigmoid", 2, "input", 1.0, 0.0, float("inf"), True, 28)
    assert {(b.norm1.stream_factor, b.norm1.eps) for b in model.blocks} == {(1.75, 1e-5)} and model.blocks[0].norm2.stream_factor == 1.75
    assert model.final_norm.stream_factor == 1.0
    # no mask: every earlier key; no scaling; no shared expert
    doc = json.loads(json.dumps(BASE))
    del doc["layers"][2]["mixer"]["mask"], doc["layers"][1]["mixer"]["mask"], doc["layers"][1]["mixer"]["rot"]["scaling"]
    doc["layers"][1]["mlp"]["shared"] = None
    _, _, again = build(doc)
    assert again.groups[again.bindings[0]["mixer"].group].need.window is None and again.blocks[0].mixer.window == 9
    assert again.blocks[1].mixer.chunk is None and again.blocks[1].mixer.rotary.gain == 1.0 and again.blocks[1].ffn.shared_inner == 0


@pytest.mark.parametrize("path,value", [(("layers", 1, "type"), "mlstm"), (("layers", 1, "mixer", "kv_heads"), 4), (("layers", 1, "mixer", "heads"), 0),
                                        (("layers", 1, "mixer", "rot", "dims"), 5), (("layers", 1, "mixer", "rot", "dims"), 14),
                                        (("layers", 1, "mixer", "rot"), None), (("layers", 1, "mixer", "rot", "scaling", "factor"), 0),
                                        (("layers", 1, "mixer", "rot", "scaling", "slow"), None), (("layers", 1, "mixer", "mask", "size"), 0),
                                        (("layers", 0, "mixer", "rot", "dims"), 2), (("layers", 0, "mixer", "kv_rank"), None),
                                        (("layers", 0, "mixer", "scale"), "big"), (("layers", 2, "mixer", "kv_from"), 1),
                                        (("layers", 2, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "kv_from"), 3),
                                        (("layers", 2, "mixer", "kv_from"), -1), (("layers", 4, "mixer", "kv_from"), 2),
                                        (("layers", 2, "mixer", "kv_rank"), 20), (("layers", 2, "mixer", "rot", "base"), 101.0),
                                        (("layers", 1, "mlp", "kind"), "dense"), (("layers", 1, "mlp", "router", "top"), 7),
                                        (("layers", 1, "mlp", "expert", "ff"), 0), (("layers", 1, "mlp", "shared"), 3),
                                        (("norm",), {}), (("postln_alpha",), None), (("width",), 0), (("layers",), [])])
def test_bad_values_are_refused(path, value):
    from ayaka_py_b200.config.model import ConfigError, TomodraConfig
    doc = json.loads(json.dumps(BASE))
    at = doc
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        TomodraConfig.from_dict(doc)


def test_arrangement_takes_its_feed_forward_whole_or_not_at_all():
    from ayaka_py_b200.parts import make_block
    parts = dict.fromkeys(("copy", "mixer", "norm1"))
    make_block("normed_sum", parts)
    make_block("normed_sum", dict(parts, ffn=None, norm2=None))
    for wrong in (dict(parts, ffn=None), dict(parts, norm2=None), dict(parts, extra=None), {"mixer": None, "norm1": None}):
        with pytest.raises(ValueError):
            make_block("normed_sum", wrong)


def test_parts_refuse_what_they_cannot_do():
    from ayaka_py_b200.parts import PartSpec, make_part
    common = {"width": 16, "experts": 4, "top": 2, "inner": 8, "limit": None, "shared_inner": 0, "shared_limit": None}
    make_part(PartSpec("moe", dict(common, router="sigmoid", weigh="input")), torch.float32, "meta")
    for wrong in ({"weigh": "both"}, {"weigh": "input", "activation": "relu2"}, {"router": "argmax"}):
        with pytest.raises(ValueError):
            make_part(PartSpec("moe", dict(common, **wrong)), torch.float32, "meta")
    att = {"width": 16, "heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.0}
    with pytest.raises(ValueError):
        make_part(PartSpec("rotary_attention", dict(att, sink="loud")), torch.float32, "meta")
    lat = {"width": 16, "heads": 2, "dim": 8, "rot_dim": 0, "vdim": 8, "kv_rank": 8, "scale": 1.0, "eps": 1e-5, "rot": None}
    for wrong in ({"gate": "row"}, {"window": 0}):
        with pytest.raises(ValueError):
            make_part(PartSpec("latent_attention", dict(lat, **wrong)), torch.float32, "meta")


def test_needs_of_readers_of_one_cache():
    """What is kept is what either reader may read; pages of another geometry are refused."""
    from ayaka_py_b200.parts import KVNeed
    need = lambda **kw: KVNeed(kv_heads=2, head_dim=8, value_dim=6, **kw)
    assert need(window=5).together(need(window=9)) == need(window=9)
    assert need(window=5).together(need()) == need() and need().together(need(window=5)) == need()
    assert need(window=5, keep_first=3).together(need(window=4, keep_first=7)) == need(window=5, keep_first=7)
    assert need(chunk=16).together(need(chunk=16)) == need(chunk=16)
    assert need(chunk=16).together(need(chunk=8)) == need() and need(chunk=16).together(need(window=9)) == need()
    assert need(window=5, chunk=8).together(need(window=6, chunk=8)) == need(window=6, chunk=8)
    with pytest.raises(ValueError):
        need().together(KVNeed(kv_heads=2, head_dim=8, value_dim=7))


def test_run_steps_that_read_a_cache_must_fit():
    from dataclasses import replace

    from ayaka_py_b200.models.model import Model
    from ayaka_py_b200.parts import RunStep
    arch, config, _ = build(BASE)
    spec = arch.build_spec(config)
    # a reader of a reader reads the owner's cache, which then keeps what all three need
    longer = {"type": "latent_attention", "mlp": None, "mixer": dict(_LAT["mixer"], kv_from=0, mask={"size": 50})}
    doc = dict(BASE, layers=[_LAT, reader(0), longer])
    arch3 = build(doc)[0]
    spec3 = arch3.build_spec(arch3.config_class.from_dict(doc))
    model = Model(replace(spec3, order=(RunStep(0), RunStep(1, cache_of=0), RunStep(2, cache_of=1))), torch.bfloat16, "meta")
    assert [g.need.window for g in model.groups] == [50] and [b["mixer"].layer for b in model.bindings] == [0, 0, 0]
    for order in ((RunStep(0), RunStep(1, cache_of=0)), (RunStep(0, cache_of=0),), (RunStep(2, cache_of=1), RunStep(0))):
        with pytest.raises(ValueError):
            Model(replace(spec, order=order), torch.bfloat16, "meta")


def test_pages_stay_for_the_longest_window_that_reads_them():
    """Page size 4; the cache of a layer with a window of 9 that a window of 30 reads as well holds the latter's pages."""
    from ayaka_py_b200.cache import CacheManager
    _, _, model = build(BASE)
    m = CacheManager(model.groups, kv_pages=40, page_size=4, max_requests=2, max_len=128, device=None)
    a, n = m.open("a"), 0
    wide, narrow, chunk = (model.bindings[i]["mixer"].group for i in (0, 3, 1))
    for step in (3, 20, 1, 1, 18, 1, 2, 31, 1, 1):
        m.commit(m.reserve([(a, n, step)]))
        n += step
        m.check_invariants()
        for group, first in ((wide, max(0, n - 29)), (narrow, max(0, n - 8)), (chunk, n // 21 * 21)):
            held = [p for p in range(-(-n // 4)) if m.tables[group][a, p] > 0]
            assert held == list(range(first // 4, -(-n // 4))), (n, group, held)
    m.close(a)
    m.assert_clean()


# ------------------------------------------------- the plain implementation --

def test_masks_of_the_plain_model():
    w, c = plain.window_mask(12, 4), plain.chunk_mask(12, 5)
    for i in range(12):
        assert np.flatnonzero(w[i]).tolist() == list(range(max(0, i - 3), i + 1))
        assert np.flatnonzero(c[i]).tolist() == list(range(i // 5 * 5, i + 1))
    assert plain.window_mask(6, None).sum() == plain.chunk_mask(6, None).sum() == 21


def test_softmax_of_the_plain_model():
    s = np.array([[[0.3, -1.0, 2.0]], [[5.0, 1.0, -2.0]]])
    seen = np.array([[True, False, True]])
    e = np.exp(s) * seen
    assert np.allclose(plain.softmax(s, seen), e / e.sum(-1, keepdims=True))
    sink = np.array([0.7, -3.0])
    assert np.allclose(plain.softmax(s, seen, sink), e / (e.sum(-1, keepdims=True) + np.exp(sink)[:, None, None]))
    assert np.allclose(plain.softmax(s - 1000, seen, sink), 0) and np.allclose(plain.softmax(s, seen, sink + 800), 0)


def test_rotation_of_the_plain_model():
    """A product of two rotated vectors depends on their distance alone; each pair turns by its own angle; the
    dimensions beyond pass; the framework's frequencies are the same."""
    from ayaka_py_b200.parts.position import rotary_frequencies
    rs = np.random.RandomState(0)
    for scaling in (None, {"factor": 8.0, "original": 100, "fast": 16.0, "slow": 1.0}, {"factor": 2.5, "original": 30, "fast": 1.0, "slow": 1.0}):
        rot = {"dims": 8, "base": 300.0, "scaling": scaling}
        f, gain = plain.frequencies(rot)
        f2, gain2 = rotary_frequencies(8, 300.0, scaling)
        assert np.allclose(f, f2, rtol=1e-14) and gain == pytest.approx(gain2)
        if scaling is None:
            assert gain == 1.0 and np.allclose(f, 300.0 ** (-np.arange(4) / 4))
        else:
            assert np.all(f <= 300.0 ** (-np.arange(4) / 4) + 1e-15) and np.all(f >= 300.0 ** (-np.arange(4) / 4) / scaling["factor"] - 1e-15)
        for turn, pair in ((plain.rotate_neighbours, lambda i: (2 * i, 2 * i + 1)), (plain.rotate_halves, lambda i: (i, i + 4))):
            q, k = np.tile(rs.randn(10), (20, 1, 1)), np.tile(rs.randn(10), (20, 1, 1))
            rq, rk = turn(q, rot)[:, 0], turn(k, rot)[:, 0]
            dots = rq @ rk.T
            assert np.allclose([dots[7, 3], dots[11, 7]], dots[4, 0]) and not np.isclose(dots[7, 3], dots[7, 2])
            assert np.allclose(rq[:, 8:], q[:, 0, 8:])
            for i in range(4):
                u, v = (q[5, 0, j] for j in pair(i))
                a = 5 * f[i]
                assert np.allclose(rq[5, list(pair(i))], [gain * (u * np.cos(a) - v * np.sin(a)), gain * (v * np.cos(a) + u * np.sin(a))])


def test_routing_of_the_plain_model():
    chosen, w = plain.route(np.array([0.5, 2.0, -1.0, 2.0, 1.0]), 3)
    assert chosen == [1, 3, 4] and np.allclose(w, 1 / (1 + np.exp(-np.array([2.0, 2.0, 1.0])))) and w.sum() > 1
    margin = []
    plain.route(np.array([0.5, 2.0, -1.0]), 2, margin)
    plain.route(np.array([0.5, 2.0]), 2, margin)
    assert margin == [1.5, np.inf]


def test_weights_in_front_of_an_expert_are_another_function_than_behind_it():
    rs = np.random.RandomState(1)
    t = {n: rs.randn(*s) for n, s in (("gate", (6, 5)), ("up", (6, 5)), ("down", (5, 6)))}
    h = rs.randn(1, 5)
    assert np.allclose(plain.expert(1.0 * h, t, ""), plain.expert(h, t, ""))
    assert np.abs(plain.expert(0.6 * h, t, "") - 0.6 * plain.expert(h, t, "")).max() > 0.05


def test_plain_model_is_causal_and_respects_windows_and_chunks():
    """Changing a token moves the logits of later positions only, and only those that the windows, one after the other,
    or the token's chunk reach."""
    lat = lambda **kw: {"type": "latent_attention", "mlp": _MOE, "mixer": dict(_LAT["mixer"], mask={"size": 5}, **kw)}
    cfg = dict(BASE, layers=[lat(), lat(kv_from=0)])
    t = {k: v.astype(np.float64) for k, v in plain.random_tensors(cfg, 3).items()}
    toks = np.random.RandomState(0).randint(0, 97, 30).tolist()
    other = list(toks)
    other[9] = (other[9] + 1) % 97
    moved = np.abs(plain.forward(cfg, t, other) - plain.forward(cfg, t, toks)).max(axis=1)
    # the second layer reads the first one's latents, made of the embeddings: the two windows do not add up
    assert (moved[:9] == 0).all() and (moved[9:14] > 0).all() and (moved[14:] == 0).all()
    cfg = dict(BASE, layers=[dict(_ATT, mixer=dict(_ATT["mixer"], mask={"size": 7}))] * 2)
    t = {k: v.astype(np.float64) for k, v in plain.random_tensors(cfg, 4).items()}
    moved = np.abs(plain.forward(cfg, t, other) - plain.forward(cfg, t, toks)).max(axis=1)
    assert (moved[:9] == 0).all() and (moved[9:14] > 0).all() and (moved[14:] == 0).all()
