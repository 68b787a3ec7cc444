"""Murutar: every mechanism alone against the plain functions of ``plain_murutar``, then whole models of
several shapes replayed whole, decoded, in portions and mixed, and greedy generation through the engine's own
entry point."""

import copy
import json
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_murutar as plain
import trace_tools
from test_gpu_vedadra import DT, bind, context_for, dev, host, mixer_alone, standing_out_rows, step_of, tol

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ configs --

def dense(n, limit=1.5):
    return {"kind": "dense", "ff": n, "limit": limit}


def moe(experts, top, count, keep, ff):
    router = {"experts": experts, "top": top}
    if count is not None:
        router["groups"] = {"count": count, "keep": keep}
    return {"kind": "moe", "router": router, "expert": {"ff": ff}}


def attention(heads, kv, dim, vdim, size, rot, scale, v_mix, mlp, base=10000.0):
    mixer = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix,
             "rot": {"base": base, "dims": rot}}
    if size is not None:
        mixer["mask"] = {"size": size}
    return {"type": "attention", "mlp": mlp, "mixer": mixer}


def lightning(dim, vdim, decay, mlp):
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def document(layers, vocab, width, side=8, cap=12.0, scale=None, eps=1e-5):
    return {"architecture": "Murutar", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": float(width) ** 0.5 if scale is None else scale}, "token_side": {"dim": side},
            "logit_softcap": cap, "layers": layers}


# A: odd sizes; a window that is no multiple of a page; layers without feed-forward; the recurrence first, so that its
# state meets the first tokens of the stream; a layer of attention that does not mix values between two that do.
CONFIG_A = document([lightning(10, 14, (0.7, 0.95, 0.999), moe(6, 2, 3, 2, 20)), attention(4, 2, 20, 12, 23, 12, 0.22, True, dense(40, 0.8)),
                     attention(2, 2, 12, 28, 7, 12, 0.3, False, None), attention(6, 2, 16, 12, 40, 2, 0.25, True, moe(8, 3, 2, 1, 16)),
                     lightning(7, 9, (0.5, 1.0), None)], vocab=211, width=72, side=12, scale=4.0)
# B: every head with keys of its own; a window of one token (a query sees itself and the sink); a window longer than any
# request; an attention without a window; every expert chosen; no groups; embedding scale 1; the first attention does not mix.
CONFIG_B = document([attention(4, 4, 16, 16, 1000, 8, 0.25, False, dense(48, 6.0)), lightning(32, 16, (0.3,), moe(4, 4, None, None, 24)),
                     attention(3, 3, 16, 40, 1, 16, 0.25, True, None), lightning(16, 48, (0.99, 0.9, 0.0), dense(30)),
                     attention(6, 3, 8, 40, None, 4, 0.35, True, moe(12, 2, 4, 2, 8), base=500.0)], vocab=130, width=64, side=20, cap=30.0, scale=1.0)
# C: sizes of the tensor-core kernels (heads of 64 and 128, eight query heads on two key/value heads), windows of a few
# pages, sixteen experts in eight groups.
CONFIG_C = document([attention(8, 2, 64, 128, 80, 32, 0.125, True, moe(16, 4, 8, 3, 64)), lightning(64, 128, (0.8, 0.99), dense(192, 2.0)),
                     lightning(32, 32, (0.6, 0.9, 0.97, 0.999), None), attention(4, 2, 128, 128, 48, 128, 0.09, True, moe(16, 4, 4, 2, 64)),
                     lightning(128, 64, (0.95, 0.998), dense(160, 1.0))], vocab=300, width=128, side=32, cap=20.0, eps=1e-6)
CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C}
LENGTHS = {"A": [1, 2, 19, 77, 150], "B": [3, 33, 64, 129], "C": [5, 48, 100, 300]}
PAGE = {"A": 16, "B": 8, "C": 16}


class Logits(np.ndarray):
    """Logits [T, V] with ``close``: the places where a router's choice was a close call."""


def oracle(cfg, t64, toks):
    margins = []
    out = plain.forward(cfg, t64, toks, margins=margins).view(Logits)
    out.close = np.min(np.stack(margins), axis=0) < 0.06 if margins else np.zeros(len(toks), dtype=bool)
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    base = tmp_path_factory.mktemp("murutar")
    out = {}
    for tag, cfg in CONFIGS.items():
        tensors = plain.random_tensors(cfg, seed=60 + ord(tag))
        folder = plain.write_folder(base / tag, cfg, tensors)
        rs = np.random.RandomState(ord(tag))
        reqs = {f"{tag.lower()}{i}": rs.randint(0, cfg["vocab"], n).tolist() for i, n in enumerate(LENGTHS[tag])}
        t64 = {k: v.astype(np.float64) for k, v in tensors.items()}
        want = {rid: oracle(cfg, t64, toks) for rid, toks in reqs.items()}
        out[tag] = (folder, cfg, t64, reqs, want)
    return out


def limit(dtype, want):
    big = max(float(np.abs(w).max()) for w in want.values())
    return (3e-5 if dtype == "float32" else 0.05) * big


def replay(folder, dtype, trace, page_size, max_tokens=None):
    from ayaka_py_b200.replay import ReplaySession
    session = ReplaySession(folder, dtype, max_tokens or trace_tools.tokens_needed(trace), page_size)
    outputs = []
    for record in trace:
        logits = session.step(record)
        outputs.append(None if logits is None or logits.shape[0] == 0 else logits.cpu().numpy())
    session.cache.assert_clean()
    return outputs, session


def check(models, tag, dtype, trace, want=None, **kw):
    """In 32-bit every position must agree.  In bfloat16 rounding can turn a router's close call, which moves
    that position's logits visibly and, through the caches and the recurrence, later ones a little: the places
    that the plain model marks as close calls are not compared, and of the others at most 2 in 100 may differ,
    which a lost state, a wrong page or a wrong edge would exceed at once."""
    folder = models[tag][0]
    want = want or models[tag][4]
    outputs, session = replay(folder, dtype, trace, PAGE[tag], **kw)
    got = trace_tools.collect(trace, outputs)
    if dtype == "float32":
        bad = trace_tools.first_difference(got, want, limit(dtype, want))
        assert bad is None, f"first wrong place: request {bad[0]} position {bad[1]} |diff| {bad[2]:.3e} (limit {limit(dtype, want):.3e})"
        return session
    over, total, first = 0, 0, None
    for rid, rows in want.items():
        for p in range(rows.shape[0]):
            assert p in got.get(rid, {}), f"request {rid} position {p} was not answered"
            if rows.close[p]:
                continue
            d = float(np.abs(got[rid][p] - np.asarray(rows[p])).max())
            total += 1
            if not d <= limit(dtype, want):
                over += 1
                first = first or (rid, p, d)
    assert over <= 0.02 * total, f"{over} of {total} places differ; the first: request {first[0]} position {first[1]} |diff| {first[2]:.3e}"
    return session


def layer_tensors(layer, d, seed, prefix="l0.mix.", side=4):
    t = plain.random_tensors(document([layer], 4, d, side), seed)
    return {k: v.astype(np.float64) for k, v in t.items()}, {k[len(prefix):]: v for k, v in t.items() if k.startswith(prefix)}


def put(t64, w, prefix="l0.mix."):
    for name, v in w.items():
        t64[prefix + name] = v.astype(np.float64)


def make(kind, params, dtype):
    from ayaka_py_b200.parts import PartSpec, make_part
    return make_part(PartSpec(kind, params), DT[dtype], "cuda")


# ------------------------------------------- the stream between the products --

STREAM_CASES = [72, 64, 6, 1537, 1, 2048, 4096, 5000]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", STREAM_CASES)
def test_gated_update_of_the_stream_and_the_norm_that_follows(dtype, d):
    """x += y s sigmoid(r) and, from the same kernel, the next layer norm, RMS norm or copy of it; y a row, or the
    weighted rows of chosen experts.  The gates are columns of a wider matrix."""
    from ayaka_py_b200 import ops
    rs = np.random.RandomState(d)
    for n in (1, 37):
        x, y = (rs.randn(n, d) * 2 + 9.0).astype(np.float32), rs.randn(n, d).astype(np.float32)      # a mean far from zero
        wide = rs.randn(n, d + 8).astype(np.float32) * 2
        s, w2 = rs.randn(d).astype(np.float32), (1.0 + 0.2 * rs.randn(d)).astype(np.float32)
        b2 = rs.randn(d).astype(np.float32)
        r = wide[:, 4:4 + d]
        want = x + y * s * plain.sigmoid(r.astype(np.float64))
        gates = dev(wide)[:, 4:4 + d]
        stream = dev(x)
        assert ops.stream_update(stream, dev(y), dev(s), gate=gates) is None
        assert np.abs(host(stream) - want).max() < 1e-4
        follow = {"copy": want, "layernorm": plain.layer_norm(want, w2.astype(np.float64), 3e-5) + b2,
                  "rmsnorm": plain.unit_rms(want, 3e-5) * w2}
        for post, expect in follow.items():
            stream = dev(x)
            got = ops.stream_update(stream, dev(y), dev(s), gate=gates, post=post, next_weight=dev(w2),
                                    next_bias=dev(b2) if post == "layernorm" else None, next_eps=3e-5, out_dtype=DT[dtype])
            assert got.dtype == DT[dtype] and np.abs(host(stream) - want).max() < 1e-4
            assert np.abs(host(got) - expect).max() < (5e-4 if dtype == "float32" else 2e-2) * max(1.0, float(np.abs(expect).max())), post
        # the rows of chosen experts, in order and at places of their own
        top = 3
        rows, weights = rs.randn(n * top, d).astype(np.float32), rs.rand(n, top).astype(np.float32)
        route = SimpleNamespace(weights=dev(weights), top=top)
        want = x + np.einsum("nk,nkd->nd", weights.astype(np.float64), rows.reshape(n, top, d)) * s * plain.sigmoid(r.astype(np.float64))
        place = rs.permutation(n * top + 5)[:n * top].astype(np.int32)
        spread = np.zeros((n * top + 5, d), dtype=np.float32)
        spread[place] = rows
        for picked in (ops.PickedRows(dev(rows), route, None), ops.PickedRows(dev(spread), route, torch.from_numpy(place).cuda())):
            stream = dev(x)
            got = ops.stream_update(stream, picked, dev(s), gate=gates, post="layernorm", next_weight=dev(w2), next_eps=3e-5, out_dtype=DT[dtype])
            assert np.abs(host(stream) - want).max() < 1e-4
            expect = plain.layer_norm(want, w2.astype(np.float64), 3e-5)
            assert np.abs(host(got) - expect).max() < (5e-4 if dtype == "float32" else 2e-2) * max(1.0, float(np.abs(expect).max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", STREAM_CASES)
def test_rms_normed_update_of_the_stream_and_the_norm_that_follows(dtype, d):
    from ayaka_py_b200 import ops
    rs = np.random.RandomState(d + 1)
    for n in (1, 37):
        x, y = rs.randn(n, d).astype(np.float32), (rs.randn(n, d) * 0.01 + 0.02).astype(np.float32)
        s, w2 = rs.randn(d).astype(np.float32), (1.0 + 0.2 * rs.randn(d)).astype(np.float32)
        want = x + plain.unit_rms(y.astype(np.float64), 2e-4) * s                       # an eps that matters
        for post in ("none", "layernorm"):
            stream = dev(x)
            got = ops.stream_update(stream, dev(y), dev(s), eps=2e-4, post=post, next_weight=dev(w2), next_eps=1e-5, out_dtype=DT[dtype])
            assert np.abs(host(stream) - want).max() < 1e-4
        expect = plain.layer_norm(want, w2.astype(np.float64), 1e-5)
        assert np.abs(host(got) - expect).max() < (5e-4 if dtype == "float32" else 2e-2) * max(1.0, float(np.abs(expect).max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", [72, 1, 6, 640])
def test_layer_norm_without_a_bias(dtype, d):
    rs = np.random.RandomState(d)
    x, w = (rs.randn(9, d) * 3 + 20).astype(np.float32), (1.0 + 0.2 * rs.randn(d)).astype(np.float32)
    part = make("layernorm", {"width": d, "eps": 1e-5, "bias": False}, dtype)
    assert set(part.tensors()) == {"weight"}
    part.bind({"weight": dev(w)})
    want = plain.layer_norm(x.astype(np.float64), w.astype(np.float64), 1e-5)
    assert np.abs(host(part.forward(dev(x), None)) - want).max() < (2e-4 if dtype == "float32" else 2e-2) * max(1.0, float(np.abs(want).max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,n,layers", [(72, 12, 3), (64, 5, 2), (128, 32, 1), (100, 64, 4), (50, 1, 2)])
def test_token_side_input_alone(dtype, d, n, layers):
    """The layer's own columns of the table, the tokens' own rows; a few rows (straight from the stream) and many."""
    from ayaka_py_b200 import ops
    rs = np.random.RandomState(n)
    vocab = 40
    lay = lightning(4, 4, (0.5,), None)
    t = plain.random_tensors(document([lay] * layers, vocab, d, n), 5)
    t64 = {k: v.astype(np.float64) for k, v in t.items()}
    for layer in range(layers):
        part = make("token_side", {"vocab": vocab, "width": d, "dim": n, "columns": n * layers, "col0": layer * n, "eps": 1e-4}, dtype)
        p = f"l{layer}.side."
        part.bind({"table": dev(t["side.embed"], DT[dtype]), "gate_weight": dev(t[p + "gate"], DT[dtype]),
                   "proj_weight": dev(t[p + "proj"], DT[dtype]), "norm": dev(t[p + "norm"])})
        for rows in (1, 5, 150):
            x = plain.round_bf16(rs.randn(rows, d).astype(np.float32))
            toks = rs.randint(0, vocab, rows)
            ctx = SimpleNamespace(tokens=torch.from_numpy(toks.astype(np.int32)).cuda())
            stream = dev(x)
            copy_ = stream.to(DT[dtype]) if part.reads_copy(rows) else None
            y = part.forward(stream, copy_, ctx)
            ops.stream_update(stream, y, part.norm, eps=part.eps)
            want = plain.token_input(x.astype(np.float64), toks, t64, f"l{layer}.", layer, n, 1e-4)
            assert np.abs(host(stream) - x - want).max() < (1e-4 if dtype == "float32" else 4e-2) * max(1.0, float(np.abs(want).max())), (layer, rows)
    other = plain.token_input(x.astype(np.float64), (toks + 1) % vocab, t64, f"l{layer}.", layer, n, 1e-4)
    assert np.abs(other - want).max() > 0.1


@pytest.mark.parametrize("shape", [(3, 640), (1, 7), (5, 1001)])
def test_soft_cap_of_the_logits(shape):
    from ayaka_py_b200 import ops
    z = (np.random.RandomState(1).randn(*shape) * 40).astype(np.float32)
    for cap in (15.0, 2.5):
        assert np.abs(host(ops.softcap_(dev(z), cap)) - cap * np.tanh(z.astype(np.float64) / cap)).max() < 1e-5 * cap


# -------------------------------------------------------------- feed-forward --

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,inner,bound", [(72, 40, 0.5), (64, 30, 1.0), (128, 192, 7.0), (48, 7, 1.3)])
def test_limited_gated_feed_forward_alone(dtype, d, inner, bound):
    """The gate is limited from above only, the up projection from both sides; another product rides along."""
    rs = np.random.RandomState(3)
    t64, w = layer_tensors(lightning(4, 4, (0.5,), dense(inner, bound)), d, 19, prefix="l0.mlp.")
    part = make("gated_mlp", {"width": d, "inner": inner, "activation": "limited_glu", "limit": bound}, dtype)
    bind(part, w, {"gate": "gate_weight", "up": "up_weight", "down": "down_weight"}, dtype)
    extra, bias = plain.round_bf16(rs.randn(d, d).astype(np.float32) / 8), rs.randn(d).astype(np.float32)
    for joined in (False, True):
        if joined:
            view = part.join_input(dev(extra, DT[dtype]), dev(bias))
            assert np.array_equal(host(view), extra)
        for n in (1, 5, 150):
            h = plain.round_bf16(rs.randn(n, d).astype(np.float32) * 2)
            ctx = SimpleNamespace(carry={})
            want = plain.limited_glu_ff(h.astype(np.float64), t64, "l0.mlp.", bound)
            got = part.forward(dev(h, DT[dtype]), None, ctx)
            assert np.abs(host(got) - want).max() < tol(dtype, 3 * float(np.abs(want).max()))
            if joined:
                assert np.abs(host(ctx.carry[part]) - (h.astype(np.float64) @ extra.T + bias)).max() < tol(dtype, 3.0)
    g, u = h.astype(np.float64) @ t64["l0.mlp.gate"].T, h.astype(np.float64) @ t64["l0.mlp.up"].T
    other = (np.clip(g, -bound, bound) * plain.sigmoid(1.702 * np.clip(g, -bound, bound)) * (np.clip(u, -bound, bound) + 1)) @ t64["l0.mlp.down"].T
    if bound < 2:                                      # a gate limited from below as well is another function
        assert np.abs(other - want).max() > 0.01


MOE_CASES = [(12, 3, 3, 2, 16), (8, 2, 1, 1, 24), (16, 4, 8, 3, 8), (6, 2, 6, 2, 20), (4, 4, 2, 2, 64), (64, 6, 8, 4, 8), (5, 5, 1, 1, 12),
             (32, 1, 2, 1, 40)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,top,count,keep,ff", MOE_CASES)
def test_experts_routed_by_softmax_scores_in_groups_alone(dtype, E, top, count, keep, ff):
    """Routing and output for a single token, a few and many (the experts' products run through different kernels),
    as rows and as a sum; the best expert of a dropped group scores more than some chosen one; the weights are the
    scores themselves."""
    from ayaka_py_b200 import ops
    d = 48
    mlp = moe(E, top, count, keep, ff)
    t64, w = layer_tensors(lightning(4, 4, (0.5,), mlp), d, 100 + E, prefix="l0.mlp.")
    part = make("moe", {"width": d, "experts": E, "top": top, "inner": ff, "limit": None, "shared_inner": 0, "shared_limit": None,
                        "router": "softmax_groups", "groups": count, "keep": keep, "activation": "relu2"}, dtype)
    names = {"router": "router_weight"}
    for e in range(E):
        names.update({f"e{e}.up": f"up_{e}", f"e{e}.down": f"down_{e}"})
    bind(part, w, names, dtype)
    rs = np.random.RandomState(E)
    extra, bias = plain.round_bf16(rs.randn(d, d).astype(np.float32) / 7), rs.randn(d).astype(np.float32)
    part.join_input(dev(extra, DT[dtype]), dev(bias))
    passed_over = False
    for n in (1, 7, 150):
        h = plain.round_bf16(rs.randn(n, d).astype(np.float32) * 1.5)
        margins = []
        want = plain.moe_ff(h.astype(np.float64), t64, "l0.mlp.", mlp, margins)
        clear = margins[0] > 1e-4
        z = h.astype(np.float64) @ t64["l0.mlp.router"].T
        route = ops.moe_route(dev(z.astype(np.float32)), E, top, {"groups": count, "keep": keep, "scores": "softmax", "group_best": 1,
                                                                  "normalize": False})
        ids, weights = route.ids.cpu().numpy(), host(route.weights)
        for t in np.flatnonzero(clear):
            chosen, wt = plain.route(z[t], top, count, keep)
            assert ids[t].tolist() == chosen, (t, ids[t], chosen)
            assert np.abs(weights[t] - wt).max() < 1e-6
            left = [e for e in range(E) if e not in chosen]
            passed_over = passed_over or (len(left) > 0 and z[t][left].max() > z[t][chosen].min())
        ctx = SimpleNamespace(carry={})
        x = dev(h, DT[dtype])
        big = float(np.abs(want).max())
        assert np.abs(host(part.forward(x, None, ctx)) - want)[clear].max() < tol(dtype, 4 * big), n
        assert np.abs(host(ctx.carry[part]) - (h.astype(np.float64) @ extra.T + bias)).max() < tol(dtype, 3.0)
        stream = torch.zeros(n, d, device="cuda")
        ops.stream_update(stream, part.forward_rows(x, ctx), torch.ones(d, device="cuda"), gate=torch.full((n, d), 40.0, device="cuda"))
        assert np.abs(host(stream) - want)[clear].max() < tol(dtype, 4 * big), n
        assert clear.mean() > 0.9
    assert passed_over or keep == count or count == E or top == 1      # in the last two cases the best experts are the chosen ones


def test_routing_where_scores_underflow():
    """Experts are ranked by their logits, so also among scores that are zero in 32-bit."""
    from ayaka_py_b200 import ops
    z = np.array([[300.0, -10.0, 5.0, 7.0, 6.0, -400.0]], dtype=np.float32)
    route = ops.moe_route(dev(z), 6, 4, {"groups": 2, "keep": 2, "scores": "softmax", "group_best": 1, "normalize": False})
    assert route.ids.cpu().numpy().tolist() == [[0, 3, 4, 2]]
    assert host(route.weights).tolist() == [[1.0, 0.0, 0.0, 0.0]]


# ---------------------------------------------------------------- attention --

ATT_NAMES = {"q": "q_weight", "k": "k_weight", "v": "v_weight", "vmix": "mix", "o": "out_weight"}


def attention_part(layer, d, dtype, value_mix=None, rot=True):
    mx = layer["mixer"]
    return make("rotary_attention", {"width": d, "heads": mx["heads"], "kv_heads": mx["kv_heads"], "dim": mx["dim"], "vdim": mx["vdim"],
                                     "scale": mx["scale"], "rot": mx["rot"] if rot else None, "window": (mx.get("mask") or {}).get("size"),
                                     "sink": 0.0, "value_mix": value_mix}, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv,size,rot", [(4, 2, 20, 12, 23, 12), (3, 3, 16, 40, 1, 16), (4, 1, 8, 16, None, 2), (8, 2, 64, 128, 80, 32),
                                               (2, 2, 12, 28, 7, 6), (4, 4, 32, 32, 130, 24), (2, 1, 128, 64, 1000, 128), (5, 1, 16, 256, 16, 8)])
def test_windowed_rotary_attention_with_a_sink_alone(dtype, H, G, D, Dv, size, rot):
    d = 48
    layer = attention(H, G, D, Dv, size, rot, 1.5 / np.sqrt(D), False, None)
    t64, w = layer_tensors(layer, d, 29)
    part = attention_part(layer, d, dtype)
    bind(part, w, ATT_NAMES, dtype)
    fn = lambda h: plain.sink_attention(h, t64, "l0.mix.", layer["mixer"], 1e-5, [])
    mixer_alone(part, dtype, d, fn, {0: 150, 1: 9, 2: 70})


@pytest.mark.parametrize("sink,gain", [(0.0, 0.2), (0.0, 6.0), (3.0, 1.0), (-40.0, 1.0), (30.0, 1.0)])
def test_the_sinks_share_of_the_denominator(sink, gain):
    """Scores far below, around and far above the sink's, in both kernels and both forms (with the context cut into
    parts and whole): the output is the softmax over the keys and one more without a value."""
    from ayaka_py_b200 import ops
    from ayaka_py_b200.cache import CacheGroupSpec
    from ayaka_py_b200.parts import KVNeed
    H, G, D, Dv, n = 4, 2, 32, 32, 200
    rs = np.random.RandomState(8)
    for window in (None, 70):
        for dtype in ("float32", "bfloat16"):
            q, k, v = (plain.round_bf16(rs.randn(n, h, e).astype(np.float32)) for h, e in ((H, D), (G, D), (G, Dv)))
            cache, runner = context_for([CacheGroupSpec("g", KVNeed(G, D, window=window, value_heads=G, value_dim=Dv), 1)], dtype,
                                        max_requests=2, page_size=8, pages=64)
            kp, vp = cache.kv_layer(0, 0)
            sinks = torch.full((H,), sink, device="cuda")
            s = np.einsum("ihd,jhd->hij", q.astype(np.float64), k.astype(np.float64)[:, np.arange(H) // 2]) * gain / np.sqrt(D)
            seen = plain.window_mask(n, window)
            s = np.where(seen, s, -np.inf)
            top = np.maximum(s.max(axis=-1, keepdims=True), sink)
            e = np.exp(s - top)
            p = e / (np.exp(sink - top) + e.sum(axis=-1, keepdims=True))
            want = np.einsum("hij,jhd->ihd", p, v.astype(np.float64)[:, np.arange(H) // 2]).reshape(n, H * Dv)
            at = 0
            for count in (150, 1, 1, 48):
                ctx, res = step_of(cache, runner, {0: count})
                rows = slice(at, at + count)
                ops.kv_append(kp, vp, dev(k[rows].reshape(count, -1), DT[dtype]), dev(v[rows].reshape(count, -1), DT[dtype]), ctx.row_req,
                              ctx.positions, ctx.tables[0])
                for tensor_cores in (True, False):
                    got = ops.grouped_attention(dev(q[rows].reshape(count, -1), DT[dtype]), kp, vp, ctx.tables[0], ctx, heads=H, key_heads=G,
                                                key_dim=D, scale=gain / np.sqrt(D), window=window, sinks=sinks, tensor_cores=tensor_cores)
                    worst = np.abs(host(got) - want[rows]).max()
                    assert worst < (3e-5 if dtype == "float32" else 2e-2) * np.abs(want).max() + 1e-12, (window, dtype, count, tensor_cores, worst)
                cache.commit(res)
                at += count


def edge_places(P, size, n):
    """The first tokens, page borders, keys just inside and just outside the windows of the last queries, and the end."""
    out = {0, 2, P - 1, P, P + 1, 5 * P - 1, 5 * P, n - 1, n - 2, n - size, n - size - 1, n - size + 1, n - 3}
    return sorted(p for p in out if 0 <= p < n)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv,size,gain", [(4, 2, 20, 12, 37, 4.0), (8, 2, 64, 128, 70, 4.0), (2, 1, 32, 64, 1000, 4.0), (4, 1, 16, 16, 24, 4.0),
                                                (3, 3, 16, 24, 129, 1.0)])
def test_attention_with_keys_that_stand_out_at_window_and_page_borders(dtype, H, G, D, Dv, size, gain):
    """Keys made from the queries' matrix at chosen places score high against one another (the rotation turns two
    dimensions only, slowly).  A window that is one position longer or shorter gives another output at a checked place."""
    rs = np.random.RandomState(17)
    d, P = 48, 8
    layer = attention(H, G, D, Dv, size, 2, gain / D, False, None, base=2.0)
    t64, w = layer_tensors(layer, d, 37)
    q = w["q"].reshape(H, D, d)
    q[:, :2] = 0                                              # nothing on the dimensions that turn
    w["q"] = q.reshape(H * D, d)
    w["k"] = q[::H // G].reshape(G * D, d).copy()
    put(t64, w)
    part = attention_part(layer, d, dtype)
    bind(part, w, ATT_NAMES, dtype)
    lengths = {0: 330, 1: 9, 2: 70}
    places = {0: edge_places(P, size, 330), 1: [0, 8], 2: [3, 2 * P, 69]}
    rows = {i: standing_out_rows(rs, n, d, places[i]) for i, n in lengths.items()}
    want = mixer_alone(part, dtype, d, lambda h: plain.sink_attention(h, t64, "l0.mix.", layer["mixer"], 1e-5, []), lengths, rows=rows, page_size=P)
    if size < 330:
        for other_size in (size + 1, size - 1):
            other_mx = copy.deepcopy(layer["mixer"])
            other_mx["mask"]["size"] = other_size
            other = plain.sink_attention(rows[0].astype(np.float64), t64, "l0.mix.", other_mx, 1e-5, [])
            worst = max(np.abs(other[p] - want[0][p]).max() for p in (329, 328))
            assert worst > 0.01 * np.abs(want[0]).max(), other_size


def test_rotation_of_every_pair_and_only_those():
    """Queries and keys of one row each at far positions, dimension by dimension: pairs (i, i + dims/2), the rest passes;
    a base for which the slow pairs hardly move and one for which all do; vector and scalar forms."""
    from ayaka_py_b200 import ops
    from ayaka_py_b200.cache import CacheGroupSpec
    from ayaka_py_b200.parts import KVNeed
    from ayaka_py_b200.parts.position import rotary_frequencies
    rs = np.random.RandomState(2)
    for H, G, D, Dv, dims, base in ((3, 1, 20, 12, 12, 1e4), (2, 2, 64, 48, 16, 5e5), (4, 2, 16, 8, 16, 3.0), (2, 1, 7, 5, 6, 100.0), (2, 1, 24, 4, 8, 50.0)):
        n = 600
        cache, runner = context_for([CacheGroupSpec("g", KVNeed(G, D, value_heads=G, value_dim=Dv), 1)], "float32", max_requests=2, page_size=8, pages=128)
        ctx, res = step_of(cache, runner, {0: n})
        proj = rs.randn(n, (H + G) * D + G * Dv + 3).astype(np.float32)
        kp, vp = cache.kv_layer(0, 0)
        freq = torch.tensor(rotary_frequencies(dims, base, None)[0], dtype=torch.float64).float().cuda()
        first = rs.randn(n, G * Dv).astype(np.float32)
        q = ops.rotary_prepare(dev(proj), kp, vp, freq, dims, ctx, ctx.tables[0], H, True, torch.float32, first=dev(first), mix=0.3)
        both = plain.rotate_halves(proj[:, :(H + G) * D].astype(np.float64).reshape(n, H + G, D), base, dims)
        assert np.abs(host(q).reshape(n, H, D) - both[:, :H]).max() < 2e-4
        table = cache.table_rows(0, [cache.slot_of[0]])[0]
        cells = [(int(table[p // 8]), p % 8) for p in range(n)]
        keys = np.stack([host(kp)[c] for c in cells])
        values = np.stack([host(vp)[c] for c in cells])
        assert np.abs(keys - both[:, H:]).max() < 2e-4
        own = proj[:, (H + G) * D:(H + G) * D + G * Dv].reshape(n, G, Dv)
        assert np.abs(values - (0.7 * own + 0.3 * first.reshape(n, G, Dv))).max() < 1e-5
        cache.commit(res)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_values_blended_with_an_earlier_layers(dtype):
    """The values filed are the blended ones (decoding reads them from the cache), the first layer's are its own."""
    d, H, G, D, Dv = 48, 4, 2, 16, 24
    layer = attention(H, G, D, Dv, 19, 8, 0.3, True, None)
    t64, w = layer_tensors(layer, d, 31)
    for lam in (0.4, -0.5, 1.0):
        w["vmix"] = np.float32(lam)
        put(t64, w)
        t64["l0.mix.vmix"] = np.asarray(lam)
        part = attention_part(layer, d, dtype, "blend")
        bind(part, w, ATT_NAMES, dtype)
        head = attention_part(layer, d, dtype, "first")
        bind(head, w, ATT_NAMES, dtype)
        earlier = plain.round_bf16(np.random.RandomState(3).randn(G * Dv, d).astype(np.float32) / 7)

        class Second:
            def cache_need(self):
                return part.cache_need()

            def forward(self, x, residual, ctx, binding):
                ctx.carry["first_values"] = (x.float() @ dev(earlier).t()).contiguous()
                return part.forward(x, residual, ctx, binding)

        def second(h):
            return plain.sink_attention(h, t64, "l0.mix.", layer["mixer"], 1e-5, [(h @ earlier.T).reshape(-1, G, Dv)])
        want = mixer_alone(Second(), dtype, d, second, {0: 80, 1: 9, 2: 30})
        unmixed = mixer_alone(head, dtype, d, lambda h: plain.sink_attention(h, t64, "l0.mix.", layer["mixer"], 1e-5, []), {0: 80, 1: 9, 2: 30})
        assert np.abs(want[0] - unmixed[0]).max() > 0.1


# -------------------------------------------------------------- recurrence --

LIGHT_NAMES = {"q": "q_weight", "k": "k_weight", "v": "v_weight", "g": "gate_weight", "norm": "norm", "o": "out_weight"}


def lightning_part(layer, d, dtype, eps=1e-5):
    mx = layer["mixer"]
    return make("lightning", {"width": d, "heads": mx["heads"], "dim": mx["dim"], "vdim": mx["vdim"], "decay": mx["decay"], "eps": eps}, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D,Dv,decay", [(10, 14, (0.7, 0.95, 0.999)), (32, 64, (0.5,)), (64, 128, (0.8, 0.99)), (32, 32, (0.6, 0.9, 1.0, 0.0)),
                                        (7, 5, (0.97, 0.3)), (20, 256, (0.9,)), (128, 40, (0.99,)), (256, 16, (0.95,)), (300, 8, (0.95,))])
def test_lightning_alone(dtype, D, Dv, decay):
    """Whole, token by token, in ragged portions (the chunked kernel meets chunks of every length), batched, and in
    slots that were used before; decays of 1 and 0; heads of 300 numbers take the token-by-token kernel for prompts too."""
    d = 48
    layer = lightning(D, Dv, decay, None)
    t64, w = layer_tensors(layer, d, 43)
    part = lightning_part(layer, d, dtype)
    bind(part, w, LIGHT_NAMES, dtype)
    mixer_alone(part, dtype, d, lambda h: plain.lightning(h, t64, "l0.mix.", layer["mixer"], 1e-5), {0: 150, 1: 9, 2: 70})


def test_lightning_remembers_far_tokens():
    """A token 300 back that stands out still counts under a decay near one, not under a small one."""
    d = 48
    rs = np.random.RandomState(3)
    rows = {0: standing_out_rows(rs, 330, d, [5, 29]), 1: standing_out_rows(rs, 9, d, [0]), 2: standing_out_rows(rs, 70, d, [3])}
    for decay, felt in (((0.9995, 0.9999), True), ((0.5, 0.8), False)):
        layer = lightning(16, 24, decay, None)
        t64, w = layer_tensors(layer, d, 47)
        for dtype in ("float32", "bfloat16"):
            part = lightning_part(layer, d, dtype)
            bind(part, w, LIGHT_NAMES, dtype)
            want = mixer_alone(part, dtype, d, lambda h: plain.lightning(h, t64, "l0.mix.", layer["mixer"], 1e-5), {0: 330, 1: 9, 2: 70}, rows=rows)
        x = rows[0].astype(np.float64).copy()
        x[5] = 0.0
        other = plain.lightning(x, t64, "l0.mix.", layer["mixer"], 1e-5)
        assert (np.abs(other[320] - want[0][320]).max() > 1e-3 * np.abs(want[0]).max()) == felt


@pytest.mark.parametrize("H,D,Dv", [(2, 16, 24), (3, 64, 128), (2, 40, 33), (1, 128, 128), (2, 7, 70)])
def test_the_two_kernels_of_the_recurrence_against_one_another(H, D, Dv):
    """Chunks of 64 tokens on the tensor cores (one after the other in blocks of 16 and of 32 value columns, and side by
    side) and token by token: the same inputs
    (exact in bfloat16), 32-bit outputs and 32-bit states, over portions that leave ragged chunks."""
    from ayaka_py_b200 import ops
    from ayaka_py_b200.cache import CacheGroupSpec
    from ayaka_py_b200.parts import StateNeed
    rs = np.random.RandomState(D)
    decay = np.linspace(0.6, 0.9995, H)
    powers = dev((decay[:, None] ** np.arange(65)[None, :]).astype(np.float32))
    n = H * (2 * D + Dv)
    z = rs.randn(300, n).astype(np.float32) * 2
    act = plain.round_bf16((z / (1 + np.exp(-z))).astype(np.float32))
    a64 = act.astype(np.float64)
    q, k, v = a64[:, :H * D].reshape(-1, H, D), a64[:, H * D:2 * H * D].reshape(-1, H, D), a64[:, 2 * H * D:].reshape(-1, H, Dv)
    want = plain.decayed_recurrence(q, k, v, decay).reshape(300, H * Dv)
    S = np.zeros((H, D, Dv))
    for t in range(300):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
    for cols, side in ((16, False), (32, False), (0, True)):
        if side and Dv % 8:
            continue
        cache, runner = context_for([CacheGroupSpec("g", StateNeed((H, D, Dv), torch.float32), 1)], "bfloat16", max_requests=2, page_size=8, pages=8)
        got, at = [], 0
        for count in (130, 2, 63, 64, 41):
            ctx, res = step_of(cache, runner, {0: count})
            got.append(host(ops.decay_recurrence(dev(act[at:at + count], torch.bfloat16), cache.state_layer(0, 0), powers, ctx, H, D, Dv, slice_cols=cols,
                                                side_by_side=side)))
            cache.commit(res)
            at += count
        assert np.abs(np.concatenate(got) - want).max() < 1e-4 * np.abs(want).max()
        assert np.abs(host(cache.state_layer(0, 0)[cache.slot_of[0]]) - S).max() < 1e-4 * np.abs(S).max()
    cache, runner = context_for([CacheGroupSpec("g", StateNeed((H, D, Dv), torch.float32), 1)], "float32", max_requests=2, page_size=8, pages=8)
    ctx, res = step_of(cache, runner, {0: 300})
    got = host(ops.decay_recurrence(dev(z), cache.state_layer(0, 0), powers, ctx, H, D, Dv))
    z64 = z.astype(np.float64)
    s64 = plain.silu(z64)
    want = plain.decayed_recurrence(s64[:, :H * D].reshape(-1, H, D), s64[:, H * D:2 * H * D].reshape(-1, H, D), s64[:, 2 * H * D:].reshape(-1, H, Dv), decay)
    assert np.abs(got - want.reshape(300, H * Dv)).max() < 2e-5 * np.abs(want).max()
    cache.commit(res)


# --------------------------------------------------------------- whole models --

def test_layers_one_by_one_in_32_bit(models):
    """The residual stream after every layer against the plain model."""
    from ayaka_py_b200.replay import ReplaySession
    for tag in CONFIGS:
        folder, cfg, t64, reqs, _ = models[tag]
        toks = list(reqs.values())[2]
        after = []
        plain.forward(cfg, t64, toks, after)
        s = ReplaySession(folder, "float32", 256, PAGE[tag])
        seen = []
        for block in s.model.blocks:
            inner = block.forward
            def outer(x, ctx, caches, inner=inner):
                y = inner(x, ctx, caches)
                seen.append(host(y))
                return y
            block.forward = outer
        s.step({"step": 0, "entries": [{"id": "x", "tokens": toks, "want": [0]}], "end": ["x"]})
        assert len(seen) == len(after) == len(cfg["layers"])
        for i, (got, want) in enumerate(zip(seen, after)):
            assert np.abs(got - want).max() < 1e-4 * max(1.0, float(np.abs(want).max())), (tag, i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C"])
def test_each_request_alone_and_whole(models, tag, dtype):
    check(models, tag, dtype, trace_tools.whole(models[tag][3]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C"])
def test_prefill_against_token_by_token_decoding(models, tag, dtype):
    check(models, tag, dtype, trace_tools.tail_decoded(models[tag][3], 40))
    few = dict(list(models[tag][3].items())[:3])
    check(models, tag, dtype, trace_tools.tail_decoded(few, 10_000), want={k: models[tag][4][k] for k in few})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C"])
def test_portions_down_to_two_tokens(models, tag, dtype):
    check(models, tag, dtype, trace_tools.portions(models[tag][3]))
    check(models, tag, dtype, trace_tools.portions(models[tag][3], sizes=(2, 2, 1, 2, 3, 2)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C"])
def test_mixed_batches_with_pages_and_slots_used_again(models, tag, dtype):
    reqs = dict(models[tag][3])
    extra = {f"{rid}+": toks[::-1] for rid, toks in reqs.items()}      # more requests than slots
    _, cfg, t64, _, want = models[tag]
    want = dict(want)
    want.update({rid: oracle(cfg, t64, toks) for rid, toks in extra.items()})
    reqs.update(extra)
    for seed in (0, 1):
        trace = trace_tools.mixed(reqs, seed=seed)
        assert max(len(s["entries"]) for s in trace) >= 3
        session = check(models, tag, dtype, trace, want=want)
        assert any(g["reused"] > 0 for g in session.cache.stats()["groups"].values())
    longer = {rid: toks for rid, toks in reqs.items() if len(toks) >= 19}
    check(models, tag, dtype, trace_tools.reopened(longer, seed=3), want={rid: want[rid] for rid in longer})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "C"])
def test_long_decoding_past_many_windows(models, tag, dtype):
    folder, cfg, t64, _, _ = models[tag]
    toks = np.random.RandomState(11).randint(0, cfg["vocab"], 420).tolist()
    want = {"long": oracle(cfg, t64, toks)}
    check(models, tag, dtype, trace_tools.tail_decoded({"long": toks}, 400), want=want)


def test_the_batch_does_not_change_a_request(models):
    """A request alone, cut one way, and the same request beside others, cut another way (32-bit)."""
    folder, cfg, _, reqs, _ = models["A"]
    alone = trace_tools.portions({"a4": reqs["a4"]}, sizes=(16, 1, 5))
    out_alone, _ = replay(folder, "float32", alone, 16)
    got_alone = trace_tools.collect(alone, out_alone)["a4"]
    both = trace_tools.mixed(reqs, seed=4)
    out_both, _ = replay(folder, "float32", both, 16)
    got_both = trace_tools.collect(both, out_both)["a4"]
    worst = max(float(np.abs(got_alone[p] - got_both[p]).max()) for p in got_alone)
    assert worst < 5e-5


def test_pages_behind_the_window_come_back(tmp_path):
    """A model of windowed attentions only, a long request in a pool smaller than its length: the pages that no window
    reaches any more are handed out again."""
    cfg = document([attention(4, 2, 12, 16, 37, 8, 0.3, True, dense(40)), attention(2, 2, 12, 16, 37, 4, 0.3, True, None)], 90, 48, side=6)
    tensors = plain.random_tensors(cfg, 77)
    folder = plain.write_folder(tmp_path, cfg, tensors)
    t64 = {k: v.astype(np.float64) for k, v in tensors.items()}
    toks = np.random.RandomState(12).randint(0, cfg["vocab"], 300).tolist()
    want = {"long": plain.forward(cfg, t64, toks)}
    trace = trace_tools.portions({"long": toks}, sizes=(5, 2, 11, 1, 1, 7))
    outputs, session = replay(folder, "float32", trace, 8, max_tokens=320)
    got = trace_tools.collect(trace, outputs)
    assert trace_tools.first_difference(got, want, limit("float32", want)) is None
    stats = session.cache.stats()["groups"]
    assert stats and all(g["high_water"] < 300 // 8 // 2 and g["reused"] > 0 for g in stats.values())


OTHER_SHAPES = {
    # no attention at all: no pages, only state slots
    "only_lightning": document([lightning(9, 11, (0.9, 0.99), dense(33)), lightning(6, 10, (0.4, 0.7, 0.8, 0.9, 1.0), None)], 101, 50, side=3),
    # one layer, one head, a side table of one column per layer, one expert of one
    "smallest": document([attention(1, 1, 2, 1, 5, 2, 0.7, True, moe(1, 1, None, None, 3))], 17, 8, side=1, cap=3.0),
    # a width that is no multiple of 8, heads of 50 and 20, every group kept; two different windows
    "odd_width": document([attention(5, 5, 20, 20, 33, 10, 0.2, True, moe(9, 3, 3, 3, 28)), lightning(50, 50, (0.98, 0.6), dense(77)),
                           attention(10, 5, 16, 20, 64, 6, 0.25, True, dense(64, 0.3))], 257, 100, side=20),
    # values of 256 numbers in the attention and of 320 in the recurrence, keys of 300
    "wide_heads": document([lightning(16, 320, (0.97,), dense(64)), attention(2, 1, 300, 256, 300, 128, 0.06, False, None),
                            lightning(300, 24, (0.93, 0.5), None)], 64, 64, side=16),
    # 32 experts of which 8 are chosen from 2 of 4 groups; 24 in 12 groups of two; two experts, both chosen
    "many_experts": document([attention(2, 1, 64, 64, 128, 64, 0.125, False, moe(32, 8, 4, 2, 32)), lightning(16, 16, [0.5 + 0.06 * i for i in range(8)],
                                                                                                           moe(24, 6, 12, 3, 16)),
                              attention(4, 2, 32, 64, 100, 16, 0.18, True, moe(2, 2, 2, 2, 8))], 512, 128, side=64, cap=50.0),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(OTHER_SHAPES))
def test_other_shapes_whole_decoded_in_portions_and_mixed(tmp_path, name, dtype):
    cfg = OTHER_SHAPES[name]
    tensors = plain.random_tensors(cfg, seed=len(name))
    t64 = {k: v.astype(np.float64) for k, v in tensors.items()}
    rs = np.random.RandomState(1)
    reqs = {f"r{i}": rs.randint(0, cfg["vocab"], n).tolist() for i, n in enumerate([1, 37, 130])}
    want = {rid: oracle(cfg, t64, toks) for rid, toks in reqs.items()}
    folder = plain.write_folder(tmp_path / name, cfg, tensors)
    models = {name: (folder, cfg, t64, reqs, want)}
    PAGE[name] = 16
    for trace in (trace_tools.whole(reqs), trace_tools.tail_decoded(reqs, 40), trace_tools.portions(reqs), trace_tools.mixed(reqs, seed=2)):
        check(models, name, dtype, trace)


# --------------------------------------------- the engine's own entry point --

@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation_through_the_scheduler(models, graphs):
    from ayaka_py_b200.engine.llm import LLM
    from ayaka_py_b200.engine.request import StopCriteria
    from ayaka_py_b200.sampling.params import SamplingParams
    folder, cfg, t64, reqs, _ = models["A"]
    prompts = [reqs["a2"], reqs["a3"][:40], reqs["a0"], reqs["a3"][5:30], reqs["a1"], reqs["a4"][:70]]
    llm = LLM(folder, dtype="float32", kv_pages=24, page_size=16, max_requests=3, batch_tokens=48, prefill_chunk=20,
              max_model_len=128, decode_graph=graphs)
    results = llm.generate(prompts, SamplingParams(temperature=0.0), StopCriteria(max_tokens=12, ignore_eos=True))
    for prompt, result in zip(prompts, results):
        want = plain.greedy_generate(cfg, t64, prompt, 12)
        k = next((i for i, (a, b) in enumerate(zip(result.token_ids, want)) if a != b), None)
        if k is not None:                     # a near tie may turn a token
            logits = plain.forward(cfg, t64, prompt + want[:k])[-1]
            assert abs(logits[result.token_ids[k]] - logits[want[k]]) < 1e-3
        else:
            assert result.token_ids == want
    llm.engine.cache.assert_clean()


def test_bfloat16_generation_with_decode_graphs_equals_eager(models):
    from ayaka_py_b200.engine.llm import LLM
    from ayaka_py_b200.engine.request import StopCriteria
    from ayaka_py_b200.sampling.params import SamplingParams
    folder, cfg, _, reqs, _ = models["C"]
    prompts = [reqs["c1"], reqs["c0"], reqs["c2"][:33]]
    out = []
    for graphs in (True, False):
        llm = LLM(folder, dtype="bfloat16", kv_pages=40, page_size=16, max_requests=4, max_model_len=160, decode_graph=graphs)
        out.append([r.token_ids for r in llm.generate(prompts, SamplingParams(temperature=0.0),
                                                      StopCriteria(max_tokens=16, ignore_eos=True))])
    assert out[0] == out[1]


def test_random_weights_mode_and_command_line(tmp_path):
    """A folder written by the engine's own random-weights mode loads, generates from the command line and replays a trace."""
    import subprocess
    import sys
    from pathlib import Path
    from ayaka_py_b200.config.model import MurutarConfig
    from ayaka_py_b200.weights import write_random_model
    folder = write_random_model(tmp_path / "m", MurutarConfig.from_dict(CONFIG_B), seed=3)
    assert json.loads((folder / "config.json").read_text())["architecture"] == "Murutar"
    root = Path(__file__).resolve().parent.parent
    proc = subprocess.run([sys.executable, "-m", "ayaka_py_b200", "generate", str(folder), "--prompt-ids", "1,2,3,4,5",
                           "--max-tokens", "5", "--temperature", "0", "--ignore-eos", "--max-model-len", "64", "--kv-pages", "16"],
                          cwd=root, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    line = json.loads(proc.stdout.strip().splitlines()[-1])
    assert len(line["token_ids"]) == 5
    steps = "\n".join(json.dumps(s) for s in [{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []},
                                              {"step": 1, "entries": [{"id": "a", "tokens": [9], "want": [0]}], "end": ["a"]}])
    proc = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path / "out"),
                           "--max-tokens", "64"], input=steps + "\n", cwd=root, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert "done 0" in proc.stdout and "done 1" in proc.stdout
    assert np.fromfile(tmp_path / "out" / "0.f32", dtype="<f4").shape == (2 * CONFIG_B["vocab"],)
