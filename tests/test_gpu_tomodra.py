"""Tomodra: every mechanism alone against the plain functions of ``plain_tomodra``, then whole models of several
shapes replayed whole, decoded, in portions and mixed, and greedy generation through the engine's own entry point."""

import copy
import json
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_tomodra as plain
import trace_tools
from test_gpu_vedadra import DT, bind, context_for, dev, host, mixer_alone, standing_out_rows, step_of, tol

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ configs --

def moe(experts, top, ff, shared):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def yarn(factor, original, fast=32.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention(heads, kv, dim, vdim, size, rot, scale, mlp, base=10000.0, scaling=None):
    mixer = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}
    if scaling is not None:
        mixer["rot"]["scaling"] = scaling
    if size is not None:
        mixer["mask"] = {"size": size}
    return {"type": "attention", "mlp": mlp, "mixer": mixer}


def latent(heads, dim, rot_dim, vdim, rank, size, scale, mlp, base=10000.0, kv_from=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
             "rot": {"base": base, "dims": rot_dim}}
    if size is not None:
        mixer["mask"] = {"size": size}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": mlp, "mixer": mixer}


def document(layers, vocab, width, alpha=1.5, eps=1e-5):
    return {"architecture": "Tomodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": layers}


# A: odd sizes that only the plain kernels take; a latent read by two later layers of other head counts, a longer and a
# shorter window, with other layers between; layers without feed-forward; chunk and windows that are no multiple of a page.
CONFIG_A = document([latent(3, 10, 6, 14, 20, 11, 0.3, moe(6, 2, 20, 28)), attention(4, 2, 20, 12, 23, 12, 0.22, moe(5, 1, 24, 16), scaling=yarn(4.0, 50)),
                     latent(5, 7, 6, 9, 20, 29, 0.35, None, kv_from=0), attention(2, 1, 12, 28, 7, 2, 0.3, None),
                     latent(2, 16, 6, 12, 20, 4, 0.3, moe(4, 3, 12, 8), kv_from=0)], vocab=211, width=72)
# B: every head with keys of its own; a chunk and a window of one token (a query sees itself, and the sink); no masks at
# all; every expert chosen; no shared expert; the stream's factor 1 and below; a latent next to its reader.
CONFIG_B = document([attention(4, 4, 16, 16, 1, 8, 0.25, moe(4, 4, 24, 0)), latent(2, 32, 8, 16, 40, 1, 0.2, None),
                     latent(6, 8, 8, 24, 40, None, 0.25, moe(3, 1, 32, 40), kv_from=1), attention(3, 3, 16, 40, None, 16, 0.25, None, base=500.0),
                     latent(1, 24, 2, 20, 12, 1000, 0.2, moe(8, 2, 16, 12), base=50.0)], vocab=130, width=64, alpha=1.0)
# C: sizes of the tensor-core kernels (heads of 64 and 128, eight query heads on two key/value heads, a latent of 128),
# windows and chunks of a few pages, sixteen experts.
CONFIG_C = document([attention(8, 2, 64, 128, 80, 32, 0.125, moe(16, 2, 64, 96), scaling=yarn(8.0, 64, 8.0)), latent(8, 64, 32, 64, 128, 70, 0.1, moe(16, 4, 64, 128)),
                     latent(4, 128, 32, 128, 128, 48, 0.08, moe(16, 1, 96, 64), kv_from=1), attention(4, 2, 128, 64, 48, 128, 0.09, None),
                     latent(16, 32, 16, 32, 64, 33, 0.14, moe(8, 2, 128, 64), base=500000.0)], vocab=300, width=128, alpha=2.5, eps=1e-6)
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
    base = tmp_path_factory.mktemp("tomodra")
    out = {}
    for tag, cfg in CONFIGS.items():
        tensors = plain.random_tensors(cfg, seed=70 + ord(tag))
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
    """In 32-bit every position must agree.  In bfloat16 rounding can turn a router's close call, which moves that
    position's logits visibly and, through the caches, later ones a little: the places that the plain model marks as close
    calls are not compared, and of the others at most 2 in 100 may differ, which a wrong page or a wrong edge would
    exceed at once."""
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


def layer_tensors(layer, d, seed, prefix="l0.mix."):
    t = plain.random_tensors(document([layer], 4, d), seed)
    return {k: v.astype(np.float64) for k, v in t.items()}, {k[len(prefix):]: v for k, v in t.items() if k.startswith(prefix)}


def put(t64, w, prefix="l0.mix."):
    for name, v in w.items():
        t64[prefix + name] = v.astype(np.float64)


def make(kind, params, dtype):
    from ayaka_py_b200.parts import PartSpec, make_part
    return make_part(PartSpec(kind, params), DT[dtype], "cuda")


# ----------------------------------------------------------- the normed sum --

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d", [72, 64, 6, 1537, 1, 2048, 4096, 5000])
def test_norm_of_the_sum_with_the_stream_and_what_follows(dtype, d):
    """x = norm(a x + y) with y a row; the rows of chosen experts (in order and at places of their own), weighted or as
    they are; the shared expert's row beside them, as it is and behind a gate.  From the same kernel a copy or a norm."""
    from ayaka_py_b200 import ops
    rs = np.random.RandomState(d)
    for n, a in ((1, 1.0), (37, 2.25), (5, 0.0)):
        x, y = rs.randn(n, d).astype(np.float32) * 2, rs.randn(n, d).astype(np.float32) * 3
        w, w2 = (1.0 + 0.2 * rs.randn(d)).astype(np.float32), (1.0 + 0.2 * rs.randn(d)).astype(np.float32)
        eps, top = 3e-2, 3                                                   # an eps that matters
        rows, weights = rs.randn(n * top, d).astype(np.float32), rs.rand(n, top).astype(np.float32)
        wide = rs.randn(n, 5).astype(np.float32) * 2
        place = rs.permutation(n * top + 5)[:n * top].astype(np.int32)
        spread = np.full((n * top + 5, d), np.nan, dtype=np.float32)
        spread[place] = rows
        route = SimpleNamespace(weights=dev(weights), top=top)
        p64, y64 = rows.astype(np.float64).reshape(n, top, d), y.astype(np.float64)
        gate = plain.sigmoid(wide[:, 3:4].astype(np.float64))
        cases = [(dev(y), y64), (ops.PickedRows(dev(rows), route, None), np.einsum("nk,nkd->nd", weights.astype(np.float64), p64)),
                 (ops.PickedRows(dev(rows), route, None, weighted=False), p64.sum(axis=1)),
                 (ops.PickedRows(dev(spread), route, torch.from_numpy(place).cuda(), weighted=False, shared=dev(y)), p64.sum(axis=1) + y64),
                 (ops.PickedRows(dev(spread), route, torch.from_numpy(place).cuda(), shared=dev(y), mix=dev(wide)[:, 3]),
                  np.einsum("nk,nkd->nd", weights.astype(np.float64), p64) + gate * y64)]
        for result, value in cases:
            want = plain.rms_norm(a * x.astype(np.float64) + value, w.astype(np.float64), eps)
            stream = dev(x)
            assert ops.stream_update(stream, result, dev(w), factor=a, eps=eps) is None
            assert np.abs(host(stream) - want).max() < 2e-5 * max(1.0, np.abs(want).max())
            for post, expect in (("copy", want), ("rmsnorm", plain.rms_norm(want, w2.astype(np.float64), 1e-3))):
                stream = dev(x)
                got = ops.stream_update(stream, result, dev(w), factor=a, eps=eps, post=post, next_weight=dev(w2), next_eps=1e-3, out_dtype=DT[dtype])
                assert got.dtype == DT[dtype] and np.abs(host(stream) - want).max() < 2e-5 * max(1.0, np.abs(want).max())
                assert np.abs(host(got) - expect).max() < (5e-5 if dtype == "float32" else 1e-2) * max(1.0, np.abs(expect).max())
        part = make("rmsnorm", {"width": d, "eps": eps, "stream_factor": a}, dtype)
        part.bind({"weight": dev(w)})
        copy_ = make("stream_copy", {"width": d}, dtype)
        stream = dev(x)
        h = part.sum_normed(stream, dev(y), copy_, None)
        assert h.dtype == DT[dtype] and np.array_equal(host(h), host(copy_.forward(stream, None)))
        # the same kernel's other forms take rows of chosen experts beside a shared one too
        s, gates = rs.randn(d).astype(np.float32), rs.randn(n, d).astype(np.float32)
        stream = dev(x)
        ops.stream_update(stream, cases[4][0], dev(s), gate=dev(gates))
        assert np.abs(host(stream) - (x + cases[4][1] * s * plain.sigmoid(gates.astype(np.float64)))).max() < 1e-4


# ------------------------------------------------------------------ experts --

def moe_part(mlp, d, dtype, **kw):
    shared = (mlp.get("shared") or {}).get("ff", 0)
    return make("moe", {"width": d, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "inner": mlp["expert"]["ff"], "limit": None,
                        "shared_inner": shared, "shared_limit": None, "router": "sigmoid", "slope": 1.0, "plus": 0.0, "weigh": "input", **kw}, dtype)


def moe_names(mlp):
    names = {"router": "router_weight"}
    if mlp.get("shared"):
        names.update({"shared.gate": "shared_gate", "shared.up": "shared_up", "shared.down": "shared_down", "shared.sg": "shared_mix"})
    for e in range(mlp["router"]["experts"]):
        names.update({f"e{e}.gate": f"gate_{e}", f"e{e}.up": f"up_{e}", f"e{e}.down": f"down_{e}"})
    return names


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,E,top,ff,sf", [(48, 8, 1, 16, 24), (48, 6, 2, 20, 12), (40, 5, 5, 24, 0), (64, 16, 4, 64, 96), (128, 12, 3, 72, 7), (36, 9, 2, 15, 30),
                                           (64, 40, 8, 16, 8)])
def test_experts_with_weighted_inputs_alone(dtype, d, E, top, ff, sf):
    """Routing and output for a single token, a few and many (the experts' products run through different kernels), as a
    sum and as rows.  The weights in front of the experts: behind them the result is another."""
    from ayaka_py_b200 import ops
    mlp = moe(E, top, ff, sf)
    t64, w = layer_tensors(latent(1, 4, 2, 4, 4, 4, 1.0, mlp), d, 100 + E, prefix="l0.mlp.")
    part = moe_part(mlp, d, dtype)
    bind(part, w, moe_names(mlp), dtype)
    rs = np.random.RandomState(E)
    for n in (1, 7, 150):
        h = plain.round_bf16(rs.randn(n, d).astype(np.float32) * 1.5)
        margins = []
        want = plain.moe_ff(h.astype(np.float64), t64, "l0.mlp.", mlp, margins)
        clear = margins[0] > 1e-4
        z = h.astype(np.float64) @ t64["l0.mlp.router"].T
        route = ops.moe_route(dev(z.astype(np.float32)), E, top, {"normalize": False})
        for t in np.flatnonzero(clear):
            chosen, wt = plain.route(z[t], top)
            assert route.ids[t].tolist() == chosen and np.abs(host(route.weights[t]) - wt).max() < 1e-6
        x = dev(h, DT[dtype])
        big = float(np.abs(want).max())
        ctx = SimpleNamespace(carry={})
        assert np.abs(host(part.forward(x, None, ctx)) - want)[clear].max() < tol(dtype, 4 * big), n
        stream = dev(h)
        ops.stream_update(stream, part.forward_rows(x, ctx), torch.ones(d, device="cuda"), factor=1.5, eps=1e-5)
        normed = plain.rms_norm(1.5 * h.astype(np.float64) + want, 1.0, 1e-5)
        assert np.abs(host(stream) - normed)[clear].max() < tol(dtype, 4.0), n
        assert clear.mean() > 0.9
        behind = moe_part(mlp, d, dtype, weigh="output")
        bind(behind, w, moe_names(mlp), dtype)
        assert np.abs(host(behind.forward(x, None, ctx)) - want).max() > 10 * tol("float32", 4 * big) + (0.02 * big if n > 1 else 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_form_of_the_experts_products_weights_its_rows(dtype):
    """The same pairs through each kernel that the dtype has; weights that differ widely."""
    from ayaka_py_b200 import ops
    rs = np.random.RandomState(6)
    d, E, ff, n, top = 64, 5, 40, 90, 2
    h = plain.round_bf16(rs.randn(n, d).astype(np.float32))
    w_in, w_down = (plain.round_bf16(rs.randn(*s).astype(np.float32) / 8) for s in ((E, 2 * ff, d), (E, d, ff)))
    logits = (rs.randn(n, E) * 4 - 2).astype(np.float32)
    route = ops.moe_route(dev(logits), E, top, {"normalize": False})
    ids, wt = route.ids.cpu().numpy(), host(route.weights)
    want = np.zeros((n, top, d))
    for t in range(n):
        for k in range(top):
            g, u = wt[t, k] * h[t].astype(np.float64) @ w_in[ids[t, k], :ff].T, wt[t, k] * h[t].astype(np.float64) @ w_in[ids[t, k], ff:].T
            want[t, k] = (g * plain.sigmoid(g) * u) @ w_down[ids[t, k]].T
    assert wt.min() < 0.1 and wt.max() > 0.9
    x, a, b = dev(h, DT[dtype]), dev(w_in, DT[dtype]), dev(w_down, DT[dtype])
    glu = (float("inf"), 1.0, 0.0)
    forms = {"tiles": ops.moe_gemm(ops.moe_gemm(x, a, route, glu, DT[dtype], weigh_input=True), b, route, None, torch.float32)}
    if dtype == "bfloat16":
        forms["pairs"] = ops.moe_gemv(ops.moe_gemv(x, a, route, glu, weigh_input=True), b, route, None)
        rows, where = ops.moe_experts_tc(x, a, b, route, *glu, weigh_input=True)
        forms["tcgen05"] = rows[where.long()]
    for form, got in forms.items():
        assert np.abs(host(got).reshape(n, top, d) - want).max() < tol(dtype, 2 * np.abs(want).max()), form


def test_routing_where_scores_saturate():
    """Experts are ranked by their logits, so also among scores that are 1 or 0 in 32-bit."""
    from ayaka_py_b200 import ops
    z = np.array([[40.0, -200.0, 60.0, 50.0, -150.0, -300.0], [-150.0, -140.0, -160.0, -130.0, -170.0, -180.0]], dtype=np.float32)
    route = ops.moe_route(dev(z), 6, 4, {"normalize": False})
    assert route.ids.cpu().numpy().tolist() == [[2, 3, 0, 4], [3, 1, 0, 2]]
    assert host(route.weights).tolist() == [[1.0, 1.0, 1.0, 0.0], [0.0, 0.0, 0.0, 0.0]]


# --------------------------------------------------------- latent attention --

LAT_NAMES = {"q": "q_weight", "dkv": "down_weight", "dkv.norm": "down_norm", "uk": "uk_weight", "uv": "uv_weight", "o": "out_weight"}


def latent_part(layer, d, dtype, own=True, eps=1e-5):
    mx = layer["mixer"]
    return make("latent_attention", {"width": d, "heads": mx["heads"], "dim": mx["dim"], "rot_dim": mx["rot_dim"], "vdim": mx["vdim"],
                                     "kv_rank": mx["kv_rank"], "scale": mx["scale"], "eps": eps, "rot": dict(mx["rot"], layout="halves"), "gate": None,
                                     "window": (mx.get("mask") or {}).get("size"), "own_latent": own}, dtype)


def plain_latent(layer, t64, eps=1e-5):
    return lambda h: plain.latent_attention(h, t64, "l0.mix.", layer["mixer"], eps, plain.latent_of(h, t64, "l0.mix.", layer["mixer"], eps))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,R,Dv,rank,size", [(3, 10, 6, 14, 20, 11), (4, 64, 32, 64, 128, 40), (1, 24, 2, 20, 12, 1), (6, 16, 8, 24, 40, None),
                                                (8, 32, 16, 48, 64, 33), (2, 24, 8, 40, 256, 130), (40, 8, 8, 8, 32, 64), (16, 16, 16, 16, 272, 1000),
                                                (5, 12, 4, 8, 36, 32), (2, 128, 64, 128, 512, 96)])
def test_windowed_latent_attention_alone(dtype, H, D, R, Dv, rank, size):
    d = 48
    layer = latent(H, D, R, Dv, rank, size, 1.5 / np.sqrt(D + R), None)
    t64, w = layer_tensors(layer, d, 53)
    part = latent_part(layer, d, dtype)
    assert "gate_weight" not in part.tensors()
    bind(part, w, LAT_NAMES, dtype)
    mixer_alone(part, dtype, d, plain_latent(layer, t64), {0: 150, 1: 9, 2: 70})


def latent_edge_weights(rs, layer, d, seed):
    """Tensors of a layer whose score of query i and key j is about gain * c_i . c_j, without a rotated part in it."""
    mx = layer["mixer"]
    H, D, R, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"]
    t64, w = layer_tensors(layer, d, seed)
    uk = np.linalg.qr(rs.randn(rank, rank))[0][:D].astype(np.float32)
    w["uk"] = plain.round_bf16(np.tile(uk, (H, 1)) * 4)
    q = np.zeros((H, D + R, d), dtype=np.float32)
    q[:, :D] = (uk.astype(np.float64) * 4 @ w["dkv"][:rank].astype(np.float64)).astype(np.float32)
    w["q"] = plain.round_bf16(q.reshape(H * (D + R), d))
    w["dkv.norm"][:] = 1
    put(t64, w)
    return t64, w


def edge_places(P, size, n):
    """The first tokens, page borders, keys just inside and just outside the windows of the last queries, and the end."""
    out = {0, 2, P - 1, P, P + 1, 5 * P - 1, 5 * P, n - 1, n - 2, n - size, n - size - 1, n - size + 1, n - 3}
    return sorted(p for p in out if 0 <= p < n)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,R,Dv,rank,size", [(2, 16, 8, 24, 32, 37), (4, 24, 6, 12, 28, 24), (3, 32, 16, 64, 128, 129), (2, 16, 8, 16, 64, 1000), (8, 32, 32, 32, 64, 32)])
def test_latents_that_stand_out_at_window_and_page_borders(dtype, H, D, R, Dv, rank, size):
    """Chosen places score high against one another, in prompts and in decoding.  A window that is one position longer or
    shorter gives another output at a checked place."""
    rs = np.random.RandomState(19)
    d, P = 48, 8
    layer = latent(H, D, R, Dv, rank, size, 0.15 / D if size < 330 else 0.4 / D, None)
    t64, w = latent_edge_weights(rs, layer, d, 59)
    part = latent_part(layer, d, dtype)
    bind(part, w, LAT_NAMES, dtype)
    lengths = {0: 330, 1: 9, 2: 70}
    places = {0: edge_places(P, size, 330) if size < 330 else [7, 8, 5 * P - 1, 328], 1: [0, 8], 2: [3, 2 * P, 69]}
    rows = {i: standing_out_rows(rs, n, d, places[i]) for i, n in lengths.items()}
    want = mixer_alone(part, dtype, d, plain_latent(layer, t64), lengths, rows=rows, page_size=P)
    for other_size in (size + 1, size - 1) if size < 330 else ():
        changed = dict(layer, mixer=dict(layer["mixer"], mask={"size": other_size}))
        other = plain_latent(changed, t64)(rows[0].astype(np.float64))
        assert max(np.abs(other[p] - want[0][p]).max() for p in (329, 328)) > 0.01 * np.abs(want[0]).max(), other_size
    if size >= 330:                                             # without a far key the output at 328 is another
        x = rows[0].astype(np.float64).copy()
        x[7] = rs.randn(d)
        assert np.abs(plain_latent(layer, t64)(x)[328] - want[0][328]).max() > 0.01 * np.abs(want[0]).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("own_size,size,H,D,Dv,rank,R", [(20, 45, 5, 7, 9, 20, 6), (45, 20, 3, 32, 40, 64, 16), (30, None, 2, 16, 24, 40, 8), (None, 12, 8, 64, 32, 128, 32),
                                                         (16, 16, 4, 24, 16, 24, 8)])
def test_a_layer_that_reads_anothers_latent(dtype, own_size, size, H, D, Dv, rank, R):
    """Queries, up-projections, head count and window of its own over what the other layer cached of another input; the
    cache keeps what the longer window needs, whichever layer has it."""
    d = 48
    first = latent(3, 12, R, 10, rank, own_size, 0.3, None)
    second = latent(H, D, R, Dv, rank, size, 1.5 / np.sqrt(D + R), None)
    t1, w1 = layer_tensors(first, d, 61)
    t2, w2 = layer_tensors(dict(second, mixer=dict(second["mixer"], kv_from=0)), d, 67)
    assert "dkv" not in w2
    one, two = latent_part(first, d, dtype), latent_part(second, d, dtype, own=False)
    assert set(two.tensors()) == {"q_weight", "uk_weight", "uv_weight", "out_weight"}
    bind(one, w1, LAT_NAMES, dtype)
    bind(two, w2, LAT_NAMES, dtype)
    turn = np.random.RandomState(7).permutation(d)              # the second layer's input is another row

    class Pair:
        def cache_need(self):
            return one.cache_need().together(two.cache_need())

        def forward(self, x, residual, ctx, binding):
            from ayaka_py_b200.cache import CacheBinding
            one.forward(x, None, ctx, binding)
            return two.forward(x[:, torch.from_numpy(turn).cuda()].contiguous(), residual, ctx, CacheBinding(binding.group, binding.name, binding.layer, writes=False))

    def want(h):
        return plain.latent_attention(h[:, turn], t2, "l0.mix.", second["mixer"], 1e-5, plain.latent_of(h, t1, "l0.mix.", first["mixer"], 1e-5))
    mixer_alone(Pair(), dtype, d, want, {0: 150, 1: 9, 2: 70})


def test_the_latent_is_made_exactly_where_it_is_kept():
    from ayaka_py_b200.cache import CacheBinding
    layer = latent(2, 8, 4, 8, 16, None, 0.3, None)
    for own, writes in ((True, False), (False, True)):
        with pytest.raises(ValueError):
            latent_part(layer, 16, "float32", own=own).forward(torch.zeros(1, 16, device="cuda"), None, None, CacheBinding(0, "g", 0, writes))


@pytest.mark.parametrize("H,rank,rot,P", [(4, 72, 24, 16), (16, 512, 64, 16), (6, 40, 8, 8), (40, 32, 8, 16), (1, 264, 24, 16)])
@pytest.mark.parametrize("window", [1, 32, 40, 100, 500, 1000])
def test_tensor_core_latent_attention_in_windows_against_the_32_bit_pipes(H, rank, rot, P, window):
    """Prompts, portions on top of a cached context, single rows (whose window is cut into partitions and merged): both
    kernels read the same pages; positions hundreds of tokens on, windows of one partition and of many."""
    from ayaka_py_b200 import ops
    from ayaka_py_b200.cache import CacheGroupSpec
    from ayaka_py_b200.parts import KVNeed
    cache, runner = context_for([CacheGroupSpec("g", KVNeed(1, rot, None, 1, rank), 1)], "bfloat16", max_requests=4, page_size=P, pages=2048 // P,
                                positions=1024)
    rope, lat = (pages[:, :, 0] for pages in cache.kv_layer(0, 0))
    gen = torch.Generator(device="cuda").manual_seed(1)
    for pages in (lat, rope):
        pages.copy_(torch.randn(pages.shape, generator=gen, device="cuda"))
    for plan in ({0: 500, 1: 33, 2: 1}, {0: 7, 2: 130}, {0: 1, 1: 1, 2: 1}, {1: 1}, {0: 64, 1: 1, 2: 1, 3: 17}, {0: 1, 1: 1, 2: 1, 3: 1}):
        ctx, res = step_of(cache, runner, plan)
        q = torch.randn(ctx.num_rows, H, rank + rot, generator=gen, device="cuda") * 0.5
        a = ops.latent_attention(q, lat, rope, ctx.tables[0], ctx, 0.2, tensor_cores=False, window=window)
        b = ops.latent_attention(q, lat, rope, ctx.tables[0], ctx, 0.2, tensor_cores=True, window=window)
        assert not torch.isnan(b).any()
        assert float((a - b).abs().max()) < 0.01 * float(a.abs().max()) + 1e-3, plan
        if window == 1:                                          # a row sees itself alone
            table = cache.table_rows(0, [cache.slot_of[i] for i in plan])
            own = {i: int(cache.length[cache.slot_of[i]]) for i in plan}
            order = [list(plan)[int(k)] for k in ctx.host["order"]]
            at = 0
            for i in order:
                for e in range(plan[i]):
                    p = own[i] + e
                    cell = lat[int(table[list(plan).index(i)][p // P]), p % P].float()
                    assert float((a[at] - cell).abs().max()) < 1e-4
                    at += 1
        cache.commit(res)


def test_both_layouts_of_the_rotated_part():
    """Every pair of queries and of the shared key part at far positions, one base for which the slow pairs hardly move
    and one for which all do; with and without writing."""
    from ayaka_py_b200 import ops
    from ayaka_py_b200.cache import CacheGroupSpec
    from ayaka_py_b200.parts import KVNeed
    from ayaka_py_b200.parts.position import rotary_frequencies
    rs = np.random.RandomState(2)
    for H, D, R, rank, dims, base, scaling in ((3, 5, 8, 12, 8, 1e4, None), (1, 4, 6, 40, 4, 3.0, None), (2, 16, 64, 24, 64, 5e5, yarn(4.0, 100))):
        n, rot = 600, {"dims": dims, "base": base, "scaling": scaling}
        f, gain = rotary_frequencies(dims, base, scaling)
        freq = torch.tensor(f, dtype=torch.float64).float().cuda()
        proj = rs.randn(n, H * (D + R) + rank + R + 2).astype(np.float32)
        w = (1.0 + 0.2 * rs.randn(rank)).astype(np.float32)
        q64 = proj[:, :H * (D + R)].astype(np.float64).reshape(n, H, D + R)[:, :, D:]
        down = proj[:, H * (D + R):].astype(np.float64)
        for halves in (True, False):
            cache, runner = context_for([CacheGroupSpec("g", KVNeed(1, R, None, 1, rank), 1)], "float32", max_requests=2, page_size=8, pages=128)
            ctx, res = step_of(cache, runner, {0: n})
            rope, lat = cache.kv_layer(0, 0)
            turn = plain.rotate_halves if halves else plain.rotate_neighbours
            query = ops.latent_prepare(dev(proj), lat, rope, dev(w), freq, gain, dims, ctx, ctx.tables[0], H, D, R, rank, 1e-4, True, halves)
            assert np.abs(host(query)[:, :, rank:] - turn(q64, rot)).max() < 3e-4
            table = cache.table_rows(0, [cache.slot_of[0]])[0]
            cells = [(int(table[p // 8]), p % 8, 0) for p in range(n)]
            assert np.abs(np.stack([host(rope[c]) for c in cells]) - turn(down[:, None, rank:rank + R], rot)[:, 0]).max() < 3e-4
            assert np.abs(np.stack([host(lat[c]) for c in cells]) - plain.rms_norm(down[:, :rank], w.astype(np.float64), 1e-4)).max() < 2e-5
            before = rope.clone(), lat.clone()
            again = ops.latent_prepare(dev(proj[:, :H * (D + R)]), lat, rope, None, freq, gain, dims, ctx, ctx.tables[0], H, D, R, rank, 1e-4, False, halves)
            assert torch.equal(again[:, :, rank:], query[:, :, rank:]) and torch.equal(rope, before[0]) and torch.equal(lat, before[1])
            cache.commit(res)


# -------------------------------------------------------- chunked attention --

ATT_NAMES = {"q": "q_weight", "k": "k_weight", "v": "v_weight", "q.norm": "q_norm", "k.norm": "k_norm", "sink": "sink", "o": "out_weight"}


def attention_part(layer, d, dtype, eps=1e-5):
    mx = layer["mixer"]
    return make("rotary_attention", {"width": d, "heads": mx["heads"], "kv_heads": mx["kv_heads"], "dim": mx["dim"], "vdim": mx["vdim"],
                                     "scale": mx["scale"], "rot": dict(mx["rot"], layout="interleaved"), "chunk": (mx.get("mask") or {}).get("size"),
                                     "sink": "learned", "qk_norm_eps": eps}, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv,size,rot,scaling", [(4, 2, 20, 12, 23, 12, yarn(4.0, 50)), (3, 3, 16, 40, 1, 16, None), (4, 1, 8, 16, None, 2, None),
                                                       (8, 2, 64, 128, 80, 32, yarn(8.0, 64, 8.0)), (2, 2, 12, 28, 7, 6, yarn(2.0, 20, 4.0, 2.0)),
                                                       (4, 4, 32, 32, 130, 24, None), (2, 1, 128, 64, 1000, 128, yarn(16.0, 128)), (5, 1, 16, 256, 16, 8, None),
                                                       (16, 2, 32, 32, 64, 20, None)])
def test_chunked_attention_with_head_norms_and_learned_sinks_alone(dtype, H, G, D, Dv, size, rot, scaling):
    d = 48
    layer = attention(H, G, D, Dv, size, rot, 2.0 / np.sqrt(D), None, base=500.0, scaling=scaling)
    t64, w = layer_tensors(layer, d, 29)
    w["sink"] = plain.round_bf16(np.linspace(-3.0, 3.0, H).astype(np.float32))      # a sink that counts, another for every head
    put(t64, w)
    part = attention_part(layer, d, dtype)
    bind(part, w, ATT_NAMES, dtype)
    fn = lambda h: plain.attention(h, t64, "l0.mix.", layer["mixer"], 1e-5)
    want = mixer_alone(part, dtype, d, fn, {0: 150, 1: 9, 2: 70})
    without = dict(t64)
    without["l0.mix.sink"] = np.full(H, -1e9)
    assert np.abs(plain.attention(np.random.RandomState(5).randn(20, d), without, "l0.mix.", layer["mixer"], 1e-5) -
                  fn(np.random.RandomState(5).randn(20, d))).max() > 0.01 * np.abs(want[0]).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv,size,gain", [(4, 2, 20, 12, 41, 6.0), (8, 2, 64, 128, 80, 6.0), (2, 1, 32, 64, 1000, 6.0), (4, 1, 16, 16, 24, 6.0), (3, 3, 16, 24, 109, 6.0)])
def test_keys_that_stand_out_at_chunk_and_page_borders(dtype, H, G, D, Dv, size, gain):
    """Keys made from the queries' matrix at chosen places score high against one another; chunks that are one position
    longer or shorter give another output right behind a border, in prompts and in decoding."""
    rs = np.random.RandomState(17)
    d, P, n = 48, 8, 330
    layer = attention(H, G, D, Dv, size, 2, gain / D, None, base=2.0)
    t64, w = layer_tensors(layer, d, 37)
    q = w["q"].reshape(H, D, d)
    q[:, :2] = 0                                              # nothing on the dimensions that turn
    w["q"] = q.reshape(H * D, d)
    w["k"] = q[::H // G].reshape(G * D, d).copy()
    w["q.norm"][:], w["k.norm"][:] = 1, 1
    w["sink"][:] = -1.0
    put(t64, w)
    part = attention_part(layer, d, dtype)
    bind(part, w, ATT_NAMES, dtype)
    last = n // size * size
    places = {p for p in (0, 2, P - 1, P, 5 * P - 1, 5 * P, last - 2, last - 1, last, last + 1, n - 2, n - 1) if 0 <= p < n}
    lengths = {0: n, 1: 9, 2: 70}
    spots = {0: sorted(places), 1: [0, 8], 2: [3, 2 * P, 69]}
    rows = {i: standing_out_rows(rs, m, d, spots[i]) for i, m in lengths.items()}
    want = mixer_alone(part, dtype, d, lambda h: plain.attention(h, t64, "l0.mix.", layer["mixer"], 1e-5), lengths, rows=rows, page_size=P)
    if size < n:
        for other_size in (size + 1, size - 1):
            changed = copy.deepcopy(layer["mixer"])
            changed["mask"]["size"] = other_size
            other = plain.attention(rows[0].astype(np.float64), t64, "l0.mix.", changed, 1e-5)
            assert max(np.abs(other[p] - want[0][p]).max() for p in (last - 1, last, last + 1)) > 0.01 * np.abs(want[0]).max(), other_size


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,chunk", [(None, 1), (None, 5), (None, 64), (None, 200), (None, 333), (70, 100), (100, 70), (None, None)])
def test_decode_steps_read_the_parts_of_their_own_chunk(dtype, window, chunk):
    """Single rows at positions around chunk borders, hundreds of tokens on: the parts counted from the chunk's (or the
    window's) first key are the whole of what a row sees; a sink counts once."""
    from ayaka_py_b200 import ops
    from ayaka_py_b200.cache import CacheGroupSpec
    from ayaka_py_b200.parts import KVNeed
    H, G, D, Dv, n = 4, 2, 32, 32, 420
    rs = np.random.RandomState(8)
    q, k, v = (plain.round_bf16(rs.randn(n, h, e).astype(np.float32)) for h, e in ((H, D), (G, D), (G, Dv)))
    sinks = np.array([-2.0, 0.0, 1.0, 4.0], dtype=np.float32)
    of = np.arange(H) // 2
    s = np.einsum("ihd,jhd->hij", q.astype(np.float64), k.astype(np.float64)[:, of]) * 0.4
    p = plain.softmax(s, plain.window_mask(n, window) & plain.chunk_mask(n, chunk), sinks.astype(np.float64))
    want = np.einsum("hij,jhd->ihd", p, v.astype(np.float64)[:, of]).reshape(n, H * Dv)
    cache, runner = context_for([CacheGroupSpec("g", KVNeed(G, D, value_heads=G, value_dim=Dv), 1)], dtype, max_requests=2, page_size=8, pages=128)
    kp, vp = cache.kv_layer(0, 0)
    size, at = chunk or 64, 0
    cuts = []
    for border in range(size, n, size) if size > 40 else (40, 200, 390):
        cuts += [border - 2 - sum(cuts)] + [1] * 4 if border - 2 > sum(cuts) else []
    cuts += [n - 3 - sum(cuts), 1, 1, 1]
    for count in cuts:
        ctx, res = step_of(cache, runner, {0: count})
        rows = slice(at, at + count)
        ops.kv_append(kp, vp, dev(k[rows].reshape(count, -1), DT[dtype]), dev(v[rows].reshape(count, -1), DT[dtype]), ctx.row_req, ctx.positions,
                      ctx.tables[0])
        for tensor_cores in (True, False):
            got = ops.grouped_attention(dev(q[rows].reshape(count, -1), DT[dtype]), kp, vp, ctx.tables[0], ctx, heads=H, key_heads=G, key_dim=D,
                                        scale=0.4, window=window, chunk=chunk, sinks=dev(sinks), tensor_cores=tensor_cores)
            assert np.abs(host(got) - want[rows]).max() < (3e-5 if dtype == "float32" else 2e-2) * np.abs(want).max(), (at, count, tensor_cores)
        cache.commit(res)
        at += count
    assert at == n


def test_head_norms_and_rotation_of_every_pair():
    """Queries and keys at far positions in both layouts, with and without norms, with stretched frequencies and a gain;
    sizes of the vector and of the scalar form."""
    from ayaka_py_b200 import ops
    from ayaka_py_b200.cache import CacheGroupSpec
    from ayaka_py_b200.parts import KVNeed
    from ayaka_py_b200.parts.position import rotary_frequencies
    rs = np.random.RandomState(2)
    for H, G, D, Dv, dims, base, scaling in ((3, 1, 20, 12, 12, 1e4, None), (2, 2, 64, 48, 16, 5e5, yarn(8.0, 100)), (4, 2, 16, 8, 16, 3.0, None),
                                             (2, 1, 7, 5, 6, 100.0, yarn(2.0, 30, 4.0)), (2, 1, 24, 4, 4, 50.0, None), (2, 1, 24, 4, 10, 50.0, None),
                                             (1, 1, 200, 8, 200, 1e5, None)):
        n, rot = 600, {"dims": dims, "base": base, "scaling": scaling}
        f, gain = rotary_frequencies(dims, base, scaling)
        freq = torch.tensor(f, dtype=torch.float64).float().cuda()
        proj = (rs.randn(n, (H + G) * D + G * Dv) * np.exp(rs.randn(n, 1))).astype(np.float32)
        proj = np.pad(proj, ((0, 0), (0, -proj.shape[1] % 4)))
        qw, kw = ((1.0 + 0.3 * rs.randn(D)).astype(np.float32) for _ in range(2))
        heads = proj[:, :(H + G) * D].astype(np.float64).reshape(n, H + G, D)
        for normed in (True, False):
            x = heads
            if normed:
                x = np.concatenate([plain.rms_norm(heads[:, :H], qw.astype(np.float64), 1e-3), plain.rms_norm(heads[:, H:], kw.astype(np.float64), 1e-3)], axis=1)
            for halves in (True, False):
                cache, runner = context_for([CacheGroupSpec("g", KVNeed(G, D, value_heads=G, value_dim=Dv), 1)], "float32", max_requests=2, page_size=8, pages=128)
                ctx, res = step_of(cache, runner, {0: n})
                kp, vp = cache.kv_layer(0, 0)
                q = ops.rotary_prepare(dev(proj), kp, vp, freq, dims, ctx, ctx.tables[0], H, True, torch.float32, gain=gain, halves=halves,
                                       q_norm=dev(qw) if normed else None, k_norm=dev(kw) if normed else None, eps=1e-3)
                want = (plain.rotate_halves if halves else plain.rotate_neighbours)(x, rot)
                bound = 1e-4 * np.abs(want).max()
                assert np.abs(host(q).reshape(n, H, D) - want[:, :H]).max() < bound, (D, dims, normed, halves)
                table = cache.table_rows(0, [cache.slot_of[0]])[0]
                cells = [(int(table[p // 8]), p % 8) for p in range(n)]
                assert np.abs(np.stack([host(kp[c]) for c in cells]) - want[:, H:]).max() < bound
                own = proj[:, (H + G) * D:(H + G) * D + G * Dv].reshape(n, G, Dv)
                assert np.array_equal(np.stack([vp[c].cpu().numpy() for c in cells]), own)
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
            assert np.abs(got - want).max() < 3e-5 * max(1.0, float(np.abs(want).max())), (tag, i)


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
def test_long_decoding_past_many_windows_and_chunks(models, tag, dtype):
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
    assert max(float(np.abs(got_alone[p] - got_both[p]).max()) for p in got_alone) < 5e-5


def test_pages_behind_windows_and_chunks_come_back(tmp_path):
    """A long request in a pool smaller than its length: pages that no window reaches (the reader's, which is the longer
    one, counts) and pages before the chunk are handed out again."""
    cfg = document([latent(4, 12, 8, 16, 24, 21, 0.3, moe(4, 1, 16, 8)), attention(2, 2, 12, 16, 30, 8, 0.3, None),
                    latent(2, 12, 8, 16, 24, 37, 0.3, None, kv_from=0)], 90, 48)
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
    # one layer, one head, heads of one and two numbers, one expert of one
    "smallest": document([attention(1, 1, 2, 1, 5, 2, 0.7, moe(1, 1, 3, 1))], 17, 8),
    "smallest_latent": document([latent(1, 1, 2, 1, 1, 3, 0.7, None), latent(1, 2, 2, 3, 1, 2, 0.7, moe(2, 1, 5, 3), kv_from=0)], 19, 12, alpha=0.5),
    # only latents, three readers of one and a chain of owners; a rotated part wider than the plain one
    "only_latent": document([latent(3, 24, 32, 16, 48, 50, 0.2, moe(5, 1, 24, 12)), latent(6, 16, 32, 32, 48, 64, 0.25, moe(5, 2, 24, 12), kv_from=0),
                             latent(2, 8, 16, 24, 32, 18, 0.3, None), latent(4, 48, 32, 8, 48, 7, 0.2, None, kv_from=0),
                             latent(2, 12, 32, 12, 48, None, 0.2, moe(3, 3, 8, 4), kv_from=0)], 333, 96),
    # a width that is no multiple of 8, inner widths that are none of 4
    "odd_width": document([attention(5, 5, 20, 20, 33, 10, 0.2, moe(9, 3, 30, 18)), latent(2, 50, 10, 50, 56, 41, 0.14, moe(7, 2, 21, 33)),
                           attention(10, 5, 16, 20, 64, 6, 0.25, moe(6, 2, 14, 0), scaling=yarn(3.0, 40, 16.0))], 257, 100, alpha=3.0),
    # values of 256 numbers, keys of 300, a latent of 512 + 64
    "wide_heads": document([attention(2, 1, 300, 256, 300, 128, 0.06, None), latent(2, 128, 64, 256, 512, 40, 0.08, moe(4, 2, 64, 64)),
                            latent(20, 16, 64, 16, 512, 128, 0.1, None, kv_from=1)], 64, 64),
    # 32 experts of which 8 are chosen; ten of 24; two experts, both chosen
    "many_experts": document([attention(2, 1, 64, 64, 128, 64, 0.125, moe(32, 8, 32, 64)), latent(8, 16, 16, 16, 64, 100, 0.2, moe(24, 10, 16, 8)),
                              attention(4, 2, 32, 64, 100, 16, 0.18, moe(2, 2, 8, 24))], 512, 128, alpha=1.25),
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
    from ayaka_py_b200.config.model import TomodraConfig
    from ayaka_py_b200.weights import write_random_model
    folder = write_random_model(tmp_path / "m", TomodraConfig.from_dict(CONFIG_B), seed=3)
    assert json.loads((folder / "config.json").read_text())["architecture"] == "Tomodra"
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
