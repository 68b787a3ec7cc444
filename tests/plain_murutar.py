"""Murutar in plain NumPy, one function per mechanism, whole sequences, no cache.  Slow and
simple on purpose: it shares no code with the package and is what the kernels are compared
with.  Everything runs in the dtype of the tensors it is given (float64 in the tests).

Notation: x is the residual stream [T, d]; W are [out, in] and applied as W @ x; i is a
query's position and j a key's, both counted from 0; t counts time steps of a recurrence."""

from __future__ import annotations

import numpy as np

from plain_vedadra import round_bf16, write_folder, write_safetensors  # noqa: F401  (file helpers only)


# ----------------------------------------------------------- small functions --

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    """Division of the last axis by its root mean square, eps under the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, eps):
    mu = x.mean(axis=-1, keepdims=True)
    var = ((x - mu) ** 2).mean(axis=-1, keepdims=True)
    return (x - mu) / np.sqrt(var + eps) * w


def window_mask(T, size):
    """visible[i, j]: j is i itself or one of the size - 1 positions before it (size None: any earlier one)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size is not None else True)


def sink_softmax(s, visible):
    """Softmax over the visible keys and one more whose score is 0 and which has no value."""
    s = np.where(visible, s, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.where(visible, np.exp(s - top), 0.0)
    return e / (np.exp(-top) + e.sum(axis=-1, keepdims=True))


def rotate_halves(x, base, dims):
    """x [T, heads, D]: dimension i < dims/2 and dimension i + dims/2 are a pair that turns by the position
    times base^(-2i / dims); the dimensions from ``dims`` on pass."""
    half = dims // 2
    angle = np.arange(x.shape[0])[:, None] * (float(base) ** (-2.0 * np.arange(half) / dims))[None, :]
    c, s = np.cos(angle)[:, None, :].astype(x.dtype), np.sin(angle)[:, None, :].astype(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


# -------------------------------------------------------------------- mixers --

def sink_attention(h, t, p, mx, eps, first_values):
    """Windowed softmax attention with a sink.  ``first_values``: a list, empty until the model's first layer
    that mixes values leaves its own there; the later ones blend theirs with them."""
    T = h.shape[0]
    H, G, D, Dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = (h @ t[p + "q"].T).reshape(T, H, D)
    k = (h @ t[p + "k"].T).reshape(T, G, D)
    v = (h @ t[p + "v"].T).reshape(T, G, Dv)
    q, k = (rotate_halves(z, mx["rot"]["base"], mx["rot"]["dims"]) for z in (q, k))
    if mx.get("v_mix"):
        if first_values:
            lam = float(np.asarray(t[p + "vmix"]).reshape(()))
            v = (1.0 - lam) * v + lam * first_values[0]
        else:
            first_values.append(v)
    kv_of = np.arange(H) // (H // G)
    s = np.einsum("ihd,jhd->hij", q, k[:, kv_of]) * mx["scale"]
    w = sink_softmax(s, window_mask(T, (mx.get("mask") or {}).get("size")))
    return np.einsum("hij,jhd->ihd", w, v[:, kv_of]).reshape(T, H * Dv) @ t[p + "o"].T


def decayed_recurrence(q, k, v, decay):
    """S <- decay S + k v^T per head, read by q after the write, from an empty state.  q, k [T, H, D], v [T, H, Dv]."""
    T, H, D = q.shape
    lam = np.asarray(decay, dtype=q.dtype)[:, None, None]
    S = np.zeros((H, D, v.shape[2]), dtype=q.dtype)
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for n in range(T):
        S = lam * S + k[n][:, :, None] * v[n][:, None, :]
        out[n] = np.einsum("hdv,hd->hv", S, q[n])
    return out


def lightning(h, t, p, mx, eps, first_values=None):
    T = h.shape[0]
    H, D, Dv = mx["heads"], mx["dim"], mx["vdim"]
    q = silu(h @ t[p + "q"].T).reshape(T, H, D)
    k = silu(h @ t[p + "k"].T).reshape(T, H, D)
    v = silu(h @ t[p + "v"].T).reshape(T, H, Dv)
    o = decayed_recurrence(q, k, v, mx["decay"]).reshape(T, H * Dv)
    o = unit_rms(o, eps) * t[p + "norm"] * sigmoid(h @ t[p + "g"].T)
    return o @ t[p + "o"].T


MIXERS = {"attention": sink_attention, "lightning": lightning}


# -------------------------------------------------------------- feed-forward --

def limited_glu_ff(h, t, p, limit):
    g = np.minimum(h @ t[p + "gate"].T, limit)
    u = np.clip(h @ t[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ t[p + "down"].T


def relu2_expert(h, t, p):
    return (np.maximum(h @ t[p + "up"].T, 0.0) ** 2) @ t[p + "down"].T


def route(z, top, count, keep, margin=None):
    """One token's routing from its logits z [E]: (chosen experts, their weights).  ``margin``: a list that
    receives how far the choice was from turning out otherwise, in logits (the smaller of the gap between the
    last kept group and the next one, and between the last chosen expert and the next allowed one)."""
    E = z.shape[0]
    e = np.exp(z - z.max())
    s = e / e.sum()
    per = E // count
    best = z.reshape(count, per).max(axis=1)
    order = sorted(range(count), key=lambda g: (-best[g], g))
    allowed = [e for g in order[:keep] for e in range(g * per, (g + 1) * per)]
    ranked = sorted(allowed, key=lambda e: (-z[e], e))
    chosen = ranked[:top]
    if margin is not None:
        gaps = [best[order[keep - 1]] - best[order[keep]]] if keep < count else []
        if top < len(ranked):
            gaps.append(z[ranked[top - 1]] - z[ranked[top]])
        margin.append(min(gaps) if gaps else np.inf)
    return chosen, s[chosen]


def moe_ff(h, t, p, mlp, margins=None):
    """``margins``: a list that receives one array [T] of this layer's routing margins (see ``route``)."""
    r = mlp["router"]
    mine = [] if margins is not None else None
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ t[p + "router"].T
    out = np.zeros_like(h)
    for n in range(h.shape[0]):
        chosen, w = route(z[n], r["top"], groups["count"], groups["keep"], mine)
        for e, we in zip(chosen, w):
            out[n] += we * relu2_expert(h[n:n + 1], t, f"{p}e{e}.")[0]
    if margins is not None:
        margins.append(np.asarray(mine))
    return out


def feed_forward(h, t, p, mlp, margins=None):
    return limited_glu_ff(h, t, p, mlp["limit"]) if mlp["kind"] == "dense" else moe_ff(h, t, p, mlp, margins)


# --------------------------------------------------------------------- model --

def gated(y, h, t, p, which):
    """A sublayer's result times a constant per channel and a gate per channel from the sublayer's input."""
    return y * t[f"{p}ls{which}"] * sigmoid(h @ t[f"{p}rg{which}"].T + t[f"{p}rg{which}.b"])


def token_input(x, tokens, t, p, layer, dim, eps):
    """What the layer adds for its tokens: the layer's part of the side table's row, gated by the stream."""
    e = t["side.embed"][np.asarray(tokens), layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ t[p + "side.gate"].T) * e) @ t[p + "side.proj"].T
    return unit_rms(y, eps) * t[p + "side.norm"]


def forward(cfg, t, tokens, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence from position 0.  ``layers_out``: a list that receives the
    residual stream after every layer; ``margins``: see ``moe_ff``."""
    eps = cfg["norm"]["eps"]
    x = t["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    first_values = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = layer_norm(x, t[p + "norm1"], eps)
        x = x + gated(MIXERS[layer["type"]](h, t, p + "mix.", layer["mixer"], eps, first_values), h, t, p, 1)
        if layer.get("mlp") is not None:
            h = layer_norm(x, t[p + "norm2"], eps)
            x = x + gated(feed_forward(h, t, p + "mlp.", layer["mlp"], margins), h, t, p, 2)
        x = x + token_input(x, tokens, t, p, i, cfg["token_side"]["dim"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    cap = cfg["logit_softcap"]
    return cap * np.tanh(layer_norm(x, t["final.norm"], eps) @ t["embed"].T / cap)


# ------------------------------------------------- tensors, files, configs --

def tensor_shapes(cfg):
    d, sd = cfg["width"], cfg["token_side"]["dim"]
    out = {"embed": (cfg["vocab"], d), "side.embed": (cfg["vocab"], len(cfg["layers"]) * sd), "final.norm": (d,)}
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        for n in (1, 2) if layer.get("mlp") is not None else (1,):
            out.update({f"{p}norm{n}": (d,), f"{p}ls{n}": (d,), f"{p}rg{n}": (d, d), f"{p}rg{n}.b": (d,)})
        out.update({p + "side.gate": (sd, d), p + "side.proj": (d, sd), p + "side.norm": (d,)})
        m = p + "mix."
        H, D, Dv = mx["heads"], mx["dim"], mx["vdim"]
        G = mx["kv_heads"] if layer["type"] == "attention" else H
        out.update({m + "q": (H * D, d), m + "k": (G * D, d), m + "v": (G * Dv, d), m + "o": (d, H * Dv)})
        if layer["type"] == "lightning":
            out.update({m + "g": (H * Dv, d), m + "norm": (H * Dv,)})
        elif mx.get("v_mix"):
            out[m + "vmix"] = ()
        mlp, f = layer.get("mlp"), p + "mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            out.update({f + "gate": (mlp["ff"], d), f + "up": (mlp["ff"], d), f + "down": (d, mlp["ff"])})
            continue
        out[f + "router"] = (mlp["router"]["experts"], d)
        for e in range(mlp["router"]["experts"]):
            out.update({f"{f}e{e}.up": (mlp["expert"]["ff"], d), f"{f}e{e}.down": (d, mlp["expert"]["ff"])})
    return out


def random_tensors(cfg, seed, gain=1.0):
    """Every tensor as float32 values that bfloat16 holds exactly."""
    rs = np.random.RandomState(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        g = rs.standard_normal(shape).astype(np.float32)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            w = g / np.sqrt(shape[-1])
        elif name == "side.embed":
            w = g
        elif last in ("norm1", "norm2", "norm"):
            w = 1.0 + 0.1 * g
        elif last in ("ls1", "ls2"):
            w = 0.8 + 0.2 * g
        elif last == "b":
            w = 0.5 * g
        elif last == "vmix":
            w = np.float32(0.4) + 0.1 * g
        elif last == "router":
            w = 2.0 * g / np.sqrt(shape[-1])
        else:
            w = gain * g / np.sqrt(shape[-1])
        out[name] = round_bf16(np.asarray(w, dtype=np.float32))
    return out


def greedy_generate(cfg, t, prompt, n):
    """n tokens, each the arg max of the last position's logits (the whole sequence is run again every time)."""
    toks, out = list(prompt), []
    for _ in range(n):
        nxt = int(np.argmax(forward(cfg, t, toks)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out
