"""Tomodra in plain NumPy, one function per mechanism, whole sequences, no cache.  Slow and
simple on purpose: it shares no code with the package and is what the kernels are compared
with.  Everything runs in the dtype of the tensors it is given (float64 in the tests).

Notation: x is the residual stream [T, d]; W are [out, in] and applied as W @ x; i is a
query's position and j a key's, both counted from 0."""

from __future__ import annotations

import numpy as np

from plain_vedadra import round_bf16, write_folder, write_safetensors  # noqa: F401  (file helpers only)


# ----------------------------------------------------------- small functions --

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms_norm(x, w, eps):
    """The last axis over its root mean square (eps under the root), times a weight."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def softmax(s, visible, sink=None):
    """Softmax of s [H, T, T] over the visible keys; ``sink`` [H]: one more key per head with that score and no value."""
    s = np.where(visible, s, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, np.asarray(sink)[:, None, None])
    e = np.where(visible, np.exp(s - top), 0.0)
    below = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        below = below + np.exp(np.asarray(sink)[:, None, None] - top)
    return e / below


def window_mask(T, size):
    """visible[i, j]: j is i itself or one of the size - 1 positions before it (size None: any earlier one)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size is not None else True)


def chunk_mask(T, size):
    """visible[i, j]: j is not later than i and lies in the same run of ``size`` positions (None: any run)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i // size == j // size) if size is not None else True)


# ------------------------------------------------------------------ rotation --

def frequencies(rot):
    """(turns per position in radians of every pair, factor on cos and sin)."""
    n, base = rot["dims"], float(rot["base"])
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    stretch = rot.get("scaling")
    if not stretch:
        return f, 1.0
    where = lambda turns: n * np.log(stretch["original"] / (2 * np.pi * turns)) / (2 * np.log(base))
    first = max(np.floor(where(stretch["fast"])), 0)
    last = min(np.ceil(where(stretch["slow"])), n - 1)
    share = np.clip((np.arange(n // 2) - first) / max(last - first, 0.001), 0.0, 1.0)
    return f / stretch["factor"] * share + f * (1.0 - share), 0.1 * np.log(stretch["factor"]) + 1.0


def _cos_sin(x, rot):
    f, gain = frequencies(rot)
    angle = np.arange(x.shape[0])[:, None] * f[None, :]
    return (gain * np.cos(angle))[:, None, :].astype(x.dtype), (gain * np.sin(angle))[:, None, :].astype(x.dtype)


def rotate_neighbours(x, rot):
    """x [T, heads, D]: dimensions 2i and 2i + 1 below ``dims`` are a pair that turns; the rest passes."""
    c, s = _cos_sin(x, rot)
    out, n = x.copy(), rot["dims"]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2], out[..., 1:n:2] = u * c - v * s, v * c + u * s
    return out


def rotate_halves(x, rot):
    """The same for the pairs i and i + dims/2."""
    c, s = _cos_sin(x, rot)
    n = rot["dims"]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., n:]], axis=-1)


# -------------------------------------------------------------------- mixers --

def latent_of(h, t, p, mx, eps):
    """What a latent layer keeps of its tokens: (c [T, rank], rotated key part [T, rot_dim])."""
    both = h @ t[p + "dkv"].T
    c = rms_norm(both[:, :mx["kv_rank"]], t[p + "dkv.norm"], eps)
    return c, rotate_halves(both[:, None, mx["kv_rank"]:], mx["rot"])[:, 0]


def latent_attention(h, t, p, mx, eps, kept):
    """``kept``: the pair of ``latent_of``, this layer's own or an earlier layer's."""
    T = h.shape[0]
    H, D, R, Dv = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    c, kr = kept
    q = (h @ t[p + "q"].T).reshape(T, H, D + R)
    qn, qr = q[..., :D], rotate_halves(q[..., D:], mx["rot"])
    kn = (c @ t[p + "uk"].T).reshape(T, H, D)
    v = (c @ t[p + "uv"].T).reshape(T, H, Dv)
    s = (np.einsum("ihd,jhd->hij", qn, kn) + np.einsum("ihd,jd->hij", qr, kr)) * mx["scale"]
    w = softmax(s, window_mask(T, (mx.get("mask") or {}).get("size")))
    return np.einsum("hij,jhd->ihd", w, v).reshape(T, H * Dv) @ t[p + "o"].T


def attention(h, t, p, mx, eps):
    T = h.shape[0]
    H, G, D, Dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = rms_norm((h @ t[p + "q"].T).reshape(T, H, D), t[p + "q.norm"], eps)
    k = rms_norm((h @ t[p + "k"].T).reshape(T, G, D), t[p + "k.norm"], eps)
    v = (h @ t[p + "v"].T).reshape(T, G, Dv)
    q, k = rotate_neighbours(q, mx["rot"]), rotate_neighbours(k, mx["rot"])
    of = np.arange(H) // (H // G)
    s = np.einsum("ihd,jhd->hij", q, k[:, of]) * mx["scale"]
    w = softmax(s, chunk_mask(T, (mx.get("mask") or {}).get("size")), t[p + "sink"])
    return np.einsum("hij,jhd->ihd", w, v[:, of]).reshape(T, H * Dv) @ t[p + "o"].T


# -------------------------------------------------------------- feed-forward --

def expert(h, t, p):
    g = h @ t[p + "gate"].T
    return (g * sigmoid(g) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def route(z, top, margin=None):
    """One token's routing from its logits z [E]: (chosen experts, their weights).  ``margin``: a list that receives
    the gap between the last chosen expert and the next, in logits."""
    ranked = sorted(range(z.shape[0]), key=lambda e: (-z[e], e))
    if margin is not None:
        margin.append(z[ranked[top - 1]] - z[ranked[top]] if top < len(ranked) else np.inf)
    return ranked[:top], sigmoid(z[ranked[:top]])


def moe_ff(h, t, p, mlp, margins=None):
    """``margins``: a list that receives one array [T] of this layer's routing margins (see ``route``)."""
    mine = [] if margins is not None else None
    z = h @ t[p + "router"].T
    out = np.zeros_like(h)
    for n in range(h.shape[0]):
        for e, w in zip(*route(z[n], mlp["router"]["top"], mine)):
            out[n] += expert(w * h[n:n + 1], t, f"{p}e{e}.")[0]
    if margins is not None:
        margins.append(np.asarray(mine))
    if mlp.get("shared"):
        out = out + sigmoid(h @ t[p + "shared.sg"].T) * expert(h, t, p + "shared.")
    return out


# --------------------------------------------------------------------- model --

def forward(cfg, t, tokens, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence from position 0.  ``layers_out``: a list that receives the
    residual stream after every layer; ``margins``: see ``moe_ff``."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = t["embed"][np.asarray(tokens)]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            y = attention(x, t, p + "mix.", mx, eps)
        else:
            if mx.get("kv_from") is None:
                kept[i] = latent_of(x, t, p + "mix.", mx, eps)
            y = latent_attention(x, t, p + "mix.", mx, eps, kept[i if mx.get("kv_from") is None else mx["kv_from"]])
        x = rms_norm(alpha * x + y, t[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = rms_norm(alpha * x + moe_ff(x, t, p + "mlp.", layer["mlp"], margins), t[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, t["final.norm"], eps) @ t["head"].T


# ------------------------------------------------- tensors, files, configs --

def tensor_shapes(cfg):
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d), "head": (cfg["vocab"], d), "final.norm": (d,)}
    for i, layer in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        m, f = p + "mix.", p + "mlp."
        out[p + "norm1"] = (d,)
        H, D, Dv = mx["heads"], mx["dim"], mx["vdim"]
        if layer["type"] == "attention":
            G = mx["kv_heads"]
            out.update({m + "q": (H * D, d), m + "k": (G * D, d), m + "v": (G * Dv, d), m + "q.norm": (D,), m + "k.norm": (D,),
                        m + "sink": (H,), m + "o": (d, H * Dv)})
        else:
            R, K = mx["rot_dim"], mx["kv_rank"]
            out.update({m + "q": (H * (D + R), d), m + "uk": (H * D, K), m + "uv": (H * Dv, K), m + "o": (d, H * Dv)})
            if mx.get("kv_from") is None:
                out.update({m + "dkv": (K + R, d), m + "dkv.norm": (K,)})
        if mlp is None:
            continue
        out[p + "norm2"] = (d,)
        out[f + "router"] = (mlp["router"]["experts"], d)
        experts = [(f"{f}e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            experts.append((f + "shared.", mlp["shared"]["ff"]))
            out[f + "shared.sg"] = (1, d)
        for at, ff in experts:
            out.update({at + "gate": (ff, d), at + "up": (ff, d), at + "down": (d, ff)})
    return out


def random_tensors(cfg, seed, gain=1.0):
    """Every tensor as float32 values that bfloat16 holds exactly."""
    rs = np.random.RandomState(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        g = rs.standard_normal(shape).astype(np.float32)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            w = g
        elif last in ("norm1", "norm2", "norm"):
            w = 1.0 + 0.1 * g
        elif last == "sink":
            w = 0.5 * g
        elif last in ("router", "head"):
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
