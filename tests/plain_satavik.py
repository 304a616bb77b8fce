"""A plain, slow restatement of the Satavik decoder, one function per mechanism.

It shares no code with the library: tensors come in as a dict name -> torch
tensor, the configuration as the parsed config.json, and everything runs on the
CPU in one dtype (float64 by default).  ``forward`` returns logits for a whole
sequence and, optionally, the residual stream after every layer.

Notation: T tokens, D width, H heads, G key/value heads, K channels of one map
of a query or key head, V value channels per head, E experts.
"""
from __future__ import annotations

import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


# ---------------------------------------------------------------------------------------------------------
def rotate_halves(x, positions, dims, base):
    """x [T, ..., K]: of the first ``dims`` channels, channel i is rotated with channel i + dims/2."""
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * (float(base) ** (-2.0 * i / dims))[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    cos, sin = torch.cos(ang).to(x.dtype).view(shape), torch.sin(ang).to(x.dtype).view(shape)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def visible_keys(T, chunk):
    """[T, T]: row i sees column j iff j <= i and both lie in one block of ``chunk`` positions (None: no blocks)."""
    t = torch.arange(T)
    seen = t[None, :] <= t[:, None]
    if chunk is not None:
        seen = seen & (t[None, :] // chunk == t[:, None] // chunk)
    return seen


def capped(scores, cap):
    return scores if cap is None else cap * torch.tanh(scores / cap)


def softmax_rows(scores, visible):
    s = scores.masked_fill(~visible, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def map_weights(q, k, scale, cap, visible):
    """Attention weights [H, T, T] of one map: q [T, H, K], k [T, G, K]."""
    k = k.repeat_interleave(q.shape[1] // k.shape[1], dim=1)
    return softmax_rows(capped(torch.einsum("thk,shk->hts", q, k) * scale, cap), visible)


def second_map_weight(w, pre, diff):
    """How much of the second map is taken off the first, one number for the layer."""
    return torch.exp((w[pre + "lq1"] * w[pre + "lk1"]).sum()) - torch.exp((w[pre + "lq2"] * w[pre + "lk2"]).sum()) + diff


def keys_and_values(h, w, pre, mix, eps, positions):
    """(k [T, G, 2, K] normed and rotated, v [T, G, V])."""
    T, G, K, V = h.shape[0], mix["kv_heads"], mix["dim"], mix["vdim"]
    k = rms_norm((h @ w[pre + "k"].T).view(T, G, 2, K), w[pre + "k.norm"], eps)
    if mix.get("rot"):
        k = rotate_halves(k, positions, mix["rot"]["dims"], mix["rot"]["base"])
    return k, (h @ w[pre + "v"].T).view(T, G, V)


def differential_attention(h, w, pre, mix, eps, positions, shared=None):
    """Two maps per head over the same values, the second taken off the first.  ``shared``: another layer's keys and
    values (a layer that reads them has no projections of its own).  Returns (output, (keys, values))."""
    T, H, K, V = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q = rms_norm((h @ w[pre + "q"].T).view(T, H, 2, K), w[pre + "q.norm"], eps)
    if mix.get("rot"):
        q = rotate_halves(q, positions, mix["rot"]["dims"], mix["rot"]["base"])
    k, v = keys_and_values(h, w, pre, mix, eps, positions) if shared is None else shared
    seen = visible_keys(T, mix["mask"]["size"] if mix.get("mask") else None)
    vals = v.repeat_interleave(H // v.shape[1], dim=1)
    a = [torch.einsum("hts,shv->thv", map_weights(q[:, :, m], k[:, :, m], mix["scale"], mix.get("softcap"), seen), vals)
         for m in (0, 1)]
    o = a[0] - second_map_weight(w, pre, mix["diff"]) * a[1]
    o = unit_rms(o, eps) * (1 - mix["diff"])
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w[pre + "o"].T, (k, v)


# ---------------------------------------------------------------------------------------------------------
def clamped_unit(h, w, pre, limit):
    g = torch.clamp(h @ w[pre + "gate"].T, max=limit)
    u = torch.clamp(h @ w[pre + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[pre + "down"].T


def route(h, w, pre, top):
    """(ids [T, top], weights [T, top], logits [T, E]): the largest logits, softmax over them alone."""
    z = h @ w[pre + "router"].T + w[pre + "router.b"]
    ids = torch.topk(z, top, dim=-1).indices
    return ids, chosen_weights(z, ids), z


def chosen_weights(z, ids):
    c = torch.gather(z, 1, ids)
    e = torch.exp(c - c.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def moe_ffn(h, w, pre, mlp, forced=None):
    """``forced`` (ids [T, top]): use these experts instead of the router's choice."""
    ids, wts, z = route(h, w, pre, mlp["router"]["top"])
    if forced is not None:
        ids, wts = forced, chosen_weights(z, forced)
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        part = (wts * (ids == e)).sum(-1)
        rows = torch.nonzero((ids == e).any(-1)).flatten()
        if len(rows):
            y[rows] += part[rows, None] * clamped_unit(h[rows], w, f"{pre}e{e}.", mlp["expert"]["limit"])
    if mlp.get("shared"):
        y = y + clamped_unit(h, w, pre + "shared.", mlp["shared"]["limit"])
    return y


# ---------------------------------------------------------------------------------------------------------
def forward(cfg, weights, tokens, dtype=torch.float64, trace=None, forced_routing=None):
    """Logits [T, vocab].  ``trace``: a list that receives the residual stream behind every layer.
    ``forced_routing``: {layer index: ids [T, top]}."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        shared = kept[mix["kv_from"]] if mix.get("kv_from") is not None else None
        y, kept[i] = differential_attention(x, w, p + "mix.", mix, eps, positions, shared)
        x = x + rms_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            y = moe_ffn(x, w, p + "mlp.", layer["mlp"], None if forced_routing is None else forced_routing.get(i))
            x = x + rms_norm(y, w[p + "norm2"], eps)
        if trace is not None:
            trace.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def tensor_shapes(cfg):
    """name -> shape of every tensor a model folder of this design holds."""
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D), "final.norm": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q, H, G, K, V = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (D,), q + "q": (H * 2 * K, D), q + "q.norm": (K,), q + "g": (H, D), q + "o": (D, H * V)})
        out.update({q + n: (K,) for n in ("lq1", "lk1", "lq2", "lk2")})
        if m.get("kv_from") is None:
            out.update({q + "k": (G * 2 * K, D), q + "v": (G * V, D), q + "k.norm": (K,)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        f, r = p + "mlp.", mlp["router"]
        out.update({p + "norm2": (D,), f + "router": (r["experts"], D), f + "router.b": (r["experts"],)})
        units = [(f"{f}e{e}.", mlp["expert"]["ff"]) for e in range(r["experts"])]
        if mlp.get("shared"):
            units.append((f + "shared.", mlp["shared"]["ff"]))
        for u, ff in units:
            out.update({u + "gate": (ff, D), u + "up": (ff, D), u + "down": (D, ff)})
    return out


def random_weights(cfg, seed, gain=1.0):
    """name -> bfloat16 tensor (what a model folder stores), in ranges where every mechanism matters: the stream of
    order one, scores that reach the soft cap's bend, gates and up branches that reach their limits."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(tuple(s), generator=g)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = rn(*shape) / cfg["embedding"]["scale"]
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            t = 0.7 + 0.2 * rn(*shape)
        elif leaf == "norm":
            t = 1 + 0.3 * rn(*shape)
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = rn(*shape) * (0.4 / shape[0] ** 0.25)
        elif leaf == "b":
            t = rn(*shape) * 0.5
        elif len(shape) == 2:
            t = rn(*shape) * (gain / math.sqrt(shape[1]))
        else:
            raise ValueError(name)
        out[name] = t.to(torch.bfloat16)
    return out


def greedy(cfg, weights, prompt, count):
    """Greedy continuation by running the whole sequence anew for every token; returns (tokens, the margin between
    the best and the second logit at every choice)."""
    tokens, margins = list(prompt), []
    for _ in range(count):
        top = torch.topk(forward(cfg, weights, tokens)[-1], 2)
        margins.append(float(top.values[0] - top.values[1]))
        tokens.append(int(top.indices[0]))
    return tokens[len(prompt):], margins
