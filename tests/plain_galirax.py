"""A plain, slow restatement of the Galirax decoder, one function per mechanism.

It shares no code with the library: tensors come in as a dict name -> torch
tensor, the configuration as the parsed config.json, and everything runs on the
CPU in one dtype (float64 by default), token by token where the design has a
recurrence.  ``forward`` returns logits for a whole sequence and, optionally,
the residual stream after every layer run.

Notation: T tokens, D width, H heads, G key/value heads, K key channels per
head, V value channels per head, E experts.
"""
from __future__ import annotations

import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    """Mean off, divided by the root of the mean squared deviation (eps inside the root), times w, plus b."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


# ---------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """float64 [dims / 2]: base^(-2i/dims).  With scaling, a channel pair whose period (in positions) is shorter than
    original / high keeps its frequency, one whose period is longer than original / low has it divided by the factor, and
    between the two the frequency is a blend that is linear in original / period."""
    i = torch.arange(rot["dims"] // 2, dtype=torch.float64)
    f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
    sc = rot.get("scaling")
    if not sc:
        return f
    out = []
    for v in f.tolist():
        period, slow = 2 * math.pi / v, v / sc["factor"]
        if period < sc["original"] / sc["high"]:
            out.append(v)
        elif period > sc["original"] / sc["low"]:
            out.append(slow)
        else:
            share = (sc["original"] / period - sc["low"]) / (sc["high"] - sc["low"])
            out.append(slow + share * (v - slow))
    return torch.tensor(out, dtype=torch.float64)


def rotate_neighbours(x, positions, rot):
    """x [T, heads, K]: of the first rot.dims channels of every head, channel 2i is rotated with channel 2i + 1."""
    dims = rot["dims"]
    ang = positions.to(torch.float64)[:, None] * frequencies(rot)[None, :]
    cos, sin = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = a * cos - b * sin
    out[..., 1:dims:2] = b * cos + a * sin
    return out


def visible_keys(T, mask):
    """[T, T] bool: row i, column j.  Causal; with a mask only the last ``size`` positions and the first ``keep_first``."""
    t = torch.arange(T)
    dist = t[:, None] - t[None, :]
    vis = dist >= 0
    if mask:
        vis = vis & ((dist < mask["size"]) | (t[None, :] < mask.get("keep_first", 0)))
    return vis


def sink_softmax(scores, visible, sink):
    """scores [H, T, T]; sink [H]: one more term exp(sink_h) in every row's denominator."""
    s = scores.masked_fill(~visible[None], -math.inf)
    m = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


def attention(h, w, pre, mix, eps, positions, wide):
    """``wide``: biases on q, k and v, and one RMS norm over all heads of q (of k) together, ahead of the rotation."""
    T = h.shape[0]
    H, G, K, V = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q, k, v = (h @ w[pre + t].T for t in "qkv")
    if wide:
        q, k, v = q + w[pre + "q.b"], k + w[pre + "k.b"], v + w[pre + "v.b"]
        q, k = unit_rms(q, eps) * w[pre + "q.norm"], unit_rms(k, eps) * w[pre + "k.norm"]
    q, k, v = q.view(T, H, K), k.view(T, G, K), v.view(T, G, V)
    if mix.get("rot"):
        q, k = rotate_neighbours(q, positions, mix["rot"]), rotate_neighbours(k, positions, mix["rot"])
    rep = H // G
    scores = torch.einsum("thk,shk->hts", q, k.repeat_interleave(rep, dim=1)) * mix["scale"]
    p = sink_softmax(scores, visible_keys(T, mix.get("mask")), w[pre + "sink"].to(h.dtype))
    o = torch.einsum("hts,shv->thv", p, v.repeat_interleave(rep, dim=1))
    return o.reshape(T, H * V) @ w[pre + "o"].T


def decayed_sums(q, k, v, decay, state=None):
    """q, k [T, H, K]; v [T, H, V]; decay [H]: S <- decay_h S + k v^T, o = S^T q, token by token.  ([T, H, V], S)."""
    T, H, K = q.shape
    S = torch.zeros(H, K, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def lightning(h, w, pre, mix, eps):
    T = h.shape[0]
    H, K, V = mix["heads"], mix["dim"], mix["vdim"]
    q, k, v = (silu(h @ w[pre + t].T) for t in "qkv")
    o, _ = decayed_sums(q.view(T, H, K), k.view(T, H, K), v.view(T, H, V), torch.tensor(mix["decay"], dtype=h.dtype))
    o = unit_rms(o.reshape(T, H * V), eps) * w[pre + "norm"]
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------------------
def gated_expert(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def choose(s, correction, router):
    """s [T, E] scores: ids [T, top] of the experts with the largest corrected scores within the best groups, a group's
    score being the sum of its two largest corrected scores."""
    choice = s + correction
    groups = router.get("groups")
    if groups and groups["count"] > 1:
        T, n = choice.shape
        per = n // groups["count"]
        best = choice.view(T, groups["count"], per).topk(min(2, per), dim=-1).values.sum(-1)
        keep = torch.topk(best, groups["keep"], dim=-1).indices
        allowed = torch.zeros(T, groups["count"], dtype=torch.bool)
        allowed.scatter_(1, keep, True)
        choice = choice.masked_fill(~allowed.repeat_interleave(per, dim=1), -math.inf)
    return torch.topk(choice, router["top"], dim=-1).indices


def route_weights(s, ids, scale):
    """The chosen scores (without the correction) over their sum, times ``scale``."""
    c = torch.gather(s, 1, ids)
    return c / (c.sum(-1, keepdim=True) + 1e-20) * scale


def moe(h, w, pre, mlp, forced=None):
    """``forced`` (ids [T, top]): use these experts instead of the router's choice (the weights stay the scores')."""
    router = mlp["router"]
    s = sigmoid(h @ w[pre + "router"].T)
    ids = choose(s, w[pre + "correction"], router) if forced is None else forced
    wts = route_weights(s, ids, router["scale"])
    y = torch.zeros_like(h)
    for e in range(router["experts"]):
        t, j = (ids == e).nonzero(as_tuple=True)
        if t.numel():
            y[t] = y[t] + wts[t, j][:, None] * gated_expert(h[t], w, f"{pre}e{e}.")
    return y


# ---------------------------------------------------------------------------------------------------------
def layer_runs(cfg):
    """Indices of the layers in the order in which they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    inside = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inside * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, weights, tokens, dtype=torch.float64, trace=None, forced_routing=None):
    """Logits [T, vocab].  ``trace``: a list that receives the residual stream behind every layer run.
    ``forced_routing``: {layer run: ids [T, top]}."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for run, i in enumerate(layer_runs(cfg)):
        layer, p = cfg["layers"][i], f"l{i}."
        mix, mlp = layer["mixer"], layer.get("mlp")
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        if layer["type"] == "lightning":
            y = lightning(h, w, p + "mix.", mix, eps)
        else:
            y = attention(h, w, p + "mix.", mix, eps, positions, layer["type"] == "attention_2")
        if mlp is not None:
            y = y + moe(h, w, p + "mlp.", mlp, None if forced_routing is None else forced_routing.get(run))
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def tensor_shapes(cfg):
    """name -> shape of every tensor a model folder of this design holds."""
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D), "final.norm": (D,), "final.norm.b": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        out.update({p + "norm1": (D,), p + "norm1.b": (D,)})
        if layer["type"] == "lightning":
            H, K, V = m["heads"], m["dim"], m["vdim"]
            out.update({q + "q": (H * K, D), q + "k": (H * K, D), q + "v": (H * V, D), q + "g": (H * V, D), q + "norm": (H * V,),
                        q + "o": (D, H * V)})
        else:
            H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({q + "q": (H * K, D), q + "k": (G * K, D), q + "v": (G * V, D), q + "sink": (H,), q + "o": (D, H * V)})
            if layer["type"] == "attention_2":
                out.update({q + "q.b": (H * K,), q + "k.b": (G * K,), q + "v.b": (G * V,), q + "q.norm": (H * K,),
                            q + "k.norm": (G * K,)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        f, E, ff = p + "mlp.", mlp["router"]["experts"], mlp["expert"]["ff"]
        for e in range(E):
            out.update({f"{f}e{e}.gate": (ff, D), f"{f}e{e}.up": (ff, D), f"{f}e{e}.down": (D, ff)})
        out.update({f + "router": (E, D), f + "correction": (E,)})
    return out


def random_weights(cfg, seed, gain=1.0):
    """name -> bfloat16 tensor (what a model folder stores), in ranges where every mechanism matters: norm biases and
    sinks of the order of what they are added to, corrections large enough to change choices and to make some choice
    scores negative."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(tuple(s), generator=g)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = rn(*shape) * 0.7
        elif leaf == "norm1" or leaf == "norm":
            t = 1 + 0.2 * rn(*shape)
        elif leaf == "b":
            t = rn(*shape) * 0.3
        elif leaf == "sink":
            t = rn(*shape) * 1.5
        elif leaf == "correction":
            t = rn(*shape) * 0.5
        elif leaf == "router":
            t = rn(*shape) * (1.5 / math.sqrt(shape[1]))
        else:
            t = rn(*shape) * (gain / math.sqrt(shape[1]))
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
