"""A plain statement of the Setotar decoder: whole sequences, no cache, no batches, float64, one function per
mechanism.  It shares no code with the package and is slow on purpose.

The design: several residual streams per token that a sublayer reads as one weighted sum and writes through a
mixing matrix (hyper-connections), each sublayer's output scaled per channel; two mixers (``attention``:
grouped-query attention over all keys, queries and keys normed over their whole projections and turned by
YaRN-stretched rotary positions, where a layer may read another layer's keys and values; ``parallel``:
window attention that keeps the first tokens, behind biased projections and short convolutions, with linearly
stretched positions, unit-RMS values and capped scores, next to a linear recurrence in which one
gate a channel sets what is kept and what is written); a mixture of gated experts on rows scaled by the router's
sigmoid, or none.
"""

import json
import math
import os

import torch

F = torch.float64


def read_model_folder(path):
    """(config dict, {name: float64 tensor})."""
    from safetensors.torch import load_file

    with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as handle:
        cfg = json.load(handle)
    weights = {k: v.to(F) for k, v in load_file(os.path.join(path, "model.safetensors")).items()}
    return cfg, weights


# ------------------------------------------------------------------------------------------ small things

def rms(x, eps):
    """``x / sqrt(mean(x^2) + eps)`` over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(x, taps):
    """``x`` ``[T, C]``, ``taps`` ``[C, K]``: the last column multiplies the current token, the one before it the
    token before, and so on; nothing stands in front of the sequence."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for back in range(min(K, t + 1)):
            y[t] += taps[:, K - 1 - back] * x[t - back]
    return y


def frequencies(rot):
    """``(f [dims / 2], multiplier of cos and sin)`` of a rotation: plain, with every frequency divided by a factor
    (``scaling`` has only that), or YaRN (``scaling`` has ``original``, ``fast`` and ``slow`` too)."""
    dims, base = rot["dims"], rot["base"]
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    scaling = rot.get("scaling")
    if scaling is None:
        return f, 1.0
    factor = scaling["factor"]
    if "original" not in scaling:
        return f / factor, 1.0

    def turns(t):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turns(scaling["fast"])), 0)
    hi = min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(float(f[i]) / factor * ramp + float(f[i]) * (1.0 - ramp))
    return torch.tensor(out, dtype=F), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot):
    """Turns the first ``dims`` entries of the heads of ``x`` ``[T, heads, D]``: entry ``i`` with entry ``i + dims/2``."""
    if rot is None:
        return x
    f, mult = frequencies(rot)
    half = rot["dims"] // 2
    angle = positions.to(F)[:, None] * f[None, :]
    cos, sin = (angle.cos() * mult)[:, None, :], (angle.sin() * mult)[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * cos - v * sin
    out[..., half:2 * half] = v * cos + u * sin
    return out


def visible(i, j, window=None, keep_first=0):
    """Whether query ``i`` sees key ``j`` (tensors of positions)."""
    if window is None:
        return j <= i
    return (j <= i) & ((i - j < window) | (j < keep_first))


def attend(q, k, v, scale, cap=None, window=None, keep_first=0):
    """``q`` ``[T, H, D]``, ``k`` ``[T, G, D]``, ``v`` ``[T, G, V]`` -> ``[T, H, V]``."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = visible(torch.arange(T)[:, None], torch.arange(T)[None, :], window, keep_first)
    out = torch.zeros((T, H, v.shape[-1]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if cap is not None:
            s = cap * torch.tanh(s / cap)
        out[:, h] = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1) @ v[:, g]
    return out


# ------------------------------------------------------------------------------------------ attention

def keys_values(h, w, p, m, eps, positions):
    """A layer's keys (normed over the whole projection, turned) and values."""
    T = h.shape[0]
    k = norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, m["kv_heads"], m["dim"])
    v = (h @ w[p + "v"].T).reshape(T, m["kv_heads"], m["vdim"])
    return rotate(k, positions, m.get("rot")), v


def attention_mixer(h, w, p, m, eps, positions, kv):
    T = h.shape[0]
    q = norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, m["heads"], m["dim"])
    q = rotate(q, positions, m.get("rot"))
    return attend(q, *kv, m["scale"]).reshape(T, -1) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------ parallel

def left_mixer(h, w, p, m, eps, positions):
    T = h.shape[0]

    def project(name):
        x = h @ w[p + name].T + w[p + name + ".b"]
        return causal_conv(x, w[p + name + ".conv"]) if m.get("conv") is not None else x

    q = rotate(project("q").reshape(T, m["heads"], m["dim"]), positions, m.get("rot"))
    k = rotate(project("k").reshape(T, m["kv_heads"], m["dim"]), positions, m.get("rot"))
    v = rms(project("v").reshape(T, m["kv_heads"], m["vdim"]), eps)
    mask = m.get("mask") or {}
    a = attend(q, k, v, m["scale"], m.get("softcap"), mask.get("size"), mask.get("keep_first", 0))
    return a.reshape(T, -1) @ w[p + "o"].T


def forget_recurrence(q, f, v):
    """``q``/``f`` ``[T, H, D]``, ``v`` ``[T, H, V]``: per head ``S <- diag(f) S + (1 - f) v^T`` from zero, ``o = S^T q``."""
    T, H, D = q.shape
    S = torch.zeros((H, D, v.shape[-1]), dtype=q.dtype)
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out.append((q[t][:, :, None] * S).sum(dim=1))
    return torch.stack(out)


def right_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    low = w[p + "lower"]
    f = (low + (1.0 - low) * torch.sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).reshape(T, H, D)
    o = norm(forget_recurrence(q, f, v), w[p + "norm"], eps)
    return o.reshape(T, -1) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps, positions):
    return (m["left_scale"] * left_mixer(h, w, p + "left.", m["left"], eps, positions)
            + m["right_scale"] * right_mixer(h, w, p + "right.", m["right"], eps))


# ------------------------------------------------------------------------------------------ experts

def expert(x, w, p):
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, router):
    """(indices ``[T, top]``, all scores ``[T, E]``): the largest sigmoids, the lower index first among equals."""
    s = torch.sigmoid(h @ w[p + "router"].T)
    return torch.argsort(s, dim=-1, descending=True, stable=True)[:, :router["top"]], s


def routed_feed_forward(h, w, p, mlp, chosen=None):
    """``chosen`` (``[T, top]``): these experts instead of the router's choice (weights still from the scores), for
    comparisons in which a near-tie may fall either way."""
    index, s = route(h, w, p, mlp["router"])
    if chosen is not None:
        index = torch.as_tensor(chosen).long()
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in index[t].tolist():
            out[t] += expert(s[t, e] * h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


# ------------------------------------------------------------------------------------------ the model

def through_streams(xs, w, p, sublayer):
    """One sublayer around the streams ``xs`` ``[S, T, W]``: read, run, write every stream from the old ones."""
    u = (w[p + "in"][:, None, None] * xs).sum(dim=0)
    y = sublayer(u)
    mix, out = w[p + "mix"], w[p + "out"]
    new = []
    for t in range(xs.shape[0]):
        x = out[t] * y
        for s in range(xs.shape[0]):
            x = x + mix[s, t] * xs[s]
        new.append(x)
    return torch.stack(new)


def forward(cfg, w, tokens, layers_out=None, routes=None):
    """Logits ``[T, vocab]`` of one sequence from its first token; ``layers_out`` (a list) receives the sum of the
    streams after every layer; ``routes`` ({layer: ``[T, top]``}) fixes the experts of routed layers."""
    eps = cfg["norm"]["eps"]
    positions = torch.arange(len(tokens))
    xs = w["embed"][torch.as_tensor(tokens)][None].repeat(cfg["streams"], 1, 1)
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]

        def mixer(u):
            h = norm(u, w[p + "norm1"], eps)
            if layer["type"] == "parallel":
                y = parallel_mixer(h, w, p + "mix.", m, eps, positions)
            else:
                source = m.get("kv_from")
                if source is None:
                    kept[i] = keys_values(h, w, p + "mix.", m, eps, positions)
                y = attention_mixer(h, w, p + "mix.", m, eps, positions, kept[i if source is None else source])
            return y * w[p + "ls1"]

        xs = through_streams(xs, w, p + "hc1.", mixer)
        if layer.get("mlp") is not None:
            def feed_forward(u):
                h = norm(u, w[p + "norm2"], eps)
                return routed_feed_forward(h, w, p + "mlp.", layer["mlp"], None if routes is None else routes.get(i)) * w[p + "ls2"]

            xs = through_streams(xs, w, p + "hc2.", feed_forward)
        if layers_out is not None:
            layers_out.append(xs.sum(dim=0))
    return norm(xs.sum(dim=0), w["final.norm"], eps) @ w["head"].T


def generate(cfg, w, prompt, n):
    """Greedy continuation: ``n`` tokens, each the largest logit (the lowest index among equals)."""
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(torch.argmax(forward(cfg, w, seq)[-1]))
        out.append(tok)
        seq.append(tok)
    return out
