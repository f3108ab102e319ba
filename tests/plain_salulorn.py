"""A plain statement of the Salulorn decoder: whole sequences, no cache, no batches, float64, one function per
mechanism.  It shares no code with the package and is slow on purpose.

The design: one residual stream; layers whose two sublayers read the same norm and are added together; a run of layers
that is passed through several times with the same weights, each pass opened by a projection of the stream and the
embedding side by side; three mixers (``gla``: a linear recurrence with a matrix state and a decay per key channel;
``attention``: window attention behind biased projections, short convolutions and norms over whole rows, with turned
queries and keys, capped scores and a sink; ``latent_attention``: attention over a low-rank latent with YaRN-stretched
positions, a sink and an output gate); a gated feed-forward, or none.
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

def norm(x, w, eps):
    """``x / sqrt(mean(x^2) + eps) * w`` over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(x, taps):
    """``x`` ``[T, C]``, ``taps`` ``[C, K]``: the last column multiplies the current token, the one before it the
    token before, and so on; nothing stands in front of the sequence."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for back in range(min(K, T)):
        y[back:] += taps[:, K - 1 - back] * x[:T - back]
    return y


def frequencies(rot):
    """``(f [dims / 2], multiplier of cos and sin)``: plain, or stretched by parts (YaRN) with ``scaling``."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if scaling is None:
        return torch.tensor(f, dtype=F), 1.0

    def index_at(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_at(scaling["fast"])), 0)
    hi = min(math.ceil(index_at(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot):
    """Turns the first ``dims`` entries of the heads of ``x`` ``[T, heads, D]``: entry ``2i`` with entry ``2i + 1``."""
    if rot is None:
        return x
    f, mult = frequencies(rot)
    angle = positions.to(F)[:, None] * f[None, :]
    cos, sin = (angle.cos() * mult)[:, None, :], (angle.sin() * mult)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * cos - v * sin
    out[..., 1:rot["dims"]:2] = v * cos + u * sin
    return out


def sink_softmax(s, seen, sink):
    """Weights ``exp(s) / (exp(sink) + sum exp(s))`` over the seen keys of ``s`` ``[T, T]``; ``sink`` None: no term."""
    s = s.masked_fill(~seen, -math.inf)
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = top.clamp(min=float(sink))
    e = torch.exp(s - top)
    below = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        below = below + torch.exp(sink - top)
    return e / below


def visible(T, window=None):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if window is None else (j <= i) & (i - j < window)


def attend(q, k, v, scale, cap=None, window=None, sink=None):
    """``q`` ``[T, H, D]``, ``k`` ``[T, G, D]``, ``v`` ``[T, G, V]``, ``sink`` ``[H]`` or None -> ``[T, H, V]``."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = visible(T, window)
    out = torch.zeros((T, H, v.shape[-1]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if cap is not None:
            s = cap * torch.tanh(s / cap)
        out[:, h] = sink_softmax(s, seen, None if sink is None else sink[h]) @ v[:, g]
    return out


# ------------------------------------------------------------------------------------------ the mixers

def attention_mixer(h, w, p, m, eps, positions):
    T = h.shape[0]

    def project(name):
        x = h @ w[p + name].T + w[p + name + ".b"]
        return causal_conv(x, w[p + name + ".conv"]) if m.get("conv") is not None else x

    q = norm(project("q"), w[p + "q.norm"], eps).reshape(T, m["heads"], m["dim"])
    k = norm(project("k"), w[p + "k.norm"], eps).reshape(T, m["kv_heads"], m["dim"])
    v = project("v").reshape(T, m["kv_heads"], m["vdim"])
    q, k = rotate(q, positions, m.get("rot")), rotate(k, positions, m.get("rot"))
    window = m["mask"]["size"] if m.get("mask") else None
    a = attend(q, k, v, m["scale"], m.get("softcap"), window, w[p + "sink"])
    return a.reshape(T, -1) @ w[p + "o"].T


def latent_mixer(h, w, p, m, eps, positions):
    T, H, D, R, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    q = (norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = norm(down[:, :rank], w[p + "dkv.norm"], eps)
    shared = rotate(down[:, None, rank:], positions, m["rot"])
    k = torch.cat([(c @ w[p + "uk"].T).reshape(T, H, D), shared.expand(T, H, R)], dim=-1)
    v = (c @ w[p + "uv"].T).reshape(T, H, m["vdim"])
    q = torch.cat([q[..., :D], rotate(q[..., D:], positions, m["rot"])], dim=-1)
    a = attend(q, k, v, m["scale"], sink=w[p + "sink"]).reshape(T, -1)
    return (a * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def decayed_recurrence(q, k, v, alpha):
    """``q``/``k``/``alpha`` ``[T, H, D]``, ``v`` ``[T, H, V]``: ``S <- diag(alpha) S + k v^T`` from zero, ``o = S^T q``."""
    T, H, D = q.shape
    S = torch.zeros((H, D, v.shape[-1]), dtype=q.dtype)
    out = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((q[t][:, :, None] * S).sum(dim=1))
    return torch.stack(out)


def channel_decay(z, tau):
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def gla_mixer(h, w, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    o = norm(decayed_recurrence(q, k, v, channel_decay(z, m["tau"]).reshape(T, H, D)), w[p + "norm"], eps)
    return (o.reshape(T, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------ the model

def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def run_order(cfg):
    """``[(layer, whether a pass begins in front of it)]``: the looped layers as often as the loop says."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        order += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence from its first token; ``layers_out`` (a list) receives the stream after
    every run of a layer."""
    eps = cfg["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x0 = w["embed"][torch.as_tensor(tokens)]
    x = x0
    for i, opens in run_order(cfg):
        if opens:
            x = torch.cat([x, x0], dim=-1) @ w["loop.in"].T
        layer, p = cfg["layers"][i], f"l{i}."
        m = layer["mixer"]
        h = norm(x, w[p + "norm1"], eps)
        if layer["type"] == "gla":
            y = gla_mixer(h, w, p + "mix.", m, eps)
        elif layer["type"] == "attention":
            y = attention_mixer(h, w, p + "mix.", m, eps, positions)
        else:
            y = latent_mixer(h, w, p + "mix.", m, eps, positions)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, w, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, w["final.norm"], eps) @ w["head"].T


def generate(cfg, w, prompt, n):
    """Greedy continuation: ``n`` tokens, each the largest logit (the lowest index among equals)."""
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(torch.argmax(forward(cfg, w, seq)[-1]))
        out.append(tok)
        seq.append(tok)
    return out
