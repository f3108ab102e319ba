"""Tiny Setotar configurations for the tests: they differ in every size, constant and layer order."""

import os

import torch


def rot(base, dims, *scaling):
    """``scaling``: nothing, a factor, or a factor with the original length, fast and slow."""
    out = dict(base=base, dims=dims)
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def attention(heads, kv_heads, dim, vdim, scale, mlp, turn=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if turn is not None:
        m["rot"] = turn
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m, mlp=mlp)


def left(heads, kv_heads, dim, vdim, scale, conv=None, turn=None, window=None, keep=None, cap=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if conv is not None:
        m["conv"] = conv
    if turn is not None:
        m["rot"] = turn
    if window is not None:
        m["mask"] = dict(size=window) if keep is None else dict(size=window, keep_first=keep)
    if cap is not None:
        m["softcap"] = cap
    return m


def right(heads, dim, vdim):
    return dict(heads=heads, dim=dim, vdim=vdim)


def parallel(left_side, right_side, left_scale, right_scale, mlp):
    return dict(type="parallel", mixer=dict(left=left_side, right=right_side, left_scale=left_scale,
                                            right_scale=right_scale), mlp=mlp)


def moe(experts, top, ff):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


# the parallel mixer first, three taps, values wider than keys, a window of 10 that keeps three keys, a low cap; an
# attention without a feed-forward whose keys and values two later layers read (one of them behind another mixer),
# with another number of query heads; a parallel mixer that sees everything, without a cap, with one tap
_YARN_A = rot(500.0, 12, 8.0, 64, 4.0, 0.5)
S_A = dict(architecture="Setotar", vocab=200, width=64, streams=2, norm=dict(eps=1e-5), layers=[
    parallel(left(4, 2, 16, 24, 0.3, 3, rot(100.0, 8, 4.0), 10, 3, 4.0), right(3, 12, 8), 0.7, 0.9, moe(5, 2, 24)),
    attention(4, 2, 16, 8, 0.25, None, _YARN_A),
    attention(6, 2, 16, 8, 0.3, moe(4, 1, 40), _YARN_A, kv_from=1),
    parallel(left(2, 2, 8, 16, 0.4, 1, rot(50.0, 2)), right(1, 20, 24), -0.4, 1.3, None),
    attention(4, 2, 16, 8, 0.2, moe(3, 2, 16), _YARN_A, kv_from=1),
])

# one stream; one head of 24 without rotation, all of three experts; a window of 3 that keeps one key, no convolution,
# no cap, the whole head turned; a state of 40 x 33; a window that keeps nothing, four taps, sizes that are no multiples
# of 8
S_B = dict(architecture="Setotar", vocab=131, width=96, streams=1, norm=dict(eps=1e-6), layers=[
    attention(1, 1, 24, 40, 0.2, moe(3, 3, 32)),
    parallel(left(2, 1, 24, 24, 0.2, None, rot(10000.0, 24), 3, 1), right(1, 40, 33), 0.5, 0.5, moe(4, 1, 16)),
    attention(1, 1, 24, 40, 0.15, moe(4, 3, 24), kv_from=0),
    parallel(left(3, 3, 10, 12, 0.3, 4, rot(1000.0, 6, 2.0), 17, None, 30.0), right(2, 6, 10), 1.0, -0.25, None),
])

# sizes the tensor-core kernels take: keys of 64 with values of 80, windows of 65 and 64 around a page border that keep
# 70 keys (more than a page) and one, four query heads a key/value head and one; keys of 128 with values of 48; states
# of 128 and 64 rows; four streams; one expert of eight; an attention with heads of 64 read by one with twice the heads
S_C = dict(architecture="Setotar", vocab=257, width=128, streams=4, norm=dict(eps=1e-5), layers=[
    attention(4, 2, 64, 64, 0.125, moe(8, 1, 64), rot(10000.0, 32, 4.0, 128, 32.0, 1.0)),
    parallel(left(8, 2, 64, 80, 0.11, 3, rot(10000.0, 32, 2.0), 65, 70, 20.0), right(2, 128, 64), 0.65, 0.55, moe(8, 2, 32)),
    attention(8, 2, 64, 64, 0.125, None, rot(10000.0, 32, 4.0, 128, 32.0, 1.0), kv_from=0),
    parallel(left(4, 4, 128, 48, 0.09, 2, rot(30000.0, 64), 64, 1, 45.0), right(4, 64, 32), 0.8, 0.7, moe(8, 3, 32)),
])

TINY_S = {"SA": S_A, "SB": S_B, "SC": S_C}


def random_config(rng):
    """A configuration drawn from ``rng`` (a ``random.Random``): two to six layers of any kind in any order, some of
    them reading an earlier layer's keys and values, every size, head count, window, cap, tap count and constant drawn
    anew."""
    def feed_forward():
        if rng.random() < 0.2:
            return None
        experts = rng.choice([1, 2, 3, 4, 6, 8, 12, 17])
        return moe(experts, rng.randint(1, min(experts, 4)), rng.choice([16, 24, 32, 48, 64]))

    def turn(dim, kinds=(0, 1, 4)):
        if rng.random() < 0.15:
            return None
        kind = rng.choice(kinds)
        scaling = {0: (), 1: (rng.choice([1.0, 2.0, 5.5]),),
                   4: (rng.choice([1.0, 2.0, 4.0, 16.0]), rng.choice([32, 100, 4096]), rng.choice([8.0, 32.0]), rng.choice([0.5, 1.0]))}[kind]
        return rot(rng.choice([100.0, 1e4, 1e6]), rng.choice([d for d in (2, 4, 8, 16, 32, 64, 128) if d <= dim]), *scaling)

    layers = []
    for i in range(rng.randint(2, 6)):
        own = [j for j, made in enumerate(layers) if made["type"] == "attention" and "kv_from" not in made["mixer"]]
        if own and rng.random() < 0.4:
            source = rng.choice(own)
            m = layers[source]["mixer"]
            layers.append(attention(m["kv_heads"] * rng.choice([1, 2, 3]), m["kv_heads"], m["dim"], m["vdim"],
                                    rng.choice([m["scale"], 0.2]), feed_forward(), m.get("rot"), kv_from=source))
            continue
        kv, dim, vdim = rng.choice([1, 2, 4]), rng.choice([8, 16, 24, 32, 48, 64, 128]), rng.choice([8, 16, 32, 40, 64, 80, 128])
        heads, scale = kv * rng.choice([1, 2, 3, 4]), rng.choice([dim ** -0.5, 0.2, 0.1])
        if rng.random() < 0.5:
            layers.append(attention(heads, kv, dim, vdim, scale, feed_forward(), turn(dim)))
            continue
        window = rng.choice([None, 1, 2, 5, 17, 40, 64, 65, 100, 300])
        side = left(heads, kv, dim, vdim, scale, rng.choice([None, 1, 2, 3, 4]), turn(dim),
                    window, rng.choice([None, 0, 1, 4, 63, 64, 66]), rng.choice([None, 2.0, 15.0, 50.0]))
        layers.append(parallel(side, right(rng.choice([1, 2, 3]), rng.choice([4, 16, 24, 64, 100, 128]), rng.choice([8, 24, 33, 64])),
                               rng.choice([0.3, 1.0, -0.7]), rng.choice([0.5, 1.2]), feed_forward()))
    return dict(architecture="Setotar", vocab=rng.choice([97, 200, 333, 500, 1000]), width=rng.choice([48, 64, 72, 96, 128, 160, 256]),
                streams=rng.choice([1, 2, 3, 4, 8]), norm=dict(eps=rng.choice([1e-6, 1e-5])), layers=layers)


def make_setotar_folder(tmp_path, name, seed=0, dtype=torch.float32, raw=None):
    """A model folder of the tiny configuration ``name`` (or of ``raw``, a configuration given as it is)."""
    from starter_b200.config import config_from_dict
    from starter_b200.weights import write_model_folder

    raw = TINY_S[name] if raw is None else raw
    path = os.path.join(str(tmp_path), f"tiny_{name}_{seed}")
    write_model_folder(path, config_from_dict(raw), seed, dtype)
    # The library draws matrices from N(0, 0.02): with those every score is near 0, every softmax near uniform, every
    # forget gate the same, and a wrong key, a lost state or a window that is one token off would hardly show.  Larger
    # matrices give scores of order one and routers that decide; forget gates spread from short to long memory; the
    # mixing matrices stay near the identity so that early layers still count at the end.
    from safetensors.torch import load_file, save_file

    file = os.path.join(path, "model.safetensors")
    tensors = load_file(file)
    for key, value in tensors.items():
        v = value.float()
        if key == "embed":
            v = v * 100.0
        elif key.endswith((".left.q", ".left.k")):
            v = v * 14.0
        elif key.endswith((".q.norm", ".k.norm")):
            v = v * 1.5
        elif key.endswith(".router"):
            v = v * 40.0
        elif key.endswith(".lower"):
            v = (torch.linspace(0.0, 0.9, v.numel()) + 0.3 * (v - 0.4)).clamp(0.0, 0.97)
        elif key.endswith(".f.b"):
            v = torch.linspace(6.0, -2.0, v.numel()) + v
        elif key.endswith(".conv"):
            v = v * 5.0
        elif key.endswith(".mix"):
            v = 0.75 * torch.eye(v.shape[0]) + 0.3 * v
        elif value.dim() == 2:
            v = v * 5.0
        elif key.endswith(".b"):
            v = v * 10.0
        tensors[key] = v.to(value.dtype)
    save_file(tensors, file, metadata={"format": "pt"})
    return path
