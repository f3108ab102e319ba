"""Tiny Salulorn configurations for the tests: they differ in every size, constant and layer order."""

import json
import os

import torch


def rot(base, dims, *scaling):
    """``scaling``: nothing, or a factor with the original length, fast and slow."""
    out = dict(base=base, dims=dims)
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def dense(ff):
    return dict(kind="dense", ff=ff)


def gla(heads, dim, vdim, tau, rank, mlp):
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau, decay_rank=rank), mlp=mlp)


def attention(heads, kv_heads, dim, vdim, scale, mlp, conv=None, turn=None, window=None, cap=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if conv is not None:
        m["conv"] = conv
    if turn is not None:
        m["rot"] = turn
    if window is not None:
        m["mask"] = dict(size=window)
    if cap is not None:
        m["softcap"] = cap
    return dict(type="attention", mixer=m, mlp=mlp)


def latent(heads, dim, turn, vdim, q_rank, kv_rank, scale, mlp):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=turn["dims"], vdim=vdim, q_rank=q_rank,
                                                    kv_rank=kv_rank, scale=scale, rot=turn), mlp=mlp)


# the loop in the middle, three passes over an attention and a latent attention; a recurrence without a feed-forward in
# front, values wider and narrower than keys, half of a head turned, a window of 10, a low cap, four taps; an attention
# that has none of the optional things; sizes the plain kernels take
L_A = dict(architecture="Salulorn", vocab=210, width=72, norm=dict(eps=1e-6), loop=dict(start=1, stop=3, times=3), layers=[
    gla(3, 12, 8, 4.0, 5, None),
    attention(4, 2, 16, 24, 0.3, dense(40), 4, rot(100.0, 8), 10, 6.0),
    latent(3, 20, rot(500.0, 8, 3.0, 60, 4.0, 0.5), 12, 24, 40, 0.25, dense(56)),
    gla(2, 24, 36, 9.0, 11, dense(24)),
    attention(3, 1, 24, 8, 0.2, None),
])

# no loop; sizes that are no multiples of 8, one head of everything, tau 1, one tap, a window of 3, plain frequencies in
# the latent attention
L_B = dict(architecture="Salulorn", vocab=131, width=50, norm=dict(eps=1e-5), layers=[
    attention(2, 1, 10, 12, 0.4, dense(30), 1, rot(1000.0, 6), 3, 20.0),
    gla(1, 40, 33, 1.0, 3, dense(20)),
    latent(1, 7, rot(10000.0, 6), 9, 13, 21, 0.3, None),
    attention(3, 3, 9, 7, 0.3, dense(18), 3, None, 17),
])

# sizes the tensor-core kernels take: keys of 64 with values of 80 and of 128 with 48, windows of 65 and 64 around a page
# border, four query heads a key/value head and one; a recurrence of 128 x 64; latents of 96 and 208; the loop over the
# whole model, twice
L_C = dict(architecture="Salulorn", vocab=257, width=128, norm=dict(eps=1e-5), loop=dict(start=0, stop=4, times=2), layers=[
    latent(6, 48, rot(10000.0, 32, 8.0, 128, 32.0, 1.0), 64, 72, 96, 0.11, dense(192)),
    attention(8, 2, 64, 80, 0.12, dense(64), 3, rot(1e5, 64), 65, 30.0),
    gla(2, 128, 64, 16.0, 24, dense(128)),
    attention(4, 4, 128, 48, 0.09, None, 2, rot(30000.0, 64), 64, 45.0),
])

TINY_L = {"LA": L_A, "LB": L_B, "LC": L_C}


def random_config(rng):
    """A configuration drawn from ``rng`` (a ``random.Random``): two to six layers of any kind in any order, looped or not,
    every size, head count, window, cap, tap count and constant drawn anew."""
    def feed_forward():
        return None if rng.random() < 0.2 else dense(rng.choice([16, 40, 64, 96, 128, 200]))

    def turn(dims, stretched):
        scaling = ()
        if rng.random() < stretched:
            scaling = (rng.choice([1.0, 2.0, 4.0, 16.0]), rng.choice([32, 100, 4096]), rng.choice([8.0, 32.0]), rng.choice([0.5, 1.0]))
        return rot(rng.choice([100.0, 1e4, 1e6]), dims, *scaling)

    layers = []
    for _ in range(rng.randint(2, 6)):
        kind = rng.choice(["gla", "attention", "latent_attention"])
        if kind == "gla":
            layers.append(gla(rng.choice([1, 2, 3, 5]), rng.choice([4, 16, 24, 64, 100, 128, 200]), rng.choice([8, 24, 33, 64, 96]),
                              rng.choice([1.0, 5.0, 16.0]), rng.choice([1, 4, 16, 40]), feed_forward()))
        elif kind == "attention":
            kv, dim = rng.choice([1, 2, 4]), rng.choice([8, 16, 24, 32, 48, 64, 128])
            turned = None if rng.random() < 0.15 else turn(rng.choice([d for d in (2, 4, 8, 16, 32, 64, 128) if d <= dim]), 0.0)
            layers.append(attention(kv * rng.choice([1, 2, 3, 4]), kv, dim, rng.choice([8, 16, 32, 40, 64, 80, 128]),
                                    rng.choice([dim ** -0.5, 0.2, 0.1]), feed_forward(), rng.choice([None, 1, 2, 3, 4]), turned,
                                    rng.choice([None, 1, 2, 5, 17, 40, 64, 65, 100, 300]), rng.choice([None, 3.0, 15.0, 50.0])))
        else:
            layers.append(latent(rng.choice([1, 2, 3, 6]), rng.choice([8, 20, 32, 64]), turn(rng.choice([2, 8, 16, 32]), 0.7),
                                 rng.choice([8, 24, 64]), rng.choice([12, 40, 64]), rng.choice([16, 30, 64, 112, 256]),
                                 rng.choice([0.3, 0.15]), feed_forward()))
    out = dict(architecture="Salulorn", vocab=rng.choice([97, 200, 333, 500, 1000]), width=rng.choice([48, 64, 72, 96, 128, 160, 256]),
               norm=dict(eps=rng.choice([1e-6, 1e-5])), layers=layers)
    if rng.random() < 0.8:
        start = rng.randrange(len(layers))
        out["loop"] = dict(start=start, stop=rng.randint(start + 1, len(layers)), times=rng.choice([1, 2, 3]))
    return out


def make_salulorn_folder(tmp_path, name, seed=0, dtype=torch.float32, raw=None):
    """A model folder of the tiny configuration ``name`` (or of ``raw``, a configuration given as it is)."""
    from starter_b200.config import config_from_dict
    from starter_b200.weights import write_model_folder

    raw = TINY_L[name] if raw is None else raw
    path = os.path.join(str(tmp_path), f"tiny_{name}_{seed}")
    write_model_folder(path, config_from_dict(raw), seed, dtype)
    # the rank of a decay is left to the checkpoint, as in a model that was not drawn by the library
    with open(os.path.join(path, "config.json")) as handle:
        stored = json.load(handle)
    for layer in stored["layers"]:
        layer["mixer"].pop("decay_rank", None)
    with open(os.path.join(path, "config.json"), "w") as handle:
        json.dump(stored, handle)
    # The library draws matrices from N(0, 0.02): with those every score is near 0, every softmax near uniform, every
    # decay the same, and a wrong key, a lost state or a window that is one token off would hardly show.  Larger
    # matrices give scores of order one, the sinks spread from next to nothing to most of the softmax, the decays from
    # short to long memory; the loop's projection keeps some of the stream so that early passes still count.
    from safetensors.torch import load_file, save_file

    file = os.path.join(path, "model.safetensors")
    tensors = load_file(file)
    for key, value in tensors.items():
        v = value.float()
        if key == "embed":
            v = v * 100.0
        elif key == "loop.in":
            v = v * 4.0
            v[:, :v.shape[0]] += 0.6 * torch.eye(v.shape[0])
        elif key.endswith((".q.norm", ".k.norm")):
            v = v * 1.5
        elif key.endswith(".sink"):
            v = torch.linspace(-1.0, 3.0, v.numel()) + v
        elif key.endswith(".a2"):
            v = v * 20.0
        elif key.endswith(".a2.b"):
            v = torch.linspace(5.0, -2.0, v.numel()) + v
        elif key.endswith(".conv"):
            v = v * 5.0
            v[:, -1] += 0.5
        elif key.endswith((".uq", ".uk")):
            v = v * 10.0
        elif value.dim() == 2:
            v = v * 5.0
        elif key.endswith(".b"):
            v = v * 10.0
        tensors[key] = v.to(value.dtype)
    save_file(tensors, file, metadata={"format": "pt"})
    return path
