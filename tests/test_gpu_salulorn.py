"""Salulorn on the GPU against the plain statement: each mechanism alone, then the model through the step function, the
cache, the state slots and the generation loop, cut into steps and batches in every way."""

import copy

import pytest
import torch

import plain_salulorn as plain
from gpu_helpers import DTYPES, FP32_TOL
from tiny import random_prompt
from tiny_salulorn import TINY_L, make_salulorn_folder, rot

pytestmark = pytest.mark.gpu

CONFIGS = ["LA", "LB", "LC"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64
_cases, _runners, _wanted = {}, {}, {}


def case(tmp_path_factory, name, seed=1):
    if (name, seed) not in _cases:
        folder = make_salulorn_folder(tmp_path_factory.mktemp(f"l{name}{seed}"), name, seed=seed)
        _cases[(name, seed)] = (folder,) + plain.read_model_folder(folder)
    return _cases[(name, seed)]


def runner_for(tmp_path_factory, name, dtype, max_tokens=64 * 40):
    from starter_b200.engine import ModelRunner, load_model

    if (name, dtype) not in _runners:
        folder, _, _ = case(tmp_path_factory, name)
        _runners[(name, dtype)] = ModelRunner(load_model(folder, dtype), max_tokens=max_tokens, max_sequences=12)
    return _runners[(name, dtype)]


def wanted(name, cfg, w, prompt):
    """The plain logits, computed once for both number formats."""
    key = (name, tuple(prompt))
    if key not in _wanted:
        _wanted[key] = plain.forward(cfg, w, prompt)
    return _wanted[key]


def close(got, want, dtype, what, fp32=2e-5, bf16=2e-2):
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(want.shape)}"
    tol = (fp32 if dtype in ("float32", torch.float32) else bf16) * float(want.abs().max())
    err = (got - want).abs()
    assert float(err.max()) <= tol, f"{what}: off by {float(err.max()):.3e} (allowed {tol:.3e}) at {tuple(int(i) for i in (err == err.max()).nonzero()[0])}"


# Bounds of the model-level comparisons, relative to the largest logit of the case: float32 as for the other designs;
# bfloat16 against the float64 statement a row may be off by 6e-2 and the mean over a comparison by 1e-2.  A lost state,
# a key that is one off or a skipped layer moves rows by 1e-1 and more, and the float32 runs of the same kernels hold
# every row to 2e-5.
BF16_ROW_TOL = 6e-2
BF16_MEAN_TOL = 1e-2


def assert_close(got, want, dtype, what=""):
    """Fails with the first wrong row named: its place is the clue (a prompt's end, the first single-token step, a
    page border, a window's edge)."""
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(want.shape)}"
    scale = float(want.abs().max())
    tol = (FP32_TOL if dtype == "float32" else BF16_ROW_TOL) * scale
    err = (got - want).abs().reshape(want.shape[0], -1).max(dim=1).values
    bad = (~(err <= tol)).nonzero().flatten().tolist()
    assert not bad, (f"{what}: {len(bad)} of {len(err)} rows off by more than {tol:.2e}; first wrong row {bad[0]} "
                     f"(error {err[bad[0]].item():.3e}), largest error {err.max().item():.3e}")
    if dtype != "float32":
        mean = (got - want).abs().mean().item()
        assert mean <= BF16_MEAN_TOL * scale, f"{what}: mean error {mean:.3e} above {BF16_MEAN_TOL * scale:.3e}"


def dev(v, ty=torch.float32):
    return v.to("cuda", ty).contiguous()


def ints(a):
    return torch.tensor(a, dtype=torch.int32, device="cuda")


def packed(lengths, slots):
    """(seq_slot, seq_q_start, seq_q_len) on the device for sequences packed one after another."""
    starts = [sum(lengths[:i]) for i in range(len(lengths))]
    return ints(slots), ints(starts), ints(lengths)


def turned(turn, t, length=400):
    from starter_b200.config.salulorn import _position
    from starter_b200.parts.rotary import InterleavedRotaryTable

    if turn is None:
        return None
    table = InterleavedRotaryTable(_position(turn), t, "cuda")
    table.ensure(length)
    return table.rotation()


# ------------------------------------------------------------------------------ mechanisms alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [40, 37, 600, 5000])
def test_two_outputs_added_together_and_a_norm(hidden, dtype):
    """The sum that closes a layer whose sublayers ran side by side, and the next norm, in one kernel; selected rows leave
    the stream as it was."""
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(hidden)
    x, y, z, gain = (torch.randn(*s, generator=g, dtype=F) for s in ((9, hidden), (9, hidden), (9, hidden), (hidden,)))
    x[3], y[3], z[3] = x[3] * 1e-3, y[3] * 1e-3, z[3] * 1e-3          # a row whose eps matters
    xd, yd, zd = dev(x), dev(y, t), dev(z, t)
    new = xd.double().cpu() + yd.double().cpu() + zd.double().cpu()
    want = plain.norm(new, gain.float().double(), 1e-5)
    got = ops.residual_norm(xd, t, 1e-5, (yd, None, None, 0.0, zd), dev(gain), rows=ints([8, 3]))
    close(got, want[[8, 3]], dtype, "selected rows", fp32=1e-6, bf16=8e-3)
    assert torch.equal(xd, dev(x))
    got = ops.residual_norm(xd, t, 1e-5, (yd, None, None, 0.0, zd), dev(gain))
    close(got, want, dtype, "norm of the sum", fp32=1e-6, bf16=8e-3)
    close(xd, new, "float32", "the stream", fp32=1e-6)
    # one output alone, in both spellings
    one, two = dev(x), dev(x)
    ops.residual_norm(one, t, 1e-5, (yd, None, None, 0.0), dev(gain))
    ops.residual_norm(two, t, 1e-5, (yd, None, None, 0.0, None), dev(gain))
    assert torch.equal(one, two)
    close(one, x.float().double() + yd.double().cpu(), "float32", "one output", fp32=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [40, 37, 600, 5000])
def test_stream_and_embedding_side_by_side(hidden, dtype):
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(hidden + 1)
    x, y, z, table = (torch.randn(n, hidden, generator=g, dtype=F) for n in (6, 6, 6, 11))
    tokens = [10, 0, 3, 3, 7, 1]
    xd, yd, zd, td = dev(x), dev(y, t), dev(z, t), dev(table, t)
    embedded = td.double().cpu()[tokens]
    for pending, total in ((None, xd.double().cpu()), ((yd, None, None, 0.0), xd.double().cpu() + yd.double().cpu()),
                           ((yd, None, None, 0.0, zd), xd.double().cpu() + yd.double().cpu() + zd.double().cpu())):
        got = ops.residual_join(xd, pending, ints(tokens), td, 0.5)
        close(got, torch.cat([total, 0.5 * embedded], dim=1), dtype, "joined row", fp32=1e-6, bf16=8e-3)
        assert got.dtype == t and torch.equal(xd, dev(x))
    with pytest.raises(ops.KernelError, match="norm"):
        ops.residual_join(xd, (yd, dev(torch.ones(hidden)), None, 1e-5), ints(tokens), td)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, cols", [(64, 200), (37, 41), (1024, 3000), (8, 8)])
def test_output_gate_alone(width, cols, dtype):
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(width)
    a, z = dev(torch.randn(7, width, generator=g, dtype=F), t), dev(torch.randn(7, cols, generator=g, dtype=F) * 4.0, t)
    for at in {0, cols - width, (cols - width) // 2}:
        b = a.clone()
        ops.sigmoid_gate(b, z, at)
        close(b, a.double().cpu() * torch.sigmoid(z.double().cpu()[:, at:at + width]), dtype, f"from {at}", fp32=1e-6, bf16=8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tau", [1.0, 7.0, 16.0])
@pytest.mark.parametrize("rank, channels, tokens", [(1, 12, 1), (5, 40, 9), (16, 300, 70), (100, 129, 8), (24, 256, 33)])
def test_low_rank_decay_alone(rank, channels, tokens, tau, dtype):
    """Decays from next to nothing to next to one; the complement keeps its digits where the decay is close to one."""
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(rank * 10 + channels)
    u = dev(torch.randn(tokens, rank + 6, generator=g, dtype=F), t)
    a2 = torch.randn(rank, channels, generator=g, dtype=F) / rank ** 0.5
    bias = torch.linspace(12.0, -12.0, channels, dtype=F)
    z = u.double().cpu()[:, 3:3 + rank] @ a2.float().double() + bias.float().double()
    want = -torch.expm1(torch.nn.functional.logsigmoid(z) / tau)
    got = ops.low_rank_decay(u, 3, dev(a2), dev(bias), tau).double().cpu()
    assert got.shape == want.shape
    assert float(((got - want).abs() / want).max()) < 3e-5
    close(1.0 - got, plain.channel_decay(z, tau), "float32", "decay", fp32=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, n, v", [(3, 12, 8), (1, 40, 33), (2, 128, 64), (4, 64, 32), (2, 1, 1), (1, 256, 20), (5, 5, 100), (48, 100, 32)])
def test_decayed_recurrence_alone(heads, n, v, dtype):
    """Three sequences whole, then in portions down to one token that cross the kernel's chunks, in state slots with
    floats of others around them; decays from next to nothing to next to one, and a first value that must still show at
    the end."""
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(heads * 1000 + n)
    lengths, slots = [300, 1, 17], [2, 0, 3]
    total = sum(lengths)
    q, k = torch.randn(total, heads * n, generator=g, dtype=F), torch.randn(total, heads * n, generator=g, dtype=F)
    val = torch.randn(total, heads * v, generator=g, dtype=F)
    val[0] = 60.0
    let_go = torch.rand(total, heads * n, generator=g, dtype=F) * torch.logspace(-5, 0, heads * n, dtype=F).flip(0)[None]
    let_go[:, 0] = 1e-4                                   # a row that forgets next to nothing
    decay = dev(let_go)
    proj = dev(torch.cat([torch.zeros(total, 3, dtype=F), q, k, val], dim=1), t)
    seen = proj.double().cpu()[:, 3:].split([heads * n, heads * n, heads * v], dim=1)
    qq, kk = (x.reshape(total, heads, n) for x in seen[:2])
    vv, alpha = seen[2].reshape(total, heads, v), 1.0 - decay.double().cpu().reshape(total, heads, n)
    want, at = [], 0
    for length in lengths:
        part = slice(at, at + length)
        want.append(plain.decayed_recurrence(qq[part] * n ** -0.5, kk[part], vv[part], alpha[part]))
        at += length
    forgot = vv[:300].clone()
    forgot[0] = 0.0
    forgot = plain.decayed_recurrence(qq[:300] * n ** -0.5, kk[:300], forgot, alpha[:300])
    assert float((forgot[280:] - want[0][280:]).abs().max()) > 0.02
    want = torch.cat(want).reshape(total, heads * v)
    state_at = 5
    state = torch.zeros(4, state_at + heads * n * v + 2, device="cuda")
    state[:, :state_at] = 7.0
    state[:, -2:] = 8.0

    def run(p, d, lens, sl):
        return ops.state_scan("channel_decay", (p, 3), (p, 3 + heads * n), (p, 3 + 2 * heads * n), None, None, None, None, None,
                              state, state_at, *packed(lens, sl), heads, heads, n, v, decay=d)

    close(run(proj, decay, lengths, slots), want, dtype, "whole", fp32=2e-5, bf16=2e-5)        # (the inputs are the same bits)
    assert float((state[:, :state_at] - 7.0).abs().max()) == 0.0 and float((state[:, -2:] - 8.0).abs().max()) == 0.0
    assert float(state[1, state_at:-2].abs().max()) == 0.0
    state[:, state_at:-2] = 0.0
    got, done, bases = [[], [], []], [0, 0, 0], [0, 300, 301]
    for sizes in ([1, 1, 1], [2, 0, 1], [16, 0, 15], [33, 0, 0], [248, 0, 0]):
        live = [i for i in range(3) if sizes[i]]
        rows = torch.cat([torch.arange(bases[i] + done[i], bases[i] + done[i] + sizes[i]) for i in live]).cuda()
        out = run(proj[rows].contiguous(), decay[rows].contiguous(), [sizes[i] for i in live], [slots[i] for i in live])
        at = 0
        for i in live:
            got[i].append(out[at:at + sizes[i]])
            at += sizes[i]
            done[i] += sizes[i]
    close(torch.cat([torch.cat(p) for p in got]), want, dtype, "in portions", fp32=2e-5, bf16=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, turn, row_norm, unit", [
    (4, 2, 16, 24, rot(100.0, 8), True, False), (3, 1, 64, 32, rot(2e3, 24, 3.0, 300, 20.0, 2.0), True, True),
    (1, 1, 9, 7, None, True, False), (3, 3, 10, 12, rot(1e3, 6), True, False), (8, 1, 128, 80, rot(1e4, 128), True, False),
    (2, 2, 8, 16, rot(30.0, 2), True, False), (12, 4, 40, 40, rot(1e5, 12), False, True)])
def test_row_norms_with_turned_pairs(heads, kv_heads, dim, vdim, turn, row_norm, unit, dtype):
    """Norm over the whole row, neighbouring entries turned together: queries in place, keys and values in the cache on
    both sides of page borders."""
    from starter_b200 import ops

    t, n, eps = TORCH[dtype], 200, 1e-5
    g = torch.Generator().manual_seed(heads * 100 + dim)
    widths = [heads * dim, kv_heads * dim, kv_heads * vdim]
    proj = torch.randn(n, sum(widths) + (-sum(widths) % 8), generator=g, dtype=F) * 2.0
    proj[3] *= 1e-3                                      # a row whose eps matters
    proj = dev(proj, t)
    q, k, v = (p.double().cpu() for p in proj[:, :sum(widths)].split(widths, dim=1))
    gains = (torch.randn(widths[0], generator=g, dtype=F), torch.randn(widths[1], generator=g, dtype=F))
    if row_norm:
        q, k = plain.norm(q, gains[0].float().double(), eps), plain.norm(k, gains[1].float().double(), eps)
    place = torch.arange(n) + 37
    q = plain.rotate(q.reshape(n, heads, dim), place, turn)
    k = plain.rotate(k.reshape(n, kv_heads, dim), place, turn)
    v = v.reshape(n, kv_heads, vdim)
    v = plain.norm(v, torch.ones(vdim, dtype=F), eps) if unit else v
    table = torch.zeros(3, 8, dtype=torch.int32, device="cuda")
    table[1, :5] = ints([5, 2, 7, 0, 3])
    ks = torch.zeros(8, kv_heads, 64, dim, dtype=t, device="cuda")
    vs = torch.zeros(8, kv_heads, 64, vdim, dtype=t, device="cuda")
    pos, slot = dev(place, torch.int32), ints([1] * n)
    norms = (dev(gains[0]), dev(gains[1])) if row_norm else None
    ops.sink_prepare_norm(proj, heads, kv_heads, dim, vdim, pos, slot, table, ks, vs, turned(turn, t), norms, unit, eps)
    close(proj[:, :widths[0]], q.reshape(n, -1), dtype, "queries", fp32=1e-6, bf16=8e-3)
    pages = torch.tensor([5, 2, 7, 0, 3])[place // 64]
    close(ks[pages.cuda(), :, (place % 64).cuda()], k, dtype, "keys", fp32=1e-6, bf16=8e-3)
    close(vs[pages.cuda(), :, (place % 64).cuda()], v, dtype, "values", fp32=1e-6, bf16=8e-3)
    assert float(ks[5, :, :37].abs().max()) == 0.0 and float(vs[3].abs().max()) == 0.0, "nothing else was written"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, cap", [
    (4, 2, 16, 24, 10, 20.0), (1, 1, 24, 40, 3, None), (8, 2, 64, 80, 65, 30.0), (4, 4, 128, 48, 64, 50.0), (5, 1, 128, 72, 99, 25.0),
    (2, 2, 10, 12, 17, 20.0), (3, 1, 64, 128, 130, None), (6, 2, 64, 64, None, 15.0), (2, 2, 128, 128, 1, 40.0), (1, 1, 200, 136, 70, 30.0)])
def test_window_attention_with_a_sink_and_a_cap_alone(heads, kv_heads, dim, vdim, window, cap, dtype):
    """A sequence of 300 over five scattered pages.  Queries late in the sequence aim at one key, so that its score stands
    out: the oldest inside their window, the one just outside it, keys on either side of a page border, their own place.
    Sinks from far below the scores to above the largest.  Plain, ``mma.sync`` and tcgen05 kernels, whole, as a later
    portion and as the last token alone in 1, 3 and 7 parts."""
    from starter_b200 import ops

    t, n, scale = TORCH[dtype], 300, 0.25
    g = torch.Generator().manual_seed(heads * 100 + dim + vdim)
    group = heads // kv_heads
    q = torch.randn(n, heads, dim, generator=g, dtype=F)
    k = torch.randn(n, kv_heads, dim, generator=g, dtype=F)
    v = torch.randn(n, kv_heads, vdim, generator=g, dtype=F)
    span = window or n
    aim = 12.0
    probes = {280: 280, 299: 0, 250: 191, 251: 192, 130: 63, 131: 64}
    for at in (298, 257, 200, 193, 128):
        probes[at] = max(at - span + 1, 0)               # the oldest key inside the window
        probes[at - 1] = max(at - 1 - span, 0)           # the key just outside it
    for at, key in probes.items():
        for h in range(heads):
            target = k[key, h // group]
            q[at, h] = target / target.norm() ** 2 * (aim / scale)
    sink = torch.linspace(8.0, -2.0, heads, dtype=F) if heads > 1 else torch.tensor([6.0], dtype=F)
    width = heads * dim
    proj = torch.zeros(n, width + (-width % 8), dtype=F)
    proj[:, :width] = q.reshape(n, -1)
    proj = dev(proj, t)
    table = torch.zeros(3, 8, dtype=torch.int32, device="cuda")
    pages = [5, 2, 7, 0, 3]
    table[1, :5] = ints(pages)
    ks = dev(torch.randn(8, kv_heads, 64, dim, generator=g) * 50.0, t)        # stale contents everywhere else
    vs = dev(torch.randn(8, kv_heads, 64, vdim, generator=g) * 50.0, t)
    place = torch.arange(n)
    where = torch.tensor(pages)[place // 64].cuda(), (place % 64).cuda()
    ks[where[0], :, where[1]] = dev(k, t)
    vs[where[0], :, where[1]] = dev(v, t)
    args = (proj.double().cpu()[:, :width].reshape(n, heads, dim), dev(k, t).double().cpu(), dev(v, t).double().cpu(), scale, cap)
    sk = sink.float().double()
    want = plain.attend(*args, window, sk).reshape(n, heads * vdim)
    others = [(None, "no sink")] + ([] if window is None else [(window + 1, "wider")] + ([(window - 1, "narrower")] if window > 1 else []))
    for wrong, what in others:                           # an edge that is one off, or a lost sink, must show
        other = plain.attend(*args, window if what == "no sink" else wrong, None if what == "no sink" else sk)
        assert float((other.reshape(n, -1) - want).abs().max()) > 0.1, what
    pos, slot = dev(place, torch.int32), ints([1] * n)
    rest = dict(window=window, softcap=cap, sink=dev(sink))
    out = ops.sink_attention(proj, ks, vs, table, slot, pos, heads, kv_heads, dim, vdim, scale, **rest)
    close(out, want, dtype, "plain kernel, whole", bf16=3e-2)
    if dtype == "float32" or not ops.sink_tc_takes(proj, heads, kv_heads, dim, vdim):
        assert dtype == "float32" or max(dim, vdim) > 128 or dim % 8 or vdim % 8
        return
    out = ops.sink_attention_tc(proj, ks, vs, table, ints([1]), ints([0]), ints([n]), ints([n]), ints([0, 0, 0, 0, 0]),
                                ints([128, 0, 256, 192, 64]), heads, kv_heads, dim, vdim, scale, **rest)
    close(out, want, dtype, "tensor cores, whole", bf16=3e-2)
    out = ops.sink_attention_tc(proj[260:].contiguous(), ks, vs, table, ints([1]), ints([0]), ints([40]), ints([n]), ints([0]),
                                ints([0]), heads, kv_heads, dim, vdim, scale, **rest)
    close(out, want[260:], dtype, "tensor cores, a later portion", bf16=3e-2)
    for last in (300, 299, 296):
        for parts in (1, 3, 7):
            out = ops.sink_attention_tc(proj[last - 1:last].contiguous(), ks, vs, table, ints([1]), ints([0]), ints([1]), ints([last]),
                                        ints([0]), ints([0]), heads, kv_heads, dim, vdim, scale, n_splits=parts, **rest)
            close(out, want[last - 1:last], dtype, f"tensor cores, token {last - 1} in {parts} parts", bf16=3e-2)
    if not ops.sink_tcgen05_takes(proj, dim, vdim):
        return
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    out = ops.sink_attention_tcgen05(proj, ks, vs, table, ints([1]), ints([0]), ints([n]), ints([n]), ints([0, 0, 0, 0, 0]),
                                     ints([128, 0, 256, 192, 64]), heads, kv_heads, dim, scale, status=status,
                                     blocks=(ints([0, 0]), ints([0, 256])), vdim=vdim, **rest)
    close(out, want, dtype, "tcgen05, whole", bf16=3e-2)
    late = slice(130, 300)
    out = ops.sink_attention_tcgen05(proj[late].contiguous(), ks, vs, table, ints([1]), ints([0]), ints([170]), ints([n]),
                                     ints([0, 0, 0]), ints([0, 64, 128]), heads, kv_heads, dim, scale, status=status, vdim=vdim, **rest)
    close(out, want[late], dtype, "tcgen05, a later portion", bf16=3e-2)
    assert int(status.item()) == 0


def absorbed(q, c, shared, scale, window, sink):
    """The latent attention with the key up-projection folded into the queries: ``q`` ``[T, H, rank + rot]``, ``c`` ``[T, rank]``,
    ``shared`` ``[T, rot]`` -> the weighted sums of the latents ``[T, H, rank]``."""
    return plain.attend(q, torch.cat([c, shared], dim=1)[:, None], c[:, None], scale, None, window, sink)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, rank, rot_dim, window", [(3, 40, 8, None), (1, 21, 6, None), (6, 96, 32, None), (16, 128, 64, None),
                                                          (70, 64, 16, None), (4, 512, 64, None), (5, 208, 16, 70)])
def test_latent_attention_with_a_sink_alone(heads, rank, rot_dim, window, dtype):
    """A sequence of 300 over five scattered pages; queries that aim at the first key, at keys around page borders and at
    their own; sinks from far below the scores to above them.  Whole, as a later portion, single tokens in parts."""
    from starter_b200 import ops

    t, n, scale, row = TORCH[dtype], 300, 0.2, rank + rot_dim
    g = torch.Generator().manual_seed(heads * 10 + rank)
    q = torch.randn(n, heads, row, generator=g, dtype=F)
    rows = torch.randn(n, row, generator=g, dtype=F)
    for at, key in {299: 0, 298: 298, 297: 64, 250: 63, 130: 127, 131: 128, 40: 31, 41: 32}.items():
        q[at] = rows[key] / rows[key].norm() ** 2 * (12.0 / scale)
    q, rows = dev(q, t), dev(rows, t)
    sink = torch.linspace(9.0, -2.0, heads, dtype=F) if heads > 1 else torch.tensor([5.0], dtype=F)
    table = torch.zeros(3, 8, dtype=torch.int32, device="cuda")
    pages = [5, 2, 7, 0, 3]
    table[1, :5] = ints(pages)
    store = dev(torch.randn(8, 1, 64, row, generator=g) * 50.0, t)             # stale contents everywhere else
    place = torch.arange(n)
    store[torch.tensor(pages)[place // 64].cuda(), 0, (place % 64).cuda()] = rows
    r64 = rows.double().cpu()
    args = (q.double().cpu(), r64[:, :rank], r64[:, rank:], scale, window)
    want = absorbed(*args, sink.float().double())
    assert float((absorbed(*args, None) - want).abs().max()) > 0.1             # a lost sink must show
    sd, pos, slot = dev(sink), dev(place, torch.int32), ints([1] * n)
    out = ops.latent_attention(q, store, table, slot, pos, heads, rank, rot_dim, scale, window, sd)
    close(out, want, dtype, "plain kernel, whole", bf16=3e-2)
    if not ops.latent_tc_takes(t, rank, rot_dim):
        assert dtype == "float32" or rank % 16 or rot_dim % 16
        return
    out = ops.latent_attention_tc(q, store, table, ints([1]), ints([0]), ints([n]), ints([n]), ints([0, 0, 0, 0, 0]),
                                  ints([128, 0, 256, 192, 64]), heads, rank, rot_dim, scale, window, sink=sd)
    close(out, want, dtype, "tensor cores, whole", bf16=3e-2)
    out = ops.latent_attention_tc(q[260:].contiguous(), store, table, ints([1]), ints([0]), ints([40]), ints([n]), ints([0]), ints([0]),
                                  heads, rank, rot_dim, scale, window, sink=sd)
    close(out, want[260:], dtype, "tensor cores, a later portion", bf16=3e-2)
    for last in (300, 299, 298, 42):
        for parts in (1, 3, 7, 32):
            out = ops.latent_attention_tc(q[last - 1:last].contiguous(), store, table, ints([1]), ints([0]), ints([1]), ints([last]),
                                          ints([0]), ints([0]), heads, rank, rot_dim, scale, window, n_splits=parts, max_q_len=1, sink=sd)
            close(out, want[last - 1:last], dtype, f"tensor cores, token {last - 1} in {parts} parts", bf16=3e-2)


# ------------------------------------------------------------------------------ the model

def all_places(n):
    return list(range(n))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_each_request_alone_and_whole(tmp_path_factory, name, dtype):
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    for length, seed in ((1, 1), (2, 2), (9, 3), (64, 4), (65, 5), (200, 6)):
        prompt = random_prompt(length, cfg["vocab"], seed)
        slot = runner.open_sequence()
        got = runner.step([StepEntry(slot, prompt, all_places(length))])
        runner.close_sequence(slot)
        want = wanted(name, cfg, w, prompt)
        assert_close(got, want, dtype, f"{name} whole, length {length}")
        assert_close(got[:3], want[:3], dtype, f"{name}: the first tokens of a sequence")
    runner.check_status()
    runner.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_every_layer_against_the_plain_layers(tmp_path_factory, name, dtype):
    """The stream after each run of a layer, which names the first one that differs."""
    from starter_b200 import ops
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    model = runner.model
    prompt = random_prompt(90, cfg["vocab"], 8)
    slot = runner.open_sequence()
    ctx = runner.make_context([StepEntry(slot, prompt, [])])
    x, pending, got = ops.embedding32(ctx.tokens, model.embed, 1.0, ctx.status), None, []
    for entry in model.spec.schedule:
        if entry.junction is not None:
            x, pending = model.junctions[entry.junction](x, pending, ctx, model.embed, 1.0), None
        x, pending = model.blocks[entry.layer](x, pending, ctx, entry.cache, entry.writes_cache)
        after = x.double() + pending.value.double()
        got.append(after if pending.second is None else after + pending.second.double())
    runner.close_sequence(slot)
    want = []
    plain.forward(cfg, w, prompt, layers_out=want)
    assert len(want) == len(plain.run_order(cfg)) == len(got)
    for i in range(len(want)):
        close(got[i], want[i], dtype, f"{name} after run {i}", fp32=2e-5, bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_then_tokens_one_by_one(tmp_path_factory, name, dtype):
    """Windows of 3, 10, 17, 64 and 65 pass over decoded tokens, and a page border is crossed while decoding."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    for length, tail in ((40, 39), (100, 45), (150, 90)):
        prompt = random_prompt(length, cfg["vocab"], 20 + length)
        slot = runner.open_sequence()
        head = length - tail
        rows = [runner.step([StepEntry(slot, prompt[:head], all_places(head))])]
        for tok in prompt[head:]:
            rows.append(runner.step([StepEntry(slot, [tok], [0])]))
        runner.close_sequence(slot)
        got, want = torch.cat(rows), wanted(name, cfg, w, prompt)
        assert_close(got, want, dtype, f"{name} last {tail} one by one, length {length}")
        assert_close(got[head:head + 1], want[head:head + 1], dtype, "the first single-token step")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["LA", "LC"])
def test_long_decoding_over_many_pages(tmp_path_factory, name, dtype):
    """Two requests of unequal lengths decoded together for 300 steps, the longer one over six pages; the shorter one
    ends on the way; every logit is held to the plain statement."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    lengths, heads = (380, 150), (80, 3)
    prompts = [random_prompt(n, cfg["vocab"], 300 + n) for n in lengths]
    slots = [runner.open_sequence() for _ in prompts]
    first = runner.step([StepEntry(s, p[:h], all_places(h)) for s, p, h in zip(slots, prompts, heads)])
    got = [[first[:heads[0]]], [first[heads[0]:]]]
    at = list(heads)
    while at[0] < lengths[0]:
        live = [i for i in range(2) if at[i] < lengths[i]]
        rows = runner.step([StepEntry(slots[i], [prompts[i][at[i]]], [0]) for i in live])
        for k, i in enumerate(live):
            got[i].append(rows[k:k + 1])
            at[i] += 1
            if at[i] == lengths[i]:
                runner.close_sequence(slots[i])
    for i in range(2):
        assert_close(torch.cat(got[i]), wanted(name, cfg, w, prompts[i]), dtype, f"{name} request {i} decoded to {lengths[i]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_portions_of_several_sizes(tmp_path_factory, name, dtype):
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    prompt = random_prompt(171, cfg["vocab"], 77)
    for sizes in ((2, 2, 3, 57, 64, 1, 40, 2), (63, 2, 63, 43), (5, 128, 38), (30, 141)):
        slot = runner.open_sequence()
        rows, at = [], 0
        for n in sizes:
            rows.append(runner.step([StepEntry(slot, prompt[at:at + n], all_places(n))]))
            at += n
        assert at == len(prompt)
        runner.close_sequence(slot)
        assert_close(torch.cat(rows), wanted(name, cfg, w, prompt), dtype, f"{name} portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_unequal_batches_with_slots_pages_and_states_used_again(tmp_path_factory, name, dtype):
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    batches = [[(70, 9), (5, 3), (33, 12), (1, 6)], [(2, 40), (129, 2), (64, 5)], [(17, 0), (63, 3)]]
    seed = 300
    for batch in batches:
        seqs, slots, got = [], [], []
        for plen, extra in batch:
            seed += 1
            seqs.append(random_prompt(plen + extra, cfg["vocab"], seed))
            slots.append(runner.open_sequence())
            got.append([])
        first = runner.step([StepEntry(slots[i], seqs[i][:plen], all_places(plen)) for i, (plen, _) in enumerate(batch)])
        offset = 0
        for i, (plen, _) in enumerate(batch):
            got[i].append(first[offset:offset + plen])
            offset += plen
        live = [i for i, (_, extra) in enumerate(batch) if extra > 0]
        for i, (_, extra) in enumerate(batch):
            if extra == 0:
                runner.close_sequence(slots[i])
        step = 0
        while live:
            out = runner.step([StepEntry(slots[i], [seqs[i][batch[i][0] + step]], [0]) for i in live])
            for row, i in enumerate(live):
                got[i].append(out[row:row + 1])
            step += 1
            for i in [i for i in live if batch[i][1] == step]:
                runner.close_sequence(slots[i])
            live = [i for i in live if batch[i][1] > step]
        for i, seq in enumerate(seqs):
            assert_close(torch.cat(got[i]), wanted(name, cfg, w, seq), dtype, f"{name} batch {batch}, request {i}")
        runner.cache.check()
    assert runner.cache.slots.held_count == 0 and runner.cache.pages.held_count == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["LA", "LC"])
def test_portions_prompts_and_single_tokens_in_one_step(tmp_path_factory, name, dtype):
    """One step that begins a sequence, brings a later portion of another and a single token of a third."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    prompts = [random_prompt(n, cfg["vocab"], 500 + n) for n in (66, 140, 90)]
    slots = [runner.open_sequence() for _ in prompts]
    got = [[], [], []]
    done = [0, 0, 0]
    for sizes in ((0, 70, 64), (40, 2, 1), (25, 67, 1), (1, 1, 24)):
        live = [i for i in range(3) if sizes[i]]
        out = runner.step([StepEntry(slots[i], prompts[i][done[i]:done[i] + sizes[i]], all_places(sizes[i])) for i in live])
        at = 0
        for i in live:
            got[i].append(out[at:at + sizes[i]])
            at += sizes[i]
            done[i] += sizes[i]
    for i in range(3):
        runner.close_sequence(slots[i])
        assert done[i] == len(prompts[i])
        assert_close(torch.cat(got[i]), wanted(name, cfg, w, prompts[i]), dtype, f"{name} mixed steps, request {i}")


@pytest.mark.parametrize("what", ["a far key through the latent", "a far key through the recurrence", "the window's edge"])
def test_a_key_far_away_decides(tmp_path_factory, what):
    """A single token changed far back, or at a window's edge, moves the logits as it moves the plain statement's, in a
    prompt and while decoding: through the latent attention, through the recurrence's state, and not at all once it has
    left the only window."""
    from safetensors.torch import load_file, save_file
    from starter_b200.engine import ModelRunner, StepEntry, load_model

    raw = copy.deepcopy(TINY_L["LA"])
    layer = {"a far key through the latent": 2, "a far key through the recurrence": 0, "the window's edge": 1}[what]
    raw["layers"] = [raw["layers"][layer]]
    raw["loop"] = dict(start=0, stop=1, times=1)
    window = 60
    if layer == 1:
        raw["layers"][0]["mixer"]["mask"]["size"] = window
        raw["layers"][0]["mixer"].pop("conv")               # (else the taps reach over the edge)
    folder = make_salulorn_folder(tmp_path_factory.mktemp("far"), "FAR", seed=3, raw=raw)
    file = folder + "/model.safetensors"
    tensors = load_file(file)
    if layer == 0:
        tensors["l0.mix.a2.b"] = torch.full_like(tensors["l0.mix.a2.b"], 7.0)
    elif layer == 2:
        tensors["l0.mix.uq"] = tensors["l0.mix.uq"] * 3.0
        tensors["l0.mix.sink"] = tensors["l0.mix.sink"] - 3.0
    else:
        tensors["l0.mix.sink"] = tensors["l0.mix.sink"] - 3.0
    save_file(tensors, file, metadata={"format": "pt"})
    cfg, w = plain.read_model_folder(folder)
    a = random_prompt(330, cfg["vocab"], 4)
    changed = 2 if layer != 1 else 265
    b = list(a)
    b[changed] = (b[changed] + 1) % cfg["vocab"]
    want_a, want_b = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    moved = (want_a - want_b).abs().max(dim=1).values / float(want_a.abs().max())
    if layer == 1:
        assert float(moved[changed + window - 1]) > 20 * FP32_TOL and float(moved[changed + window]) == 0.0
    else:
        assert float(moved[311:].max()) > 10 * FP32_TOL
    runner = ModelRunner(load_model(folder, "float32"), max_tokens=64 * 8, max_sequences=4, use_graphs=False)
    for prompt, want in ((a, want_a), (b, want_b)):
        for head in (310, 330):
            slot = runner.open_sequence()
            got = [runner.step([StepEntry(slot, prompt[:head], all_places(head))])]
            got += [runner.step([StepEntry(slot, [tok], [0])]) for tok in prompt[head:]]
            runner.close_sequence(slot)
            assert_close(torch.cat(got), want, "float32", what)


@pytest.mark.parametrize("seed", range(14))
def test_configurations_drawn_at_random(tmp_path_factory, seed):
    """Layer kinds, their order, the loop, every size, head count, window, tap count and constant drawn anew: three
    unequal requests whole and alone, then begun together and decoded together, then one in portions, in float32 and,
    whole and decoded, in bfloat16.  The bounds are wider than elsewhere: some drawn models are ill-conditioned."""
    import random

    from starter_b200.engine import ModelRunner, StepEntry, load_model
    from tiny_salulorn import random_config

    rng = random.Random(3000 + seed)
    raw = random_config(rng)
    folder = make_salulorn_folder(tmp_path_factory.mktemp(f"r{seed}"), f"R{seed}", seed=seed, dtype=torch.bfloat16, raw=raw)
    cfg, w = plain.read_model_folder(folder)
    lengths = [rng.choice([1, 3, 40, 130]), rng.choice([2, 70, 150]), rng.choice([5, 64, 65, 200])]
    prompts = [random_prompt(n, cfg["vocab"], seed * 10 + i) for i, n in enumerate(lengths)]
    want = [plain.forward(cfg, w, p) for p in prompts]

    def held(got, wanted, dtype, what):
        if dtype == "float32":
            close(got, wanted, dtype, what, fp32=3e-4)
        else:
            mean = float((got.double().cpu() - wanted).abs().mean()) / float(wanted.abs().max())
            assert mean <= 2e-2, f"bfloat16, {what}: mean error {mean:.3e} of the largest logit"

    for dtype in DTYPES:
        runner = ModelRunner(load_model(folder, dtype), max_tokens=64 * 40, max_sequences=8, use_graphs=False)
        for p, wanted_rows in zip(prompts, want):
            slot = runner.open_sequence()
            got = runner.step([StepEntry(slot, p, all_places(len(p)))])
            runner.close_sequence(slot)
            held(got, wanted_rows, dtype, f"whole, length {len(p)}")
        tails = [min(len(p) - 1, 20) for p in prompts]
        heads = [len(p) - t for p, t in zip(prompts, tails)]
        slots = [runner.open_sequence() for _ in prompts]
        first = runner.step([StepEntry(s, p[:h], all_places(h)) for s, p, h in zip(slots, prompts, heads)])
        got, at = [[] for _ in prompts], 0
        for i, h in enumerate(heads):
            got[i].append(first[at:at + h])
            at += h
        for step in range(max(tails)):
            live = [i for i in range(3) if step < tails[i]]
            out = runner.step([StepEntry(slots[i], [prompts[i][heads[i] + step]], [0]) for i in live])
            for row, i in enumerate(live):
                got[i].append(out[row:row + 1])
        for i in range(3):
            runner.close_sequence(slots[i])
            held(torch.cat(got[i]), want[i], dtype, f"begun and decoded together, request {i}")
        slot, rows, at = runner.open_sequence(), [], 0
        for n in (2, 1, 3, 61, 70, 200):
            part = prompts[2][at:at + n]
            if part:
                rows.append(runner.step([StepEntry(slot, part, all_places(len(part)))]))
                at += len(part)
        runner.close_sequence(slot)
        held(torch.cat(rows), want[2], dtype, "in portions")
        runner.check_status()
        runner.cache.check()
        assert runner.cache.slots.held_count == 0 and runner.cache.pages.held_count == 0


@pytest.mark.parametrize("name", CONFIGS)
def test_greedy_generation_through_the_entry_point(tmp_path_factory, name):
    """Unequal prompts through ``Engine.generate`` (the scheduler, the captured single-token step with its saved and
    restored state, the sampler): 70 tokens each, past a page border and past every window, equal to the plain
    statement's greedy continuation."""
    from starter_b200 import Engine

    folder, cfg, w = case(tmp_path_factory, name)
    engine = Engine(folder, dtype="float32", max_batch=4)
    prompts = [random_prompt(n, cfg["vocab"], 900 + n) for n in (50, 3, 21)]
    steps = list(engine.generate(prompts, 70))
    assert len(steps) == 70
    for i, prompt in enumerate(prompts):
        seq = list(prompt) + [s[i] for s in steps]
        logits = plain.forward(cfg, w, seq[:-1])            # one pass over the whole: each token is the largest logit
        assert [int(torch.argmax(row)) for row in logits[len(prompt) - 1:]] == [s[i] for s in steps], f"request {i}"


def test_random_weights_from_the_library_run_in_bfloat16():
    """``random_model`` places every tensor as the loader would, and sampling with temperature runs."""
    from starter_b200 import Engine
    from starter_b200.config import config_from_dict
    from starter_b200.engine.runner import random_model

    model = random_model(config_from_dict(TINY_L["LC"]), seed=5, dtype="bfloat16")
    engine = Engine.from_model(model, max_batch=2)
    out = engine.complete([[1, 2, 3], [4]], 12, temperature=0.8, seed=3)
    assert [len(c.tokens) for c in out] == [12, 12]
    assert all(0 <= t < 257 for c in out for t in c.tokens)


# ------------------------------------------------------------------------------ the programs

def test_command_line_and_trace_replay(tmp_path_factory, tmp_path):
    """``python -m starter_b200 generate`` and ``bin/trace_run`` pick the design by its config.json."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    folder, cfg, w = case(tmp_path_factory, "LB")
    prompts = [random_prompt(5, cfg["vocab"], 1), random_prompt(19, cfg["vocab"], 2)]
    text = ";".join(",".join(str(t) for t in p) for p in prompts)
    out = subprocess.run([sys.executable, "-m", "starter_b200", "generate", "--model-path", folder, "--input-ids", text,
                          "--max-new-tokens", "6", "--dtype", "float32"], cwd=root, capture_output=True, text=True,
                         timeout=600)
    assert out.returncode == 0, out.stderr
    lines = [json.loads(line) for line in out.stdout.splitlines() if line.startswith("{")]
    assert [line["tokens"] for line in lines] == [plain.generate(cfg, w, p, 6) for p in prompts]

    # a trace: two unequal requests start together, are decoded together, the shorter one ends first
    a, b = random_prompt(140, cfg["vocab"], 5), random_prompt(70, cfg["vocab"], 6)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:130], "want": [0, 129]},
                                     {"id": "b", "tokens": b[:66], "want": [65]}], "end": []}]
    for i in range(10):
        entries = [{"id": "a", "tokens": [a[130 + i]], "want": [0]}]
        if i < 4:
            entries.append({"id": "b", "tokens": [b[66 + i]], "want": [0] if i % 2 else []})
        steps.append({"step": 1 + i, "entries": entries, "end": (["b"] if i == 3 else []) + (["a"] if i == 9 else [])})
    out_dir = str(tmp_path / "float32")
    proc = subprocess.Popen([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                             "--out", out_dir, "--max-tokens", "210"], stdin=subprocess.PIPE, stdout=subprocess.PIPE,
                            text=True)
    for record in steps:
        proc.stdin.write(json.dumps(record) + "\n")
        proc.stdin.flush()
        assert proc.stdout.readline().strip() == f"done {record['step']}"
    proc.stdin.close()
    assert proc.wait(timeout=120) == 0
    want_a, want_b = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    read = lambda s: torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{s}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]))  # noqa: E731
    assert_close(read(0), torch.stack([want_a[0], want_a[129], want_b[65]]), "float32", "the first step")
    for i in range(10):
        rows = [want_a[130 + i]] + ([want_b[66 + i]] if i < 4 and i % 2 else [])
        assert_close(read(1 + i), torch.stack(rows), "float32", f"step {1 + i}")
