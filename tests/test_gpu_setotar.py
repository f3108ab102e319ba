"""Setotar on the GPU against the plain statement: each mechanism alone, then the model through the step function, the
cache, the state slots and the generation loop, cut into steps and batches in every way."""

import pytest
import torch

import plain_setotar as plain
from gpu_helpers import DTYPES, FP32_TOL
from tiny import random_prompt
from tiny_setotar import TINY_S, make_setotar_folder, rot

pytestmark = pytest.mark.gpu

CONFIGS = ["SA", "SB", "SC"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64
_cases, _runners = {}, {}


def case(tmp_path_factory, name, seed=1):
    if (name, seed) not in _cases:
        folder = make_setotar_folder(tmp_path_factory.mktemp(f"s{name}{seed}"), name, seed=seed)
        _cases[(name, seed)] = (folder,) + plain.read_model_folder(folder)
    return _cases[(name, seed)]


def runner_for(tmp_path_factory, name, dtype, max_tokens=64 * 40):
    from starter_b200.engine import ModelRunner, load_model

    if (name, dtype) not in _runners:
        folder, _, _ = case(tmp_path_factory, name)
        _runners[(name, dtype)] = ModelRunner(load_model(folder, dtype), max_tokens=max_tokens, max_sequences=12)
    return _runners[(name, dtype)]


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


class Routed:
    """Runs steps and notes, per request, which experts every routed layer chose for each of its tokens.  The 32-bit
    comparisons do not use the notes (there the choice itself is held to the plain statement); the bfloat16
    comparisons hand them to the plain statement, because a near-tie may fall either way once the router's input is
    rounded to 8 bits."""

    def __init__(self, runner):
        self.runner = runner
        blocks = [runner.model.blocks[e.layer] for e in runner.model.spec.schedule]
        self.runs = {i: b.feed_forward for i, b in enumerate(blocks) if b.feed_forward is not None}
        self.notes = {}

    def step(self, entries, keys):
        out = self.runner.step(entries)
        at = 0
        for entry, key in zip(entries, keys):
            n = len(entry.tokens)
            for place, ff in self.runs.items():
                self.notes.setdefault(key, {}).setdefault(place, []).append(ff.last_ids[at:at + n].cpu())
            at += n
        return out

    def routes(self, key, dtype):
        if dtype == "float32" or not self.runs:
            return None
        return {place: torch.cat(parts) for place, parts in self.notes[key].items()}


# ------------------------------------------------------------------------------ mechanisms alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [40, 37, 600, 5000])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8])
def test_stream_step_with_a_layer_scale_and_an_rms_norm(streams, hidden, dtype):
    """The pending output scaled per channel and written, the next read and its RMS norm in one kernel; the matrix is
    [from, to], every stream comes from the OLD ones, and selected rows leave the streams as they were."""
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(10 + streams)
    rnd = lambda *shape: torch.randn(*shape, generator=g, dtype=F)  # noqa: E731
    x, y = rnd(7, streams, hidden), rnd(7, hidden)
    mix, out, read, scale, gain = rnd(streams, streams), rnd(streams), rnd(streams), rnd(hidden), rnd(hidden)
    xd, yd = dev(x), dev(y, t)
    w = {"in": read.float().double(), "out": out.float().double(), "mix": mix.float().double()}
    seen, written = xd.double().cpu().transpose(0, 1), yd.double().cpu() * scale.float().double()
    new = plain.through_streams(seen, w, "", lambda u: written)
    pending = (yd, dev(mix), dev(out), None, dev(scale))
    norm = (dev(gain), 1e-5)
    rows = ints([6, 2])
    got = ops.hyper_step(xd, t, pending, None, norm, rows=rows)
    close(got, plain.norm(new.sum(dim=0)[[6, 2]], gain, 1e-5), dtype, "closing rows", bf16=8e-3)
    assert torch.equal(xd, dev(x))
    got = ops.hyper_step(xd, t, pending, dev(read), norm)
    close(got, plain.norm((w["in"][:, None, None] * new).sum(dim=0), gain, 1e-5), dtype, "write, read, norm", bf16=8e-3)
    close(xd, new.transpose(0, 1), "float32", "the streams after the write", fp32=1e-5)
    got = ops.hyper_step(xd, t, None, dev(read), norm)
    close(got, plain.norm((w["in"][:, None, None] * xd.double().cpu().transpose(0, 1)).sum(dim=0), gain, 1e-5), dtype,
          "read and norm alone", bf16=8e-3)
    # the scale without a norm, and behind a bias
    bias = rnd(hidden)
    again = xd.double().cpu().transpose(0, 1)
    written = (yd.double().cpu() + bias.float().double()) * scale.float().double()
    new = plain.through_streams(again, w, "", lambda u: written)
    got = ops.hyper_step(xd, t, (yd, dev(mix), dev(out), dev(bias), dev(scale)), None, None)
    close(got, new.sum(dim=0), dtype, "bias, scale, plain sum", bf16=8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, turn, row_norm, unit", [
    (4, 2, 16, 24, rot(100.0, 8), False, True), (6, 3, 64, 32, rot(2e3, 24, 3.0, 300, 20.0, 2.0), True, False),
    (1, 1, 24, 40, None, True, False), (3, 3, 10, 12, rot(1e3, 6, 2.0), True, True), (8, 1, 128, 80, rot(1e4, 128), True, True),
    (16, 2, 128, 128, rot(1e4, 64, 2.0), False, True)])
def test_prepare_alone(heads, kv_heads, dim, vdim, turn, row_norm, unit, dtype):
    """Norm over the whole row, half-split turn, values over their root mean square: queries in place, keys and values
    in the cache on both sides of page borders; a reading layer's queries alone."""
    from starter_b200 import ops
    from starter_b200.config.setotar import _position
    from starter_b200.parts.rotary import PartialRotaryTable

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
    v = plain.rms(v, eps) if unit else v
    rotation = None
    if turn is not None:
        table_part = PartialRotaryTable(_position(turn), t, "cuda")
        table_part.ensure(300)
        rotation = table_part.rotation()
    table = torch.zeros(3, 8, dtype=torch.int32, device="cuda")
    table[1, :5] = ints([5, 2, 7, 0, 3])
    ks = torch.zeros(8, kv_heads, 64, dim, dtype=t, device="cuda")
    vs = torch.zeros(8, kv_heads, 64, vdim, dtype=t, device="cuda")
    pos, slot = dev(place, torch.int32), ints([1] * n)
    norms = (dev(gains[0]), dev(gains[1])) if row_norm else None
    alone = proj[:, :widths[0]].contiguous()
    ops.sink_prepare_norm(proj, heads, kv_heads, dim, vdim, pos, slot, table, ks, vs, rotation, norms, unit, eps)
    close(proj[:, :widths[0]], q.reshape(n, -1), dtype, "queries", fp32=1e-6, bf16=8e-3)
    pages = torch.tensor([5, 2, 7, 0, 3])[place // 64]
    close(ks[pages.cuda(), :, (place % 64).cuda()], k, dtype, "keys", fp32=1e-6, bf16=8e-3)
    close(vs[pages.cuda(), :, (place % 64).cuda()], v, dtype, "values", fp32=1e-6, bf16=8e-3)
    assert float(ks[5, :, :37].abs().max()) == 0.0 and float(vs[3].abs().max()) == 0.0, "nothing else was written"
    kept = ks.clone()
    ops.sink_prepare_norm(alone, heads, kv_heads, dim, vdim, pos, slot, table, ks, vs, rotation,
                          (norms[0], None) if row_norm else None, False, eps, write_cache=False)
    assert torch.equal(ks, kept)
    close(alone, q.reshape(n, -1), dtype, "a reading layer's queries", fp32=1e-6, bf16=8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, keep, cap", [
    (4, 2, 16, 24, 10, 3, 20.0), (1, 1, 24, 40, 3, 1, None), (8, 2, 64, 80, 65, 70, 30.0), (4, 4, 128, 48, 64, 1, 50.0),
    (5, 1, 128, 72, 99, 6, 25.0), (2, 2, 10, 12, 17, 0, 20.0), (3, 1, 64, 128, 130, 64, None), (2, 1, 96, 72, None, 0, 25.0),
    (6, 2, 64, 64, None, 0, None), (2, 2, 128, 128, 1, 65, 40.0), (1, 1, 200, 136, 70, 5, 30.0), (8, 8, 32, 16, 40, 128, None)])
def test_window_attention_with_kept_keys_and_a_cap_alone(heads, kv_heads, dim, vdim, window, keep, cap, dtype):
    """A sequence of 300 over five scattered pages.  Queries late in the sequence aim at one key, so that its score stands
    out: the oldest inside their window, the one just outside it, the last kept key and the first that is not kept, keys
    on either side of a page border, their own place.  Plain, ``mma.sync`` and tcgen05 kernels, whole, as a later portion
    and as the last token alone in 1, 3 and 7 parts."""
    from starter_b200 import ops

    t, n, scale = TORCH[dtype], 300, 0.25
    g = torch.Generator().manual_seed(heads * 100 + dim + vdim)
    group = heads // kv_heads
    q = torch.randn(n, heads, dim, generator=g, dtype=F)
    k = torch.randn(n, kv_heads, dim, generator=g, dtype=F)
    v = torch.randn(n, kv_heads, vdim, generator=g, dtype=F)
    span = window or n
    probes = {280: 280, 299: 0, 250: 191, 251: 192, 130: 63, 131: 64}
    for at in (298, 257, 200, 193, 128):
        probes[at] = max(at - span + 1, 0)               # the oldest key inside the window
        probes[at - 1] = max(at - 1 - span, 0)           # the key just outside it
    for at in (295, 290, 221, 150):
        probes[at] = max(keep - 1, 0)                    # the last kept key
        probes[at - 1] = keep                            # the first that is not kept
    for at, key in probes.items():
        for h in range(heads):
            target = k[key, h // group]
            q[at, h] = target / target.norm() ** 2 * (30.0 / scale)
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
    want = plain.attend(*args, window, keep).reshape(n, heads * vdim)
    if window is not None:
        # an edge that is one off must show
        for wrong in ((window + 1, keep), (window, keep + 1)) + (((window - 1, keep),) if window > 1 else ()):
            other = plain.attend(*args, *wrong).reshape(n, heads * vdim)
            assert float((other - want).abs().max()) > 0.3, wrong
    pos, slot = dev(place, torch.int32), ints([1] * n)
    rest = dict(window=window, keep_first=keep, softcap=cap)
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
    assert ops.sink_tcgen05_takes(proj, dim, vdim) == (dim % 16 == 0)
    if dim % 16:
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


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, n, v", [(3, 12, 8), (1, 40, 33), (2, 128, 64), (4, 64, 32), (2, 1, 1), (1, 256, 20), (5, 5, 100)])
def test_forget_write_recurrence_alone(heads, n, v, dtype):
    """Three sequences whole, then in portions down to one token that cross the kernel's chunks, in state slots with
    floats of others around them; forget gates from next to nothing to next to one, and a first value that must still
    show at the end."""
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(heads * 1000 + n)
    lengths, slots = [300, 1, 17], [2, 0, 3]
    total = sum(lengths)
    z, raw = torch.randn(total, heads * n, generator=g, dtype=F), torch.randn(total, heads * n, generator=g, dtype=F)
    val = torch.randn(total, heads * v, generator=g, dtype=F)
    val[0] = 40.0
    bias = torch.linspace(6.0, -3.0, heads * n, dtype=F)
    lower = torch.linspace(0.0, 0.95, heads * n, dtype=F)
    lower[0] = 0.0
    proj = dev(torch.cat([torch.zeros(total, 3, dtype=F), raw, z, val], dim=1), t)
    seen = proj.double().cpu()[:, 3:].split([heads * n, heads * n, heads * v], dim=1)
    low, b = lower.float().double(), bias.float().double()
    q = plain.silu(seen[0]).reshape(total, heads, n)
    f = (low + (1.0 - low) * torch.sigmoid(seen[1] + b)).reshape(total, heads, n)
    vv = seen[2].reshape(total, heads, v)
    want, at = [], 0
    for length in lengths:
        want.append(plain.forget_recurrence(q[at:at + length], f[at:at + length], vv[at:at + length]))
        at += length
    forgot = vv[:300].clone()
    forgot[0] = 0.0
    forgot = plain.forget_recurrence(q[:300], f[:300], forgot)
    assert float((forgot[280:] - want[0][280:]).abs().max()) > 0.02
    want = torch.cat(want).reshape(total, heads * v)
    state_at = 5
    state = torch.zeros(4, state_at + heads * n * v + 2, device="cuda")
    state[:, :state_at] = 7.0
    state[:, -2:] = 8.0

    def run(p, lens, sl):
        return ops.state_scan("forget_write", (p, 3), (p, 3 + heads * n), (p, 3 + 2 * heads * n), None, None, dev(lower), dev(bias),
                              None, state, state_at, *packed(lens, sl), heads, heads, n, v)

    close(run(proj, lengths, slots), want, dtype, "whole", fp32=2e-5, bf16=2e-5)        # (the inputs are the same bits)
    assert float((state[:, :state_at] - 7.0).abs().max()) == 0.0 and float((state[:, -2:] - 8.0).abs().max()) == 0.0
    assert float(state[1, state_at:-2].abs().max()) == 0.0
    state[:, state_at:-2] = 0.0
    got, done, bases = [[], [], []], [0, 0, 0], [0, 300, 301]
    for sizes in ([1, 1, 1], [2, 0, 1], [16, 0, 15], [33, 0, 0], [248, 0, 0]):
        live = [i for i in range(3) if sizes[i]]
        rows = torch.cat([torch.arange(bases[i] + done[i], bases[i] + done[i] + sizes[i]) for i in live]).cuda()
        out = run(proj[rows].contiguous(), [sizes[i] for i in live], [slots[i] for i in live])
        at = 0
        for i in live:
            got[i].append(out[at:at + sizes[i]])
            at += sizes[i]
            done[i] += sizes[i]
    close(torch.cat([torch.cat(p) for p in got]), want, dtype, "in portions", fp32=2e-5, bf16=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_in_parts_without_a_gate_and_a_scaled_sum(dtype):
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(3)
    for parts, psize, shared in ((1, 40, False), (3, 8, True), (4, 64, True), (5, 7, True), (2, 600, False)):
        o = dev(torch.randn(6, parts * psize, generator=g, dtype=F) * 3.0)
        w = torch.randn(psize if shared else parts * psize, generator=g, dtype=F)
        want = plain.rms(o.double().cpu().reshape(6, parts, psize), 1e-5).reshape(6, -1) * (w.repeat(parts) if shared else w)
        close(ops.group_norm_gate(o, None, 0, dev(w), parts, 1e-5, False, t), want, dtype, f"{parts} x {psize}", fp32=1e-6, bf16=8e-3)
    for width in (37, 64, 1000, 5000):
        a, b = (dev(torch.randn(5, width, generator=g, dtype=F), t) for _ in range(2))
        close(ops.scaled_sum(a, b, 0.7, -1.5), 0.7 * a.double().cpu() - 1.5 * b.double().cpu(), dtype, f"width {width}", fp32=1e-6, bf16=8e-3)


@pytest.mark.parametrize("taps", [1, 2, 3, 4])
@pytest.mark.parametrize("dtype", DTYPES)
def test_biased_convolution_has_zeros_in_front_of_the_sequence(taps, dtype):
    """The bias belongs to the projection: a sequence's first tokens see zeros, not biases, in front of them."""
    from starter_b200 import ops

    t, channels = TORCH[dtype], 48
    g = torch.Generator().manual_seed(taps)
    x = dev(torch.randn(90, channels, generator=g, dtype=F), t)
    w, bias = torch.randn(channels, taps, generator=g, dtype=F), torch.randn(channels, generator=g, dtype=F) * 5.0
    want = torch.cat([plain.causal_conv(part + bias.float().double(), w.float().double()) for part in x.double().cpu().split([70, 20])])
    state = torch.zeros(3, (taps - 1) * channels, device="cuda") if taps > 1 else None
    out = ops.short_conv(x, 0, channels, dev(w), None, dev(bias), state, 0, *packed([70, 20], [2, 0]), 70)
    close(out, want, dtype, "whole", fp32=1e-6, bf16=8e-3)
    if taps > 1:
        state.zero_()
    rows, at = [], 0
    for n in (1, 2, 1, 35, 31):
        rows.append(ops.short_conv(x[at:at + n].contiguous(), 0, channels, dev(w), None, dev(bias), state, 0, *packed([n], [1]), n))
        at += n
    close(torch.cat(rows), want[:70], dtype, "in portions", fp32=1e-6, bf16=8e-3)


@pytest.mark.parametrize("experts, top", [(5, 2), (3, 3), (16, 1), (64, 8), (1, 1)])
def test_router_of_plain_sigmoids_alone(experts, top):
    from starter_b200 import ops

    g = torch.Generator().manual_seed(experts * 10 + top)
    h = torch.randn(40, 48, generator=g, dtype=F)
    h[5] = 0.0                                                   # every score equal: the first experts win
    router = torch.randn(experts, 48, generator=g, dtype=F) * 0.3
    if experts > 1:
        router[1] = router[0]                                    # two that always tie
    hh = dev(h)
    index, s = plain.route(hh.double().cpu(), {"r.router": router.float().double()}, "r.", dict(top=top))
    ids, weights = ops.moe_route(hh, dev(router), None, top, "sigmoid")
    assert torch.equal(ids.cpu().long(), index)
    close(weights, s.gather(1, index), "float32", "weights", fp32=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 5, 70, 700])
@pytest.mark.parametrize("experts, top, width, inner", [(5, 2, 64, 24), (3, 3, 96, 32), (8, 1, 128, 64), (4, 2, 40, 20), (1, 1, 64, 64)])
def test_experts_that_take_the_weighted_input_alone(experts, top, width, inner, rows, dtype):
    """Given choices on whichever tile kernel the step's shape picks, then on every kind; weights from next to nothing to
    one, so that a weight behind the expert instead of in front of it shows."""
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(rows + experts)
    h = dev(torch.randn(rows, width, generator=g, dtype=F), t)
    gate_up = dev(torch.randn(experts, 2 * inner, width, generator=g, dtype=F) * 0.3, t)
    down = dev(torch.randn(experts, width, inner, generator=g, dtype=F) * 0.3, t)
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(rows)]).int()
    weights = torch.rand(rows, top, generator=g, dtype=F).float()
    h64 = h.double().cpu()
    want, behind = torch.zeros(rows, width, dtype=F), torch.zeros(rows, width, dtype=F)
    for e in range(experts):
        w = {"e.gate": gate_up[e, :inner].double().cpu(), "e.up": gate_up[e, inner:].double().cpu(), "e.down": down[e].double().cpu()}
        share = (weights * (ids == e)).sum(dim=1).double()
        used = (ids == e).any(dim=1)
        want[used] += plain.expert(share[used, None] * h64[used], w, "e.")
        behind[used] += share[used, None] * plain.expert(h64[used], w, "e.")
    assert float((want - behind).abs().max()) > 0.1 * float(want.abs().max())
    out = ops.moe_experts(h, ids.cuda(), weights.cuda(), gate_up, down, expert="gated_silu", weigh_input=True)
    close(out, want, dtype, "the step's own tiles", bf16=2.5e-2)
    if dtype == "bfloat16" and width % 16 == 0 and inner % 16 == 0:
        for tile_rows in (4, 32, 64, 128, 256):
            out = ops.moe_experts(h, ids.cuda(), weights.cuda(), gate_up, down, expert="gated_silu", tile_rows=tile_rows, weigh_input=True)
            close(out, want, dtype, f"tiles of {tile_rows} rows", bf16=2.5e-2)


# ------------------------------------------------------------------------------ the model

def all_places(n):
    return list(range(n))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_each_request_alone_and_whole(tmp_path_factory, name, dtype):
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    routed = Routed(runner_for(tmp_path_factory, name, dtype))
    runner = routed.runner
    for length, seed in ((1, 1), (2, 2), (9, 3), (64, 4), (65, 5), (200, 6)):
        prompt = random_prompt(length, cfg["vocab"], seed)
        slot = runner.open_sequence()
        got = routed.step([StepEntry(slot, prompt, all_places(length))], [length])
        runner.close_sequence(slot)
        want = plain.forward(cfg, w, prompt, routes=routed.routes(length, dtype))
        assert_close(got, want, dtype, f"{name} whole, length {length}")
        assert_close(got[:3], want[:3], dtype, f"{name}: the first tokens of a sequence")
    runner.check_status()
    runner.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_every_layer_against_the_plain_layers(tmp_path_factory, name, dtype):
    """The sum of the streams after each layer, which names the first one that differs."""
    from starter_b200 import ops
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    model = runner.model
    prompt = random_prompt(90, cfg["vocab"], 8)
    slot = runner.open_sequence()
    ctx = runner.make_context([StepEntry(slot, prompt, [])])
    streams = ops.embedding_streams(ctx.tokens, model.embed, model.spec.streams, ctx.status)
    rows = torch.arange(90, dtype=torch.int32, device="cuda")
    pending, got, routes = None, [], {}
    for i, entry in enumerate(model.spec.schedule):
        streams, pending = model.blocks[entry.layer](streams, pending, ctx, entry.cache, entry.writes_cache)
        after = (pending.value.float(),) + pending.for_kernel()[1:]
        got.append(ops.hyper_step(streams, torch.float32, after, None, None, rows=rows))
        if model.blocks[entry.layer].feed_forward is not None:
            routes[i] = model.blocks[entry.layer].feed_forward.last_ids.cpu()
    runner.close_sequence(slot)
    want = []
    plain.forward(cfg, w, prompt, layers_out=want, routes=None if dtype == "float32" else routes)
    assert len(want) == len(cfg["layers"]) == len(got)
    for i in range(len(want)):
        close(got[i], want[i], dtype, f"{name} after layer {i}", fp32=2e-5, bf16=2.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_then_tokens_one_by_one(tmp_path_factory, name, dtype):
    """Windows of 3, 10, 17, 64 and 65 pass over decoded tokens, and a page border is crossed while decoding."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    routed = Routed(runner_for(tmp_path_factory, name, dtype))
    runner = routed.runner
    for length, tail in ((40, 39), (100, 45), (150, 90)):
        prompt = random_prompt(length, cfg["vocab"], 20 + length)
        slot = runner.open_sequence()
        head = length - tail
        rows = [routed.step([StepEntry(slot, prompt[:head], all_places(head))], [length])]
        for tok in prompt[head:]:
            rows.append(routed.step([StepEntry(slot, [tok], [0])], [length]))
        runner.close_sequence(slot)
        got = torch.cat(rows)
        want = plain.forward(cfg, w, prompt, routes=routed.routes(length, dtype))
        assert_close(got, want, dtype, f"{name} last {tail} one by one, length {length}")
        assert_close(got[head:head + 1], want[head:head + 1], dtype, "the first single-token step")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["SA", "SC"])
def test_long_decoding_over_many_pages(tmp_path_factory, name, dtype):
    """Two requests of unequal lengths decoded together for 300 steps, the longer one over six pages; the shorter one
    ends on the way; every logit is held to the plain statement."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    routed = Routed(runner_for(tmp_path_factory, name, dtype))
    runner = routed.runner
    lengths, heads = (380, 150), (80, 3)
    prompts = [random_prompt(n, cfg["vocab"], 300 + n) for n in lengths]
    slots = [runner.open_sequence() for _ in prompts]
    first = routed.step([StepEntry(s, p[:h], all_places(h)) for s, p, h in zip(slots, prompts, heads)], [0, 1])
    got = [[first[:heads[0]]], [first[heads[0]:]]]
    at = list(heads)
    while at[0] < lengths[0]:
        live = [i for i in range(2) if at[i] < lengths[i]]
        rows = routed.step([StepEntry(slots[i], [prompts[i][at[i]]], [0]) for i in live], live)
        for k, i in enumerate(live):
            got[i].append(rows[k:k + 1])
            at[i] += 1
            if at[i] == lengths[i]:
                runner.close_sequence(slots[i])
    for i in range(2):
        want = plain.forward(cfg, w, prompts[i], routes=routed.routes(i, dtype))
        assert_close(torch.cat(got[i]), want, dtype, f"{name} request {i} decoded to {lengths[i]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_portions_of_several_sizes(tmp_path_factory, name, dtype):
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    prompt = random_prompt(171, cfg["vocab"], 77)
    for sizes in ((2, 2, 3, 57, 64, 1, 40, 2), (63, 2, 63, 43), (5, 128, 38), (30, 141)):
        routed = Routed(runner_for(tmp_path_factory, name, dtype))
        runner = routed.runner
        slot = runner.open_sequence()
        rows, at = [], 0
        for n in sizes:
            rows.append(routed.step([StepEntry(slot, prompt[at:at + n], all_places(n))], [0]))
            at += n
        assert at == len(prompt)
        runner.close_sequence(slot)
        want = plain.forward(cfg, w, prompt, routes=routed.routes(0, dtype))
        assert_close(torch.cat(rows), want, dtype, f"{name} portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_unequal_batches_with_slots_pages_and_states_used_again(tmp_path_factory, name, dtype):
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    batches = [[(70, 9), (5, 3), (33, 12), (1, 6)], [(2, 40), (129, 2), (64, 5)], [(17, 0), (63, 3)]]
    seed = 300
    for batch in batches:
        routed = Routed(runner)
        seqs, slots, got = [], [], []
        for plen, extra in batch:
            seed += 1
            seqs.append(random_prompt(plen + extra, cfg["vocab"], seed))
            slots.append(runner.open_sequence())
            got.append([])
        first = routed.step([StepEntry(slots[i], seqs[i][:plen], all_places(plen)) for i, (plen, _) in enumerate(batch)],
                            list(range(len(batch))))
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
            out = routed.step([StepEntry(slots[i], [seqs[i][batch[i][0] + step]], [0]) for i in live], live)
            for row, i in enumerate(live):
                got[i].append(out[row:row + 1])
            step += 1
            for i in [i for i in live if batch[i][1] == step]:
                runner.close_sequence(slots[i])
            live = [i for i in live if batch[i][1] > step]
        for i, seq in enumerate(seqs):
            want = plain.forward(cfg, w, seq, routes=routed.routes(i, dtype))
            assert_close(torch.cat(got[i]), want, dtype, f"{name} batch {batch}, request {i}")
        runner.cache.check()
    assert runner.cache.slots.held_count == 0 and runner.cache.pages.held_count == 0


def test_a_far_key_decides_through_a_reading_layer(tmp_path_factory):
    """A key hundreds of tokens back, made to stand out in the layer that owns it, moves the logits of a layer that only
    reads it, in a prompt and while decoding; and it is the cached key that is read, not a key of the reading layer."""
    import copy

    from safetensors.torch import load_file, save_file
    from starter_b200.engine import ModelRunner, StepEntry, load_model

    raw = copy.deepcopy(TINY_S["SA"])
    raw["layers"] = [dict(raw["layers"][1]), dict(raw["layers"][2])]
    raw["layers"][1]["mixer"] = dict(raw["layers"][1]["mixer"], kv_from=0, scale=3.0)
    folder = make_setotar_folder(tmp_path_factory.mktemp("far"), "FAR", seed=3, raw=raw)
    file = folder + "/model.safetensors"
    tensors = load_file(file)
    tensors["l0.mix.o"] = tensors["l0.mix.o"] * 0.0               # the owner itself shows nothing of what it attends to
    save_file(tensors, file, metadata={"format": "pt"})
    cfg, w = plain.read_model_folder(folder)
    a = random_prompt(330, cfg["vocab"], 4)
    b = list(a)
    b[2] = (b[2] + 1) % cfg["vocab"]
    want_a, want_b = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    assert float((want_a[311:] - want_b[311:]).abs().max()) > 20 * FP32_TOL * float(want_a.abs().max())
    runner = ModelRunner(load_model(folder, "float32"), max_tokens=64 * 8, max_sequences=4, use_graphs=False)
    for prompt, want in ((a, want_a), (b, want_b)):
        slot = runner.open_sequence()
        got = [runner.step([StepEntry(slot, prompt[:310], all_places(310))])]
        got += [runner.step([StepEntry(slot, [tok], [0])]) for tok in prompt[310:]]
        runner.close_sequence(slot)
        assert_close(torch.cat(got), want, "float32", "a far key through a reading layer")


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(tmp_path_factory, seed):
    """Layer kinds, their order, every size, head count, window, tap count and constant drawn anew: three unequal
    requests whole and alone, then begun together and decoded together, then one in portions, in float32 (the choice
    of experts itself is held) and, whole, in bfloat16 with the engine's choices handed over.  The float32 bound is
    wider than elsewhere: some drawn models are ill-conditioned."""
    import random

    from starter_b200.engine import ModelRunner, StepEntry, load_model
    from tiny_setotar import random_config

    rng = random.Random(2000 + seed)
    raw = random_config(rng)
    folder = make_setotar_folder(tmp_path_factory.mktemp(f"r{seed}"), f"R{seed}", seed=seed, dtype=torch.bfloat16, raw=raw)
    cfg, w = plain.read_model_folder(folder)
    lengths = [rng.choice([1, 3, 40, 130]), rng.choice([2, 70, 150]), rng.choice([5, 64, 65, 200])]
    prompts = [random_prompt(n, cfg["vocab"], seed * 10 + i) for i, n in enumerate(lengths)]
    want = [plain.forward(cfg, w, p) for p in prompts]
    runner = ModelRunner(load_model(folder, "float32"), max_tokens=64 * 40, max_sequences=8, use_graphs=False)
    for p, wanted in zip(prompts, want):
        slot = runner.open_sequence()
        got = runner.step([StepEntry(slot, p, all_places(len(p)))])
        runner.close_sequence(slot)
        close(got, wanted, "float32", f"whole, length {len(p)}", fp32=3e-4)
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
        close(torch.cat(got[i]), want[i], "float32", f"begun and decoded together, request {i}", fp32=3e-4)
    slot, rows, at = runner.open_sequence(), [], 0
    for n in (2, 1, 3, 61, 70, 200):
        part = prompts[2][at:at + n]
        if part:
            rows.append(runner.step([StepEntry(slot, part, all_places(len(part)))]))
            at += len(part)
    runner.close_sequence(slot)
    close(torch.cat(rows), want[2], "float32", "in portions", fp32=3e-4)
    runner.check_status()
    runner.cache.check()
    assert runner.cache.slots.held_count == 0 and runner.cache.pages.held_count == 0
    routed = Routed(ModelRunner(load_model(folder, "bfloat16"), max_tokens=64 * 40, max_sequences=8, use_graphs=False))
    for p in prompts:
        slot = routed.runner.open_sequence()
        got = routed.step([StepEntry(slot, p, all_places(len(p)))], [len(p)])
        routed.runner.close_sequence(slot)
        held = plain.forward(cfg, w, p, routes=routed.routes(len(p), "bfloat16"))
        # a drawn model may be ill-conditioned: the mean error says whether the mechanisms are right
        mean = float((got.double().cpu() - held).abs().mean()) / float(held.abs().max())
        assert mean <= 2e-2, f"bfloat16, length {len(p)}: mean error {mean:.3e} of the largest logit"


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
        assert [s[i] for s in steps] == plain.generate(cfg, w, prompt, 70), f"request {i}"


def test_random_weights_from_the_library_run_in_bfloat16():
    """``random_model`` places every tensor as the loader would, and sampling with temperature runs."""
    from starter_b200 import Engine
    from starter_b200.config import config_from_dict
    from starter_b200.engine.runner import random_model

    model = random_model(config_from_dict(TINY_S["SC"]), seed=5, dtype="bfloat16")
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
    folder, cfg, w = case(tmp_path_factory, "SB")
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
