"""Korurax on the GPU against the plain statement: each mechanism alone, then the model through the step
function, the cache and the generation loop, cut into steps and batches in every way."""

import math

import pytest
import torch

import plain_korurax as plain
from gpu_helpers import DTYPES, FP32_TOL
from tiny import random_prompt
from tiny_korurax import TINY_R, make_korurax_folder

pytestmark = pytest.mark.gpu

CONFIGS = ["RA", "RB", "RC"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64
_cases, _runners = {}, {}


def case(tmp_path_factory, name, seed=1):
    if (name, seed) not in _cases:
        folder = make_korurax_folder(tmp_path_factory.mktemp(f"r{name}{seed}"), name, seed=seed)
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


# Bounds of the model-level comparisons, relative to the largest logit of the case.  float32: as for the
# other designs.  bfloat16 against the float64 statement: the largest row and the mean of a comparison, from
# measurements on these configurations (a lost key, a chunk that is one off or a skipped layer moves rows by
# 1e-1 and more, and the float32 runs of the same kernels hold every row to 2e-5).
BF16_ROW_TOL = 5e-2
BF16_MEAN_TOL = 8e-3


def assert_close(got, want, dtype, what="", stray=0.0):
    """Fails with the first wrong row named: its place is the clue (a prompt's end, the first single-token
    step, a page boundary, a chunk's edge).  ``stray`` (bfloat16 only, for comparisons of hundreds of rows):
    the share of rows that may pass the row bound, none of them by more than twice; among hundreds of rows the
    tail of bfloat16 rounding (one sharp softmax) reaches further than among a tiny case's dozens, while a
    lost key or a misplaced tile moves whole runs of rows, and by far more.  float32 holds every row."""
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(want.shape)}"
    scale = float(want.abs().max())
    tol = (FP32_TOL if dtype == "float32" else BF16_ROW_TOL) * scale
    err = (got - want).abs().reshape(want.shape[0], -1).max(dim=1).values
    bad = (~(err <= tol)).nonzero().flatten().tolist()
    if dtype != "float32" and stray > 0.0 and len(bad) <= stray * len(err) and float(err.max()) <= 2.0 * tol:
        bad = []
    assert not bad, (f"{what}: {len(bad)} of {len(err)} rows off by more than {tol:.2e}; first wrong row {bad[0]} "
                     f"(error {err[bad[0]].item():.3e}), largest error {err.max().item():.3e}")
    if dtype != "float32":
        mean = (got - want).abs().mean().item()
        assert mean <= BF16_MEAN_TOL * scale, f"{what}: mean error {mean:.3e} above {BF16_MEAN_TOL * scale:.3e}"


def dev(v, ty=torch.float32):
    return v.to("cuda", ty).contiguous()


def ints(a):
    return torch.tensor(a, dtype=torch.int32, device="cuda")


class Routed:
    """Runs steps and notes, per request, which experts every routed layer chose for each of its tokens.
    The 32-bit comparisons do not use the notes (there the choice itself is held to the plain statement);
    the bfloat16 comparisons hand them to the plain statement, because a near-tie between two experts may
    fall either way once the router's input is rounded to 8 bits, and that is no fault."""

    def __init__(self, runner):
        self.runner = runner
        self.layers = [i for i, b in enumerate(runner.model.blocks)
                       if getattr(b, "feed_forward", None) is not None and hasattr(b.feed_forward, "last_ids")]
        self.notes = {}

    def step(self, entries, keys):
        out = self.runner.step(entries)
        at = 0
        for entry, key in zip(entries, keys):
            n = len(entry.tokens)
            for layer in self.layers:
                ids = self.runner.model.blocks[layer].feed_forward.last_ids[at:at + n].cpu()
                self.notes.setdefault(key, {}).setdefault(layer, []).append(ids)
            at += n
        return out

    def routes(self, key, dtype):
        if dtype == "float32" or not self.layers:
            return None
        return {layer: torch.cat(parts) for layer, parts in self.notes[key].items()}


# ------------------------------------------------------------------------------ mechanisms alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("norm", ["layernorm", "rmsnorm"])
@pytest.mark.parametrize("hidden", [40, 37, 600, 13000])
def test_the_stream_step_alone(hidden, norm, dtype):
    """The sum inside a layer, a layer's end (filing, the sum over 1 to 5 levels), the model's end on chosen
    rows, and the norm alone; rows with a large mean, which a layer norm must take off."""
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(hidden)
    n, mult, eps = 7, 0.3, 1e-5
    gain = torch.randn(hidden, generator=g, dtype=F) * 0.3 + 1.0

    def normed(x):
        return plain.layer_norm(x, gain, eps) if norm == "layernorm" else plain.rms_norm(x, gain, eps)

    for levels in (1, 2, 5):
        history = torch.randn(levels, n, hidden, generator=g, dtype=F) * 2.0 + 3.0
        base = torch.randn(n, hidden, generator=g, dtype=F) + 5.0
        y = dev(torch.randn(n, hidden, generator=g, dtype=F), t)
        mix = torch.rand(levels, generator=g, dtype=F) + 0.1
        hd, bd = dev(history), dev(base)
        # inside a layer
        dst = torch.zeros(n, hidden, device="cuda")
        out = ops.depth_step(bd, t, y, mult, dst=dst, norm=(norm, dev(gain), eps))
        x = bd.double().cpu() + mult * y.double().cpu()
        close(dst, x, "float32", "the sum inside a layer")
        close(out, normed(x), dtype, "its norm", bf16=1e-2)
        # a layer's end
        dst = torch.zeros(n, hidden, device="cuda")
        out = ops.depth_step(bd, t, y, mult, hd, dev(mix), dst, (norm, dev(gain), eps))
        close(hd[levels - 1], x, "float32", "the layer's result, filed")
        joined = mix[levels - 1] * x + sum(mix[j] * history[j] for j in range(levels - 1))
        close(dst, joined, "float32", f"the sum over {levels} levels")
        close(out, normed(joined), dtype, "its norm", bf16=1e-2)
        # the model's end on chosen rows: nothing is written
        hd2, before = dev(history), dev(history)
        rows = ints([5, 0, 5, 2])
        out = ops.depth_step(bd, t, y, mult, hd2, dev(mix), None, (norm, dev(gain), eps), rows=rows)
        assert torch.equal(hd2, before)
        close(out, normed(joined)[[5, 0, 5, 2]], dtype, "chosen rows", bf16=1e-2)
    out = ops.depth_step(bd, t, norm=(norm, dev(gain), eps))
    close(out, normed(bd.double().cpu()), dtype, "the norm alone", bf16=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_cap_and_clamped_gate_alone(dtype):
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(3)
    logits = torch.randn(5, 77, generator=g, dtype=F) * 20.0
    got = ops.softcap(dev(logits), 6.5)
    close(got, 6.5 * torch.tanh(logits / 6.5), "float32", "the cap")
    gu = dev(torch.randn(9, 2 * 52, generator=g, dtype=F) * 2.0, t)       # most entries past a limit of 0.8
    got = ops.gated_clamped(gu, 0.8)
    a, b = gu.double().cpu()[:, :52].clamp(max=0.8), gu.double().cpu()[:, 52:].clamp(-0.8, 0.8)
    close(got, a * torch.sigmoid(1.702 * a) * (b + 1.0), dtype, "the clamped gate", bf16=5e-3)


@pytest.mark.parametrize("rows", [1, 8, 40, 128, 200, 512, 700])
@pytest.mark.parametrize("width, inner, limit", [(256, 192, 0.9), (128, 64, 2.0), (136, 72, 1.0)])
def test_clamped_gated_product_fused_and_not(rows, width, inner, limit):
    """The activation inside the tensor-core products' epilogues (few rows; 512 and more) and behind a plain
    product (in between, and sizes the tensor-core products refuse): all against the plain statement."""
    from starter_b200 import ops

    g = torch.Generator().manual_seed(rows + inner)
    x = dev(torch.randn(rows, width, generator=g, dtype=F), torch.bfloat16)
    w = dev(torch.randn(2 * inner, width, generator=g, dtype=F) * 0.12, torch.bfloat16)     # many entries past the limits
    got = ops.linear_gated_clamped(x, w, limit)
    gu = (x.double().cpu() @ w.double().cpu().T).to(torch.bfloat16).double()
    a, b = gu[:, :inner].clamp(max=limit), gu[:, inner:].clamp(-limit, limit)
    close(got, a * torch.sigmoid(1.702 * a) * (b + 1.0), "bfloat16", f"{rows} rows", bf16=1.2e-2)
    x32, w32 = x.float(), w.float()
    got = ops.linear_gated_clamped(x32, w32, limit)
    gu = x32.double().cpu() @ w32.double().cpu().T
    a, b = gu[:, :inner].clamp(max=limit), gu[:, inner:].clamp(-limit, limit)
    close(got, a * torch.sigmoid(1.702 * a) * (b + 1.0), "float32", f"{rows} rows, float32", fp32=1e-5)


def paged(k, v, t, pages=(5, 2, 7, 0, 3)):
    """Keys ``[T, G, D]`` and values ``[T, G, Dv]`` of one sequence filed in scattered pages of slot 1."""
    n, kv_heads, dim = k.shape
    vdim = v.shape[2]
    table = torch.zeros(3, 8, dtype=torch.int32, device="cuda")
    table[1, :len(pages)] = torch.tensor(pages, dtype=torch.int32)
    ks = torch.zeros(8, kv_heads, 64, dim, dtype=t, device="cuda")
    vs = torch.zeros(8, kv_heads, 64, vdim, dtype=t, device="cuda")
    for i, page in enumerate(pages):
        part = slice(64 * i, min(n, 64 * (i + 1)))
        if part.start >= n:
            break
        ks[page, :, :part.stop - part.start] = k[part].transpose(0, 1).to(t)
        vs[page, :, :part.stop - part.start] = v[part].transpose(0, 1).to(t)
    return ks, vs, table


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, chunk, window, extras", [
    (4, 2, 16, 32, 10, None, "psg"), (6, 1, 24, 40, 3, None, "psg"), (4, 2, 32, 64, 64, None, "psg"),
    (6, 2, 64, 32, 100, None, "psg"), (8, 1, 16, 16, 130, None, "psg"), (2, 2, 128, 128, 65, None, "psg"),
    (3, 3, 64, 64, None, None, "s"), (4, 1, 32, 32, None, 70, "p"), (2, 1, 64, 16, 128, 33, "g"),
    (5, 5, 16, 64, 1000, None, ""), (4, 4, 8, 8, 1, None, "psg"), (4, 2, 64, 64, 100, None, "psg"),
    (2, 1, 128, 128, None, 90, "pg"), (2, 2, 64, 64, 200, 150, "")])
def test_attention_alone_with_one_key_that_stands_out(heads, kv_heads, dim, vdim, chunk, window, extras, dtype):
    """Queries late in a sequence of 300 (five scattered pages) score one key far above the rest: the first
    key of the query's chunk and the key just before it, keys on either side of a page border, the query's
    own place, a key far back in the chunk; the answer must hold that key's value, or must not.  The plain
    kernel and the tensor-core kernel, whole, as a later portion, and the last token alone with its pages in
    1, 3 and 7 parts; each of penalty, sink and gate switched on and off."""
    from starter_b200 import ops

    t = TORCH[dtype]
    n, scale = 300, 0.2
    g = torch.Generator().manual_seed(heads * 100 + dim + (chunk or 0))
    q = torch.randn(n, heads, dim, generator=g, dtype=F)
    k = torch.randn(n, kv_heads, dim, generator=g, dtype=F)
    v = torch.randn(n, kv_heads, vdim, generator=g, dtype=F)
    r1 = torch.rand(heads, generator=g, dtype=F) * 0.8 + 0.05 if "p" in extras else None
    r2 = torch.rand(heads, generator=g, dtype=F) * 1.5 + 0.05 if "p" in extras else None
    sink = torch.randn(heads, generator=g, dtype=F) + 1.0 if "s" in extras else None
    gate = torch.rand(n, heads, generator=g, dtype=F) if "g" in extras else None
    group = heads // kv_heads
    c = chunk or n
    probes = {}                                   # query position -> the key made to stand out
    for q_pos in (299, 257, 250, 200, 193, 130, 129, 64):
        start = max(q_pos // c * c, q_pos - (window or n) + 1, 0)
        for key in (start, start - 1):
            if 0 <= key <= q_pos and q_pos not in probes:
                probes[q_pos] = key
        q_pos2 = q_pos - 3
        if q_pos2 not in probes and q_pos2 - 1 >= 0:
            probes[q_pos2] = start - 1 if start >= 1 else 0
    probes[280] = 280                             # its own place
    probes[191] = 128                             # across a page border, far back
    for q_pos, key in probes.items():
        for h in range(heads):
            direction = k[key, h // group] / k[key, h // group].norm()
            q[q_pos, h] = direction * (60.0 / scale / max(1.0, float(k[key, h // group].norm())) * 1.0)
    qd, kd, vd = dev(q, t), dev(k, t), dev(v, t)
    qr, kr, vr = qd.double().cpu(), kd.double().cpu(), vd.double().cpu()
    want = plain.attend(qr, kr, vr, scale, r1, r2, sink, gate, chunk, window).reshape(n, heads * vdim)
    ks, vs, table = paged(kd, vd, t)
    pos, slot = torch.arange(n, dtype=torch.int32, device="cuda"), torch.ones(n, dtype=torch.int32, device="cuda")
    pen = (dev(r1), dev(r2)) if r1 is not None else None
    sk = dev(sink) if sink is not None else None
    gt = dev(gate) if gate is not None else None
    q2 = qd.reshape(n, heads * dim)
    out = ops.sink_attention(q2, ks, vs, table, slot, pos, heads, kv_heads, dim, vdim, scale, pen, sk, gt, chunk, window)
    close(out, want, dtype, "plain kernel, whole")
    tail = torch.arange(260, 300, device="cuda")
    out = ops.sink_attention(q2[tail].contiguous(), ks, vs, table, slot[tail].contiguous(), pos[tail].contiguous(), heads,
                             kv_heads, dim, vdim, scale, pen, sk, gt[tail].contiguous() if gt is not None else None,
                             chunk, window)
    close(out, want[260:], dtype, "plain kernel, single tokens")
    if not ops.sink_tc_takes(q2, heads, kv_heads, dim, vdim):
        return
    out = ops.sink_attention_tc(q2, ks, vs, table, ints([1]), ints([0]), ints([n]), ints([n]), ints([0, 0, 0, 0, 0]),
                                ints([128, 0, 256, 192, 64]), heads, kv_heads, dim, vdim, scale, pen, sk, gt, chunk, window)
    close(out, want, dtype, "tensor cores, whole")
    out = ops.sink_attention_tc(q2[tail].contiguous(), ks, vs, table, ints([1]), ints([0]), ints([40]), ints([n]), ints([0]),
                                ints([0]), heads, kv_heads, dim, vdim, scale, pen, sk,
                                gt[tail].contiguous() if gt is not None else None, chunk, window)
    close(out, want[260:], dtype, "tensor cores, a later portion")
    for parts in (1, 3, 7):
        out = ops.sink_attention_tc(q2[299:].contiguous(), ks, vs, table, ints([1]), ints([0]), ints([1]), ints([n]),
                                    ints([0]), ints([0]), heads, kv_heads, dim, vdim, scale, pen, sk,
                                    gt[299:].contiguous() if gt is not None else None, chunk, window, n_splits=parts)
        close(out, want[299:], dtype, f"tensor cores, one token in {parts} parts")
    if not ops.sink_tcgen05_takes(q2, dim, vdim):
        return
    # the tcgen05 kernel: blocks of 256 queries (one full, one of 44), from the list of blocks and from the
    # list of tiles; then a later portion of 170 tokens
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    for blocks in ((ints([0, 0]), ints([0, 256])), None):
        out = ops.sink_attention_tcgen05(q2, ks, vs, table, ints([1]), ints([0]), ints([n]), ints([n]), ints([0, 0, 0, 0, 0]),
                                         ints([128, 0, 256, 192, 64]), heads, kv_heads, dim, scale, pen, sk, gt, chunk, window,
                                         status, blocks, vdim)
        close(out, want, dtype, "tcgen05, whole")
    late = torch.arange(130, 300, device="cuda")
    out = ops.sink_attention_tcgen05(q2[late].contiguous(), ks, vs, table, ints([1]), ints([0]), ints([170]), ints([n]),
                                     ints([0, 0, 0]), ints([0, 64, 128]), heads, kv_heads, dim, scale, pen, sk,
                                     gt[late].contiguous() if gt is not None else None, chunk, window, status,
                                     (ints([0]), ints([0])), vdim)
    close(out, want[130:], dtype, "tcgen05, a later portion")
    assert int(status.item()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_prepare_alone(dtype):
    """Keys and values filed on both sides of a page border, gates formed, padding behind the gates ignored."""
    from starter_b200 import ops

    t = TORCH[dtype]
    heads, kv_heads, dim, vdim = 3, 3, 8, 24
    width = heads * dim + kv_heads * (dim + vdim) + heads
    pad = -width % 8
    g = torch.Generator().manual_seed(5)
    proj = dev(torch.randn(6, width + pad, generator=g, dtype=F) * 2.0, t)
    table = torch.zeros(4, 4, dtype=torch.int32, device="cuda")
    table[2, :3] = ints([6, 1, 4])
    pos, slot = ints([62, 63, 64, 65, 127, 128]), ints([2] * 6)
    ks = torch.zeros(8, kv_heads, 64, dim, dtype=t, device="cuda")
    vs = torch.zeros(8, kv_heads, 64, vdim, dtype=t, device="cuda")
    gate = ops.sink_prepare(proj, heads, kv_heads, dim, vdim, pos, slot, table, ks, vs)
    close(gate, torch.sigmoid(proj.double().cpu()[:, width - heads:width]), "float32", "gates", fp32=1e-6)
    for row, p in enumerate(pos.tolist()):
        page = int(table[2, p // 64])
        kk = proj[row, heads * dim:heads * dim + kv_heads * dim].reshape(kv_heads, dim)
        vv = proj[row, heads * dim + kv_heads * dim:width - heads].reshape(kv_heads, vdim)
        assert torch.equal(ks[page, :, p % 64], kk) and torch.equal(vs[page, :, p % 64], vv), p
    assert int((ks != 0).any(dim=-1).sum()) == 6 * kv_heads


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [8, 4])
def test_half_split_rotation_of_the_latent_parts_alone(dims, dtype):
    """The shared key part in the cache row and the queries' rotated parts, entry i with entry i + dims / 2."""
    from starter_b200 import ops
    from starter_b200.config import PartialRopeSpec
    from starter_b200.parts import PartialRotaryTable

    t = TORCH[dtype]
    heads, dim, rot, q_rank, rank, base = 3, 8, 8, 12, 16, 100.0
    table_part = PartialRotaryTable(PartialRopeSpec(dims=dims, base=base), t, "cuda")
    table_part.ensure(200)
    rotation = table_part.rotation()
    cos, sin = ops.latent_tables(rotation, dims)
    g = torch.Generator().manual_seed(dims)
    n = 5
    proj = dev(torch.randn(n, q_rank + rank + rot, generator=g, dtype=F), t)
    qg, kg = torch.rand(q_rank, generator=g, dtype=F) + 0.5, torch.rand(rank, generator=g, dtype=F) + 0.5
    pos, slot = ints([0, 63, 64, 130, 199]), ints([1] * n)
    table = torch.zeros(2, 4, dtype=torch.int32, device="cuda")
    table[1] = ints([3, 0, 2, 1])
    store = torch.zeros(4, 1, 64, rank + rot, dtype=t, device="cuda")
    cq = ops.latent_prepare(proj, dev(qg), dev(kg), 1e-5, cos, sin, pos, slot, table, store, q_rank, rank, rot, dims,
                            layout=rotation.layout)
    pr = proj.double().cpu()
    close(cq, plain.rms_norm(pr[:, :q_rank], qg, 1e-5), dtype, "the query latent", bf16=1e-2)
    want_c = plain.rms_norm(pr[:, q_rank:q_rank + rank], kg, 1e-5)
    want_r = plain.rotate_half_split(pr[:, q_rank + rank:], pos.cpu(), base, dims)
    for row, p in enumerate(pos.tolist()):
        got = store[int(table[1, p // 64]), 0, p % 64]
        close(got[:rank], want_c[row], dtype, f"latent at {p}", bf16=1e-2)
        close(got[rank:], want_r[row], dtype, f"shared key part at {p}", bf16=1e-2)
    q = dev(torch.randn(n, heads * (dim + rot), generator=g, dtype=F), t)
    qa = torch.zeros(n, heads, rank + rot, dtype=t, device="cuda")
    ops.latent_rotate_q(q, qa, cos, sin, pos, heads, dim, rot, dims, rank, layout=rotation.layout)
    want_q = plain.rotate_half_split(q.double().cpu().reshape(n, heads, dim + rot)[..., dim:], pos.cpu(), base, dims)
    close(qa[..., rank:], want_q, dtype, "the queries' rotated parts", bf16=1e-2)


@pytest.mark.parametrize("experts, top, scale", [(5, 2, 2.0), (3, 1, 0.7), (3, 3, 1.0), (12, 5, 1.5), (64, 8, 3.0)])
def test_router_with_sigmoid_scores_alone(experts, top, scale):
    from starter_b200 import ops

    g = torch.Generator().manual_seed(experts)
    h = torch.randn(33, 48, generator=g, dtype=F)
    router = torch.randn(experts, 48, generator=g, dtype=F) * 0.5
    ids, weights = ops.moe_route(dev(h), dev(router), None, top, "sigmoid_normalised", scale)
    want_ids, want_w = plain.route(dev(h).double().cpu(), dev(router).double().cpu(), top, scale)
    assert torch.equal(ids.cpu().long(), want_ids)
    close(weights, want_w, "float32", "weights", fp32=1e-5)
    assert torch.allclose(weights.sum(dim=1).cpu().double(), torch.full((33,), scale, dtype=F), atol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 5, 70, 300])
@pytest.mark.parametrize("experts, top, width, inner", [(5, 2, 64, 24), (3, 3, 96, 16), (8, 2, 128, 64), (6, 1, 40, 36)])
def test_squared_relu_experts_alone(experts, top, width, inner, rows, dtype):
    from starter_b200 import ops

    t = TORCH[dtype]
    g = torch.Generator().manual_seed(rows + experts)
    h = dev(torch.randn(rows, width, generator=g, dtype=F), t)
    up = dev(torch.randn(experts, inner, width, generator=g, dtype=F) * 0.2, t)
    down = dev(torch.randn(experts, width, inner, generator=g, dtype=F) * 0.2, t)
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(rows)]).to(torch.int32)
    weights = torch.rand(rows, top, generator=g, dtype=F) + 0.1
    got = ops.moe_experts(h, dev(ids, torch.int32), dev(weights), up, down, expert="relu2")
    hd, ud, dd = h.double().cpu(), up.double().cpu(), down.double().cpu()
    want = torch.zeros(rows, width, dtype=F)
    for r in range(rows):
        for c in range(top):
            e = int(ids[r, c])
            want[r] += weights[r, c] * ((torch.relu(ud[e] @ hd[r]) ** 2) @ dd[e].T)
    close(got, want, dtype, "experts", bf16=2.5e-2)


@pytest.mark.parametrize("rows", [3, 700])
@pytest.mark.parametrize("experts, top, width, inner", [(3, 2, 144, 80), (4, 1, 256, 128), (5, 3, 48, 272)])
def test_squared_relu_experts_on_every_tile_kind(experts, top, width, inner, rows):
    """The plain tiles and both tensor-core tiles (64 rows; 128 rows, which steps with many rows an expert
    choose) against the experts one by one: inner sizes and widths that end inside a k-slice and inside a
    tile's outputs, one expert with a handful of rows next to experts with hundreds."""
    from starter_b200 import ops

    g = torch.Generator().manual_seed(rows * experts + width)
    h = dev(torch.randn(rows, width, generator=g, dtype=F), torch.bfloat16)
    up = dev(torch.randn(experts, inner, width, generator=g, dtype=F) * 0.2, torch.bfloat16)
    down = dev(torch.randn(experts, width, inner, generator=g, dtype=F) * 0.2, torch.bfloat16)
    ids = torch.stack([torch.randperm(experts - 1, generator=g)[:top] for _ in range(rows)]).to(torch.int32)
    ids[:min(rows, 5), 0] = experts - 1          # the last expert serves five rows at most
    if top > 1:
        ids[:min(rows, 5), 1:] = torch.arange(top - 1, dtype=torch.int32)
    weights = torch.rand(rows, top, generator=g, dtype=F) + 0.1
    hd, ud, dd = h.double().cpu(), up.double().cpu(), down.double().cpu()
    want = torch.zeros(rows, width, dtype=F)
    for e in range(experts):
        chosen = (ids == e)
        share = (weights * chosen).sum(dim=1)
        used = share > 0
        want[used] += share[used, None] * ((torch.relu(hd[used] @ ud[e].T) ** 2) @ dd[e].T)
    if rows * top >= 128 * experts:
        assert ops._lib("moe").sb_moe_tile_rows_for(1, width, inner, rows * top, experts) in (128, 256)
    got = ops.moe_experts(h, dev(ids, torch.int32), dev(weights), up, down, expert="relu2")
    close(got, want, "bfloat16", "the tiles the step chooses", bf16=2.5e-2)
    for tile_rows in (4, 32, 64, 128, 256):
        got = ops.moe_experts(h, dev(ids, torch.int32), dev(weights), up, down, expert="relu2", tile_rows=tile_rows)
        close(got, want, "bfloat16", f"tiles of {tile_rows} rows", bf16=2.5e-2)


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
        want = plain.forward(cfg, w, prompt, expert_ids=routed.routes(length, dtype))
        assert_close(got, want, dtype, f"{name} whole, length {length}")
        assert_close(got[:3], want[:3], dtype, f"{name}: the first tokens of a sequence")
    runner.check_status()
    runner.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_of_a_wider_model(tmp_path_factory, dtype):
    """Prompts of hundreds of tokens on a wider model, where a step's shape chooses the large tiles (hundreds of
    rows an expert, keys and values of 128): whole, then the same request as a long portion, a short one and
    single tokens, next to a second request."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, "RD")
    routed = Routed(runner_for(tmp_path_factory, "RD", dtype))
    runner = routed.runner
    prompt, other = random_prompt(700, cfg["vocab"], 71), random_prompt(333, cfg["vocab"], 72)
    slot = runner.open_sequence()
    got = routed.step([StepEntry(slot, prompt, all_places(700))], ["whole"])
    runner.close_sequence(slot)
    want = plain.forward(cfg, w, prompt, expert_ids=routed.routes("whole", dtype))
    assert_close(got, want, dtype, "RD whole, 700 tokens", stray=0.01)
    a, b = runner.open_sequence(), runner.open_sequence()
    rows = [routed.step([StepEntry(a, prompt[:600], all_places(600)), StepEntry(b, other, all_places(333))], ["a", "b"])]
    got_b = rows[0][600:]
    rows = [rows[0][:600], routed.step([StepEntry(a, prompt[600:690], all_places(90))], ["a"])]
    runner.close_sequence(b)
    for tok in prompt[690:]:
        rows.append(routed.step([StepEntry(a, [tok], [0])], ["a"]))
    runner.close_sequence(a)
    assert_close(torch.cat(rows), plain.forward(cfg, w, prompt, expert_ids=routed.routes("a", dtype)), dtype,
                 "RD in portions of 600, 90 and single tokens", stray=0.01)
    assert_close(got_b, plain.forward(cfg, w, other, expert_ids=routed.routes("b", dtype)), dtype,
                 "RD: the request beside it", stray=0.01)
    runner.check_status()
    runner.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_every_layer_against_the_plain_layers(tmp_path_factory, name, dtype):
    """The stream behind each layer (summed over depth), which names the first layer that differs."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    model = runner.model
    prompt = random_prompt(90, cfg["vocab"], 8)
    slot = runner.open_sequence()
    ctx = runner.make_context([StepEntry(slot, prompt, [len(prompt) - 1])])
    stream, pending = model.hidden(ctx)
    model.logits(stream, pending, ctx.want_rows, ctx.status)
    runner.close_sequence(slot)
    routes = {i: b.feed_forward.last_ids.cpu() for i, b in enumerate(model.blocks)
              if getattr(b, "feed_forward", None) is not None and hasattr(b.feed_forward, "last_ids")}
    _, want = plain.forward(cfg, w, prompt, expert_ids=None if dtype == "float32" else routes, return_layers=True)
    history = stream.history.double().cpu()
    for i in range(len(cfg["layers"]) - 1):           # the last layer's result is never filed: the end takes chosen rows
        mix = model.blocks[i].connection.weights.double().cpu()
        got = sum(mix[j] * history[j] for j in range(i + 2))
        close(got, want[i], dtype, f"{name} behind layer {i}", fp32=2e-5, bf16=2.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_then_tokens_one_by_one(tmp_path_factory, name, dtype):
    """Chunks of 3, 10, 64, 65, 100 and 130 begin and end among decoded tokens, and page borders are crossed
    while decoding."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    routed = Routed(runner_for(tmp_path_factory, name, dtype))
    runner = routed.runner
    for length, tail in ((40, 39), (100, 45), (150, 90), (270, 20)):
        prompt = random_prompt(length, cfg["vocab"], 20 + length)
        slot = runner.open_sequence()
        head = length - tail
        rows = [routed.step([StepEntry(slot, prompt[:head], all_places(head))], [length])]
        for tok in prompt[head:]:
            rows.append(routed.step([StepEntry(slot, [tok], [0])], [length]))
        runner.close_sequence(slot)
        got = torch.cat(rows)
        want = plain.forward(cfg, w, prompt, expert_ids=routed.routes(length, dtype))
        assert_close(got, want, dtype, f"{name} last {tail} one by one, length {length}")
        assert_close(got[head:head + 1], want[head:head + 1], dtype, "the first single-token step")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["RA", "RC"])
def test_long_decoding_over_many_pages(tmp_path_factory, name, dtype):
    """Two requests of unequal lengths decoded together for 300 steps, the longer one over six pages; the
    shorter one ends on the way; every logit is held to the plain statement."""
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
        want = plain.forward(cfg, w, prompts[i], expert_ids=routed.routes(i, dtype))
        assert_close(torch.cat(got[i]), want, dtype, f"{name} request {i} decoded to {lengths[i]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_portions_of_several_sizes(tmp_path_factory, name, dtype):
    """Portions cut inside chunks, at their edges and across pages; chunks are counted from the sequence's
    start wherever a portion begins."""
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    prompt = random_prompt(171, cfg["vocab"], 77)
    for sizes in ((2, 2, 3, 57, 64, 1, 40, 2), (63, 2, 63, 43), (5, 128, 38), (10, 90, 30, 41)):
        routed = Routed(runner_for(tmp_path_factory, name, dtype))
        runner = routed.runner
        slot = runner.open_sequence()
        rows, at = [], 0
        for n in sizes:
            rows.append(routed.step([StepEntry(slot, prompt[at:at + n], all_places(n))], [0]))
            at += n
        assert at == len(prompt)
        runner.close_sequence(slot)
        want = plain.forward(cfg, w, prompt, expert_ids=routed.routes(0, dtype))
        assert_close(torch.cat(rows), want, dtype, f"{name} portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_unequal_batches_with_slots_and_pages_used_again(tmp_path_factory, name, dtype):
    from starter_b200.engine import StepEntry

    _, cfg, w = case(tmp_path_factory, name)
    runner = runner_for(tmp_path_factory, name, dtype)
    vocab = cfg["vocab"]
    batches = [[(70, 9), (5, 3), (33, 12), (1, 6)], [(2, 40), (129, 2), (64, 5)], [(17, 0), (63, 3)]]
    seed = 300
    for batch in batches:
        routed = Routed(runner)
        seqs, slots, got = [], [], []
        for plen, extra in batch:
            seed += 1
            seqs.append(random_prompt(plen + extra, vocab, seed))
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
            want = plain.forward(cfg, w, seq, expert_ids=routed.routes(i, dtype))
            assert_close(torch.cat(got[i]), want, dtype, f"{name} batch {batch}, request {i}")
        runner.cache.check()
    assert runner.cache.slots.held_count == 0 and runner.cache.pages.held_count == 0


@pytest.mark.parametrize("name", CONFIGS)
def test_greedy_generation_through_the_entry_point(tmp_path_factory, name):
    """Unequal prompts through ``Engine.generate`` (the scheduler, the captured single-token step, the
    sampler): 70 tokens each, past a page border and past chunk edges, equal to the plain statement's greedy
    continuation."""
    from starter_b200 import Engine

    folder, cfg, w = case(tmp_path_factory, name)
    engine = Engine(folder, dtype="float32", max_batch=4)
    prompts = [random_prompt(n, cfg["vocab"], 900 + n) for n in (50, 3, 21)]
    steps = list(engine.generate(prompts, 70))
    assert len(steps) == 70
    for i, prompt in enumerate(prompts):
        assert [s[i] for s in steps] == plain.generate(cfg, w, prompt, 70), f"request {i}"


def test_random_weights_from_the_library_run_in_bfloat16():
    """``random_model`` places every tensor as the loader would, and sampling with temperature runs through
    the captured step on tensor cores."""
    from starter_b200 import Engine
    from starter_b200.config import config_from_dict
    from starter_b200.engine.runner import random_model

    model = random_model(config_from_dict(TINY_R["RC"]), seed=5, dtype="bfloat16")
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
    folder, cfg, w = case(tmp_path_factory, "RB")
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
    for dtype in ("float32", "bfloat16"):
        out_dir = str(tmp_path / dtype)
        proc = subprocess.Popen([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                                 "--out", out_dir, "--max-tokens", "210"], stdin=subprocess.PIPE, stdout=subprocess.PIPE,
                                text=True)
        for record in steps:
            proc.stdin.write(json.dumps(record) + "\n")
            proc.stdin.flush()
            assert proc.stdout.readline().strip() == f"done {record['step']}"
        proc.stdin.close()
        assert proc.wait(timeout=120) == 0
        if dtype != "float32":
            continue                 # (the routing of a bfloat16 run is not known here: it ran, with the files in place)
        want_a, want_b = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
        read = lambda s: torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{s}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]))  # noqa: E731
        assert_close(read(0), torch.stack([want_a[0], want_a[129], want_b[65]]), "float32", "the first step")
        for i in range(10):
            rows = [want_a[130 + i]] + ([want_b[66 + i]] if i < 4 and i % 2 else [])
            assert_close(read(1 + i), torch.stack(rows), "float32", f"step {1 + i}")
