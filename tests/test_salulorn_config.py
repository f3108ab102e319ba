"""Salulorn's configuration on the CPU: what config.json means, what is refused, the run order of looped layers, tensor
names, rotation tables, and the plain statement on cases whose answer is known."""

import copy
import math

import pytest
import torch

import plain_salulorn as plain
from tiny_salulorn import L_A, L_B, L_C, TINY_L, rot

F = torch.float64


def spec_of(raw):
    from starter_b200.config import config_from_dict

    return config_from_dict(raw).to_model_spec()


def test_every_size_and_constant_comes_from_the_config():
    spec = spec_of(L_A)
    assert (spec.architecture, spec.vocab_size, spec.hidden_size, spec.streams) == ("Salulorn", 210, 72, 1)
    assert not spec.tie_embeddings and spec.lm_head_name == "head" and spec.final_norm.gain_32bit and spec.final_norm.eps == 1e-6
    first, second, third, fourth, fifth = spec.layers
    s = first.mixer
    assert (s.kind, s.num_heads, s.head_dim, s.value_dim, s.tau, s.decay_rank, s.norm_eps) == \
        ("gated_linear_attention", 3, 12, 8, 4.0, 5, 1e-6)
    assert first.arrangement == "prenorm32_mixer_only" and set(first.parts) == {"mixer", "norm1"}
    a = second.mixer
    assert (a.kind, a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.scale) == ("sink_attention", 4, 2, 16, 24, 0.3)
    assert (a.window, a.softcap, a.conv, a.bias, a.row_norm, a.sink, a.norm_eps) == (10, 6.0, 4, True, True, True, 1e-6)
    assert not (a.unit_values or a.head_gate or a.distance_penalty or a.values_from_keys or a.keep_first) and a.fixed_sink is None
    assert (a.position.kind, a.position.base, a.position.dims, a.position.scaling) == ("rope_interleaved", 100.0, 8, None)
    assert second.arrangement == "parallel32" and second.feed_forward.intermediate_size == 40
    assert second.feed_forward.activation == "silu" and "norm2" not in second.parts
    m = third.mixer
    assert (m.kind, m.num_heads, m.head_dim, m.rot_dim, m.value_dim, m.q_rank, m.kv_rank, m.scale) == \
        ("latent_attention", 3, 20, 8, 12, 24, 40, 0.25)
    assert (m.sink, m.output_gate, m.window, m.own_kv, m.norm_eps) == (True, True, None, True, 1e-6)
    y = m.position.scaling
    assert (m.position.base, m.position.dims, y.factor, y.original, y.fast, y.slow) == (500.0, 8, 3.0, 60.0, 4.0, 0.5)
    assert fourth.mixer.decay_rank == 11
    b = fifth.mixer
    assert (b.position, b.window, b.softcap, b.conv, b.bias, b.row_norm, b.sink) == (None, None, None, None, True, True, True)


def test_run_order_of_looped_layers():
    """Every pass has cache entries of its own, and the junction stands in front of each pass's first layer."""
    spec = spec_of(L_A)
    assert [(e.layer, e.cache, e.junction) for e in spec.schedule] == \
        [(0, 0, None), (1, 1, 0), (2, 2, None), (1, 3, 0), (2, 4, None), (1, 5, 0), (2, 6, None), (3, 7, None), (4, 8, None)]
    assert all(e.writes_cache for e in spec.schedule) and len(spec.junctions) == 1 and spec.junctions[0].names == {"weight": "loop.in"}
    once = dict(L_A, loop=dict(start=0, stop=1, times=1))
    assert [(e.layer, e.junction) for e in spec_of(once).schedule] == [(0, 0), (1, None), (2, None), (3, None), (4, None)]
    assert [(e.layer, e.junction) for e in spec_of(L_B).schedule] == [(i, None) for i in range(4)] and not spec_of(L_B).junctions
    for raw in (*TINY_L.values(), once):
        assert [(e.layer, e.junction is not None) for e in spec_of(raw).schedule] == plain.run_order(raw)


def test_cache_and_state_needs():
    from starter_b200.engine.model import build_layers

    blocks, positions = build_layers(spec_of(L_A), torch.float32, "cpu")
    assert len(positions) == 2
    kv = [b.mixer.kv_need() for b in blocks]
    assert kv[0] is None and kv[3] is None
    assert (kv[1].num_kv_heads, kv[1].head_dim, kv[1].value_size, kv[1].window) == (2, 16, 24, 10)
    assert (kv[2].num_kv_heads, kv[2].head_dim, kv[2].value_size, kv[2].window) == (1, 48, 0, None)
    assert blocks[0].mixer.state_need().shape == (3 * 12 * 8,)
    assert blocks[1].mixer.state_need().shape == (3 * (4 * 16 + 2 * 16 + 2 * 24),)
    assert blocks[2].mixer.state_need() is None and blocks[4].mixer.state_need() is None
    assert build_layers(spec_of(L_B), torch.float32, "cpu")[0][0].mixer.state_need() is None       # one tap keeps nothing


def test_tensor_names():
    from starter_b200.engine.model import expected_tensors

    names = expected_tensors(spec_of(L_A))
    for name, shape in {"embed": (210, 72), "head": (210, 72), "final.norm": (72,), "loop.in": (72, 144), "l0.norm1": (72,),
                        "l0.mix.q": (36, 72), "l0.mix.v": (24, 72), "l0.mix.g": (24, 72), "l0.mix.a1": (5, 72), "l0.mix.a2": (36, 5),
                        "l0.mix.a2.b": (36,), "l0.mix.norm": (8,), "l0.mix.o": (72, 24), "l1.mix.q.b": (64,), "l1.mix.k.norm": (32,),
                        "l1.mix.v.conv": (48, 4), "l1.mix.sink": (4,), "l1.mix.o": (72, 96), "l1.mlp.gate": (40, 72),
                        "l1.mlp.down": (72, 40), "l2.mix.dq": (24, 72), "l2.mix.dq.norm": (24,), "l2.mix.uq": (84, 24),
                        "l2.mix.dkv": (48, 72), "l2.mix.dkv.norm": (40,), "l2.mix.uk": (60, 40), "l2.mix.uv": (36, 40),
                        "l2.mix.sink": (3,), "l2.mix.g": (36, 72), "l2.mix.o": (72, 36)}.items():
        assert tuple(names[name].shape) == shape, name
    for name in ("l0.mlp.gate", "l1.norm2", "l4.mix.q.conv", "l4.mlp.up"):
        assert name not in names, name
    assert "loop.in" not in expected_tensors(spec_of(L_B))


def test_the_decay_rank_comes_from_the_checkpoint():
    from starter_b200.config import ConfigError, config_from_dict

    raw = copy.deepcopy(L_A)
    for layer in raw["layers"]:
        layer["mixer"].pop("decay_rank", None)
    cfg = config_from_dict(raw)
    with pytest.raises(ConfigError, match="decay_rank"):
        cfg.to_model_spec()
    full = cfg.with_tensor_shapes({"l0.mix.a1": (7, 72), "l3.mix.a1": (2, 72), "l1.mix.q": (64, 72)})
    assert [full.to_model_spec().layers[i].mixer.decay_rank for i in (0, 3)] == [7, 2]
    with pytest.raises(ConfigError, match="rows"):
        config_from_dict(L_A).with_tensor_shapes({"l0.mix.a1": (6, 72)})


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="lstm"), "mixers"),
    (lambda c: c["layers"][0]["mixer"].update(extra=1), "extra"),
    (lambda c: c["layers"][0]["mixer"].update(tau=0.0), "positive"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "key/value heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][1]["mixer"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=0.0), "positive"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=6), "rot_dim"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(factor=0), "positive"),
    (lambda c: c["layers"][2]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "feed-forward"),
    (lambda c: c["layers"][1]["mlp"].update(ff=0), "ff"),
    (lambda c: c["loop"].update(stop=6), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["loop"].pop("start"), "start"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(streams=3), "streams"),
])
def test_what_is_refused(change, text):
    from starter_b200.config import ConfigError, config_from_dict

    raw = copy.deepcopy(L_A)
    change(raw)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(raw)


def test_config_round_trip():
    from starter_b200.config import config_from_dict

    for raw in TINY_L.values():
        cfg = config_from_dict(raw)
        assert config_from_dict(cfg.to_dict()) == cfg


def test_a_junction_needs_a_stream_it_can_stand_in():
    from dataclasses import replace

    from starter_b200.config import ScheduleEntry
    from starter_b200.engine import DecoderModel
    from tiny import TINY_A

    spec = spec_of(L_A)
    with pytest.raises(ValueError, match="junction"):
        DecoderModel(replace(spec_of(TINY_A), junctions=spec.junctions), torch.float32, "cpu")
    with pytest.raises(ValueError, match="junction 1"):
        DecoderModel(replace(spec, schedule=(ScheduleEntry(0, 0, junction=1),)), torch.float32, "cpu")


@pytest.mark.parametrize("turn", [rot(100.0, 8), rot(10000.0, 24, 5.0, 640, 24.0, 1.5), rot(1e6, 128, 8.0, 64, 4.0, 0.5),
                                  rot(500.0, 12, 1.0, 100, 8.0, 8.0), rot(10000.0, 2, 3.0, 32, 32.0, 1.0)])
def test_rotation_tables(turn):
    """The library's tables against the plain frequencies, far out too; growing them keeps what was there."""
    from starter_b200.config.salulorn import _position
    from starter_b200.parts.rotary import InterleavedRotaryTable

    table = InterleavedRotaryTable(_position(turn), torch.float32, "cpu")
    assert table.ensure(10) and not table.ensure(4096)
    before = table.cos.clone()
    assert table.ensure(5000)
    assert torch.equal(table.cos[:4096], before) and table.rotation().rotary_dim == turn["dims"]
    assert table.rotation().layout == "interleaved"
    f, mult = plain.frequencies(turn)
    pos = torch.arange(table.length, dtype=F)
    for got, want in ((table.cos, (pos[:, None] * f).cos() * mult), (table.sin, (pos[:, None] * f).sin() * mult)):
        assert float((got.double() - want).abs().max()) < 2e-7 * mult


# ------------------------------------------------------------------------------ the plain statement, by hand

def test_plain_frequencies_stretch_by_parts():
    # index(t) = 8 ln(40 pi / (2 pi t)) / (2 ln 10): 20 turns at 0, 2 turns at 4: ramps 0, 1/4, 2/4, 3/4
    f, mult = plain.frequencies(rot(10.0, 8, 2.0, 40.0 * math.pi, 20.0, 2.0))
    plain_f = [10.0 ** (-2 * i / 8) for i in range(4)]
    assert f.tolist() == pytest.approx([p * (1 - r / 2) for p, r in zip(plain_f, (0, 0.25, 0.5, 0.75))])
    assert mult == pytest.approx(1 + 0.1 * math.log(2.0))


def test_plain_rotation_pairs_neighbours_and_leaves_the_rest():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0, 6.0]]], dtype=F).repeat(2, 1, 1)
    y = plain.rotate(x, torch.tensor([0, 3]), rot(100.0, 4))
    assert torch.equal(y[0], x[0])
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    assert y[1, 0].tolist() == pytest.approx([math.cos(a0), math.sin(a0), -2 * math.sin(a1), 2 * math.cos(a1), 5.0, 6.0])


def test_plain_window_sink_and_cap():
    q = torch.zeros((4, 1, 2), dtype=F)
    k = torch.zeros((4, 1, 2), dtype=F)
    v = torch.tensor([[[1.0]], [[2.0]], [[4.0]], [[8.0]]], dtype=F)
    sink = torch.tensor([math.log(3.0)], dtype=F)
    # every score is 0 and the sink weighs as much as three keys; two keys are seen
    assert plain.attend(q, k, v, 1.0, None, 2, sink)[:, 0, 0].tolist() == pytest.approx([1 / 4, 3 / 5, 6 / 5, 12 / 5])
    assert plain.attend(q, k, v, 1.0, None, None, sink)[3, 0, 0].item() == pytest.approx(15 / 7)
    q[3, 0, 0], k[2, 0, 0] = 1.0, 3.0
    w = math.exp(2.0 * math.tanh(3.0 / 2.0))              # the sink itself is not capped
    assert plain.attend(q, k, v, 1.0, 2.0, 2, sink)[3, 0, 0].item() == pytest.approx((w * 4 + 8) / (w + 1 + 3))


def test_plain_recurrence_decays_the_rows_of_key_channels():
    q = torch.tensor([[[1.0, 2.0]], [[1.0, 1.0]]], dtype=F)
    k = torch.tensor([[[3.0, 5.0]], [[1.0, -1.0]]], dtype=F)
    alpha = torch.tensor([[[0.1, 0.2]], [[0.5, 0.25]]], dtype=F)
    v = torch.tensor([[[4.0]], [[8.0]]], dtype=F)
    o = plain.decayed_recurrence(q, k, v, alpha)[:, 0, 0]
    assert o.tolist() == pytest.approx([12.0 + 40.0, 0.5 * 12 + 8 + 0.25 * 20 - 8])
    assert float(plain.channel_decay(torch.tensor(0.0, dtype=F), 2.0)) == pytest.approx(0.5 ** 0.5)


def test_plain_convolution_puts_the_last_tap_on_the_current_token():
    x = torch.tensor([[1.0], [10.0], [100.0], [1000.0]], dtype=F)
    assert plain.causal_conv(x, torch.tensor([[3.0, 2.0, 1.0]], dtype=F))[:, 0].tolist() == [1.0, 12.0, 123.0, 1230.0]


def test_plain_model_runs_the_loop_with_the_embedding():
    """One looped layer that adds nothing: the stream is the loop's projection applied as often as the loop says."""
    from starter_b200.engine.model import expected_tensors

    cfg = dict(copy.deepcopy(L_C), loop=dict(start=1, stop=2, times=3))
    cfg["layers"] = cfg["layers"][:2]
    torch.manual_seed(0)
    w = {n: torch.randn(tuple(p.shape), dtype=F) * 0.1 for n, p in expected_tensors(spec_of(cfg)).items()}
    for n in ("l0.mix.o", "l1.mix.o", "l0.mlp.down", "l1.mlp.down"):
        w[n] = torch.zeros_like(w[n])
    x0 = w["embed"][[3, 5]]
    x, seen = x0, []
    plain.forward(cfg, w, [3, 5], seen)
    assert len(seen) == 4 and torch.equal(seen[0], x0)
    for got in seen[1:]:
        x = x @ w["loop.in"][:, :128].T + x0 @ w["loop.in"][:, 128:].T
        assert torch.allclose(got, x)
