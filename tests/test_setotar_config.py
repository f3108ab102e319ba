"""Setotar's configuration on the CPU: what config.json means, what is refused, the run order of layers that read
another layer's keys and values, tensor names, rotation tables, and the plain statement on cases whose answer is known."""

import copy
import math

import pytest
import torch

import plain_setotar as plain
from tiny_setotar import S_A, S_B, S_C, TINY_S, rot

F = torch.float64


def spec_of(raw):
    from starter_b200.config import config_from_dict

    return config_from_dict(raw).to_model_spec()


def test_every_size_and_constant_comes_from_the_config():
    spec = spec_of(S_A)
    assert (spec.architecture, spec.vocab_size, spec.hidden_size, spec.streams) == ("Setotar", 200, 64, 2)
    assert not spec.tie_embeddings and spec.lm_head_name == "head" and spec.final_norm.gain_32bit
    first, second, third, fourth, fifth = spec.layers
    m = first.mixer
    assert (m.kind, m.join, m.left_scale, m.right_scale) == ("parallel", "scaled_sum", 0.7, 0.9)
    a, s = m.left, m.right
    assert (a.kind, a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.scale) == ("sink_attention", 4, 2, 16, 24, 0.3)
    assert (a.window, a.keep_first, a.softcap, a.conv, a.bias, a.unit_values, a.norm_eps) == (10, 3, 4.0, 3, True, True, 1e-5)
    assert not (a.row_norm or a.sink or a.head_gate or a.distance_penalty or a.values_from_keys) and a.fixed_sink is None
    assert (a.position.kind, a.position.base, a.position.dims, a.position.scaling.factor) == ("rope_partial", 100.0, 8, 4.0)
    assert (s.kind, s.num_heads, s.head_dim, s.value_dim, s.norm_eps) == ("forget_write", 3, 12, 8, 1e-5)
    ff = first.feed_forward
    assert (ff.experts, ff.top, ff.intermediate_size, ff.expert, ff.scoring, ff.weigh_input, ff.router_bias) == \
        (5, 2, 24, "gated_silu", "sigmoid", True, False)
    b = second.mixer
    assert (b.kind, b.row_norm, b.own_kv, b.window, b.softcap, b.conv, b.bias, b.unit_values) == \
        ("sink_attention", True, True, None, None, None, False, False)
    y = b.position.scaling
    assert (y.factor, y.original, y.fast, y.slow) == (8.0, 64.0, 4.0, 0.5)
    assert second.arrangement == "hyper_mixer_only" and "feed_forward" not in second.parts
    assert not third.mixer.own_kv and third.mixer.num_heads == 6 and third.mixer.position == b.position
    assert (fourth.mixer.left.window, fourth.mixer.left.keep_first, fourth.mixer.left.softcap, fourth.mixer.left.conv) == (None, 0, None, 1)
    assert fourth.mixer.left.position.scaling is None and fifth.arrangement == "hyper_prenorm"
    assert all(layer.connection1.streams == 2 and layer.connection1.channel_scale == 64 for layer in spec.layers)
    assert spec_of(S_B).layers[0].mixer.position is None and spec_of(S_B).layers[1].mixer.left.conv is None


def test_run_order_of_layers_that_read_another_layers_keys_and_values():
    order = spec_of(S_A).schedule
    assert [(e.layer, e.cache, e.writes_cache) for e in order] == \
        [(0, 0, True), (1, 1, True), (2, 1, False), (3, 3, True), (4, 1, False)]


def test_cache_and_state_needs():
    """A reading layer asks for nothing; both halves of a parallel mixer share one slot of floats."""
    from starter_b200.engine.model import build_layers

    blocks, positions = build_layers(spec_of(S_A), torch.float32, "cpu")
    assert len(positions) == 3                         # equal rotations share their tables
    kv = [b.mixer.kv_need() for b in blocks]
    assert (kv[0].num_kv_heads, kv[0].head_dim, kv[0].value_size, kv[0].window) == (2, 16, 24, 10)
    assert (kv[1].head_dim, kv[1].value_size, kv[1].window) == (16, 8, None) and kv[2] is None and kv[4] is None
    conv = 2 * (4 * 16 + 2 * 16 + 2 * 24)
    assert blocks[0].mixer.state_need().shape == (conv + 3 * 12 * 8,)
    assert blocks[0].mixer.sides["left"].state_at == 0 and blocks[0].mixer.sides["right"].state_at == conv
    assert blocks[1].mixer.state_need() is None
    assert blocks[3].mixer.state_need().shape == (20 * 24,)       # one tap keeps nothing


def test_tensor_names():
    from starter_b200.engine.model import expected_tensors

    spec = spec_of(S_A)
    names = expected_tensors(spec)
    for name, shape in {"embed": (200, 64), "head": (200, 64), "final.norm": (64,), "l0.mix.left.q": (64, 64),
                        "l0.mix.left.k.b": (32,), "l0.mix.left.v.conv": (48, 3), "l0.mix.left.o": (64, 96),
                        "l0.mix.right.f": (36, 64), "l0.mix.right.f.b": (36,), "l0.mix.right.lower": (36,),
                        "l0.mix.right.norm": (8,), "l0.mix.right.o": (64, 24), "l0.ls1": (64,), "l0.ls2": (64,),
                        "l0.hc1.in": (2,), "l0.hc2.mix": (2, 2), "l0.mlp.router": (5, 64), "l0.mlp.e4.down": (64, 24),
                        "l1.mix.q.norm": (64,), "l1.mix.k.norm": (32,), "l2.mix.q.norm": (96,), "l2.mix.o": (64, 48),
                        "l3.mix.left.q.conv": (16, 1)}.items():
        assert tuple(names[name].shape) == shape, name
    for name in ("l2.mix.k", "l2.mix.v", "l2.mix.k.norm", "l1.norm2", "l1.ls2", "l1.hc2.in", "l1.mlp.router"):
        assert name not in names, name
    # what a layer without a feed-forward may still store is not read and not missed
    assert set(spec.ignored_tensors) == {f"l{i}.{n}" for i in (1, 3) for n in ("norm2", "ls2", "hc2.in", "hc2.out", "hc2.mix")}
    assert "l1.mix.left.q.conv" not in expected_tensors(spec_of(S_B))


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="lstm"), "mixers"),
    (lambda c: c["layers"][0]["mixer"].update(extra=1), "extra"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "key/value heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "positive"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), "count"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=0.0), "positive"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(state=4), "state"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "feed-forward"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "attention layer"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "of its own"),
    (lambda c: c["layers"][4]["mixer"].update(vdim=16), "vdim"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.update(window=3), "window"),
])
def test_what_is_refused(change, text):
    from starter_b200.config import ConfigError, config_from_dict

    raw = copy.deepcopy(S_A)
    change(raw)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(raw)


def test_config_round_trip():
    from starter_b200.config import config_from_dict

    for raw in TINY_S.values():
        cfg = config_from_dict(raw)
        assert config_from_dict(cfg.to_dict()) == cfg


@pytest.mark.parametrize("turn", [rot(100.0, 8), rot(30000.0, 64, 3.0), rot(10000.0, 24, 5.0, 640, 24.0, 1.5), rot(1e6, 128, 8.0, 64, 4.0, 0.5),
                                  rot(500.0, 12, 1.0, 100, 8.0, 8.0), rot(10000.0, 2, 3.0, 32, 32.0, 1.0)])
def test_rotation_tables(turn):
    """The library's tables against the plain frequencies, far out too; growing them keeps what was there."""
    from starter_b200.config.setotar import _position
    from starter_b200.parts.rotary import PartialRotaryTable

    table = PartialRotaryTable(_position(turn), torch.float32, "cpu")
    assert table.ensure(10) and not table.ensure(4096)
    before = table.cos.clone()
    assert table.ensure(5000)
    assert torch.equal(table.cos[:4096], before) and table.rotation().rotary_dim == turn["dims"]
    f, mult = plain.frequencies(turn)
    pos = torch.arange(table.length, dtype=F)
    for got, want in ((table.cos, (pos[:, None] * f).cos() * mult), (table.sin, (pos[:, None] * f).sin() * mult)):
        assert float((got.double() - want).abs().max()) < 2e-7 * mult


# ------------------------------------------------------------------------------ the plain statement, by hand

def test_plain_frequencies_stretch_by_parts():
    f, mult = plain.frequencies(rot(100.0, 4, 8.0))
    assert f.tolist() == pytest.approx([1 / 8, 0.1 / 8]) and mult == 1.0
    # d(t) = 8 ln(40 pi / (2 pi t)) / (2 ln 10): 20 turns at 0, 2 turns at 4: lo 0, hi 4, ramps 0, 1/4, 2/4, 3/4
    f, mult = plain.frequencies(rot(10.0, 8, 2.0, 40.0 * math.pi, 20.0, 2.0))
    plain_f = [10.0 ** (-2 * i / 8) for i in range(4)]
    assert f.tolist() == pytest.approx([p * (1 - r / 2) for p, r in zip(plain_f, (0, 0.25, 0.5, 0.75))])
    assert mult == pytest.approx(1 + 0.1 * math.log(2.0))


def test_plain_rotation_pairs_the_halves_and_leaves_the_rest():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0, 6.0]]], dtype=F).repeat(2, 1, 1)
    y = plain.rotate(x, torch.tensor([0, 3]), rot(100.0, 4))
    assert torch.equal(y[0], x[0])
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    assert y[1, 0].tolist() == pytest.approx([math.cos(a0), -2 * math.sin(a1), math.sin(a0), 2 * math.cos(a1), 5.0, 6.0])


def test_plain_window_keeps_the_first_keys_and_caps_scores():
    q = torch.zeros((5, 1, 2), dtype=F)
    k = torch.zeros((5, 1, 2), dtype=F)
    v = torch.tensor([[[1.0]], [[2.0]], [[4.0]], [[8.0]], [[16.0]]], dtype=F)
    out = plain.attend(q, k, v, 1.0, None, 2, 1)
    # every score is 0: the mean of what is seen; the first key stays when it has left the window of two
    assert out[:, 0, 0].tolist() == pytest.approx([1.0, 3 / 2, 7 / 3, 13 / 3, 25 / 3])
    q[4, 0, 0], k[0, 0, 0] = 1.0, 3.0
    w = math.exp(2.0 * math.tanh(3.0 / 2.0))
    assert float(plain.attend(q, k, v, 1.0, 2.0, 2, 1)[4, 0, 0]) == pytest.approx((w * 1 + 8 + 16) / (w + 2))
    assert float(plain.attend(q, k, v, 1.0, 2.0, 2, 0)[4, 0, 0]) == pytest.approx(12.0)


def test_plain_recurrence_forgets_and_writes_by_one_gate():
    q = torch.tensor([[[1.0, 2.0]], [[1.0, 1.0]]], dtype=F)
    f = torch.tensor([[[0.5, 0.9]], [[0.25, 1.0]]], dtype=F)
    v = torch.tensor([[[4.0]], [[8.0]]], dtype=F)
    o = plain.forget_recurrence(q, f, v)[:, 0, 0]
    s = (0.5 * 4, 0.1 * 4)
    assert o.tolist() == pytest.approx([s[0] + 2 * s[1], 0.25 * s[0] + 0.75 * 8 + s[1]])


def test_plain_convolution_puts_the_last_tap_on_the_current_token():
    x = torch.tensor([[1.0], [10.0], [100.0], [1000.0]], dtype=F)
    assert plain.causal_conv(x, torch.tensor([[3.0, 2.0, 1.0]], dtype=F))[:, 0].tolist() == [1.0, 12.0, 123.0, 1230.0]


def test_plain_experts_take_the_weighted_input():
    w = {"m.router": torch.tensor([[1.0], [3.0], [2.0]], dtype=F)}
    for e in range(3):
        w.update({f"m.e{e}.gate": torch.tensor([[1.0]], dtype=F), f"m.e{e}.up": torch.tensor([[10.0 ** e]], dtype=F),
                  f"m.e{e}.down": torch.tensor([[1.0]], dtype=F)})
    h = torch.tensor([[0.5]], dtype=F)
    out = plain.routed_feed_forward(h, w, "m.", dict(router=dict(top=2)))
    want = 0.0
    for e, z in ((1, 1.5), (2, 1.0)):
        x = 0.5 / (1 + math.exp(-z))
        want += x / (1 + math.exp(-x)) * 10.0 ** e * x
    assert float(out) == pytest.approx(want)


def test_plain_streams_are_written_from_the_old_ones():
    xs = torch.tensor([[[1.0]], [[10.0]]], dtype=F)
    w = {"h.in": torch.tensor([2.0, 1.0], dtype=F), "h.out": torch.tensor([1.0, -1.0], dtype=F),
         "h.mix": torch.tensor([[0.5, 3.0], [0.25, 0.0]], dtype=F)}
    new = plain.through_streams(xs, w, "h.", lambda u: u * 100.0)
    assert new[:, 0, 0].tolist() == pytest.approx([0.5 + 2.5 + 1200.0, 3.0 - 1200.0])


def test_a_reading_layer_uses_the_other_layers_keys():
    """Changing the source layer's key projection moves the reading layer; its own has none."""
    from starter_b200.engine.model import expected_tensors

    torch.manual_seed(0)
    cfg = copy.deepcopy(S_C)
    cfg["layers"] = [cfg["layers"][0], cfg["layers"][2]]
    w = {n: torch.randn(tuple(p.shape), dtype=F) * 0.3 for n, p in expected_tensors(spec_of(cfg)).items()}
    base, moved, other = [], [], dict(w)
    other["l0.mix.o"] = torch.zeros_like(w["l0.mix.o"])           # layer 0 itself no longer shows what it attends to
    plain.forward(cfg, other, [1, 2, 3, 4], base)
    other["l0.mix.v"] = w["l0.mix.v"] * 2.0
    plain.forward(cfg, other, [1, 2, 3, 4], moved)
    assert torch.equal(base[0], moved[0]) and not torch.allclose(base[1], moved[1])
