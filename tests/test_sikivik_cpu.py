"""Sikivik without a GPU: configuration, tensor plan, registry, and the oracle's mechanisms against closed forms."""
import json

import numpy as np
import pytest

import sikivik_cases as cases
from oracle import sikivik as ref
from zeninfer_b200 import blocks, registry
from zeninfer_b200.sikivik import AttentionConfig, Rotation, SikivikConfig, StateConfig, projection_rows, rotation_tables, tensor_plan


# ---- configuration and files ----
def test_config_reads_every_size():
    c, cfg, _, _ = cases.model("ragged")
    assert (cfg.width, cfg.vocab, cfg.eps) == (90, 203, 1e-5)
    a, r, b, g, last = (layer.mixer for layer in cfg.layers)
    assert isinstance(a, AttentionConfig) and (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.conv, a.rot, a.v_mix) == (6, 3, 40, 24, 17, 4, Rotation(5e3, 22), False)
    assert a.scale == 1.3 * 40 ** -0.5 and a.pitch == 64
    assert isinstance(r, StateConfig) and (r.heads, r.dim, r.vdim, r.decay, r.rot, r.tau) == (3, 20, 28, (0.9, 0.99, 0.999), Rotation(500.0, 12), None)
    assert (g.heads, g.dim, g.vdim, g.tau, g.decay, g.rot) == (2, 33, 18, 8.0, None, None) and b.v_mix and last.conv == 1
    assert [layer.ff for layer in cfg.layers] == [None, 123, 61, None, 75] and cfg.first_values() == 2
    assert [n for n, _ in projection_rows(g, 10)] == ["q", "k", "v", "g", "a1"] and [n for n, _ in projection_rows(r, 10)] == ["q", "k", "v", "g"]


def test_first_values_without_mixing_layers():
    c, _ = cases.CASES["ragged"]
    c = json.loads(json.dumps(c))
    for layer in c["layers"]:
        layer["mixer"].pop("v_mix", None)
    assert SikivikConfig.from_dict(c).first_values() is None


def test_config_refuses_what_it_does_not_know():
    c, _ = cases.CASES["ragged"]
    changes = (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][1]["mlp"].update(kind="experts"), lambda d: d["layers"][0]["mixer"].update(kv_heads=4),
               lambda d: d["layers"][1]["mixer"].update(decay=[0.9]), lambda d: d["layers"][1]["mixer"]["rot"].update(dims=22), lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7),
               lambda d: d["layers"][4]["mixer"].update(vdim=28))
    for change in changes:
        bad = json.loads(json.dumps(c))
        change(bad)
        with pytest.raises(ValueError):
            SikivikConfig.from_dict(bad)


def test_bf16_keeps_shapes():
    for shape in ((), (3,), (2, 5)):
        w = np.full(shape, 0.5, np.float32)
        assert blocks.to_bf16(w).shape == shape and np.array_equal(blocks.from_bf16(blocks.to_bf16(w)), w)


def test_registry_chooses_by_config(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Sikivik"}))
    assert registry.architecture_of(str(tmp_path)) == "Sikivik"


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_plan_covers_the_oracle(name):
    # the oracle runs on the tensors the plan lists: none missing; the first mixing layer's share is the only one that changes nothing
    c, cfg, bits, weights = cases.model(name)
    assert set(bits) == {n for n, _ in tensor_plan(cfg, cases.CASES[name][1])}
    ids = cases.tokens_for(c, 4)
    base, _ = ref.forward(c, weights, ids)
    unused = set()
    for n in bits:
        try:
            moved, _ = ref.forward(c, {**weights, n: weights[n] + np.float32(0.5)}, ids)
            if np.array_equal(moved, base):
                unused.add(n)
            less = {k: t for k, t in weights.items() if k != n}
            if n not in unused:
                with pytest.raises(KeyError):
                    ref.forward(c, less, ids)
        except KeyError as e:
            pytest.fail(f"{n}: {e}")
    first = cfg.first_values()
    alone = {n for n in bits for i, layer in enumerate(cfg.layers) if getattr(layer.mixer, "window", 0) == 1 and n.startswith((f"l{i}.mix.q", f"l{i}.mix.k"))}
    assert unused == ({f"l{first}.mix.vmix"} if first is not None else set()) | alone          # a window of one key has nothing to weigh


def test_rotation_tables():
    cos, sin = rotation_tables(Rotation(100.0, 6), 5)
    assert cos.shape == sin.shape == (5, 3) and cos.dtype == np.float32
    assert np.allclose(cos[4], np.cos(4 * 100.0 ** (-np.arange(3) / 3)), atol=1e-7) and np.allclose(sin[2], np.sin(2 * 100.0 ** (-np.arange(3) / 3)), atol=1e-7)
    assert rotation_tables(Rotation(10.0, 0), 5)[0].shape == (5, 0)


# ---- the oracle's mechanisms against other forms of the same equations ----
def test_oracle_decayed_write_is_a_weighted_sum():
    rng = np.random.default_rng(1)
    q, k, g, v = rng.standard_normal((6, 2, 3)), rng.standard_normal((6, 2, 3)), rng.uniform(0.3, 1.0, (6, 2, 3)), rng.standard_normal((6, 2, 4))
    o = ref.decayed_write(q, k, v, g)
    for h in range(2):
        for t in range(6):
            want = sum((q[t, h] * k[s, h] * np.prod(g[s + 1:t + 1, h], axis=0)).sum() * v[s, h] for s in range(t + 1))
            assert np.allclose(o[t, h], want)


def test_oracle_channel_decay():
    z = np.array([-30.0, -1.0, 0.0, 2.0, 40.0])
    assert np.allclose(ref.channel_decay(z, 4.0), (1 / (1 + np.exp(-z))) ** 0.25)
    assert np.allclose(ref.channel_decay(z, 1.0), 1 / (1 + np.exp(-z)))


def test_oracle_rotation_depends_on_distance_only():
    rng = np.random.default_rng(2)
    a, b = rng.standard_normal(10), rng.standard_normal(10)
    x = np.tile(np.stack([a, b])[None], (9, 1, 1))
    r = ref.rotate_half(x, 6, 50.0)
    assert np.allclose(r[0], x[0]) and np.allclose(r[:, :, 6:], x[:, :, 6:])
    assert np.isclose(r[7, 0] @ r[4, 1], r[3, 0] @ r[0, 1]) and not np.isclose(r[7, 0] @ r[4, 1], r[7, 0] @ r[5, 1])
    # the pair (0, half) turns by one radian per token
    assert np.isclose(r[1, 0, 0], a[0] * np.cos(1.0) - a[3] * np.sin(1.0)) and np.isclose(r[1, 0, 3], a[3] * np.cos(1.0) + a[0] * np.sin(1.0))
    back = cases.undo_rotation(r, 6, 50.0)
    assert np.allclose(back, x)


def test_undone_convolution():
    rng = np.random.default_rng(3)
    w, x = cases.short_taps(5, 4, rng).astype(np.float64), rng.standard_normal((20, 5))
    assert np.allclose(ref.causal_conv(cases.undo_conv(x, w), w), x)


@pytest.mark.parametrize("size,off", [(16, 1), (16, -1), (40, 1), (2, -1)])
def test_planted_keys_show_a_window_that_is_one_off(size, off):
    # what the GPU tests rely on: with the planted keys a window one position too long or short changes outputs by far more than the
    # tolerance used there
    T, m = 90, dict(heads=4, kv_heads=2, dim=24, vdim=20, conv=3, rot=dict(base=100.0, dims=10), scale=20.0 / 24, mask=dict(size=size))
    proj, taps = cases.standout_projections(T, m, [30, 50], 5)
    rows = [("q", 96), ("k", 48), ("v", 40), ("g", 80)]
    w = {**cases.selectors(rows), **{f"{n}.b": 0.0 for n in "qkvo"}, **{f"{n}.conv": t for n, t in zip("qkv", taps)}, "o": np.eye(80)}
    good, _ = ref.attention(proj.astype(np.float64), w, m, None)
    bad, _ = ref.attention(proj.astype(np.float64), w, {**m, "mask": dict(size=size + off)}, None)
    assert np.abs(good - bad).max() > 0.5


def test_faults_show_in_the_logits():
    # a lost state, a convolution that forgets, a window one off, values that are not mixed: each far above the tolerances of the GPU tests
    c, _, _, weights = cases.model("ragged")
    ids = cases.tokens_for(c, 60)
    whole, _ = ref.forward(c, weights, ids)
    lost, _ = ref.forward(c, weights, ids[20:])
    assert cases.logit_error(lost, whole[20:]) > 0.05
    for i, change in ((0, dict(mask=dict(size=16))), (2, dict(mask=dict(size=10))), (4, dict(mask=dict(size=39))), (4, dict(v_mix=False)), (0, dict(rot=dict(base=5e3, dims=20)))):
        other = json.loads(json.dumps(c))
        other["layers"][i]["mixer"].update(change)
        assert cases.logit_error(ref.forward(other, weights, ids)[0], whole) > 2e-3, (i, change)
    gone = {**weights, "l0.mix.k.conv": weights["l0.mix.k.conv"] * np.array([0, 1, 1, 1])}
    assert cases.logit_error(ref.forward(c, gone, ids)[0], whole) > 2e-3
