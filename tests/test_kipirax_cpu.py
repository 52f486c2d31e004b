"""Kipirax without a GPU: configuration, files, registry, trace replay, and the oracle's mechanisms against closed forms."""
import io
import json

import numpy as np
import pytest

import kipirax_cases as cases
from oracle import kipirax as ref
from zeninfer_b200 import blocks, registry, safetensors, trace
from zeninfer_b200.decoder import Decoder
from zeninfer_b200.kipirax import DeltaConfig, KipiraxConfig, ParallelConfig, tensor_plan


# ---- configuration and files ----
def test_config_reads_every_size():
    c, cfg, _, _ = cases.model("ragged")
    assert (cfg.width, cfg.vocab, cfg.groups, cfg.eps, cfg.logit_softcap, cfg.max_positions) == (90, 203, 3, 1e-5, 20.0, 640)
    first, second = cfg.layers[0].mixer, cfg.layers[1].mixer
    assert isinstance(first, DeltaConfig) and (first.heads, first.kv_heads, first.dim, first.vdim, first.conv) == (4, 2, 20, 28, 3)
    assert isinstance(second, ParallelConfig) and (second.left.window, second.left.keep_first, second.left.scale) == (17, 3, 0.21)
    assert (second.right.heads, second.right.dim, second.right.vdim) == (3, 12, 37) and second.left.pitch == 64
    assert [layer.ff for layer in cfg.layers] == [122, None, None, 75]


def test_config_refuses_what_it_does_not_know():
    c, _, _, _ = cases.model("ragged")
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="experts"), lambda d: d["norm"].update(groups=4),
                   lambda d: d["layers"][0]["mixer"].update(kv_heads=3)):
        bad = json.loads(json.dumps(c))
        change(bad)
        with pytest.raises(ValueError):
            KipiraxConfig.from_dict(bad)


def test_bf16_round_trip():
    w = np.array([1.0, -2.5, 3.14159, 1e-8, 0.0, 65504.0], np.float32)
    import torch
    assert np.array_equal(blocks.to_bf16(w), torch.from_numpy(w).to(torch.bfloat16).view(torch.int16).numpy().view(np.uint16))
    bits = np.arange(0, 0x7F80, 7, dtype=np.uint16)
    assert np.array_equal(blocks.to_bf16(blocks.from_bf16(bits)), bits)


def test_safetensors_round_trip(tmp_path):
    rng = np.random.default_rng(0)
    tensors = {"a": blocks.to_bf16(rng.standard_normal((3, 5), dtype=np.float32)), "b": rng.standard_normal(7).astype(np.float32), "t": np.arange(6, dtype=np.int32)}
    path = str(tmp_path / "m.safetensors")
    safetensors.write(path, tensors)
    with safetensors.SafetensorsFile(path) as f:
        assert set(f.tensors) == set(tensors) and f.dtype("a") == "BF16" and f.shape("a") == (3, 5)
        for n, a in tensors.items():
            assert np.array_equal(f.array(n), a)
        with pytest.raises(safetensors.SafetensorsError):
            f.array("missing")
    raw = open(path, "rb").read()
    open(path, "wb").write(raw[:-4])      # data cut short
    with pytest.raises(safetensors.SafetensorsError):
        safetensors.SafetensorsFile(path)
    open(path, "wb").write(b"\x00")
    with pytest.raises(safetensors.SafetensorsError):
        safetensors.SafetensorsFile(path)


def test_registry_chooses_by_config(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Kipirax"}))
    assert registry.architecture_of(str(tmp_path)) == "Kipirax"
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "unheard-of"}))
    with pytest.raises(registry.UnknownModel):
        registry.architecture_of(str(tmp_path))
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(None, str(tmp_path), dtype="float16")


def test_plan_covers_the_oracle():
    # the oracle runs on exactly the tensors the plan lists: none missing, none unused
    c, cfg, bits, weights = cases.model("ragged")
    used = set()

    class Watch(dict):
        def items(self):
            for n, t in super().items():
                used.add(n)
                yield n, t
    ref.forward(c, Watch(weights), cases.tokens_for(c, 3))
    assert used == {n for n, _ in tensor_plan(cfg, 10, 7)} == set(bits)
    for name in bits:
        less = {n: t for n, t in weights.items() if n != name}
        with pytest.raises(KeyError):
            ref.forward(c, less, cases.tokens_for(c, 3))


# ---- trace replay on a decoder that only counts ----
class Counting(Decoder):
    vocab = 4

    def __init__(self):
        self.seen, self.resets = [], 0

    def reset(self):
        self.seen, self.resets = [], self.resets + 1

    def feed(self, tokens, want=()):
        base = len(self.seen)
        self.seen += tokens
        return np.array([[sum(self.seen[:base + w + 1]), w, base, 0] for w in want], np.float32).reshape(len(want), 4)


def test_replay_keeps_one_request_at_a_time(monkeypatch, tmp_path, capsys):
    r = trace.Replay(Counting())
    assert r.step([{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}], []).tolist() == [[6, 2, 0, 0], [1, 0, 0, 0]]
    with pytest.raises(ValueError):
        r.step([{"id": "b", "tokens": [1], "want": []}], [])
    assert r.step([{"id": "a", "tokens": [5], "want": [0]}], ["a"]).tolist() == [[11, 0, 3, 0]]
    assert r.step([{"id": "b", "tokens": [7], "want": [0]}], ["b"]).tolist() == [[7, 0, 0, 0]]       # nothing of `a` is left
    # the command: answers, files and order
    dec = Counting()
    dec.close = lambda: None
    monkeypatch.setattr("zeninfer_b200.build.build", lambda: "")
    monkeypatch.setattr("zeninfer_b200.backend.Backend", lambda: None)
    monkeypatch.setattr("zeninfer_b200.registry.load_model", lambda *a: dec)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": [4, 4], "want": []}], "end": []}, {"step": 1, "entries": [{"id": "x", "tokens": [1], "want": [0]}], "end": ["x"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace.main(["--model", "m", "--dtype", "bfloat16", "--out", str(tmp_path), "--max-tokens", "8"]) == 0
    assert capsys.readouterr().out.split("\n")[:2] == ["done 0", "done 1"]
    assert not (tmp_path / "0.f32").exists() and np.fromfile(tmp_path / "1.f32", "<f4").tolist() == [9, 0, 2, 0]

    def refuse(*a):
        raise registry.UnsupportedDtype("no")
    monkeypatch.setattr("zeninfer_b200.registry.load_model", refuse)
    assert trace.main(["--model", "m", "--dtype", "float32", "--out", str(tmp_path)]) == 3


# ---- the oracle's mechanisms against other forms of the same equations ----
def test_oracle_delta_rule_writes_and_reads():
    # unit decay, beta 1, orthonormal keys: the state recalls every value written, and a repeated key replaces its value
    D, V = 4, 3
    k = np.eye(D)[[0, 1, 2, 1]][:, None]
    v = np.random.default_rng(0).standard_normal((4, 1, V))
    one = np.ones((4, 1, D))
    o = ref.delta_rule(k, k, v, one, np.ones((4, 1)))
    assert np.allclose(o, v)                                     # the read-out sees the current token's write
    o = ref.delta_rule(np.repeat(np.eye(D)[1][None, None], 4, 0), k, v, one, np.ones((4, 1)))
    assert np.allclose(o[:, 0], [np.zeros(V), v[1, 0], v[1, 0], v[3, 0]])
    decayed = ref.delta_rule(np.repeat(np.eye(D)[0][None, None], 4, 0), k, v, 0.5 * one, np.ones((4, 1)))
    assert np.allclose(decayed[:, 0], v[0, 0] * 0.5 ** np.arange(4)[:, None])


def test_oracle_gated_write_is_a_running_average():
    f = np.random.default_rng(1).uniform(0.2, 0.9, (5, 1, 2))
    v = np.random.default_rng(2).standard_normal((5, 1, 3))
    q = np.ones((5, 1, 2))
    want = [sum((1 - f[s, 0, d]) * np.prod(f[s + 1:t + 1, 0, d]) * v[s, 0] for s in range(t + 1) for d in range(2)) for t in range(5)]
    assert np.allclose(ref.gated_write(q, f, v)[:, 0], want)


def test_oracle_convolution_and_shift():
    x = np.arange(1.0, 6.0)[:, None]
    assert np.allclose(ref.causal_conv(x, np.array([[100.0, 10.0, 1.0]]))[:, 0], [1, 12, 123, 234, 345])
    assert np.allclose(ref.token_shift(x, np.array([0.25]))[:, 0], [0.75, 1.75, 2.75, 3.75, 4.75])


def test_oracle_grouped_norm():
    x = np.array([3.0, 4.0, 0.5, -0.5])
    assert np.allclose(ref.grouped_rms_norm(x, np.array([1.0, 1.0, 2.0, 1.0]), 2, 0.0), [3 / np.sqrt(12.5), 4 / np.sqrt(12.5), 2.0, -1.0])


@pytest.mark.parametrize("size,keep,off", [(16, 3, (1, 0)), (16, 3, (-1, 0)), (16, 3, (0, 1)), (16, 3, (0, -1)), (16, 0, (1, 0)), (40, 35, (0, -1))])
def test_planted_keys_show_a_mask_that_is_one_off(size, keep, off):
    # what the GPU tests rely on: with the planted keys a window or a kept token too many or too few changes outputs by far more
    # than the tolerance used there
    T = 120
    planted = [j for j in (keep - 1, keep, 50) if 0 <= j < T]
    q, k, v, qw, kw = cases.standout_attention(T, 4, 2, 24, 20, planted, 5)
    qn, kn = ref.rms(q.astype(np.float64), 1e-6) * qw, ref.rms(k.astype(np.float64), 1e-6) * kw
    good = ref.window_attention(qn, kn, v, 2.0, size, keep)
    bad = ref.window_attention(qn, kn, v, 2.0, size + off[0], keep + off[1])
    assert np.abs(good - bad).max() > 0.5


def test_far_and_first_tokens_show_in_the_logits():
    # a state that is lost between two portions changes what comes after it
    c, _, _, weights = cases.model("ragged")
    ids = cases.tokens_for(c, 40)
    whole, _ = ref.forward(c, weights, ids)
    lost, _ = ref.forward(c, weights, ids[20:])
    assert cases.logit_error(lost, whole[20:]) > 0.05
