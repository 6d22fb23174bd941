"""CPU checks around the block models: the plain statement agrees with itself however a sequence is cut, model folders
are read and refused with a reason before any device is touched, and sessions keep their slots."""
import copy
import json

import numpy as np
import pytest

import block_models as bm
import plain_blocks as pb


@pytest.mark.parametrize("name", list(bm.CONFIGS))
def test_plain_model_does_not_depend_on_cuts(name):
    cfg, t = bm.make(bm.CONFIGS[name])
    toks = bm.tokens(cfg, 60)
    whole = pb.PlainModel(cfg, t).run(toks)
    m = pb.PlainModel(cfg, t)
    parts, at = [], 0
    for n in bm.cuts_of(60, 1, 2, 17):
        parts.append(m.run(toks[at:at + n]))
        at += n
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-9


def test_layer_runs():
    lay = [{}] * 5
    assert pb.layer_runs({"layers": lay}) == [0, 1, 2, 3, 4]
    assert pb.layer_runs({"layers": lay, "loop": {"start": 1, "stop": 3, "times": 3}}) == [0, 1, 2, 1, 2, 1, 2, 3, 4]


def test_rotation_scaling_leaves_fast_pairs_and_divides_slow_ones():
    rot = {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    f, amp = pb.rotary_frequencies(rot)
    g, _ = pb.rotary_frequencies({"base": 10000.0, "dims": 64})
    assert np.allclose(f[:5], g[:5]) and np.allclose(f[-1], g[-1] / 4) and np.isclose(amp, 1 + 0.1 * np.log(4.0))


def test_chunked_mask_and_sink_of_the_plain_model():
    assert [pb.seen_keys(p, {"size": 3}) for p in range(7)] == [0, 0, 0, 3, 3, 3, 6]
    w = pb.sink_weights(np.array([[0.0, 0.0, 0.0], [50.0, 0.0, 0.0], [-50.0, -50.0, -50.0]]))
    assert np.allclose(w[0], 0.25) and np.allclose(w[1], [1, 0, 0]) and w[2].sum() < 1e-20


def test_recurrence_of_the_plain_model_keeps_its_variance():
    """a^2 + (sqrt(1 - a^2))^2 = 1: white noise through an open input gate keeps unit variance."""
    rng = np.random.default_rng(0)
    u = rng.standard_normal((4000, 50))
    out, _ = pb.gated_recurrence(u, np.full_like(u, 0.5), np.ones_like(u), rng.normal(-3, 1, 50), np.zeros(50))
    assert 0.8 < out[500:].var() < 1.2


def refused(pkg, tmp_path, match, change=None, tensors=None, name="odd"):
    cfg, t = bm.make(bm.CONFIGS[name])
    cfg = copy.deepcopy(cfg)
    if change:
        change(cfg)
    if tensors:
        tensors(t)
    folder = pb.write_model(tmp_path / "m", cfg, t)
    with pytest.raises(pkg.B200Error, match=match):
        pkg.Engine.from_model(folder)


def test_model_folder_is_read_and_stops_at_the_missing_gpu(pkg, tmp_path):
    if pkg.api.device_count() > 0:
        pytest.skip("a GPU is present")
    for name in bm.CONFIGS:
        refused(pkg, tmp_path, "no CUDA device", name=name)


def test_model_folder_errors(pkg, tmp_path):
    def setter(*path, value):
        def f(c):
            for p in path[:-1]:
                c = c[p]
            c[path[-1]] = value
        return f

    refused(pkg, tmp_path, "unknown architecture 'Other'", setter("architecture", value="Other"))
    refused(pkg, tmp_path, "unknown architecture 'llama'", setter("architecture", value="llama"))
    refused(pkg, tmp_path, "unknown mixer 'conv'", setter("layers", 0, "type", value="conv"))
    refused(pkg, tmp_path, "unknown feed-forward 'moe'", setter("layers", 0, "mlp", "kind", value="moe"))
    refused(pkg, tmp_path, "'loop' lies outside", setter("loop", "stop", value=9))
    refused(pkg, tmp_path, "missing field 'width'", lambda c: c.pop("width"))
    refused(pkg, tmp_path, "'heads' must be positive", setter("layers", 0, "mixer", "heads", value=0))
    refused(pkg, tmp_path, "not an integer", setter("vocab", value=10.5))
    refused(pkg, tmp_path, "l2.mix.uv has an unexpected shape", setter("layers", 2, "mixer", "vdim", value=10))
    refused(pkg, tmp_path, "l0.mix.dq.norm is missing", tensors=lambda t: t.pop("l0.mix.dq.norm"))
    refused(pkg, tmp_path, "w1 is missing", tensors=lambda t: t.pop("l1.mix.w1"))
    def piz(match, change=None, tensors=None):
        refused(pkg, tmp_path, match, change, tensors, name="piz_odd")

    piz("unknown mixer 'wkv'", setter("layers", 1, "type", value="wkv"))
    piz("heads must be a multiple of kv_heads", setter("layers", 0, "mixer", "kv_heads", value=4))
    piz("vdim must equal dim", setter("layers", 0, "mixer", "vdim", value=10))
    piz("rot.dims exceeds dim", setter("layers", 0, "mixer", "rot", "dims", value=22))
    piz("rot.dims must be even", setter("layers", 0, "mixer", "rot", "dims", value=5))
    piz("width must be a multiple of blocks", setter("layers", 1, "mixer", "blocks", value=5))
    piz("missing field 'scale'", lambda c: c["layers"][0]["mixer"].pop("scale"))
    piz("l1.mix.conv has an unexpected shape", setter("layers", 1, "mixer", "conv", value=4))
    piz("l3.mix.ri.b is missing", tensors=lambda t: t.pop("l3.mix.ri.b"))
    with pytest.raises(pkg.B200Error, match="cannot open"):
        pkg.Engine.from_model(str(tmp_path / "nowhere"))
    (tmp_path / "m" / "config.json").write_text('{"architecture": "Nezolix", "layers": [}')
    with pytest.raises(pkg.B200Error, match="malformed JSON"):
        pkg.Engine.from_model(str(tmp_path / "m"))


def test_damaged_weights_file(pkg, tmp_path):
    cfg, t = bm.make(bm.CONFIGS["odd"])
    folder = pb.write_model(tmp_path / "m", cfg, t)
    raw = (tmp_path / "m" / "model.safetensors").read_bytes()
    for bad, why in ((raw[:6], "not a safetensors file"), (raw[:5000], "header longer|does not match|malformed"), (raw[:-10], "does not match its shape")):
        (tmp_path / "m" / "model.safetensors").write_bytes(bad)
        with pytest.raises(pkg.B200Error, match=why):
            pkg.Engine.from_model(folder)


class FakeEngine:
    """Records calls; logits carry (slot, position, token)."""
    vocab = 3

    def __init__(self, n):
        self.desc = type("D", (), {"max_seqs": n})
        self.calls = []

    def decode(self, toks, pos, slots, want_logits, want_argmax):
        self.calls.append(("decode", slots[0], pos[0], list(toks)))
        return np.array([[slots[0], pos[0], toks[0]]], np.float32), None

    def prefill_rows(self, toks, want, slot, start_pos):
        self.calls.append(("prefill", slot, start_pos, list(toks)))
        return np.array([[slot, start_pos + w, toks[w]] for w in want], np.float32).reshape(len(want), 3)

    def kv_reset(self, slot):
        self.calls.append(("reset", slot))


def test_sessions_keep_slots_and_positions(pkg):
    e = FakeEngine(2)
    s = pkg.Sessions(e)
    assert s.feed("a", [7, 8, 9], [2, 0]).tolist() == [[0, 2, 9], [0, 0, 7]]
    assert s.feed("a", [4], [0]).tolist() == [[0, 3, 4]]
    assert s.feed("b", [5]).shape == (0, 3)
    with pytest.raises(RuntimeError):
        s.feed("c", [1])
    s.end("a")
    assert s.feed("c", [1, 2], [1]).tolist() == [[0, 1, 2]]
    assert [c[:3] for c in e.calls] == [("prefill", 0, 0), ("decode", 0, 3), ("decode", 1, 0), ("reset", 0), ("prefill", 0, 0)]
    with pytest.raises(KeyError):
        s.open("b")
    assert json.dumps(sorted(s.live)) == '["b", "c"]'
