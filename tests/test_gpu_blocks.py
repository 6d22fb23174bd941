"""Block models on the GPU (the engine's own entry points) against the plain statement of their mechanisms.

Errors are measured per position: root mean square over the vocabulary of the difference of the logits (mean taken off),
over the root mean square of the logits. Limits: 1e-4 for a 32-bit engine; for a bfloat16 one, three times what rounding
the operands of the matrix products to bfloat16 does to the plain model's logits of the same tokens.
"""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import block_models as bm
import plain_blocks as pb

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


def err(got, ref):
    d = np.asarray(got, np.float64) - ref
    d = d - d.mean(axis=-1, keepdims=True)
    r = ref - ref.mean(axis=-1, keepdims=True)
    return float((np.sqrt((d * d).mean(axis=-1)) / np.sqrt((r * r).mean())).max())


class Case:
    def __init__(self, folder, cfg, tensors):
        self.folder, self.cfg, self.tensors = folder, cfg, tensors
        self.cache = {}

    def plain(self, toks):
        key = tuple(toks)
        if key not in self.cache:
            self.cache[key] = pb.PlainModel(self.cfg, self.tensors).run(toks)
        return self.cache[key]

    def limit(self, dtype, toks):
        if dtype == "float32":
            return 1e-4
        key = ("limit", *toks)
        if key not in self.cache:
            self.cache[key] = 3 * err(pb.PlainModel(self.cfg, self.tensors, pb.to_bf16).run(toks), self.plain(toks))
        return self.cache[key]


@pytest.fixture(scope="module")
def case(tmp_path_factory):
    made = {}

    def get(name, sharp=1.0, cfg=None):
        if (name, sharp) not in made:
            c, t = bm.make(cfg or bm.CONFIGS[name], seed=len(made) + 5, sharp=sharp)
            made[name, sharp] = Case(pb.write_model(tmp_path_factory.mktemp("block") / name, c, t), c, t)
        return made[name, sharp]

    return get


def engine(pkg, c, dtype, max_seqs=2, max_ctx=512):
    return pkg.Engine.from_model(c.folder, dtype=dtype, max_seqs=max_seqs, max_ctx=max_ctx)


def feed(sess, sid, toks, cuts):
    """All logits of a sequence fed in portions."""
    out, at = [], 0
    for n in cuts:
        out.append(sess.feed(sid, toks[at:at + n], range(n)))
        at += n
    assert at == len(toks)
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(bm.CONFIGS))
def test_prompt_and_decode_match_the_plain_model(pkg, case, name, dtype):
    c = case(name)
    toks = bm.tokens(c.cfg, 150)
    ref = c.plain(toks)
    sess = pkg.Sessions(engine(pkg, c, dtype))
    assert err(feed(sess, "whole", toks, [150]), ref) < c.limit(dtype, toks)
    assert err(feed(sess, "single", toks[:110], [1] * 110), ref[:110]) < c.limit(dtype, toks)
    sess.end("whole")
    sess.end("single")


MECHANISMS = {  # one layer, one mechanism; the rest of the model is as plain as it gets
    "latent attention": [bm.latent(ff=0)],
    "latent attention, rotation of part of rot_dim": [bm.latent(ff=0, rot_dim=12, rot={"base": 9.0, "dims": 4})],
    "yarn": [bm.latent(ff=0, rot_dim=16, rot=bm.YARN, window=90)],
    "wkv": [bm.wkv(ff=0)],
    "feed-forward": [bm.latent(window=1, ff=77)],
}
PIZILIX_MECHANISMS = {
    "attention": [bm.attention(ff=0)],
    "attention, rotation of the whole head": [bm.attention(ff=0, dim=16, rot={"base": 9.0, "dims": 16})],
    "attention, one head each": [bm.attention(ff=0, heads=4, kv_heads=4, chunk=33)],
    "attention, vectorised": [bm.attention(ff=0, heads=4, kv_heads=2, dim=32, chunk=40, rot={"base": 50.0, "dims": 16})],
    "attention, yarn": [bm.attention(ff=0, dim=24, chunk=50, rot=bm.CHUNK_YARN)],
    "attention, everything seen": [bm.attention(ff=0, chunk=0)],
    "recurrence": [bm.rglru(ff=0)],
    "recurrence, wide blocks": [bm.rglru(ff=0, width=192, blocks=1, conv=4)],
    "feed-forward, silu": [bm.attention(chunk=1, ff=77)],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", [*MECHANISMS, *PIZILIX_MECHANISMS])
def test_each_mechanism_alone(pkg, case, name, dtype):
    cfg = bm.config(MECHANISMS[name]) if name in MECHANISMS else bm.pizilix(PIZILIX_MECHANISMS[name])
    c = case(name.replace(" ", "_").replace(",", ""), cfg=cfg)
    toks = bm.tokens(c.cfg, 70)
    ref = c.plain(toks)
    sess = pkg.Sessions(engine(pkg, c, dtype))
    assert err(feed(sess, 0, toks, [70]), ref) < c.limit(dtype, toks)
    assert err(feed(sess, 1, toks, [33] + [1] * 37), ref) < c.limit(dtype, toks)


MISTAKES = {  # planted in the plain model: what a missing or wrong piece would do to the logits
    "no sink": ("sink_weights", lambda s: np.exp(s - s.max(-1, keepdims=True)) / np.exp(s - s.max(-1, keepdims=True)).sum(-1, keepdims=True)),
    "no cap on scores": ("softcap", None),
    "sliding instead of chunked": ("seen_keys", lambda p, mask: max(0, p - mask["size"] + 1) if mask else 0),
    "no rotation": ("rotate", lambda x, positions, rot: x),
    "conv without history": ("causal_conv", lambda x, w, b, before: (x * w[:, -1] + b, before)),
    "first token unscaled": ("gated_recurrence", None),
    "relu for silu": ("silu", lambda z: np.maximum(z, 0)),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_mistakes_would_show(pkg, case, name, monkeypatch):
    """The engine agrees with the plain model, and a plain model with one mistake does not."""
    c = case("piz_mistakes", cfg=bm.pizilix([bm.attention(scale=1.0), bm.rglru(), bm.attention(chunk=20, scale=1.0)], loop={"start": 0, "stop": 2, "times": 2}))
    toks = bm.tokens(c.cfg, 60)
    ref, limit = c.plain(toks), c.limit("bfloat16", toks)
    got = pkg.Sessions(engine(pkg, c, "bfloat16")).feed(0, toks, range(60))
    assert err(got, ref) < limit
    what, wrong = MISTAKES[name]
    if name == "no cap on scores":
        right = pb.softcap
        wrong = lambda z, cap: z if cap == 6.0 else right(z, cap)
    if name == "first token unscaled":
        right_rec = pb.gated_recurrence

        def wrong(u, r, i, lam, S):  # starts where the first token's state comes out as i u
            a = np.exp(-8 * r[0] * np.logaddexp(0, lam))
            return right_rec(u, r, i, lam, (1 - np.sqrt(1 - a * a)) / a * i[0] * u[0])
    monkeypatch.setattr(pb, what, wrong)
    assert err(pb.PlainModel(c.cfg, c.tensors).run(toks), ref) > 2 * limit


def test_embedding_joins_every_further_pass(pkg, case):
    """With one pass, or with layers unrolled under other names, the embedding is not added again: both differ from the loop."""
    c = case("piz_mistakes", cfg=bm.pizilix([bm.attention(scale=1.0), bm.rglru(), bm.attention(chunk=20, scale=1.0)], loop={"start": 0, "stop": 2, "times": 2}))
    toks = bm.tokens(c.cfg, 40)
    unrolled = copy.deepcopy(c.cfg)
    unrolled["loop"] = None
    unrolled["layers"] = [c.cfg["layers"][l] for l in pb.layer_runs(c.cfg)]
    t = {k: v for k, v in c.tensors.items() if not k.startswith("l")}
    for i, l in enumerate(pb.layer_runs(c.cfg)):
        t.update({f"l{i}." + k.split(".", 1)[1]: v for k, v in c.tensors.items() if k.startswith(f"l{l}.")})
    assert err(pb.PlainModel(unrolled, t).run(toks), c.plain(toks)) > 0.1
    from pathlib import Path
    u = Case(pb.write_model(Path(c.folder).parent / "unrolled", unrolled, t), unrolled, t)
    for x in (c, u):
        sess = pkg.Sessions(engine(pkg, x, "float32"))
        assert err(feed(sess, 0, toks, [21] + [1] * 19), x.plain(toks)) < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_stream_of_one_token_pizilix(pkg, case, dtype):
    """The same for a loop that adds the embedding again: what is handed in counts as the embedding."""
    c = case("piz_odd")
    eng = engine(pkg, c, dtype)
    trace = []
    ref = pb.PlainModel(c.cfg, c.tensors).run([42], trace)
    x = eng.lookup_embedding(42)
    logits = eng.forward(x, 0)
    assert np.abs(x - trace[-1][0]).max() < (1e-4 if dtype == "float32" else 5e-2) * np.abs(trace[-1]).max()
    assert err(logits[None], ref) < c.limit(dtype, [42])


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_stream_of_one_token(pkg, case, dtype):
    """b200_forward takes and returns the residual stream: embedding row (scaled) in, the stream after all layer runs out."""
    c = case("odd")
    eng = engine(pkg, c, dtype)
    trace = []
    ref = pb.PlainModel(c.cfg, c.tensors).run([42], trace)
    x = eng.lookup_embedding(42)
    assert np.allclose(x, c.tensors["embed"][42] * c.cfg["embedding"]["scale"], rtol=1e-6)
    logits = eng.forward(x, 0)
    assert np.abs(x - trace[-1][0]).max() < (1e-4 if dtype == "float32" else 5e-2) * np.abs(trace[-1]).max()
    assert err(logits[None], ref) < c.limit(dtype, [42])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(2,), (3, 2), (7, 1, 16), (64, 65, 3), (31,)])
@pytest.mark.parametrize("name", ["odd", "aligned", "piz_odd", "piz_aligned"])
def test_portions_of_several_sizes(pkg, case, name, sizes, dtype):
    c = case(name)
    toks = bm.tokens(c.cfg, 170)
    sess = pkg.Sessions(engine(pkg, c, dtype))
    assert err(feed(sess, 0, toks, bm.cuts_of(170, *sizes)), c.plain(toks)) < c.limit(dtype, toks)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [5, 16])
def test_small_chunks_and_wrapping_rings(pkg, case, dtype, chunk, monkeypatch):
    """A prompt longer than a chunk is cut by the engine; the windowed caches are rings of window - 1 + chunk rows, which
    wrap many times here, in prompts and in decoding."""
    monkeypatch.setenv("B200_PREFILL_CHUNK", str(chunk))
    for name in ("odd", "aligned", "piz_odd", "piz_aligned"):
        c = case(name)
        toks = bm.tokens(c.cfg, 230)
        sess = pkg.Sessions(engine(pkg, c, dtype))
        assert err(feed(sess, 0, toks, [120] + [1] * 60 + [50]), c.plain(toks)) < c.limit(dtype, toks)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65])
def test_window_edges(pkg, case, window, dtype):
    """Sharp scores: single keys carry most of the weight, so a window one token off changes the logits. The mistake is
    planted in the plain model: windows one smaller and one larger must be told apart with room to spare."""
    cfg = bm.config([bm.latent(window=window, ff=0), bm.latent(window=window, heads=2, dim=16, vdim=24, ff=0)])
    c = case(f"edge{window}", sharp=2.0, cfg=cfg)
    toks = bm.tokens(c.cfg, 150)
    ref = c.plain(toks)
    mistake = np.inf
    for off in (-1, 1):
        if window + off < 1:
            continue
        wrong = copy.deepcopy(c.cfg)
        for l in wrong["layers"]:
            l["mixer"]["mask"]["size"] = window + off
        bad = pb.PlainModel(wrong, c.tensors).run(toks)
        mistake = min(mistake, err(bad, ref))
    limit = c.limit(dtype, toks)
    assert mistake > 3 * limit
    sess = pkg.Sessions(engine(pkg, c, dtype))
    for sid, cuts in enumerate(([150], [90] + [1] * 60, bm.cuts_of(150, 2, 5, 64, 1))):
        assert err(feed(sess, sid, toks, cuts), ref) < limit
        sess.end(sid)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [1, 2, 16, 63, 64, 65])
def test_chunk_edges(pkg, case, chunk, dtype):
    """The same for chunked masks: chunks one smaller or larger must be told apart, and so must chunks counted from where a
    portion starts (positions restarting there)."""
    cfg = bm.pizilix([bm.attention(chunk=chunk, ff=0), bm.attention(chunk=chunk, heads=4, kv_heads=1, dim=32, rot={"base": 40.0, "dims": 16}, ff=0)])
    c = case(f"chunk{chunk}", sharp=3.0, cfg=cfg)
    toks = bm.tokens(c.cfg, 150)
    ref = c.plain(toks)
    limit = c.limit(dtype, toks)
    for off in (-1, 1):
        if chunk + off < 1:
            continue
        wrong = copy.deepcopy(c.cfg)
        for l in wrong["layers"]:
            l["mixer"]["mask"]["size"] = chunk + off
        assert err(pb.PlainModel(wrong, c.tensors).run(toks), ref) > 3 * limit
    sess = pkg.Sessions(engine(pkg, c, dtype))
    for sid, cuts in enumerate(([150], [90] + [1] * 60, bm.cuts_of(150, 2, 5, 64, 1))):
        assert err(feed(sess, sid, toks, cuts), ref) < limit
        sess.end(sid)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", [(2, 1, 32), (40, 2, 12)])
def test_a_far_key_in_its_chunk(pkg, case, heads, dtype):
    """An early token's key stands out for late queries until their chunk ends: in prompts, in decoding, and (many splits of the
    context) at the splits' edges. The sink's share of the weight shows in the queries that see nothing alike."""
    n, chunk, early = 660, 300, 305
    H, G, D = heads
    c = case(f"far_chunk{H}", cfg=bm.pizilix([bm.attention(heads=H, kv_heads=G, dim=D, chunk=chunk, scale=0.02, cap=30.0, rot={"base": 10.0, "dims": 4}, ff=0)]))
    t = {k: v.copy() for k, v in c.tensors.items()}
    W = c.cfg["width"]
    t["embed"][:, :2] = 0
    t["embed"][1], t["embed"][2] = np.eye(W)[0], np.eye(W)[1]
    t["l0.norm1"][:] = 0
    t["l0.mix.k"][:, 0] = 0
    t["l0.mix.k"][5::D, 0] = 4
    t["l0.mix.q"][:, 1] = 0
    t["l0.mix.q"][5::D, 1] = 8
    t = {k: pb.bf16_round(v) for k, v in t.items()}
    from pathlib import Path
    c2 = Case(pb.write_model(Path(c.folder).parent / f"far_chunk{H}b", c.cfg, t), c.cfg, t)
    toks = [3 + v % (c.cfg["vocab"] - 3) for v in bm.tokens(c.cfg, n)]
    toks[early] = 1
    places = (early + 1, early + 64, early + 150, 2 * chunk - 1, 2 * chunk)
    for p in places:
        toks[p] = 2
    ref = c2.plain(toks)
    assert err(ref[places[-2]][None], ref[places[-1]][None]) > 0.3
    sess = pkg.Sessions(engine(pkg, c2, dtype, max_ctx=700))
    for sid, cuts in enumerate(([n], [early + 140] + [1] * (n - early - 140), bm.cuts_of(n, 50, 3))):
        got = feed(sess, sid, toks, cuts)
        for p in places:
            assert err(got[p:p + 1], ref[p:p + 1]) < c2.limit(dtype, toks), p
        sess.end(sid)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_recurrence_that_remembers(pkg, case, dtype):
    """Channels that hardly decay: what an early token left is still there hundreds of tokens later, across tiles and portions."""
    c = case("remember", cfg=bm.pizilix([bm.rglru(width=72, blocks=2, conv=4, ff=0)]))
    t = {k: v.copy() for k, v in c.tensors.items()}
    t["l0.mix.lam"][:] = -9.0
    t = {k: pb.bf16_round(v) for k, v in t.items()}
    from pathlib import Path
    c2 = Case(pb.write_model(Path(c.folder).parent / "remember2", c.cfg, t), c.cfg, t)
    toks = bm.tokens(c.cfg, 330)
    other = list(toks)
    other[3] = (toks[3] + 1) % c.cfg["vocab"]
    assert err(c2.plain(other)[-50:], c2.plain(toks)[-50:]) > 3e-3
    sess = pkg.Sessions(engine(pkg, c2, dtype))
    for sid, cuts in enumerate(([330], [65] * 5 + [5], [3, 127] + [1] * 200)):
        assert err(feed(sess, sid, toks, cuts), c2.plain(toks)) < c2.limit(dtype, toks)
        sess.end(sid)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds(pkg, case, dtype):
    """One early token's latent points along one direction and a late query asks for it: its score stands out among
    hundreds of keys as long as it is inside the window, and the logits change the moment it leaves."""
    n, window, early = 400, 300, 60
    c = case("far", cfg=bm.config([bm.latent(heads=2, dim=32, rot_dim=4, vdim=32, q_rank=24, kv_rank=40, window=window, ff=0, rot={"base": 10.0, "dims": 0}, scale=0.5)]))
    # token 1's embedding is its own direction; queries of token 2 look for it in every head
    t = {k: v.copy() for k, v in c.tensors.items()}
    W = c.cfg["width"]
    t["embed"][:, :2] = 0
    t["embed"][1], t["embed"][2] = np.eye(W)[0], np.eye(W)[1]
    t["l0.norm1"][:] = 1
    t["l0.mix.dkv"][:40, 0] = 0
    t["l0.mix.dkv"][5, 0] = 1
    t["l0.mix.uk"][:, 5] = 4
    t["l0.mix.dq"][:, 1] = 0
    t["l0.mix.dq"][3, 1] = 1
    t["l0.mix.uq"][:, 3] = 4
    t = {k: pb.bf16_round(v) for k, v in t.items()}
    from pathlib import Path
    c2 = Case(pb.write_model(Path(c.folder).parent / "far2", c.cfg, t), c.cfg, t)
    toks = [3 + v % (c.cfg["vocab"] - 3) for v in bm.tokens(c.cfg, n)]
    toks[early] = 1
    for p in (early + 1, early + 150, early + window - 1, early + window):
        toks[p] = 2
    ref = c2.plain(toks)
    inside, outside = ref[early + window - 1], ref[early + window]
    assert err(inside[None], outside[None]) > 0.3  # the key's leaving shows
    sess = pkg.Sessions(engine(pkg, c2, dtype))
    for sid, cuts in enumerate(([n], [early + 140] + [1] * (n - early - 140), bm.cuts_of(n, 50, 3))):
        got = feed(sess, sid, toks, cuts)
        for p in (early + 1, early + 150, early + window - 1, early + window):
            assert err(got[p:p + 1], ref[p:p + 1]) < c2.limit(dtype, toks), p
        sess.end(sid)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "piz_odd"])
def test_first_tokens_and_short_sequences(pkg, case, name, dtype):
    c = case(name)
    sess = pkg.Sessions(engine(pkg, c, dtype))
    for n in (1, 2, 3, 4, 5, 9):
        toks = bm.tokens(c.cfg, n, seed=50 + n)
        for cuts in ([n], [1] * n):
            assert err(feed(sess, n, toks, cuts), c.plain(toks)) < c.limit(dtype, toks)
            sess.end(n)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "piz_odd"])
def test_slots_that_are_freed_and_used_again(pkg, case, name, dtype):
    c = case(name)
    eng = engine(pkg, c, dtype, max_seqs=1)
    sess = pkg.Sessions(eng)
    long, short = bm.tokens(c.cfg, 140, seed=8), bm.tokens(c.cfg, 45, seed=9)
    feed(sess, "a", long, [100] + [1] * 40)
    with pytest.raises(RuntimeError):
        sess.feed("b", short)
    sess.end("a")
    assert err(feed(sess, "b", short, [20] + [1] * 25), c.plain(short)) < c.limit(dtype, short)
    # starting over at position 0 without a reset
    got = eng.prefill_rows(short[:30], range(30), slot=0, start_pos=0)
    assert err(got, c.plain(short)[:30]) < c.limit(dtype, short)
    # a slot only continues where it stands
    for bad in (29, 31, 5):
        with pytest.raises(pkg.B200Error, match="next position is 30"):
            eng.decode([1], [bad])
    with pytest.raises(pkg.B200Error, match="exceeds"):
        eng.prefill(bm.tokens(c.cfg, 500), start_pos=30)
    assert err(eng.decode([short[30]], [30])[0], c.plain(short)[30:31]) < c.limit(dtype, short)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch", [2, 4, 7, 12, 19])
@pytest.mark.parametrize("name", ["odd", "piz_odd", "piz_aligned"])
def test_batches_of_unequal_requests_match_each_alone(pkg, case, name, dtype, batch):
    """Prompts of unequal length in one call (runs share chunks), then joint decode steps in mixed slot order, on the
    matvec path (small batches) and on the row path (large ones)."""
    c = case(name)
    eng = engine(pkg, c, dtype, max_seqs=batch + 2)
    lens = [3 + 11 * i % 37 for i in range(batch)]
    seqs = [bm.tokens(c.cfg, n + 6, seed=100 + i) for i, n in enumerate(lens)]
    slots = list(np.random.default_rng(3).permutation(batch + 2)[:batch])
    first = eng.prefill_batch([s[:n] for s, n in zip(seqs, lens)], slots=slots)
    refs = [c.plain(s) for s in seqs]
    limit = max(c.limit(dtype, s) for s in seqs)
    for i, n in enumerate(lens):
        assert err(first[i:i + 1], refs[i][n - 1:n]) < limit
    for k in range(5):
        order = np.random.default_rng(k).permutation(batch)
        logits, amax = eng.decode([seqs[i][lens[i] + k] for i in order], [lens[i] + k for i in order], slots=[slots[i] for i in order])
        assert np.array_equal(amax, logits.argmax(axis=1))
        for row, i in zip(logits, order):
            assert err(row[None], refs[i][lens[i] + k][None]) < limit
    # the prompt continues in a second joint call
    tail = eng.prefill_batch([s[-1:] for s in seqs], slots=slots, start_pos=[n + 5 for n in lens])
    for i in range(batch):
        assert err(tail[i:i + 1], refs[i][-1:]) < limit


@pytest.mark.parametrize("name", ["odd", "wkv_only", "piz_odd", "piz_wide"])
def test_greedy_generation(pkg, case, name):
    """The device-resident loop of a 32-bit engine chooses the plain model's ids."""
    c = case(name)
    prompt = bm.tokens(c.cfg, 23, seed=77)
    ids, gap = pb.greedy(c.cfg, c.tensors, prompt, 40)
    assert gap > 1e-4
    sess = pkg.Sessions(engine(pkg, c, "float32"))
    assert sess.generate_greedy("g", prompt, 40) == ids
    assert sess.live["g"][1] == 23 + 39


@pytest.mark.parametrize("name", ["aligned", "piz_aligned"])
def test_greedy_batch_and_penalty(pkg, case, name):
    c = case(name)
    eng = engine(pkg, c, "float32", max_seqs=3)
    prompts = [bm.tokens(c.cfg, n, seed=n) for n in (9, 30, 17)]
    first = eng.prefill_batch(prompts).argmax(axis=1)
    out, _ = eng.generate_greedy(first, [len(p) for p in prompts], 20)
    for i, p in enumerate(prompts):
        ids, gap = pb.greedy(c.cfg, c.tensors, p, 21)
        assert gap > 1e-4 and [int(first[i])] + [int(v) for v in out[:, i]] == ids
    # repetition penalty: every occurrence among the generated ids divides (or multiplies) that id's logit
    eng.kv_reset(0)
    p = prompts[0]
    tok = int(eng.prefill(p).argmax())
    got, _ = eng.generate_greedy_penalized([tok], [len(p)], 12, 1.5, histories=[[tok]])
    m = pb.PlainModel(c.cfg, c.tensors)
    m.run(p)
    seen = [tok]
    for g in got[:, 0]:
        l = m.run([seen[-1]])[-1]
        for s in seen:
            l[s] = l[s] / 1.5 if l[s] > 0 else l[s] * 1.5
        assert int(g) == int(l.argmax())
        seen.append(int(g))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "piz_odd"])
def test_long_decoding(pkg, case, name, dtype):
    """400 decoded tokens: dozens of windows, and a recurrence that has forgotten its start."""
    c = case(name)
    toks = bm.tokens(c.cfg, 420, seed=4)
    sess = pkg.Sessions(engine(pkg, c, dtype))
    assert err(feed(sess, 0, toks, [20] + [1] * 400), c.plain(toks)) < c.limit(dtype, toks)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["yarn", "piz_aligned"])
def test_results_do_not_depend_on_cuts_or_company(pkg, case, name, dtype):
    """The same tokens as one prompt, in portions, and beside other requests: equal beyond rounding."""
    c = case(name)
    toks = bm.tokens(c.cfg, 130, seed=12)
    eng = engine(pkg, c, dtype, max_seqs=4)
    a = eng.prefill(toks, slot=0)
    eng.prefill(toks[:77], slot=1)
    b = eng.prefill(toks[77:], slot=1, start_pos=77)
    m = eng.prefill_batch([bm.tokens(c.cfg, 50), toks, bm.tokens(c.cfg, 3)], slots=[3, 2, 0])[1]
    for other in (b, m):
        assert err(other[None], a[None].astype(np.float64)) < (1e-5 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "piz_odd"])
def test_trace_replay_program(pkg, case, tmp_path, name, dtype):
    c = case(name)
    a, b = bm.tokens(c.cfg, 40, seed=1), bm.tokens(c.cfg, 12, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:25], "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[25:39], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[39:], "want": [0]}], "end": ["a"]},
             {"step": 7, "entries": [{"id": "b", "tokens": b, "want": [3, 11]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", c.folder, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 7"]
    assert not (tmp_path / "1.f32").exists()
    V = c.cfg["vocab"]
    for step, toks, rows in ((0, a, [0, 24]), (2, a, [39]), (7, b, [3, 11])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(rows), V)
        assert err(got, c.plain(toks)[rows]) < c.limit(dtype, toks)
