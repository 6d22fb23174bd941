"""Small random block models for the tests: configurations of odd sizes and weights that make faults visible."""
import copy

import numpy as np

import plain_blocks as pb

ROT = {"base": 10000.0, "dims": 8}
YARN = {"base": 300.0, "dims": 16, "scaling": {"factor": 5.0, "original": 96, "fast": 6.0, "slow": 0.5}}


def latent(heads=3, dim=24, rot_dim=8, vdim=40, q_rank=20, kv_rank=36, window=7, scale=0.4, rot=None, ff=52):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "mask": {"size": window}, "rot": dict(rot or ROT)}}


def wkv(heads=3, dim=20, rank=6, ff=44):
    return {"type": "wkv", "mlp": {"kind": "dense", "ff": ff} if ff else None, "mixer": {"heads": heads, "dim": dim}, "rank": rank}


def config(layers, width=72, vocab=101, eps=1e-5, embed_scale=3.0, loop=None):
    return {"architecture": "Nezolix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers, "loop": loop}


CHUNK_YARN = {"base": 200.0, "dims": 8, "scaling": {"factor": 3.0, "original": 64, "fast": 5.0, "slow": 0.4}}


def attention(heads=6, kv_heads=2, dim=20, chunk=7, scale=0.35, cap=6.0, rot=None, ff=52):
    """Shared-kv attention: values are the keys as projected."""
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": cap,
                      "mask": {"size": chunk} if chunk else None, "rot": dict(rot or {"base": 1000.0, "dims": 6})}}


def rglru(width=36, blocks=3, conv=3, ff=44):
    return {"type": "rglru", "mlp": {"kind": "dense", "ff": ff} if ff else None, "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def pizilix(layers, width=72, vocab=101, eps=1e-5, cap=9.0, loop=None):
    return {"architecture": "Pizilix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers, "loop": loop}


# name -> configuration: every size differs from its neighbours, and each covers another branch
CONFIGS = {
    # sizes that are multiples of nothing; a layer without feed-forward; a stretch in the middle runs three times
    "odd": config([latent(), wkv(ff=0), latent(heads=5, dim=10, rot_dim=6, vdim=9, q_rank=11, kv_rank=13, window=4, rot={"base": 77.0, "dims": 6}, ff=35), wkv()],
                  width=70, vocab=99, loop={"start": 1, "stop": 3, "times": 3}),
    # one head; YaRN; vectors of one size class up; every layer once
    "yarn": config([latent(heads=1, dim=32, rot_dim=16, vdim=200, q_rank=48, kv_rank=24, window=33, rot=YARN), wkv(heads=1, dim=96, rank=16),
                    latent(heads=2, dim=48, rot_dim=16, vdim=64, q_rank=16, kv_rank=72, window=65, rot=YARN, ff=0)], width=96, vocab=130, embed_scale=1.0),
    # aligned sizes (the vectorised paths), loop over everything
    "aligned": config([latent(heads=4, dim=64, rot_dim=32, vdim=128, q_rank=96, kv_rank=128, window=50, rot={"base": 5000.0, "dims": 32}, ff=192, scale=0.15),
                       wkv(heads=2, dim=64, rank=16, ff=320)], width=192, vocab=256, loop={"start": 0, "stop": 2, "times": 2}),
    "wkv_only": config([wkv(heads=2, dim=128, rank=9), wkv(heads=5, dim=7, rank=1, ff=0), wkv(heads=1, dim=160, rank=24)], width=88),
    # odd head dimensions; a window wider than the context; seventeen heads (one more than a group of the decode kernel)
    "wide_window": config([latent(heads=17, dim=7, rot_dim=5, vdim=3, q_rank=9, kv_rank=19, window=5000, rot={"base": 31.0, "dims": 2}), wkv(heads=2, dim=33, rank=70)],
                          width=65, vocab=77),
    # Pizilix: sizes that are multiples of nothing, a stretch in the middle that runs three times
    "piz_odd": pizilix([attention(), rglru(ff=0), attention(heads=5, kv_heads=5, dim=9, chunk=4, rot={"base": 77.0, "dims": 2}, ff=35), rglru(width=35, blocks=5, conv=2)],
                       width=70, vocab=99, loop={"start": 1, "stop": 3, "times": 3}),
    # aligned sizes (the vectorised paths), YaRN, loop over everything
    "piz_aligned": pizilix([attention(heads=8, kv_heads=2, dim=64, chunk=50, scale=0.15, rot=dict(CHUNK_YARN, dims=32), ff=192), rglru(width=256, blocks=2, conv=4, ff=320)],
                           width=192, vocab=256, loop={"start": 0, "stop": 2, "times": 2}),
    # more query heads per key head than a group of the decode kernel holds; one gate block wider than a tile; more taps than
    # the register window; a chunk longer than the context
    "piz_wide": pizilix([rglru(width=130, blocks=1, conv=6), attention(heads=19, kv_heads=1, dim=11, chunk=5000, rot={"base": 31.0, "dims": 10})], width=65, vocab=77),
    # whole-head rotation with YaRN, no mask, no caps; one tap; gate blocks of one channel; a layer without feed-forward
    "piz_plain": pizilix([attention(heads=3, kv_heads=3, dim=32, chunk=0, cap=None, scale=0.2, rot=dict(CHUNK_YARN, dims=32), ff=0), rglru(width=24, blocks=24, conv=1)],
                         width=80, cap=None),
    # the widest value size class, no rotation at all, wide gate blocks
    "piz_deep": pizilix([attention(heads=2, kv_heads=1, dim=200, chunk=65, scale=0.08, rot={"base": 10.0, "dims": 0}), rglru(width=400, blocks=2, conv=4, ff=0)], width=104),
    "window_1": config([latent(window=1), latent(window=2, rot={"base": 50.0, "dims": 4})], loop={"start": 0, "stop": 1, "times": 2}),
}


def make(cfg, seed=0, sharp=1.0):
    """(config.json contents, tensors rounded to bfloat16). sharp multiplies the attention scores' scale."""
    cfg = copy.deepcopy(cfg)
    ranks = [l.pop("rank", 0) for l in cfg["layers"]]
    pizi = cfg["architecture"] == "Pizilix"
    for l in cfg["layers"]:
        if "scale" in l["mixer"]:
            l["mixer"]["scale"] *= sharp
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    t = {}

    def mat(name, rows, cols, gain=1.0):
        t[name] = rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    def norm(name, n):
        t[name] = (0.0 if pizi else 1.0) + 0.3 * rng.standard_normal(n)

    t["embed"] = rng.standard_normal((cfg["vocab"], W)) * 0.5
    for i, (l, rank) in enumerate(zip(cfg["layers"], ranks)):
        L, m = f"l{i}.", l["mixer"]
        H, D = m.get("heads"), m.get("dim")
        norm(L + "norm1", W)
        if not pizi:
            norm(L + "norm1b", W)
        if l["type"] == "latent_attention":
            mat(L + "mix.dq", m["q_rank"], W)
            norm(L + "mix.dq.norm", m["q_rank"])
            mat(L + "mix.uq", H * (D + m["rot_dim"]), m["q_rank"])
            mat(L + "mix.dkv", m["kv_rank"] + m["rot_dim"], W)
            norm(L + "mix.dkv.norm", m["kv_rank"])
            mat(L + "mix.uk", H * D, m["kv_rank"])
            mat(L + "mix.uv", H * m["vdim"], m["kv_rank"])
            mat(L + "mix.g", H * m["vdim"], W)
            mat(L + "mix.o", W, H * m["vdim"])
        elif l["type"] == "attention":
            mat(L + "mix.q", H * D, W)
            mat(L + "mix.k", m["kv_heads"] * D, W)
            mat(L + "mix.o", W, H * D)
        elif l["type"] == "rglru":
            N, B = m["width"], m["blocks"]
            for s in "yx":
                mat(L + "mix." + s, N, W)
                t[L + "mix." + s + ".b"] = rng.standard_normal(N) * 0.3
            t[L + "mix.conv"] = rng.standard_normal((N, m["conv"])) * 0.8
            t[L + "mix.conv.b"] = rng.standard_normal(N) * 0.3
            for s in ("ra", "ri"):
                t[L + "mix." + s] = rng.standard_normal((B, N // B, N // B)) * 1.5 / np.sqrt(N // B)
                t[L + "mix." + s + ".b"] = rng.standard_normal((B, N // B)) * 0.5
            t[L + "mix.lam"] = rng.normal(-4.0, 2.0, N)  # memories from one token to thousands
            mat(L + "mix.o", W, N)
        else:
            for s in "rkvgw":
                t[L + "mix.mu." + s] = rng.uniform(0, 1, W)
            for s in "rkvg":
                mat(L + "mix." + s, H * D, W)
            mat(L + "mix.w1", rank, W)
            mat(L + "mix.w2", H * D, rank)
            t[L + "mix.w0"] = rng.normal(-2.5, 1.5, H * D)
            t[L + "mix.u"] = rng.standard_normal((H, D)) * 0.7
            norm(L + "mix.norm", H * D)
            mat(L + "mix.o", W, H * D)
        if l.get("mlp"):
            norm(L + "norm2", W)
            if not pizi:
                norm(L + "norm2b", W)
            mat(L + "mlp.gate", l["mlp"]["ff"], W)
            mat(L + "mlp.up", l["mlp"]["ff"], W)
            mat(L + "mlp.down", W, l["mlp"]["ff"])
    norm("final.norm", W)
    if not pizi:
        mat("head", cfg["vocab"], W)
    return cfg, {k: pb.bf16_round(v) for k, v in t.items()}


def tokens(cfg, n, seed=1):
    return [int(v) for v in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def cuts_of(n, *sizes):
    """n tokens cut into portions that repeat the given sizes."""
    out, i = [], 0
    while n:
        c = min(n, sizes[i % len(sizes)])
        out.append(c)
        n -= c
        i += 1
    return out
