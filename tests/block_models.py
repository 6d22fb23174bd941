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
    "window_1": config([latent(window=1), latent(window=2, rot={"base": 50.0, "dims": 4})], loop={"start": 0, "stop": 1, "times": 2}),
}


def make(cfg, seed=0, sharp=1.0):
    """(config.json contents, tensors rounded to bfloat16). sharp multiplies the attention scores' scale."""
    cfg = copy.deepcopy(cfg)
    ranks = [l.pop("rank", 0) for l in cfg["layers"]]
    for l in cfg["layers"]:
        if l["type"] == "latent_attention":
            l["mixer"]["scale"] *= sharp
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    t = {}

    def mat(name, rows, cols, gain=1.0):
        t[name] = rng.standard_normal((rows, cols)) * gain / np.sqrt(cols)

    def norm(name, n):
        t[name] = 1.0 + 0.3 * rng.standard_normal(n)

    t["embed"] = rng.standard_normal((cfg["vocab"], W)) * 0.5
    for i, (l, rank) in enumerate(zip(cfg["layers"], ranks)):
        L, m = f"l{i}.", l["mixer"]
        H, D = m["heads"], m["dim"]
        norm(L + "norm1", W)
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
            norm(L + "norm2b", W)
            mat(L + "mlp.gate", l["mlp"]["ff"], W)
            mat(L + "mlp.up", l["mlp"]["ff"], W)
            mat(L + "mlp.down", W, l["mlp"]["ff"])
    norm("final.norm", W)
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
