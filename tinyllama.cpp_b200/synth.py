"""Synthetic models: named shapes from the benchmark configurations and a ctypes front end to the
GGUF writer / quantizers in csrc/synth.cpp."""
import ctypes
import json
import os
import struct

import numpy as np

from . import _build

Q8_0, Q4_K, Q6_K, F32 = 8, 12, 14, 0
BLOCK_ELEMS = {Q8_0: 32, Q4_K: 256, Q6_K: 256, F32: 1}
BLOCK_BYTES = {Q8_0: 34, Q4_K: 144, Q6_K: 210, F32: 4}

# scheme: 0 = every linear Q8_0; 1 = Q4_K with Q6_K for attn_v / ffn_down / output ("Q4_K_M-style");
#         2 = every linear Q6_K; 3 = every linear Q4_K
SHAPES = {
    "tiny": dict(hidden=256, ffn=512, n_heads=4, n_kv_heads=2, n_layers=2, vocab=512, max_pos=128, theta=10000.0),
    "tiny_mha": dict(hidden=512, ffn=768, n_heads=4, n_kv_heads=4, n_layers=2, vocab=1024, max_pos=256, theta=10000.0),
    "tinyllama-1.1b": dict(hidden=2048, ffn=5632, n_heads=32, n_kv_heads=4, n_layers=22, vocab=32000, max_pos=2048, theta=10000.0),
    "llama2-7b": dict(hidden=4096, ffn=11008, n_heads=32, n_kv_heads=32, n_layers=32, vocab=32000, max_pos=4096, theta=10000.0),
    "llama3-8b": dict(hidden=4096, ffn=14336, n_heads=32, n_kv_heads=8, n_layers=32, vocab=128256, max_pos=8192, theta=500000.0),
    "llama2-70b": dict(hidden=8192, ffn=28672, n_heads=64, n_kv_heads=8, n_layers=80, vocab=32000, max_pos=8192, theta=10000.0),
}


class _Cfg(ctypes.Structure):
    _fields_ = [(n, ctypes.c_int32) for n in "hidden ffn n_heads n_kv_heads n_layers vocab max_pos".split()] + [
        ("eps", ctypes.c_float), ("theta", ctypes.c_float), ("scheme", ctypes.c_int32),
        ("norm_random", ctypes.c_int32), ("seed", ctypes.c_uint64), ("sigma", ctypes.c_float)]


_lib = None


def lib():
    global _lib
    if _lib is None:
        _lib = ctypes.CDLL(_build.build_synth())
        _lib.b200_synth_write_gguf.argtypes = [ctypes.c_char_p, ctypes.POINTER(_Cfg)]
        _lib.b200_synth_quantize.argtypes = [ctypes.c_int, ctypes.c_void_p, ctypes.c_int64, ctypes.c_void_p]
        _lib.b200_synth_fill_normal.argtypes = [ctypes.c_void_p, ctypes.c_int64, ctypes.c_uint64, ctypes.c_uint64, ctypes.c_float]
        _lib.b200_synth_fill_normal.restype = None
        _lib.b200_synth_set_threads.argtypes = [ctypes.c_int]
        _lib.b200_synth_set_threads.restype = None
        # a launcher (torchrun) may have pinned OMP_NUM_THREADS to 1 for the process: the writer uses the cores it may run on
        try:
            _lib.b200_synth_set_threads(len(os.sched_getaffinity(0)))
        except AttributeError:
            _lib.b200_synth_set_threads(os.cpu_count() or 1)
    return _lib


def write_gguf(path, shape, scheme, seed=1234, sigma=0.02, norm_random=False, eps=1e-5, embd_quant=False, **overrides):
    """Writes a synthetic model file. `shape` is a key of SHAPES or a dict with the same fields.
    embd_quant: token_embd is quantised like attn_q (what real checkpoints ship) instead of F32."""
    s = dict(SHAPES[shape]) if isinstance(shape, str) else dict(shape)
    s.update(overrides)
    cfg = _Cfg(s["hidden"], s["ffn"], s["n_heads"], s["n_kv_heads"], s["n_layers"], s["vocab"], s["max_pos"],
               eps, s["theta"], scheme, int(bool(norm_random)) | (2 if embd_quant else 0), seed, sigma)
    rc = lib().b200_synth_write_gguf(os.fsencode(path), ctypes.byref(cfg))
    if rc:
        raise RuntimeError(f"b200_synth_write_gguf failed with status {rc}")
    return path


def fill_normal(n, seed, stream=1, sigma=0.02):
    out = np.empty(n, np.float32)
    lib().b200_synth_fill_normal(out.ctypes.data, n, seed, stream, sigma)
    return out


def quantize(ggml_type, x):
    """Quantizes a float32 array (size a multiple of the block size) into packed blocks (uint8 array)."""
    x = np.ascontiguousarray(x, np.float32).ravel()
    out = np.empty(x.size // BLOCK_ELEMS[ggml_type] * BLOCK_BYTES[ggml_type], np.uint8)
    rc = lib().b200_synth_quantize(ggml_type, x.ctypes.data, x.size, out.ctypes.data)
    if rc:
        raise RuntimeError(f"b200_synth_quantize failed with status {rc}")
    return out


# Block models of a real model's layer sizes. Nezolix: three latent-attention layers, then one WKV layer, repeated; Pizilix:
# attention and RG-LRU layers in turn.
BLOCK_SHAPES = {
    "pizilix-w2048": dict(design="Pizilix", width=2048, ff=5632, vocab=32000, n_layers=8, heads=16, kv_heads=4, dim=128, rot_dims=64, window=1024,
                          lru_width=2048, lru_blocks=16, conv=4),
    "pizilix-w4096": dict(design="Pizilix", width=4096, ff=11008, vocab=32000, n_layers=8, heads=32, kv_heads=8, dim=128, rot_dims=64, window=1024,
                          lru_width=4096, lru_blocks=16, conv=4),
    "nezolix-w2048": dict(design="Nezolix", width=2048, ff=5632, vocab=32000, n_layers=8, heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=256,
                          window=1024, wkv_heads=32, wkv_dim=64, decay_rank=64),
    "nezolix-w4096": dict(design="Nezolix", width=4096, ff=11008, vocab=32000, n_layers=8, heads=32, dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512,
                          window=1024, wkv_heads=64, wkv_dim=64, decay_rank=64),
}


def block_config(shape):
    s = BLOCK_SHAPES[shape] if isinstance(shape, str) else shape
    if s["design"] == "Pizilix":
        mlp = {"kind": "dense", "ff": s["ff"]}
        attn = {"type": "attention", "mlp": mlp,
                "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5, "softcap": 50.0,
                          "mask": {"size": s["window"]},
                          "rot": {"base": 10000.0, "dims": s["rot_dims"], "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
        lru = {"type": "rglru", "mlp": mlp, "mixer": {"width": s["lru_width"], "blocks": s["lru_blocks"], "conv": s["conv"]}}
        return {"architecture": "Pizilix", "width": s["width"], "vocab": s["vocab"], "norm": {"eps": 1e-6}, "logit_softcap": 30.0, "loop": None,
                "layers": [lru if l % 2 else attn for l in range(s["n_layers"])]}
    attn = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": s["ff"]},
            "mixer": {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot_dim"], "vdim": s["vdim"], "q_rank": s["q_rank"], "kv_rank": s["kv_rank"],
                      "scale": (s["dim"] + s["rot_dim"]) ** -0.5, "mask": {"size": s["window"]},
                      "rot": {"base": 10000.0, "dims": s["rot_dim"], "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    wkv = {"type": "wkv", "mlp": {"kind": "dense", "ff": s["ff"]}, "mixer": {"heads": s["wkv_heads"], "dim": s["wkv_dim"]}}
    return {"architecture": "Nezolix", "width": s["width"], "vocab": s["vocab"], "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "loop": None,
            "layers": [wkv if l % 4 == 3 else attn for l in range(s["n_layers"])]}


def block_tensors(cfg, decay_rank=0):
    """(name, shape) of every tensor of a block model."""
    W = cfg["width"]
    pizilix = cfg["architecture"] == "Pizilix"
    out = [("embed", (cfg["vocab"], W))]
    for i, l in enumerate(cfg["layers"]):
        L, m = f"l{i}.", l["mixer"]
        H, D = m.get("heads"), m.get("dim")
        out += [(L + "norm1", (W,))] + ([] if pizilix else [(L + "norm1b", (W,))])
        if l["type"] == "latent_attention":
            out += [(L + "mix." + n, s) for n, s in (
                ("dq", (m["q_rank"], W)), ("dq.norm", (m["q_rank"],)), ("uq", (H * (D + m["rot_dim"]), m["q_rank"])), ("dkv", (m["kv_rank"] + m["rot_dim"], W)),
                ("dkv.norm", (m["kv_rank"],)), ("uk", (H * D, m["kv_rank"])), ("uv", (H * m["vdim"], m["kv_rank"])), ("g", (H * m["vdim"], W)), ("o", (W, H * m["vdim"])))]
        elif l["type"] == "attention":
            out += [(L + "mix.q", (H * D, W)), (L + "mix.k", (m["kv_heads"] * D, W)), (L + "mix.o", (W, H * D))]
        elif l["type"] == "rglru":
            N, B = m["width"], m["blocks"]
            S = N // B
            out += [(L + "mix." + n, s) for n, s in (
                ("y", (N, W)), ("y.b", (N,)), ("x", (N, W)), ("x.b", (N,)), ("conv", (N, m["conv"])), ("conv.b", (N,)), ("ra", (B, S, S)), ("ra.b", (B, S)),
                ("ri", (B, S, S)), ("ri.b", (B, S)), ("lam", (N,)), ("o", (W, N)))]
        else:
            out += [(L + "mix.mu." + n, (W,)) for n in "rkvgw"] + [(L + "mix." + n, (H * D, W)) for n in "rkvg"]
            out += [(L + "mix." + n, s) for n, s in (("w1", (decay_rank, W)), ("w2", (H * D, decay_rank)), ("w0", (H * D,)), ("u", (H, D)), ("norm", (H * D,)), ("o", (W, H * D)))]
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            out += [(L + "norm2", (W,))] + ([] if pizilix else [(L + "norm2b", (W,))]) + [(L + "mlp.gate", (ff, W)), (L + "mlp.up", (ff, W)), (L + "mlp.down", (W, ff))]
    return out + [("final.norm", (W,))] + ([] if pizilix else [("head", (cfg["vocab"], W))])


def write_block_model(folder, shape, seed=1234, sigma=0.02):
    """Writes config.json and model.safetensors of a BLOCK_SHAPES entry: N(0, sigma) matrices (slices of one seeded block of
    16 Mi values at seeded offsets), unit norms, token-shift mixes in [0, 1), decay biases around -3 (WKV) and -5 (RG-LRU)."""
    os.makedirs(folder, exist_ok=True)
    s = BLOCK_SHAPES[shape] if isinstance(shape, str) else shape
    cfg = block_config(shape)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    names = block_tensors(cfg, s.get("decay_rank", 0))
    head, at = {}, 0
    for name, shp in names:
        n = int(np.prod(shp)) * 2
        head[name] = {"dtype": "BF16", "shape": list(shp), "data_offsets": [at, at + n]}
        at += n
    rng = np.random.default_rng(seed)
    block = rng.standard_normal(1 << 24, dtype=np.float32) * sigma
    block = (block.view(np.uint32) >> 16).astype(np.uint16)

    def bits(a):
        return (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)

    h = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for name, shp in names:
            n = int(np.prod(shp))
            if "norm" in name:
                f.write(bits(np.zeros(n) if s["design"] == "Pizilix" else np.ones(n)).tobytes())
            elif ".mu." in name:
                f.write(bits(rng.uniform(0, 1, n)).tobytes())
            elif name.endswith(".lam"):
                f.write(bits(rng.normal(-5, 1, n)).tobytes())
            elif name.endswith(".w0"):
                f.write(bits(rng.normal(-3, 1, n)).tobytes())
            else:
                while n:
                    o = int(rng.integers(0, block.size))
                    k = min(n, block.size - o)
                    f.write(block[o:o + k].tobytes())
                    n -= k
    return folder
