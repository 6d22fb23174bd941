"""Plain, slow numpy statement of the layer mechanisms of the block models (one function per mechanism): the oracle of
the tests. Shares no code with the package. Everything is computed in float64; `rnd` is applied to what enters a matrix product
(identity, or rounding to bfloat16 to learn how far that alone moves the results)."""
import json
import math
import struct

import numpy as np


# ---- files -------------------------------------------------------------------------------------------------------
def bf16_round(a):
    """float32 -> nearest bfloat16 (ties to even), returned as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return u.view(np.float32)


def write_model(folder, cfg, tensors):
    """config.json and model.safetensors with every tensor in bfloat16 (values must already be bfloat16)."""
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    head, blobs, at = {}, [], 0
    for name, a in tensors.items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    h = json.dumps(head).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return str(folder)


def read_model(folder):
    cfg = json.load(open(f"{folder}/config.json"))
    raw = open(f"{folder}/model.safetensors", "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    out = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        u = np.frombuffer(raw[8 + n + lo:8 + n + hi], "<u2").astype(np.uint32) << 16
        out[name] = u.view(np.float32).reshape(t["shape"]).astype(np.float64)
    return cfg, out


# ---- small pieces ------------------------------------------------------------------------------------------------
def exact(a):
    return a


def to_bf16(a):
    return bf16_round(np.asarray(a, np.float32)).astype(np.float64)


def rms(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rotary_frequencies(rot):
    """(frequency per pair, factor on cos and sin) of a rotation entry: base, dims and, if given, a YaRN scaling."""
    dims, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def where(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(where(s["fast"])), 0)
    hi = min(math.ceil(where(s["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T][..., n]: dimension 2i is paired with 2i+1 over the first rot.dims dimensions."""
    f, m = rotary_frequencies(rot)
    a = np.asarray(positions, np.float64)[:, None] * f[None, :]
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (len(f),)
    c, s = (np.cos(a) * m).reshape(shape), (np.sin(a) * m).reshape(shape)
    out = x.copy()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * c - v * s
    out[..., 1:rot["dims"]:2] = v * c + u * s
    return out


# ---- mixers ------------------------------------------------------------------------------------------------------
def latent_attention(h, W, m, eps, start=0, cache=None, rnd=exact):
    """h [T][width] at positions start..; W(name) gives the mixer's tensors. cache: (latents, rotated keys) of the
    positions before `start`. Returns (output, new cache)."""
    T, H, D, R, VD = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = np.arange(start, start + T)
    h = rnd(h)
    q = (rnd(rms(h @ W("dq").T, W("dq.norm"), eps)) @ W("uq").T).reshape(T, H, D + R)
    qn, qr = rnd(q[..., :D]), rnd(rotate(q[..., D:], pos, m["rot"]))
    low = h @ W("dkv").T
    c = rnd(rms(low[:, :m["kv_rank"]], W("dkv.norm"), eps))
    kr = rnd(rotate(low[:, m["kv_rank"]:], pos, m["rot"]))
    if cache is not None:
        c, kr = np.concatenate([cache[0], c]), np.concatenate([cache[1], kr])
    N = len(c)
    kn = rnd(c @ W("uk").T).reshape(N, H, D)
    v = rnd(c @ W("uv").T).reshape(N, H, VD)
    out = np.empty((T, H, VD))
    window = (m.get("mask") or {}).get("size")
    for t in range(T):
        p = start + t
        lo = max(0, p - window + 1) if window else 0
        s = (np.einsum("hd,jhd->hj", qn[t], kn[lo:p + 1]) + qr[t] @ kr[lo:p + 1].T) * m["scale"]
        e = np.exp(s - s.max(axis=1, keepdims=True))
        e /= e.sum(axis=1, keepdims=True)
        out[t] = np.einsum("hj,jhv->hv", rnd(e), v[lo:p + 1])
    o = out.reshape(T, H * VD) * sigmoid(h @ W("g").T)
    return rnd(o) @ W("o").T, (c, kr)


def wkv_recurrence(r, k, v, w, u, S):
    """r, k, v, w [T][heads][dim], u [heads][dim], S [heads][key][value]. Returns (o [T][heads][dim], S after)."""
    S = S.copy()
    out = np.empty_like(v)
    for t in range(len(r)):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hk,hkv->hv", r[t], S + u[:, :, None] * kv)
        S = w[t][:, :, None] * S + kv
    return out, S


def wkv(h, W, m, eps, state=None, rnd=exact):
    """state: (last h, S). Returns (output, new state)."""
    T, H, D = len(h), m["heads"], m["dim"]
    last, S = state if state is not None else (np.zeros(h.shape[1]), np.zeros((H, D, D)))
    prev = np.concatenate([last[None], h[:-1]])
    mix = {s: rnd(h + (prev - h) * W("mu." + s)) for s in "rkvgw"}
    r, k, v = ((mix[s] @ W(s).T).reshape(T, H, D) for s in "rkv")
    gate = silu(mix["g"] @ W("g").T)
    w = np.exp(-np.exp(rnd(np.tanh(mix["w"] @ W("w1").T)) @ W("w2").T + W("w0"))).reshape(T, H, D)
    o, S = wkv_recurrence(r, k, v, w, W("u"), S)
    o = o / np.sqrt(np.mean(o * o, axis=-1, keepdims=True) + eps)
    return rnd(o.reshape(T, H * D) * W("norm") * gate) @ W("o").T, (h[-1], S)


def softcap(z, cap):
    return z if not cap else cap * np.tanh(z / cap)


def seen_keys(p, mask):
    """First key position that the query at position p sees, by a chunked mask (blocks of `size` positions)."""
    return p // mask["size"] * mask["size"] if mask else 0


def sink_weights(s):
    """Softmax over the last axis with one more term, exp(0), in the denominator."""
    top = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - top)
    return e / (np.exp(-top) + e.sum(axis=-1, keepdims=True))


def shared_kv_attention(h, W, m, start=0, cache=None, rnd=exact):
    """Grouped-query attention whose values are its unrotated keys; chunked mask, capped scores, sink. cache: (unrotated keys,
    rotated keys) of the positions before `start`, each [positions][kv_heads][dim]. Returns (output, new cache)."""
    T, H, G, D = len(h), m["heads"], m["kv_heads"], m["dim"]
    pos = np.arange(start, start + T)
    h = rnd(h)
    q = rnd(rotate((h @ W("q").T).reshape(T, H, D), pos, m["rot"]))
    raw = (h @ W("k").T).reshape(T, G, D)
    v, k = rnd(raw), rnd(rotate(raw, pos, m["rot"]))
    if cache is not None:
        v, k = np.concatenate([cache[0], v]), np.concatenate([cache[1], k])
    out = np.empty((T, H, D))
    for t in range(T):
        p = start + t
        lo = seen_keys(p, m.get("mask"))
        for x in range(H):
            g = x // (H // G)
            s = softcap(k[lo:p + 1, g] @ q[t, x] * m["scale"], m.get("softcap"))
            out[t, x] = rnd(sink_weights(s)) @ v[lo:p + 1, g]
    return rnd(out.reshape(T, H * D)) @ W("o").T, (v, k)


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(x, w, b, before):
    """x [T][channels]; w [channels][taps], last column = the current token; before [taps - 1][channels] = earlier inputs."""
    taps = w.shape[1]
    full = np.concatenate([before, x])
    return sum(full[k:k + len(x)] * w[:, k] for k in range(taps)) + b, full[len(full) - taps + 1:]


def gated_recurrence(u, r, i, lam, S):
    """Per channel: a = exp(-8 r softplus(lam)), S <- a S + sqrt(1 - a^2) i u. All [T][channels]. Returns (S of every token, S after)."""
    log_a = -8.0 * r * np.logaddexp(0.0, lam)
    a, x = np.exp(log_a), np.sqrt(-np.expm1(2 * log_a)) * i * u
    out = np.empty_like(u)
    for t in range(len(u)):
        S = a[t] * S + x[t]
        out[t] = S
    return out, S


def rglru(h, W, m, state=None, rnd=exact):
    """state: (last taps - 1 inputs of the convolution, S). Returns (output, new state)."""
    T, N, B = len(h), m["width"], m["blocks"]
    before, S = state if state is not None else (np.zeros((m["conv"] - 1, N)), np.zeros(N))
    h = rnd(h)
    y = gelu_tanh(h @ W("y").T + W("y.b"))
    u, before = causal_conv(h @ W("x").T + W("x.b"), W("conv"), W("conv.b"), before)
    ub = u.reshape(T, B, N // B)
    r = sigmoid(np.einsum("boi,tbi->tbo", W("ra"), ub) + W("ra.b")).reshape(T, N)
    i = sigmoid(np.einsum("boi,tbi->tbo", W("ri"), ub) + W("ri.b")).reshape(T, N)
    out, S = gated_recurrence(u, r, i, W("lam"), S)
    return rnd(out * y) @ W("o").T, (before, S)


def dense_relu(h, W, rnd=exact):
    h = rnd(h)
    return rnd(np.maximum(h @ W("gate").T, 0) * (h @ W("up").T)) @ W("down").T


def dense_silu(h, W, rnd=exact):
    h = rnd(h)
    return rnd(silu(h @ W("gate").T) * (h @ W("up").T)) @ W("down").T


# ---- model -------------------------------------------------------------------------------------------------------
def layer_runs(cfg):
    """Layer index of every run, in order (a looped stretch counts once per pass)."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


class PlainModel:
    """Nezolix (each sublayer normalised before and after, own head) or Pizilix (normalised before, norm weights stored around
    zero, embedding added again before every further pass of a loop, tied and capped head)."""

    def __init__(self, cfg, tensors, rnd=exact):
        self.rnd = rnd
        self.cfg, self.t = cfg, {k: np.asarray(v, np.float64) for k, v in tensors.items()}
        self.reset()

    def reset(self):
        self.pos, self.state = 0, [None] * len(layer_runs(self.cfg))

    def run(self, tokens, trace=None):
        """The next tokens of the sequence; returns their logits [T][vocab]."""
        x = (self.run_pizilix if self.cfg["architecture"] == "Pizilix" else self.run_nezolix)(np.asarray(tokens), trace)
        self.pos += len(x)
        return x

    def run_nezolix(self, tokens, trace):
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        x = self.t["embed"][tokens] * cfg["embedding"]["scale"]
        for i, l in enumerate(layer_runs(cfg)):
            lay = cfg["layers"][l]
            N = lambda s: self.t[f"l{l}.{s}"]
            W = lambda s: self.t[f"l{l}.mix.{s}"]
            h = rms(x, N("norm1"), eps)
            if lay["type"] == "wkv":
                y, self.state[i] = wkv(h, W, lay["mixer"], eps, self.state[i], self.rnd)
            else:
                y, self.state[i] = latent_attention(h, W, lay["mixer"], eps, self.pos, self.state[i], self.rnd)
            x = x + rms(y, N("norm1b"), eps)
            if lay.get("mlp"):
                y = dense_relu(rms(x, N("norm2"), eps), lambda s: self.t[f"l{l}.mlp.{s}"], self.rnd)
                x = x + rms(y, N("norm2b"), eps)
            if trace is not None:
                trace.append(x.copy())
        return self.rnd(rms(x, self.t["final.norm"], eps)) @ self.t["head"].T

    def run_pizilix(self, tokens, trace):
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        x = first = self.t["embed"][tokens]
        runs, loop = layer_runs(cfg), cfg.get("loop")
        again = {loop["start"] + n * (loop["stop"] - loop["start"]) for n in range(1, loop["times"])} if loop else set()
        for i, l in enumerate(runs):
            lay = cfg["layers"][l]
            W = lambda s: self.t[f"l{l}.mix.{s}"]
            norm = lambda s: rms(x, 1 + self.t[f"l{l}.{s}"], eps)
            if i in again:
                x = x + first
            if lay["type"] == "rglru":
                y, self.state[i] = rglru(norm("norm1"), W, lay["mixer"], self.state[i], self.rnd)
            else:
                y, self.state[i] = shared_kv_attention(norm("norm1"), W, lay["mixer"], self.pos, self.state[i], self.rnd)
            x = x + y
            if lay.get("mlp"):
                x = x + dense_silu(norm("norm2"), lambda s: self.t[f"l{l}.mlp.{s}"], self.rnd)
            if trace is not None:
                trace.append(x.copy())
        return softcap(self.rnd(rms(x, 1 + self.t["final.norm"], eps)) @ self.t["embed"].T, cfg.get("logit_softcap"))


def greedy(cfg, tensors, prompt, steps):
    """(ids, smallest gap between the two largest logits over the steps)."""
    m = PlainModel(cfg, tensors)
    l = m.run(prompt)[-1]
    ids, gap = [], math.inf
    for _ in range(steps):
        top = np.sort(l)[-2:]
        gap = min(gap, float(top[1] - top[0]))
        ids.append(int(l.argmax()))
        l = m.run([ids[-1]])[-1]
    return ids, gap
