"""Fezozen in plain numpy float64, one function per mechanism, whole sequences only.

It shares nothing with the package: it reads a config.json object and a {tensor name: array}
dictionary and walks a sequence from its first token.  Attention builds every score of every query
against every key, from keys and values expanded per head, and masks afterwards; a routed token
runs its experts one by one, each on the token's input times its weight.

Notation: T tokens, W model width; ``h`` [T, W] is a sublayer's normed input; a matrix M stored
[out, in] is applied as ``h @ M.T``.
"""
import math

import numpy as np


# ---- small functions
def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def capped(z, cap):
    """cap tanh(z / cap); no cap (None or 0): z."""
    return cap * np.tanh(z / cap) if cap else z


def unit_rms(x, eps):
    """x divided by sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


# ---- rotation
def frequencies(base, dims, scaling):
    """([dims / 2] angles per position, the factor on the cosines and sines).  With ``scaling`` the
    frequencies that turn fewer than ``slow`` times over ``original`` positions are divided by
    ``factor``, those that turn more than ``fast`` times stay, and the ones between are blended
    linearly along their index."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0

    def place(turns):                # the (real) index of the frequency that makes ``turns`` turns
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(place(scaling["fast"])), 0)
    last = min(math.ceil(place(scaling["slow"])), dims - 1)
    mix = np.array([min(max((i - first) / max(last - first, 0.001), 0.0), 1.0) for i in range(dims // 2)])
    return f / scaling["factor"] * mix + f * (1.0 - mix), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, positions, rot):
    """x [T, H, D]: dimensions 2i and 2i + 1 below ``rot.dims`` are a pair that turns by position *
    frequency i; dimensions from ``rot.dims`` on pass unchanged."""
    dims = int(rot["dims"]) if rot else 0
    if dims == 0:
        return x
    freq, stretch = frequencies(rot["base"], dims, rot.get("scaling"))
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    c, s = stretch * np.cos(ang)[:, None, :], stretch * np.sin(ang)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.copy()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ---- softmax attention
def visible(T, window):
    """[T, T]: whether query i sees key j: itself and all before it, or itself and the window - 1 before it."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < window) if window else True)


def masked_attention(q, k, v, scale, cap, window):
    """q [T, H, D], k [T, G, D], v [T, G, Vd] of one sequence from its start; head h reads kv head
    h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = visible(T, window)
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, capped((q[:, h] @ k[:, g].T) * scale, cap), -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e / e.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def window_of(m):
    return (m.get("mask") or {}).get("size")


def heads_of(x, heads):
    return x.reshape(x.shape[0], heads, -1)


def biased_attention_mixer(h, P, m, eps):
    """'attention': biases, a partial and stretched rotation, capped scores, every key before."""
    pos = np.arange(h.shape[0])
    q = rotate_pairs(heads_of(h @ P["q"].T + P["q.b"], m["heads"]), pos, m["rot"])
    k = rotate_pairs(heads_of(h @ P["k"].T + P["k.b"], m["kv_heads"]), pos, m["rot"])
    v = heads_of(h @ P["v"].T + P["v.b"], m["kv_heads"])
    o = masked_attention(q, k, v, m["scale"], m.get("softcap"), window_of(m))
    return o.reshape(h.shape[0], -1) @ P["o"].T


def unit_attention_mixer(h, P, m, eps):
    """'attention_2': no biases, q and k of every head divided by their root mean square after the
    rotation, a window."""
    pos = np.arange(h.shape[0])
    q = unit_rms(rotate_pairs(heads_of(h @ P["q"].T, m["heads"]), pos, m["rot"]), eps)
    k = unit_rms(rotate_pairs(heads_of(h @ P["k"].T, m["kv_heads"]), pos, m["rot"]), eps)
    v = heads_of(h @ P["v"].T, m["kv_heads"])
    o = masked_attention(q, k, v, m["scale"], m.get("softcap"), window_of(m))
    return o.reshape(h.shape[0], -1) @ P["o"].T


def latent_attention_mixer(h, P, m, eps):
    """Keys and values of a head are expansions of one normed latent, beside a rotated key part that all
    heads share; a window; a sigmoid gate on every number of the heads' outputs."""
    T = h.shape[0]
    H, D, R, Vd, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = heads_of(h @ P["q"].T, H)
    q = np.concatenate([q[..., :D], rotate_pairs(q[..., D:], pos, m.get("rot"))], axis=-1)
    down = h @ P["dkv"].T
    c = rms_norm(down[:, :rank], P["dkv.norm"], eps)
    shared = rotate_pairs(down[:, None, rank:], pos, m.get("rot"))                       # [T, 1, R]
    k = np.concatenate([(c @ P["uk"].T).reshape(T, H, D), np.repeat(shared, H, axis=1)], axis=-1)
    v = (c @ P["uv"].T).reshape(T, H, Vd)
    o = masked_attention(q, k, v, m["scale"], None, window_of(m)).reshape(T, H * Vd)
    return (o * output_gate(h, P["g"])) @ P["o"].T


def output_gate(h, g):
    return sigmoid(h @ g.T)


# ---- feed-forward
def choose(z, top):
    """z [experts]: the ``top`` largest sigmoid(z) (the lower index first among equals) and those scores."""
    s = sigmoid(z)
    order = sorted(range(len(z)), key=lambda e: (-s[e], e))[:top]
    return order, s[order]


def expert(x, P, e):
    return (silu(x @ P[f"e{e}.gate"].T) * (x @ P[f"e{e}.up"].T)) @ P[f"e{e}.down"].T


def routed_ffn(h, P, mlp):
    """Every chosen expert sees the token's input times its score."""
    out = np.zeros((h.shape[0], P["e0.down"].shape[0]))
    z = h @ P["router"].T
    for t in range(h.shape[0]):
        for e, s in zip(*choose(z[t], mlp["router"]["top"])):
            out[t] += expert(s * h[t], P, e)
    return out


# ---- the model
def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


MIXERS = {"attention": biased_attention_mixer, "attention_2": unit_attention_mixer, "latent_attention": latent_attention_mixer}


def tensors_of(config, i):
    """The layer whose tensors layer i runs."""
    while "weights_of" in config["layers"][i]:
        i = config["layers"][i]["weights_of"]
    return i


def forward(config, tensors, tokens, return_layers=False):
    """Logits [T, vocab] of a whole sequence; with ``return_layers`` also the residual stream after
    every layer."""
    eps = config["norm"]["eps"]
    x = tensors["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    layers = []
    for i, layer in enumerate(config["layers"]):
        L = f"l{tensors_of(config, i)}."
        y = MIXERS[layer["type"]](rms_norm(x, tensors[L + "norm1"], eps), sub(tensors, L + "mix."), layer["mixer"], eps)
        x = x + rms_norm(y, tensors[L + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = routed_ffn(rms_norm(x, tensors[L + "norm2"], eps), sub(tensors, L + "mlp."), layer["mlp"])
            x = x + rms_norm(y, tensors[L + "norm2b"], eps)
        layers.append(x.copy())
    logits = rms_norm(x, tensors["final.norm"], eps) @ tensors["head"].T
    return (logits, layers) if return_layers else logits


def load_folder(folder):
    """(config.json object, {tensor name: float64 array}) of a model folder; the safetensors file
    is read here, by hand: 8 bytes of header length, the JSON header, then the data."""
    import json
    import os
    import struct
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    tensors = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw = data[lo:hi]
        if info["dtype"] == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        elif info["dtype"] == "F32":
            a = np.frombuffer(raw, dtype="<f4")
        else:
            raise ValueError(f"{name}: dtype {info['dtype']}")
        tensors[name] = a.astype(np.float64).reshape(info["shape"])
    return config, tensors


def generate(config, tensors, prompt, n, stop=()):
    """Greedy continuation: (tokens, reason); the first largest logit wins; a stop token ends the
    run and is the last token returned."""
    toks, out = list(prompt), []
    for _ in range(n):
        nxt = int(np.argmax(forward(config, tensors, toks)[-1]))
        out.append(nxt)
        if nxt in stop:
            return out, "stop"
        toks.append(nxt)
    return out, "length"
