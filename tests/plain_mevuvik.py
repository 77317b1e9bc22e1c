"""Mevuvik in plain numpy float64, one function per mechanism, whole sequences only.

It shares nothing with the package: it reads a config.json object and a {tensor name: array}
dictionary and walks a sequence from its first token.  Attention builds every score of a query
against every key before it, from keys and values expanded per head; the recurrent mixer runs token
by token exactly as its update is written.

Notation: T tokens, W model width; ``h`` [T, W] is a sublayer's normed input; a matrix M stored
[out, in] is applied as ``h @ M.T``.
"""
import math

import numpy as np


# ---- small functions
def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def capped(z, cap):
    """cap tanh(z / cap); no cap (None or 0): z."""
    return cap * np.tanh(z / cap) if cap else z


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def rms_scale(x, eps):
    """x divided by sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_scale(x, eps) * w


def number_norm(x, g, eps):
    """The model's norm: one number for all coordinates."""
    return rms_scale(x, eps) * float(np.asarray(g).reshape(()))


# ---- rotation
def rotate_half(x, positions, base, dims):
    """x [T, H, D]: dimension i < dims/2 pairs with dimension i + dims/2 and the pair turns by
    positions * base^(-2i/dims); dimensions from ``dims`` on pass unchanged."""
    half = dims // 2
    if half == 0:
        return x
    freq = np.array([base ** (-2.0 * i / dims) for i in range(half)])
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    out = x.copy()
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


# ---- softmax attention
def causal_attention(q, k, v, scale):
    """q [T, H, D], k [T, G, D], v [T, G, Vd] of one sequence from its start; head h reads kv head
    h // (H / G)."""
    T, H, _ = q.shape
    G, vd = k.shape[1], v.shape[2]
    out = np.zeros((T, H, vd))
    for a in range(T):
        for h in range(H):
            g = h // (H // G)
            s = (k[:a + 1, g] @ q[a, h]) * scale
            e = np.exp(s - s.max())
            out[a, h] = (e / e.sum()) @ v[:a + 1, g]
    return out


def latent_attention_mixer(h, P, m, eps):
    """Queries and keys/values both pass a normed latent; the keys of a head are its expansion of the
    latent beside one rotated part that all heads share."""
    T = h.shape[0]
    H, D, R, Vd, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    cq = rms_norm(h @ P["dq"].T, P["dq.norm"], eps)
    q = (cq @ P["uq"].T).reshape(T, H, D + R)
    down = h @ P["dkv"].T
    c = rms_norm(down[:, :rank], P["dkv.norm"], eps)
    shared = rotate_half(down[:, None, rank:], pos, rot["base"], rot["dims"])        # [T, 1, R]
    q = np.concatenate([q[..., :D], rotate_half(q[..., D:], pos, rot["base"], rot["dims"])], axis=-1)
    k = np.concatenate([(c @ P["uk"].T).reshape(T, H, D), np.repeat(shared, H, axis=1)], axis=-1)
    v = (c @ P["uv"].T).reshape(T, H, Vd)
    return causal_attention(q, k, v, m["scale"]).reshape(T, H * Vd) @ P["o"].T


def head_gated_attention_mixer(h, P, m):
    """The left branch: grouped attention without positions, one sigmoid gate per head."""
    T = h.shape[0]
    H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ P["q"].T).reshape(T, H, D)
    k = (h @ P["k"].T).reshape(T, G, D)
    v = (h @ P["v"].T).reshape(T, G, Vd)
    o = causal_attention(q, k, v, m["scale"]) * sigmoid(h @ P["g"].T)[:, :, None]
    return o.reshape(T, H * Vd) @ P["o"].T


# ---- matrix memory
def matrix_memory_scan(q, k, v, log_in, log_forget, state=None):
    """q, k [T, H, D], v [T, H, Vd], log_in, log_forget [T, H].  Per head and token, with m a running
    maximum (0 at the start) that keeps the exponentials small:
    m' = max(f + m, i); S <- e^(f + m - m') S + e^(i - m') k v^T; n the same with k alone;
    o = S^T q / (max(|n . q|, e^(-m')) + 1e-6).  Returns (o, (S, n, m))."""
    T, H, D = q.shape
    Vd = v.shape[2]
    if state is None:
        state = (np.zeros((H, D, Vd)), np.zeros((H, D)), np.zeros(H))
    S, n, m = (a.copy() for a in state)
    o = np.zeros((T, H, Vd))
    for t in range(T):
        for h in range(H):
            i, f = log_in[t, h], log_forget[t, h]
            new = max(f + m[h], i)
            keep, write = math.exp(f + m[h] - new), math.exp(i - new)
            S[h] = keep * S[h] + write * np.outer(k[t, h], v[t, h])
            n[h] = keep * n[h] + write * k[t, h]
            m[h] = new
            o[t, h] = (S[h].T @ q[t, h]) / (max(abs(n[h] @ q[t, h]), math.exp(-new)) + 1e-6)
    return o, (S, n, m)


def matrix_memory_mixer(h, P, m, eps):
    """The right branch."""
    T = h.shape[0]
    H, D, Vd, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ P["q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ P["k"].T).reshape(T, H, D)
    v = (h @ P["v"].T).reshape(T, H, Vd)
    log_in = capped(h @ P["i"].T + P["i.b"], cap)
    log_forget = log_sigmoid(capped(h @ P["f"].T + P["f.b"], cap))
    o, _ = matrix_memory_scan(q, k, v, log_in, log_forget)
    o = rms_scale(o, eps).reshape(T, H * Vd) * P["norm"] * sigmoid(h @ P["g"].T)
    return o @ P["o"].T


def two_branch_mixer(h, P, m, eps):
    left = head_gated_attention_mixer(h, sub(P, "left."), m["left"])
    right = matrix_memory_mixer(h, sub(P, "right."), m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


# ---- feed-forward
def dense_ffn(h, P):
    return relu_squared(h @ P["up"].T) @ P["down"].T


def route_sigmoid(z, correction, top, scale):
    """z [experts]: s = sigmoid(z); the ``top`` largest s + correction are chosen (the lower index
    first among equals); their weights are s over the chosen ones' sum (+ 1e-20), times scale."""
    s = sigmoid(z)
    choice = s + correction
    order = sorted(range(len(z)), key=lambda e: (-choice[e], e))[:top]
    return order, s[order] / (s[order].sum() + 1e-20) * scale


def routed_ffn(h, P, mlp):
    out = np.zeros((h.shape[0], P["e0.down"].shape[0]))
    z = h @ P["router"].T
    r = mlp["router"]
    for t in range(h.shape[0]):
        chosen, weights = route_sigmoid(z[t], P["correction"], r["top"], r["scale"])
        for e, wt in zip(chosen, weights):
            out[t] += wt * (relu_squared(h[t] @ P[f"e{e}.up"].T) @ P[f"e{e}.down"].T)
    return out


# ---- the model
def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


MIXERS = {"latent_attention": latent_attention_mixer, "parallel": two_branch_mixer}


def runs(config):
    """[(layer, loop pass that starts with this run or None)] in the order of the runs."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, None) for i in range(start)]
    for t in range(times):
        out += [(i, t if i == start else None) for i in range(start, stop)]
    return out + [(i, None) for i in range(stop, n)]


def forward(config, tensors, tokens, return_layers=False):
    """Logits [T, vocab] of a whole sequence; with ``return_layers`` also the residual stream after
    every run of a layer."""
    tokens = np.asarray(tokens)
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = number_norm(tensors["embed"][tokens], tensors["embed.norm"], eps)
    layers = []
    for i, loop_pass in runs(config):
        if loop_pass is not None:
            x = x + tensors["loop.step"][loop_pass]
        layer = config["layers"][i]
        h = number_norm(x, tensors[f"l{i}.norm1"], eps)
        x = x + m * (MIXERS[layer["type"]](h, sub(tensors, f"l{i}.mix."), layer["mixer"], eps) * tensors[f"l{i}.ls1"])
        mlp = layer.get("mlp")
        if mlp is not None:
            h, P = number_norm(x, tensors[f"l{i}.norm2"], eps), sub(tensors, f"l{i}.mlp.")
            y = dense_ffn(h, P) if mlp["kind"] == "dense" else routed_ffn(h, P, mlp)
            x = x + m * (y * tensors[f"l{i}.ls2"])
        layers.append(x.copy())
    logits = capped(number_norm(x, tensors["final.norm"], eps) @ tensors["head"].T, config.get("logit_softcap"))
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
