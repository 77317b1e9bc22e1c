"""Fezozen: configuration, plan, tensor names.

A decoder with an RMS norm on both sides of every sublayer: x += norm1b(mixer(norm1(x))), then
x += norm2b(ffn(norm2(x))).  The configuration lists the layers one by one; a layer with
``weights_of: j`` runs layer j's tensors (j before or after it) with a cache of its own.  Three mixers,
all softmax attention with positions turned in pairs (dims 2i and 2i + 1):

* ``attention``: every key before; biases on q, k and v; the first ``rot.dims`` dims of every head
  turned with frequencies blended along the index and stretched cosines and sines (``rot.scaling``);
  capped scores.
* ``attention_2``: a sliding window; no biases; q and k of every head divided by their root mean square
  after the rotation, without weights.
* ``latent_attention``: keys and values expanded from one normed latent per position, beside a rotated
  key part that all heads share; a sliding window; a sigmoid gate on every number of the heads' outputs.

The feed-forward routes every token to ``top`` of ``experts`` small gated layers (SiLU) by sigmoid scores
that are not renormalized, and a score multiplies its expert's input: the sum of expert(score * h); or
there is none (``mlp: null``).

config.json::

    {"architecture": "Fezozen", "vocab": V, "width": W, "embedding": {"scale": s}, "norm": {"eps": e},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap": null | c,
                           "rot": {"base", "dims", "scaling": null | {"factor", "original", "fast", "slow"}}},
                 "mlp": null | {"kind": "moe", "router": {"experts", "top"}, "expert": {"ff"}}},
                {"type": "attention_2",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}, "rot": {...}}, "mlp": ...},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "mask": {"size"}, "rot": {...}},
                 "mlp": ...},
                {"type": ..., "weights_of": j, ...}, ...]}

Tensors: ``embed``, ``l<i>.{norm1,norm1b,norm2,norm2b}``, ``final.norm``, ``head``;
``l<i>.mix.{q,q.b,k,k.b,v,v.b,o}`` (attention), ``l<i>.mix.{q,k,v,o}`` (attention_2),
``l<i>.mix.{q,dkv,dkv.norm,uk,uv,g,o}`` (latent_attention); ``l<i>.mlp.{router,e<j>.gate,e<j>.up,e<j>.down}``.

This module is all that knows the architecture: it turns the configuration into a ``ModelPlan`` of
generic parts (``sandwich`` block, ``capped_attention``, ``latent_attention``, ``moe``, ``rmsnorm``, ``rotary``).
"""
from __future__ import annotations

import dataclasses
from typing import Tuple

from ..config.base import ConfigError, ModelConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

MIXERS = ("attention", "attention_2", "latent_attention")


def _num(problems, where, obj, name, kind=int, allow_zero=False, optional=False, signed=False):
    v = obj.get(name) if isinstance(obj, dict) else None
    if v is None and optional:
        return None
    if kind is int and isinstance(v, float) and v.is_integer():
        v = int(v)                                   # a count written as 256.0
    ok = isinstance(v, int) and not isinstance(v, bool) if kind is int else (
        isinstance(v, (int, float)) and not isinstance(v, bool))
    if not ok:
        problems.append(f"{where}.{name}: expected {'an integer' if kind is int else 'a number'}, got {v!r}")
        return None
    if not signed and (v < 0 or (v == 0 and not allow_zero)):
        problems.append(f"{where}.{name}: must be positive, got {v!r}")
        return None
    return kind(v)


def _check_mask_and_rotation(p, w, m, turned, what):
    """``turned``: the width of the vector that is rotated, ``what`` its name in the configuration."""
    if m.get("mask") is not None:
        _num(p, w + ".mask", m["mask"], "size")
    rot = m.get("rot")
    if rot is None:
        return
    dims = _num(p, w + ".rot", rot, "dims", allow_zero=True)
    if not dims:
        return
    base = _num(p, w + ".rot", rot, "base", float)
    if turned is not None and (dims % 2 or dims > turned):
        p.append(f"{w}.rot.dims: {dims} is odd or more than {what} ({turned})")
    scaling = rot.get("scaling")
    if scaling is not None:
        for name in ("factor", "original", "fast", "slow"):
            _num(p, w + ".rot.scaling", scaling, name, float)
        if base is not None and base <= 1.0:
            p.append(f"{w}.rot.base: {base} must be above 1 beside a scaling")


def _check_attention(p, w, m):
    heads, g = _num(p, w, m, "heads"), _num(p, w, m, "kv_heads")
    if heads and g and heads % g:
        p.append(f"{w}: {heads} heads are not a multiple of {g} kv_heads")
    dim = _num(p, w, m, "dim")
    _num(p, w, m, "vdim")
    _num(p, w, m, "scale", float, signed=True)
    _num(p, w, m, "softcap", float, allow_zero=True, optional=True)
    _check_mask_and_rotation(p, w, m, dim, "dim")


def _check_latent(p, w, m):
    for name in ("heads", "vdim", "kv_rank"):
        _num(p, w, m, name)
    dim, rd = _num(p, w, m, "dim", allow_zero=True), _num(p, w, m, "rot_dim", allow_zero=True)
    if dim == 0 and rd == 0:
        p.append(f"{w}: dim and rot_dim are both 0")
    _num(p, w, m, "scale", float, signed=True)
    _check_mask_and_rotation(p, w, m, rd, "rot_dim")


def _check_mlp(p, w, mlp):
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        got = mlp.get("kind") if isinstance(mlp, dict) else mlp
        p.append(f"{w}.kind: unknown feed-forward {got!r} (known: moe)")
        return
    experts, top = _num(p, w + ".router", mlp.get("router"), "experts"), _num(p, w + ".router", mlp.get("router"), "top")
    if experts and top and top > experts:
        p.append(f"{w}.router.top: {top} of {experts} experts")
    _num(p, w + ".expert", mlp.get("expert"), "ff")


def _check_owner(p, w, layers, i, kind):
    j = layers[i]["weights_of"]
    if not isinstance(j, int) or isinstance(j, bool) or not 0 <= j < len(layers) or j == i or not isinstance(layers[j], dict):
        p.append(f"{w}.weights_of: {j!r} is not another layer")
        return
    if layers[j].get("type") != kind:
        p.append(f"{w}.weights_of: layer {j} is a {layers[j].get('type')!r} layer, this one {kind!r}")
        return
    at, steps = j, 0                                 # the chain of owners must end at a layer with tensors of its own
    while isinstance(layers[at], dict) and "weights_of" in layers[at]:
        at, steps = layers[at]["weights_of"], steps + 1
        if not isinstance(at, int) or isinstance(at, bool) or not 0 <= at < len(layers):
            return                                   # reported at the layer that says so
        if steps > len(layers):
            p.append(f"{w}.weights_of: the layers that share tensors name one another in a circle")
            return


@dataclasses.dataclass(frozen=True)
class FezozenConfig(ModelConfig):
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    #: one entry per layer, as config.json lists them (checked; plain dicts)
    layers: Tuple[dict, ...]

    @classmethod
    def from_dict(cls, raw):
        if not isinstance(raw, dict):
            raise ConfigError("config.json: the top level must be an object")
        p = []
        vocab = _num(p, "config", raw, "vocab")
        width = _num(p, "config", raw, "width")
        emb = _num(p, "embedding", raw.get("embedding"), "scale", float, signed=True)
        if emb == 0.0:
            p.append("embedding.scale: must not be 0")
        eps = _num(p, "norm", raw.get("norm"), "eps", float, allow_zero=True)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            p.append("layers: expected a list of at least one layer")
            layers = []
        for i, layer in enumerate(layers):
            w = f"layers[{i}]"
            if not isinstance(layer, dict):
                p.append(f"{w}: expected an object")
                continue
            kind, m = layer.get("type"), layer.get("mixer")
            if kind not in MIXERS:
                p.append(f"{w}.type: unknown mixer {kind!r} (known: {', '.join(MIXERS)})")
                continue
            if not isinstance(m, dict):
                p.append(f"{w}.mixer: expected an object")
                continue
            (_check_latent if kind == "latent_attention" else _check_attention)(p, w + ".mixer", m)
            if layer.get("mlp") is not None:
                _check_mlp(p, w + ".mlp", layer["mlp"])
            if layer.get("weights_of") is not None:
                _check_owner(p, w, layers, i, kind)
        if p:
            raise ConfigError("config.json: " + "; ".join(p))
        # a null weights_of is the same as none
        layers = tuple({k: v for k, v in layer.items() if k != "weights_of" or v is not None} for layer in layers)
        return cls(vocab=vocab, width=width, embedding_scale=emb, norm_eps=eps, layers=layers)

    def to_dict(self):
        return {"architecture": "Fezozen", "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
                "layers": [dict(layer) for layer in self.layers]}


def owner(cfg, i: int) -> int:
    """The layer whose tensors layer ``i`` runs: itself, or the end of its chain of ``weights_of``."""
    while "weights_of" in cfg.layers[i]:
        i = int(cfg.layers[i]["weights_of"])
    return i


def _window(m):
    mask = m.get("mask")
    return int(mask["size"]) if mask else None


def _rotation(m, width):
    rot = m.get("rot") or {}
    dims = int(rot.get("dims") or 0)
    if not dims:
        return None
    return PartSpec("rotary", {"head_dim": width, "rotary_dim": dims, "theta": float(rot["base"]), "layout": "interleaved",
                               "scaling": rot.get("scaling")})


def _attention_spec(cfg, kind, m, prefix) -> PartSpec:
    names = {k: prefix + k for k in ("q", "k", "v", "o")}
    bias = kind == "attention"
    if bias:
        names.update({f"{k}_bias": f"{prefix}{k}.b" for k in ("q", "k", "v")})
    return PartSpec("capped_attention", {
        "hidden_size": cfg.width, "heads": int(m["heads"]), "kv_heads": int(m["kv_heads"]), "dim": int(m["dim"]),
        "vdim": int(m["vdim"]), "bias": bias, "scale": float(m["scale"]), "softcap": float(m.get("softcap") or 0.0),
        "window": _window(m), "qk_unit": cfg.norm_eps if kind == "attention_2" else None,
        "position": _rotation(m, int(m["dim"]))}, names)


def _latent_spec(cfg, m, prefix) -> PartSpec:
    names = {k: prefix + k for k in ("q", "dkv", "uk", "uv", "g", "o")}
    names["dkv_norm"] = prefix + "dkv.norm"
    return PartSpec("latent_attention", {
        "hidden_size": cfg.width, "num_heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": int(m["rot_dim"]),
        "vdim": int(m["vdim"]), "rank": int(m["kv_rank"]), "scale": float(m["scale"]), "norm_eps": cfg.norm_eps,
        "gate": "channel", "window": _window(m), "position": _rotation(m, int(m["rot_dim"]))}, names)


def _ffn_spec(cfg, mlp, prefix) -> PartSpec:
    experts = int(mlp["router"]["experts"])
    names = {"router": prefix + "router"}
    names.update({f"e{e}.{part}": f"{prefix}e{e}.{part}" for e in range(experts) for part in ("gate", "up", "down")})
    return PartSpec("moe", {"hidden_size": cfg.width, "experts": experts, "top": int(mlp["router"]["top"]),
                            "ff": int(mlp["expert"]["ff"]), "limit": None, "alpha": 1.0, "shift": 0.0, "router_bias": False,
                            "routing": "sigmoid_raw", "weigh": "input", "shared": None}, names)


def build_plan(cfg: FezozenConfig, names=None) -> ModelPlan:
    def norm(name, after_sublayer=False):
        params = {"size": cfg.width, "eps": cfg.norm_eps}
        return PartSpec("rmsnorm", {**params, "after_sublayer": True} if after_sublayer else params, {"weight": name})

    layers, place, ignored = [], {}, []
    for i, layer in enumerate(cfg.layers):
        if "weights_of" in layer:
            continue
        m, prefix = layer["mixer"], f"l{i}.mix."
        mixer = _latent_spec(cfg, m, prefix) if layer["type"] == "latent_attention" else _attention_spec(cfg, layer["type"], m, prefix)
        parts = {"mixer_norm": norm(f"l{i}.norm1"), "mixer": mixer, "mixer_post_norm": norm(f"l{i}.norm1b", True)}
        if layer.get("mlp") is not None:
            parts.update({"ffn_norm": norm(f"l{i}.norm2"), "ffn": _ffn_spec(cfg, layer["mlp"], f"l{i}.mlp."),
                          "ffn_post_norm": norm(f"l{i}.norm2b", True)})
        else:
            ignored += [f"l{i}.norm2", f"l{i}.norm2b"]          # a layer without feed-forward has no use for them
        place[i] = len(layers)
        layers.append(LayerSpec(parts, "sandwich"))
    # every run of a layer, with tensors of its own or another layer's, keeps its own cache
    schedule = [ScheduleEntry(place[owner(cfg, i)]) for i in range(len(cfg.layers))]
    plan = ModelPlan(
        hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "scale": cfg.embedding_scale},
                           {"weight": "embed"}),
        layers=layers, schedule=schedule, final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width}, {"weight": "head"}),
        max_positions=0, stop_ids=[], ignored_tensors=ignored)
    plan.validate()
    return plan


def checkpoint_layout(cfg: FezozenConfig) -> dict:
    """{tensor name: (shape, kind)} of a complete checkpoint (kind as weights.random_init reads it)."""
    w = cfg.width
    out = {"embed": ((cfg.vocab, w), "matrix")}
    for i, layer in enumerate(cfg.layers):
        if "weights_of" in layer:
            continue
        m, p = layer["mixer"], f"l{i}.mix."
        out.update({f"l{i}.norm1": ((w,), "norm"), f"l{i}.norm1b": ((w,), "norm")})
        if layer["type"] == "latent_attention":
            nh, d, rd, vd, r = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
            out.update({p + "q": ((nh * (d + rd), w), "matrix"), p + "dkv": ((r + rd, w), "matrix"), p + "dkv.norm": ((r,), "norm"),
                        p + "uk": ((nh * d, r), "matrix"), p + "uv": ((nh * vd, r), "matrix"), p + "g": ((nh * vd, w), "matrix"),
                        p + "o": ((w, nh * vd), "matrix")})
        else:
            nh, g, d, vd = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
            for s, rows in (("q", nh * d), ("k", g * d), ("v", g * vd)):
                out[p + s] = ((rows, w), "matrix")
                if layer["type"] == "attention":
                    out[f"{p}{s}.b"] = ((rows,), "bias")
            out[p + "o"] = ((w, nh * vd), "matrix")
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        out.update({f"l{i}.norm2": ((w,), "norm"), f"l{i}.norm2b": ((w,), "norm")})
        p = f"l{i}.mlp."
        ff, experts = int(mlp["expert"]["ff"]), int(mlp["router"]["experts"])
        for e in range(experts):
            out.update({f"{p}e{e}.gate": ((ff, w), "matrix"), f"{p}e{e}.up": ((ff, w), "matrix"), f"{p}e{e}.down": ((w, ff), "matrix")})
        out[p + "router"] = ((experts, w), "matrix")
    out["final.norm"] = ((w,), "norm")
    out["head"] = ((cfg.vocab, w), "matrix")
    return out


register_architecture(["Fezozen", "fezozen"], FezozenConfig, build_plan, checkpoint_layout)
