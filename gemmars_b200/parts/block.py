"""The arrangement of a layer's parts.

``prenorm`` (src/qwen.rs:682-696): x += mixer(norm(x)); x += ffn(norm(x)), the residual stream
``x`` in float32; a layer may lack the feed-forward and its norm, and each sublayer's output may have a
factor per feature (``mixer_scale``, ``ffn_scale``).  ``parallel``: x += mixer(norm(x)) + ffn(norm(x)) with one norm, or with a norm of its own for the feed-forward.  ``sandwich``:
a norm on both sides of each sublayer, x += post(mixer(pre(x))); x += post(ffn(pre(x))).  Another
arrangement (a third norm) is another class like these, registered under its own kind
and reading its own part names from the layer's spec."""
from __future__ import annotations

import torch

from .. import kernels
from .base import Block, Part, TensorWant, register_part
from .norm import RMSNorm


class PreNormBlock(Block):
    def __init__(self, layer_spec, compute):
        super().__init__(layer_spec, compute)
        self.mixer_norm = self.need("mixer_norm", "norm")
        self.mixer = self.need("mixer", "mixer")
        has_ffn = "ffn" in layer_spec.parts
        self.ffn_norm = self.need("ffn_norm", "norm") if has_ffn else None
        self.ffn = self.need("ffn", "ffn") if has_ffn else None
        self.scales = {}
        for name, part in (("mixer_scale", self.mixer), ("ffn_scale", self.ffn)):
            if name in layer_spec.parts and part is not None:
                if not hasattr(part, "set_output_scale"):
                    raise ValueError(f"block {layer_spec.block!r}: the {part.category} {part.spec.kind!r} takes no factor on its output")
                self.scales[name] = self.need(name, "scale")
                self.scales[name].give_to(part)

    def parts(self):
        out = {"mixer_norm": self.mixer_norm, "mixer": self.mixer}
        if self.ffn is not None:
            out.update({"ffn_norm": self.ffn_norm, "ffn": self.ffn})
        out.update(self.scales)          # loaded after the parts they are handed to
        return out

    #: forward takes ``h_in`` / ``next_norm`` and returns what its last product left for the next block's first norm
    chains_norms = True

    def first_norm(self):
        """The norm that reads the residual first: the block before may be asked to feed it."""
        return self.mixer_norm

    @property
    def takes_unscaled_rows(self):
        return getattr(self.mixer, "links_norms", False)

    def forward(self, ctx, x, caches, writes_cache=True, h_in=None, next_norm=None):
        """Runs the layer on ``x`` in place.  In decode steps the RMSNorms are taken into the
        products around them where the parts can (kernels.UnscaledRows): ``h_in`` is what the block
        before left for this block's first norm (None: the norm runs by itself), ``next_norm`` the
        first norm of the block after; returns what the feed-forward's last product left for it."""
        mine = self.split_caches(caches)
        linking = (kernels.NORM_LINKS and self.compute == "bfloat16" and ctx.n_tokens <= kernels.LINK_MAX_TOKENS)
        h = h_in if h_in is not None else self.mixer_norm.forward(ctx, x)
        left = None
        # the norm that reads the residual after the mixer, if what follows it can take its unscaled rows
        after = next_norm if self.ffn is None else (self.ffn_norm if getattr(self.ffn, "links_norms", False) else None)
        if getattr(self.mixer, "links_norms", False):
            then = after if linking and getattr(after, "linkable", False) else None
            left = self.mixer.forward(ctx, h, x, mine["mixer"], writes_cache, then_norm=then)
        else:
            self.mixer.forward(ctx, _plain(h), x, mine["mixer"], writes_cache)
        if self.ffn is None:
            return left
        h = left if left is not None else self.ffn_norm.forward(ctx, x)
        if getattr(self.ffn, "links_norms", False):
            then = next_norm if linking and getattr(next_norm, "linkable", False) else None
            return self.ffn.forward(ctx, h, x, then_norm=then)
        self.ffn.forward(ctx, _plain(h), x)
        return None


class ChannelScale(Part):
    """``channel_scale``: a factor per feature on a sublayer's output, ``factor`` times the tensor
    ``weight`` [size], applied in float32 where the sublayer's last product adds into the stream."""
    category = "scale"

    def __init__(self, spec, compute):
        super().__init__(spec, compute)
        self.size = int(spec.params["size"])
        self.constant = float(spec.params.get("factor", 1.0))
        self.weight = self._part = None

    def give_to(self, part):
        self._part = part

    def factor(self):
        return self.weight

    def wants(self):
        return {"weight": TensorWant((self.size,), "vector")}

    def load(self, tensors):
        self.weight = (tensors["weight"].to(torch.float32) * self.constant).contiguous()
        if self._part is not None:
            self._part.set_output_scale(self.factor())

    def weight_bytes(self):
        return 0 if self.weight is None else 4 * self.weight.numel()


class AddRow(Part):
    """``add_row``: row ``row`` of the tensor ``weight`` [rows, size] is added to every row of the stream."""
    category = "stream"

    def __init__(self, spec, compute):
        super().__init__(spec, compute)
        self.size, self.rows, self.row = (int(spec.params[k]) for k in ("size", "rows", "row"))
        if not 0 <= self.row < self.rows:
            raise ValueError(f"add_row: row {self.row} of {self.rows}")
        self.vector = None

    def wants(self):
        return {"weight": TensorWant((self.rows, self.size), "vector")}

    def load(self, tensors):
        self.vector = tensors["weight"][self.row].to(torch.float32).contiguous()

    def kernel_units(self):
        return [("rows", ())]

    def weight_bytes(self):
        return 0 if self.vector is None else 4 * self.vector.numel()

    def forward(self, ctx, x, then_norm=None):
        """``then_norm``: an RMSNorm part that reads the stream next; its output is made in the same pass."""
        if not isinstance(then_norm, RMSNorm):
            kernels.add_row(self.vector, x)
            return None
        out = torch.empty(x.shape, dtype=then_norm.act_dtype, device=x.device)
        kernels.add_row(self.vector, x, (then_norm.weight, then_norm.eps, out))
        return out


class ParallelBlock(Block):
    """``parallel``: h = norm(x); x += mixer(h) + ffn(h).  One norm, and both branches read its
    output; each branch adds its result into the float32 residual stream, the mixer first.  The
    layer's spec lists ``norm``, ``mixer`` and, when the layer has a feed-forward, ``ffn``.  With
    ``ffn_norm`` in the spec the feed-forward reads a norm of its own of the same x:
    x += mixer(norm(x)) + ffn(ffn_norm(x)), both norms taken before either branch changes x."""

    def __init__(self, layer_spec, compute):
        super().__init__(layer_spec, compute)
        self.norm = self.need("norm", "norm")
        self.mixer = self.need("mixer", "mixer")
        self.ffn = self.need("ffn", "ffn") if "ffn" in layer_spec.parts else None
        self.ffn_norm = self.need("ffn_norm", "norm") if self.ffn is not None and "ffn_norm" in layer_spec.parts else None

    def parts(self):
        out = {"norm": self.norm, "mixer": self.mixer}
        if self.ffn_norm is not None:
            out["ffn_norm"] = self.ffn_norm
        if self.ffn is not None:
            out["ffn"] = self.ffn
        return out

    def forward(self, ctx, x, caches, writes_cache=True):
        mine = self.split_caches(caches)
        # read by both branches before either changes x; two norms of the same x are one pass where they can be
        if self.ffn_norm is not None and hasattr(self.norm, "forward_with"):
            h, h_ffn = self.norm.forward_with(ctx, x, self.ffn_norm)
        else:
            h = self.norm.forward(ctx, x)
            h_ffn = self.ffn_norm.forward(ctx, x) if self.ffn_norm is not None else h
        self.mixer.forward(ctx, h, x, mine["mixer"], writes_cache)
        if self.ffn is not None:
            self.ffn.forward(ctx, h_ffn, x)


class SandwichBlock(Block):
    """``sandwich``: x += mixer_post_norm(mixer(mixer_norm(x))); x += ffn_post_norm(ffn(ffn_norm(x))).
    A sublayer's output goes into float32 rows of its own instead of the residual stream (stored there by
    parts that can, else added into zeros); the norm after it reads those rows, adds the normed rows into
    the stream and makes the output of the norm that reads the stream next, the next layer's first one
    included, in the same pass.  The layer's spec lists
    ``mixer_norm``, ``mixer``, ``mixer_post_norm`` and, when the layer has a feed-forward,
    ``ffn_norm``, ``ffn``, ``ffn_post_norm``."""

    def __init__(self, layer_spec, compute):
        super().__init__(layer_spec, compute)
        self.mixer_norm = self.need("mixer_norm", "norm")
        self.mixer = self.need("mixer", "mixer")
        self.mixer_post_norm = self.need("mixer_post_norm", "norm")
        self.ffn = self.need("ffn", "ffn") if "ffn" in layer_spec.parts else None
        self.ffn_norm = self.need("ffn_norm", "norm") if self.ffn is not None else None
        self.ffn_post_norm = self.need("ffn_post_norm", "norm") if self.ffn is not None else None
        for part in (self.mixer, self.ffn):
            if hasattr(part, "set_output_store"):
                part.set_output_store()

    def parts(self):
        out = {"mixer_norm": self.mixer_norm, "mixer": self.mixer, "mixer_post_norm": self.mixer_post_norm}
        if self.ffn is not None:
            out.update({"ffn_norm": self.ffn_norm, "ffn": self.ffn, "ffn_post_norm": self.ffn_post_norm})
        return out

    #: forward takes ``h_in`` / ``next_norm``: the norm before may be made by the pass of the norm after
    chains_norms = True
    takes_unscaled_rows = True

    def first_norm(self):
        return self.mixer_norm

    @staticmethod
    def _rows_for(part, x):
        """Float32 rows for the part's output: as they come for a part that stores, else zeros."""
        return torch.empty_like(x) if _stores(part) else torch.zeros_like(x)

    def forward(self, ctx, x, caches, writes_cache=True, h_in=None, next_norm=None):
        mine = self.split_caches(caches)
        y = self._rows_for(self.mixer, x)
        self.mixer.forward(ctx, _plain(h_in) if h_in is not None else self.mixer_norm.forward(ctx, x), y, mine["mixer"], writes_cache)
        if self.ffn is None:
            return self.mixer_post_norm.add_normed(ctx, y, x, _same_kind(self.mixer_post_norm, next_norm))
        h = self.mixer_post_norm.add_normed(ctx, y, x, _same_kind(self.mixer_post_norm, self.ffn_norm))
        if h is None:
            h = self.ffn_norm.forward(ctx, x)
        if not _stores(self.ffn):
            y.zero_()
        self.ffn.forward(ctx, h, y)
        return self.ffn_post_norm.add_normed(ctx, y, x, _same_kind(self.ffn_post_norm, next_norm))


def _stores(part):
    """Whether the part stores its output instead of adding it (it was asked to, and could)."""
    return getattr(part, "stores", False)


def _same_kind(norm, then):
    """``then`` if ``norm``'s pass over a sublayer's output can make its output as well, else None."""
    return then if isinstance(then, type(norm)) and hasattr(then, "weight") else None


def _plain(h):
    return h.materialize() if isinstance(h, kernels.UnscaledRows) else h


register_part("block", "prenorm", PreNormBlock)
register_part("block", "parallel", ParallelBlock)
register_part("block", "sandwich", SandwichBlock)
register_part("scale", "channel_scale", ChannelScale)
register_part("stream", "add_row", AddRow)
