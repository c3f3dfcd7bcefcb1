"""Arrangements of a layer's parts."""

from __future__ import annotations

from .base import Block, FixedState, NormedUpdate, StreamUpdate
from .registry import BLOCKS
from .spec import TensorSpec


@BLOCKS.register("prenorm")
class PreNormBlock(Block):
    """h = x + mixer(norm(x)); out = h + feed_forward(norm(h)). Each residual add is fused
    with the norm that follows it, so the block returns its last output unadded; a part that
    ``fuses_residual`` may instead add its output into the stream itself and return None.
    A layer without a feed-forward ends after the mixer. Parameter ``residual_scale`` (1): the
    factor m in h = x + m mixer(norm(x)); out = h + m feed_forward(norm(h)). The factor is
    applied where the output is added: by the part itself if it adds into the stream and
    ``scales_residual``, else by the norm that follows (``delta_scale``).
    Reference: src/mlx_one/models/language/lfm2/reference_math.py:160-179."""

    def __init__(self, spec, tensors, runtime, **roles):
        super().__init__(spec, tensors, runtime, **roles)
        self.scale = float(spec.get("residual_scale", 1.0))
        self.pending_scale = self.scale
        for part in (self.mixer, self.feed_forward):
            if part is not None:
                part.residual_scale = self.scale

    @staticmethod
    def _norm(norm, residual, delta, consumer, scale=1.0):
        extra = {} if scale == 1.0 else {"delta_scale": scale}
        if consumer.accepts_normed_input and norm.supports_lazy:
            return norm.forward(residual, delta, lazy=True, **extra)
        return norm.forward(residual, delta, **extra)

    def _fuses(self, part):
        return part.fuses_residual and (self.scale == 1.0 or part.scales_residual)

    def forward(self, residual, delta, ctx, cache, write, delta_scale=1.0):
        normed = self._norm(self.mixer_norm, residual, delta, self.mixer, delta_scale)
        if self._fuses(self.mixer):
            mixed = self.mixer.forward(normed, ctx, cache, write, residual=residual)
        else:
            mixed = self.mixer.forward(normed, ctx, cache, write)
        if self.feed_forward is None:
            return mixed
        normed = self._norm(self.feed_forward_norm, residual, mixed, self.feed_forward, self.scale)
        if self._fuses(self.feed_forward):
            return self.feed_forward.forward(normed, ctx, residual=residual)
        return self.feed_forward.forward(normed, ctx)


@BLOCKS.register("outnorm")
class OutputNormBlock(Block):
    """x <- x + norm1(mixer(in1(x))); x <- x + norm2(feed_forward(in2(x))): the norms are applied
    to the parts' outputs, the parts read the stream itself (rounded to the compute dtype).
    A layer without a feed-forward ends after the mixer. Parameters:

    ``taps`` (None: in(x) = x): in(x) = x + conv(x), a causal convolution over time on every
    channel of the 32-bit stream, conv(x)_t = sum_j w[:, j] x_(t - taps + 1 + j) with nothing
    before a sequence's start; ``conv1`` and ``conv2`` [hidden, taps] are the two sublayers'
    weights. The last taps - 1 rows of x that each sublayer read are kept per request in 32-bit.

    ``streams`` (None: the layer's result goes on as it is): the number n of streams that are
    averaged after the layer, with the stored weights ``average`` [n]: what the next layer reads
    is sum_j average[j] X_j, X_0 the embedding's output and X_(j+1) the result of the call j of
    the order (before any averaging), so n is this call's number plus two."""

    @classmethod
    def tensors(cls, spec):
        out = {}
        if spec.get("taps"):
            out["conv1"] = TensorSpec((spec["hidden"], spec["taps"]), "wide")
            if spec.get("feed_forward", True):
                out["conv2"] = TensorSpec((spec["hidden"], spec["taps"]), "wide")
        if spec.get("streams"):
            out["average"] = TensorSpec((spec["streams"],), "wide")
        return out

    @classmethod
    def cache_need(cls, spec):
        taps = spec.get("taps")
        if not taps or taps < 2:
            return None
        sublayers = 2 if spec.get("feed_forward", True) else 1
        return {"inputs": FixedState((sublayers, taps - 1, spec["hidden"]), "float32")}

    def __init__(self, spec, tensors, runtime, **roles):
        super().__init__(spec, tensors, runtime, **roles)
        self.taps = spec.get("taps") or 0
        self.conv1 = self.vector(tensors["conv1"]) if "conv1" in tensors else None
        self.conv2 = self.vector(tensors["conv2"]) if "conv2" in tensors else None
        self.average = self.vector(tensors["average"]) if "average" in tensors else None
        self.keeps_streams = self.average is not None
        for norm in (self.mixer_norm, self.feed_forward_norm):
            if norm is not None and not hasattr(norm, "add_normed"):
                raise ValueError("this block needs norms that can be applied to a part's output")

    def _read(self, residual, kernel, ctx, own_cache, write, sublayer):
        """What a sublayer reads: the stream (plus its convolution over time) in the compute dtype."""
        view = (own_cache or {}).get("inputs")
        return self.ops.stream_conv(residual, kernel, taps=self.taps, ctx=ctx, view=view,
                                    sublayer=sublayer, write=write, dtype=self.runtime.dtype)

    def forward(self, residual, delta, ctx, cache, write, own_cache=None, streams=None,
                delta_scale=1.0):
        if delta is not None:
            raise ValueError("this block takes a stream with nothing pending")
        mixed = self.mixer.forward(self._read(residual, self.conv1, ctx, own_cache, write, 0),
                                   ctx, cache, write)
        self.mixer_norm.add_normed(residual, mixed)
        if self.feed_forward is not None:
            out = self.feed_forward.forward(
                self._read(residual, self.conv2, ctx, own_cache, write, 1), ctx)
            self.feed_forward_norm.add_normed(residual, out)
        if self.average is None:
            return None
        kept, place = streams
        if self.average.numel() != place + 2:
            raise ValueError(f"call {place} of the order averages {place + 2} streams, "
                             f"{self.average.numel()} weights are stored")
        return self.ops.stream_average(kept, self.average, place + 2, kept[place + 2]), None


@BLOCKS.register("sandwich")
class SandwichBlock(Block):
    """x <- x + post1(mixer(norm1(x))); x <- x + post2(feed_forward(norm2(x))): every part reads
    the normed stream and its output is normed once more before it is added. The norms ahead of
    the parts are the layer's ``mixer_norm`` and ``feed_forward_norm``; the norms behind them are
    the block's own: v / rms(v) * (offset + weight) over the model width, with the stored weights
    ``post_mixer`` and ``post_feed_forward``, taken and added in 32-bit. A layer without a
    feed-forward ends after the mixer. Parameters: ``size``, ``eps``, ``offset`` (0; 1 for
    weights stored around zero), ``feed_forward`` (True: the layer has one), ``norm``
    (``rmsnorm``; ``layernorm``: the norms behind the parts are (v - mean) / sqrt(variance + eps) *
    weight + bias, with the stored ``post_mixer.bias`` and ``post_feed_forward.bias``).

    With layer norms a part's output is handed on as a ``NormedUpdate``: one kernel norms it, adds it
    to the stream and applies the norm ahead of the next part (of the next layer, at the end)."""

    @classmethod
    def tensors(cls, spec):
        init = "norm0" if spec.get("offset") else "norm"
        names = ["post_mixer"] + (["post_feed_forward"] if spec.get("feed_forward", True) else [])
        out = {name: TensorSpec((spec["size"],), init) for name in names}
        if cls._layer_norms(spec):
            out.update({name + ".bias": TensorSpec((spec["size"],), "bias") for name in names})
        return out

    @staticmethod
    def _layer_norms(spec):
        kind = spec.get("norm") or "rmsnorm"
        if kind not in ("rmsnorm", "layernorm"):
            raise ValueError(f"unknown norm {kind!r}")
        return kind == "layernorm"

    def __init__(self, spec, tensors, runtime, **roles):
        super().__init__(spec, tensors, runtime, **roles)
        self.eps = float(spec["eps"])
        offset = float(spec.get("offset") or 0.0)
        weight = lambda name: (self.vector(tensors[name]) + offset).contiguous()
        self.post_mixer = weight("post_mixer")
        self.post_feed_forward = weight("post_feed_forward") if "post_feed_forward" in tensors else None
        if (self.feed_forward is None) != (self.post_feed_forward is None):
            raise ValueError("a feed-forward and the norm behind it come together")
        self.normed_updates = self._layer_norms(spec)
        self.biases = {}
        if self.normed_updates:
            self.biases = {name[:-len(".bias")]: self.vector(tensors[name])
                           for name in tensors if name.endswith(".bias")}

    def _read(self, norm, residual, delta, consumer, scale=1.0):
        extra = {} if scale == 1.0 else {"delta_scale": scale}
        if delta is None and consumer.accepts_normed_input and norm.supports_lazy:
            return norm.forward(residual, delta, lazy=True, **extra)
        return norm.forward(residual, delta, **extra)

    def _forward_updates(self, residual, delta, ctx, cache, write):
        normed = self.mixer_norm.forward(residual, delta)
        out = self.mixer.forward(normed, ctx, cache, write)
        delta = NormedUpdate(out, self.post_mixer, self.biases["post_mixer"], self.eps)
        if self.feed_forward is not None:
            out = self.feed_forward.forward(self.feed_forward_norm.forward(residual, delta), ctx)
            delta = NormedUpdate(out, self.post_feed_forward, self.biases["post_feed_forward"], self.eps)
        return delta

    def forward(self, residual, delta, ctx, cache, write, delta_scale=1.0):
        if self.normed_updates:
            return self._forward_updates(residual, delta, ctx, cache, write)
        normed = self._read(self.mixer_norm, residual, delta, self.mixer, delta_scale)
        mixed = self.mixer.forward(normed, ctx, cache, write)
        self.ops.normed_mean_add(residual, [mixed], [self.post_mixer], self.eps)
        if self.feed_forward is not None:
            normed = self._read(self.feed_forward_norm, residual, None, self.feed_forward)
            out = self.feed_forward.forward(normed, ctx)
            self.ops.normed_mean_add(residual, [out], [self.post_feed_forward], self.eps)
        return None


@BLOCKS.register("hyper")
class HyperConnectedBlock(Block):
    """Hyper-connections: ``streams`` residual streams X_1 .. X_n instead of one, all equal to the
    embedding's output at the start. A sublayer reads u = sum_s in[s] X_s, and with y =
    part(norm(u)) every stream is replaced at once: X_t <- sum_s mix[s, t] X_s + out[t] y. The
    stored ``in1``, ``out1`` [streams] and ``mix1`` [streams, streams] (indexed [from, to]) belong
    to the mixer, ``in2``, ``out2``, ``mix2`` to the feed-forward. A layer without a feed-forward
    ends after the mixer. Parameters: ``streams``, ``feed_forward`` (True: the layer has one).

    The streams are 32-bit [tokens, streams, hidden]. One kernel stands between two sublayers: it
    writes the last one's output into the streams, reads the next one's input from them and norms
    it, so each stream is read and written once per sublayer. Ahead of the first sublayer there is
    one stream that stands for all: reading it takes the sum of ``in``, and the first write makes
    ``streams`` of it with the sums of ``mix``'s columns."""

    parallel_streams = True

    @classmethod
    def tensors(cls, spec):
        count = spec["streams"]
        out = {}
        for which in ("1", "2") if spec.get("feed_forward", True) else ("1",):
            out["in" + which] = TensorSpec((count,), "wide")
            out["out" + which] = TensorSpec((count,), "norm")
            out["mix" + which] = TensorSpec((count, count), "mix")
        return out

    def __init__(self, spec, tensors, runtime, **roles):
        super().__init__(spec, tensors, runtime, **roles)
        self.streams = int(spec["streams"])
        if (self.feed_forward is None) == bool(spec.get("feed_forward", True)):
            raise ValueError("a feed-forward and its connections come together")
        for norm in (self.mixer_norm, self.feed_forward_norm):
            if norm is not None and not hasattr(norm, "read_streams"):
                raise ValueError("this block needs norms that can read parallel streams")
        # per sublayer: (reading weights, mix, out), for all streams and for the one at the start
        self.connections = []
        for which in ("1", "2") if self.feed_forward is not None else ("1",):
            read, mix = self.vector(tensors["in" + which]), self.vector(tensors["mix" + which])
            out = self.vector(tensors["out" + which])
            self.connections.append({
                self.streams: (read, mix, out),
                1: (read.sum(0, keepdim=True), mix.sum(0, keepdim=True).contiguous(), out)})

    def _sublayer(self, which, norm, residual, delta, run):
        before = residual.shape[1] if delta is None else delta.mix.shape[1]
        read, mix, out = self.connections[which][before]
        residual, normed = norm.read_streams(residual, delta, read)
        return residual, StreamUpdate(run(normed), mix, out)

    def forward(self, residual, delta, ctx, cache, write):
        residual, delta = self._sublayer(0, self.mixer_norm, residual, delta,
                                         lambda x: self.mixer.forward(x, ctx, cache, write))
        if self.feed_forward is not None:
            residual, delta = self._sublayer(1, self.feed_forward_norm, residual, delta,
                                             lambda x: self.feed_forward.forward(x, ctx))
        return residual, delta
