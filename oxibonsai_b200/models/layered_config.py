"""Configuration of decoders that are described layer by layer in a ``config.json``.

A model directory holds ``config.json`` and ``model.safetensors``.  The configuration lists the layers; each entry names its
mixer (a kind of attention, a recurrence, or several side by side) with its sizes and its feed-forward block.  The specs below
are the mechanisms with their constants as fields; a *design* (``models.registry.ARCHITECTURES``) is a function that reads a
``config.json`` into a :class:`LayeredConfig` and fixes the constants the file does not carry.

Every mixer spec names its tensors: ``sections`` (the matrices that read the mixer's input, as row ranges), ``vectors``, ``inner``
(matrices that read something else) and the output matrix "o" with ``out_width`` inputs.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field

import torch

from .rope_scaling import llama31_frequencies

MAX_HEAD_DIM = 256          # attention head sizes the kernels cover
MAX_STATE_DIM = 512         # key sizes of a matrix memory
MAX_GROUP = 64              # query heads per kv head
MAX_RANK = 512              # latent size of a compressed cache
MAX_LATENT_ROW = 640        # that and the shared key part, each padded to 16
MAX_EXPERTS = 512
MAX_CHOSEN = 32             # experts of a token
MAX_TAPS = 16               # of a convolution over tokens
MAX_SCAN_STATES = 256       # per channel


class LayeredConfigError(ValueError):
    """A ``config.json`` that is incomplete or describes something the kernels do not cover."""


class MixerSpec:
    """What all mixers have in common: the branches of a layer (one, unless mixers stand side by side)."""

    @property
    def branches(self) -> tuple["Branch", ...]:
        return (Branch("", self, 1.0),)

    @property
    def inner(self) -> dict[str, tuple[int, int]]:
        return {}

    @property
    def out_bias(self) -> bool:
        """Whether the output projection has a bias ("o.b")."""
        return False


@dataclass(frozen=True)
class Branch:
    """A mixer of a layer: the prefix of its tensors and the factor of its output in the layer's sum."""
    prefix: str
    spec: "AttentionSpec | LatentAttentionSpec | MlstmSpec | LinearRecurrenceSpec | MinGruSpec | SelectiveScanSpec"
    scale: float


@dataclass(frozen=True)
class FrequencyScaling:
    """Rotary frequencies for contexts longer than ``original``: wavelengths above original / low are stretched by ``factor``, those
    below original / high are kept, with a linear ramp in between."""
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first ``dims`` dimensions of a head: dimension i paired with i + dims / 2, or with ``interleaved`` 2i
    with 2i + 1."""
    base: float
    dims: int
    interleaved: bool = False
    scaling: FrequencyScaling | None = None

    @property
    def frequencies(self) -> list[float]:
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if self.scaling is None:
            return f
        s = self.scaling
        return llama31_frequencies(torch.tensor(f, dtype=torch.float64), s.factor, s.low, s.high, s.original).tolist()


@dataclass(frozen=True)
class AttentionSpec(MixerSpec):
    """Softmax attention; everything from ``vdim`` on is optional."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    vdim: int | None = None     # None: the values are the un-normalised keys (cache rows that are key and value)
    window: int = 0             # positions a query sees, its own included; 0 = all
    chunk: int = 0              # a query sees its own chunk of that many positions only, counted from position 0
    keep_first: int = 0         # first positions that stay visible
    slope_exponent: float | None = None    # geometric slopes of a linear distance bias
    norm_weights: bool = False  # weights of the query and key norms
    gated: bool = False         # one sigmoid gate per head on the output
    element_gate: bool = False  # one sigmoid gate per output element instead
    softcap: float = 0.0        # scores become softcap * tanh(score / softcap), with separate values; 0 = as they are
    temp_coef: float = 0.0      # queries are multiplied by 1 + temp_coef * ln(floor((position + 1) / temp_every) + 1)
    temp_every: float = 1.0
    normed: bool = True         # queries and keys are divided by their root mean square
    rotary: RotarySpec | None = None
    sink: bool = False          # a learned term per head in the softmax denominator, without a key and a value
    kv_from: int | None = None  # the layer whose cached keys and values are used; None: this layer has its own
    biases: bool = False        # projections with biases
    difference: float | None = None    # two softmax maps per head: o = a1 - lambda a2 over its root mean square, times 1 - difference,
    #                             with lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + difference
    kind = "attention"

    @property
    def maps(self) -> int:
        return 1 if self.difference is None else 2

    @property
    def row_dim(self) -> int:
        """Elements a cache row must hold: the keys of all maps, or the value."""
        return max(self.maps * self.dim, self.value_dim)

    @property
    def visible(self) -> int:
        """Most cached tokens a query sees (0: no bound)."""
        return self.window + self.keep_first if self.window > 0 else self.chunk

    @property
    def out_bias(self) -> bool:
        return self.biases

    @property
    def value_dim(self) -> int:
        return self.dim if self.vdim is None else self.vdim

    @property
    def out_width(self) -> int:
        return self.heads * self.value_dim

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads

    @property
    def sections(self) -> list[tuple[str, int]]:
        s = [("q", self.heads * self.maps * self.dim)]
        if self.kv_from is None:
            s.append(("k", self.kv_heads * self.maps * self.dim))
            if self.vdim is not None:
                s.append(("v", self.kv_heads * self.vdim))
        return s + ([("g", self.out_width if self.element_gate else self.heads)] if self.gated or self.element_gate else [])

    @property
    def vectors(self) -> dict[str, tuple[int, ...]]:
        v: dict[str, tuple[int, ...]] = {"q.norm": (self.dim,), "k.norm": (self.dim,)} if self.norm_weights else {}
        if self.sink:
            v["sink"] = (self.heads,)
        if self.biases:
            v.update({n + ".b": (rows,) for n, rows in self.sections if n != "g"})
        if self.difference is not None:
            v.update({n: (self.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        return v


@dataclass(frozen=True)
class LatentAttentionSpec(MixerSpec):
    """Softmax attention whose keys and values are linear in one normalised latent per token ("dkv", its first ``rank`` rows): the
    cache holds the latent and one rotated key part that all heads share.  The output has one sigmoid gate per element."""
    heads: int
    dim: int                    # unrotated query / key dimensions of a head
    rot_dim: int                # rotated ones, behind them
    vdim: int
    rank: int
    scale: float
    rotary: RotarySpec
    kind = "latent"

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def sections(self) -> list[tuple[str, int]]:
        return [("q", self.heads * (self.dim + self.rot_dim)), ("dkv", self.rank), ("dkv", self.rot_dim), ("g", self.out_width)]

    @property
    def vectors(self) -> dict[str, tuple[int, ...]]:
        return {"dkv.norm": (self.rank,)}

    @property
    def inner(self) -> dict[str, tuple[int, int]]:
        return {"uk": (self.heads * self.dim, self.rank), "uv": (self.out_width, self.rank)}


@dataclass(frozen=True)
class MlstmSpec(MixerSpec):
    """Matrix-memory recurrence with capped exponential gates (mLSTM)."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    den_eps: float = 1e-6
    kind = "mlstm"

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def sections(self) -> list[tuple[str, int]]:
        qk = self.heads * self.dim
        return [("q", qk), ("k", qk), ("v", self.out_width), ("g", self.out_width), ("i", self.heads), ("f", self.heads)]

    @property
    def vectors(self) -> dict[str, tuple[int, ...]]:
        return {"i.b": (self.heads,), "f.b": (self.heads,), "norm": (self.out_width,)}


@dataclass(frozen=True)
class LinearRecurrenceSpec(MixerSpec):
    """``S <- a S + b k v^T, o = S^T q`` with one decay per head and token, then a gated norm in ``norm_parts`` equal parts.

    ``decay`` lists fixed decays (b = 1); without it they come from the input (state-space duality): dt = softplus(raw + bias),
    a = exp(-exp(A_log) dt), b = dt, a skip D per head, and one matrix "in" for all projections.  ``conv`` > 0: a causal
    convolution of that many taps on values, keys and queries."""
    heads: int
    dim: int
    vdim: int
    groups: int                         # heads / groups heads share queries and keys
    norm_parts: int
    gate: str                           # "silu" or "sigmoid"
    decay: tuple[float, ...] | None = None
    activation: bool = False            # silu on queries, keys and values (after the convolution)
    rotary: RotarySpec | None = None
    key_scale: float = 1.0
    conv: int = 0
    gate_first: bool = False            # the gate comes before the norm
    norm_weight: bool = False
    kind = "recurrence"

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_channels(self) -> int:
        return self.out_width + 2 * self.groups * self.dim

    @property
    def sections(self) -> list[tuple[str, int]]:
        if self.decay is None:          # z, then x, B, C (values, keys, queries), then dt
            return [("in", self.out_width), ("in", self.conv_channels), ("in", self.heads)]
        qk = self.groups * self.dim
        return [("q", qk), ("k", qk), ("v", self.out_width), ("g", self.out_width)]

    @property
    def vectors(self) -> dict[str, tuple[int, ...]]:
        v: dict[str, tuple[int, ...]] = {"norm": (self.out_width,)} if self.norm_weight else {}
        if self.conv:
            v.update({"conv": (self.conv_channels, self.conv), "conv.b": (self.conv_channels,)})
        if self.decay is None:
            v.update({"dt_bias": (self.heads,), "A_log": (self.heads,), "D": (self.heads,)})
        return v


@dataclass(frozen=True)
class MinGruSpec(MixerSpec):
    """An element-wise gated recurrence whose gates read the current token only (minGRU), with a silu gate on the output."""
    width: int
    kind = "mingru"

    @property
    def out_width(self) -> int:
        return self.width

    @property
    def sections(self) -> list[tuple[str, int]]:
        return [("z", self.width), ("x", self.width), ("g", self.width)]

    @property
    def vectors(self) -> dict[str, tuple[int, ...]]:
        return {"z.b": (self.width,), "x.b": (self.width,)}


@dataclass(frozen=True)
class SelectiveScanSpec(MixerSpec):
    """A state-space recurrence with ``states`` decays per channel, whose step sizes (through a product of rank ``rank``), inputs and
    outputs are read from the convolved channels (Mamba)."""
    channels: int
    states: int
    rank: int
    conv: int
    kind = "selective"

    @property
    def out_width(self) -> int:
        return self.channels

    @property
    def sections(self) -> list[tuple[str, int]]:
        return [("in", self.channels), ("in", self.channels)]      # the channels, then their gates

    @property
    def vectors(self) -> dict[str, tuple[int, ...]]:
        c = self.channels
        return {"conv": (c, self.conv), "conv.b": (c,), "dt.b": (c,), "A_log": (c, self.states), "D": (c,)}

    @property
    def inner(self) -> dict[str, tuple[int, int]]:
        return {"x": (self.rank + 2 * self.states, self.channels), "dt": (self.channels, self.rank)}


RECURRENT = ("mlstm", "recurrence", "mingru", "selective")


@dataclass(frozen=True)
class ParallelSpec(MixerSpec):
    """Mixers side by side that read the same input; the scaled sum of their outputs is the layer's."""
    parts: tuple[Branch, ...]
    kind = "parallel"

    @property
    def branches(self) -> tuple[Branch, ...]:
        return self.parts


@dataclass(frozen=True)
class GatedMlpSpec:
    """``W_down [g * sigmoid(alpha (g + cubic g^3)) * (u + offset)]`` with ``g = min(W_gate h, limit)``, ``u = clamp(W_up h, -limit,
    limit)``."""
    ff: int
    limit: float
    alpha: float
    offset: float
    cubic: float = 0.0
    matrices = ("gate", "up")


def gelu_mlp(ff: int) -> GatedMlpSpec:
    """A gate through the tanh form of gelu: (1 + tanh(y)) / 2 = sigmoid(2 y)."""
    return GatedMlpSpec(ff, math.inf, alpha=2.0 * math.sqrt(2.0 / math.pi), offset=0.0, cubic=0.044715)


@dataclass(frozen=True)
class SquaredReluMlpSpec:
    """``W_down relu(W_up h)^2``."""
    ff: int
    matrices = ("up",)


@dataclass(frozen=True)
class RouterSpec:
    """Chooses ``top`` of ``experts`` per token.  Scores are sigmoids, or with ``softmax`` that of all logits; what is compared is the
    score, plus a learned correction where the router has one.  Experts form ``groups`` equal groups of neighbours, of which only the
    ``keep`` with the largest sums of their two best are eligible.  The weights are the chosen scores, over (their sum + ``den_eps``)
    if ``normalized``, times ``scale``."""
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    den_eps: float = 1e-20
    softmax: bool = False
    normalized: bool = True
    corrected: bool = True


@dataclass(frozen=True)
class ExpertsSpec:
    """A weighted sum of the chosen experts; each is a gated block of ``ff`` hidden units as in :class:`GatedMlpSpec`.  ``shared``: one more
    block that every token runs, times the sigmoid of one number per token ("shared.sg")."""
    router: RouterSpec
    ff: int
    limit: float = math.inf
    alpha: float = 1.0
    offset: float = 0.0
    shared: GatedMlpSpec | None = None


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    mlp: GatedMlpSpec | SquaredReluMlpSpec | ExpertsSpec | None


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start`` .. ``stop`` - 1 run ``times`` times in a row with the same weights and a cache or state per pass.  Ahead of pass t
    x grows by row t of "loop.step" and, from the second pass on, by the embedding."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class Run:
    """One run of a layer; ``begins``: the pass it is the first run of (None: it begins none)."""
    layer: int
    begins: int | None = None


@dataclass(frozen=True)
class LayeredConfig:
    arch: str
    name: str
    width: int
    vocab: int
    eps: float
    layer_specs: tuple[LayerSpec, ...] = field(repr=False)
    embed_scale: float = 1.0
    pre_norm: bool = False      # a norm ahead of each sublayer too ("norm1", "norm2"; those on the outputs are then "norm1b", "norm2b")
    side_by_side: bool = False  # mixer and feed-forward read the same norm ("norm1"); x grows by residual_mult times their sum
    residual_mult: float = 1.0
    layer_norm: bool = False    # norms take the mean off first
    norm_groups: int | None = None     # norms divide that many equal parts by their own root mean square (None: one part)
    input_taps: int = 0         # what a sublayer reads, h, becomes h + conv(h), a convolution over that many tokens ("canon1", "canon2"); 0: no
    loop: LoopSpec | None = None
    own_head: bool = False      # the head is a tensor of its own ("head")
    logit_cap: float = 0.0      # logits become cap * tanh(logits / cap); 0: as they are

    @property
    def layers(self) -> int:
        return len(self.layer_specs)

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def runs(self) -> tuple[Run, ...]:
        """The layers in the order they run; caches and states belong to runs."""
        lo = self.loop
        if lo is None:
            return tuple(Run(i) for i in range(self.layers))
        body = [Run(i, t if i == lo.start else None) for t in range(lo.times) for i in range(lo.start, lo.stop)]
        return tuple([Run(i) for i in range(lo.start)] + body + [Run(i) for i in range(lo.stop, self.layers)])

    @property
    def row_steps(self) -> bool:
        """Whether what happens between sublayers takes the general row kernel."""
        return self.norm_groups is not None or self.input_taps > 0 or self.loop is not None

    @property
    def has_state(self) -> bool:
        """Whether a sequence has state besides the pages of attention layers."""
        return bool(self.recurrent_layers) or self.input_taps > 0

    def branches(self, i: int, *kinds: str) -> list[Branch]:
        """The mixers of layer ``i`` of the given kinds."""
        return [b for b in self.layer_specs[i].mixer.branches if b.spec.kind in kinds]

    @property
    def attention_layers(self) -> list[int]:
        return [i for i in range(self.layers) if self.branches(i, "attention", "latent")]

    @property
    def recurrent_layers(self) -> list[int]:
        return [i for i in range(self.layers) if self.branches(i, *RECURRENT)]

    def attention(self, i: int) -> AttentionSpec | LatentAttentionSpec:
        return self.branches(i, "attention", "latent")[0].spec

    def recurrence(self, i: int) -> "MlstmSpec | LinearRecurrenceSpec | MinGruSpec | SelectiveScanSpec":
        return self.branches(i, *RECURRENT)[0].spec

    @property
    def max_visible(self) -> int | None:
        """Most cached tokens a query of any attention layer can see (None: no bound, or no attention layer)."""
        seen = [self.attention(i) for i in self.attention_layers]
        if not seen or any(isinstance(m, LatentAttentionSpec) or m.visible <= 0 for m in seen):
            return None
        return max(m.visible for m in seen)

    @property
    def expert_layers(self) -> list[int]:
        return [i for i in range(self.layers) if isinstance(self.layer_specs[i].mlp, ExpertsSpec)]

    def experts(self, i: int) -> ExpertsSpec:
        return self.layer_specs[i].mlp

    def norm_names(self, i: int) -> list[tuple[str | None, str | None]]:
        """Per sublayer of layer ``i`` the names of the norms of its input and of its output (None: none).  Sublayers side by side
        count as one."""
        p = f"l{i}."
        if self.side_by_side:
            return [(p + "norm1", None)]
        names = [(p + f"norm{n}", p + f"norm{n}b") if self.pre_norm else (None, p + f"norm{n}") for n in (1, 2)]
        return names if self.layer_specs[i].mlp is not None else names[:1]

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Name and shape of every tensor of the checkpoint."""
        w = self.width
        s: dict[str, tuple[int, ...]] = {"embed": (self.vocab, w), "final.norm": (w,)}
        if self.own_head:
            s["head"] = (self.vocab, w)
        if self.loop is not None:
            s["loop.step"] = (self.loop.times, w)
        for i, layer in enumerate(self.layer_specs):
            if self.input_taps:
                s.update({f"l{i}.canon{n + 1}": (w, self.input_taps) for n in range(len(self.norm_names(i)))})
            s.update({n: (w,) for pair in self.norm_names(i) for n in pair if n is not None})
            for b in layer.mixer.branches:
                x = f"l{i}.mix.{b.prefix}"
                for name, rows in b.spec.sections:
                    s[x + name] = (s.get(x + name, (0, w))[0] + rows, w)
                s.update({x + n: shape for n, shape in {**b.spec.vectors, **b.spec.inner}.items()})
                s[x + "o"] = (w, b.spec.out_width)
                if b.spec.out_bias:
                    s[x + "o.b"] = (w,)
            if isinstance(layer.mlp, ExpertsSpec):
                f, n = layer.mlp.ff, layer.mlp.router.experts
                s[f"l{i}.mlp.router"] = (n, w)
                if layer.mlp.router.corrected:
                    s[f"l{i}.mlp.correction"] = (n,)
                if layer.mlp.shared is not None:
                    sf, sp = layer.mlp.shared.ff, f"l{i}.mlp.shared."
                    s.update({sp + "gate": (sf, w), sp + "up": (sf, w), sp + "down": (w, sf), sp + "sg": (1, w)})
                for e in range(n):
                    s.update({f"l{i}.mlp.e{e}.gate": (f, w), f"l{i}.mlp.e{e}.up": (f, w), f"l{i}.mlp.e{e}.down": (w, f)})
            elif layer.mlp is not None:
                f = layer.mlp.ff
                s.update({f"l{i}.mlp.{n}": (f, w) for n in layer.mlp.matrices})
                s[f"l{i}.mlp.down"] = (w, f)
        return s

    def param_count(self) -> int:
        n = 0
        for shape in self.tensor_shapes().values():
            k = 1
            for d in shape:
                k *= d
            n += k
        return n


def _get(d: dict, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise LayeredConfigError(f"config.json: {where} has no '{key}'")
    return d[key]


def _size(d: dict, key: str, where: str, lowest: int = 1) -> int:
    v = _get(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v or int(v) < lowest:
        raise LayeredConfigError(f"config.json: {where}.{key} must be an integer >= {lowest}, got {v!r}")
    return int(v)


def _number(d: dict, key: str, where: str) -> float:
    v = _get(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise LayeredConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
    return float(v)


def _positive(d: dict, key: str, where: str) -> float:
    v = _number(d, key, where)
    if not v > 0:
        raise LayeredConfigError(f"config.json: {where}.{key} must be positive, got {v!r}")
    return v


def _attention_sizes(m: dict, where: str) -> tuple[int, int, int, int]:
    heads, kv, dim, vdim = (_size(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim"))
    if heads % kv or heads // kv > MAX_GROUP:
        raise LayeredConfigError(f"config.json: {where}: {heads} heads over {kv} key/value heads")
    if max(dim, vdim) > MAX_HEAD_DIM:
        raise LayeredConfigError(f"config.json: {where}: head size {max(dim, vdim)} exceeds {MAX_HEAD_DIM}")
    return heads, kv, dim, vdim


def _rotary(m: dict, dim: int, where: str, interleaved: bool = False) -> RotarySpec | None:
    """The rotation of heads of ``dim`` dimensions (None: nothing is rotated)."""
    rot, where = _get(m, "rot", where), where + ".rot"
    dims = _size(rot, "dims", where, 0)
    if dims % 2 or dims > dim:
        raise LayeredConfigError(f"config.json: {where}.dims must be even and at most {dim}, got {dims}")
    scaling, raw = None, rot.get("scaling") if interleaved else None
    if raw is not None:
        scaling = FrequencyScaling(*(_positive(raw, k, where + ".scaling") for k in ("factor", "low", "high", "original")))
        if scaling.low >= scaling.high:
            raise LayeredConfigError(f"config.json: {where}.scaling: low ({scaling.low}) must be below high ({scaling.high})")
    return RotarySpec(_positive(rot, "base", where), dims, interleaved, scaling) if dims else None


def _state_dim(dim: int, where: str) -> int:
    if dim > MAX_STATE_DIM:
        raise LayeredConfigError(f"config.json: {where}: key size {dim} exceeds {MAX_STATE_DIM}")
    return dim


def _layers(raw: dict, mixers: dict, mlps: dict) -> tuple[LayerSpec, ...]:
    """The layer list: ``mixers`` reads a mixer by its type, ``mlps`` a feed-forward block by its kind."""
    layers = []
    for i, entry in enumerate(_get(raw, "layers", "the model")):
        where = f"layers[{i}]"
        kind = _get(entry, "type", where)
        if kind not in mixers:
            raise LayeredConfigError(f"config.json: {where}: unknown mixer type {kind!r}")
        ff = _get(entry, "mlp", where)
        if ff is not None and _get(ff, "kind", where + ".mlp") not in mlps:
            raise LayeredConfigError(f"config.json: {where}.mlp: unknown kind {ff['kind']!r}")
        layers.append(LayerSpec(mixers[kind](_get(entry, "mixer", where), where + ".mixer"), None if ff is None else mlps[ff["kind"]](ff, where + ".mlp")))
    if not layers:
        raise LayeredConfigError("config.json: the model has no layers")
    return tuple(layers)


def _model(raw: dict, design: str, name: str, layers: tuple[LayerSpec, ...], **extra) -> LayeredConfig:
    arch = raw.get("architecture", design)
    return LayeredConfig(arch, name or arch, _size(raw, "width", "the model"), _size(raw, "vocab", "the model"),
                         _number(_get(raw, "norm", "the model"), "eps", "norm"), layers, **extra)


# ---- Keripel ----------------------------------------------------------------------------------------------------------------------
def _windowed_attention(m: dict, where: str) -> AttentionSpec:
    heads, kv, dim, vdim = _attention_sizes(m, where)
    mask = _get(m, "mask", where)
    if vdim != dim:
        raise LayeredConfigError(f"config.json: {where}: the values are the keys, so vdim ({vdim}) must equal dim ({dim})")
    return AttentionSpec(heads, kv, dim, _number(m, "scale", where), window=_size(mask, "size", where + ".mask"),
                         keep_first=_size(mask, "keep_first", where + ".mask", 0), slope_exponent=8.0, norm_weights=True, gated=True)


def _mlstm(m: dict, where: str) -> MlstmSpec:
    heads, dim, vdim = (_size(m, k, where) for k in ("heads", "dim", "vdim"))
    return MlstmSpec(heads, _state_dim(dim, where), vdim, _number(m, "gate_cap", where))


def keripel_config(raw: dict, name: str = "") -> LayeredConfig:
    """The Keripel design: mLSTM and windowed-attention mixers in the order the file lists, output norms, gated feed-forward
    blocks where a layer has one, and a head tied to the embedding."""
    mlp = lambda m, where: GatedMlpSpec(_size(m, "ff", where), _number(m, "limit", where), alpha=1.702, offset=1.0)
    return _model(raw, "Keripel", name, _layers(raw, {"attention": _windowed_attention, "mlstm": _mlstm}, {"dense": mlp}))


# ---- Kekevik ----------------------------------------------------------------------------------------------------------------------
def _decays(m: dict, heads: int, where: str) -> tuple[float, ...]:
    d = _get(m, "decay", where)
    if not isinstance(d, list) or len(d) != heads or any(isinstance(x, bool) or not isinstance(x, (int, float)) or not 0 <= x <= 1 for x in d):
        raise LayeredConfigError(f"config.json: {where}.decay must list {heads} numbers from 0 to 1")
    return tuple(float(x) for x in d)


def _retention(m: dict, where: str) -> LinearRecurrenceSpec:
    heads, dim, vdim = (_size(m, k, where) for k in ("heads", "dim", "vdim"))
    return LinearRecurrenceSpec(heads, _state_dim(dim, where), vdim, groups=heads, norm_parts=heads, gate="silu", decay=_decays(m, heads, where),
                                rotary=_rotary(m, dim, where), key_scale=dim ** -0.5)


def _lightning(m: dict, where: str) -> LinearRecurrenceSpec:
    heads, dim, vdim = (_size(m, k, where) for k in ("heads", "dim", "vdim"))
    return LinearRecurrenceSpec(heads, _state_dim(dim, where), vdim, groups=heads, norm_parts=1, gate="sigmoid", decay=_decays(m, heads, where),
                                activation=True, norm_weight=True)


def _capped_attention(m: dict, where: str) -> AttentionSpec:
    heads, kv, dim, vdim = _attention_sizes(m, where)
    temp = _get(m, "q_temp", where)
    return AttentionSpec(heads, kv, dim, _number(m, "scale", where), vdim=vdim, softcap=_positive(m, "softcap", where),
                         temp_coef=_number(temp, "coef", where + ".q_temp"), temp_every=_positive(temp, "every", where + ".q_temp"))


def _mamba2(m: dict, where: str) -> LinearRecurrenceSpec:
    heads, vdim, state, groups, parts, taps = (_size(m, k, where) for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv"))
    if heads % groups or heads * vdim % parts:
        raise LayeredConfigError(f"config.json: {where}: {heads} heads of {vdim} values over {groups} groups and {parts} norm groups")
    return LinearRecurrenceSpec(heads, _state_dim(state, where), vdim, groups=groups, norm_parts=parts, gate="silu", activation=True, conv=taps,
                                gate_first=True, norm_weight=True)


def _side_by_side(m: dict, where: str) -> ParallelSpec:
    return ParallelSpec((Branch("left.", _capped_attention(_get(m, "left", where), where + ".left"), _number(m, "left_scale", where)),
                         Branch("right.", _mamba2(_get(m, "right", where), where + ".right"), _number(m, "right_scale", where))))


def kekevik_config(raw: dict, name: str = "") -> LayeredConfig:
    """The Kekevik design: retention, lightning attention, and capped attention beside a state-space mixer, in the order the
    file lists; norms before and after each sublayer, squared-relu feed-forward blocks, a scaled embedding tied to the head."""
    layers = _layers(raw, {"retention": _retention, "lightning": _lightning, "parallel": _side_by_side},
                     {"dense": lambda m, where: SquaredReluMlpSpec(_size(m, "ff", where))})
    scale = _number(_get(raw, "embedding", "the model"), "scale", "embedding")
    return _model(raw, "Kekevik", name, layers, embed_scale=scale, pre_norm=True)


# ---- Kutepel ----------------------------------------------------------------------------------------------------------------------
def _rotary_attention(m: dict, where: str) -> AttentionSpec:
    heads, kv, dim, vdim = _attention_sizes(m, where)
    source = None if m.get("kv_from") is None else _size(m, "kv_from", where, 0)
    return AttentionSpec(heads, kv, dim, _number(m, "scale", where), vdim=vdim, normed=False, rotary=_rotary(m, dim, where, interleaved=True), sink=True,
                         kv_from=source)


def _latent_attention(m: dict, where: str) -> LatentAttentionSpec:
    heads, dim, rot_dim, vdim, rank = (_size(m, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    rotary = _rotary(m, rot_dim, where, interleaved=True)
    if rotary is None or rotary.dims != rot_dim:
        raise LayeredConfigError(f"config.json: {where}: rot.dims must be rot_dim ({rot_dim}), which must be even")
    up = lambda n, m: -(-n // m) * m
    if up(dim, 8) + up(rot_dim, 8) > MAX_HEAD_DIM or vdim > MAX_HEAD_DIM:
        raise LayeredConfigError(f"config.json: {where}: head sizes {dim} + {rot_dim} and {vdim} exceed {MAX_HEAD_DIM}")
    if rank > MAX_RANK or up(rank, 16) + up(rot_dim, 16) > MAX_LATENT_ROW:
        raise LayeredConfigError(f"config.json: {where}: a latent of {rank} + {rot_dim} exceeds {MAX_RANK} or {MAX_LATENT_ROW} together")
    return LatentAttentionSpec(heads, dim, rot_dim, vdim, rank, _number(m, "scale", where), rotary)


def _choice(r: dict, where: str) -> tuple[int, int]:
    """Experts, and how many of them a token uses."""
    experts, top = _size(r, "experts", where), _size(r, "top", where)
    if experts > MAX_EXPERTS or top > min(MAX_CHOSEN, experts):
        raise LayeredConfigError(f"config.json: {where}: {top} of {experts} experts (at most {MAX_CHOSEN} of {MAX_EXPERTS})")
    return experts, top


def _experts(m: dict, where: str) -> ExpertsSpec:
    r, ff = _get(m, "router", where), _size(_get(m, "expert", where), "ff", where + ".expert")
    experts, top = _choice(r, where + ".router")
    where += ".router"
    g = r.get("groups")
    count, keep = (1, 1) if g is None else (_size(g, "count", where + ".groups"), _size(g, "keep", where + ".groups"))
    if experts % count or keep > count or top > keep * (experts // count):
        raise LayeredConfigError(f"config.json: {where}: {top} of {experts} experts in {keep} of {count} groups")
    return ExpertsSpec(RouterSpec(experts, top, count, keep, _number(r, "scale", where)), ff)


def kutepel_config(raw: dict, name: str = "") -> LayeredConfig:
    """The Kutepel design: latent attention and rotary attention with sinks (some layers on an earlier one's keys and values) in the
    order the file lists, side by side with a mixture of experts behind one layer norm, and a head tied to the embedding."""
    layers = _layers(raw, {"attention": _rotary_attention, "latent_attention": _latent_attention}, {"moe": _experts})
    for i, layer in enumerate(layers):
        j = getattr(layer.mixer, "kv_from", None)
        if j is None:
            continue
        source = layers[j].mixer if j < i else None
        if not isinstance(source, AttentionSpec) or source.kv_from is not None:
            raise LayeredConfigError(f"config.json: layers[{i}].mixer.kv_from: layer {j} is no earlier attention layer with keys and values of its own")
        if (source.kv_heads, source.dim, source.vdim) != (layer.mixer.kv_heads, layer.mixer.dim, layer.mixer.vdim):
            raise LayeredConfigError(f"config.json: layers[{i}].mixer.kv_from: layer {j} has other key/value heads")
    return _model(raw, "Kutepel", name, layers, side_by_side=True, residual_mult=_number(raw, "residual_mult", "the model"), layer_norm=True)


# ---- Naforax ----------------------------------------------------------------------------------------------------------------------
SWISH_ALPHA = 1.702         # of the clamped units


def _differential_attention(m: dict, where: str) -> AttentionSpec:
    heads, kv, dim, vdim = _attention_sizes(m, where)
    if 2 * dim > MAX_HEAD_DIM:
        raise LayeredConfigError(f"config.json: {where}: two maps of {dim} dimensions exceed {MAX_HEAD_DIM}")
    return AttentionSpec(heads, kv, dim, _number(m, "scale", where), vdim=vdim, chunk=_size(_get(m, "mask", where), "size", where + ".mask"), norm_weights=True,
                         element_gate=True, rotary=_rotary(m, dim, where, interleaved=True), biases=True, difference=_number(m, "diff", where))


def _taps(d: dict, key: str, where: str) -> int:
    taps = _size(d, key, where)
    if taps > MAX_TAPS:
        raise LayeredConfigError(f"config.json: {where}.{key}: a convolution over {taps} tokens exceeds {MAX_TAPS}")
    return taps


def _mingru(m: dict, where: str) -> MinGruSpec:
    return MinGruSpec(_size(m, "width", where))


def _mamba1(m: dict, where: str) -> SelectiveScanSpec:
    states = _size(m, "state", where)
    if states > MAX_SCAN_STATES:
        raise LayeredConfigError(f"config.json: {where}: {states} states per channel exceed {MAX_SCAN_STATES}")
    return SelectiveScanSpec(_size(m, "inner", where), states, _size(m, "dt_rank", where), _taps(m, "conv", where))


def _clamped_unit(m: dict, where: str) -> GatedMlpSpec:
    return GatedMlpSpec(_size(m, "ff", where), _positive(m, "limit", where), alpha=SWISH_ALPHA, offset=1.0)


def _softmax_experts(m: dict, where: str) -> ExpertsSpec:
    experts, top = _choice(_get(m, "router", where), where + ".router")
    e, shared = _clamped_unit(_get(m, "expert", where), where + ".expert"), m.get("shared")
    return ExpertsSpec(RouterSpec(experts, top, softmax=True, normalized=False, corrected=False), e.ff, e.limit, e.alpha, e.offset,
                       None if shared is None else _clamped_unit(shared, where + ".shared"))


def _loop(raw: dict, layers: int) -> LoopSpec | None:
    if raw.get("loop") is None:
        return None
    lo = LoopSpec(*(_size(raw["loop"], k, "loop", least) for k, least in (("start", 0), ("stop", 1), ("times", 1))))
    if not lo.start < lo.stop <= layers:
        raise LayeredConfigError(f"config.json: loop: layers {lo.start} .. {lo.stop - 1} of {layers}")
    return lo


def naforax_config(raw: dict, name: str = "") -> LayeredConfig:
    """The Naforax design: differential attention in chunks, minGRU and selective-scan mixers in the order the file lists, a loop over some
    of the layers, grouped norms before and after each sublayer, a convolution ahead of each, dense blocks and experts with a shared
    one, and a capped head of its own."""
    layers = _layers(raw, {"attention": _differential_attention, "mingru": _mingru, "mamba1": _mamba1},
                     {"dense": lambda m, where: gelu_mlp(_size(m, "ff", where)), "moe": _softmax_experts})
    groups, width = _size(_get(raw, "norm", "the model"), "groups", "norm"), _size(raw, "width", "the model")
    if width % groups or groups << max(0, -(-(width // groups) // 16) - 1).bit_length() > 1024:     # a power of two of threads per part, 16 columns each
        raise LayeredConfigError(f"config.json: norm.groups: {groups} equal parts of {width}")
    return _model(raw, "Naforax", name, layers, pre_norm=True, residual_mult=_number(raw, "residual_mult", "the model"), norm_groups=groups,
                  input_taps=_taps(_get(raw, "canon", "the model"), "taps", "canon"), loop=_loop(raw, len(layers)), own_head=True,
                  logit_cap=_positive(raw, "logit_softcap", "the model"))
