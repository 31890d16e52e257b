"""Configuration of decoders that are described layer by layer in a ``config.json``.

A model directory holds ``config.json`` and ``model.safetensors``.  The configuration lists the layers; each entry names its
mixer (a kind of attention or a recurrence) with its sizes and its feed-forward block.  The specs below are the mechanisms
with their constants as fields; a *design* (``models.registry.ARCHITECTURES``) is a function that reads a ``config.json`` into
a :class:`LayeredConfig` and fixes the constants the file does not carry.
"""
from __future__ import annotations

from dataclasses import dataclass, field

MAX_HEAD_DIM = 256          # attention head sizes the kernels cover
MAX_STATE_DIM = 512         # key sizes of a matrix memory
MAX_GROUP = 64              # query heads per kv head


class LayeredConfigError(ValueError):
    """A ``config.json`` that is incomplete or describes something the kernels do not cover."""


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention over rows that are key and value at once (the values are the un-normalised keys), with query / key norm,
    a linear distance bias, a sliding window that keeps the first tokens, and one sigmoid gate per head."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int                 # positions a query sees, its own included; 0 = all
    keep_first: int             # first positions that stay visible
    slope_exponent: float = 8.0
    kind = "attention"

    @property
    def out_width(self) -> int:
        return self.heads * self.dim

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads


@dataclass(frozen=True)
class MlstmSpec:
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


@dataclass(frozen=True)
class GatedMlpSpec:
    """``W_down [g * sigmoid(alpha g) * (u + offset)]`` with ``g = min(W_gate h, limit)``, ``u = clamp(W_up h, -limit, limit)``."""
    ff: int
    limit: float
    alpha: float
    offset: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec | MlstmSpec
    mlp: GatedMlpSpec | None


@dataclass(frozen=True)
class LayeredConfig:
    arch: str
    name: str
    width: int
    vocab: int
    eps: float
    layer_specs: tuple[LayerSpec, ...] = field(repr=False)

    @property
    def layers(self) -> int:
        return len(self.layer_specs)

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def attention_layers(self) -> list[int]:
        return [i for i, l in enumerate(self.layer_specs) if l.mixer.kind == "attention"]

    @property
    def recurrent_layers(self) -> list[int]:
        return [i for i, l in enumerate(self.layer_specs) if l.mixer.kind == "mlstm"]

    @property
    def max_visible(self) -> int | None:
        """Most cached tokens a query of any attention layer can see (None: no bound, or no attention layer)."""
        seen = [self.layer_specs[i].mixer for i in self.attention_layers]
        return None if not seen or any(m.window <= 0 for m in seen) else max(m.window + m.keep_first for m in seen)

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Name and shape of every tensor of the checkpoint."""
        w = self.width
        s: dict[str, tuple[int, ...]] = {"embed": (self.vocab, w), "final.norm": (w,)}
        for i, layer in enumerate(self.layer_specs):
            p, m = f"l{i}.", layer.mixer
            x = p + "mix."
            s[p + "norm1"] = (w,)
            s[x + "q"], s[x + "o"] = (m.heads * m.dim, w), (w, m.out_width)
            if m.kind == "attention":
                s.update({x + "k": (m.kv_heads * m.dim, w), x + "q.norm": (m.dim,), x + "k.norm": (m.dim,), x + "g": (m.heads, w)})
            else:
                s.update({x + "k": (m.heads * m.dim, w), x + "v": (m.out_width, w), x + "g": (m.out_width, w), x + "norm": (m.out_width,),
                          x + "i": (m.heads, w), x + "i.b": (m.heads,), x + "f": (m.heads, w), x + "f.b": (m.heads,)})
            if layer.mlp is not None:
                f = layer.mlp.ff
                s.update({p + "norm2": (w,), p + "mlp.gate": (f, w), p + "mlp.up": (f, w), p + "mlp.down": (w, f)})
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


def _attention(m: dict, where: str) -> AttentionSpec:
    heads, kv, dim, vdim = (_size(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim"))
    mask = _get(m, "mask", where)
    if vdim != dim:
        raise LayeredConfigError(f"config.json: {where}: the values are the keys, so vdim ({vdim}) must equal dim ({dim})")
    if heads % kv or heads // kv > MAX_GROUP:
        raise LayeredConfigError(f"config.json: {where}: {heads} heads over {kv} key/value heads")
    if dim > MAX_HEAD_DIM:
        raise LayeredConfigError(f"config.json: {where}: head size {dim} exceeds {MAX_HEAD_DIM}")
    return AttentionSpec(heads, kv, dim, _number(m, "scale", where), _size(mask, "size", where + ".mask"), _size(mask, "keep_first", where + ".mask", 0))


def _mlstm(m: dict, where: str) -> MlstmSpec:
    heads, dim, vdim = (_size(m, k, where) for k in ("heads", "dim", "vdim"))
    if dim > MAX_STATE_DIM:
        raise LayeredConfigError(f"config.json: {where}: key size {dim} exceeds {MAX_STATE_DIM}")
    return MlstmSpec(heads, dim, vdim, _number(m, "gate_cap", where))


def keripel_config(raw: dict, name: str = "") -> LayeredConfig:
    """The Keripel design: mLSTM and windowed-attention mixers in the order the file lists, output norms, gated feed-forward
    blocks where a layer has one, and a head tied to the embedding."""
    mixers = {"attention": _attention, "mlstm": _mlstm}
    layers = []
    for i, entry in enumerate(_get(raw, "layers", "the model")):
        where = f"layers[{i}]"
        kind = _get(entry, "type", where)
        if kind not in mixers:
            raise LayeredConfigError(f"config.json: {where}: unknown mixer type {kind!r}")
        mixer = mixers[kind](_get(entry, "mixer", where), where + ".mixer")
        mlp = _get(entry, "mlp", where)
        if mlp is not None:
            if _get(mlp, "kind", where + ".mlp") != "dense":
                raise LayeredConfigError(f"config.json: {where}.mlp: unknown kind {mlp['kind']!r}")
            mlp = GatedMlpSpec(_size(mlp, "ff", where + ".mlp"), _number(mlp, "limit", where + ".mlp"), alpha=1.702, offset=1.0)
        layers.append(LayerSpec(mixer, mlp))
    if not layers:
        raise LayeredConfigError("config.json: the model has no layers")
    arch = raw.get("architecture", "Keripel")
    return LayeredConfig(arch, name or arch, _size(raw, "width", "the model"), _size(raw, "vocab", "the model"),
                         _number(_get(raw, "norm", "the model"), "eps", "norm"), tuple(layers))
