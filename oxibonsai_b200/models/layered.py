"""Decoders described layer by layer (``layered_config``): weights, mixers and the step runner.

A step is a batch of rows (tokens).  Rows of single tokens (decode) come first, portions of prompts follow, each portion
contiguous, short ones first; every projection runs over all rows, a mixer runs its single-token kernel over the first group and
its prompt kernel over the second (latent attention takes short portions for single tokens).  Mixers that stand side by side in a
layer share one projection and one output projection over their joined outputs; a feed-forward block beside the mixer shares the
projection too.  A row carries its position and its slot; the slot's block-table row names the pages of its sequence
and the state table its recurrent state row, so which pages, rows and companions a token has does not enter its arithmetic.

Two modes: bf16 (tensor-core projections and attention, f32 residual stream, norms, scores, gates and recurrent state) and
the exact mode, f32 throughout.  Decode steps of slots 0 .. n-1 are captured into CUDA graphs; mixed batches are issued
eagerly with the same kernels.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from pathlib import Path
from typing import Sequence

import numpy as np
import torch

from ..ops import cuda_ops as K
from ..ops import layered_ops as L
from ..ops import nvtx
from .layered_config import (AttentionSpec, Branch, ExpertsSpec, GatedMlpSpec, LatentAttentionSpec, LayeredConfig, LinearRecurrenceSpec, MinGruSpec,
                             MlstmSpec, RotarySpec, SelectiveScanSpec, SquaredReluMlpSpec)
from .paged import RowCache, StatePool
from .rope_scaling import geometric_slopes
from .slot_state import SlotState


def _tensor(t) -> torch.Tensor:
    """A checkpoint tensor as a host torch tensor (bf16 kept, everything else widened to f32)."""
    if t.dtype == "BF16":
        return torch.from_numpy(np.array(np.frombuffer(t.data, dtype="<i2"))).view(torch.bfloat16).reshape(t.shape)
    return torch.from_numpy(np.array(t.to_f32()))


@dataclass
class MlpWeights:
    pre_norm: torch.Tensor | None
    norm: torch.Tensor | None
    up: L.DenseWeight                # gated blocks: gate and up rows interleaved
    down: L.DenseWeight
    act: L.Glu | str
    ff: int

    @classmethod
    def gated(cls, spec: GatedMlpSpec, matrix, prefix: str, norms, device) -> "MlpWeights":
        """``matrix``: a checkpoint matrix by its name."""
        return cls(*norms, L.DenseWeight([matrix(prefix + "gate"), matrix(prefix + "up")], device, interleave=True), L.DenseWeight([matrix(prefix + "down")], device),
                   L.Glu(spec.limit, spec.alpha, spec.offset, spec.cubic), spec.ff)

    @property
    def nbytes(self) -> int:
        return self.up.nbytes + self.down.nbytes


@dataclass
class ExpertWeights:
    """A mixture of experts.  Beside the mixer its router is part of the layer's projection; behind it, ``router`` reads the
    feed-forward's input: the router's rows and the shared block's gate."""
    column: int                      # first router logit in that projection
    correction: torch.Tensor | None
    up: L.DenseWeight                # all experts' gate and up rows, interleaved, one expert below the other
    down: L.DenseWeight
    experts: int
    top: int
    pre_norm: torch.Tensor | None = None
    norm: torch.Tensor | None = None
    router: L.DenseWeight | None = None
    shared: MlpWeights | None = None

    @property
    def nbytes(self) -> int:
        """Bytes a decode step must stream for one token."""
        n = (self.up.nbytes + self.down.nbytes) * self.top // self.experts
        return n + (0 if self.router is None else self.router.nbytes) + (0 if self.shared is None else self.shared.nbytes)


@dataclass
class LatentWeights:
    """The expansions of a latent in the forms the kernels read (sizes padded with zeros)."""
    keys: torch.Tensor               # [heads, rank to 16, dim to 32]
    values: torch.Tensor             # [heads, vdim, rank to 32]
    expand: L.DenseWeight            # per head dim to 8 key rows, vdim to 8 value rows

    @classmethod
    def load(cls, m: LatentAttentionSpec, uk: torch.Tensor, uv: torch.Tensor, device) -> "LatentWeights":
        H, R, up = m.heads, m.rank, L.round_up
        uk, uv = uk.view(H, m.dim, R), uv.view(H, m.vdim, R)
        pad = torch.nn.functional.pad
        keys = pad(uk.transpose(1, 2), (0, up(m.dim, 32) - m.dim, 0, up(R, 16) - R))
        both = torch.cat([pad(uk, (0, 0, 0, up(m.dim, 8) - m.dim)), pad(uv, (0, 0, 0, up(m.vdim, 8) - m.vdim))], dim=1)
        return cls(keys.contiguous().to(device), pad(uv, (0, up(R, 32) - R)).contiguous().to(device), L.DenseWeight([both.reshape(-1, R)], device))

    @property
    def nbytes(self) -> int:
        """Bytes a decode step must stream."""
        return 2 * (self.keys.numel() + self.values.numel())


@dataclass
class ScanWeights:
    """The projections inside a selective scan."""
    read: L.DenseWeight              # three parts: step sizes (low rank), inputs, outputs
    step: L.DenseWeight

    @classmethod
    def load(cls, m: SelectiveScanSpec, x: torch.Tensor, dt: torch.Tensor, device) -> "ScanWeights":
        return cls(L.DenseWeight(list(torch.split(x, [m.rank, m.states, m.states])), device), L.DenseWeight([dt], device))

    @property
    def nbytes(self) -> int:
        return self.read.nbytes + self.step.nbytes


@dataclass
class BranchWeights:
    columns: list[int]               # first output of each section in the layer's projection
    vectors: dict[str, torch.Tensor]
    offset: int                      # first column in the input of the output projection
    inner: LatentWeights | ScanWeights | None = None


@dataclass
class LayerWeights:
    pre_norm: torch.Tensor | None
    norm: torch.Tensor | None
    proj: L.DenseWeight              # every projection that reads the mixers' input, one matrix
    out: L.DenseWeight               # the branches' output projections side by side
    branches: list[BranchWeights]
    mlp: MlpWeights | ExpertWeights | None
    convs: list[torch.Tensor]        # per sublayer: the convolution of its input [taps, width], the current token's tap first
    out_bias: torch.Tensor | None = None


def branch_offsets(widths: Sequence[int]) -> tuple[list[int], int]:
    """First columns of the branches' outputs in their joined buffer (16-byte boundaries in either mode), and its width."""
    at, offsets = 0, []
    for w in widths:
        at = L.round_up(at, 8)
        offsets.append(at)
        at += w
    return offsets, at


class LayeredWeights:
    """Device-resident weights of a model directory (``model.safetensors``)."""

    def __init__(self, cfg: LayeredConfig, tensors: dict[str, torch.Tensor], device):
        shapes = cfg.tensor_shapes()
        for n, s in shapes.items():
            if n not in tensors:
                raise ValueError(f"checkpoint has no tensor {n}")
            if tuple(tensors[n].shape) != s:
                raise ValueError(f"tensor {n} is {list(tensors[n].shape)}, expected {list(s)}")
        self.cfg, self.device = cfg, torch.device(device)
        m = lambda n: tensors[n].to(torch.bfloat16)
        v = lambda n: None if n is None else tensors[n].float().to(self.device)
        self.embed = L.DenseWeight([m("embed")], self.device)
        self.head = L.DenseWeight([m("head")], self.device) if cfg.own_head else self.embed
        self.final_norm = v("final.norm")
        self.loop_step = v("loop.step") if cfg.loop is not None else None
        self.layers: list[LayerWeights] = []
        for i, spec in enumerate(cfg.layer_specs):
            norms, p, parts, counts = cfg.norm_names(i), f"l{i}.mlp.", [], []
            for b in spec.mixer.branches:
                first: dict[str, int] = {}
                for name, rows in b.spec.sections:
                    at = first.get(name, 0)
                    parts.append(m(f"l{i}.mix.{b.prefix}{name}")[at:at + rows])
                    first[name] = at + rows
                counts.append(len(b.spec.sections))
            moe = spec.mlp if isinstance(spec.mlp, ExpertsSpec) else None
            if moe is not None and cfg.side_by_side:
                parts.append(m(p + "router"))
            proj = L.DenseWeight(parts, self.device)
            offsets, width = branch_offsets([b.spec.out_width for b in spec.mixer.branches])
            out = torch.zeros((cfg.width, width), dtype=torch.bfloat16)
            branches, at = [], 0
            for b, off, count in zip(spec.mixer.branches, offsets, counts):
                x = f"l{i}.mix.{b.prefix}"
                out[:, off:off + b.spec.out_width] = m(x + "o")
                inner = None
                if isinstance(b.spec, LatentAttentionSpec):
                    inner = LatentWeights.load(b.spec, m(x + "uk"), m(x + "uv"), self.device)
                elif isinstance(b.spec, SelectiveScanSpec):
                    inner = ScanWeights.load(b.spec, m(x + "x"), m(x + "dt"), self.device)
                branches.append(BranchWeights(proj.columns[at:at + count], {n: v(x + n) for n in b.spec.vectors}, off, inner))
                at += count
            mlp = None
            assert moe is not None or not cfg.side_by_side or spec.mlp is None, "dense blocks stand behind the mixer"
            if moe is not None:
                r, names = moe.router, [f"{p}e{e}." for e in range(moe.router.experts)]
                up = L.DenseWeight([torch.cat([m(n + c) for n in names]) for c in ("gate", "up")], self.device, interleave=True)
                mlp = ExpertWeights(proj.columns[at] if cfg.side_by_side else 0, v(p + "correction") if r.corrected else None, up,
                                    L.DenseWeight([torch.cat([m(n + "down") for n in names])], self.device), r.experts, r.top)
                if not cfg.side_by_side:
                    mlp.pre_norm, mlp.norm = map(v, norms[1])
                    mlp.router = L.DenseWeight([m(p + "router")] + ([m(p + "shared.sg")] if moe.shared is not None else []), self.device)
                if moe.shared is not None:
                    mlp.shared = MlpWeights.gated(moe.shared, m, p + "shared.", (None, None), self.device)
            elif isinstance(spec.mlp, GatedMlpSpec):
                mlp = MlpWeights.gated(spec.mlp, m, p, map(v, norms[1]), self.device)
            elif isinstance(spec.mlp, SquaredReluMlpSpec):
                mlp = MlpWeights(*map(v, norms[1]), L.DenseWeight([m(p + "up")], self.device), L.DenseWeight([m(p + "down")], self.device), L.SQUARED_RELU, spec.mlp.ff)
            convs = [L.conv_weight(v(f"l{i}.canon{n + 1}")) for n in range(len(norms))] if cfg.input_taps else []
            biased = [b.prefix for b in spec.mixer.branches if b.spec.out_bias]
            bias = sum(v(f"l{i}.mix.{x}o.b") for x in biased) if biased else None
            self.layers.append(LayerWeights(*map(v, norms[0]), proj, L.DenseWeight([out], self.device), branches, mlp, convs, bias))
        torch.cuda.synchronize(self.device)

    @classmethod
    def from_dir(cls, cfg: LayeredConfig, path, device) -> "LayeredWeights":
        from ..convert import read_safetensors
        return cls(cfg, {t.name: _tensor(t) for t in read_safetensors(str(Path(path) / "model.safetensors"))}, device)

    @property
    def packed_bytes(self) -> int:
        """Bytes a decode step must stream."""
        layer = [l.proj.nbytes + l.out.nbytes + (0 if l.mlp is None else l.mlp.nbytes) + sum(b.inner.nbytes for b in l.branches if b.inner is not None)
                 for l in self.layers]
        return self.head.nbytes + sum(layer[r.layer] for r in self.cfg.runs)


def new_row_cache(cfg: LayeredConfig, num_pages: int, page_size: int, exact: bool, device) -> RowCache:
    """Rows by the number of a layer's run."""
    layers = {}
    for n, run in enumerate(cfg.runs):
        if run.layer not in cfg.attention_layers:
            continue
        s = cfg.attention(run.layer)
        if isinstance(s, LatentAttentionSpec):
            layers[n] = (1, L.lib().bonsai_lay_latent_row(s.rank, s.rot_dim), "latent")
        elif s.kv_from is None:
            layers[n] = (s.kv_heads, L.lib().bonsai_lay_attn_row(s.row_dim), "shared" if s.vdim is None else "separate")
    return RowCache(layers, num_pages, page_size, K.KV_F32 if exact else K.KV_BF16, torch.float32 if exact else torch.bfloat16, device)


def state_dims(m: MlstmSpec | LinearRecurrenceSpec) -> tuple[int, int]:
    """Padded rows and columns of a head's state."""
    l = L.lib()
    if isinstance(m, MlstmSpec):
        return l.bonsai_lay_mlstm_dim(m.dim), l.bonsai_lay_mlstm_vdim(m.vdim)
    return l.bonsai_lay_rec_dim(m.dim), l.bonsai_lay_rec_vdim(m.vdim)


def runs_chunked(m) -> bool:
    """Whether portions of prompts go to the tensor cores (longer keys take the token-by-token kernel)."""
    if not isinstance(m, (MlstmSpec, LinearRecurrenceSpec)):
        return False
    return m.dim <= (L.lib().bonsai_lay_mlstm_chunk_dim() if isinstance(m, MlstmSpec) else L.lib().bonsai_lay_rec_chunk_dim())


def new_state_pool(cfg: LayeredConfig, num_rows: int, device) -> StatePool:
    """State by the number of a layer's run."""
    layers = {}
    for n, run in enumerate(cfg.runs):
        state = {f"canon{i + 1}": (cfg.input_taps, cfg.width) for i in range(len(cfg.norm_names(run.layer)))} if cfg.input_taps else {}
        if run.layer in cfg.recurrent_layers:
            m = cfg.recurrence(run.layer)
            if isinstance(m, MinGruSpec):
                state["S"] = (m.width,)
            elif isinstance(m, SelectiveScanSpec):
                state.update({"S": (m.channels, L.lib().bonsai_lay_scan_states(m.states)), "conv": (m.conv, m.channels)})
            else:
                d, e = state_dims(m)
                state["S"] = (m.heads, d, e)
                if isinstance(m, MlstmSpec):
                    state.update({"n": (m.heads, e // 64, d), "m": (m.heads, e // 64)})
                elif m.conv:
                    state["conv"] = (m.conv, m.conv_channels)
        if state:
            layers[n] = state
    return StatePool(layers, num_rows, device)


@dataclass
class Rows:
    """Row metadata the kernels read: one set for decode steps (row = slot), one that mixed batches fill."""
    tokens: torch.Tensor
    positions: torch.Tensor
    slots: torch.Tensor


@dataclass
class StepShape:
    """How a step's rows split: ``singles`` single-token rows, then ``portions`` (device address of the int4 list and of the
    query tiles per tokens-per-tile).  ``short``: the rows up to the first portion of more than ``SHORT`` tokens."""
    rows: int
    singles: int
    short: int
    portions: int = 0
    entries: int = 0
    tiles: dict[int, tuple[int, int]] | None = None      # tokens per tile -> (device address, tiles)
    segments: dict["SegmentPlan", tuple[int, int, int]] | None = None    # recurrences that cut the portions: segments, device addresses of the two lists
    contexts: list["ContextGroup"] = field(default_factory=list)

    def cut(self, plan: "SegmentPlan | None") -> tuple[int, int, int]:
        """Segment list, segments (0: portions as a whole) and prompt list of a recurrence."""
        n, segs, prompts = (self.segments or {}).get(plan, (0, 0, 0))
        return segs, n, prompts


SHORT = 32                  # tokens of a portion whose rows latent attention treats as single tokens
SHORT_ROWS = 256            # such rows in a step, at least
CONTEXT_TILE = 128          # query tokens per tile over expanded keys


@dataclass
class ContextGroup:
    """Long portions whose cached latents are expanded together: device addresses of the portions, of {first scratch row, cached
    tokens, slot, 0} for each, and of the query tiles."""
    portions: int
    contexts: int
    count: int
    tiles: int
    n_tiles: int
    rows: int                   # scratch rows in all
    longest: int


def group_contexts(lists: Sequence[tuple[int, int, int, int]], limit: int) -> list[list[tuple[int, int, int, int]]]:
    """Cuts portions (first row, tokens, slot, first position) into runs whose cached tokens together stay within ``limit`` rows."""
    groups: list[list[tuple[int, int, int, int]]] = []
    rows = 0
    for e in lists:
        n = e[1] + e[3]
        if not groups or rows + n > limit:
            groups.append([])
            rows = 0
        groups[-1].append(e)
        rows += n
    return groups


MAX_SEGMENTS = 24           # segment states the scratch of the recurrent layers holds
CHUNK = 64                  # tokens per chunk of the recurrences


@dataclass(frozen=True)
class SegmentCost:
    """What running a recurrence in segments costs, in times of one chunk of a lone CTA.  Segments run side by side, but their
    state products run twice.  Fitted to measured times."""
    resident: int           # CTAs an SM holds
    crowded: float          # time of a chunk when an SM is full
    twice: float            # both passes of a segment over one pass
    fixed: float
    each: float             # per segment
    shortest: int           # chunks
    share: float = 0.0      # > 0: CTAs share an SM evenly, and a chunk takes so long per CTA on it, but no less than alone

    def waves(self, ctas: int, sms: int) -> float:
        if self.share > 0:
            return max(1.0, self.share * ctas / sms)
        if self.resident > 1 and ctas <= 0.6 * sms:        # more of them do not spread evenly
            return 1.0
        return self.crowded * -(-ctas // (self.resident * sms))


# mLSTM, 8 heads of 256 x 512: 4096 tokens 600 us whole, 443 us in 2 segments, 451 in 4, 548 in 16; 512 tokens 76 us whole, 64 us in 2.
# Linear recurrence, 32 heads of 128 x 128: 4096 tokens 306 us whole, 166 in 4, 174 in 8, 210 in 32; 512 tokens 38 whole, 30 in 4.
# 16 heads of 256 x 256: 4096 tokens 424 us whole, 315 in 2, 324 in 4; 512 tokens 55 whole, 49 in 2.
MLSTM_COST = SegmentCost(1, 1.0, 1.5, 0.5, 0.6, 4)
RECURRENCE_COST = SegmentCost(2, 1.55, 1.45, 2.0, 0.3, 2)
WIDE_RECURRENCE_COST = SegmentCost(1, 1.0, 1.35, 1.2, 0.6, 2)
# Selective scan, 16 states: 4096 tokens of 512 channels 252 us whole, 122 in 4 segments, 63 in 16; of 2048 channels 253, 209, 131; of 8192
# channels 392 whole, 472 in 4.
SCAN_COST = SegmentCost(8, 1.0, 1.68, 1.5, 0.4, 2, share=0.38)


@dataclass(frozen=True)
class SegmentPlan:
    """Layers with as many CTAs per portion and the same costs cut a step's portions alike."""
    ctas: int
    cost: SegmentCost


def segment_plan(m: MlstmSpec | LinearRecurrenceSpec | SelectiveScanSpec) -> SegmentPlan:
    if isinstance(m, SelectiveScanSpec):
        return SegmentPlan(-(-m.channels // L.lib().bonsai_lay_scan_channels(m.states)), SCAN_COST)
    d, e = state_dims(m)
    cost = MLSTM_COST if isinstance(m, MlstmSpec) else (RECURRENCE_COST if d <= 128 else WIDE_RECURRENCE_COST)
    return SegmentPlan(m.heads * e // 64, cost)


def plan_segments(lengths: Sequence[int], plan: SegmentPlan, sms: int) -> int:
    """Chunks per segment for portions of ``lengths`` tokens; 0 = do not cut."""
    c = plan.cost
    chunks = [-(-n // CHUNK) for n in lengths]
    best, best_cost = 0, max(chunks) * c.waves(plan.ctas * len(chunks), sms)
    for size in range(c.shortest, max(chunks)):
        segs = sum(-(-n // size) for n in chunks)
        if segs > MAX_SEGMENTS:
            continue
        cost = c.twice * size * c.waves(plan.ctas * segs, sms) + c.fixed + c.each * segs
        if cost < best_cost:
            best, best_cost = size, cost
    return best


class AttentionMixer:
    """``index``: the number of the layer's run, here and below."""

    def __init__(self, r: "LayeredRunner", index: int, branch: Branch, w: BranchWeights, out: torch.Tensor):
        self.r, self.spec, self.out = r, branch.spec, out
        spec, cols = self.spec, dict(zip((n for n, _ in branch.spec.sections), w.columns))
        self.tile = 64 // spec.group
        source = index if spec.kv_from is None else spec.kv_from          # the layer whose rows are used
        self.appends, rot = spec.kv_from is None, spec.rotary
        slopes = None if spec.slope_exponent is None else geometric_slopes(spec.heads, spec.slope_exponent).to(r.device)
        ints = [r.proj.stride(0), cols["q"], cols.get("k", -1), cols.get("v", 0), cols.get("g", -1), out.stride(0), spec.heads, spec.kv_heads, spec.dim,
                spec.value_dim, r.max_pages, r.kv.page_size, spec.window, spec.keep_first, int(spec.normed), 0 if rot is None else rot.dims,
                int(rot is not None and rot.interleaved), spec.chunk, spec.maps, int(spec.element_gate)]
        vec, lam, left = dict(w.vectors), 0.0, 1.0
        if spec.difference is not None:
            dot = lambda i: float(torch.exp((vec[f"lq{i}"].double() * vec[f"lk{i}"].double()).sum()))
            lam, left = dot(1) - dot(2) + spec.difference, 1.0 - spec.difference
            for n, rows in spec.sections:                    # the kernels have both here
                if n != "g" and not spec.biases:
                    vec[n + ".b"] = torch.zeros(rows, dtype=torch.float32, device=r.device)
            if not spec.norm_weights:
                vec["q.norm"] = vec["k.norm"] = torch.ones(spec.dim, dtype=torch.float32, device=r.device)
        floats = [r.cfg.eps, spec.scale, branch.scale, spec.softcap, spec.temp_coef, spec.temp_every, lam, left]
        self.call = {id(rows): L.MixerCall([r.proj, vec.get("q.norm"), vec.get("k.norm"), slopes, rows.positions, rows.slots, r.block_table,
                                            r.kv.rows[source], r.kv.factors.get(source), r.kv.values.get(source), out, vec.get("sink"),
                                            None if rot is None else r.angles(rot), vec.get("q.b"), vec.get("k.b"), vec.get("v.b")], ints, floats)
                     for rows in (r.slot_rows, r.batch_rows)}

    def splits(self, batch: int) -> int:
        """KV splits of one row's decode attention: about a CTA per SM, and no more than there are 16-token tiles per warp."""
        s = self.spec
        seen = self.r.max_seq if s.visible <= 0 else min(self.r.max_seq, s.visible + 32)
        n, ctas = 1, batch * s.kv_heads * (-(-s.maps * s.group // 16))
        while n < 8 and ctas * n * 2 <= 160 and n * 2 * 128 <= seen + 127:
            n *= 2
        return n

    def __call__(self, rows: Rows, st: StepShape, stream: int, early: bool) -> None:
        lib, a = L.lib(), self.call[id(rows)].args
        if self.r.exact:
            if self.appends:
                K.check(lib.bonsai_lay_attn_append(*a, 0, st.rows, 1, stream), "attn_append")
            K.check(lib.bonsai_lay_attn_f32(*a, st.rows, stream), "attn_f32")
            return
        if st.singles:
            K.check(lib.bonsai_lay_attn_decode(*a, st.singles, self.splits(st.singles), stream), "attn_decode")
        if st.portions:
            tiles, n = st.tiles[self.tile]
            if self.appends:
                K.check(lib.bonsai_lay_attn_append(*a, st.singles, st.rows - st.singles, 0, stream), "attn_append")
            K.check(lib.bonsai_lay_attn_prompt(*a, st.entries, tiles, n, stream), "attn_prompt")

    def launches(self) -> int:
        return 1 + int(self.r.exact and self.appends)


class LatentAttentionMixer:
    """Single tokens and short portions attend to the latents themselves, longer portions to keys and values expanded from them."""

    def __init__(self, r: "LayeredRunner", index: int, branch: Branch, w: BranchWeights, out: torch.Tensor):
        self.r, self.spec, self.w, s = r, branch.spec, w, branch.spec
        q, c, rot, g = w.columns
        row = self.row = r.kv.rows[index].shape[-1]
        self.groups = -(-s.heads // L.lib().bonsai_lay_latent_group(s.heads))
        self.lat_ld, self.kv_ld = max(row, w.inner.expand.kp), w.inner.expand.n
        absorbed, partial, sums = r.latent_scratch(row, self.lat_ld, s.heads, L.round_up(s.rank, 16), self.kv_ld)
        ints = [r.proj.stride(0), q, c, rot, g, out.stride(0), s.heads, s.dim, s.rot_dim, s.vdim, s.rank, r.max_pages, r.kv.page_size,
                absorbed.shape[0], partial.shape[0], r.kv.num_pages]
        self.call = {id(rows): L.MixerCall([r.proj, w.vectors["dkv.norm"], r.angles(s.rotary), rows.positions, rows.slots, r.block_table, r.kv.rows[index],
                                            w.inner.keys, w.inner.values, absorbed, partial, sums, r.status, out], ints, [r.cfg.eps, s.scale, branch.scale])
                     for rows in (r.slot_rows, r.batch_rows)}

    def splits(self, rows: int) -> tuple[int, int]:
        """KV splits of the absorbed form, a power of two, and how many of them share a sum: at most a CTA per SM (of those that clusters
        reach), and no more than there are tiles of 64 keys at full length."""
        lib, n = L.lib(), 1
        while 2 * n <= min(lib.bonsai_lay_latent_max_splits(), self.r.scratch.sms // (rows * self.groups), -(-self.r.max_seq // 64)):
            n *= 2
        # large clusters do not fill the GPU: two of eight in a GPC of 16 to 20 SMs
        return n, min(n, lib.bonsai_lay_latent_max_cluster() if rows * self.groups * n <= 64 else 4)

    def __call__(self, rows: Rows, st: StepShape, stream: int, early: bool) -> None:
        lib, a, r = L.lib(), self.call[id(rows)].args, self.r
        if r.exact:
            K.check(lib.bonsai_lay_latent_append(*a, 0, st.rows, 1, stream), "latent_append")
            K.check(lib.bonsai_lay_latent_f32(*a, st.rows, stream), "latent_f32")
            return
        if st.short:
            n, cluster = self.splits(st.short)
            K.check(lib.bonsai_lay_latent_query(*a, st.short, stream), "latent_query")
            K.check(lib.bonsai_lay_latent_decode(*a, st.short, n, cluster, stream), "latent_decode")
            K.check(lib.bonsai_lay_latent_value(*a, st.short, n // cluster, stream), "latent_value")
        if st.rows > st.short:
            K.check(lib.bonsai_lay_latent_append(*a, st.short, st.rows - st.short, 0, stream), "latent_append")
        for g in st.contexts:
            lat, kv = r.latents[self.row, self.lat_ld], r.expanded[: r.context_rows * self.kv_ld].view(-1, self.kv_ld)
            K.check(lib.bonsai_lay_latent_gather(*a, g.contexts, g.count, g.longest, lat.data_ptr(), self.lat_ld, stream), "latent_gather")
            L.linear(self.w.inner.expand, lat, g.rows, kv, r.scratch)
            K.check(lib.bonsai_lay_latent_prompt(*a, g.portions, g.contexts, g.tiles, g.n_tiles, kv.data_ptr(), self.kv_ld, lat.data_ptr(), self.lat_ld, stream),
                    "latent_prompt")

    def launches(self) -> int:
        return 2 if self.r.exact else 3


class MlstmMixer:
    def __init__(self, r: "LayeredRunner", index: int, branch: Branch, w: BranchWeights, out: torch.Tensor):
        self.r, self.spec, self.w, self.out, cfg = r, branch.spec, w, out, r.cfg
        spec, s = self.spec, r.states.tensors[index]
        assert branch.scale == 1.0, "an mLSTM output is not scaled"
        q, k, v, self.g_col, i, f = w.columns
        self.chunked = not r.exact and runs_chunked(spec)
        self.plan = segment_plan(spec)
        self.fused = spec.vdim <= L.lib().bonsai_lay_mlstm_fused_vdim()
        floats = [spec.gate_cap, cfg.eps, spec.den_eps, spec.dim ** -0.5]

        def call(rows, out):
            return L.MixerCall([r.proj, self.w.vectors["i.b"], self.w.vectors["f.b"], self.w.vectors["norm"], s["S"], s["n"], s["m"], rows.positions,
                                rows.slots, r.state_table, out, *r.segment_scratch],
                               [r.proj.stride(0), q, k, v, self.g_col, i, f, out.stride(0), spec.heads, spec.dim, spec.vdim], floats)
        # o f32 for the gated head norm, and the finished activations of the fused single-token step
        self.raw = {id(rows): call(rows, r.head_out) for rows in (r.slot_rows, r.batch_rows)}
        self.done = {id(rows): call(rows, self.out) for rows in (r.slot_rows, r.batch_rows)}

    def _finish(self, row0: int, count: int) -> None:
        s = self.spec
        L.gated_norm(self.r.head_out, row0, self.r.proj, self.g_col, self.w.vectors["norm"], self.r.cfg.eps, count, s.heads, s.vdim, self.out)

    def __call__(self, rows: Rows, st: StepShape, stream: int, early: bool) -> None:
        lib = L.lib()
        if st.singles and self.fused:
            K.check(lib.bonsai_lay_mlstm_step(*self.done[id(rows)].args, None, st.singles, 2 if self.r.exact else 1, stream), "mlstm_step")
        elif st.singles:
            K.check(lib.bonsai_lay_mlstm_step(*self.raw[id(rows)].args, None, st.singles, 3, stream), "mlstm_step")
            self._finish(0, st.singles)
        if st.portions:
            a = self.raw[id(rows)].args
            if self.chunked:
                K.check(lib.bonsai_lay_mlstm_chunk(*a, st.entries, st.portions, *st.cut(self.plan), stream), "mlstm_chunk")
            else:
                K.check(lib.bonsai_lay_mlstm_step(*a, st.entries, st.portions, 0, stream), "mlstm_step")
            self._finish(st.singles, st.rows - st.singles)

    def launches(self) -> int:
        return 1 if self.fused else 2


class LinearRecurrenceMixer:
    def __init__(self, r: "LayeredRunner", index: int, branch: Branch, w: BranchWeights, out: torch.Tensor):
        self.r, self.spec, self.scale, self.out, cfg = r, branch.spec, branch.scale, out, r.cfg
        spec, s, lib, vec = self.spec, r.states.tensors[index], L.lib(), w.vectors
        self.norm = vec.get("norm")
        self.chunked = not r.exact and runs_chunked(spec)
        self.plan = segment_plan(spec)
        # the single-token step finishes its outputs itself when the norm is per head
        self.fused = spec.norm_parts == spec.heads and not spec.gate_first and spec.vdim <= lib.bonsai_lay_rec_fused_vdim()
        decay = rate = conv_w = freq = None
        if spec.decay is None:
            self.g_col, conv, dt = w.columns
            v, k, q = conv, conv + spec.out_width, conv + spec.out_width + spec.groups * spec.dim
            rate = torch.exp(vec["A_log"])
        else:
            q, k, v, self.g_col = w.columns
            conv = dt = 0
            decay = torch.tensor(spec.decay, dtype=torch.float32, device=r.device)
        if spec.conv:
            conv_w = vec["conv"].flip(1).t().contiguous()              # [taps][channels], the current token's tap first
        if spec.rotary is not None:
            freq = torch.tensor(spec.rotary.frequencies, dtype=torch.float64, device=r.device)
        floats = [cfg.eps, spec.key_scale, self.scale]

        def call(rows, dst):
            return L.MixerCall([r.proj, decay, rate, vec.get("dt_bias"), vec.get("D"), self.norm, conv_w, vec.get("conv.b"), s.get("conv"), freq, s["S"],
                                rows.positions, rows.slots, r.state_table, dst, r.features, r.segment_scratch[0], r.segment_scratch[3]],
                               [r.proj.stride(0), q, k, v, self.g_col, dt, conv, dst.stride(0), r.features.stride(0), spec.heads, spec.groups, spec.dim,
                                spec.vdim, int(spec.activation), spec.conv, spec.conv_channels if spec.conv else 0,
                                spec.rotary.dims if spec.rotary else 0, int(spec.gate == "silu")], floats)
        # o f32 for the gated norm, and the finished activations of the fused single-token step
        self.raw = {id(rows): call(rows, r.head_out) for rows in (r.slot_rows, r.batch_rows)}
        self.done = {id(rows): call(rows, out) for rows in (r.slot_rows, r.batch_rows)}

    def _finish(self, row0: int, count: int) -> None:
        s = self.spec
        L.gated_norm(self.r.head_out, row0, self.r.proj, self.g_col, self.norm, self.r.cfg.eps, count, s.norm_parts, s.out_width // s.norm_parts, self.out,
                     s.gate, s.gate_first, self.scale)

    def __call__(self, rows: Rows, st: StepShape, stream: int, early: bool) -> None:
        lib, exact = L.lib(), int(self.r.exact)
        if st.singles and self.fused:
            K.check(lib.bonsai_lay_rec_step(*self.done[id(rows)].args, None, st.singles, 2, exact, int(early), stream), "rec_step")
        elif st.singles:
            K.check(lib.bonsai_lay_rec_step(*self.raw[id(rows)].args, None, st.singles, 1, exact, int(early), stream), "rec_step")
            self._finish(0, st.singles)
        if st.portions:
            a = self.raw[id(rows)].args
            K.check(lib.bonsai_lay_rec_features(*a, st.singles, st.rows - st.singles, exact, stream), "rec_features")
            if self.spec.conv:
                K.check(lib.bonsai_lay_rec_ring(*a, st.entries, st.portions, stream), "rec_ring")
            if self.chunked:
                K.check(lib.bonsai_lay_rec_chunk(*a, st.entries, st.portions, *st.cut(self.plan), stream), "rec_chunk")
            else:
                K.check(lib.bonsai_lay_rec_step(*a, st.entries, st.portions, 0, exact, 0, stream), "rec_step")
            self._finish(st.singles, st.rows - st.singles)

    def launches(self) -> int:
        return 1 if self.fused else 2


class MinGruMixer:
    def __init__(self, r: "LayeredRunner", index: int, branch: Branch, w: BranchWeights, out: torch.Tensor):
        self.r, self.spec, vec = r, branch.spec, w.vectors
        assert branch.scale == 1.0, "a minGRU output is not scaled"
        self.call = {id(rows): L.MixerCall([r.proj, vec["z.b"], vec["x.b"], r.states.tensors[index]["S"], rows.positions, rows.slots, r.state_table, out],
                                           [r.proj.stride(0), *w.columns, out.stride(0), self.spec.width], [])
                     for rows in (r.slot_rows, r.batch_rows)}

    def cluster(self, portions: int, tokens: int) -> int:
        """CTAs that share a portion: about four per SM, and no more than have tokens at a time."""
        n, ctas = 1, portions * -(-self.spec.width // 32)
        while n < 8 and 2 * n * ctas <= 4 * self.r.scratch.sms and 2 * n * L.lib().bonsai_lay_gru_tokens() <= tokens:
            n *= 2
        return n

    def __call__(self, rows: Rows, st: StepShape, stream: int, early: bool) -> None:
        lib, a, exact = L.lib(), self.call[id(rows)].args, int(self.r.exact)
        if st.singles:
            K.check(lib.bonsai_lay_gru_step(*a, st.singles, exact, stream), "gru_step")
        if st.portions:
            n = self.cluster(st.portions, (st.rows - st.singles) // st.portions)
            K.check(lib.bonsai_lay_gru_scan(*a, st.entries, st.portions, n, exact, stream), "gru_scan")

    def launches(self) -> int:
        return 1


class SelectiveScanMixer:
    def __init__(self, r: "LayeredRunner", index: int, branch: Branch, w: BranchWeights, out: torch.Tensor):
        self.r, self.spec, self.w, s, vec = r, branch.spec, w.inner, branch.spec, w.vectors
        assert branch.scale == 1.0, "a selective scan's output is not scaled"
        self.plan = segment_plan(s)
        state, (x_col, z_col), (dt_col, b_col, c_col) = r.states.tensors[index], w.columns, w.inner.read.columns
        self.x, self.bc, self.dt, self.low = r.scan_buffers(s, w.inner)
        A = torch.zeros((s.channels, state["S"].shape[-1]), dtype=torch.float32, device=r.device)
        A[:, : s.states] = -torch.exp(vec["A_log"])
        taps = L.conv_weight(vec["conv"])
        ints = [r.proj.stride(0), z_col, self.bc.stride(0), b_col, c_col, self.dt.stride(0), self.x.stride(0), out.stride(0), s.channels, s.states]
        self.call, self.conv = {}, {}
        for rows in (r.slot_rows, r.batch_rows):
            self.call[id(rows)] = L.MixerCall([r.proj, self.bc, self.dt, self.x, vec["dt.b"], A, vec["D"], state["S"], rows.positions, rows.slots, r.state_table, out,
                                               *r.scan_scratch], ints, [])
            self.conv[id(rows)] = L.Conv(r.proj, x_col, s.channels, taps, vec["conv.b"], state["conv"], rows, r.state_table, self.x, silu=True)

    def __call__(self, rows: Rows, st: StepShape, stream: int, early: bool) -> None:
        lib, a, r, s, T = L.lib(), self.call[id(rows)].args, self.r, self.spec, st.rows
        exact = int(r.exact)
        self.conv[id(rows)](st)
        L.linear(self.w.read, self.x, T, self.bc, r.scratch)
        if not r.exact:
            L.narrow(self.bc, 0, s.rank, T, self.low)
        L.linear(self.w.step, self.bc if r.exact else self.low, T, self.dt, r.scratch)
        if st.singles:
            K.check(lib.bonsai_lay_scan_step(*a, st.singles, exact, stream), "scan_step")
        if st.portions:
            segs, n, prompts = (0, 0, 0) if r.exact else st.cut(self.plan)
            K.check(lib.bonsai_lay_scan(*a, st.entries, st.portions, segs, n, prompts, exact, stream), "scan")

    def launches(self) -> int:
        return 4 if self.r.exact else 5


MIXERS = {"attention": AttentionMixer, "latent": LatentAttentionMixer, "mlstm": MlstmMixer, "recurrence": LinearRecurrenceMixer, "mingru": MinGruMixer,
          "selective": SelectiveScanMixer}


class LayeredRunner(SlotState):
    """Owns the activation buffers, the caches and the captured decode steps of a layer-list decoder.  Same surface as
    ``Qwen3Runner`` where the engine and the scheduler use it."""

    sample_fn = staticmethod(L.sample)

    def __init__(self, weights: LayeredWeights, kv: RowCache, states: StatePool, max_batch: int, max_seq: int, exact: bool = False,
                 prefill_chunk: int = 4096):
        self.w, self.kv, self.states, self.exact = weights, kv, states, exact
        self.cfg, self.device = weights.cfg, weights.device
        self.max_batch, self.max_seq = max_batch, max_seq
        self.max_pages = -(-max_seq // kv.page_size)
        self.capacity = max(int(prefill_chunk), 64, max_batch)         # rows of a step
        self.prefill_capacity = self.capacity
        cfg, dev, cap = self.cfg, self.device, self.capacity
        f32, i32 = dict(dtype=torch.float32, device=dev), dict(dtype=torch.int32, device=dev)
        self.init_slots(max_batch, self.max_pages, cfg.vocab, dev)
        self.logits = torch.zeros((max_batch, cfg.vocab), **f32)
        self.state_table = torch.zeros(max_batch, **i32)
        self._state_row: dict[int, int] = {}
        self.kv_pools = {kv.kvt: kv}
        self.slot_formats = [kv.kvt] * max_batch
        self.scratch = L.GemmScratch(dev, self.status)
        # activations; the padding columns of the bf16 buffers stay zero for the projections that read them
        self._acts: dict[int, torch.Tensor] = {}
        self.x = torch.zeros((cap, cfg.width), **f32)
        # input of the next projection; without a norm in between, that of the exact mode is the stream itself
        self.h = self.x if exact and not (cfg.pre_norm or cfg.side_by_side) else self.act_buffer(cfg.width, shared=False)
        self.n32 = torch.zeros((cap if cfg.input_taps else 1, L.round_up(cfg.width, 4)), **f32)     # what a convolution reads
        self.normed = self.act_buffer(cfg.width, shared=False)
        self.y = torch.zeros((cap, L.round_up(cfg.width, 4)), **f32)
        self.proj = torch.zeros((cap, max(L.round_up(l.proj.n, 4) for l in weights.layers)), **f32)
        recurrent = [cfg.recurrence(i) for i in cfg.recurrent_layers]
        heads = [m.out_width for m in recurrent if isinstance(m, (MlstmSpec, LinearRecurrenceSpec))]
        self.head_out = torch.zeros((cap if heads else 1, L.round_up(max(heads, default=4), 4)), **f32)
        # prepared queries, keys and values of prompt rows
        linear = [m for m in recurrent if isinstance(m, LinearRecurrenceSpec)]
        width = max((L.lib().bonsai_lay_rec_features_width(m.heads, m.groups, m.dim, m.vdim) for m in linear), default=8)
        self.features = torch.zeros((cap if linear else 1, width), dtype=torch.float32 if exact else torch.bfloat16, device=dev)
        # states of the segments a long prompt is cut into (layers run one after another and share them)
        chunked = [] if exact else [m for m in recurrent if runs_chunked(m)]
        shapes = [(m.heads, *state_dims(m)) for m in chunked]
        scans = [m for m in recurrent if isinstance(m, SelectiveScanSpec)]
        self.segment_plans = sorted({segment_plan(m) for m in chunked + ([] if exact else scans)}, key=lambda p: p.ctas)
        parts = 0 if exact else MAX_SEGMENTS
        self.scan_scratch = [torch.empty(max(1, parts * max((m.channels * n(m) for m in scans), default=0)), **f32) for n in
                             (lambda m: L.lib().bonsai_lay_scan_states(m.states), lambda m: 1)]
        self._scan_buffers: dict[tuple, list[torch.Tensor]] = {}
        segs = MAX_SEGMENTS if shapes else 0
        self.segment_scratch = [torch.empty(max(1, segs * max((f(*s) for s in shapes), default=0)), **f32) for f in
                                (lambda h, d, e: h * d * e, lambda h, d, e: h * d * e // 64, lambda h, d, e: h * e // 64, lambda h, d, e: h * e // 32)]
        # tables of rotations and the scratch of latent attention, filled by the mixers that need them
        self._angles: dict[RotarySpec, torch.Tensor] = {}
        self.short_rows = max(SHORT_ROWS, max_batch)
        self.context_rows = max(cap, L.round_up(max_seq, kv.page_size))
        self.latents: dict[tuple[int, int], torch.Tensor] = {}
        self.expanded = torch.empty(0, dtype=torch.bfloat16, device=dev)
        self._absorbed: dict[tuple, list[torch.Tensor]] = {}
        # row metadata: decode steps use the slot tensors as they are; a mixed batch uploads [tokens | positions | slots | lists]
        self.slot_rows = Rows(self.tokens, self.positions, torch.arange(max_batch, **i32))
        attention = [cfg.attention(i) for i in cfg.attention_layers]
        conv = {L.lib().bonsai_lay_conv_rows()} if cfg.input_taps or scans else set()
        self._tile_sizes = sorted({64 // s.group for s in attention if isinstance(s, AttentionSpec)} | conv)
        self._expands = not exact and any(isinstance(s, LatentAttentionSpec) for s in attention)
        self._meta = torch.zeros(3 * cap + 4 * cap + 8 * MAX_SEGMENTS * len(self.segment_plans) + 2 * cap * len(self._tile_sizes) + 2 * cap + 12 * max_batch + 64, **i32)
        self.batch_rows = Rows(*(self._meta[i * cap:(i + 1) * cap] for i in range(3)))
        self._host = [torch.zeros(self._meta.numel(), dtype=torch.int32).pin_memory() for _ in range(2)]
        self._host_free = [torch.cuda.Event() for _ in range(2)]
        self._turn = 0
        self.runs = cfg.runs
        self.mixers, self.mixer_out = [], []           # per run: the branches' mixers and the buffer they write
        for n, run in enumerate(self.runs):
            spec, w = cfg.layer_specs[run.layer], weights.layers[run.layer]
            widths = tuple(b.spec.out_width for b in spec.mixer.branches)
            out = self.act_buffer(*widths)
            self.mixer_out.append(out)
            self.mixers.append([MIXERS[b.spec.kind](self, n, b, bw, out[:, bw.offset:]) for b, bw in zip(spec.mixer.branches, w.branches)])
        specs = [cfg.experts(i) for i in cfg.expert_layers]
        shared = L.ExpertScratch(cap, cfg.width, specs, exact, dev) if specs else None
        routers = [weights.layers[i].mlp.router for i in cfg.expert_layers]
        self.router_out = torch.zeros((cap, max((L.round_up(w.n, 4) for w in routers if w is not None), default=4)), **f32) if routers and not cfg.side_by_side else self.proj
        self.experts = {i: L.Routing(cfg.experts(i), w.mlp.up, w.mlp.down, w.mlp.correction, self.router_out, w.mlp.column, shared)
                        for i, w in enumerate(weights.layers) if i in cfg.expert_layers}
        self.row_steps = {id(rows): self._row_steps(rows) for rows in (self.slot_rows, self.batch_rows)} if cfg.row_steps else None
        self._branch, self._forked = torch.cuda.Stream(dev), False
        self._graphs: dict[tuple, torch.cuda.CUDAGraph] = {}

    def angles(self, rot: RotarySpec) -> torch.Tensor:
        """Cosines and sines of a rotation at every position the pages can hold, from angles in double precision."""
        if rot not in self._angles:
            f64 = dict(dtype=torch.float64, device=self.device)
            a = torch.outer(torch.arange(self.max_pages * self.kv.page_size, **f64), torch.tensor(rot.frequencies, **f64))
            self._angles[rot] = torch.stack([a.cos(), a.sin()], dim=-1).float().contiguous()
        return self._angles[rot]

    def latent_scratch(self, row: int, lat_ld: int, heads: int, rank: int, kv_ld: int) -> list[torch.Tensor]:
        """Absorbed queries, partial sums and their maxima for rows of one latent attention layer (layers of equal sizes share them);
        also makes room for its gathered and expanded rows."""
        bf16, f32 = dict(dtype=torch.bfloat16, device=self.device), dict(dtype=torch.float32, device=self.device)
        if not self.exact:
            if (row, lat_ld) not in self.latents:
                self.latents[row, lat_ld] = torch.zeros((self.context_rows, lat_ld), **bf16)
            if self.expanded.numel() < self.context_rows * kv_ld:
                self.expanded = torch.empty(self.context_rows * kv_ld, **bf16)
        if (row, heads, rank) not in self._absorbed:
            rows, parts = (1, 1) if self.exact else (self.short_rows, max(self.short_rows, self.scratch.sms))
            self._absorbed[row, heads, rank] = [torch.zeros((rows, heads, row), **bf16), torch.empty((parts, heads, rank), **f32),
                                                torch.empty((parts, heads, 2), **f32)]
        return self._absorbed[row, heads, rank]

    def scan_buffers(self, m: SelectiveScanSpec, w: ScanWeights) -> list[torch.Tensor]:
        """Convolved channels, their projection, step sizes, and the 16-bit low-rank part of one selective-scan layer (layers of equal
        sizes share them; the padding of what projections read stays zero)."""
        key = (m.channels, m.states, m.rank)
        if key not in self._scan_buffers:
            new = lambda n, ld, dtype: torch.zeros((n, ld), dtype=dtype, device=self.device)
            act, cap = torch.float32 if self.exact else torch.bfloat16, self.capacity
            self._scan_buffers[key] = [new(cap, L.round_up(m.channels, 4) if self.exact else w.read.kp, act), new(cap, L.round_up(w.read.n, 4), torch.float32),
                                       new(cap, L.round_up(m.channels, 4), torch.float32), new(1 if self.exact else cap, w.step.kp, torch.bfloat16)]
        return self._scan_buffers[key]

    def act_buffer(self, *widths: int, shared: bool = True) -> torch.Tensor:
        """Input buffer of a projection that reads blocks of ``widths`` columns (:func:`branch_offsets`): f32 in the exact mode, else
        bf16 padded to the tensor-core width.  One per layout, so that the padding never holds another layer's values."""
        if shared and widths in self._acts:
            return self._acts[widths]
        ld = L.round_up(branch_offsets(widths)[1], 4 if self.exact else L.K_ALIGN)
        t = torch.zeros((self.capacity, ld), dtype=torch.float32 if self.exact else torch.bfloat16, device=self.device)
        if shared:
            self._acts[widths] = t
        return t

    # ---- slots ------------------------------------------------------------------------------------------------------------------
    def bind_state(self, slot: int) -> None:
        if self.cfg.has_state and slot not in self._state_row:
            row = self._state_row[slot] = self.states.alloc()
            self.state_table[slot] = row

    def release_state(self, slot: int) -> None:
        row = self._state_row.pop(slot, None)
        if row is not None:
            self.states.release(row)

    def move_state(self, src: int, dst: int) -> None:
        self.release_state(dst)
        if src in self._state_row:
            self._state_row[dst] = self._state_row.pop(src)
            self.state_table[dst].copy_(self.state_table[src], non_blocking=True)

    def set_slot_format(self, slot: int, kvt: int) -> None:
        if kvt != self.kv.kvt:
            raise ValueError("the layer-list decoders have one cache format per engine")

    # ---- one step ------------------------------------------------------------------------------------------------------------------
    def _row_steps(self, rows: Rows) -> list[L.RowStep]:
        """The row steps of designs that take the general kernel: the start, one behind each sublayer of each run, and the final norm of
        listed rows.  Each leaves the next sublayer's input; the last one behind a sublayer the final norm of all rows."""
        cfg, w = self.cfg, self.w
        common = dict(eps=cfg.eps, groups=cfg.norm_groups or 1)
        subs = [(n, run, j) for n, run in enumerate(self.runs) for j in range(len(cfg.norm_names(run.layer)))]

        def following(k: int) -> dict:
            """What comes between sublayer ``k`` - 1 and sublayer ``k``."""
            if k == len(subs):
                return dict(h=self.normed, next_norm=w.final_norm)
            n, run, j = subs[k]
            l = w.layers[run.layer]
            a = dict(h=self.h, next_norm=l.pre_norm if j == 0 else l.mlp.pre_norm)
            if cfg.input_taps:
                a.update(conv=(l.convs[j], self.states.tensors[n][f"canon{j + 1}"]), n32=self.n32)
            if j == 0 and run.begins is not None:
                a["step"] = w.loop_step[run.begins]
                if run.begins > 0:
                    a.update(table=w.embed.data, scale=cfg.embed_scale)
            return a
        new = lambda **a: L.RowStep(self.x, a.pop("h"), rows, self.state_table, **common, **a)
        steps = [new(fresh=True, **{**following(0), "table": w.embed.data, "scale": cfg.embed_scale})]
        for k, (n, run, j) in enumerate(subs):
            l, a = w.layers[run.layer], following(k + 1)
            if j == 0:
                a.update(y=self.y, bias=l.out_bias, w=l.norm)
            else:
                moe = isinstance(l.mlp, ExpertWeights)
                a["w"] = l.mlp.norm
                if not moe or l.mlp.shared is not None:
                    a["y"] = self.y
                if moe and l.mlp.shared is not None:
                    a["gate"] = self.router_out[:, l.mlp.router.columns[1]:]
            steps.append(new(mult=cfg.residual_mult, **a))
        steps.append(new(h=self.normed, next_norm=w.final_norm))
        return steps

    def _looped_layers(self, rows: Rows, st: StepShape) -> None:
        """:meth:`_layers` of designs whose row steps take the general kernel."""
        T, s, steps = st.rows, K.stream(), iter(self.row_steps[id(rows)])
        next(steps)(T, st)
        for n, run in enumerate(self.runs):
            w = self.w.layers[run.layer]
            L.linear(w.proj, self.h, T, self.proj, self.scratch)
            for k, mixer in enumerate(self.mixers[n]):
                mixer(rows, st, s, early=k > 0)
            L.linear(w.out, self.mixer_out[n], T, self.y, self.scratch)
            next(steps)(T, st)
            if w.mlp is None:
                continue
            experts = self.experts.get(run.layer)
            block = w.mlp
            if experts is not None:
                L.linear(w.mlp.router, self.h, T, self.router_out, self.scratch)
                self._beside(experts, self.h, T)
                block = w.mlp.shared
            if block is not None:
                act = self.act_buffer(block.ff)
                L.linear(block.up, self.h, T, act, self.scratch, block.act)
                L.linear(block.down, act, T, self.y, self.scratch)
            if experts is not None:
                self._join()
            next(steps)(T, st, experts)

    def _layers(self, rows: Rows, st: StepShape, final: bool = False) -> None:
        """Embedding and layers.  ``final``: the last residual step leaves the final norm of all rows in ``normed``."""
        if self.row_steps is not None:
            return self._looped_layers(rows, st)
        cfg, T, s = self.cfg, st.rows, K.stream()
        x, h, layers = self.x, self.h, self.w.layers
        copy = None if h is x else h
        L.embed(self.w.embed.data, rows.tokens, cfg.embed_scale, T, cfg.width, x, copy, layers[0].pre_norm, cfg.eps, cfg.layer_norm)
        for i, (spec, w) in enumerate(zip(cfg.layer_specs, layers)):
            last = i + 1 == len(layers)
            after, following = (self.normed, self.w.final_norm) if last and final else (copy, None if last else layers[i + 1].pre_norm)
            L.linear(w.proj, h, T, self.proj, self.scratch)
            experts = self.experts.get(i)
            if experts is not None:
                self._beside(experts, h, T)
            for n, mixer in enumerate(self.mixers[i]):
                mixer(rows, st, s, early=n > 0)            # only the first one follows the projection directly
            L.linear(w.out, self.mixer_out[i], T, self.y, self.scratch)
            if cfg.side_by_side:
                if experts is not None:
                    self._join()
                L.side_by_side(x, self.y, experts, cfg.residual_mult, T, after, following, cfg.eps, cfg.layer_norm)
            elif w.mlp is None:
                L.norm_add(x, self.y, w.norm, cfg.eps, T, after, following)
            else:
                L.norm_add(x, self.y, w.norm, cfg.eps, T, copy, w.mlp.pre_norm)
                act = self.act_buffer(spec.mlp.ff)
                L.linear(w.mlp.up, h, T, act, self.scratch, w.mlp.act)
                L.linear(w.mlp.down, act, T, self.y, self.scratch)
                L.norm_add(x, self.y, w.mlp.norm, cfg.eps, T, after, following)

    def _beside(self, experts: L.Routing, h: torch.Tensor, T: int) -> None:
        """The experts of a layer, which need the router's projection only: in a captured decode step, a branch beside the mixer's kernels
        or the shared block."""
        main = torch.cuda.current_stream(self.device)
        self._forked = torch.cuda.is_current_stream_capturing()
        if not self._forked:
            experts(h, T, self.scratch)
            return
        self._branch.wait_stream(main)
        with torch.cuda.stream(self._branch):
            experts(h, T, self.scratch)

    def _join(self) -> None:
        if self._forked:
            torch.cuda.current_stream(self.device).wait_stream(self._branch)

    def _head(self, row_list: int, count: int, out: torch.Tensor) -> None:
        """Logits of ``count`` rows (device address of their indices) into ``out`` [count, vocab]."""
        if self.row_steps is None:
            L.norm_rows(self.x, row_list, count, self.w.final_norm, self.cfg.eps, self.normed, self.cfg.layer_norm)
        else:
            self.row_steps[id(self.batch_rows)][-1](count, None, norm_of=row_list)
        self._logits(count, out)

    def _logits(self, count: int, out: torch.Tensor) -> None:
        """The head over the first rows of ``normed``."""
        L.linear(self.w.head, self.normed, count, out, self.scratch, L.SoftCap(self.cfg.logit_cap) if self.cfg.logit_cap > 0 else None)

    def step_eager(self, batch: int, sample: bool = True, lm_head: bool = True, masked: bool = False) -> None:
        """One token for each of the slots 0 .. batch-1 (tokens and positions are read from the slot tensors)."""
        self._layers(self.slot_rows, StepShape(batch, batch, batch), final=lm_head)
        if lm_head:
            self._logits(batch, self.logits)
        if sample:
            self.sample_rows(0, batch, masked, advance=True)

    def step(self, batch: int, sample: bool = True, masked: bool = False) -> None:
        """:meth:`step_eager` replayed from a CUDA graph captured at its first call."""
        key = (batch, sample, masked)
        g = self._graphs.get(key)
        if g is None:
            for w in self.w.layers:                            # allocated outside the capture
                block = w.mlp.shared if isinstance(w.mlp, ExpertWeights) else w.mlp
                if block is not None:
                    self.act_buffer(block.ff)
            g = self._graphs[key] = K.capture_graph(self.device, lambda: self.step_eager(batch, sample, masked=masked))
        mark = nvtx.push(f"decode_step[batch={batch}]")
        g.replay()
        nvtx.pop(mark)

    def run_batch(self, entries: Sequence[tuple[int, Sequence[int], int]], want: Sequence[Sequence[int]], device_tokens: bool = False) -> torch.Tensor:
        """Runs portions of several sequences as one batch.  ``entries``: (slot, tokens, first position) each, the slots
        distinct; ``want``: per entry the places among its tokens whose logits are asked for.  Returns them as f32
        [wanted, vocab], in the order of the entries and of their places.  ``device_tokens``: single-token entries take their
        token from ``tokens[slot]`` on the device (the host's value is ignored)."""
        T = sum(len(e[1]) for e in entries)
        if T == 0 or T > self.capacity:
            raise ValueError(f"a step takes 1 to {self.capacity} tokens, got {T}")
        if len({e[0] for e in entries}) != len(entries):
            raise ValueError("a step takes one entry per slot")
        sizes = [len(e[1]) for e in entries]
        order = sorted(range(len(entries)), key=lambda i: (sizes[i] != 1, sizes[i] > SHORT, i))     # single tokens, then short portions
        cap = self.capacity
        turn = self._turn = (self._turn + 1) % 2
        self._host_free[turn].synchronize()                    # the copy that read this buffer has finished
        host = self._host[turn].numpy()
        lists, row, row0 = [], 0, [0] * len(entries)
        for i in order:
            slot, toks, pos0 = entries[i]
            n = len(toks)
            t = np.asarray(toks, dtype=np.int64)
            if n == 0 or t.min() < 0 or t.max() >= self.cfg.vocab:
                raise ValueError(f"entry of slot {slot}: needs tokens in [0, {self.cfg.vocab})")
            if not 0 <= slot < self.max_batch or pos0 < 0 or pos0 + n > self.max_seq:
                raise ValueError(f"entry of slot {slot}: {n} tokens at position {pos0} do not fit {self.max_batch} slots of {self.max_seq} tokens")
            host[row:row + n] = t
            host[cap + row:cap + row + n] = np.arange(pos0, pos0 + n)
            host[2 * cap + row:2 * cap + row + n] = slot
            if n > 1:
                lists.append((row, n, slot, pos0))
            row0[i] = row
            row += n
        singles = short = sum(n == 1 for n in sizes)
        for _, n, _, _ in lists:
            if n > SHORT or short + n > self.short_rows:
                break
            short += n
        end = -(-3 * cap // 4) * 4
        put = lambda a: (end, end + a.size)
        base = self._meta.data_ptr()
        st = StepShape(T, singles, short, len(lists), base + 4 * end, {}, {})
        if lists:
            a = np.asarray(lists, dtype=np.int32).reshape(-1)
            lo, hi = put(a)
            host[lo:hi] = a
            end = hi
            lengths = [n for _, n, _, _ in lists]
            for plan in self.segment_plans:
                size = plan_segments(lengths, plan, self.scratch.sms)
                if not size:
                    continue
                segs, prompts = [], []
                for first, n, slot, pos0 in lists:
                    cuts = range(0, n, size * CHUNK)
                    prompts.append((slot, pos0, len(segs), len(cuts)))
                    segs += [(first + c, min(size * CHUNK, n - c), slot, int(c == cuts[-1])) for c in cuts]
                a = np.asarray(segs + prompts, dtype=np.int32).reshape(-1)
                lo, hi = put(a)
                host[lo:hi] = a
                st.segments[plan] = (len(segs), base + 4 * lo, base + 4 * (lo + 4 * len(segs)))
                end = hi
            groups = group_contexts([e for e in lists if e[0] >= short], self.context_rows) if self._expands else []
            for g in groups:                                      # blocks of four words, ahead of the lists of two
                first = np.cumsum([0] + [n + pos0 for _, n, _, pos0 in g])
                a = np.asarray(g + [(f, n + pos0, slot, 0) for f, (_, n, slot, pos0) in zip(first, g)], dtype=np.int32).reshape(-1)
                lo, hi = put(a)
                host[lo:hi] = a
                at = base + 4 * lo
                st.contexts.append(ContextGroup(at, at + 16 * len(g), len(g), 0, 0, int(first[-1]), max(n + pos0 for _, n, _, pos0 in g)))
                end = hi
            for c, g in zip(st.contexts, groups):
                a = np.asarray([(e, t) for e, (_, n, _, _) in enumerate(g) for t in range(0, n, CONTEXT_TILE)], dtype=np.int32).reshape(-1)
                lo, hi = put(a)
                host[lo:hi] = a
                c.tiles, c.n_tiles, end = base + 4 * lo, a.size // 2, hi
            for size in self._tile_sizes:
                a = np.asarray([(e, t) for e, (_, n, _, _) in enumerate(lists) for t in range(0, n, size)], dtype=np.int32).reshape(-1)
                lo, hi = put(a)
                host[lo:hi] = a
                st.tiles[size] = (base + 4 * lo, a.size // 2)
                end = hi
        wanted = np.asarray([row0[i] + p for i, ps in enumerate(want) for p in ps], dtype=np.int32)
        host[end:end + wanted.size] = wanted
        rows_at = base + 4 * end
        end += wanted.size
        self._meta[:end].copy_(self._host[turn][:end], non_blocking=True)
        self._host_free[turn].record()
        if device_tokens and singles:
            idx = self.batch_rows.slots[:singles].long()
            self.batch_rows.tokens[:singles].copy_(torch.index_select(self.tokens, 0, idx))
        mark = nvtx.push(f"batch[rows={T},singles={singles},portions={len(lists)}]")
        self._layers(self.batch_rows, st)
        out = torch.empty((wanted.size, self.cfg.vocab), dtype=torch.float32, device=self.device)
        if wanted.size:
            self._head(rows_at, wanted.size, out)
        nvtx.pop(mark)
        return out

    def prefill(self, tokens: Sequence[int], slot: int, pos0: int = 0, chunk: int = 4096) -> None:
        """Runs prompt ``tokens`` of the sequence in ``slot`` from position ``pos0`` on; leaves the logits of the last one in
        ``logits[slot]``."""
        n, chunk = len(tokens), max(1, min(chunk, self.capacity))
        for done in range(0, n, chunk):
            part = tokens[done:done + chunk]
            last = done + len(part) == n
            out = self.run_batch([(slot, part, pos0 + done)], [[len(part) - 1] if last else []])
            if last:
                self.logits[slot].copy_(out[0], non_blocking=True)

    def kernel_launches(self, batch: int, sample: bool = True) -> int:
        """Launches of one decode step (each is one of this library's kernels)."""
        n = 2 + int(sample)
        for run, mixers in zip(self.runs, self.mixers):
            mlp = self.w.layers[run.layer].mlp
            if mlp is None:
                k = 0
            elif isinstance(mlp, ExpertWeights):       # behind the mixer: its own projection and row step, and the shared block
                k = self.experts[run.layer].launches(batch) + (0 if self.cfg.side_by_side else 2) + (0 if mlp.shared is None else 2)
            else:
                k = 3
            n += 3 + sum(m.launches() for m in mixers) + k
        return n
