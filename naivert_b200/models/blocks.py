"""Models described as an ordered list of layers: each layer has a token mixer and, optionally, a feed-forward.

The mechanisms are independent of one another and carry their own sizes and constants, so a design is a list of
``LayerSpec`` plus the sizes of its stream.  ``StackSpec`` offers what the rest of the framework asks of a model
(vocabulary, stop tokens, cache bytes); the runtime that executes it is ``runtime/stack.py``.

A *run* is one execution of a layer: a layer inside the loop runs once per pass with the same weights, and every run
has its own cache or state.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Dict, List, Optional, Tuple, Union

from .spec import MoeRoutingSpec

# widths of the kernels (csrc/stack*.cu, csrc/router.cuh)
MAX_EXPERTS, MAX_TOP_K, MAX_GROUPS = 256, 32, 32
MAX_HEAD_DIM = 512
MAX_RANK = 4096
MAX_STEP_INPUT = 40000           # values a product of the one-token step can take in
MAX_STATE_DIM = 512              # key width of a matrix state


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Causal softmax attention without positions over one cached, normed latent per token, with an output gate."""

    heads: int
    dim: int                # query / key width of a head
    vdim: int               # value width of a head
    kv_rank: int            # cached latent
    q_rank: int             # query latent
    scale: float
    kind: str = "latent_attention"


@dataclass(frozen=True)
class GatedRecurrenceSpec:
    """Two branches of ``width``: a GELU gate and a short causal convolution feeding a gated linear recurrence whose
    gates are block-diagonal products (``log a = -decay * r * softplus(lam)``)."""

    width: int
    blocks: int
    taps: int
    decay: float = 8.0
    kind: str = "rglru"

    @property
    def block(self) -> int:
        return self.width // self.blocks

    @property
    def hist_rows(self) -> int:
        """Ring rows of the convolution history: a step writes its input while the previous ``taps - 1`` are read."""
        return max(1, 2 * (self.taps - 1))


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first ``dims`` columns of a head (column i paired with i + dims / 2) by position * freq[i]."""

    dims: int
    base: float
    factor: float = 1.0              # linear scaling: every frequency is divided by it

    def frequencies(self) -> List[float]:
        return [self.base ** (-2.0 * i / self.dims) / self.factor for i in range(self.dims // 2)]


@dataclass(frozen=True)
class GroupedAttentionSpec:
    """Softmax attention with shared key / value heads, norms per head, rotary positions and biases; with ``window`` > 0
    positions fall into chunks [0, window), [window, 2 window), ... and a query sees its own chunk only."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: Optional[RotarySpec] = None
    window: int = 0
    kind: str = "grouped_attention"


@dataclass(frozen=True)
class DeltaStateSpec:
    """Gated delta rule with a decay per head and key channel; short convolutions ahead of q, k and v; the decay and the
    output gate come through low-rank products (``decay_rank``, ``gate_rank``)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int
    gate_rank: int
    kind: str = "channel_delta"

    @property
    def conv_columns(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def hist_rows(self) -> int:
        """Ring rows of the convolution history (see ``GatedRecurrenceSpec.hist_rows``)."""
        return max(1, 2 * (self.taps - 1))

    def state_floats(self, hidden: int) -> int:
        return _pad(self.heads * self.vdim * _pad(self.dim, 4), 4)


@dataclass(frozen=True)
class BonusStateSpec:
    """Time mixing with the previous token ahead of every product, a data-dependent decay per channel (low-rank) and a bonus
    for the current token."""

    heads: int
    dim: int
    decay_rank: int
    kind: str = "wkv"

    @property
    def vdim(self) -> int:
        return self.dim

    def state_floats(self, hidden: int) -> int:
        """The matrices, then the previous token's input."""
        return self.shift_at + _pad(hidden, 4)

    @property
    def shift_at(self) -> int:
        return self.heads * self.dim * _pad(self.dim, 4)


@dataclass(frozen=True)
class NormalizedStateSpec:
    """Matrix memory with exponential gates (log gates capped at ``cap``), a normaliser and a running maximum."""

    heads: int
    dim: int
    vdim: int
    cap: float
    kind: str = "mlstm"

    def state_floats(self, hidden: int) -> int:
        """The matrices with the normaliser as one more column, then the maxima."""
        return _pad(self.heads * (self.vdim + 1) * _pad(self.dim, 4) + self.heads, 4)


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers over one input; the sublayer is the mean of the two branches after an RMS norm each."""

    left: GroupedAttentionSpec
    right: NormalizedStateSpec
    kind: str = "parallel"


@dataclass(frozen=True)
class ClampedGluSpec:
    """min(g, limit) * sigmoid(alpha * g) * (clamp(u, -limit, limit) + 1) between two products."""

    ff: int
    limit: float
    alpha: float = 1.702
    kind: str = "dense"


@dataclass(frozen=True)
class SquaredReluSpec:
    """relu(.)^2 between two products."""

    ff: int
    kind: str = "relu2"


@dataclass(frozen=True)
class ExpertsSpec:
    """Routed SiLU-GLU experts; ``routing`` carries scores, group limit and weights."""

    routing: MoeRoutingSpec
    kind: str = "moe"

    @property
    def ff(self) -> int:
        return self.routing.intermediate


Mixer = Union[LatentAttentionSpec, GatedRecurrenceSpec, DeltaStateSpec, BonusStateSpec, ParallelSpec]
FeedForward = Union[ClampedGluSpec, SquaredReluSpec, ExpertsSpec]


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mixer
    mlp: Optional[FeedForward]
    weights_of: Optional[int] = None     # layer whose tensors this one uses (cache and state stay its own)


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start .. stop - 1`` run ``times`` times in a row; a learned vector is added to the stream ahead of each pass."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerRun:
    run: int                         # index among all runs: owns a cache or state
    layer: int                       # whose weights
    pass_start: Optional[int]        # pass whose vector is added to the stream first


@dataclass(frozen=True)
class StackSpec:
    name: str
    architecture: str
    hidden: int
    vocab: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    loop: Optional[LoopSpec] = None
    norm: str = "rms"                # kind of the norms around a sublayer and of the last one: "rms" or "layer"
    pre_norm: bool = True            # a sublayer reads the normed stream (else the stream itself); its output is always normed
    tied_head: bool = True           # the output product uses the embedding table
    stop_token_ids: Tuple[int, ...] = ()
    think_end_token_id: int = -1
    draft: None = None               # no block draft: rounds commit one token

    @property
    def layer_count(self) -> int:
        return len(self.layers)

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ValueError(f"{self.name}: layer {i} borrows its weights in a circle")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def runs(self) -> List[LayerRun]:
        out: List[Tuple[int, Optional[int]]] = []
        n, lp = len(self.layers), self.loop
        if lp is None:
            out = [(i, None) for i in range(n)]
        else:
            out = [(i, None) for i in range(lp.start)]
            for t in range(lp.times):
                out += [(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
            out += [(i, None) for i in range(lp.stop, n)]
        return [LayerRun(k, i, t) for k, (i, t) in enumerate(out)]

    def vocab_shard(self, tp: int) -> int:
        if tp != 1:
            raise ValueError(f"{self.architecture} runs on one GPU (tp=1); tp={tp} was asked for")
        return self.vocab

    def with_layers(self, n: int) -> "StackSpec":
        """The first ``n`` layers (a loop that would be cut is dropped)."""
        if not 1 <= n <= len(self.layers):
            raise ValueError(f"layer count {n} outside 1..{len(self.layers)}")
        loop = self.loop if self.loop is not None and self.loop.stop <= n else None
        first: Dict[int, int] = {}                     # borrowers of a layer that is cut share among themselves
        layers = []
        for i, layer in enumerate(self.layers[:n]):
            j = self.owner(i)
            j = first.setdefault(j, i) if j >= n else j
            layers.append(replace(layer, weights_of=None if j == i else j))
        return replace(self, name=f"{self.name}-L{n}", layers=tuple(layers), loop=loop)

    def kv_bytes_per_token(self, tp: int = 1, element_bytes: int = 2) -> int:
        self.vocab_shard(tp)
        total = 0
        for r in self.runs():
            m = self.layers[r.layer].mixer
            if m.kind == "latent_attention":
                total += _pad(m.kv_rank, 16) * element_bytes
            elif m.kind == "parallel":
                total += m.left.kv_heads * (_pad(m.left.dim, 8) + _pad(m.left.vdim, 8)) * element_bytes
        return total

    def validate(self) -> "StackSpec":
        """Refuse what the kernels cannot run, by name, before anything is allocated."""
        def need(ok: bool, what: str) -> None:
            if not ok:
                raise ValueError(f"{self.name}: {what}")
        need(self.hidden >= 1 and self.vocab >= 1 and len(self.layers) >= 1, "empty model")
        need(self.hidden <= 25600, "width above 25600")
        for i, layer in enumerate(self.layers):
            m, f = layer.mixer, layer.mlp
            if m.kind == "parallel":
                widest = max(m.left.heads * _pad(m.left.vdim, 8), m.right.heads * m.right.vdim)
            else:
                widest = m.width if m.kind == "rglru" else m.heads * _pad(m.vdim, 8)
            if f is not None:
                widest = max(widest, _pad(f.ff, 8) * (f.routing.top_k if f.kind == "moe" else 1))
            need(widest <= MAX_STEP_INPUT, f"layer {i}: a product of the step would take in {widest} values, at most {MAX_STEP_INPUT}")
        need(self.norm in ("rms", "layer"), f"unknown norm {self.norm!r}")
        for i, layer in enumerate(self.layers):
            j = layer.weights_of
            if j is not None:
                need(0 <= j < len(self.layers), f"layer {i}: no layer {j} to take weights from")
                own = self.layers[self.owner(i)]
                need((own.mixer, own.mlp) == (layer.mixer, layer.mlp), f"layer {i}: differs from layer {j}, whose weights it uses")
        for i, layer in enumerate(self.layers):
            m, f = layer.mixer, layer.mlp
            if m.kind == "latent_attention":
                need(min(m.heads, m.dim, m.vdim, m.kv_rank, m.q_rank) >= 1, f"layer {i}: empty attention size")
                need(m.dim <= MAX_HEAD_DIM and m.vdim <= MAX_HEAD_DIM, f"layer {i}: head width above {MAX_HEAD_DIM}")
                need(m.kv_rank <= MAX_RANK, f"layer {i}: kv_rank above {MAX_RANK}")
            elif m.kind == "rglru":
                need(min(m.width, m.blocks, m.taps) >= 1 and m.width % m.blocks == 0, f"layer {i}: width does not split into blocks")
            elif m.kind in ("channel_delta", "wkv"):
                need(min(m.heads, m.dim, m.vdim, m.decay_rank) >= 1, f"layer {i}: empty mixer size")
                need(m.dim <= MAX_STATE_DIM and m.vdim <= MAX_STATE_DIM, f"layer {i}: head width above {MAX_STATE_DIM}")
                need(m.decay_rank <= MAX_RANK, f"layer {i}: decay rank above {MAX_RANK}")
                if m.kind == "channel_delta":
                    need(min(m.kv_heads, m.taps, m.gate_rank) >= 1, f"layer {i}: empty mixer size")
                    need(m.gate_rank <= MAX_RANK, f"layer {i}: gate rank above {MAX_RANK}")
                    need(m.heads % m.kv_heads == 0, f"layer {i}: {m.heads} heads over {m.kv_heads} key heads")
            elif m.kind == "parallel":
                a, b = m.left, m.right
                need(min(a.heads, a.kv_heads, a.dim, a.vdim, b.heads, b.dim, b.vdim) >= 1, f"layer {i}: empty mixer size")
                need(max(a.dim, a.vdim) <= MAX_HEAD_DIM and b.dim <= MAX_STATE_DIM, f"layer {i}: head width above {MAX_HEAD_DIM}")
                need(b.vdim <= 4096, f"layer {i}: value width above 4096")
                need(a.heads % a.kv_heads == 0, f"layer {i}: {a.heads} heads over {a.kv_heads} key heads")
                need(a.window >= 0, f"layer {i}: negative chunk length")
                need(a.rotary is None or (a.rotary.dims % 2 == 0 and 0 <= a.rotary.dims <= a.dim), f"layer {i}: rotated columns")
                need(b.cap > 0, f"layer {i}: gate cap")
            else:
                need(False, f"layer {i}: unknown mixer {m.kind!r}")
            if f is not None and f.kind == "moe":
                r = f.routing
                need(r.score_func == "sigmoid", f"layer {i}: router scores {r.score_func!r}")
                need(1 <= r.top_k <= min(MAX_TOP_K, r.expert_count) and r.expert_count <= MAX_EXPERTS,
                     f"layer {i}: router of {r.expert_count} experts, top {r.top_k}")
                need(1 <= r.limited_group_count <= r.group_count <= MAX_GROUPS and r.expert_count % r.group_count == 0,
                     f"layer {i}: expert groups")
                need(r.top_k <= r.expert_count // r.group_count * r.limited_group_count, f"layer {i}: fewer eligible experts than top_k")
            elif f is not None and f.kind not in ("dense", "relu2"):
                need(False, f"layer {i}: unknown feed-forward {f.kind!r}")
        if self.loop is not None:
            need(0 <= self.loop.start < self.loop.stop <= len(self.layers) and self.loop.times >= 1, "loop bounds")
        return self


def _pad(n: int, to: int) -> int:
    return -(-n // to) * to
