"""Decoder whose layers each choose a mixer -- recurrent (HGRN2, gated delta rule, matrix memories with one decay per head) or attention
(over paged latents, over keys that are the values, differential) -- and a feed-forward (gated or not, routed experts), on hyper-connected
residual streams or on one stream normed before -- and behind -- every sublayer.  A range of layers may run several times in a row with
the same weights.

A design of this kind is a :class:`HybridConfig` (layer specs plus constants) and a :class:`HybridWeights`;
``models/registry.py`` says which checkpoint architectures map here and how their files are read.  The executor lowers
a layer run to a fixed list of launches over buffers allocated once:

    hyper_step (fold the last sublayer's output into the streams, read-out, norm, token shift), or
    norm_step  (x += norm(the last sublayer's output), norm; sums the rows of routed experts on the way), or
    norm_conv_step (x += the last sublayer's output, norm, causal convolution of what the sublayer reads); both passes take the
                bias and the gate of an output on its way to x: gemm(residual gate) over the normed rows stands behind them
    pass:       norm_step (x += the last sublayer's output, copy beside the embedding) | gemm(x | embedding, fp32 out)
    recurrent:  gemm(q | gate | v, fp32 out) | hgrn2 | head_rmsnorm | gemm(o)
    delta:      gemm(gate | q | k | v) | gemm(decay | step size, fp32 out) | conv_unit_gates | delta_rule | head_rmsnorm * gate | gemm(o)
    latent:     gemm(q | latent | rotated key | head gates) | latent_append (norm, rotations) | gemm per head (W_uk^T q) |
                latent_attention (head gates in its epilogue) | gemm per head (W_uv o) | gemm(o);
                prompts over wide latents: latent_gather | gemm (K | V pages) | paged_prefill | gemm(o)
    tied:       gemm(q | k | head gates) | tied_append (biases, norms, pages) | tied_attention (bias by distance, cap, sink, head gates) | gemm(o)
    memory:     gemm(q | k | v | gate) | gemm(input | forget gates, fp32 out) | decay_memory (rotations, gates, read-out) | head_rmsnorm * gate |
                gemm(o)
    diff:       gemm(q | k | v) | conv_rope_append | diff_attention (both maps, difference and norm) | gemm(o)
    dense:      gemm(gate_up or up, activation in the epilogue) | gemm(down)
    experts:    gemm(router | shared gate, fp32 out) | route, permute, gather | grouped gemm(up, activation epilogue) | grouped gemm(down)
                shared expert: gemm(gate_up, gated epilogue) | gemm(down)

The residual streams, norms, gates and recurrent state are fp32 in every engine; matrix products and the activations
between them are bf16, or fp32 throughout in the 32-bit engine (``EngineConfig.compute_dtype``).

Widths that are not multiples of 8 are padded with zero weights at load time, so every product meets the tensor-map
rules of the bf16 kernels whatever the model's sizes.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from .. import ops
from ..ops import hybrid as hops
from ..ops import moe as moe_ops
from ..ops.hybrid import Act, DynamicTanh, ExpertRows, GatedRows, HyperConnection, LatentRope, RmsNorm
from .decoder import pad_mlp, pick_swiglu_half


def pad8(n: int) -> int:
    return n + (-n) % 8


# ------------------------------------------------------------------------------------------
# configuration
# ------------------------------------------------------------------------------------------
@dataclass
class RecurrentSpec:
    """HGRN2: ``heads`` states of ``dim`` x ``vdim``."""
    heads: int
    dim: int
    vdim: int


@dataclass
class LatentSpec:
    """Latent attention: ``window`` 0 means every earlier token; ``kv_from`` names the layer whose latents are read.  ``rot_dim``: rotated
    dimensions of every query head, and of a key part that all heads share and that lies behind the latent in its page row;
    ``gated``: every head's output is multiplied by the sigmoid of a projection of the mixer's input."""
    heads: int
    dim: int
    vdim: int
    rank: int
    scale: float
    window: int = 0
    kv_from: int | None = None
    rot_dim: int = 0
    rot_base: float = 10000.0
    gated: bool = False

    @property
    def q_width(self) -> int:
        """Columns of a projected query head."""
        return pad8(self.dim) + pad8(self.rot_dim)

    @property
    def key_width(self) -> int:
        """Columns of a page row, and of a query head folded to meet it."""
        return pad8(self.rank) + pad8(self.rot_dim)

    @property
    def latent_col(self) -> int:
        """Where the latent begins in a projected row."""
        return self.heads * self.q_width

    @property
    def gate_col(self) -> int:
        return self.latent_col + (self.key_width if self.kv_from is None else 0)

    @property
    def proj_width(self) -> int:
        return self.gate_col + (self.heads if self.gated else 0)


@dataclass
class DeltaSpec:
    """Gated delta rule: ``heads`` states of ``dim`` x ``vdim`` over ``kv_heads`` query / key heads, behind convolutions of ``taps``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @property
    def conv_width(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass
class DiffSpec:
    """Differential attention: two maps of ``dim`` per head over values of ``vdim``, behind convolutions of ``taps``; ``window`` 0 means
    every earlier token, otherwise the last ``window`` and the first ``keep``.  The first ``rot_dims`` of every map are rotated."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    scale: float
    diff: float
    window: int = 0
    keep: int = 0
    rot_dims: int = 0
    rot_base: float = 10000.0

    @property
    def conv_width(self) -> int:
        return 2 * (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim

    @property
    def page_elems(self) -> int:
        return self.kv_heads * ops.PAGE * (2 * pad8(self.dim) + pad8(self.vdim))


@dataclass
class TiedSpec:
    """Attention whose values are its keys before their norm: ``heads`` queries of ``dim`` over ``kv_heads`` keys, both normed over the whole
    projection.  Scores times ``scale`` are capped to softcap tanh(s / softcap) (0: not), and lose a number per head times the distance;
    ``sink``: a number per head joins the softmax; ``window`` 0 means every earlier token; ``gated``: a sigmoid per head."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: float = 0.0
    window: int = 0
    sink: bool = True
    gated: bool = True

    @property
    def gate_col(self) -> int:
        return (self.heads + self.kv_heads) * self.dim

    @property
    def proj_width(self) -> int:
        return self.gate_col + (self.heads if self.gated else 0)

    @property
    def factor(self) -> float:
        """What a page's factors hold besides the key's norm."""
        return self.scale / self.softcap if self.softcap > 0 else self.scale

    @property
    def page_elems(self) -> int:
        return hops.tied_page_elems(self.kv_heads, pad8(self.dim))


@dataclass
class MemorySpec:
    """Matrix memories of ``dim`` x ``vdim`` with one decay per head and an output gate.  ``gate_cap`` 0: retention -- fixed decays, queries and
    keys rotated in their first ``rot_dims``, keys scaled by dim^-1/2, a silu gate; otherwise mLSTM -- exponential input gates and
    sigmoid forget gates capped at +-gate_cap under a running maximum, a normalizer, queries scaled, a sigmoid gate."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float = 0.0
    decay: tuple = ()                  # a fixed one per head
    rot_dims: int = 0
    rot_base: float = 10000.0

    @property
    def gated(self) -> bool:
        return self.gate_cap > 0

    @property
    def gate_col(self) -> int:
        return self.heads * (2 * self.dim + self.vdim)

    @property
    def proj_width(self) -> int:
        return self.gate_col + self.heads * self.vdim


@dataclass
class MlpSpec:
    """``act``: a gated activation, or "xielu" (one projection, two numbers per layer)."""
    inter: int
    act: str = "gelu_tanh"


@dataclass
class MoeSpec:
    """Routed experts down(act(up h)), ``top`` of ``experts`` per token, chosen from the ``keep`` best of ``groups`` equal groups, which score as
    their ``group_best`` best experts; ``score``: "softmax" (``bias``: added to the logits) or "sigmoid" (added to the scores that are
    compared).  ``act``: "relu2", or with a gate "silu" or "clamp_glu" (``limit``).  ``shared_inter`` > 0: an expert of that size (and ``shared_limit``) runs for every
    token, times the sigmoid of a projection."""
    experts: int
    top: int
    inter: int
    groups: int = 1
    keep: int = 1
    renormalize: bool = False
    act: str = "relu2"
    limit: float = 0.0
    shared_inter: int = 0
    shared_limit: float = 0.0
    bias: bool = False
    score: str = "softmax"
    group_best: int = 1

    @property
    def gated(self) -> bool:
        return Act(self.act).gated

    @property
    def logits(self) -> int:
        """Columns of the router's product: experts, and the shared expert's gate."""
        return self.experts + (self.shared_inter > 0)


@dataclass
class LayerSpec:
    mixer: RecurrentSpec | LatentSpec | DeltaSpec | DiffSpec | TiedSpec | MemorySpec
    mlp: MlpSpec | MoeSpec | None = None


@dataclass
class LoopSpec:
    """Layers start .. stop - 1 run ``times`` times in a row.  Ahead of every pass the residual becomes a projection of itself and the
    embedding, plus a vector of the pass."""
    start: int
    stop: int
    times: int


@dataclass
class HybridConfig:
    vocab: int
    hidden: int
    layers: list
    streams: int = 1
    norm_eps: float = 1e-6
    name: str = "hybrid"
    logit_scale: float = 1.0           # folded into the final norm's weight
    residual: str = "hyper"            # "hyper": connected streams, Dynamic-Tanh norms, token shift; "sandwich": RMS norms around a sublayer;
                                       # "pre": RMS norms before a sublayer
    input_taps: int = 0                # "pre": what a sublayer reads is h plus a causal convolution of h over this many taps (0: h)
    ff_input_conv: bool = True         # feed-forwards too, not only mixers
    residual_gates: bool = False       # "pre": a sublayer's output reaches the residual times sigmoid(W h + b), h the normed residual
    norm_groups: int = 1
    embed_scale: float = 1.0
    embed_normed: bool = True          # "pre": random weights have a norm of the embedding
    loop: LoopSpec | None = None
    eos_token: int = -1
    max_position: int = 1 << 20        # no positional table: bounded by the pool only
    default_seq_len: int = 8192        # sequence limit when neither the caller nor the package names one

    @property
    def runs(self) -> list:
        """The layers in the order they run; every run has a cache and state of its own."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return list(range(n))
        return [*range(lp.start), *list(range(lp.start, lp.stop)) * lp.times, *range(lp.stop, n)]

    @property
    def num_layers(self) -> int:
        """Layer runs: what caches and state are counted by."""
        return len(self.runs)

    @property
    def latent_layers(self) -> list:
        return [l.mixer for l in self.layers if isinstance(l.mixer, LatentSpec)]

    @property
    def attention_layers(self) -> list:
        return [l.mixer for l in self.layers if isinstance(l.mixer, (LatentSpec, DiffSpec, TiedSpec))]

    @property
    def num_heads(self) -> int:
        return max((m.heads for m in self.attention_layers), default=1)

    num_kv_heads = 1

    @property
    def sliding_window(self) -> int:
        """Tokens a sequence has to keep pages of: the widest window, 0 when some layer sees everything."""
        windows = [m.window for m in self.attention_layers]
        return 0 if any(w <= 0 for w in windows) else max(windows, default=1)

    @property
    def attention_sinks(self) -> int:
        """First tokens of a sequence whose pages stay for good."""
        return max((m.keep for m in self.attention_layers if isinstance(m, DiffSpec) and m.window > 0), default=0)

    has_state = True                   # token shift, convolutions and recurrences are per-sequence state

    def kv_page_shape(self, layer: int, kv_heads: int = 1):
        """Shape of one KV page of a layer run, None when it caches nothing of its own."""
        m = self.layers[self.runs[layer]].mixer
        if isinstance(m, (DiffSpec, TiedSpec)):
            return (m.page_elems,)
        return (ops.PAGE, m.key_width) if isinstance(m, LatentSpec) and m.kv_from is None else None

    def state_shapes(self, layer: int) -> dict:
        """Per-sequence fp32 state of a layer run: name -> shape."""
        spec = self.layers[self.runs[layer]]
        m = spec.mixer
        shapes = {"shift": (self.hidden,)} if self.residual == "hyper" else {}
        if self.input_taps:
            shapes["input1"] = (self.input_taps - 1, self.hidden)
            if spec.mlp is not None and self.ff_input_conv:
                shapes["input2"] = (self.input_taps - 1, self.hidden)
        if isinstance(m, (DeltaSpec, DiffSpec)):
            shapes["conv"] = (m.taps - 1, m.conv_width)
        if isinstance(m, (RecurrentSpec, DeltaSpec)):
            shapes["recurrent"] = (m.heads, m.vdim, hops.state_rows(m.dim))
        if isinstance(m, MemorySpec):
            shapes["recurrent"] = (m.heads, m.vdim + m.gated, hops.state_rows(m.dim))
            if m.gated:
                shapes["peak"] = (m.heads,)
        return shapes

    def validate(self) -> None:
        if self.residual not in ("hyper", "sandwich", "pre"):
            raise ValueError(f"unknown residual {self.residual!r}")
        if self.input_taps and (self.residual != "pre" or not 0 <= self.input_taps <= 8):
            raise ValueError(f"input convolutions of {self.input_taps} taps are not supported (1 to 8, behind norms before the sublayers)")
        if self.norm_groups < 1 or self.hidden % self.norm_groups or (self.norm_groups > 1 and self.residual != "pre"):
            raise ValueError(f"norms of {self.hidden} channels in {self.norm_groups} groups are not supported (equal groups, before the sublayers)")
        quads = self.hidden // self.norm_groups % 4 == 0
        if self.input_taps and self.hidden > (8192 if quads else 4096):
            raise ValueError(f"input convolutions of {self.hidden} channels are not supported (8192, 4096 where a norm's groups are no multiple of 4)")
        if self.residual_gates and self.residual != "pre":
            raise ValueError("gates of the residual need norms before the sublayers")
        if self.norm_groups > 1 and self.hidden > (16384 if quads else 4096):
            raise ValueError(f"norms in groups of {self.hidden} channels are not supported (16384, 4096 where they are no multiple of 4)")
        if self.loop is not None:
            lp = self.loop
            if self.residual != "pre" or not 0 <= lp.start < lp.stop <= len(self.layers) or lp.times < 1:
                raise ValueError(f"a loop over layers {lp.start} .. {lp.stop} of {len(self.layers)}, {lp.times} times, is not supported "
                                 "(with norms before the sublayers only)")
            if any(isinstance(l.mixer, LatentSpec) and l.mixer.kv_from is not None for l in self.layers):
                raise ValueError("layers that read another layer's latents cannot be combined with a loop")
        if not 1 <= self.streams <= 8 or (self.residual != "hyper" and self.streams != 1):
            raise ValueError(f"{self.streams} residual streams are not supported (1 to 8, 1 with norms around the sublayers)")
        for i, layer in enumerate(self.layers):
            m, f = layer.mixer, layer.mlp
            if isinstance(f, MoeSpec):
                if self.residual == "hyper":
                    raise ValueError(f"layer {i}: routed experts need a residual of one stream")
                if f.score not in ("softmax", "sigmoid") or f.group_best < 1 or f.group_best > 2:
                    raise ValueError(f"layer {i}: routing by {f.score!r} scores and the {f.group_best} best experts of a group is not supported")
                if f.act not in ("relu2", "silu", "clamp_glu"):
                    raise ValueError(f"layer {i}: unknown activation {f.act!r} of routed experts")
                if f.experts > 256 or f.top > 32 or f.groups < 1 or f.experts % f.groups or not 1 <= f.keep <= f.groups:
                    raise ValueError(f"layer {i}: {f.experts} experts in {f.groups} groups, {f.keep} kept, {f.top} chosen are not supported "
                                     "(at most 256 experts in equal groups, 32 chosen)")
                if not 1 <= f.top <= f.keep * (f.experts // f.groups):
                    raise ValueError(f"layer {i}: {f.top} experts cannot be chosen from {f.keep} groups of {f.experts // f.groups}")
            if isinstance(m, (RecurrentSpec, DeltaSpec, MemorySpec)):
                hops.state_rows(m.dim)
            if isinstance(m, MemorySpec):
                if not m.gated and (len(m.decay) != m.heads or not all(0 <= a <= 1 for a in m.decay)):
                    raise ValueError(f"layer {i}: {len(m.decay)} decays for {m.heads} heads (one each, between 0 and 1)")
                if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.dim:
                    raise ValueError(f"layer {i}: {m.rot_dims} rotated dimensions of {m.dim}")
                if m.gated and m.vdim > 512:
                    raise ValueError(f"layer {i}: gated memories of {m.vdim} value channels are not supported (at most 512)")
            if isinstance(m, TiedSpec):
                if m.kv_heads < 1 or m.heads % m.kv_heads:
                    raise ValueError(f"layer {i}: {m.heads} heads do not divide over {m.kv_heads} key heads")
                if m.dim > 512:
                    raise ValueError(f"layer {i}: heads of {m.dim} are not supported (at most 512)")
            if isinstance(m, (DeltaSpec, DiffSpec)):
                if not 1 <= m.taps <= 8:
                    raise ValueError(f"layer {i}: convolutions of {m.taps} taps are not supported (1 to 8)")
                if m.kv_heads < 1 or m.heads % m.kv_heads:
                    raise ValueError(f"layer {i}: {m.heads} heads do not divide over {m.kv_heads} key heads")
            if isinstance(m, DiffSpec):
                if m.vdim > 512 or m.dim > 512:
                    raise ValueError(f"layer {i}: heads of {m.dim} x {m.vdim} are not supported (at most 512)")
                if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.dim:
                    raise ValueError(f"layer {i}: {m.rot_dims} rotated dimensions of {m.dim}")
            if not isinstance(m, LatentSpec):
                continue
            if m.key_width > 1024:
                raise ValueError(f"layer {i}: latent size {m.rank} with {m.rot_dim} rotated dimensions is not supported (at most 1024 together)")
            if m.rot_dim % 2:
                raise ValueError(f"layer {i}: {m.rot_dim} rotated dimensions")
            if m.rot_dim and m.kv_from is not None:
                raise ValueError(f"layer {i}: rotated dimensions need latents of the layer's own")
            if m.kv_from is not None:
                if not 0 <= m.kv_from < i:
                    raise ValueError(f"layer {i}: kv_from {m.kv_from} does not name an earlier layer")
                src = self.layers[m.kv_from].mixer
                if not isinstance(src, LatentSpec) or src.kv_from is not None or src.rank != m.rank:
                    raise ValueError(f"layer {i}: kv_from {m.kv_from} is not a layer with latents of its own of size {m.rank}")

    def replace(self, **kw) -> "HybridConfig":
        import dataclasses

        return dataclasses.replace(self, **kw)

    def weight_bytes(self) -> int:
        n = 2 * self.vocab * self.hidden
        for layer in self.layers:
            m = layer.mixer
            if isinstance(m, RecurrentSpec):
                n += self.hidden * m.heads * (2 * m.dim + 2 * m.vdim)
            elif isinstance(m, DeltaSpec):
                n += self.hidden * (m.conv_width + 2 * m.heads * m.vdim + 2 * m.heads)
            elif isinstance(m, DiffSpec):
                n += self.hidden * (m.conv_width + m.heads * m.vdim)
            elif isinstance(m, TiedSpec):
                n += self.hidden * (m.proj_width + m.heads * m.dim)
            elif isinstance(m, MemorySpec):
                n += self.hidden * (m.proj_width + m.heads * m.vdim + 2 * m.heads * m.gated)
            else:
                n += self.hidden * m.heads * (m.dim + m.rot_dim + m.vdim + m.gated) + m.rank * m.heads * (m.dim + m.vdim)
                n += self.hidden * (m.rank + m.rot_dim) if m.kv_from is None else 0
            if isinstance(layer.mlp, MoeSpec):
                f = layer.mlp
                n += self.hidden * (f.experts * (2 + f.gated) * f.inter + 3 * f.shared_inter + f.logits)
            elif layer.mlp:
                n += (2 + Act(layer.mlp.act).gated) * self.hidden * layer.mlp.inter
            if self.residual_gates:
                n += (1 + (layer.mlp is not None)) * self.hidden * self.hidden
        if self.loop is not None:
            n += 2 * self.hidden * self.hidden
        return 2 * n

    def kv_bytes_per_token(self, kv_dtype_bytes: int = 2) -> int:
        mixers = [self.layers[li].mixer for li in self.runs]
        return kv_dtype_bytes * (sum(m.key_width for m in mixers if isinstance(m, LatentSpec) and m.kv_from is None) +
                                 sum(m.page_elems // ops.PAGE for m in mixers if isinstance(m, (DiffSpec, TiedSpec))))


# ------------------------------------------------------------------------------------------
# weights
# ------------------------------------------------------------------------------------------
@dataclass
class RecurrentWeights:
    qfv: torch.Tensor        # [heads * (dim + dim + vdim), hidden]: query, gate and value projections
    gate_bias: torch.Tensor  # fp32 [heads * dim]
    gate_low: torch.Tensor   # fp32 [heads * dim]
    norm: torch.Tensor       # fp32 [vdim]
    o: torch.Tensor          # [hidden, heads * vdim]


@dataclass
class LatentWeights:
    qc: torch.Tensor              # [LatentSpec.proj_width, hidden]: query (latent and rotated key, head gate) projections
    c_norm: torch.Tensor | None   # fp32 [rank]
    uk: torch.Tensor              # [heads * rank_p, dim_p]: W_uk^T per head, folds the key expansion into the query
    uv: torch.Tensor              # [heads * vdim_p, rank_p]: value expansion, applied to the attended latent
    o: torch.Tensor               # [hidden, heads * vdim_p]
    kv: torch.Tensor | None = None     # [heads * (key | value chunks) * 64, key_width]: both expansions, for prompts (see expand_prompts)
    freq: torch.Tensor | None = None   # fp64 [rot_dim / 2]


@dataclass
class DeltaWeights:
    gqkv: torch.Tensor       # [heads * vdim + conv_width, hidden]: output-gate, query, key and value projections
    ab: torch.Tensor         # [2 * heads, hidden]: decay and step-size projections
    conv: torch.Tensor       # fp32 [taps, conv_width]
    a_log: torch.Tensor      # fp32 [heads]
    dt_bias: torch.Tensor    # fp32 [heads]
    norm: torch.Tensor       # fp32 [vdim]
    o: torch.Tensor          # [hidden, heads * vdim]


@dataclass
class DiffWeights:
    qkv: torch.Tensor        # [conv_width, hidden]
    bias: torch.Tensor       # fp32 [conv_width]
    conv: torch.Tensor       # fp32 [taps, conv_width]
    freq: torch.Tensor       # fp64 [rot_dims / 2]
    lam: float
    o: torch.Tensor          # [hidden, heads * vdim_p]


@dataclass
class TiedWeights:
    qkg: torch.Tensor                  # [TiedSpec.proj_width, hidden]: queries, keys, head gates
    q_bias: torch.Tensor | None        # fp32 [heads * dim]
    k_bias: torch.Tensor | None        # fp32 [kv_heads * dim]
    q_gain: torch.Tensor               # fp32 [heads * dim]: the query norm's weight times the key norm's of the head's keys
    slope: torch.Tensor | None         # fp32 [heads]
    sink: torch.Tensor | None          # fp32 [heads]
    o: torch.Tensor                    # [hidden, heads * dim_p]
    o_bias: torch.Tensor | None = None


@dataclass
class MemoryWeights:
    qkvg: torch.Tensor                 # [MemorySpec.proj_width, hidden]: queries, keys, values, output gate
    o: torch.Tensor                    # [hidden, heads * vdim]
    decay: torch.Tensor | None = None          # fp32 [2, heads]: decays, their logarithms
    gates: torch.Tensor | None = None          # [2 * heads, hidden]: input, forget
    gates_bias: torch.Tensor | None = None     # fp32 [2 * heads]
    norm: torch.Tensor | None = None           # fp32 [heads * vdim]


@dataclass
class MoeWeights:
    router: torch.Tensor     # [experts (+ the shared expert's gate), hidden]
    up: torch.Tensor         # [experts, inter_p, hidden_p]; gated: [experts, 2 inter_p, hidden_p], gate and up rows packed with ``half``
    down: torch.Tensor       # [experts, hidden, inter_p]
    half: int = 0
    bias: torch.Tensor | None = None             # fp32 [experts]
    shared_up: torch.Tensor | None = None        # [2 inter_p, hidden_p], packed with ``shared_half``
    shared_down: torch.Tensor | None = None
    shared_half: int = 0


@dataclass
class HybridLayer:
    """Norms and residual connections follow ``HybridConfig.residual``: Dynamic-Tanh, hyper-connections and a token shift, or RMS
    norms before (norm1, norm2) and, for "sandwich", behind (hc1, hc2) the sublayers."""
    norm1: DynamicTanh | RmsNorm
    hc1: HyperConnection | RmsNorm | None
    mixer: RecurrentWeights | LatentWeights | DeltaWeights | DiffWeights | TiedWeights | MemoryWeights
    shift: torch.Tensor | None = None             # fp32 [hidden]
    norm2: DynamicTanh | RmsNorm | None = None
    hc2: HyperConnection | RmsNorm | None = None
    gate_up: torch.Tensor | None = None
    down: torch.Tensor | None = None
    half: int = 0
    moe: MoeWeights | None = None
    act: Act | None = None                        # feed-forward; a gated one has gate_up packed with ``half``, another up rows alone
    conv1: torch.Tensor | None = None             # fp32 [input_taps, hidden]: what the sublayer reads, the identity included
    conv2: torch.Tensor | None = None
    gate1: torch.Tensor | None = None             # [hidden, hidden] and fp32 [hidden]: gates of what the sublayers add to the residual
    gate1_bias: torch.Tensor | None = None
    gate2: torch.Tensor | None = None
    gate2_bias: torch.Tensor | None = None


@dataclass
class HybridWeights:
    embed: torch.Tensor
    layers: list = field(default_factory=list)
    final_norm: DynamicTanh | None = None
    lm_head: torch.Tensor | None = None
    embed_norm: RmsNorm | None = None
    loop_in: torch.Tensor | None = None          # [hidden, 2 * hidden_p]: residual, embedding
    loop_step: torch.Tensor | None = None        # fp32 [times, hidden]
    unused: list = field(default_factory=list)   # tensors of the checkpoint that its configuration does not name


def pad_cols(w, to=None):
    """Zero-pad the last dimension to ``to`` (default: the next multiple of 8)."""
    extra = (to or pad8(w.shape[-1])) - w.shape[-1]
    return torch.nn.functional.pad(w, (0, extra)).contiguous() if extra else w.contiguous()


def pad_head_rows(w, heads, to):
    """[heads * n, k] -> [heads * to, k] with zero rows behind every head's n."""
    n = w.shape[0] // heads
    return w if n == to else torch.nn.functional.pad(w.reshape(heads, n, -1), (0, 0, 0, to - n)).reshape(heads * to, -1)


def pack_recurrent(spec: RecurrentSpec, q, f, f_bias, low, v, norm, o) -> RecurrentWeights:
    return RecurrentWeights(qfv=pad_cols(torch.cat([q, f, v], 0)), gate_bias=f_bias.float().contiguous(), gate_low=low.float().contiguous(),
                            norm=norm.float().contiguous(), o=pad_cols(o))


def chunks(n: int) -> int:
    """64-column chunks that hold n columns."""
    return -(-n // 64)


def expand_prompts(spec: LatentSpec, dtype) -> bool:
    """Whether prompts of a layer may run on expanded keys and values: the heads fit the paged prefill kernel, and a page row is
    wider than a head (otherwise attending to the latent itself is no more work)."""
    return (dtype == torch.bfloat16 and chunks(spec.q_width) <= 3 and chunks(spec.vdim) <= min(2, chunks(spec.q_width)) and spec.scale > 0
            and spec.key_width > spec.q_width)


def rotation(dims: int, base: float, device) -> torch.Tensor:
    """Angles per position of the pairs of ``dims`` rotated dimensions, fp64."""
    return (base ** (-2 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))).to(device)


def pack_latent(spec: LatentSpec, q, dkv, dkv_norm, uk, uv, o, g=None) -> LatentWeights:
    """q: heads of dim (+ rot_dim) rows; dkv: the latent's rows (and the rotated key part's); g: head gates."""
    h, d, r, rank = spec.heads, spec.dim, spec.rot_dim, spec.rank
    dp, rp, vp, cp, kw = pad8(d), pad8(r), pad8(spec.vdim), pad8(rank), spec.key_width
    pad = torch.nn.functional.pad

    def two_parts(w, first, second):
        """[n, first + second, k] -> both parts padded to multiples of 8 rows, [n * .., k]."""
        n, k = w.shape[0], w.shape[-1]
        return torch.cat([pad(w[:, :first], (0, 0, 0, pad8(first) - first)), pad(w[:, first:], (0, 0, 0, pad8(second) - second))], 1).reshape(-1, k)

    qc = [two_parts(q.reshape(h, d + r, -1), d, r)]
    if dkv is not None:
        qc.append(two_parts(dkv[None], rank, r))
    if g is not None:
        qc.append(g)
    ukh, uvh = uk.reshape(h, d, rank), uv.reshape(h, spec.vdim, rank)
    ukt = pad(ukh.transpose(1, 2), (0, dp - d, 0, cp - rank)).reshape(h * cp, dp)             # [h, rank, dim]
    kv = None
    if expand_prompts(spec, q.dtype):
        # a head's expanded key is [W_uk c | rotated part]: the part passes through rows of the identity
        kv = q.new_zeros(h, 64 * (chunks(spec.q_width) + chunks(spec.vdim)), kw)
        kv[:, :d, :rank] = ukh
        kv[:, dp:dp + r, cp:cp + r] = torch.eye(r, dtype=q.dtype, device=q.device)
        v0 = 64 * chunks(spec.q_width)
        kv[:, v0:v0 + spec.vdim, :rank] = uvh
        kv = kv.reshape(-1, kw)
    return LatentWeights(kv=kv, qc=pad_cols(torch.cat(qc, 0)), c_norm=None if dkv_norm is None else dkv_norm.float().contiguous(), uk=ukt.contiguous(),
                         uv=pad_cols(pad_head_rows(uv, h, vp), cp), freq=rotation(r, spec.rot_base, q.device) if r else None,
                         o=pad(o.reshape(o.shape[0], h, spec.vdim), (0, vp - spec.vdim)).reshape(o.shape[0], h * vp).contiguous())


def pack_delta(spec: DeltaSpec, q, k, v, g, a, b, conv, a_log, dt_bias, norm, o) -> DeltaWeights:
    """``conv``: filters of the q, k and v channels, [channels, taps] each."""
    f32 = lambda t: t.float().contiguous()
    return DeltaWeights(gqkv=pad_cols(torch.cat([g, q, k, v], 0)), ab=pad_cols(torch.cat([a, b], 0)), conv=f32(torch.cat(conv, 0).t()), a_log=f32(a_log),
                        dt_bias=f32(dt_bias), norm=f32(norm), o=pad_cols(o))


def pack_diff(spec: DiffSpec, q, k, v, bias, conv, lam: float, o) -> DiffWeights:
    """``bias``, ``conv``: of the q, k and v channels; ``lam``: the layer's weight of the second map."""
    vp = pad8(spec.vdim)
    f32 = lambda t: t.float().contiguous()
    return DiffWeights(qkv=pad_cols(torch.cat([q, k, v], 0)), bias=f32(torch.cat(bias, 0)), conv=f32(torch.cat(conv, 0).t()), freq=rotation(spec.rot_dims, spec.rot_base, q.device),
                       lam=float(lam), o=torch.nn.functional.pad(o.reshape(o.shape[0], spec.heads, spec.vdim), (0, vp - spec.vdim)).reshape(o.shape[0], -1).contiguous())


def pack_tied(spec: TiedSpec, q, k, g, q_bias, k_bias, q_norm, k_norm, slope, sink, o, o_bias) -> TiedWeights:
    """q_norm, k_norm: weights over the whole projections."""
    h, d, dp = spec.heads, spec.dim, pad8(spec.dim)
    f32 = lambda t: None if t is None else t.float().contiguous()
    keys = k_norm.float().view(spec.kv_heads, 1, d).expand(-1, h // spec.kv_heads, -1).reshape(-1)
    return TiedWeights(qkg=pad_cols(torch.cat([q, k] + ([g] if g is not None else []), 0)), q_bias=f32(q_bias), k_bias=f32(k_bias),
                       q_gain=(q_norm.float() * keys).contiguous(), slope=f32(slope), sink=f32(sink), o_bias=f32(o_bias),
                       o=torch.nn.functional.pad(o.reshape(o.shape[0], h, d), (0, dp - d)).reshape(o.shape[0], h * dp).contiguous())


def distance_slopes(heads: int, device) -> torch.Tensor:
    """Slopes 2^(-8 (h + 1) / heads) of biases by distance."""
    return torch.exp2(-8 * torch.arange(1, heads + 1, dtype=torch.float64) / heads).float().to(device)


def pack_memory(spec: MemorySpec, q, k, v, g, o, gates=None, gates_bias=None, norm=None) -> MemoryWeights:
    """``gates``: input and forget projections."""
    f32 = lambda t: None if t is None else t.float().contiguous()
    decay = None
    if not spec.gated:                 # a decay of zero forgets everything at once; its logarithm stays finite
        decay = torch.tensor(spec.decay, dtype=torch.float64)
        decay = torch.stack([decay, torch.log(decay).clamp(min=-1e30)]).float().to(q.device)
    return MemoryWeights(qkvg=pad_cols(torch.cat([q, k, v, g], 0)), o=pad_cols(o), decay=decay, gates=None if gates is None else pad_cols(gates),
                         gates_bias=f32(gates_bias), norm=f32(norm))


def pack_moe(router, ups, downs) -> MoeWeights:
    """``ups`` [inter, hidden] and ``downs`` [hidden, inter] of every expert."""
    inter = ups[0].shape[0]
    up = torch.nn.functional.pad(pad_cols(torch.stack(list(ups))), (0, 0, 0, pad8(inter) - inter)).contiguous()
    return MoeWeights(router=pad_cols(router), up=up, down=pad_cols(torch.stack(list(downs))))


def pack_gated(gate, up, down):
    """(gate and up rows packed for the gated epilogue, down, half-width)."""
    if gate.shape[0] % 32:
        gate, up, down = pad_mlp(gate, up, down)
    half = pick_swiglu_half(gate.shape[0])
    return pad_cols(ops.pack_gate_up(gate.contiguous(), up.contiguous(), half)), down.contiguous(), half


def pack_gated_moe(router, bias, gates, ups, downs, shared=None) -> MoeWeights:
    """Gated experts: ``gates``, ``ups`` [inter, hidden] and ``downs`` [hidden, inter] of every one; ``shared``: (gate, up, down, sigmoid gate
    [1, hidden]) of the expert that runs for every token."""
    packed = [pack_gated(*w) for w in zip(gates, ups, downs)]
    w = MoeWeights(router=pad_cols(router if shared is None else torch.cat([router, shared[3]], 0)), up=torch.stack([p[0] for p in packed]),
                   down=torch.stack([p[1] for p in packed]), half=packed[0][2], bias=bias.float().contiguous() if bias is not None else None)
    if shared is not None:
        w.shared_up, w.shared_down, w.shared_half = pack_gated(*shared[:3])
    return w


def pack_mlp(layer: HybridLayer, gate, up, down, act="gelu_tanh") -> None:
    layer.gate_up, layer.down, layer.half = pack_gated(gate, up, down)
    layer.act = hops.as_act(act)


def pack_plain_mlp(layer: HybridLayer, up, down, act: Act) -> None:
    """A feed-forward without a gate."""
    layer.gate_up = torch.nn.functional.pad(pad_cols(up), (0, 0, 0, pad8(up.shape[0]) - up.shape[0])).contiguous()
    layer.down, layer.act = pad_cols(down), act


def pack_input_conv(w) -> torch.Tensor:
    """[hidden, taps] of a sublayer that reads h + conv(h): one filter, last tap first met by the token itself."""
    f = w.float().t().clone()
    f[-1] += 1
    return f.contiguous()


def xielu(p: float, q: float) -> Act:
    """xIELU with its two numbers as they are stored."""
    soft = lambda v: float(torch.nn.functional.softplus(torch.tensor(v, dtype=torch.float64)))
    return Act("xielu", soft(p), 0.5 + soft(q))


def pack_loop_in(w) -> torch.Tensor:
    """[hidden, residual | embedding], each half padded to multiples of 8 columns."""
    n = w.shape[1] // 2
    return torch.cat([pad_cols(w[:, :n]), pad_cols(w[:, n:])], 1).contiguous()


def random_weights(cfg: HybridConfig, device, seed: int = 0, std: float = 0.02, dtype=torch.bfloat16) -> HybridWeights:
    """Seeded weights of the configuration (benchmarks and tests)."""
    dev = torch.device(device)
    gen = torch.Generator(device=dev).manual_seed(seed * 1000003 + 17)
    draw = lambda *s: (torch.randn(*s, generator=gen, device=dev) * std).to(dtype)
    rand = lambda *s: torch.rand(*s, generator=gen, device=dev)
    hid, st = cfg.hidden, cfg.streams
    if cfg.residual == "hyper":
        norm = lambda: DynamicTanh(0.5 + rand(1), 1 + 0.1 * (rand(hid) - 0.5), 0.1 * (rand(hid) - 0.5))
        conn = lambda: HyperConnection(rand(st) / st + 0.5 / st, 0.5 + rand(st), torch.eye(st, device=dev) * 0.8 + 0.2 * rand(st, st) / st)
    else:
        norm = lambda: RmsNorm(1 + 0.1 * (rand(hid) - 0.5), cfg.norm_eps, cfg.norm_groups)
        conn = norm if cfg.residual == "sandwich" else lambda: None
    taps = lambda m, *rows: [torch.randn(n, m.taps, generator=gen, device=dev) * 0.5 / m.taps for n in rows]
    input_conv = lambda: pack_input_conv(torch.randn(hid, cfg.input_taps, generator=gen, device=dev) * 0.5 / cfg.input_taps) if cfg.input_taps else None
    w = HybridWeights(embed=draw(cfg.vocab, hid))
    if cfg.residual == "pre" and cfg.embed_normed:
        w.embed_norm = norm()
    if cfg.loop is not None:
        w.loop_in, w.loop_step = pack_loop_in(draw(hid, 2 * hid)), torch.randn(cfg.loop.times, hid, generator=gen, device=dev) * std
    for spec in cfg.layers:
        m = spec.mixer
        if isinstance(m, RecurrentSpec):
            mixer = pack_recurrent(m, draw(m.heads * m.dim, hid), draw(m.heads * m.dim, hid), 2 * rand(m.heads * m.dim), 0.5 * rand(m.heads * m.dim),
                                   draw(m.heads * m.vdim, hid), torch.ones(m.vdim, device=dev), draw(hid, m.heads * m.vdim))
        elif isinstance(m, DeltaSpec):
            k, v = m.kv_heads * m.dim, m.heads * m.vdim
            mixer = pack_delta(m, draw(k, hid), draw(k, hid), draw(v, hid), draw(v, hid), draw(m.heads, hid), draw(m.heads, hid), taps(m, k, k, v),
                               -rand(m.heads), rand(m.heads) - 3, torch.ones(m.vdim, device=dev), draw(hid, v))
        elif isinstance(m, DiffSpec):
            rows = (2 * m.heads * m.dim, 2 * m.kv_heads * m.dim, m.kv_heads * m.vdim)
            mixer = pack_diff(m, *(draw(n, hid) for n in rows), [draw(n) for n in rows], taps(m, *rows), m.diff, draw(hid, m.heads * m.vdim))
        elif isinstance(m, TiedSpec):
            nq, nk = m.heads * m.dim, m.kv_heads * m.dim
            mixer = pack_tied(m, draw(nq, hid), draw(nk, hid), draw(m.heads, hid) if m.gated else None, draw(nq), draw(nk), 1 + 0.1 * (rand(nq) - 0.5),
                              1 + 0.1 * (rand(nk) - 0.5), distance_slopes(m.heads, dev), rand(m.heads) if m.sink else None, draw(hid, nq), draw(hid))
        elif isinstance(m, MemorySpec):
            k, v = m.heads * m.dim, m.heads * m.vdim
            own = dict(gates=draw(2 * m.heads, hid), gates_bias=torch.cat([rand(m.heads) - 1, rand(m.heads) + 3]), norm=1 + 0.1 * (rand(v) - 0.5)) if m.gated else {}
            mixer = pack_memory(m, draw(k, hid), draw(k, hid), draw(v, hid), draw(v, hid), draw(hid, v), **own)
        else:
            own = m.kv_from is None
            mixer = pack_latent(m, draw(m.heads * (m.dim + m.rot_dim), hid), draw(m.rank + m.rot_dim, hid) if own else None,
                                torch.ones(m.rank, device=dev) if own else None, draw(m.heads * m.dim, m.rank), draw(m.heads * m.vdim, m.rank),
                                draw(hid, m.heads * m.vdim), draw(m.heads, hid) if m.gated else None)
        layer = HybridLayer(norm1=norm(), shift=rand(hid) if cfg.residual == "hyper" else None, hc1=conn(), mixer=mixer, conv1=input_conv())
        if spec.mlp is not None:
            layer.norm2, layer.hc2, layer.conv2 = norm(), conn(), input_conv() if cfg.ff_input_conv else None
        if cfg.residual_gates:
            layer.gate1, layer.gate1_bias = pad_cols(draw(hid, hid)), rand(hid)
            if spec.mlp is not None:
                layer.gate2, layer.gate2_bias = pad_cols(draw(hid, hid)), rand(hid)
        f = spec.mlp
        if isinstance(f, MoeSpec) and f.gated:
            expert = lambda n: (draw(n, hid), draw(n, hid), draw(hid, n))
            layer.moe = pack_gated_moe(draw(f.experts, hid), torch.randn(f.experts, generator=gen, device=dev) * std if f.bias else None,
                                       *zip(*(expert(f.inter) for _ in range(f.experts))),
                                       shared=(*expert(f.shared_inter), draw(1, hid)) if f.shared_inter else None)
        elif isinstance(f, MoeSpec):
            layer.moe = pack_moe(draw(f.experts, hid), [draw(f.inter, hid) for _ in range(f.experts)], [draw(hid, f.inter) for _ in range(f.experts)])
        elif f is not None and f.act == "xielu":
            pack_plain_mlp(layer, draw(f.inter, hid), draw(hid, f.inter), xielu(0.3, -0.2))
        elif f is not None:
            pack_mlp(layer, draw(f.inter, hid), draw(f.inter, hid), draw(hid, f.inter), f.act)
        w.layers.append(layer)
    w.final_norm, w.lm_head = norm(), pad_cols(draw(cfg.vocab, hid))
    return w


# ------------------------------------------------------------------------------------------
# executor
# ------------------------------------------------------------------------------------------
class HybridModel:
    """One engine step over packed rows; the counterpart of :class:`~.decoder.DecoderModel` for hybrid configurations."""

    native = None
    fused_comm = None
    split_by_window = True             # how the engine picks decode splits (decode_ctas)

    def __init__(self, cfg: HybridConfig, weights: HybridWeights, device, max_tokens: int, max_seqs: int, tp: int = 1, rank: int = 0, comm=None):
        cfg.validate()
        if tp != 1:
            raise ValueError("hybrid models run on one GPU per replica (tp = 1)")
        self.cfg, self.w, self.device = cfg, weights, torch.device(device)
        self.tp, self.rank, self.comm = tp, rank, comm
        self.max_tokens, self.max_seqs = max_tokens, max_seqs
        dt, dev = weights.embed.dtype, self.device
        if dev.type == "cuda" and dt not in (torch.bfloat16, torch.float32):
            raise ValueError(f"hybrid models run in bf16 or fp32, not {dt}")
        z = lambda *s, dtype=dt: torch.zeros(*s, dtype=dtype, device=dev)
        hid = cfg.hidden
        # residual streams, double buffered where a row reads its neighbour
        self.xs = [z(max_tokens, cfg.streams, hid, dtype=torch.float32) for _ in range(1 if cfg.residual == "sandwich" else 2)]
        self.h, self.y = z(max_tokens, pad8(hid)), z(max_tokens, pad8(hid))
        of = lambda kind: [l.mixer for l in cfg.layers if isinstance(l.mixer, kind)]
        rec, lat, delta, diff, tied, mem = (of(kind) for kind in (RecurrentSpec, LatentSpec, DeltaSpec, DiffSpec, TiedSpec, MemorySpec))
        experts = [l.mlp for l in cfg.layers if isinstance(l.mlp, MoeSpec)]
        most = lambda widths: max(widths, default=0)
        flat = lambda width, dtype=dt: z(max_tokens * width, dtype=dtype) if width else None    # viewed per layer: rows stay contiguous
        self.qfv = flat(most(pad8(m.heads * (2 * m.dim + m.vdim)) for m in rec), torch.float32)
        self.rec_o = flat(most(m.heads * m.vdim for m in rec + delta + mem), torch.float32)
        self.factor = z(max_tokens * cfg.norm_groups, dtype=torch.float32) if cfg.input_taps else None
        self.plain, self.res_gate = (z(max_tokens, pad8(hid)) if cfg.residual_gates else None for _ in range(2))
        # rotations of a step's rows, shared by the layers that turn alike
        self.turns = {key: (rotation(*key, dev), z(max_tokens, key[0] // 2, 2, dtype=torch.float32))
                      for key in {(m.rot_dims, m.rot_base) for m in mem if m.rot_dims}}
        self.loop_in = self.loop_x = None
        if cfg.loop is not None:       # residual | embedding, and the residual a pass begins with
            self.loop_in, self.loop_x = z(max_tokens, 2 * pad8(hid)), z(max_tokens, pad8(hid), dtype=torch.float32)
        self.qc = flat(most(pad8(m.proj_width) for m in lat))
        self.qa = flat(most(m.heads * m.key_width for m in lat))
        self.oc = flat(most(m.heads * pad8(m.rank) for m in lat))
        self.proj = flat(most([pad8(m.conv_width + m.heads * m.vdim) for m in delta] + [pad8(m.conv_width) for m in diff] +
                              [pad8(m.proj_width) for m in tied + mem]))
        self.ab = flat(most([pad8(2 * m.heads) for m in delta + mem] + [pad8(f.logits) for f in experts]), torch.float32)
        self.unit_qk = flat(most(2 * m.kv_heads * m.dim for m in delta), torch.float32)
        self.unit_v = flat(most(m.heads * m.vdim for m in delta))
        self.gates = flat(most(2 * m.heads for m in delta), torch.float32)
        self.diff_q = flat(most([2 * m.heads * pad8(m.dim) for m in diff] + [m.heads * pad8(m.dim) for m in tied]))
        self.attn = flat(most([pad8(m.heads * m.vdim) for m in rec + delta + mem] + [m.heads * pad8(m.vdim) for m in lat + diff] +
                              [m.heads * pad8(m.dim) for m in tied]))
        inter = most([l.down.shape[1] for l in weights.layers if l.down is not None] +
                     [l.moe.shared_down.shape[1] for l in weights.layers if l.moe is not None and l.moe.shared_down is not None])
        self.act = flat(inter)
        self.gate_up = flat(2 * inter) if dt == torch.float32 and dev.type == "cuda" else None
        self.moe_ws = None
        if experts:
            if dev.type == "cuda":
                self.moe_ws = moe_ops.MoEWorkspace(max_tokens, most(f.top for f in experts), most(f.experts for f in experts), pad8(hid),
                                                   most(l.moe.down.shape[2] for l in weights.layers if l.moe is not None), dev, dt,
                                                   gated_f32=dt == torch.float32 and any(f.gated for f in experts))
            else:
                self.moe_ws = moe_ops.MoEWorkspace(1, 1, 1, pad8(hid), 8, dev, dt)
        self.h_last_buf = z(max_seqs, pad8(hid))
        self.h_last = self.h_last_buf[:, :hid]
        self.logits_buf = z(max_seqs, pad8(cfg.vocab) if dev.type == "cuda" else cfg.vocab)
        self.logits = self.logits_buf[:, : cfg.vocab]
        per_cta = 32 if dt == torch.bfloat16 else 4                     # latent heads a decode CTA takes
        diff_ctas = [m.kv_heads * -(-(m.heads // m.kv_heads) // 8) for m in diff] + [m.kv_heads * -(-(m.heads // m.kv_heads) // 16) for m in tied]
        self.hkv = most([-(-m.heads // per_cta) for m in lat] + diff_ctas) or 1      # CTAs per decode row ...
        per_sm = 8 if dt == torch.float32 else (2 if most(m.key_width for m in lat) <= 128 else 1)
        self.decode_ctas = per_sm * (ops.num_sms() if dev.type == "cuda" else 148)       # ... and the device's places for them
        self.decode_splits, self._split_capacity = 1, 1
        # fp32 partial results of a decode row and split: 16 rows per CTA, and (maximum, sum) of each
        self.part_rows = most([m.heads for m in lat] + [16 * n for n in diff_ctas])
        self.part_width = most([pad8(m.rank) for m in lat] + [pad8(m.vdim) for m in diff] + [pad8(m.dim) for m in tied])
        self.part_o = self.part_ml = None
        self.counters = z(max_seqs * (most([-(-m.heads // 16) for m in lat] + diff_ctas) or 1), dtype=torch.int32) if dev.type == "cuda" else None
        self.state = None
        self.scratch: dict = {}
        self.capture = None            # list: gets the summed streams [rows, hidden] after every layer (tests, debugging)

    # ---- the engine's view -------------------------------------------------------------------
    def bind_native(self, kv, max_pages_per_seq: int) -> bool:
        return False                   # layers are launched from Python, decode steps replay CUDA graphs

    def bind_state(self, state) -> None:
        self.state = state

    def native_counter(self, which: int) -> int:
        return 0

    def set_backed_pages(self, num_pages: int) -> None:
        pass

    def set_hidden_taps(self, layers) -> None:
        if layers:
            raise ValueError("hidden taps are not available for hybrid models")

    def ensure_split_scratch(self, splits: int) -> bool:
        if splits <= 1 or self.device.type != "cuda" or splits <= self._split_capacity or not self.cfg.attention_layers:
            return False
        self._split_capacity = splits
        rows = self.max_seqs * self.part_rows * splits
        self.part_o = torch.empty(rows * self.part_width, dtype=torch.float32, device=self.device)
        self.part_ml = torch.empty(rows * 2, dtype=torch.float32, device=self.device)
        return True

    def set_decode_splits(self, splits: int) -> bool:
        self.decode_splits = splits
        return self.ensure_split_scratch(splits)

    # ---- one step ----------------------------------------------------------------------------
    def _rows(self, buf, t, width):
        return buf[: t * width].view(t, width)

    def _recurrent(self, li, m: RecurrentSpec, w: RecurrentWeights, h, y, si):
        t, n = h.shape[0], m.heads * (2 * m.dim + m.vdim)
        qfv = self._rows(self.qfv, t, pad8(n))
        hops.linear(h, w.qfv, qfv[:, :n], f32_out=True)
        raw = hops.hgrn2(qfv, w.gate_bias, w.gate_low, self.state.layers[li]["recurrent"], self._rows(self.rec_o, t, m.heads * m.vdim), m.heads,
                         m.dim, m.vdim, si, scratch=lambda name, shape: self._scratch(name, shape, torch.float32),
                         split=h.dtype == torch.bfloat16)
        width = m.heads * m.vdim
        attn = self._rows(self.attn, t, pad8(width))
        if pad8(width) != width:
            attn[:, width:].zero_()    # the buffer is shared with layers of other widths
        hops.head_rmsnorm(raw, w.norm, self.cfg.norm_eps, attn, m.heads, m.vdim)
        hops.linear(attn, w.o, y)

    def _delta(self, li, m: DeltaSpec, w: DeltaWeights, h, y, si):
        t, width, st = h.shape[0], m.heads * m.vdim, self.state.layers[li]
        proj = self._rows(self.proj, t, pad8(m.conv_width + width))
        hops.linear(h, w.gqkv, proj[:, : m.conv_width + width])
        ab = self._rows(self.ab, t, pad8(2 * m.heads))
        hops.linear(h, w.ab, ab[:, : 2 * m.heads], f32_out=True)
        qk, v = self._rows(self.unit_qk, t, 2 * m.kv_heads * m.dim), self._rows(self.unit_v, t, width)
        gates = self._rows(self.gates, t, 2 * m.heads).view(t, m.heads, 2)
        hops.conv_unit_gates(proj[:, width:], w.conv, st["conv"], ab, w.a_log, w.dt_bias, qk, v, gates, si, m.kv_heads, m.heads, m.dim, m.vdim)
        raw = hops.delta_rule(qk, v, gates, st["recurrent"], self._rows(self.rec_o, t, width), m.heads, m.kv_heads, m.dim, m.vdim, si,
                              blocks=h.dtype == torch.bfloat16, scratch=lambda name, shape: self._scratch(name, shape, torch.float32))
        attn = self._rows(self.attn, t, pad8(width))
        if pad8(width) != width:
            attn[:, width:].zero_()    # the buffer is shared with layers of other widths
        hops.head_rmsnorm(raw, w.norm, self.cfg.norm_eps, attn, m.heads, m.vdim, gate=proj[:, :width])
        hops.linear(attn, w.o, y)

    def _diff(self, li, m: DiffSpec, w: DiffWeights, h, y, kv, si):
        t, dp, vp = h.shape[0], pad8(m.dim), pad8(m.vdim)
        proj = self._rows(self.proj, t, pad8(m.conv_width))
        hops.linear(h, w.qkv, proj[:, : m.conv_width])
        q, attn = self._rows(self.diff_q, t, 2 * m.heads * dp), self._rows(self.attn, t, m.heads * vp)
        hops.conv_rope_append(proj, w.conv, w.bias, self.state.layers[li]["conv"], q, kv.pools[li], w.freq, si, 2 * m.heads, 2 * m.kv_heads, m.kv_heads,
                              m.dim, m.vdim, dp, vp)
        hops.diff_attention(q, attn, kv.pools[li], si, m.heads, m.kv_heads, m.dim, m.vdim, dp, vp, m.scale, w.lam, self.cfg.norm_eps, 1 - m.diff,
                            m.window, m.keep, self.decode_splits, self.part_o, self.part_ml, self.counters)
        hops.linear(attn, w.o, y)

    def _tied(self, li, m: TiedSpec, w: TiedWeights, h, y, kv, si):
        t, dp = h.shape[0], pad8(m.dim)
        proj = self._rows(self.proj, t, pad8(m.proj_width))
        hops.linear(h, w.qkg, proj[:, : m.proj_width])
        q, attn = self._rows(self.diff_q, t, m.heads * dp), self._rows(self.attn, t, m.heads * dp)
        hops.tied_append(proj, w.q_bias, w.k_bias, w.q_gain, self.cfg.norm_eps, m.factor, q, kv.pools[li], si.slots, m.heads, m.kv_heads, m.dim, dp)
        hops.tied_attention(q, attn, kv.pools[li], si, m.heads, m.kv_heads, m.dim, dp, m.softcap, w.slope, w.sink, m.window,
                            proj[:, m.gate_col:m.gate_col + m.heads] if m.gated else None, self.decode_splits, self.part_o, self.part_ml, self.counters)
        hops.linear(attn, w.o, y)

    def _memory(self, li, m: MemorySpec, w: MemoryWeights, h, y, si):
        t, width, st = h.shape[0], m.heads * m.vdim, self.state.layers[li]
        proj = self._rows(self.proj, t, pad8(m.proj_width))
        hops.linear(h, w.qkvg, proj[:, : m.proj_width])
        logits = None
        if m.gated:
            logits = self._rows(self.ab, t, pad8(2 * m.heads))
            hops.linear(h, w.gates, logits[:, : 2 * m.heads], f32_out=True)
        turns = self.turns[m.rot_dims, m.rot_base][1][:t] if m.rot_dims else None
        unit = m.dim ** -0.5
        raw = hops.decay_memory(proj, turns, logits, w.gates_bias, m.gate_cap, w.decay, st["recurrent"], st.get("peak"),
                                self._rows(self.rec_o, t, width), m.heads, m.dim, m.vdim, unit if m.gated else 1.0, 1.0 if m.gated else unit, si,
                                blocks=h.dtype == torch.bfloat16, scratch=lambda name, shape: self._scratch(name, shape, torch.float32))
        attn = self._rows(self.attn, t, pad8(width))
        if pad8(width) != width:
            attn[:, width:].zero_()    # the buffer is shared with layers of other widths
        hops.head_rmsnorm(raw, w.norm, self.cfg.norm_eps, attn, m.heads, m.vdim, gate=proj[:, m.gate_col:m.gate_col + width],
                          gate_act="sigmoid" if m.gated else "silu")
        hops.linear(attn, w.o, y)

    def _experts(self, f: MoeSpec, w: MoeWeights, h):
        t = h.shape[0]
        logits = self._rows(self.ab, t, pad8(f.logits))
        hops.linear(h, w.router, logits[:, : f.logits], f32_out=True)
        out = moe_ops.routed_experts(h, logits[:, : f.experts], w.up, w.down, self.moe_ws, f.top, Act(f.act, f.limit), w.half, f.groups, f.keep,
                                     f.renormalize, w.bias, f.score, f.group_best)
        if w.shared_up is not None:
            y = self.y[:t]
            self._mlp(h, w.shared_up, w.shared_down, Act(f.act, f.shared_limit), w.shared_half, y[:, : self.cfg.hidden])
            out = ExpertRows(out.rows, out.pos, out.weight, y, logits[:, f.experts])
        return out

    def _mlp(self, h, up, down, act: Act, half, y):
        """y = down(act(up h)); ``up`` packed with ``half`` for a gated activation."""
        t = h.shape[0]
        mid = self._rows(self.act, t, down.shape[1])
        if act.gated:
            hops.gated_linear(h, up, half, act, mid, self._rows(self.gate_up, t, up.shape[0]) if self.gate_up is not None else None)
        else:
            hops.act_linear(h, up, act, mid)
        hops.linear(mid, down, y)

    def _latent(self, li, m: LatentSpec, w: LatentWeights, h, y, kv, si):
        t, hp = h.shape[0], m.heads
        dp, cp, vp, kw = pad8(m.dim), pad8(m.rank), pad8(m.vdim), m.key_width
        own = m.kv_from is None
        pool = kv.pools[li if own else m.kv_from]
        qc = self._rows(self.qc, t, pad8(m.proj_width))
        hops.linear(h, w.qc, qc[:, : m.proj_width])
        attn = self._rows(self.attn, t, hp * vp)
        pages = self._expanded_pages(m, w, si)
        rows = si.num_decode if pages else t      # rows that attend to the latents themselves
        qa, oc = self._rows(self.qa, rows, hp * kw), self._rows(self.oc, rows, hp * cp)
        if own:
            rope = None
            if m.rot_dim:
                rope = LatentRope(w.freq, si.positions, hp, m.dim, qa.view(rows * hp, kw) if rows else None, cp, rows)
            hops.latent_append(qc, m.latent_col, w.c_norm, self.cfg.norm_eps, si.slots, pool, m.rank, rope)
        gate = qc[:, m.gate_col:m.gate_col + hp] if m.gated else None
        if rows:
            hops.linear_batched(qc[:rows], w.uk, qa, hp, m.q_width, kw)
            hops.latent_attention(qa.view(rows * hp, kw), oc.view(rows * hp, cp), pool, si, hp, kw, m.scale, m.window, self.decode_splits,
                                  self.part_o, self.part_ml, self.counters, decode_only=bool(pages), vrank=cp, gate=gate)
            hops.linear_batched(oc, w.uv, attn[:rows], hp, cp, vp)
        if pages:
            kc, vc = chunks(m.q_width), chunks(m.vdim)
            hops.latent_prefill_expanded(qc, attn, pool, w.kv, si, hp, kc, vc, m.q_width, vp, m.scale, m.window, pages,
                                         self._scratch("dense", (pages * ops.PAGE, kw)), self._scratch("kv", (pages, hp, kc + vc, ops.PAGE, 64)),
                                         self._scratch("table", (si.num_prefill_seqs, si.page_table.shape[1]), torch.int32), gate)
        hops.linear(attn, w.o, y)

    FUSED_ROWS = 512                   # steps of more rows split norms and input convolutions in two kernels
    EXPAND_BYTES = 1 << 30             # most memory the expanded keys and values of a step may take

    def _expanded_pages(self, m: LatentSpec, w: LatentWeights, si) -> int:
        """Pages to expand for this step's prompts, 0 to attend to the latents: with few queries per visible latent the
        expansion costs more than it saves."""
        if w.kv is None or si.num_prefill_seqs == 0 or si.prefill_ctx is None or self.device.type != "cuda":
            return 0
        pages = hops.visible_pages(si, m.window)
        n, start = si.prefill_len.astype("int64"), (si.prefill_ctx - si.prefill_len).astype("int64")
        seen = start + (n + 1) // 2
        pairs = int((n * (seen.clip(max=m.window) if m.window > 0 else seen)).sum())
        # operations per head: the latent kernel computes scores once per 128 output columns of a wide latent
        head = 64 * (chunks(m.q_width) + chunks(m.vdim))
        direct = pairs * 2 * (m.key_width * max(1, -(-m.rank // 128)) + m.rank)
        expanded = pairs * 2 * head + pages * ops.PAGE * 2 * head * m.key_width
        return pages if direct > expanded and pages * ops.PAGE * m.heads * head * 2 <= self.EXPAND_BYTES else 0

    def _scratch(self, name, shape, dtype=None):
        """Step scratch that grows to the largest step seen (prompt steps only: never inside a captured graph)."""
        n = 1
        for d in shape:
            n *= d
        buf = self.scratch.get(name)
        if buf is None or buf.numel() < n:
            buf = self.scratch[name] = torch.zeros(n, dtype=dtype or self.w.embed.dtype, device=self.device)
        return buf[:n].view(shape)

    def forward(self, si, kv) -> torch.Tensor:
        """Runs one step; returns logits [num_logit_rows, vocab] (a view of a static buffer)."""
        cfg, w, t = self.cfg, self.w, si.num_tokens
        cur, nxt = self.xs[0][:t], self.xs[-1][:t]
        h, y = self.h[:t], self.y[:t]
        wp = pad8(cfg.hidden)
        hops.embed_streams(si.token_ids, w.embed, cur, w.embed_norm, self.loop_in[:t, wp:wp + cfg.hidden] if cfg.loop is not None else None,
                           cfg.embed_scale)
        for freq, table in self.turns.values():
            hops.turn_table(si.positions, freq, table[:t])
        written, out = None, None      # connection whose sublayer output the residual still has to take in, and that output
        entered, add = None, None      # residual that a pass begins with instead of ``cur``, and what is still to be added to it

        def gated(y, source, weight, gate_bias, bias=None):
            """What the residual takes of a sublayer's output: gates over the normed rows the sublayer (before its convolution) came from."""
            if weight is None:
                return y
            gate = self.res_gate[:t]
            hops.linear(source, weight, gate[:, : cfg.hidden])
            return GatedRows(y, gate, gate_bias, bias)

        def step(conn, norm, h, gather=None, conv=None, state=None, plain=None, **kw):
            nonlocal cur, nxt, entered, add
            if conv is not None:
                fold = entered is not None or out is not None
                hops.norm_conv_step(entered if entered is not None else cur[:, 0], nxt[:, 0] if fold else None, out, add, norm, conv, state, h, si,
                                    self.factor if t > self.FUSED_ROWS else None, plain)
                entered = add = None
                if fold:
                    cur, nxt = nxt, cur
                return
            if cfg.residual != "hyper":
                hops.norm_step(cur[:, 0], out, written, norm, h, gather)
                return
            fold = written is not None and gather is None
            hops.hyper_step(cur, nxt if fold else None, out, written, conn.read if conn is not None else None, norm, h, si, gather=gather, **kw)
            if fold:
                cur, nxt = nxt, cur

        lp, passes = cfg.loop, 0
        for ri, li in enumerate(cfg.runs):
            spec, lw, m = cfg.layers[li], w.layers[li], cfg.layers[li].mixer
            state = self.state.layers[ri]
            begins = lp is not None and li == lp.start
            if begins:
                step(None, None, self.loop_in[:t, : cfg.hidden])
                if self.capture is not None and ri > 0:
                    self.capture.append(cur.sum(1))
                hops.linear(self.loop_in[:t], w.loop_in, self.loop_x[:t, : cfg.hidden], f32_out=True)
                entered, add, written, out = self.loop_x[:t, : cfg.hidden], w.loop_step[passes], None, None
                passes += 1
                if lw.conv1 is None:   # the passes that follow work on the stream itself
                    torch.add(entered, add, out=cur[:, 0])
                    entered = add = None
            plain = self.plain[:t] if lw.gate1 is not None and lw.conv1 is not None else None
            step(lw.hc1, lw.norm1, h, conv=lw.conv1, state=state.get("input1"), plain=plain,
                 **({"shift": lw.shift, "prev": state["shift"]} if lw.shift is not None else {}))
            if self.capture is not None and ri > 0 and not begins:
                self.capture.append(cur.sum(1))
            if isinstance(m, RecurrentSpec):
                self._recurrent(ri, m, lw.mixer, h, y[:, : cfg.hidden], si)
            elif isinstance(m, DeltaSpec):
                self._delta(ri, m, lw.mixer, h, y[:, : cfg.hidden], si)
            elif isinstance(m, DiffSpec):
                self._diff(ri, m, lw.mixer, h, y[:, : cfg.hidden], kv, si)
            elif isinstance(m, TiedSpec):
                self._tied(ri, m, lw.mixer, h, y[:, : cfg.hidden], kv, si)
            elif isinstance(m, MemorySpec):
                self._memory(ri, m, lw.mixer, h, y[:, : cfg.hidden], si)
            else:
                self._latent(ri, m, lw.mixer, h, y[:, : cfg.hidden], kv, si)
            written, out = lw.hc1, gated(y, h if plain is None else plain, lw.gate1, lw.gate1_bias, getattr(lw.mixer, "o_bias", None))
            if spec.mlp is None:
                continue
            step(lw.hc2, lw.norm2, h, conv=lw.conv2, state=state.get("input2"))
            written, out = lw.hc2, y
            if isinstance(spec.mlp, MoeSpec):
                out = self._experts(spec.mlp, lw.moe, h)
            else:
                self._mlp(h, lw.gate_up, lw.down, lw.act, lw.half, y[:, : cfg.hidden])
            out = gated(out, h, lw.gate2, lw.gate2_bias)
        if self.capture is not None:
            step(None, None, None)
            self.capture.append(cur.sum(1))
            written, out = None, None
        r = si.num_logit_rows
        hl, logits = self.h_last_buf[:r], self.logits[:r]
        if r > 0:
            step(None, w.final_norm, hl, gather=si.logit_rows[:r])
            hops.linear(hl, w.lm_head, logits)
        return logits
