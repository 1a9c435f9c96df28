"""Decoder whose layers each choose a mixer -- recurrent (HGRN2, gated delta rule) or attention (over paged latents, differential) --
and a feed-forward (gated, routed experts), on hyper-connected residual streams or on one stream normed around every sublayer.

A design of this kind is a :class:`HybridConfig` (layer specs plus constants) and a :class:`HybridWeights`;
``models/registry.py`` says which checkpoint architectures map here and how their files are read.  The executor lowers
a layer to a fixed list of launches over buffers allocated once:

    hyper_step (fold the last sublayer's output into the streams, read-out, norm, token shift), or
    norm_step  (x += norm(the last sublayer's output), norm; sums the rows of routed experts on the way)
    recurrent:  gemm(q | gate | v, fp32 out) | hgrn2 | head_rmsnorm | gemm(o)
    delta:      gemm(gate | q | k | v) | gemm(decay | step size, fp32 out) | conv_unit_gates | delta_rule | head_rmsnorm * gate | gemm(o)
    latent:     gemm(q | latent) | latent_append | gemm per head (W_uk^T q) | latent_attention | gemm per head (W_uv o) | gemm(o);
                prompts over wide latents: latent_gather | gemm (K | V pages) | paged_prefill | gemm(o)
    diff:       gemm(q | k | v) | conv_rope_append | diff_attention (both maps, difference and norm) | gemm(o)
    dense:      hyper_step or norm_step | gemm(gate_up, gated epilogue) | gemm(down)
    experts:    norm_step | gemm(router, fp32 out) | route, permute, gather | grouped gemm(up, relu^2 epilogue) | grouped gemm(down)

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
from ..ops.hybrid import DynamicTanh, HyperConnection, RmsNorm
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
    """Latent attention: ``window`` 0 means every earlier token; ``kv_from`` names the layer whose latents are read."""
    heads: int
    dim: int
    vdim: int
    rank: int
    scale: float
    window: int = 0
    kv_from: int | None = None


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
class MlpSpec:
    inter: int
    act: str = "gelu_tanh"


@dataclass
class MoeSpec:
    """Routed experts down(relu(up h)^2), ``top`` of ``experts`` per token, chosen from the ``keep`` best of ``groups`` equal groups."""
    experts: int
    top: int
    inter: int
    groups: int = 1
    keep: int = 1
    renormalize: bool = False


@dataclass
class LayerSpec:
    mixer: RecurrentSpec | LatentSpec | DeltaSpec | DiffSpec
    mlp: MlpSpec | MoeSpec | None = None


@dataclass
class HybridConfig:
    vocab: int
    hidden: int
    layers: list
    streams: int = 1
    norm_eps: float = 1e-6
    name: str = "hybrid"
    logit_scale: float = 1.0           # folded into the final norm's weight
    residual: str = "hyper"            # "hyper": connected streams, Dynamic-Tanh norms, token shift; "sandwich": RMS norms around a sublayer
    eos_token: int = -1
    max_position: int = 1 << 20        # no positional table: bounded by the pool only
    default_seq_len: int = 8192        # sequence limit when neither the caller nor the package names one

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def latent_layers(self) -> list:
        return [l.mixer for l in self.layers if isinstance(l.mixer, LatentSpec)]

    @property
    def attention_layers(self) -> list:
        return [l.mixer for l in self.layers if isinstance(l.mixer, (LatentSpec, DiffSpec))]

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
        """Shape of one KV page of a layer, None when the layer caches nothing of its own."""
        m = self.layers[layer].mixer
        if isinstance(m, DiffSpec):
            return (m.page_elems,)
        return (ops.PAGE, pad8(m.rank)) if isinstance(m, LatentSpec) and m.kv_from is None else None

    def state_shapes(self, layer: int) -> dict:
        """Per-sequence fp32 state of a layer: name -> shape."""
        m = self.layers[layer].mixer
        shapes = {"shift": (self.hidden,)} if self.residual == "hyper" else {}
        if isinstance(m, (DeltaSpec, DiffSpec)):
            shapes["conv"] = (m.taps - 1, m.conv_width)
        if isinstance(m, (RecurrentSpec, DeltaSpec)):
            shapes["recurrent"] = (m.heads, m.vdim, hops.state_rows(m.dim))
        return shapes

    def validate(self) -> None:
        if self.residual not in ("hyper", "sandwich"):
            raise ValueError(f"unknown residual {self.residual!r}")
        if not 1 <= self.streams <= 8 or (self.residual == "sandwich" and self.streams != 1):
            raise ValueError(f"{self.streams} residual streams are not supported (1 to 8, 1 with norms around the sublayers)")
        for i, layer in enumerate(self.layers):
            m, f = layer.mixer, layer.mlp
            if isinstance(f, MoeSpec):
                if self.residual != "sandwich":
                    raise ValueError(f"layer {i}: routed experts need the residual with norms around the sublayers")
                if f.experts > 256 or f.top > 32 or f.groups < 1 or f.experts % f.groups or not 1 <= f.keep <= f.groups:
                    raise ValueError(f"layer {i}: {f.experts} experts in {f.groups} groups, {f.keep} kept, {f.top} chosen are not supported "
                                     "(at most 256 experts in equal groups, 32 chosen)")
                if not 1 <= f.top <= f.keep * (f.experts // f.groups):
                    raise ValueError(f"layer {i}: {f.top} experts cannot be chosen from {f.keep} groups of {f.experts // f.groups}")
            if isinstance(m, (RecurrentSpec, DeltaSpec)):
                hops.state_rows(m.dim)
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
            if m.rank > 1024:
                raise ValueError(f"layer {i}: latent size {m.rank} is not supported (at most 1024)")
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
            else:
                n += self.hidden * m.heads * (m.dim + m.vdim) + m.rank * m.heads * (m.dim + m.vdim)
                n += self.hidden * m.rank if m.kv_from is None else 0
            if isinstance(layer.mlp, MoeSpec):
                n += self.hidden * layer.mlp.experts * (2 * layer.mlp.inter + 1)
            elif layer.mlp:
                n += 3 * self.hidden * layer.mlp.inter
        return 2 * n

    def kv_bytes_per_token(self, kv_dtype_bytes: int = 2) -> int:
        return kv_dtype_bytes * (sum(pad8(m.rank) for m in self.latent_layers if m.kv_from is None) +
                                 sum(m.page_elems // ops.PAGE for m in self.attention_layers if isinstance(m, DiffSpec)))


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
    qc: torch.Tensor              # [heads * dim_p (+ rank_p), hidden]: query (and latent) projections
    c_norm: torch.Tensor | None   # fp32 [rank]
    uk: torch.Tensor              # [heads * rank_p, dim_p]: W_uk^T per head, folds the key expansion into the query
    uv: torch.Tensor              # [heads * vdim_p, rank_p]: value expansion, applied to the attended latent
    o: torch.Tensor               # [hidden, heads * vdim_p]
    kv: torch.Tensor | None = None   # [heads * (key | value) * dim, rank_p]: both expansions, for prompts (see expand_prompts)


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
class MoeWeights:
    router: torch.Tensor     # [experts, hidden]
    up: torch.Tensor         # [experts, inter_p, hidden_p]
    down: torch.Tensor       # [experts, hidden, inter_p]


@dataclass
class HybridLayer:
    """Norms and residual connections follow ``HybridConfig.residual``: Dynamic-Tanh, hyper-connections and a token shift, or RMS
    norms before (norm1, norm2) and behind (hc1, hc2) the sublayers."""
    norm1: DynamicTanh | RmsNorm
    hc1: HyperConnection | RmsNorm
    mixer: RecurrentWeights | LatentWeights | DeltaWeights | DiffWeights
    shift: torch.Tensor | None = None             # fp32 [hidden]
    norm2: DynamicTanh | RmsNorm | None = None
    hc2: HyperConnection | RmsNorm | None = None
    gate_up: torch.Tensor | None = None
    down: torch.Tensor | None = None
    half: int = 0
    moe: MoeWeights | None = None


@dataclass
class HybridWeights:
    embed: torch.Tensor
    layers: list = field(default_factory=list)
    final_norm: DynamicTanh | None = None
    lm_head: torch.Tensor | None = None
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


def expand_prompts(spec: LatentSpec, dtype) -> bool:
    """Whether prompts of a layer may run on expanded keys and values: the heads fit the paged prefill kernel, and a latent is
    wider than a head (otherwise attending to the latent itself is no more work)."""
    return dtype == torch.bfloat16 and spec.dim == spec.vdim and spec.dim in (64, 128) and spec.rank > spec.dim


def pack_latent(spec: LatentSpec, q, dkv, dkv_norm, uk, uv, o) -> LatentWeights:
    h, dp, rp, vp = spec.heads, pad8(spec.dim), pad8(spec.rank), pad8(spec.vdim)
    qc = pad_head_rows(q, h, dp)
    if dkv is not None:
        qc = torch.cat([qc, pad_head_rows(dkv, 1, rp)], 0)
    ukt = uk.reshape(h, spec.dim, spec.rank).transpose(1, 2)                                   # [h, rank, dim]
    ukt = torch.nn.functional.pad(ukt, (0, dp - spec.dim, 0, rp - spec.rank)).reshape(h * rp, dp)
    kv = None
    if expand_prompts(spec, q.dtype):
        kv = pad_cols(torch.stack([uk.reshape(h, spec.dim, spec.rank), uv.reshape(h, spec.vdim, spec.rank)], 1).reshape(2 * h * spec.dim, spec.rank), rp)
    return LatentWeights(kv=kv, qc=pad_cols(qc), c_norm=None if dkv_norm is None else dkv_norm.float().contiguous(), uk=ukt.contiguous(),
                         uv=pad_cols(pad_head_rows(uv, h, vp), rp),
                         o=torch.nn.functional.pad(o.reshape(o.shape[0], h, spec.vdim), (0, vp - spec.vdim)).reshape(o.shape[0], h * vp).contiguous())


def pack_delta(spec: DeltaSpec, q, k, v, g, a, b, conv, a_log, dt_bias, norm, o) -> DeltaWeights:
    """``conv``: filters of the q, k and v channels, [channels, taps] each."""
    f32 = lambda t: t.float().contiguous()
    return DeltaWeights(gqkv=pad_cols(torch.cat([g, q, k, v], 0)), ab=pad_cols(torch.cat([a, b], 0)), conv=f32(torch.cat(conv, 0).t()), a_log=f32(a_log),
                        dt_bias=f32(dt_bias), norm=f32(norm), o=pad_cols(o))


def pack_diff(spec: DiffSpec, q, k, v, bias, conv, lam: float, o) -> DiffWeights:
    """``bias``, ``conv``: of the q, k and v channels; ``lam``: the layer's weight of the second map."""
    vp = pad8(spec.vdim)
    f32 = lambda t: t.float().contiguous()
    i = torch.arange(spec.rot_dims // 2, dtype=torch.float64)
    freq = spec.rot_base ** (-2 * i / max(spec.rot_dims, 1))
    return DiffWeights(qkv=pad_cols(torch.cat([q, k, v], 0)), bias=f32(torch.cat(bias, 0)), conv=f32(torch.cat(conv, 0).t()), freq=freq.to(q.device),
                       lam=float(lam), o=torch.nn.functional.pad(o.reshape(o.shape[0], spec.heads, spec.vdim), (0, vp - spec.vdim)).reshape(o.shape[0], -1).contiguous())


def pack_moe(router, ups, downs) -> MoeWeights:
    """``ups`` [inter, hidden] and ``downs`` [hidden, inter] of every expert."""
    inter = ups[0].shape[0]
    up = torch.nn.functional.pad(pad_cols(torch.stack(list(ups))), (0, 0, 0, pad8(inter) - inter)).contiguous()
    return MoeWeights(router=pad_cols(router), up=up, down=pad_cols(torch.stack(list(downs))))


def pack_mlp(layer: HybridLayer, gate, up, down) -> None:
    if gate.shape[0] % 32:
        gate, up, down = pad_mlp(gate, up, down)
    layer.half = pick_swiglu_half(gate.shape[0])
    layer.gate_up = pad_cols(ops.pack_gate_up(gate.contiguous(), up.contiguous(), layer.half))
    layer.down = down.contiguous()


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
        norm = conn = lambda: RmsNorm(1 + 0.1 * (rand(hid) - 0.5), cfg.norm_eps)
    taps = lambda m, *rows: [torch.randn(n, m.taps, generator=gen, device=dev) * 0.5 / m.taps for n in rows]
    w = HybridWeights(embed=draw(cfg.vocab, hid))
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
        else:
            own = m.kv_from is None
            mixer = pack_latent(m, draw(m.heads * m.dim, hid), draw(m.rank, hid) if own else None, torch.ones(m.rank, device=dev) if own else None,
                                draw(m.heads * m.dim, m.rank), draw(m.heads * m.vdim, m.rank), draw(hid, m.heads * m.vdim))
        layer = HybridLayer(norm1=norm(), shift=rand(hid) if cfg.residual == "hyper" else None, hc1=conn(), mixer=mixer)
        if spec.mlp is not None:
            layer.norm2, layer.hc2 = norm(), conn()
        if isinstance(spec.mlp, MoeSpec):
            f = spec.mlp
            layer.moe = pack_moe(draw(f.experts, hid), [draw(f.inter, hid) for _ in range(f.experts)], [draw(hid, f.inter) for _ in range(f.experts)])
        elif spec.mlp is not None:
            pack_mlp(layer, draw(spec.mlp.inter, hid), draw(spec.mlp.inter, hid), draw(hid, spec.mlp.inter))
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
        self.xs = [z(max_tokens, cfg.streams, hid, dtype=torch.float32) for _ in range(2 if cfg.residual == "hyper" else 1)]
        self.h, self.y = z(max_tokens, pad8(hid)), z(max_tokens, pad8(hid))
        of = lambda kind: [l.mixer for l in cfg.layers if isinstance(l.mixer, kind)]
        rec, lat, delta, diff = of(RecurrentSpec), of(LatentSpec), of(DeltaSpec), of(DiffSpec)
        experts = [l.mlp for l in cfg.layers if isinstance(l.mlp, MoeSpec)]
        most = lambda widths: max(widths, default=0)
        flat = lambda width, dtype=dt: z(max_tokens * width, dtype=dtype) if width else None    # viewed per layer: rows stay contiguous
        self.qfv = flat(most(pad8(m.heads * (2 * m.dim + m.vdim)) for m in rec), torch.float32)
        self.rec_o = flat(most(m.heads * m.vdim for m in rec + delta), torch.float32)
        self.qc = flat(most(m.heads * pad8(m.dim) + pad8(m.rank) for m in lat))
        self.qa = flat(most(m.heads * pad8(m.rank) for m in lat))
        self.oc = flat(most(m.heads * pad8(m.rank) for m in lat))
        self.proj = flat(most([pad8(m.conv_width + m.heads * m.vdim) for m in delta] + [pad8(m.conv_width) for m in diff]))
        self.ab = flat(most([pad8(2 * m.heads) for m in delta] + [pad8(f.experts) for f in experts]), torch.float32)
        self.unit_qk = flat(most(2 * m.kv_heads * m.dim for m in delta), torch.float32)
        self.unit_v = flat(most(m.heads * m.vdim for m in delta))
        self.gates = flat(most(2 * m.heads for m in delta), torch.float32)
        self.diff_q = flat(most(2 * m.heads * pad8(m.dim) for m in diff))
        self.attn = flat(most([pad8(m.heads * m.vdim) for m in rec + delta] + [m.heads * pad8(m.vdim) for m in lat + diff]))
        inter = most(l.down.shape[1] for l in weights.layers if l.down is not None)
        self.act = flat(inter)
        self.gate_up = flat(2 * inter) if dt == torch.float32 and dev.type == "cuda" else None
        self.moe_ws = None
        if experts:
            if dev.type == "cuda":
                self.moe_ws = moe_ops.MoEWorkspace(max_tokens, most(f.top for f in experts), most(f.experts for f in experts), pad8(hid),
                                                   most(pad8(f.inter) for f in experts), dev, dt)
            else:
                self.moe_ws = moe_ops.MoEWorkspace(1, 1, 1, pad8(hid), 8, dev, dt)
        self.h_last_buf = z(max_seqs, pad8(hid))
        self.h_last = self.h_last_buf[:, :hid]
        self.logits_buf = z(max_seqs, pad8(cfg.vocab) if dev.type == "cuda" else cfg.vocab)
        self.logits = self.logits_buf[:, : cfg.vocab]
        per_cta = 32 if dt == torch.bfloat16 else 4                     # latent heads a decode CTA takes
        diff_ctas = [m.kv_heads * -(-(m.heads // m.kv_heads) // 8) for m in diff]
        self.hkv = most([-(-m.heads // per_cta) for m in lat] + diff_ctas) or 1      # CTAs per decode row ...
        per_sm = 8 if dt == torch.float32 else (2 if most(m.rank for m in lat) <= 128 else 1)
        self.decode_ctas = per_sm * (ops.num_sms() if dev.type == "cuda" else 148)       # ... and the device's places for them
        self.decode_splits, self._split_capacity = 1, 1
        # fp32 partial results of a decode row and split: 16 rows per CTA, and (maximum, sum) of each
        self.part_rows = most([m.heads for m in lat] + [16 * n for n in diff_ctas])
        self.part_width = most([pad8(m.rank) for m in lat] + [pad8(m.vdim) for m in diff])
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

    def _experts(self, f: MoeSpec, w: MoeWeights, h):
        logits = self._rows(self.ab, h.shape[0], pad8(f.experts))
        hops.linear(h, w.router, logits[:, : f.experts], f32_out=True)
        return moe_ops.relu2_experts(h, logits[:, : f.experts], w.up, w.down, self.moe_ws, f.top, f.groups, f.keep, f.renormalize)

    def _latent(self, li, m: LatentSpec, w: LatentWeights, h, y, kv, si):
        t, hp = h.shape[0], m.heads
        dp, rp, vp = pad8(m.dim), pad8(m.rank), pad8(m.vdim)
        own = m.kv_from is None
        pool = kv.pools[li if own else m.kv_from]
        qc = self._rows(self.qc, t, hp * dp + (rp if own else 0))
        hops.linear(h, w.qc, qc)
        if own:
            hops.latent_append(qc[:, hp * dp:], w.c_norm, self.cfg.norm_eps, si.slots, pool, m.rank)
        attn = self._rows(self.attn, t, hp * vp)
        pages = self._expanded_pages(m, w, si)
        rows = si.num_decode if pages else t      # rows that attend to the latents themselves
        if rows:
            qa, oc = self._rows(self.qa, rows, hp * rp), self._rows(self.oc, rows, hp * rp)
            hops.linear_batched(qc[:rows], w.uk, qa, hp, dp, rp)
            hops.latent_attention(qa.view(rows * hp, rp), oc.view(rows * hp, rp), pool, si, hp, rp, m.scale, m.window, self.decode_splits,
                                  self.part_o, self.part_ml, self.counters, decode_only=bool(pages))
            hops.linear_batched(oc, w.uv, attn[:rows], hp, rp, vp)
        if pages:
            hops.latent_prefill_expanded(qc, attn, pool, w.kv, si, hp, m.dim, m.scale, m.window, pages,
                                         self._scratch("dense", (pages * ops.PAGE, rp)), self._scratch("kv", (pages, hp, 2, ops.PAGE, m.dim)),
                                         self._scratch("table", (si.num_prefill_seqs, si.page_table.shape[1]), torch.int32))
        hops.linear(attn, w.o, y)

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
        direct = pairs * 2 * m.rank * (1 + max(1, -(-m.rank // 128)))
        expanded = pairs * 4 * m.dim + pages * ops.PAGE * 4 * m.dim * m.rank
        return pages if direct > expanded and pages * ops.PAGE * m.heads * m.dim * 4 <= self.EXPAND_BYTES else 0

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
        hops.embed_streams(si.token_ids, w.embed, cur)
        written, out = None, None      # connection whose sublayer output the residual still has to take in, and that output

        def step(conn, norm, h, gather=None, **kw):
            nonlocal cur, nxt
            if cfg.residual == "sandwich":
                hops.norm_step(cur[:, 0], out, written, norm, h, gather)
                return
            fold = written is not None and gather is None
            hops.hyper_step(cur, nxt if fold else None, out, written, conn.read if conn is not None else None, norm, h, si, gather=gather, **kw)
            if fold:
                cur, nxt = nxt, cur

        for li, (spec, lw) in enumerate(zip(cfg.layers, w.layers)):
            m = spec.mixer
            step(lw.hc1, lw.norm1, h, **({"shift": lw.shift, "prev": self.state.layers[li]["shift"]} if lw.shift is not None else {}))
            if self.capture is not None and li > 0:
                self.capture.append(cur.sum(1))
            if isinstance(m, RecurrentSpec):
                self._recurrent(li, m, lw.mixer, h, y[:, : cfg.hidden], si)
            elif isinstance(m, DeltaSpec):
                self._delta(li, m, lw.mixer, h, y[:, : cfg.hidden], si)
            elif isinstance(m, DiffSpec):
                self._diff(li, m, lw.mixer, h, y[:, : cfg.hidden], kv, si)
            else:
                self._latent(li, m, lw.mixer, h, y[:, : cfg.hidden], kv, si)
            written, out = lw.hc1, y
            if spec.mlp is None:
                continue
            step(lw.hc2, lw.norm2, h)
            written = lw.hc2
            if isinstance(spec.mlp, MoeSpec):
                out = self._experts(spec.mlp, lw.moe, h)
                continue
            act = self._rows(self.act, t, lw.down.shape[1])
            hops.gated_linear(h, lw.gate_up, lw.half, spec.mlp.act, act,
                              self._rows(self.gate_up, t, lw.gate_up.shape[0]) if self.gate_up is not None else None)
            hops.linear(act, lw.down, y[:, : cfg.hidden])
            out = y
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
