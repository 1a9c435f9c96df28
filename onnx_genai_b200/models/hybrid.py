"""Decoder whose layers each choose a mixer: recurrent (HGRN2) or attention over paged latents, on hyper-connected residual
streams.

A design of this kind is a :class:`HybridConfig` (layer specs plus constants) and a :class:`HybridWeights`;
``models/registry.py`` says which checkpoint architectures map here and how their files are read.  The executor lowers
a layer to a fixed list of launches over buffers allocated once:

    hyper_step (fold the last sublayer's output into the streams, read-out, norm, token shift)
    recurrent:  gemm(q | gate | v, fp32 out) | hgrn2 | head_rmsnorm | gemm(o)
    latent:     gemm(q | latent) | latent_append | gemm per head (W_uk^T q) | latent_attention | gemm per head (W_uv o) | gemm(o);
                prompts over wide latents: latent_gather | gemm (K | V pages) | paged_prefill | gemm(o)
    hyper_step | gemm(gate_up, gated epilogue) | gemm(down)

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
from ..ops.hybrid import DynamicTanh, HyperConnection
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
class MlpSpec:
    inter: int
    act: str = "gelu_tanh"


@dataclass
class LayerSpec:
    mixer: RecurrentSpec | LatentSpec
    mlp: MlpSpec | None = None


@dataclass
class HybridConfig:
    vocab: int
    hidden: int
    layers: list
    streams: int = 1
    norm_eps: float = 1e-6
    name: str = "hybrid"
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
    def num_heads(self) -> int:
        return max((m.heads for m in self.latent_layers), default=1)

    num_kv_heads = 1

    @property
    def sliding_window(self) -> int:
        """Tokens of latents a sequence has to keep: the widest window, 0 when some layer sees everything."""
        windows = [m.window for m in self.latent_layers]
        return 0 if any(w <= 0 for w in windows) else max(windows, default=1)

    attention_sinks = 0
    has_state = True                   # the token shift alone is per-sequence state

    def kv_page_shape(self, layer: int, kv_heads: int = 1):
        """Shape of one KV page of a layer, None when the layer caches nothing of its own."""
        m = self.layers[layer].mixer
        return (ops.PAGE, pad8(m.rank)) if isinstance(m, LatentSpec) and m.kv_from is None else None

    def state_shapes(self, layer: int) -> dict:
        """Per-sequence fp32 state of a layer: name -> shape."""
        m = self.layers[layer].mixer
        shapes = {"shift": (self.hidden,)}
        if isinstance(m, RecurrentSpec):
            shapes["recurrent"] = (m.heads, m.vdim, hops.state_rows(m.dim))
        return shapes

    def validate(self) -> None:
        if not 1 <= self.streams <= 8:
            raise ValueError(f"{self.streams} residual streams are not supported (1 to 8)")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if isinstance(m, RecurrentSpec):
                hops.state_rows(m.dim)
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
            else:
                n += self.hidden * m.heads * (m.dim + m.vdim) + m.rank * m.heads * (m.dim + m.vdim)
                n += self.hidden * m.rank if m.kv_from is None else 0
            n += 3 * self.hidden * layer.mlp.inter if layer.mlp else 0
        return 2 * n

    def kv_bytes_per_token(self, kv_dtype_bytes: int = 2) -> int:
        return sum(pad8(m.rank) for m in self.latent_layers if m.kv_from is None) * kv_dtype_bytes


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
class HybridLayer:
    norm1: DynamicTanh
    shift: torch.Tensor           # fp32 [hidden]
    hc1: HyperConnection
    mixer: RecurrentWeights | LatentWeights
    norm2: DynamicTanh | None = None
    hc2: HyperConnection | None = None
    gate_up: torch.Tensor | None = None
    down: torch.Tensor | None = None
    half: int = 0


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
    norm = lambda: DynamicTanh(0.5 + rand(1), 1 + 0.1 * (rand(hid) - 0.5), 0.1 * (rand(hid) - 0.5))
    conn = lambda: HyperConnection(rand(st) / st + 0.5 / st, 0.5 + rand(st), torch.eye(st, device=dev) * 0.8 + 0.2 * rand(st, st) / st)
    w = HybridWeights(embed=draw(cfg.vocab, hid))
    for spec in cfg.layers:
        m = spec.mixer
        if isinstance(m, RecurrentSpec):
            mixer = pack_recurrent(m, draw(m.heads * m.dim, hid), draw(m.heads * m.dim, hid), 2 * rand(m.heads * m.dim), 0.5 * rand(m.heads * m.dim),
                                   draw(m.heads * m.vdim, hid), torch.ones(m.vdim, device=dev), draw(hid, m.heads * m.vdim))
        else:
            own = m.kv_from is None
            mixer = pack_latent(m, draw(m.heads * m.dim, hid), draw(m.rank, hid) if own else None, torch.ones(m.rank, device=dev) if own else None,
                                draw(m.heads * m.dim, m.rank), draw(m.heads * m.vdim, m.rank), draw(hid, m.heads * m.vdim))
        layer = HybridLayer(norm1=norm(), shift=rand(hid), hc1=conn(), mixer=mixer)
        if spec.mlp is not None:
            layer.norm2, layer.hc2 = norm(), conn()
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
        self.xs = [z(max_tokens, cfg.streams, hid, dtype=torch.float32) for _ in range(2)]      # residual streams, double buffered
        self.h, self.y = z(max_tokens, pad8(hid)), z(max_tokens, pad8(hid))
        rec = [l.mixer for l in cfg.layers if isinstance(l.mixer, RecurrentSpec)]
        lat = cfg.latent_layers
        flat = lambda width, dtype=dt: z(max_tokens * width, dtype=dtype) if width else None    # viewed per layer: rows stay contiguous
        self.qfv = flat(max((pad8(m.heads * (2 * m.dim + m.vdim)) for m in rec), default=0), torch.float32)
        self.rec_o = flat(max((m.heads * m.vdim for m in rec), default=0), torch.float32)
        self.qc = flat(max((m.heads * pad8(m.dim) + pad8(m.rank) for m in lat), default=0))
        self.qa = flat(max((m.heads * pad8(m.rank) for m in lat), default=0))
        self.oc = flat(max((m.heads * pad8(m.rank) for m in lat), default=0))
        self.attn = flat(max([pad8(m.heads * m.vdim) for m in rec] + [m.heads * pad8(m.vdim) for m in lat], default=0))
        inter = max((l.down.shape[1] for l in weights.layers if l.down is not None), default=0)
        self.act = flat(inter)
        self.gate_up = flat(2 * inter) if dt == torch.float32 and dev.type == "cuda" else None
        self.h_last_buf = z(max_seqs, pad8(hid))
        self.h_last = self.h_last_buf[:, :hid]
        self.logits_buf = z(max_seqs, pad8(cfg.vocab) if dev.type == "cuda" else cfg.vocab)
        self.logits = self.logits_buf[:, : cfg.vocab]
        per_cta = 32 if dt == torch.bfloat16 else 4                     # heads a decode CTA takes
        self.hkv = max((-(-m.heads // per_cta) for m in lat), default=1)      # CTAs per decode row ...
        per_sm = 8 if dt == torch.float32 else (2 if max((m.rank for m in lat), default=0) <= 128 else 1)
        self.decode_ctas = per_sm * (ops.num_sms() if dev.type == "cuda" else 148)       # ... and the device's places for them
        self.decode_splits, self._split_capacity = 1, 1
        self.part_o = self.part_ml = None
        self.counters = z(max_seqs * max((-(-m.heads // 16) for m in lat), default=1), dtype=torch.int32) if dev.type == "cuda" else None
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
        if splits <= 1 or self.device.type != "cuda" or splits <= self._split_capacity or not self.cfg.latent_layers:
            return False
        self._split_capacity = splits
        rows = self.max_seqs * max(m.heads for m in self.cfg.latent_layers) * splits
        self.part_o = torch.empty(rows * max(pad8(m.rank) for m in self.cfg.latent_layers), dtype=torch.float32, device=self.device)
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
        cur, nxt = self.xs[0][:t], self.xs[1][:t]
        h, y = self.h[:t], self.y[:t]
        hops.embed_streams(si.token_ids, w.embed, cur)
        written = None                 # hyper-connection whose sublayer output (in y) the streams still have to take in

        def step(read, norm, h, **kw):
            nonlocal cur, nxt
            hops.hyper_step(cur, nxt if written is not None else None, y if written is not None else None, written, read, norm, h, si, **kw)
            if written is not None:
                cur, nxt = nxt, cur

        for li, (spec, lw) in enumerate(zip(cfg.layers, w.layers)):
            step(lw.hc1.read, lw.norm1, h, shift=lw.shift, prev=self.state.layers[li]["shift"])
            if self.capture is not None and li > 0:
                self.capture.append(cur.sum(1))
            if isinstance(spec.mixer, RecurrentSpec):
                self._recurrent(li, spec.mixer, lw.mixer, h, y[:, : cfg.hidden], si)
            else:
                self._latent(li, spec.mixer, lw.mixer, h, y[:, : cfg.hidden], kv, si)
            written = lw.hc1
            if spec.mlp is not None:
                step(lw.hc2.read, lw.norm2, h)
                act = self._rows(self.act, t, lw.down.shape[1])
                hops.gated_linear(h, lw.gate_up, lw.half, spec.mlp.act, act,
                                  self._rows(self.gate_up, t, lw.gate_up.shape[0]) if self.gate_up is not None else None)
                hops.linear(act, lw.down, y[:, : cfg.hidden])
                written = lw.hc2
        if self.capture is not None:
            hops.hyper_step(cur, nxt, y, written, None, None, None, si)
            self.capture.append(nxt.sum(1))
        r = si.num_logit_rows
        hl, logits = self.h_last_buf[:r], self.logits[:r]
        if r > 0:
            hops.hyper_step(cur, None, y, written, None, w.final_norm, hl, si, gather=si.logit_rows[:r])
            hops.linear(hl, w.lm_head, logits)
        return logits
