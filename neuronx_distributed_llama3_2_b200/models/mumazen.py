"""Mumazen: a decoder-only hybrid family of state-space mixers whose layers are listed in the configuration, one by one.

  * entry: token embedding times ``embedding.scale``; the residual stream is fp32, pre-norm, every sublayer's result times a
    layer scale vector and one constant: ``x += m * ls1 * mixer(norm1 x)``, ``x += m * ls2 * ff(norm2 x)``;
  * ``mamba1``: selective scan (``ops/state_space.py``) -- a short convolution with silu, step sizes through a low-rank pair, one
    decay per channel and state, output gate ``silu(z)``;
  * ``parallel``: two mixers on the same normed input, ``left_scale * left + right_scale * right``.  Left: softmax attention of
    grouped heads over the KV cache, partial "rotate half" rotation with linearly slowed frequencies, soft-capped scores, an
    output gate ``sigmoid(W_g h)`` per element.  Right: state-space heads with one decay per head, ``B`` and ``C`` shared by the
    heads of a group, behind one short convolution; gate ``silu(z)``, then the RMS norm over equal groups of columns;
  * feed-forward: dense with biases, ``g sigmoid(1.702 g) (u + 1)`` on clamped ``g`` and ``u``; or a mixture of experts without a
    gate (squared relu) whose softmax scores, chosen with an additive correction, are divided by their sum, with identity
    experts and a shared expert behind a sigmoid gate of its own;
  * ``loop``: a range of layers runs several times in a row with the same weights; every pass has cache and state of its own
    (``layer_runs()`` is the order, one cache index per run).  Ahead of every pass but the first the embedding output is added to
    the stream, ahead of every pass a learned vector of that pass;
  * output head of its own.

Parameter modules only; the forward over the KV cache and the recurrent state lives in
``inference/hybrid.py: MumazenInferenceModel``.  What multiplies a mixer's input is ONE fused matrix ``in_proj`` (``columns`` says
where each part starts), except the rows that make step sizes, whose products stay fp32.  Tensor parallelism is not wired
for this family.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..modules.moe.sparse import SparseMoE
from ..ops.linear import gemm_nt
from ..parallel.layers import ColumnParallelLinear, ParallelEmbedding, RowParallelLinear

COLUMN_ALIGN = 8                # parts of a fused projection start on 16-byte boundaries (bf16)
GLU_SLOPE = 1.702               # inside the sigmoid of the dense feed-forward's gate


@dataclass
class RotaryConfig:
    dims: int
    base: float
    factor: float = 1.0                # every frequency is divided by it

    @classmethod
    def from_dict(cls, d: Optional[Dict[str, Any]]) -> Optional["RotaryConfig"]:
        if not d or not d.get("dims"):
            return None
        c = cls(dims=int(d["dims"]), base=float(d["base"]), factor=float((d.get("scaling") or {}).get("factor", 1.0)))
        if c.dims % 2:
            raise ValueError(f"rotation over an odd number of dimensions ({c.dims})")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"dims": self.dims, "base": self.base}
        if self.factor != 1.0:
            d["scaling"] = {"factor": self.factor}
        return d


@dataclass
class CappedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    rot: Optional[RotaryConfig]

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "CappedAttentionConfig":
        c = cls(heads=int(d["heads"]), kv_heads=int(d.get("kv_heads", d["heads"])), dim=int(d["dim"]),
                vdim=int(d.get("vdim", d["dim"])), scale=float(d["scale"]),
                softcap=float(d["softcap"]) if d.get("softcap") else None, rot=RotaryConfig.from_dict(d.get("rot")))
        if c.heads % c.kv_heads:
            raise ValueError(f"attention: {c.heads} query heads over {c.kv_heads} key/value heads")
        if c.rot is not None and c.rot.dims > c.dim:
            raise ValueError(f"attention: rotation over {c.rot.dims} of {c.dim} dimensions")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale}
        if self.softcap:
            d["softcap"] = self.softcap
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d

    @property
    def columns(self) -> int:                       # q | k | v
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)

    @property
    def width(self) -> int:                         # of the gated heads
        return self.heads * self.vdim


@dataclass
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                          # taps of the short convolution
    norm_groups: int

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "StateSpaceConfig":
        c = cls(heads=int(d["heads"]), vdim=int(d["vdim"]), state=int(d["state"]), groups=int(d.get("groups", 1)),
                conv=int(d["conv"]), norm_groups=int(d.get("norm_groups", 1)))
        if c.heads % c.groups:
            raise ValueError(f"state-space heads: {c.heads} heads over {c.groups} groups")
        if c.inner % c.norm_groups:
            raise ValueError(f"state-space heads: {c.inner} columns in {c.norm_groups} norm groups")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:                      # x | B | C, convolved together
        return self.inner + 2 * self.groups * self.state


@dataclass
class ParallelMixerConfig:
    left: CappedAttentionConfig
    right: StateSpaceConfig
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ParallelMixerConfig":
        return cls(left=CappedAttentionConfig.from_dict(d["left"]), right=StateSpaceConfig.from_dict(d["right"]),
                   left_scale=float(d["left_scale"]), right_scale=float(d["right_scale"]))

    def to_dict(self) -> Dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                "right_scale": self.right_scale}

    def parts(self) -> List[Tuple[str, int]]:
        return [("qkv", self.left.columns), ("g", self.left.width), ("z", self.right.inner), ("xbc", self.right.channels)]


@dataclass
class SelectiveScanConfig:
    inner: int
    state: int
    dt_rank: int
    conv: int

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "SelectiveScanConfig":
        return cls(inner=int(d["inner"]), state=int(d["state"]), dt_rank=int(d["dt_rank"]), conv=int(d["conv"]))

    def to_dict(self) -> Dict[str, Any]:
        return {"inner": self.inner, "state": self.state, "dt_rank": self.dt_rank, "conv": self.conv}

    def parts(self) -> List[Tuple[str, int]]:
        return [("x", self.inner), ("z", self.inner)]


@dataclass
class FeedForwardConfig:
    kind: str                          # "dense" | "moe"
    ff: int
    limit: float = 0.0                 # dense: clamp of gate and up
    experts: int = 0
    identity: int = 0
    top: int = 0
    shared_ff: int = 0

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "FeedForwardConfig":
        kind = d.get("kind", "dense")
        if kind == "dense":
            return cls(kind="dense", ff=int(d["ff"]), limit=float(d["limit"]))
        if kind == "moe":
            r = d["router"]
            c = cls(kind="moe", ff=int(d["expert"]["ff"]), experts=int(r["experts"]), identity=int(r.get("identity") or 0),
                    top=int(r["top"]), shared_ff=int((d.get("shared") or {}).get("ff", 0)))
            if not 1 <= c.top <= c.experts + c.identity:
                raise ValueError(f"mixture of experts: top {c.top} of {c.experts} + {c.identity}")
            return c
        raise ValueError(f"unknown feed-forward kind {kind!r}")

    def to_dict(self) -> Dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff, "limit": self.limit}
        r: Dict[str, Any] = {"experts": self.experts, "top": self.top}
        if self.identity:
            r["identity"] = self.identity
        d: Dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": r}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


MIXER_CONFIGS: Dict[str, Callable[[Dict[str, Any]], Any]] = {"parallel": ParallelMixerConfig.from_dict,
                                                             "mamba1": SelectiveScanConfig.from_dict}


@dataclass
class MumazenLayerConfig:
    type: str
    mixer: Any
    mlp: Optional[FeedForwardConfig]


@dataclass
class MumazenConfig:
    vocab_size: int
    hidden_size: int
    layers: List[MumazenLayerConfig] = field(default_factory=list)
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None          # (start, stop, times): layers start .. stop-1 run `times` times
    rms_norm_eps: float = 1e-6
    torch_dtype: torch.dtype = torch.bfloat16
    model_type: str = "mumazen"
    # read by shared inference code
    sequence_parallel_enabled: bool = False
    activation_checkpointing: bool = False
    initializer_range: float = 0.02

    @property
    def num_hidden_layers(self) -> int:
        """Layer RUNS: what the cache / state manager holds an entry for."""
        return len(self.layer_runs())

    def layer_runs(self) -> List[int]:
        """The layer index of every run, in order: the looped range ``times`` times in a row, then the rest."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def pass_starts(self) -> Dict[int, int]:
        """``{run: pass}`` for the runs that begin a pass of the looped range."""
        if self.loop is None:
            return {}
        a, b, times = self.loop
        return {a + t * (b - a): t for t in range(times)}

    @classmethod
    def from_dict(cls, d: Dict[str, Any], torch_dtype: torch.dtype = torch.bfloat16) -> "MumazenConfig":
        layers: List[MumazenLayerConfig] = []
        for i, L in enumerate(d["layers"]):
            if L["type"] not in MIXER_CONFIGS:
                raise ValueError(f"layer {i}: unknown mixer type {L['type']!r} (known: {sorted(MIXER_CONFIGS)})")
            layers.append(MumazenLayerConfig(L["type"], MIXER_CONFIGS[L["type"]](L["mixer"]),
                                             FeedForwardConfig.from_dict(L["mlp"]) if L.get("mlp") else None))
        loop = None
        if d.get("loop"):
            lp = d["loop"]
            loop = (int(lp["start"]), int(lp["stop"]), int(lp.get("times", 1)))
            if not (0 <= loop[0] < loop[1] <= len(layers)) or loop[2] < 1:
                raise ValueError(f"loop {loop} over {len(layers)} layers")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   residual_mult=float(d.get("residual_mult", 1.0)), loop=loop, rms_norm_eps=float(d["norm"]["eps"]),
                   torch_dtype=torch_dtype)

    @classmethod
    def from_json(cls, path: str, torch_dtype: torch.dtype = torch.bfloat16) -> "MumazenConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path) as f:
            return cls.from_dict(json.load(f), torch_dtype)

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": "Mumazen", "vocab": self.vocab_size, "width": self.hidden_size,
                             "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult,
                             "norm": {"eps": self.rms_norm_eps},
                             "layers": [{"type": L.type, "mixer": L.mixer.to_dict(),
                                         "mlp": L.mlp.to_dict() if L.mlp else None} for L in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d


def _init(std: float) -> Callable:
    return lambda w: nn.init.normal_(w, mean=0.0, std=std)


def _up8(n: int) -> int:
    return (n + COLUMN_ALIGN - 1) // COLUMN_ALIGN * COLUMN_ALIGN


def in_proj_columns(layer: MumazenLayerConfig) -> Tuple[Dict[str, Tuple[int, int]], int]:
    """``{part: (first column, columns)}`` of a layer's fused mixer projection, and its total width.  Every part starts on a
    multiple of ``COLUMN_ALIGN`` columns (rows of zeros fill the gaps)."""
    cols, at = {}, 0
    for name, n in layer.mixer.parts():
        cols[name] = (at, n)
        at = _up8(at + n)
    return cols, at


def x_proj_columns(m: SelectiveScanConfig) -> Tuple[int, int, int, int]:
    """Of the selective scan's second projection (its products stay fp32): padded columns of the low-rank step sizes, first
    column of B and of C, total width."""
    r = _up8(m.dt_rank)
    b, c = r, r + _up8(m.state)
    return r, b, c, c + _up8(m.state)


def out_proj_columns(m: ParallelMixerConfig) -> Tuple[int, int]:
    """Of a parallel mixer's joint output projection: first column of the right branch, total width."""
    right = _up8(m.left.width)
    return right, right + _up8(m.right.inner)


def _linear_in(config: MumazenConfig, n_in: int, n_out: int, device) -> ColumnParallelLinear:
    return ColumnParallelLinear(n_in, n_out, bias=False, gather_output=False, dtype=config.torch_dtype, device=device,
                                init_method=_init(config.initializer_range))


def _linear_out(config: MumazenConfig, n_in: int, device) -> RowParallelLinear:
    return RowParallelLinear(n_in, config.hidden_size, bias=False, input_is_parallel=True, dtype=config.torch_dtype,
                             device=device, init_method=_init(config.initializer_range))


class ParallelMixer(nn.Module):
    """Both branches' own tensors (their input rows are part of the layer's ``in_proj``): rows that make the step sizes, the
    convolution ``[taps, channels]`` over x | B | C, decays, skip, norm weight (times ``right_scale``, as the norm's fp32 epilogue
    applies it); and ONE output projection over [gated attention heads | normed state-space heads], whose inputs carry the
    branch scales."""

    def __init__(self, config: MumazenConfig, m: ParallelMixerConfig, device=None):
        super().__init__()
        self.cfg = m
        r = m.right
        f32 = dict(dtype=torch.float32, device=device)
        self.dt_proj = nn.Parameter(torch.zeros(_up8(r.heads), config.hidden_size, dtype=config.torch_dtype, device=device))
        self.conv_weight = nn.Parameter(torch.empty(r.conv, r.channels, **f32).normal_(0.0, 0.3))
        self.conv_bias = nn.Parameter(torch.zeros(r.channels, **f32))
        self.dt_bias = nn.Parameter(torch.zeros(r.heads, **f32))
        self.a_log = nn.Parameter(torch.zeros(r.heads, **f32))
        self.d_skip = nn.Parameter(torch.ones(r.heads, **f32))
        self.out_norm = nn.Parameter(torch.full((r.inner,), m.right_scale, **f32))
        self.o_proj = _linear_out(config, out_proj_columns(m)[1], device)


class SelectiveScanMixer(nn.Module):
    """Convolution ``[taps, channels]``, the projection of the convolved channels to [low-rank step sizes | B | C] (fp32
    products), the step sizes' second half, decays ``[inner, state]``, skip, output projection."""

    def __init__(self, config: MumazenConfig, m: SelectiveScanConfig, device=None):
        super().__init__()
        self.cfg = m
        r, _, _, n = x_proj_columns(m)
        f32 = dict(dtype=torch.float32, device=device)
        act = dict(dtype=config.torch_dtype, device=device)
        std = config.initializer_range
        self.conv_weight = nn.Parameter(torch.empty(m.conv, m.inner, **f32).normal_(0.0, 0.3))
        self.conv_bias = nn.Parameter(torch.zeros(m.inner, **f32))
        self.x_proj = nn.Parameter(torch.empty(n, m.inner, **act).normal_(0.0, std))
        self.dt_proj = nn.Parameter(torch.empty(m.inner, r, **act).normal_(0.0, std))
        self.dt_bias = nn.Parameter(torch.zeros(m.inner, **f32))
        self.a_log = nn.Parameter(torch.zeros(m.inner, m.state, **f32))
        self.d_skip = nn.Parameter(torch.ones(m.inner, **f32))
        self.o_proj = _linear_out(config, m.inner, device)


MIXERS: Dict[str, Callable[..., nn.Module]] = {"parallel": ParallelMixer, "mamba1": SelectiveScanMixer}


class DenseClampedMlp(nn.Module):
    """``down(g sigmoid(1.702 g) (u + 1)) + b`` on clamped biased projections; gate | up rows fused, biases fp32 (added inside
    the kernels).  The inner size is padded to a multiple of 8 with zero columns of ``down``."""

    def __init__(self, config: MumazenConfig, m: FeedForwardConfig, device=None):
        super().__init__()
        self.limit, self.ff, self.ff_pad = m.limit, m.ff, _up8(m.ff)
        f32 = dict(dtype=torch.float32, device=device)
        self.gate_up_proj = _linear_in(config, config.hidden_size, 2 * self.ff_pad, device)
        self.gate_bias, self.up_bias = nn.Parameter(torch.zeros(self.ff_pad, **f32)), nn.Parameter(torch.zeros(self.ff_pad, **f32))
        self.down_proj = _linear_out(config, self.ff_pad, device)
        self.down_bias = nn.Parameter(torch.zeros(config.hidden_size, **f32))


class MumazenDecoderLayer(nn.Module):
    """``ls1`` / ``ls2`` hold the layer scales times ``residual_mult``."""

    def __init__(self, config: MumazenConfig, layer: MumazenLayerConfig, device=None):
        super().__init__()
        W = config.hidden_size
        f32 = dict(dtype=torch.float32, device=device)
        self.type = layer.type
        self.columns, n_out = in_proj_columns(layer)
        self.norm1 = nn.Parameter(torch.ones(W, **f32))
        self.ls1 = nn.Parameter(torch.full((W,), config.residual_mult, **f32))
        self.in_proj = _linear_in(config, W, n_out, device)
        self.mixer = MIXERS[layer.type](config, layer.mixer, device=device)
        self.mlp = None
        self.mlp_kind = layer.mlp.kind if layer.mlp is not None else None
        if layer.mlp is not None:
            m = layer.mlp
            self.norm2 = nn.Parameter(torch.ones(W, **f32))
            self.ls2 = nn.Parameter(torch.full((W,), config.residual_mult, **f32))
            if m.kind == "dense":
                self.mlp = DenseClampedMlp(config, m, device=device)
            else:
                self.mlp = SparseMoE(W, m.experts, m.top, m.ff, None, num_identity_experts=m.identity,
                                     shared_intermediate_size=m.shared_ff, dtype=config.torch_dtype, device=device,
                                     normalize=True, gated=False)


class Fp32LogitsHead(ColumnParallelLinear):
    """An output head of its own whose logits stay in fp32; its rows are padded to a multiple of 8 with zeros, so that every
    vocabulary runs on the same kernels."""

    def __init__(self, width: int, vocab: int, **kw):
        super().__init__(width, _up8(vocab), **kw)
        self.vocab = vocab

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        w = self.weight
        y = gemm_nt(x.reshape(-1, x.shape[-1]).to(w.dtype), w, out_dtype=torch.float32)
        if w.shape[0] != self.vocab:
            y = y[:, : self.vocab].contiguous()
        return y.reshape(x.shape[:-1] + (self.vocab,))


class MumazenForCausalLM(nn.Module):
    """``layers`` holds one module per configured layer; ``layer_sequence()`` is the list the model runs, in which a looped
    layer appears once per pass (same module, another cache / state index)."""

    def __init__(self, config: MumazenConfig, device=None):
        super().__init__()
        self.config = config
        dt = config.torch_dtype
        f32 = dict(dtype=torch.float32, device=device)
        self.embed_tokens = ParallelEmbedding(config.vocab_size, config.hidden_size, dtype=dt, device=device,
                                              init_method=_init(config.initializer_range))
        self.layers = nn.ModuleList([MumazenDecoderLayer(config, L, device=device) for L in config.layers])
        self.loop_step = nn.Parameter(torch.zeros(config.loop[2], config.hidden_size, **f32)) if config.loop is not None else None
        self.norm = nn.Parameter(torch.ones(config.hidden_size, **f32))
        self.lm_head = Fp32LogitsHead(config.hidden_size, config.vocab_size, bias=False, gather_output=False, dtype=dt,
                                      device=device, init_method=_init(config.initializer_range))

    def layer_sequence(self) -> List[MumazenDecoderLayer]:
        return [self.layers[i] for i in self.config.layer_runs()]


def _padded(w: torch.Tensor, rows: int, cols: Optional[int] = None) -> torch.Tensor:
    """``w [r, c]`` in the corner of a zero matrix ``[rows, cols]``."""
    out = w.new_zeros(rows, cols if cols is not None else w.shape[1])
    out[: w.shape[0], : w.shape[1]] = w
    return out


def convert_mumazen_state_dict(sd: Dict[str, torch.Tensor], config: MumazenConfig) -> Dict[str, torch.Tensor]:
    """Checkpoint names (``embed``, ``loop.step``, ``final.norm``, ``head``, ``l<i>.norm1 / norm2 / ls1 / ls2``,
    ``l<i>.mix.<name>``, ``l<i>.mlp.<name>``, biases ``<name>.b``; linear weights ``[out, in]``) -> this module's state dict.
    Constants of the configuration that multiply a vector are folded into it in fp32."""
    W, res = config.hidden_size, config.residual_mult
    out: Dict[str, torch.Tensor] = {"embed_tokens.weight": sd["embed"], "norm": sd["final.norm"].float(),
                                    "lm_head.weight": _padded(sd["head"], _up8(config.vocab_size))}
    if config.loop is not None:
        out["loop_step"] = sd["loop.step"].float()
    for i, L in enumerate(config.layers):
        src, dst, m = f"l{i}.", f"layers.{i}.", L.mixer
        mix = lambda n: sd[src + "mix." + n]                                          # noqa: E731
        cols, n_out = in_proj_columns(L)
        to = dst + "mixer."
        out[dst + "norm1"], out[dst + "ls1"] = sd[src + "norm1"].float(), sd[src + "ls1"].float() * res
        if L.type == "mamba1":
            parts = {"x": mix("in")[: m.inner], "z": mix("in")[m.inner:]}
            r, b, c, n = x_proj_columns(m)
            xp, rows = mix("x").new_zeros(n, m.inner), mix("x")
            xp[: m.dt_rank] = rows[: m.dt_rank]
            xp[b: b + m.state], xp[c: c + m.state] = rows[m.dt_rank: m.dt_rank + m.state], rows[m.dt_rank + m.state:]
            out[to + "x_proj"], out[to + "dt_proj"] = xp, _padded(mix("dt"), m.inner, r)
            out[to + "dt_bias"] = mix("dt.b").float()
            out[to + "conv_weight"], out[to + "conv_bias"] = mix("conv").float().t(), mix("conv.b").float()
            out[to + "a_log"], out[to + "d_skip"] = mix("A_log").float(), mix("D").float()
            out[to + "o_proj.weight"] = mix("o")
        else:
            s = m.right
            win = mix("right.in")
            parts = {"qkv": torch.cat([mix("left.q"), mix("left.k"), mix("left.v")], dim=0), "g": mix("left.g"),
                     "z": win[: s.inner], "xbc": win[s.inner: s.inner + s.channels]}
            out[to + "dt_proj"] = _padded(win[s.inner + s.channels:], _up8(s.heads))
            out[to + "dt_bias"] = mix("right.dt_bias").float()
            out[to + "conv_weight"], out[to + "conv_bias"] = mix("right.conv").float().t(), mix("right.conv.b").float()
            out[to + "a_log"], out[to + "d_skip"] = mix("right.A_log").float(), mix("right.D").float()
            out[to + "out_norm"] = mix("right.norm").float() * m.right_scale
            at, n = out_proj_columns(m)
            o = mix("left.o").new_zeros(W, n)
            o[:, : m.left.width], o[:, at: at + s.inner] = mix("left.o"), mix("right.o")
            out[to + "o_proj.weight"] = o
        first = next(iter(parts.values()))
        fused = first.new_zeros(n_out, W)
        for name, (at, n) in cols.items():
            assert parts[name].shape == (n, W), (i, name, tuple(parts[name].shape), n)
            fused[at: at + n] = parts[name]
        out[dst + "in_proj.weight"] = fused
        if L.mlp is None:
            continue
        out[dst + "norm2"], out[dst + "ls2"] = sd[src + "norm2"].float(), sd[src + "ls2"].float() * res
        ml = lambda n: sd[src + "mlp." + n]                                           # noqa: E731
        to = dst + "mlp."
        if L.mlp.kind == "dense":
            F, Fp = L.mlp.ff, _up8(L.mlp.ff)
            out[to + "gate_up_proj.weight"] = torch.cat([_padded(ml("gate"), Fp), _padded(ml("up"), Fp)], dim=0)
            for n in ("gate", "up"):
                bias = torch.zeros(Fp)
                bias[:F] = ml(n + ".b").float()
                out[to + n + "_bias"] = bias
            out[to + "down_proj.weight"], out[to + "down_bias"] = _padded(ml("down"), W, Fp), ml("down.b").float()
        else:
            E = L.mlp.experts
            out[to + "router.linear_router.weight"] = ml("router").float()
            out[to + "router.correction"] = ml("correction").float()
            out[to + "experts.up_proj.weight"] = torch.stack([ml(f"e{e}.up").t() for e in range(E)])
            out[to + "experts.down_proj.weight"] = torch.stack([ml(f"e{e}.down").t() for e in range(E)])
            if L.mlp.shared_ff:
                out[to + "shared.up_proj.weight"] = ml("shared.up").t().unsqueeze(0)
                out[to + "shared.down_proj.weight"] = ml("shared.down").t().unsqueeze(0)
                out[to + "shared_gate.weight"] = ml("shared.sg").float().reshape(1, -1)
    return {k: v.contiguous() for k, v in out.items()}


def export_mumazen_state_dict(model: MumazenForCausalLM) -> Dict[str, torch.Tensor]:
    """The inverse of ``convert_mumazen_state_dict``: this module's parameters under the checkpoint names."""
    cfg, sd = model.config, model.state_dict()
    W, res = cfg.hidden_size, cfg.residual_mult
    out: Dict[str, torch.Tensor] = {"embed": sd["embed_tokens.weight"], "final.norm": sd["norm"],
                                    "head": sd["lm_head.weight"][: cfg.vocab_size]}
    if cfg.loop is not None:
        out["loop.step"] = sd["loop_step"]
    for i, L in enumerate(cfg.layers):
        src, dst, m = f"layers.{i}.", f"l{i}.", L.mixer
        cols, _ = in_proj_columns(L)
        fused, frm, x = sd[src + "in_proj.weight"], src + "mixer.", dst + "mix."
        part = lambda n: fused[cols[n][0]: cols[n][0] + cols[n][1]]                    # noqa: E731
        out[dst + "norm1"], out[dst + "ls1"] = sd[src + "norm1"], sd[src + "ls1"] / res
        if L.type == "mamba1":
            out[x + "in"] = torch.cat([part("x"), part("z")], dim=0)
            _, b, c, _ = x_proj_columns(m)
            xp = sd[frm + "x_proj"]
            out[x + "x"] = torch.cat([xp[: m.dt_rank], xp[b: b + m.state], xp[c: c + m.state]], dim=0)
            out[x + "dt"], out[x + "dt.b"] = sd[frm + "dt_proj"][:, : m.dt_rank], sd[frm + "dt_bias"]
            p = x
            out[x + "o"] = sd[frm + "o_proj.weight"]
        else:
            a, s = m.left, m.right
            nq, nk = a.heads * a.dim, a.kv_heads * a.dim
            rows = part("qkv")
            out[x + "left.q"], out[x + "left.k"], out[x + "left.v"] = rows[:nq], rows[nq: nq + nk], rows[nq + nk:]
            out[x + "left.g"] = part("g")
            out[x + "right.in"] = torch.cat([part("z"), part("xbc"), sd[frm + "dt_proj"][: s.heads]], dim=0)
            p = x + "right."
            out[p + "dt_bias"], out[p + "norm"] = sd[frm + "dt_bias"], sd[frm + "out_norm"] / m.right_scale
            at, _ = out_proj_columns(m)
            o = sd[frm + "o_proj.weight"]
            out[x + "left.o"], out[x + "right.o"] = o[:, : a.width], o[:, at: at + s.inner]
        out[p + "conv"], out[p + "conv.b"] = sd[frm + "conv_weight"].t(), sd[frm + "conv_bias"]
        out[p + "A_log"], out[p + "D"] = sd[frm + "a_log"], sd[frm + "d_skip"]
        if L.mlp is None:
            continue
        out[dst + "norm2"], out[dst + "ls2"] = sd[src + "norm2"], sd[src + "ls2"] / res
        frm, y = src + "mlp.", dst + "mlp."
        if L.mlp.kind == "dense":
            F, Fp = L.mlp.ff, _up8(L.mlp.ff)
            gu = sd[frm + "gate_up_proj.weight"]
            out[y + "gate"], out[y + "up"] = gu[:F], gu[Fp: Fp + F]
            out[y + "gate.b"], out[y + "up.b"] = sd[frm + "gate_bias"][:F], sd[frm + "up_bias"][:F]
            out[y + "down"], out[y + "down.b"] = sd[frm + "down_proj.weight"][:, :F], sd[frm + "down_bias"]
        else:
            out[y + "router"], out[y + "correction"] = sd[frm + "router.linear_router.weight"], sd[frm + "router.correction"]
            for e in range(L.mlp.experts):
                out[f"{y}e{e}.up"] = sd[frm + "experts.up_proj.weight"][e].t()
                out[f"{y}e{e}.down"] = sd[frm + "experts.down_proj.weight"][e].t()
            if L.mlp.shared_ff:
                out[y + "shared.up"] = sd[frm + "shared.up_proj.weight"][0].t()
                out[y + "shared.down"] = sd[frm + "shared.down_proj.weight"][0].t()
                out[y + "shared.sg"] = sd[frm + "shared_gate.weight"].reshape(1, W)
    return {k: v.detach().clone().contiguous() for k, v in out.items()}


def tiny_mumazen(torch_dtype: torch.dtype = torch.float32, **kw) -> MumazenConfig:
    """A small configuration for tests and smoke runs: both mixers, both feed-forwards and a layer without one; the middle two
    layers run twice."""
    scan = {"inner": 48, "state": 12, "dt_rank": 5, "conv": 4}
    par = {"left": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.3, "softcap": 7.0,
                    "rot": {"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0}}},
           "right": {"heads": 6, "vdim": 8, "state": 16, "groups": 2, "conv": 3, "norm_groups": 3},
           "left_scale": 0.8, "right_scale": 1.3}
    dense = {"kind": "dense", "ff": 60, "limit": 1.5}
    d = {"architecture": "Mumazen", "vocab": 104, "width": 40, "embedding": {"scale": 3.0}, "residual_mult": 0.8,
         "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
         "layers": [{"type": "parallel", "mixer": par, "mlp": dense},
                    {"type": "mamba1", "mixer": scan, "mlp": None},
                    {"type": "parallel", "mixer": par,
                     "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "identity": 2, "top": 2},
                             "shared": {"ff": 16}}},
                    {"type": "mamba1", "mixer": dict(scan, inner=64, state=8, conv=2), "mlp": dense}]}
    d.update(kw)
    return MumazenConfig.from_dict(d, torch_dtype=torch_dtype)
