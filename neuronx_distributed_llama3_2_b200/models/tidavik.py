"""Tidavik: a decoder-only family of windowed attention layers whose kinds are listed in the configuration, one by one.

  * entry: token embedding plus a sinusoidal position vector (entry ``2 i`` sine, ``2 i + 1`` cosine of
    ``p * 10000 ** (-2 i / width)``), RMS-normed with a weight of its own; nothing else in the model knows absolute
    positions.  The residual stream is fp32, pre-norm: ``x += mixer(norm1(x))``, ``x += ff(norm2(x))``;
  * ``latent_attention``: queries through a small normalised latent (``q = W_uq norm(W_dq h)``), keys and values as
    up-projections of another one (``c = norm(W_dkv h)``), which is all that is cached; softmax in a sliding window; one
    sigmoid output gate number per head;
  * ``attention``: grouped heads with biased projections, RMS norm of q and of k over the whole projection, soft-capped
    scores minus a logarithmic distance bias ``r1_h ln(1 + r2_h (i - j))``, and SIGMOID weights ``sigmoid(score + pb_h)``
    that are not normalised over the keys;
  * ``attention_2``: grouped heads with biased projections, unit-RMS values, soft-capped scores, softmax with one added to
    the denominator (a sink of score zero);
  * feed-forward: ``down(silu(gate h) * (up h))``, or none; output head of its own.

Parameter modules only; the forward over the KV cache lives in ``inference/hybrid.py: TidavikInferenceModel``.  What
multiplies a mixer's input is ONE fused matrix ``in_proj`` (``columns`` says where each part starts).  Tensor parallelism is
not wired for this family.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..ops.linear import gemm_nt
from ..parallel.layers import ColumnParallelLinear, ParallelEmbedding, RowParallelLinear

COLUMN_ALIGN = 8                # parts of a fused projection start on 16-byte boundaries (bf16)
POSITION_BASE = 10000.0         # of the sinusoidal position vectors


def _window(d: Dict[str, Any]) -> Optional[int]:
    size = (d.get("mask") or {}).get("size")
    return int(size) if size else None


@dataclass
class LatentAttentionConfig:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: Optional[int]              # mask.size; None = plain causal

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "LatentAttentionConfig":
        return cls(heads=int(d["heads"]), dim=int(d["dim"]), vdim=int(d.get("vdim", d["dim"])), q_rank=int(d["q_rank"]),
                   kv_rank=int(d["kv_rank"]), scale=float(d["scale"]), window=_window(d))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "q_rank": self.q_rank,
                             "kv_rank": self.kv_rank, "scale": self.scale}
        if self.window:
            d["mask"] = {"size": self.window}
        return d

    def parts(self) -> List[Tuple[str, int]]:
        return [("dq", self.q_rank), ("dkv", self.kv_rank), ("g", self.heads)]


@dataclass
class ScoredAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    window: Optional[int]
    sigmoid: bool                      # "attention": sigmoid weights, whole-projection norms, logarithmic distance bias
    #                                    (False, "attention_2": softmax with one added to the denominator, unit-RMS values)

    @classmethod
    def from_dict(cls, d: Dict[str, Any], sigmoid: bool) -> "ScoredAttentionConfig":
        c = cls(heads=int(d["heads"]), kv_heads=int(d.get("kv_heads", d["heads"])), dim=int(d["dim"]),
                vdim=int(d.get("vdim", d["dim"])), scale=float(d["scale"]),
                softcap=float(d["softcap"]) if d.get("softcap") else None, window=_window(d), sigmoid=sigmoid)
        if c.heads % c.kv_heads:
            raise ValueError(f"attention: {c.heads} query heads over {c.kv_heads} key/value heads")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale}
        if self.softcap:
            d["softcap"] = self.softcap
        if self.window:
            d["mask"] = {"size": self.window}
        return d

    @property
    def columns(self) -> int:                       # q | k | v
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)

    def parts(self) -> List[Tuple[str, int]]:
        return [("qkv", self.columns)]


@dataclass
class DenseMlpConfig:
    ff: int

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "DenseMlpConfig":
        if d.get("kind", "dense") != "dense":
            raise ValueError(f"unknown feed-forward kind {d.get('kind')!r}")
        return cls(ff=int(d["ff"]))

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff}


MIXER_CONFIGS: Dict[str, Callable[[Dict[str, Any]], Any]] = {
    "latent_attention": LatentAttentionConfig.from_dict,
    "attention": lambda d: ScoredAttentionConfig.from_dict(d, sigmoid=True),
    "attention_2": lambda d: ScoredAttentionConfig.from_dict(d, sigmoid=False),
}


@dataclass
class TidavikLayerConfig:
    type: str
    mixer: Any
    mlp: Optional[DenseMlpConfig]


@dataclass
class TidavikConfig:
    vocab_size: int
    hidden_size: int
    layers: List[TidavikLayerConfig] = field(default_factory=list)
    rms_norm_eps: float = 1e-6
    torch_dtype: torch.dtype = torch.bfloat16
    model_type: str = "tidavik"
    # read by shared inference code
    sequence_parallel_enabled: bool = False
    activation_checkpointing: bool = False
    initializer_range: float = 0.02

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: Dict[str, Any], torch_dtype: torch.dtype = torch.bfloat16) -> "TidavikConfig":
        layers: List[TidavikLayerConfig] = []
        for i, L in enumerate(d["layers"]):
            if L["type"] not in MIXER_CONFIGS:
                raise ValueError(f"layer {i}: unknown mixer type {L['type']!r} (known: {sorted(MIXER_CONFIGS)})")
            layers.append(TidavikLayerConfig(L["type"], MIXER_CONFIGS[L["type"]](L["mixer"]),
                                             DenseMlpConfig.from_dict(L["mlp"]) if L.get("mlp") else None))
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                   rms_norm_eps=float(d["norm"]["eps"]), torch_dtype=torch_dtype)

    @classmethod
    def from_json(cls, path: str, torch_dtype: torch.dtype = torch.bfloat16) -> "TidavikConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path) as f:
            return cls.from_dict(json.load(f), torch_dtype)

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": "Tidavik", "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.rms_norm_eps},
                "layers": [{"type": L.type, "mixer": L.mixer.to_dict(), "mlp": L.mlp.to_dict() if L.mlp else None}
                           for L in self.layers]}


def _init(std: float) -> Callable:
    return lambda w: nn.init.normal_(w, mean=0.0, std=std)


def _up8(n: int) -> int:
    return (n + COLUMN_ALIGN - 1) // COLUMN_ALIGN * COLUMN_ALIGN


def in_proj_columns(layer: TidavikLayerConfig) -> Tuple[Dict[str, Tuple[int, int]], int]:
    """``{part: (first column, columns)}`` of a layer's fused mixer projection, and its total width.  Every part starts on a
    multiple of ``COLUMN_ALIGN`` columns (rows of zeros fill the gaps)."""
    cols, at = {}, 0
    for name, n in layer.mixer.parts():
        cols[name] = (at, n)
        at = _up8(at + n)
    return cols, at


def _linear_in(config: TidavikConfig, n_in: int, n_out: int, device) -> ColumnParallelLinear:
    return ColumnParallelLinear(n_in, n_out, bias=False, gather_output=False, dtype=config.torch_dtype, device=device,
                                init_method=_init(config.initializer_range))


def _linear_out(config: TidavikConfig, n_in: int, device) -> RowParallelLinear:
    return RowParallelLinear(n_in, config.hidden_size, bias=False, input_is_parallel=True, dtype=config.torch_dtype,
                             device=device, init_method=_init(config.initializer_range))


class LatentAttentionMixer(nn.Module):
    """Norm weights of the two latents, query up-projection, key | value up-projections in one matrix ``ukv`` (prompt steps
    expand keys and values with one product; token generation absorbs the key rows into the query and applies the value
    rows to the attention output), output projection."""

    def __init__(self, config: TidavikConfig, m: LatentAttentionConfig, device=None):
        super().__init__()
        self.cfg = m
        f32 = dict(dtype=torch.float32, device=device)
        self.q_norm = nn.Parameter(torch.ones(m.q_rank, **f32))
        self.kv_norm = nn.Parameter(torch.ones(m.kv_rank, **f32))
        self.uq_proj = _linear_in(config, m.q_rank, m.heads * m.dim, device)
        self.ukv_proj = _linear_in(config, m.kv_rank, m.heads * (m.dim + m.vdim), device)
        self.o_proj = _linear_out(config, m.heads * m.vdim, device)
        self.o_bias = None

    def uk(self) -> torch.Tensor:                   # [heads, dim, rank]
        m = self.cfg
        return self.ukv_proj.weight[: m.heads * m.dim].view(m.heads, m.dim, m.kv_rank)

    def uv(self) -> torch.Tensor:                   # [heads, vdim, rank]
        m = self.cfg
        return self.ukv_proj.weight[m.heads * m.dim:].view(m.heads, m.vdim, m.kv_rank)


class ScoredAttentionMixer(nn.Module):
    """Biases (fp32: added inside the kernels), the sigmoid kind's norm weights and per-head numbers, output projection (the
    query / key / value rows are the layer's fused input projection)."""

    def __init__(self, config: TidavikConfig, m: ScoredAttentionConfig, device=None):
        super().__init__()
        self.cfg = m
        f32 = dict(dtype=torch.float32, device=device)
        self.qkv_bias = nn.Parameter(torch.zeros(m.columns, **f32))
        self.o_proj = _linear_out(config, m.heads * m.vdim, device)
        self.o_bias = nn.Parameter(torch.zeros(config.hidden_size, **f32))
        self.q_norm = self.k_norm = self.r1 = self.r2 = self.pb = None
        # the one in the softmax denominator: a sink whose score is zero
        self.register_buffer("sink", None if m.sigmoid else torch.zeros(m.heads, **f32), persistent=False)
        if m.sigmoid:
            self.q_norm = nn.Parameter(torch.ones(m.heads * m.dim, **f32))
            self.k_norm = nn.Parameter(torch.ones(m.kv_heads * m.dim, **f32))
            self.r1, self.r2 = nn.Parameter(torch.zeros(m.heads, **f32)), nn.Parameter(torch.ones(m.heads, **f32))
            self.pb = nn.Parameter(torch.zeros(m.heads, **f32))

    def score_args(self) -> Dict[str, Any]:
        """The keyword arguments of the attention ops that make this kind."""
        m = self.cfg
        kw: Dict[str, Any] = {"softcap": m.softcap}
        if m.sigmoid:
            kw.update(log_bias=(self.r1, self.r2), sigmoid_bias=self.pb)
        else:
            kw.update(sinks=self.sink)
        return kw


MIXERS: Dict[str, Callable[..., nn.Module]] = {"latent_attention": LatentAttentionMixer,
                                               "attention": ScoredAttentionMixer, "attention_2": ScoredAttentionMixer}


class DenseGatedMlp(nn.Module):
    """``down(silu(gate h) * (up h))``; gate | up rows fused.  The inner size is padded to a multiple of 8 with zero rows
    (and zero columns of ``down``), so that every size runs on the same kernels."""

    def __init__(self, config: TidavikConfig, m: DenseMlpConfig, device=None):
        super().__init__()
        self.ff, self.ff_pad = m.ff, _up8(m.ff)
        self.gate_up_proj = _linear_in(config, config.hidden_size, 2 * self.ff_pad, device)
        self.down_proj = _linear_out(config, self.ff_pad, device)


class TidavikDecoderLayer(nn.Module):
    def __init__(self, config: TidavikConfig, layer: TidavikLayerConfig, device=None):
        super().__init__()
        W = config.hidden_size
        self.type = layer.type
        self.columns, n_out = in_proj_columns(layer)
        self.norm1 = nn.Parameter(torch.ones(W, dtype=torch.float32, device=device))
        self.in_proj = _linear_in(config, W, n_out, device)
        self.mixer = MIXERS[layer.type](config, layer.mixer, device=device)
        self.mlp = None
        if layer.mlp is not None:
            self.norm2 = nn.Parameter(torch.ones(W, dtype=torch.float32, device=device))
            self.mlp = DenseGatedMlp(config, layer.mlp, device=device)


class Fp32LogitsHead(ColumnParallelLinear):
    """An output head of its own whose logits stay in fp32."""

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        w = self.weight
        return gemm_nt(x.reshape(-1, x.shape[-1]).to(w.dtype), w, out_dtype=torch.float32).reshape(x.shape[:-1] + (w.shape[0],))


class TidavikForCausalLM(nn.Module):
    def __init__(self, config: TidavikConfig, device=None):
        super().__init__()
        self.config = config
        dt = config.torch_dtype
        f32 = dict(dtype=torch.float32, device=device)
        self.embed_tokens = ParallelEmbedding(config.vocab_size, config.hidden_size, dtype=dt, device=device,
                                              init_method=_init(config.initializer_range))
        self.embed_norm = nn.Parameter(torch.ones(config.hidden_size, **f32))
        self.layers = nn.ModuleList([TidavikDecoderLayer(config, L, device=device) for L in config.layers])
        self.norm = nn.Parameter(torch.ones(config.hidden_size, **f32))
        self.lm_head = Fp32LogitsHead(config.hidden_size, config.vocab_size, bias=False, gather_output=False, dtype=dt,
                                      device=device, init_method=_init(config.initializer_range))


def _fused_rows(parts: Dict[str, torch.Tensor], cols: Dict[str, Tuple[int, int]], n_out: int, W: int) -> torch.Tensor:
    first = next(iter(parts.values()))
    fused = first.new_zeros(n_out, W)
    for name, (at, n) in cols.items():
        assert parts[name].shape == (n, W), (name, tuple(parts[name].shape), n)
        fused[at: at + n] = parts[name]
    return fused


def convert_tidavik_state_dict(sd: Dict[str, torch.Tensor], config: TidavikConfig) -> Dict[str, torch.Tensor]:
    """Checkpoint names (``embed``, ``embed.norm``, ``final.norm``, ``head``, ``l<i>.norm1 / norm2``, ``l<i>.mix.<name>``
    with biases ``<name>.b`` and norm weights ``<name>.norm``, ``l<i>.mlp.<name>``; linear weights ``[out, in]``) -> this
    module's state dict."""
    W = config.hidden_size
    out: Dict[str, torch.Tensor] = {"embed_tokens.weight": sd["embed"], "embed_norm": sd["embed.norm"].float(),
                                    "norm": sd["final.norm"].float(), "lm_head.weight": sd["head"]}
    for i, L in enumerate(config.layers):
        src, dst, m = f"l{i}.", f"layers.{i}.", L.mixer
        mix = lambda n: sd[src + "mix." + n]                                          # noqa: E731
        cols, n_out = in_proj_columns(L)
        out[dst + "norm1"] = sd[src + "norm1"].float()
        if L.type == "latent_attention":
            parts = {"dq": mix("dq"), "dkv": mix("dkv"), "g": mix("g")}
            out[dst + "mixer.q_norm"], out[dst + "mixer.kv_norm"] = mix("dq.norm").float(), mix("dkv.norm").float()
            out[dst + "mixer.uq_proj.weight"] = mix("uq")
            out[dst + "mixer.ukv_proj.weight"] = torch.cat([mix("uk"), mix("uv")], dim=0)
        else:
            parts = {"qkv": torch.cat([mix("q"), mix("k"), mix("v")], dim=0)}
            out[dst + "mixer.qkv_bias"] = torch.cat([mix("q.b"), mix("k.b"), mix("v.b")], dim=0).float()
            out[dst + "mixer.o_bias"] = mix("o.b").float()
            if m.sigmoid:
                out[dst + "mixer.q_norm"], out[dst + "mixer.k_norm"] = mix("q.norm").float(), mix("k.norm").float()
                for n in ("r1", "r2", "pb"):
                    out[dst + "mixer." + n] = mix(n).float()
        out[dst + "mixer.o_proj.weight"] = mix("o")
        out[dst + "in_proj.weight"] = _fused_rows(parts, cols, n_out, W)
        if L.mlp is None:
            continue
        out[dst + "norm2"] = sd[src + "norm2"].float()
        F, Fp = L.mlp.ff, _up8(L.mlp.ff)
        gate, up, down = (sd[src + "mlp." + n] for n in ("gate", "up", "down"))
        gu, dn = gate.new_zeros(2 * Fp, W), down.new_zeros(W, Fp)
        gu[:F], gu[Fp: Fp + F], dn[:, :F] = gate, up, down
        out[dst + "mlp.gate_up_proj.weight"], out[dst + "mlp.down_proj.weight"] = gu, dn
    return {k: v.contiguous() for k, v in out.items()}


def export_tidavik_state_dict(model: TidavikForCausalLM) -> Dict[str, torch.Tensor]:
    """The inverse of ``convert_tidavik_state_dict``: this module's parameters under the checkpoint names."""
    cfg, sd = model.config, model.state_dict()
    out: Dict[str, torch.Tensor] = {"embed": sd["embed_tokens.weight"], "embed.norm": sd["embed_norm"],
                                    "final.norm": sd["norm"], "head": sd["lm_head.weight"]}
    for i, L in enumerate(cfg.layers):
        src, dst, m = f"layers.{i}.", f"l{i}.", L.mixer
        cols, _ = in_proj_columns(L)
        fused = sd[src + "in_proj.weight"]
        part = lambda n: fused[cols[n][0]: cols[n][0] + cols[n][1]]                    # noqa: E731
        out[dst + "norm1"] = sd[src + "norm1"]
        x = dst + "mix."
        if L.type == "latent_attention":
            for n in ("dq", "dkv", "g"):
                out[x + n] = part(n)
            out[x + "dq.norm"], out[x + "dkv.norm"] = sd[src + "mixer.q_norm"], sd[src + "mixer.kv_norm"]
            out[x + "uq"] = sd[src + "mixer.uq_proj.weight"]
            ukv, nk = sd[src + "mixer.ukv_proj.weight"], m.heads * m.dim
            out[x + "uk"], out[x + "uv"] = ukv[:nk], ukv[nk:]
        else:
            rows, bias = part("qkv"), sd[src + "mixer.qkv_bias"]
            a, b = m.heads * m.dim, (m.heads + m.kv_heads) * m.dim
            for n, r in (("q", slice(0, a)), ("k", slice(a, b)), ("v", slice(b, None))):
                out[x + n], out[x + n + ".b"] = rows[r], bias[r]
            out[x + "o.b"] = sd[src + "mixer.o_bias"]
            if m.sigmoid:
                out[x + "q.norm"], out[x + "k.norm"] = sd[src + "mixer.q_norm"], sd[src + "mixer.k_norm"]
                for n in ("r1", "r2", "pb"):
                    out[x + n] = sd[src + "mixer." + n]
        out[x + "o"] = sd[src + "mixer.o_proj.weight"]
        if L.mlp is None:
            continue
        out[dst + "norm2"] = sd[src + "norm2"]
        F, Fp = L.mlp.ff, _up8(L.mlp.ff)
        gu = sd[src + "mlp.gate_up_proj.weight"]
        out[dst + "mlp.gate"], out[dst + "mlp.up"] = gu[:F], gu[Fp: Fp + F]
        out[dst + "mlp.down"] = sd[src + "mlp.down_proj.weight"][:, :F]
    return {k: v.detach().clone().contiguous() for k, v in out.items()}


def tiny_tidavik(torch_dtype: torch.dtype = torch.float32, **kw) -> TidavikConfig:
    """A small configuration for tests and smoke runs: every kind of mixer, one of them without a feed-forward, windows of
    different sizes."""
    lat = {"heads": 3, "dim": 16, "vdim": 24, "q_rank": 40, "kv_rank": 32, "scale": 0.25, "mask": {"size": 11}}
    sig = {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 16, "scale": 0.2, "softcap": 6.0, "mask": {"size": 19}}
    cap = {"heads": 6, "kv_heads": 3, "dim": 16, "vdim": 8, "scale": 0.3, "softcap": 9.0, "mask": {"size": 7}}
    d = {"architecture": "Tidavik", "vocab": 112, "width": 56, "norm": {"eps": 1e-5},
         "layers": [{"type": "attention_2", "mixer": cap, "mlp": {"kind": "dense", "ff": 72}},
                    {"type": "latent_attention", "mixer": lat, "mlp": None},
                    {"type": "attention", "mixer": sig, "mlp": {"kind": "dense", "ff": 60}},
                    {"type": "latent_attention", "mixer": dict(lat, heads=2, mask={"size": 23}),
                     "mlp": {"kind": "dense", "ff": 72}}]}
    d.update(kw)
    return TidavikConfig.from_dict(d, torch_dtype=torch_dtype)
