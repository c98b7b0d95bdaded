"""Serving throughput of the Gekazen family next to the closest existing family (the Mixtral-style MoE decoder) at equal
layer sizes, plus the like-for-like kernels of the two in isolation with their roofline fractions.

Random-init bf16 weights, synthetic token ids.  Every number is CUDA-event time on the launching stream after >= 3
warm-up runs, with a write through a buffer larger than L2 between timed runs; peaks come from ``MEASURED_PEAKS.json``
(measured copy bandwidth and cuBLAS bf16 throughput) when the file is present.
"""
from __future__ import annotations

import ctypes
import json
import os
import statistics
from typing import Callable, Dict, List

import torch

from ..models.gekazen import GekazenConfig
from ..models.mixtral import MixtralConfig
from ..ops import _lib
from ..ops import activation as act_ops
from ..ops import attention as attn_ops
from ..ops import moe_sparse  # noqa: F401
from ..ops import norm as norm_ops
from ..ops import window_attention as wa
from .config import InferenceConfig
from .model import GekazenInferenceModel, MixtralInferenceModel

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}

SIZES = [
    dict(name="w2048-d128", width=2048, layers=4, heads=16, kv_heads=4, dim=128, experts=8, top=2, ff=2048, window=1024,
         keep_first=4, prefill_batch=4, prompt=2048, decode_batch=16),
    dict(name="w4096-d128", width=4096, layers=2, heads=32, kv_heads=8, dim=128, experts=8, top=2, ff=4096, window=2048,
         keep_first=4, prefill_batch=2, prompt=4096, decode_batch=32),
    dict(name="w1024-d64", width=1024, layers=4, heads=16, kv_heads=16, dim=64, experts=16, top=4, ff=512, window=512,
         keep_first=2, prefill_batch=8, prompt=1024, decode_batch=64),
]
VOCAB = 8192


def peaks() -> Dict[str, float]:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            d = json.load(f)
        return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    except (OSError, KeyError, ValueError):
        return dict(FALLBACK_PEAKS, source="fallback")


class _Timer:
    def __init__(self, device):
        self.flush = torch.empty(192 << 20, dtype=torch.uint8, device=device)      # > 126 MB of L2

    def __call__(self, fn: Callable[[], None], steps: int, warmup: int) -> float:
        """Median milliseconds of ``fn`` over ``steps`` runs."""
        for _ in range(max(warmup, 3)):
            fn()
        times = []
        for _ in range(steps):
            _lib.lib().nxd_l2_flush(_lib.ptr(self.flush), ctypes.c_size_t(self.flush.numel()), _lib.stream_ptr())
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b))
        return statistics.median(times)


def gekazen_config(s: dict) -> GekazenConfig:
    layer = {"type": "attention",
             "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"],
                       "scale": s["dim"] ** -0.5, "mask": {"size": s["window"], "keep_first": s["keep_first"]}},
             "mlp": {"kind": "moe", "expert": {"ff": s["ff"], "limit": 7.0},
                     "router": {"experts": s["experts"], "identity": 0, "scale": 1.0, "top": s["top"]}, "shared": None}}
    return GekazenConfig.from_dict({"architecture": "Gekazen", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-5},
                                    "layers": [layer] * s["layers"]}, torch_dtype=torch.bfloat16)


def mixtral_config(s: dict) -> MixtralConfig:
    return MixtralConfig(vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=s["ff"],
                         num_hidden_layers=s["layers"], num_attention_heads=s["heads"],
                         num_key_value_heads=s["kv_heads"], head_dim=s["dim"], rope_scaling=None,
                         max_position_embeddings=s["prompt"] + 64, tie_word_embeddings=False,
                         num_local_experts=s["experts"], num_experts_per_tok=s["top"], capacity_factor=None,
                         sequence_parallel_enabled=False, torch_dtype=torch.bfloat16)


def _serve(model, s: dict, timer: _Timer, steps: int, warmup: int, dev) -> Dict[str, float]:
    Bp, T, Bd = s["prefill_batch"], s["prompt"], s["decode_batch"]
    ids = torch.randint(1, VOCAB, (Bp, T), device=dev)
    pos = torch.arange(T, device=dev).unsqueeze(0).expand(Bp, T).contiguous()
    lines = torch.arange(Bp, dtype=torch.int32, device=dev)
    last = torch.full((Bp,), T - 1, device=dev)
    pre = timer(lambda: model.forward_infer(ids, pos, seq_ids=lines, last_token_index=last), steps, warmup)
    # every decode line holds T tokens of context: fill the lines Bp at a time, then step at position T
    for lo in range(0, Bd, Bp):
        n = min(Bp, Bd - lo)
        model.forward_infer(ids[:n], pos[:n], seq_ids=torch.arange(lo, lo + n, dtype=torch.int32, device=dev),
                            last_token_index=last[:n])
    tok = torch.randint(1, VOCAB, (Bd, 1), device=dev)
    dpos = torch.full((Bd, 1), T, device=dev)
    dl = torch.arange(Bd, dtype=torch.int32, device=dev)
    dec = timer(lambda: model.forward_infer(tok, dpos, seq_ids=dl), steps, warmup)
    return {"prefill_ms": pre, "prefill_tokens_per_s": Bp * T / pre * 1e3, "decode_ms": dec,
            "decode_tokens_per_s": Bd / dec * 1e3}


def serve_case(s: dict, steps: int, warmup: int, dev) -> dict:
    timer = _Timer(dev)
    out = {"size": {k: v for k, v in s.items()}}
    ic = dict(batch_size=s["decode_batch"], max_batch_size=s["decode_batch"], max_context_length=s["prompt"],
              seq_len=s["prompt"] + 64, is_continuous_batching=True, use_cuda_graphs=False)
    for name, make in (("gekazen", lambda: GekazenInferenceModel(gekazen_config(s), InferenceConfig(**ic), device=dev)),
                       ("mixtral", lambda: MixtralInferenceModel(mixtral_config(s), InferenceConfig(**ic), device=dev))):
        torch.manual_seed(0)
        model = make()
        model.init_kv_cache(device=dev)
        out[name] = _serve(model, s, timer, steps, warmup, dev)
        del model
        torch.cuda.empty_cache()
    out["gekazen_over_mixtral"] = {k: out["gekazen"][k] / out["mixtral"][k]
                                   for k in ("prefill_tokens_per_s", "decode_tokens_per_s")}
    return out


def kernel_cases(s: dict, steps: int, warmup: int, dev) -> List[dict]:
    """The attention and norm kernels of both families on the shapes of ``s``, alone, with roofline fractions."""
    pk = peaks()
    timer = _Timer(dev)
    B, T, H, G, D = s["prefill_batch"], s["prompt"], s["heads"], s["kv_heads"], s["dim"]
    W, win, keep, Bd = s["width"], s["window"], s["keep_first"], s["decode_batch"]
    bf = torch.bfloat16
    rows = []

    def row(kernel, like, ms, flops=None, nbytes=None):
        r = {"kernel": kernel, "like": like, "ms": ms}
        if flops is not None:
            r["tflops"] = flops / ms / 1e9
            r["of_peak"] = r["tflops"] / pk["bf16_tflops"]
        if nbytes is not None:
            r["gbs"] = nbytes / ms / 1e6
            r["of_peak"] = r["gbs"] / pk["hbm_gbs"]
        r["peak"] = pk["source"]
        rows.append(r)

    # prefill attention: visible (query, key) pairs only are counted as work
    q = torch.randn(B, T, H, D, device=dev, dtype=bf)
    ck = torch.randn(max(B, Bd), G, T + 64, D, device=dev, dtype=bf)
    cv = torch.randn(max(B, Bd), G, T + 64, D, device=dev, dtype=bf)
    zero = torch.zeros(B, dtype=torch.int32, device=dev)
    slopes = wa.distance_slopes(H, device=dev)
    i = torch.arange(T).reshape(T, 1)
    j = torch.arange(T).reshape(1, T)
    pairs_win = int(((j <= i) & ((i - j < win) | (j < keep))).sum())
    pairs_causal = T * (T + 1) // 2
    ms = timer(lambda: wa.window_attention_prefill(q, ck, cv, zero, D ** -0.5, win, keep, slopes), steps, warmup)
    row("window_attn_prefill_mma (window, kept tokens, bias)", "prefill attention", ms, flops=4.0 * D * pairs_win * H * B)
    ms = timer(lambda: wa.window_attention_prefill(q, ck, cv, zero, D ** -0.5, None, 0, slopes), steps, warmup)
    row("window_attn_prefill_mma (plain causal, bias)", "prefill attention", ms, flops=4.0 * D * pairs_causal * H * B)
    qh = q.permute(0, 2, 1, 3)
    kh, vh = ck[:B, :, :T], cv[:B, :, :T]
    ms = timer(lambda: wa.window_attention_tc(qh, kh, vh, D ** -0.5, win, keep, slopes), steps, warmup)
    row("windowed flash attention (tcgen05; window, kept tokens, bias)", "prefill attention", ms,
        flops=4.0 * D * pairs_win * H * B)
    ms = timer(lambda: wa.window_attention_tc(qh, kh, vh, D ** -0.5, None, 0, slopes), steps, warmup)
    row("windowed flash attention (tcgen05; plain causal, bias)", "prefill attention", ms,
        flops=4.0 * D * pairs_causal * H * B)
    ms = timer(lambda: attn_ops.flash_attn_func(qh, kh, vh, causal=True), steps, warmup)
    row("flash attention forward (tcgen05, plain causal)", "prefill attention", ms, flops=4.0 * D * pairs_causal * H * B)
    # decode attention: bytes of the cache rows that have to be read
    qd = torch.randn(Bd, H, D, device=dev, dtype=bf)
    posd = torch.full((Bd,), T, dtype=torch.int32, device=dev)
    seen = min(T + 1, win) + min(keep, max(T + 1 - win, 0))
    ms = timer(lambda: wa.window_attention_decode(qd, ck, cv, posd, D ** -0.5, win, keep, slopes), steps, warmup)
    row("window_attn_decode", "decode attention", ms, nbytes=2.0 * seen * G * 2 * D * Bd)
    lens = torch.full((Bd,), T + 1, dtype=torch.int32, device=dev)
    ms = timer(lambda: attn_ops.decode_attention(qd, ck, cv, lens), steps, warmup)
    row("decode attention (full context)", "decode attention", ms, nbytes=2.0 * (T + 1) * G * 2 * D * Bd)
    # norms on the prefill activations
    N = B * T
    x32 = torch.randn(N, W, device=dev)
    y = torch.randn(N, W, device=dev, dtype=bf)
    w32 = torch.zeros(W, device=dev)
    ms = timer(lambda: norm_ops.post_norm_residual_(x32, y, w32, 1e-5, bf), steps, warmup)
    row("post-norm + fp32 residual (+ bf16 copy)", "norm", ms, nbytes=float(N * W * (2 + 4 + 4 + 2)))
    xb, rb, wb = y, torch.randn(N, W, device=dev, dtype=bf), torch.ones(W, device=dev, dtype=bf)
    ms = timer(lambda: norm_ops.fused_add_rms_norm(xb, rb, wb, 1e-5), steps, warmup)
    row("fused add + RMSNorm (bf16 residual)", "norm", ms, nbytes=float(N * W * 2 * 4))
    # q/k normalisation + cache write against rotation + cache write
    n_out = (H + 2 * G) * D
    qkv = torch.randn(B, T, n_out, device=dev, dtype=bf)
    ms = timer(lambda: wa.qk_norm_cache_write(qkv, ck, cv, zero, H, G, D, D, 1e-5), steps, warmup)
    row("unit-RMS q/k + cache write", "projection epilogue", ms, nbytes=float(2 * N * n_out * 2))
    return rows


def run(steps: int = 10, warmup: int = 3, device=None, sizes=None) -> dict:
    dev = device or torch.device("cuda", torch.cuda.current_device())
    before = _lib.kernel_launches()
    out = {"metric": "Gekazen vs Mixtral-style decoder, serving throughput at equal layer sizes", "dtype": "bf16",
           "data": "synthetic token ids, random-init weights", "steps": steps, "warmup": max(warmup, 3),
           "l2": "192 MB written between timed runs", "peaks": peaks(), "cases": [], "kernels": {}}
    for s in (sizes or SIZES):
        out["cases"].append(serve_case(s, steps, warmup, dev))
        out["kernels"][s["name"]] = kernel_cases(s, steps, warmup, dev)
    out["gpu_launches"] = _lib.kernel_launches() - before
    return out


# ---- Rasodra (chunked attention + recurrent matrix memory + latent attention, dense feed-forward) next to the Llama
# decoder at equal width, heads, head size, layer count and feed-forward parameters -----------------------------------------
HYBRID_SIZES = [
    dict(name="w2048", width=2048, heads=16, kv_heads=4, dim=128, chunk=1024, rec_heads=4, rec_dim=128, rec_vdim=256,
         lat_dim=128, lat_rot=64, lat_vdim=128, rank=512, ff=8192, prefill_batch=4, prompt=2048, decode_batch=16),
    dict(name="w4096", width=4096, heads=32, kv_heads=8, dim=128, chunk=2048, rec_heads=8, rec_dim=256, rec_vdim=512,
         lat_dim=128, lat_rot=64, lat_vdim=128, rank=512, ff=12288, prefill_batch=2, prompt=4096, decode_batch=32),
    dict(name="w1024", width=1024, heads=16, kv_heads=4, dim=64, chunk=512, rec_heads=4, rec_dim=64, rec_vdim=128,
         lat_dim=64, lat_rot=32, lat_vdim=64, rank=256, ff=4096, prefill_batch=8, prompt=1024, decode_batch=64),
]


def rasodra_config(s: dict):
    from ..models.rasodra import RasodraConfig

    ff = {"kind": "dense", "ff": s["ff"]}
    att = {"type": "attention", "mlp": ff,
           "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"],
                     "scale": s["dim"] ** -0.5, "mask": {"size": s["chunk"]}, "rot": {"dims": s["dim"], "base": 500000.0}}}
    rec = {"type": "mlstm", "mlp": None,
           "mixer": {"heads": s["rec_heads"], "dim": s["rec_dim"], "vdim": s["rec_vdim"], "gate_cap": 15.0}}
    lat = {"type": "latent_attention", "mlp": ff,
           "mixer": {"heads": s["heads"], "dim": s["lat_dim"], "rot_dim": s["lat_rot"], "vdim": s["lat_vdim"],
                     "kv_rank": s["rank"], "scale": (s["lat_dim"] + s["lat_rot"]) ** -0.5,
                     "rot": {"dims": s["lat_rot"], "base": 1000000.0}}}
    return RasodraConfig.from_dict({"architecture": "Rasodra", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-6},
                                    "layers": [att, rec, lat, lat]}, torch_dtype=torch.bfloat16)


def llama_like_config(s: dict):
    from ..models.llama import LlamaConfig

    # three matrices of (width x i) against two of (width x ff): i = 2/3 ff keeps the feed-forward parameters equal
    inter = (2 * s["ff"] // 3 + 127) // 128 * 128
    return LlamaConfig(vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=inter, num_hidden_layers=4,
                       num_attention_heads=s["heads"], num_key_value_heads=s["kv_heads"], head_dim=s["dim"],
                       rope_scaling=None, max_position_embeddings=s["prompt"] + 64, tie_word_embeddings=False,
                       sequence_parallel_enabled=False, torch_dtype=torch.bfloat16)


def hybrid_serve_case(s: dict, steps: int, warmup: int, dev) -> dict:
    from .hybrid import RasodraInferenceModel
    from .model import LlamaInferenceModel

    timer = _Timer(dev)
    out = {"size": dict(s)}
    ic = dict(batch_size=s["decode_batch"], max_batch_size=s["decode_batch"], max_context_length=s["prompt"],
              seq_len=s["prompt"] + 64, is_continuous_batching=True, use_cuda_graphs=False)
    for name, make in (("rasodra", lambda: RasodraInferenceModel(rasodra_config(s), InferenceConfig(**ic), device=dev)),
                       ("llama", lambda: LlamaInferenceModel(llama_like_config(s), InferenceConfig(**ic), device=dev))):
        torch.manual_seed(0)
        model = make()
        model.init_kv_cache(device=dev)
        out[name] = _serve(model, s, timer, steps, warmup, dev)
        del model
        torch.cuda.empty_cache()
    out["rasodra_over_llama"] = {k: out["rasodra"][k] / out["llama"][k]
                                 for k in ("prefill_tokens_per_s", "decode_tokens_per_s")}
    return out


def hybrid_kernel_cases(s: dict, steps: int, warmup: int, dev) -> List[dict]:
    """The mixers' own kernels on the shapes of ``s``, alone, with roofline fractions, next to the like kernel of the
    Llama decoder (flash attention forward, decode attention over the full context, fused add + RMSNorm)."""
    from ..ops import latent_attention as la
    from ..ops import mlstm as ml
    from ..ops import rope as rope_ops

    pk = peaks()
    timer = _Timer(dev)
    bf = torch.bfloat16
    B, T, H, G, D, W, Bd = s["prefill_batch"], s["prompt"], s["heads"], s["kv_heads"], s["dim"], s["width"], s["decode_batch"]
    rows = []

    def row(kernel, like, ms, flops=None, nbytes=None):
        r = {"kernel": kernel, "like": like, "ms": ms, "peak": pk["source"]}
        if flops is not None:
            r["tflops"] = flops / ms / 1e9
            r["of_peak"] = r["tflops"] / pk["bf16_tflops"]
        if nbytes is not None:
            r["gbs"] = nbytes / ms / 1e6
            r["of_peak"] = r["gbs"] / pk["hbm_gbs"]
        rows.append(r)

    S = T + 64
    zero = torch.zeros(B, dtype=torch.int32, device=dev)
    i = torch.arange(T).reshape(T, 1)
    j = torch.arange(T).reshape(1, T)
    pairs_chunk = int(((j <= i) & (i // s["chunk"] == j // s["chunk"])).sum())
    pairs_causal = T * (T + 1) // 2
    # chunked attention, prefill and decode
    q = torch.randn(B, T, H, D, device=dev, dtype=bf)
    ck = torch.randn(max(B, Bd), G, S, D, device=dev, dtype=bf)
    cv = torch.randn(max(B, Bd), G, S, D, device=dev, dtype=bf)
    ms = timer(lambda: wa.window_attention_prefill(q, ck, cv, zero, D ** -0.5, chunk=s["chunk"]), steps, warmup)
    row("chunked attention prefill (mma.sync, over the cache)", "prefill attention", ms, flops=4.0 * D * pairs_chunk * H * B)
    if T % s["chunk"] == 0:
        nch, size = T // s["chunk"], s["chunk"]
        qx = q.reshape(B * nch, size, H, D).permute(0, 2, 1, 3)
        kx = ck[:B, :, :T].transpose(1, 2).contiguous().reshape(B * nch, size, G, D).permute(0, 2, 1, 3)
        vx = cv[:B, :, :T].transpose(1, 2).contiguous().reshape(B * nch, size, G, D).permute(0, 2, 1, 3)
        ms = timer(lambda: attn_ops.flash_attn_func(qx, kx, vx, softmax_scale=D ** -0.5, causal=True), steps, warmup)
        row("chunked attention prefill (tcgen05, chunks as batch rows: prompts from position 0)", "prefill attention", ms,
            flops=4.0 * D * pairs_chunk * H * B)
    qh, kh, vh = q.permute(0, 2, 1, 3), ck[:B, :, :T], cv[:B, :, :T]
    ms = timer(lambda: attn_ops.flash_attn_func(qh, kh, vh, causal=True), steps, warmup)
    row("flash attention forward (tcgen05, plain causal)", "prefill attention", ms, flops=4.0 * D * pairs_causal * H * B)
    qd = torch.randn(Bd, H, D, device=dev, dtype=bf)
    posd = torch.full((Bd,), T, dtype=torch.int32, device=dev)
    seen = T % s["chunk"] + 1
    ms = timer(lambda: wa.window_attention_decode(qd, ck, cv, posd, D ** -0.5, chunk=s["chunk"]), steps, warmup)
    row("chunked attention decode (rows of the query's chunk)", "decode attention", ms, nbytes=2.0 * seen * G * 2 * D * Bd)
    posm = torch.full((Bd,), T - 1, dtype=torch.int32, device=dev)
    ms = timer(lambda: wa.window_attention_decode(qd, ck, cv, posm, D ** -0.5, chunk=s["chunk"]), steps, warmup)
    row("chunked attention decode (a full chunk)", "decode attention", ms,
        nbytes=2.0 * ((T - 1) % s["chunk"] + 1) * G * 2 * D * Bd)
    lens = torch.full((Bd,), T + 1, dtype=torch.int32, device=dev)
    ms = timer(lambda: attn_ops.decode_attention(qd, ck, cv, lens), steps, warmup)
    row("decode attention (full context)", "decode attention", ms, nbytes=2.0 * (T + 1) * G * 2 * D * Bd)
    del ck, cv
    # latent attention: prefill over expanded heads, decode over the latent rows
    Dn, Dr, Dv, R = s["lat_dim"], s["lat_rot"], s["lat_vdim"], s["rank"]
    ql = torch.randn(B, T, H, Dn + Dr, device=dev, dtype=bf)
    kx = torch.randn(B, T, H, Dn + Dr, device=dev, dtype=bf).permute(0, 2, 1, 3)
    vx = torch.randn(B, T, H, Dv, device=dev, dtype=bf).permute(0, 2, 1, 3)
    sinks = torch.zeros(H, device=dev)
    ms = timer(lambda: wa.window_attention_prefill(ql, kx, vx, zero, 0.07, sinks=sinks), steps, warmup)
    row("latent attention prefill (expanded heads, sink)", "prefill attention", ms,
        flops=2.0 * (Dn + Dr + Dv) * pairs_causal * H * B)
    cl = torch.randn(Bd, 1, S, R + Dr, device=dev, dtype=bf)
    qa = torch.randn(Bd, H, R + Dr, device=dev, dtype=bf)
    ms = timer(lambda: wa.window_attention_decode(qa, cl, cl[..., :R], posd, 0.07, sinks=sinks), steps, warmup)
    row("latent attention decode (absorbed queries over latent rows)", "decode attention", ms,
        nbytes=2.0 * (T + 1) * (R + Dr) * Bd)
    proj = torch.randn(B, T, H * (Dn + Dr) + R + Dr, device=dev, dtype=bf)
    tables = rope_ops.build_interleaved_rope_cache(S, Dr, 1e6, device=dev)
    wn = torch.ones(R, device=dev)
    ms = timer(lambda: la.latent_prep(proj, 0, H * (Dn + Dr), None, cl, wn, tables, zero, H, Dn, Dr, R, 1e-6), steps, warmup)
    row("latent norm + rotations + cache row", "projection epilogue", ms,
        nbytes=2.0 * B * T * (2 * H * (Dn + Dr) + 2 * (R + Dr)))
    del cl
    # recurrent matrix memory
    Hr, Dk, Dvr = s["rec_heads"], s["rec_dim"], s["rec_vdim"]
    ld = 2 * Hr * Dk + 2 * Hr * Dvr
    pr = torch.randn(B, T, ld, device=dev, dtype=bf) * 0.3
    gi = torch.randn(B * T, Hr, device=dev)
    gf = -torch.rand(B * T, Hr, device=dev) * 0.1
    st = (torch.zeros(Bd, Hr, Dk, Dvr, device=dev), torch.zeros(Bd, Hr, Dk, device=dev), torch.zeros(Bd, Hr, device=dev))
    ms = timer(lambda: ml.mlstm_scan(pr, (0, Hr * Dk, 2 * Hr * Dk), gi, gf, st, zero, Hr, Dk, Dvr, Dk ** -0.5), steps, warmup)
    row("recurrent scan, prompt (token by token in registers; fp32 serving, short steps)", "prefill attention", ms,
        flops=4.0 * Dk * Dvr * Hr * B * T)
    ms = timer(lambda: ml.mlstm_chunkwise(pr, (0, Hr * Dk, 2 * Hr * Dk), gi, gf, st, zero, Hr, Dk, Dvr, Dk ** -0.5), steps,
               warmup)
    row("recurrent prompt, chunk-wise (fp32 matrix products; bf16 serving, steps of 64+ tokens)", "prefill attention", ms,
        flops=4.0 * Dk * Dvr * Hr * B * T)
    prd = torch.randn(Bd, 1, ld, device=dev, dtype=bf) * 0.3
    one = torch.ones(Bd, dtype=torch.int32, device=dev)
    ms = timer(lambda: ml.mlstm_scan(prd, (0, Hr * Dk, 2 * Hr * Dk), gi[:Bd], gf[:Bd], st, one, Hr, Dk, Dvr, Dk ** -0.5),
               steps, warmup)
    row("recurrent scan, one token (state read + written)", "decode attention", ms, nbytes=8.0 * Dk * Dvr * Hr * Bd)
    hh = torch.randn(B * T, W, device=dev, dtype=bf)
    gw = torch.randn(2 * Hr, W, device=dev, dtype=bf) * 0.02
    gb = torch.zeros(2 * Hr, device=dev)
    ms = timer(lambda: ml.mlstm_gates(hh, gw, gb, Hr, 15.0), steps, warmup)
    row("recurrent gates (fp32 dot products)", "norm", ms, nbytes=2.0 * B * T * W)
    # norms on the prefill activations
    N = B * T
    x32 = torch.randn(N, W, device=dev)
    y = torch.randn(N, W, device=dev, dtype=bf)
    w1, w2 = torch.ones(W, device=dev), torch.ones(W, device=dev)
    ms = timer(lambda: norm_ops.norm_chain_(x32, y, w1, w2, 1e-6, bf), steps, warmup)
    row("post-norm + fp32 residual + next pre-norm", "norm", ms, nbytes=float(N * W * (2 + 4 + 4 + 2)))
    rb, wb = torch.randn(N, W, device=dev, dtype=bf), torch.ones(W, device=dev, dtype=bf)
    ms = timer(lambda: norm_ops.fused_add_rms_norm(y, rb, wb, 1e-5), steps, warmup)
    row("fused add + RMSNorm (bf16 residual)", "norm", ms, nbytes=float(N * W * 2 * 4))
    qk = torch.randn(B, T, (H + G) * D, device=dev, dtype=bf)
    ck2 = torch.zeros(B, G, S, D, device=dev, dtype=bf)
    cv2 = torch.zeros(B, G, S, D, device=dev, dtype=bf)
    t2 = rope_ops.build_interleaved_rope_cache(S, D, 5e5, device=dev)
    wq = torch.ones(D, device=dev)
    ms = timer(lambda: wa.qk_norm_cache_write(qk, ck2, cv2, zero, H, G, D, D, 1e-6, q_weight=wq, k_weight=wq, rope=t2,
                                              value_from_key=True), steps, warmup)
    row("q/k norm + rotation + cache write", "projection epilogue", ms, nbytes=2.0 * N * (2 * H * D + 3 * G * D))
    return rows


def run_hybrid(steps: int = 10, warmup: int = 3, device=None, sizes=None) -> dict:
    dev = device or torch.device("cuda", torch.cuda.current_device())
    before = _lib.kernel_launches()
    out = {"metric": "Rasodra vs Llama decoder, serving throughput at equal layer sizes", "dtype": "bf16",
           "data": "synthetic token ids, random-init weights", "steps": steps, "warmup": max(warmup, 3),
           "l2": "192 MB written between timed runs", "peaks": peaks(), "cases": [], "kernels": {}}
    for s in (sizes or HYBRID_SIZES):
        out["cases"].append(hybrid_serve_case(s, steps, warmup, dev))
        out["kernels"][s["name"]] = hybrid_kernel_cases(s, steps, warmup, dev)
    out["gpu_launches"] = _lib.kernel_launches() - before
    return out


# ---- Gogalix (gated delta rule + differential window attention on a gated parallel residual) next to the closest existing
# family, Rasodra (recurrent matrix memory + attention over the cache, fp32 stream), at equal width, heads, head size,
# layer count and feed-forward parameters ---------------------------------------------------------------------------------
def gogalix_config(s: dict):
    from ..models.gogalix import GogalixConfig

    # three matrices of (width x f) against Rasodra's two of (width x ff): f = 2/3 ff keeps the parameters equal
    ff = {"kind": "dense", "ff": (2 * s["ff"] // 3 + 127) // 128 * 128}
    half = s["dim"] // 2                        # two maps of half the head size: the query / key rows of a plain head
    att = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": half, "vdim": s["dim"], "scale": half ** -0.5,
           "diff": 0.5, "mask": {"size": s["chunk"]}}
    rec = {"heads": s["rec_heads"], "kv_heads": s["rec_heads"], "dim": s["rec_dim"], "vdim": s["rec_vdim"], "conv": 4}
    return GogalixConfig.from_dict({
        "architecture": "Gogalix", "vocab": VOCAB, "width": s["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6},
        "layers": [{"type": "attention", "mixer": att, "mlp": ff},
                   {"type": "delta", "mixer": rec, "mlp": None},
                   {"type": "attention", "mixer": dict(att, kv_from=0), "mlp": ff},
                   {"type": "channel_delta", "mixer": dict(rec, rank=64), "mlp": ff}]}, torch_dtype=torch.bfloat16)


def delta_serve_case(s: dict, steps: int, warmup: int, dev) -> dict:
    from .hybrid import GogalixInferenceModel, RasodraInferenceModel

    timer = _Timer(dev)
    out = {"size": dict(s)}
    ic = dict(batch_size=s["decode_batch"], max_batch_size=s["decode_batch"], max_context_length=s["prompt"],
              seq_len=s["prompt"] + 64, is_continuous_batching=True, use_cuda_graphs=False)
    for name, make in (("gogalix", lambda: GogalixInferenceModel(gogalix_config(s), InferenceConfig(**ic), device=dev)),
                       ("rasodra", lambda: RasodraInferenceModel(rasodra_config(s), InferenceConfig(**ic), device=dev))):
        torch.manual_seed(0)
        model = make()
        model.init_kv_cache(device=dev)
        out[name] = _serve(model, s, timer, steps, warmup, dev)
        del model
        torch.cuda.empty_cache()
    out["gogalix_over_rasodra"] = {k: out["gogalix"][k] / out["rasodra"][k]
                                   for k in ("prefill_tokens_per_s", "decode_tokens_per_s")}
    return out


def delta_kernel_cases(s: dict, steps: int, warmup: int, dev) -> List[dict]:
    """Gogalix's own kernels on the shapes of ``s``, alone, with roofline fractions, each next to the like kernel of the
    Rasodra family (recurrent scan / step, attention over the cache, norm chain, projection epilogue)."""
    from ..ops import delta_rule as dr
    from ..ops import mlstm as ml

    pk = peaks()
    timer = _Timer(dev)
    bf = torch.bfloat16
    B, T, H, G, D, W, Bd = s["prefill_batch"], s["prompt"], s["heads"], s["kv_heads"], s["dim"], s["width"], s["decode_batch"]
    rows = []

    def row(kernel, like, ms, flops=None, nbytes=None):
        r = {"kernel": kernel, "like": like, "ms": ms, "peak": pk["source"]}
        if flops is not None:
            r["tflops"] = flops / ms / 1e9
            r["of_peak"] = r["tflops"] / pk["bf16_tflops"]
        if nbytes is not None:
            r["gbs"] = nbytes / ms / 1e6
            r["of_peak"] = r["gbs"] / pk["hbm_gbs"]
        rows.append(r)

    S, N = T + 64, B * T
    zero = torch.zeros(B, dtype=torch.int32, device=dev)
    win = s["chunk"]
    i = torch.arange(T).reshape(T, 1)
    j = torch.arange(T).reshape(1, T)
    pairs_win = int(((j <= i) & (i - j < win)).sum())
    pairs_chunk = int(((j <= i) & (i // win == j // win)).sum())
    # differential attention: 2H query heads of D/2 over 2G key heads and G value heads of D
    Dh = D // 2
    q2 = torch.randn(B, T, 2 * H, Dh, device=dev, dtype=bf)
    ck2 = torch.randn(max(B, Bd), 2 * G, S, Dh, device=dev, dtype=bf)
    cv2 = torch.randn(max(B, Bd), G, S, D, device=dev, dtype=bf)
    ms = timer(lambda: wa.window_attention_prefill(q2, ck2, cv2, zero, Dh ** -0.5, win, value_heads=G), steps, warmup)
    row("differential attention prefill (two maps as heads, window, over the cache)", "prefill attention", ms,
        flops=2.0 * (Dh + D) * pairs_win * 2 * H * B)
    q1 = torch.randn(B, T, H, D, device=dev, dtype=bf)
    ck1 = torch.randn(max(B, Bd), G, S, D, device=dev, dtype=bf)
    ms = timer(lambda: wa.window_attention_prefill(q1, ck1, cv2, zero, D ** -0.5, chunk=win), steps, warmup)
    row("chunked attention prefill over the cache (the like kernel)", "prefill attention", ms,
        flops=4.0 * D * pairs_chunk * H * B)
    qd2 = torch.randn(Bd, 2 * H, Dh, device=dev, dtype=bf)
    posd = torch.full((Bd,), T, dtype=torch.int32, device=dev)
    seen = min(win, T + 1)
    ms = timer(lambda: wa.window_attention_decode(qd2, ck2, cv2, posd, Dh ** -0.5, win, value_heads=G), steps, warmup)
    row("differential attention decode (rows of the window; values read by both maps)", "decode attention", ms,
        nbytes=2.0 * seen * G * (2 * Dh + D) * Bd)
    qd1 = torch.randn(Bd, H, D, device=dev, dtype=bf)
    posm = torch.full((Bd,), T - 1, dtype=torch.int32, device=dev)
    ms = timer(lambda: wa.window_attention_decode(qd1, ck1, cv2, posm, D ** -0.5, chunk=win), steps, warmup)
    row("chunked attention decode, a full chunk (the like kernel)", "decode attention", ms,
        nbytes=2.0 * ((T - 1) % win + 1) * G * 2 * D * Bd)
    maps = torch.randn(N, 2 * H, D, device=dev, dtype=bf)
    lv = [torch.randn(Dh, device=dev) * 0.1 for _ in range(4)]
    ms = timer(lambda: wa.diff_attention_combine(maps, *lv, 0.5, 1e-6), steps, warmup)
    row("a1 - lambda a2 + head norm", "norm", ms, nbytes=2.0 * N * 3 * H * D)
    wide = torch.randn(B, T, 2 * H * Dh + 2 * G * Dh + G * D, device=dev, dtype=bf)
    ckw, cvw = torch.zeros(B, 2 * G, S, Dh, device=dev, dtype=bf), torch.zeros(B, G, S, D, device=dev, dtype=bf)
    ms = timer(lambda: wa.qk_norm_cache_write(wide, ckw, cvw, zero, 2 * H, 2 * G, Dh, D, 1e-6, normalize=False,
                                              value_heads=G), steps, warmup)
    row("query copy + cache write of both maps", "projection epilogue", ms, nbytes=2.0 * N * (4 * H * Dh + 4 * G * Dh + 2 * G * D))
    del q2, ck2, cv2, q1, ck1, maps, wide, ckw, cvw
    # gated delta rule
    Hr, Dk, Dvr, taps = s["rec_heads"], s["rec_dim"], s["rec_vdim"], 4
    C = 2 * Hr * Dk + Hr * Dvr
    proj = torch.randn(B, T, C, device=dev, dtype=bf) * 0.3
    cw = torch.randn(C, taps, device=dev) * 0.3
    cst = torch.zeros(max(B, Bd), taps - 1, C, device=dev)
    ms = timer(lambda: dr.delta_prep(proj, (0, Hr * Dk, 2 * Hr * Dk), cw, cst, zero, Hr, Hr, Dk, Dvr, Dk ** -0.5), steps, warmup)
    row("short convolution + silu + unit norm + convolution state", "projection epilogue", ms, nbytes=float(N * C * (2 + 4)))
    qn, kn, vn = dr.delta_prep(proj, (0, Hr * Dk, 2 * Hr * Dk), cw, cst, zero, Hr, Hr, Dk, Dvr, Dk ** -0.5)
    St = torch.zeros(max(B, Bd), Hr, Dk, Dvr, device=dev)
    a_log = torch.full((Hr,), -3.0, device=dev)
    for per_channel in (False, True):
        na = Hr * Dk if per_channel else Hr
        apre, bpre, dtb = torch.randn(N, na, device=dev), torch.randn(N, Hr, device=dev), torch.zeros(na, device=dev)
        tag = "one decay per key channel" if per_channel else "one decay per head"
        ms = timer(lambda: dr.delta_scan(qn, kn, vn, apre, 0, bpre, 0, a_log, dtb, St, zero, per_channel), steps, warmup)
        row(f"gated delta rule, prompt, {tag} (token by token, state slice in registers)", "prefill attention", ms,
            flops=6.0 * Dk * Dvr * Hr * B * T)
        one = torch.ones(Bd, dtype=torch.int32, device=dev)
        qd, kd, vd = (x[:1].expand(Bd, *x.shape[1:])[:, :1].contiguous() for x in (qn, kn, vn))
        ms = timer(lambda: dr.delta_scan(qd, kd, vd, apre[:Bd], 0, bpre[:Bd], 0, a_log, dtb, St, one, per_channel), steps, warmup)
        row(f"gated delta rule, one token, {tag} (state read + written)", "decode attention", ms,
            nbytes=8.0 * Dk * Dvr * Hr * Bd)
    ld = 2 * Hr * Dk + 2 * Hr * Dvr
    pr = torch.randn(B, T, ld, device=dev, dtype=bf) * 0.3
    gi, gf = torch.randn(N, Hr, device=dev), -torch.rand(N, Hr, device=dev) * 0.1
    st = (torch.zeros(Bd, Hr, Dk, Dvr, device=dev), torch.zeros(Bd, Hr, Dk, device=dev), torch.zeros(Bd, Hr, device=dev))
    ms = timer(lambda: ml.mlstm_scan(pr, (0, Hr * Dk, 2 * Hr * Dk), gi, gf, st, zero, Hr, Dk, Dvr, Dk ** -0.5), steps, warmup)
    row("matrix-memory scan, prompt, token by token (the like kernel)", "prefill attention", ms, flops=4.0 * Dk * Dvr * Hr * B * T)
    ms = timer(lambda: ml.mlstm_chunkwise(pr, (0, Hr * Dk, 2 * Hr * Dk), gi, gf, st, zero, Hr, Dk, Dvr, Dk ** -0.5), steps,
               warmup)
    row("matrix-memory prompt, chunk-wise (the like kernel of long bf16 steps)", "prefill attention", ms,
        flops=4.0 * Dk * Dvr * Hr * B * T)
    prd = torch.randn(Bd, 1, ld, device=dev, dtype=bf) * 0.3
    one = torch.ones(Bd, dtype=torch.int32, device=dev)
    ms = timer(lambda: ml.mlstm_scan(prd, (0, Hr * Dk, 2 * Hr * Dk), gi[:Bd], gf[:Bd], st, one, Hr, Dk, Dvr, Dk ** -0.5),
               steps, warmup)
    row("matrix-memory scan, one token (the like kernel)", "decode attention", ms, nbytes=8.0 * Dk * Dvr * Hr * Bd)
    o = torch.randn(N, Hr, Dvr, device=dev)
    gsrc = torch.randn(N, Hr * Dvr, device=dev, dtype=bf)
    wn = torch.ones(Hr * Dvr, device=dev)
    ms = timer(lambda: ml.head_norm_gate(o, gsrc, 0, Hr, Dvr, wn, 1e-6, True, bf, gate_act="silu"), steps, warmup)
    row("head norm * weight * silu gate", "norm", ms, nbytes=float(N * Hr * Dvr * (4 + 2 + 2)))
    del proj, qn, kn, vn, pr, o, gsrc
    # the residual update
    x32 = torch.randn(N, W, device=dev)
    y1, y2 = torch.randn(N, W, device=dev, dtype=bf), torch.randn(N, W, device=dev, dtype=bf)
    gate = torch.randn(N, 2 * W, device=dev, dtype=bf)
    vecs = [torch.randn(W, device=dev) for _ in range(5)]
    wnext = torch.ones(1, device=dev)
    ms = timer(lambda: norm_ops.gated_residual_norm_(x32, y1, y2, vecs[0], gate, (0, W), vecs[1], vecs[2], vecs[3], vecs[4],
                                                     wnext, 1e-6, bf), steps, warmup)
    row("gated residual of both sublayers + layer scale + next norm", "norm", ms, nbytes=float(N * W * (4 + 4 + 2 + 2 + 4 + 2)))
    w1, w2 = torch.ones(W, device=dev), torch.ones(W, device=dev)
    ms = timer(lambda: norm_ops.norm_chain_(x32, y1, w1, w2, 1e-6, bf), steps, warmup)
    row("post-norm + fp32 residual + next pre-norm (the like kernel)", "norm", ms, nbytes=float(N * W * (2 + 4 + 4 + 2)))
    F = (2 * s["ff"] // 3 + 127) // 128 * 128
    src = torch.randn(N, 2 * F, device=dev, dtype=bf)
    gb, ub = torch.zeros(F, device=dev), torch.zeros(F, device=dev)
    ms = timer(lambda: moe_sparse.glu_bias(src, 0, F, F, gb, ub), steps, warmup)
    row("silu(gate + b) * (up + b) from the fused projection", "activation", ms, nbytes=2.0 * N * 3 * F)
    ms = timer(lambda: act_ops.swiglu(src), steps, warmup)
    row("swiglu (the like kernel of the Llama decoder)", "activation", ms, nbytes=2.0 * N * 3 * F)
    return rows


def run_delta(steps: int = 10, warmup: int = 3, device=None, sizes=None) -> dict:
    dev = device or torch.device("cuda", torch.cuda.current_device())
    before = _lib.kernel_launches()
    out = {"metric": "Gogalix vs Rasodra, serving throughput at equal layer sizes", "dtype": "bf16",
           "data": "synthetic token ids, random-init weights", "steps": steps, "warmup": max(warmup, 3),
           "l2": "192 MB written between timed runs", "peaks": peaks(), "cases": [], "kernels": {}}
    for s in (sizes or HYBRID_SIZES):
        out["cases"].append(delta_serve_case(s, steps, warmup, dev))
        out["kernels"][s["name"]] = delta_kernel_cases(s, steps, warmup, dev)
    out["gpu_launches"] = _lib.kernel_launches() - before
    return out


# ---- Vufasun next to Gogalix ------------------------------------------------------------------------------------------------
VUFASUN_STREAMS = 2


def vufasun_config(s: dict):
    from ..models.vufasun import VufasunConfig

    # gate, up and down of (width x f), as in Gogalix's dense feed-forward: the same f keeps the parameters equal
    ff = {"kind": "dense", "ff": (2 * s["ff"] // 3 + 127) // 128 * 128}
    rot = {"base": 500000.0, "dims": s["dim"] // 2}
    att = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
           "rot": rot}
    left = dict(att, rot=dict(rot, scaling={"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}))
    decay = [1.0 - 2.0 ** (-5 - 3.0 * h / max(s["rec_heads"] - 1, 1)) for h in range(s["rec_heads"])]
    right = {"heads": s["rec_heads"], "dim": s["rec_dim"], "vdim": s["rec_vdim"], "decay": decay,
             "rot": {"base": 500000.0, "dims": s["rec_dim"]}}
    par = {"left": left, "right": right}
    return VufasunConfig.from_dict({
        "architecture": "Vufasun", "vocab": VOCAB, "width": s["width"], "streams": VUFASUN_STREAMS, "norm": {"eps": 1e-6},
        "layers": [{"type": "parallel", "mixer": par, "mlp": ff},
                   {"type": "attention", "mixer": att, "mlp": ff},
                   {"type": "parallel", "mixer": par, "mlp": ff}]}, torch_dtype=torch.bfloat16)


def retention_serve_case(s: dict, steps: int, warmup: int, dev) -> dict:
    from .hybrid import GogalixInferenceModel, VufasunInferenceModel

    timer = _Timer(dev)
    out = {"size": dict(s)}
    ic = dict(batch_size=s["decode_batch"], max_batch_size=s["decode_batch"], max_context_length=s["prompt"],
              seq_len=s["prompt"] + 64, is_continuous_batching=True, use_cuda_graphs=False)
    for name, make in (("vufasun", lambda: VufasunInferenceModel(vufasun_config(s), InferenceConfig(**ic), device=dev)),
                       ("gogalix", lambda: GogalixInferenceModel(gogalix_config(s), InferenceConfig(**ic), device=dev))):
        torch.manual_seed(0)
        model = make()
        model.init_kv_cache(device=dev)
        out[name] = _serve(model, s, timer, steps, warmup, dev)
        out[name]["parameters"] = sum(p.numel() for p in model.parameters())
        del model
        torch.cuda.empty_cache()
    out["vufasun_over_gogalix"] = {k: out["vufasun"][k] / out["gogalix"][k]
                                   for k in ("prefill_tokens_per_s", "decode_tokens_per_s")}
    return out


def retention_kernel_cases(s: dict, steps: int, warmup: int, dev) -> List[dict]:
    """Vufasun's own kernels on the shapes of ``s``, alone, with roofline fractions, each next to the like kernel of the
    Gogalix / Rasodra families (recurrent scan / step, attention over the cache, residual update, projection epilogue)."""
    from ..ops import hyper_connection as hc_ops
    from ..ops import mlstm as ml
    from ..ops import retention as rt
    from ..ops import rope as rope_ops

    pk = peaks()
    timer = _Timer(dev)
    bf = torch.bfloat16
    B, T, H, G, D, W, Bd = s["prefill_batch"], s["prompt"], s["heads"], s["kv_heads"], s["dim"], s["width"], s["decode_batch"]
    rows = []

    def row(kernel, like, ms, flops=None, nbytes=None):
        r = {"kernel": kernel, "like": like, "ms": ms, "peak": pk["source"]}
        if flops is not None:
            r["tflops"] = flops / ms / 1e9
            r["of_peak"] = r["tflops"] / pk["bf16_tflops"]
        if nbytes is not None:
            r["gbs"] = nbytes / ms / 1e6
            r["of_peak"] = r["gbs"] / pk["hbm_gbs"]
        rows.append(r)

    S, N = T + 64, B * T
    zero = torch.zeros(B, dtype=torch.int32, device=dev)
    pairs = T * (T + 1) // 2
    # softmax attention with the sink term, next to the same kernels without it
    q = torch.randn(B, T, H, D, device=dev, dtype=bf)
    ck = torch.randn(max(B, Bd), G, S, D, device=dev, dtype=bf)
    cv = torch.randn(max(B, Bd), G, S, D, device=dev, dtype=bf)
    sink = torch.randn(H, device=dev)
    for name, sk in (("softmax attention prefill with a sink term, over the cache", sink),
                     ("causal attention prefill over the cache (the like kernel)", None)):
        ms = timer(lambda: wa.window_attention_prefill(q, ck, cv, zero, D ** -0.5, sinks=sk), steps, warmup)
        row(name, "prefill attention", ms, flops=4.0 * D * pairs * H * B)
    qd = torch.randn(Bd, H, D, device=dev, dtype=bf)
    posd = torch.full((Bd,), T, dtype=torch.int32, device=dev)
    for name, sk in (("softmax attention decode with a sink term", sink), ("causal attention decode (the like kernel)", None)):
        ms = timer(lambda: wa.window_attention_decode(qd, ck, cv, posd, D ** -0.5, sinks=sk), steps, warmup)
        row(name, "decode attention", ms, nbytes=2.0 * (T + 1) * G * 2 * D * Bd)
    n_qkv = H * D + 2 * G * D
    wide = torch.randn(B, T, n_qkv, device=dev, dtype=bf)
    ckw, cvw = torch.zeros(B, G, S, D, device=dev, dtype=bf), torch.zeros(B, G, S, D, device=dev, dtype=bf)
    rope = rope_ops.build_interleaved_rope_cache(S, D // 2, 500000.0, device=dev, scaling=(8.0, 1.0, 4.0, 8192))
    qw, kw = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
    ms = timer(lambda: wa.qk_norm_cache_write(wide, ckw, cvw, zero, H, G, D, D, 1e-6, normalize=True, q_weight=qw,
                                              k_weight=kw, rope=rope, rope_layout="halves", whole_norm=True), steps, warmup)
    row("whole-projection q / k norm + rotation of halves + cache write", "projection epilogue", ms,
        nbytes=2.0 * N * (2 * H * D + 4 * G * D))
    ms = timer(lambda: wa.qk_norm_cache_write(wide, ckw, cvw, zero, H, G, D, D, 1e-6, normalize=False, rope=rope,
                                              rope_layout="halves"), steps, warmup)
    row("rotation of halves + cache write (sink-attention layers)", "projection epilogue", ms,
        nbytes=2.0 * N * (2 * H * D + 4 * G * D))
    ms = timer(lambda: wa.qk_norm_cache_write(wide, ckw, cvw, zero, H, G, D, D, 1e-6, normalize=True), steps, warmup)
    row("per-head unit norm + cache write (the like kernel)", "projection epilogue", ms,
        nbytes=2.0 * N * (2 * H * D + 4 * G * D))
    del q, ck, cv, wide, ckw, cvw
    # retention next to the matrix-memory kernels
    Hr, Dk, Dvr = s["rec_heads"], s["rec_dim"], s["rec_vdim"]
    ld = 2 * Hr * Dk + 2 * Hr * Dvr
    pr = torch.randn(B, T, ld, device=dev, dtype=bf) * 0.3
    dec = torch.full((Hr,), 0.99, device=dev)
    st = torch.zeros(max(B, Bd), Hr, Dk, Dvr, device=dev)
    rrope = rope_ops.build_interleaved_rope_cache(S, Dk, 500000.0, device=dev)
    offs = (0, Hr * Dk, 2 * Hr * Dk)
    flops = 4.0 * Dk * Dvr * Hr * B * T
    if rt.chunkwise_applies(Dk, Dvr):
        ms = timer(lambda: rt.retention_chunkwise(pr, offs, dec, st, zero, Hr, Dk, Dvr, Dk ** -0.5, rope=rrope), steps, warmup)
        row("retention prompt, chunk-wise (rotation inside)", "prefill attention", ms, flops=flops)
    ms = timer(lambda: rt.retention_scan(pr, offs, dec, st, zero, Hr, Dk, Dvr, Dk ** -0.5, rope=rrope), steps, warmup)
    row("retention prompt, token by token (state slice in registers, rotation inside)", "prefill attention", ms, flops=flops)
    gi, gf = torch.randn(N, Hr, device=dev), -torch.rand(N, Hr, device=dev) * 0.1
    mst = (torch.zeros(max(B, Bd), Hr, Dk, Dvr, device=dev), torch.zeros(max(B, Bd), Hr, Dk, device=dev),
           torch.zeros(max(B, Bd), Hr, device=dev))
    ms = timer(lambda: ml.mlstm_scan(pr, offs, gi, gf, mst, zero, Hr, Dk, Dvr, Dk ** -0.5), steps, warmup)
    row("matrix-memory scan, prompt, token by token (the like kernel)", "prefill attention", ms, flops=flops)
    ms = timer(lambda: ml.mlstm_chunkwise(pr, offs, gi, gf, mst, zero, Hr, Dk, Dvr, Dk ** -0.5), steps, warmup)
    row("matrix-memory prompt, chunk-wise (the like kernel of long bf16 steps)", "prefill attention", ms, flops=flops)
    prd = torch.randn(Bd, 1, ld, device=dev, dtype=bf) * 0.3
    at = torch.full((Bd,), T, dtype=torch.int32, device=dev)
    ms = timer(lambda: rt.retention_scan(prd, offs, dec, st, at, Hr, Dk, Dvr, Dk ** -0.5, rope=rrope), steps, warmup)
    row("retention, one token (state read + written)", "decode attention", ms, nbytes=8.0 * Dk * Dvr * Hr * Bd)
    ms = timer(lambda: ml.mlstm_scan(prd, offs, gi[:Bd], gf[:Bd], mst, at, Hr, Dk, Dvr, Dk ** -0.5), steps, warmup)
    row("matrix-memory scan, one token (the like kernel)", "decode attention", ms, nbytes=8.0 * Dk * Dvr * Hr * Bd)
    o = torch.randn(N, Hr, Dvr, device=dev)
    ms = timer(lambda: ml.head_norm_gate(o, pr.view(N, ld), 2 * Hr * Dk + Hr * Dvr, Hr, Dvr, None, 1e-6, True, bf,
                                         gate_act="silu"), steps, warmup)
    row("unit head norm * silu gate", "norm", ms, nbytes=float(N * Hr * Dvr * (4 + 2 + 2)))
    del pr, o
    # the stream update next to the gated residual of the parallel-residual family
    St = VUFASUN_STREAMS
    xs = torch.randn(N, St, W, device=dev)
    y1, y2 = torch.randn(N, W, device=dev, dtype=bf), torch.randn(N, W, device=dev, dtype=bf)
    mix, ow, iw = torch.eye(St, device=dev), torch.ones(St, device=dev), torch.ones(St, device=dev)
    wn, wa_, wb = torch.ones(W, device=dev), torch.ones(W, device=dev), torch.ones(W, device=dev)
    ms = timer(lambda: hc_ops.hc_step(xs, y1, mix, ow, iw, wn, 1e-6, bf), steps, warmup)
    row(f"stream write + mixing + next read and norm ({St} streams)", "norm", ms, nbytes=float(N * W * (8 * St + 2 + 2)))
    ms = timer(lambda: hc_ops.hc_step(xs, y1, mix, ow, iw, wn, 1e-6, bf, y2=y2, branch_w=(wa_, wb)), steps, warmup)
    row(f"the same with the mean of two normed branches ({St} streams)", "norm", ms, nbytes=float(N * W * (8 * St + 4 + 2)))
    x32 = torch.randn(N, W, device=dev)
    gate = torch.randn(N, 2 * W, device=dev, dtype=bf)
    vecs = [torch.randn(W, device=dev) for _ in range(5)]
    wnext = torch.ones(1, device=dev)
    ms = timer(lambda: norm_ops.gated_residual_norm_(x32, y1, y2, vecs[0], gate, (0, W), vecs[1], vecs[2], vecs[3], vecs[4],
                                                     wnext, 1e-6, bf), steps, warmup)
    row("gated residual of both sublayers + layer scale + next norm (the like kernel)", "norm", ms,
        nbytes=float(N * W * (4 + 4 + 2 + 2 + 4 + 2)))
    del xs, x32, gate
    F = (2 * s["ff"] // 3 + 127) // 128 * 128
    src = torch.randn(N, 2 * F, device=dev, dtype=bf)
    ms = timer(lambda: moe_sparse.glu_bias(src, 0, F, F, act="gelu_tanh"), steps, warmup)
    row("gelu_tanh(gate) * up from the fused projection", "activation", ms, nbytes=2.0 * N * 3 * F)
    gb, ub = torch.zeros(F, device=dev), torch.zeros(F, device=dev)
    ms = timer(lambda: moe_sparse.glu_bias(src, 0, F, F, gb, ub), steps, warmup)
    row("silu(gate + b) * (up + b) from the fused projection (the like kernel)", "activation", ms, nbytes=2.0 * N * 3 * F)
    return rows


def run_retention(steps: int = 10, warmup: int = 3, device=None, sizes=None) -> dict:
    dev = device or torch.device("cuda", torch.cuda.current_device())
    before = _lib.kernel_launches()
    out = {"metric": "Vufasun vs Gogalix, serving throughput at equal layer sizes", "dtype": "bf16",
           "data": "synthetic token ids, random-init weights", "steps": steps, "warmup": max(warmup, 3),
           "l2": "192 MB written between timed runs", "peaks": peaks(), "cases": [], "kernels": {}}
    for s in (sizes or HYBRID_SIZES):
        out["cases"].append(retention_serve_case(s, steps, warmup, dev))
        out["kernels"][s["name"]] = retention_kernel_cases(s, steps, warmup, dev)
    out["gpu_launches"] = _lib.kernel_launches() - before
    return out


# ---- Tidavik next to Rasodra (attention over the cache and latent attention with a dense feed-forward) ------------------------
def tidavik_config(s: dict):
    from ..models.tidavik import TidavikConfig

    # gate, up and down of (width x f) against Rasodra's two matrices of (width x ff): f = 2/3 ff keeps the parameters equal
    ff = {"kind": "dense", "ff": (2 * s["ff"] // 3 + 127) // 128 * 128}
    mask = {"size": s["chunk"]}
    att = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
           "softcap": 30.0, "mask": mask}
    lat = {"heads": s["heads"], "dim": s["lat_dim"], "vdim": s["lat_vdim"], "q_rank": 2 * s["rank"], "kv_rank": s["rank"],
           "scale": s["lat_dim"] ** -0.5, "mask": mask}
    return TidavikConfig.from_dict({
        "architecture": "Tidavik", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-6},
        "layers": [{"type": "attention", "mixer": att, "mlp": ff}, {"type": "attention_2", "mixer": att, "mlp": ff},
                   {"type": "latent_attention", "mixer": lat, "mlp": ff},
                   {"type": "latent_attention", "mixer": lat, "mlp": ff}]}, torch_dtype=torch.bfloat16)


def rasodra_attention_config(s: dict):
    """Rasodra without its recurrent layer: chunked attention twice, latent attention twice."""
    from ..models.rasodra import RasodraConfig

    d = rasodra_config(s).to_dict()
    att, _, lat, _ = d["layers"]
    d["layers"] = [att, att, lat, lat]
    return RasodraConfig.from_dict(d, torch_dtype=torch.bfloat16)


def scored_serve_case(s: dict, steps: int, warmup: int, dev) -> dict:
    from .hybrid import RasodraInferenceModel, TidavikInferenceModel

    timer = _Timer(dev)
    out = {"size": dict(s)}
    ic = dict(batch_size=s["decode_batch"], max_batch_size=s["decode_batch"], max_context_length=s["prompt"],
              seq_len=s["prompt"] + 64, is_continuous_batching=True, use_cuda_graphs=False)
    for name, make in (("tidavik", lambda: TidavikInferenceModel(tidavik_config(s), InferenceConfig(**ic), device=dev)),
                       ("rasodra", lambda: RasodraInferenceModel(rasodra_attention_config(s), InferenceConfig(**ic), device=dev))):
        torch.manual_seed(0)
        model = make()
        model.init_kv_cache(device=dev)
        out[name] = _serve(model, s, timer, steps, warmup, dev)
        out[name]["parameters"] = sum(p.numel() for p in model.parameters())
        del model
        torch.cuda.empty_cache()
    out["tidavik_over_rasodra"] = {k: out["tidavik"][k] / out["rasodra"][k]
                                   for k in ("prefill_tokens_per_s", "decode_tokens_per_s")}
    return out


def scored_kernel_cases(s: dict, steps: int, warmup: int, dev) -> List[dict]:
    """Tidavik's own kernels on the shapes of ``s``, alone, with roofline fractions, each next to the like kernel of the
    Rasodra / Gekazen families (windowed attention without score modifications, latent decode, projection epilogue,
    residual and norm, activation)."""
    from ..ops import latent_attention as la
    from ..ops import rope as rope_ops
    from ..ops import stream_norm as sn

    pk = peaks()
    timer = _Timer(dev)
    bf = torch.bfloat16
    B, T, H, G, D, W, Bd = s["prefill_batch"], s["prompt"], s["heads"], s["kv_heads"], s["dim"], s["width"], s["decode_batch"]
    win, S, N = s["chunk"], T + 64, B * T
    rows = []

    def row(kernel, like, fn, flops=None, nbytes=None):
        ms = timer(fn, steps, warmup)
        r = {"kernel": kernel, "like": like, "ms": ms, "peak": pk["source"]}
        if flops is not None:
            r["tflops"] = flops / ms / 1e9
            r["of_peak"] = r["tflops"] / pk["bf16_tflops"]
        if nbytes is not None:
            r["gbs"] = nbytes / ms / 1e6
            r["of_peak"] = r["gbs"] / pk["hbm_gbs"]
        rows.append(r)

    zero = torch.zeros(B, dtype=torch.int32, device=dev)
    pairs = sum(min(i + 1, win) for i in range(T))
    r1, r2, pb = torch.full((H,), 0.5, device=dev), torch.full((H,), 0.2, device=dev), torch.full((H,), -5.0, device=dev)
    one = torch.zeros(H, device=dev)
    kinds = [("soft cap + logarithmic bias + sigmoid weights", dict(softcap=30.0, log_bias=(r1, r2), sigmoid_bias=pb)),
             ("soft cap + one in the denominator", dict(softcap=30.0, sinks=one)),
             ("plain softmax (the like kernel)", {})]
    # prompts on the tcgen05 kernel (views of the projection output), and over the cache
    qkv = torch.randn(B, T, (H + 2 * G) * D, device=dev, dtype=bf)
    view = lambda a, n: qkv[..., a * D: (a + n) * D].unflatten(-1, (n, D)).permute(0, 2, 1, 3)               # noqa: E731
    q4, k4, v4 = view(0, H), view(H, G), view(H + G, G)
    for name, kw in kinds:
        row(f"windowed prefill, tcgen05: {name}", "prefill attention",
            lambda: wa.window_attention_tc(q4, k4, v4, D ** -0.5, win, **kw), flops=4.0 * D * pairs * H * B)
    q = torch.randn(B, T, H, D, device=dev, dtype=bf)
    ck = torch.randn(max(B, Bd), G, S, D, device=dev, dtype=bf)
    cv = torch.randn(max(B, Bd), G, S, D, device=dev, dtype=bf)
    for name, kw in kinds:
        row(f"windowed prefill over the cache, mma.sync: {name}", "prefill attention",
            lambda: wa.window_attention_prefill(q, ck, cv, zero, D ** -0.5, win, **kw), flops=4.0 * D * pairs * H * B)
    qd = torch.randn(Bd, H, D, device=dev, dtype=bf)
    posd = torch.full((Bd,), T, dtype=torch.int32, device=dev)
    for name, kw in kinds:
        row(f"windowed decode: {name}", "decode attention",
            lambda: wa.window_attention_decode(qd, ck, cv, posd, D ** -0.5, win, **kw), nbytes=2.0 * win * G * 2 * D * Bd)
    ckw, cvw = torch.zeros(B, G, S, D, device=dev, dtype=bf), torch.zeros(B, G, S, D, device=dev, dtype=bf)
    bias = torch.randn((H + 2 * G) * D, device=dev)
    qw, kw_ = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
    ep = 2.0 * N * (2 * H * D + 4 * G * D)
    row("bias + whole-projection q / k norm + cache write", "projection epilogue",
        lambda: wa.qk_norm_cache_write(qkv, ckw, cvw, zero, H, G, D, D, 1e-6, q_weight=qw, k_weight=kw_, whole_norm=True,
                                       bias=bias), nbytes=ep)
    row("bias + unit-RMS values + cache write", "projection epilogue",
        lambda: wa.qk_norm_cache_write(qkv, ckw, cvw, zero, H, G, D, D, 1e-6, normalize=False, bias=bias, value_norm=True),
        nbytes=ep)
    row("per-head unit q / k norm + cache write (the like kernel)", "projection epilogue",
        lambda: wa.qk_norm_cache_write(qkv, ckw, cvw, zero, H, G, D, D, 1e-6), nbytes=ep)
    del qkv, q, ck, cv, ckw, cvw
    # latent layers
    Dl, Dv, R, Rot, Q = s["lat_dim"], s["lat_vdim"], s["rank"], s["lat_rot"], 2 * s["rank"]
    ql = torch.randn(B, T, H, Dl, device=dev, dtype=bf)
    kv = torch.randn(B, T, H * (Dl + Dv), device=dev, dtype=bf)
    gate = torch.randn(B, T, H, device=dev, dtype=bf)
    kx, vx = kv[..., : H * Dl].unflatten(-1, (H, Dl)).permute(0, 2, 1, 3), kv[..., H * Dl:].unflatten(-1, (H, Dv)).permute(0, 2, 1, 3)
    fl = 2.0 * (Dl + Dv) * pairs * H * B
    row("latent prefill, expanded heads, tcgen05, output gate inside", "prefill attention",
        lambda: wa.window_attention_tc(ql.permute(0, 2, 1, 3), kx, vx, 0.07, win, gate=gate), flops=fl)
    row("latent prefill, expanded heads, mma.sync (portions), output gate inside", "prefill attention",
        lambda: wa.window_attention_prefill(ql, kx, vx, zero, 0.07, win, gate=gate), flops=fl)
    qr = torch.randn(B, T, H, Dl + Rot, device=dev, dtype=bf)
    kr = torch.randn(B, T, H, Dl + Rot, device=dev, dtype=bf).permute(0, 2, 1, 3)
    row("latent prefill of the closest family, window added (the like kernel)", "prefill attention",
        lambda: wa.window_attention_prefill(qr, kr, vx, zero, 0.07, win, sinks=one), flops=2.0 * (Dl + Rot + Dv) * pairs * H * B)
    del qr, kr, kv, ql
    cl = torch.randn(Bd, 1, S, R, device=dev, dtype=bf)
    qa, gd = torch.randn(Bd, H, R, device=dev, dtype=bf), torch.randn(Bd, H, device=dev, dtype=bf)
    row("latent decode in the window (absorbed queries, output gate)", "decode attention",
        lambda: wa.window_attention_decode(qa, cl, cl, posd, 0.07, win, gate=gd), nbytes=2.0 * win * R * Bd)
    cr = torch.randn(Bd, 1, S, R + Rot, device=dev, dtype=bf)
    qb = torch.randn(Bd, H, R + Rot, device=dev, dtype=bf)
    posw = torch.full((Bd,), win - 1, dtype=torch.int32, device=dev)
    row("latent decode of the closest family over as many rows (the like kernel)", "decode attention",
        lambda: wa.window_attention_decode(qb, cr, cr[..., :R], posw, 0.07, sinks=one), nbytes=2.0 * win * (R + Rot) * Bd)
    proj = torch.randn(B, T, Q + R + (H + 7) // 8 * 8, device=dev, dtype=bf)
    wq, wc = torch.ones(Q, device=dev), torch.ones(R, device=dev)
    row("both latent norms + cache row", "projection epilogue",
        lambda: la.latent_norms(proj, 0, Q, Q, R, cl, wq, wc, zero, 1e-6, rows=True), nbytes=2.0 * N * (2 * Q + 3 * R))
    pr = torch.randn(B, T, H * (Dl + Rot) + R + Rot, device=dev, dtype=bf)
    tables = rope_ops.build_interleaved_rope_cache(S, Rot, 1e6, device=dev)
    row("latent norm + rotations + cache row (the like kernel)", "projection epilogue",
        lambda: la.latent_prep(pr, 0, H * (Dl + Rot), None, cr, wc, tables, zero, H, Dl, Rot, R, 1e-6),
        nbytes=2.0 * N * (2 * H * (Dl + Rot) + 2 * (R + Rot)))
    del cl, cr, proj, pr
    # the stream
    x32, y = torch.randn(N, W, device=dev), torch.randn(N, W, device=dev, dtype=bf)
    w1, w2, b1 = torch.ones(W, device=dev), torch.ones(W, device=dev), torch.zeros(W, device=dev)
    row("residual add with output bias + next norm", "norm", lambda: sn.residual_norm_(x32, y, b1, w1, 1e-6, bf),
        nbytes=float(N * W * (4 + 4 + 2 + 2)))
    row("post-norm + residual + next norm (the like kernel)", "norm", lambda: norm_ops.norm_chain_(x32, y, w1, w2, 1e-6, bf),
        nbytes=float(N * W * (4 + 4 + 2 + 2)))
    table = torch.randn(VOCAB, W, device=dev, dtype=bf)
    ids = torch.randint(0, VOCAB, (B, T), device=dev)
    pos = torch.arange(T, device=dev).expand(B, T).contiguous()
    freq = sn.position_frequencies(W, device=dev)
    row("embedding + position vector + entry norm + first norm", "norm",
        lambda: sn.embed_norm(table, ids, pos, freq, w1, 1e-6, w2, bf), nbytes=float(N * W * (2 + 4 + 2)))
    F = (2 * s["ff"] // 3 + 127) // 128 * 128
    src = torch.randn(N, 2 * F, device=dev, dtype=bf)
    row("silu(gate) * up from the fused projection", "activation", lambda: moe_sparse.glu_bias(src, 0, F, F), nbytes=2.0 * N * 3 * F)
    row("SwiGLU of the Llama decoder (the like kernel)", "activation", lambda: act_ops.swiglu(src), nbytes=2.0 * N * 3 * F)
    return rows


def run_scored(steps: int = 10, warmup: int = 3, device=None, sizes=None) -> dict:
    dev = device or torch.device("cuda", torch.cuda.current_device())
    before = _lib.kernel_launches()
    out = {"metric": "Tidavik vs Rasodra (attention layers), serving throughput at equal layer sizes", "dtype": "bf16",
           "data": "synthetic token ids, random-init weights", "steps": steps, "warmup": max(warmup, 3),
           "l2": "192 MB written between timed runs", "peaks": peaks(), "cases": [], "kernels": {}}
    for s in (sizes or HYBRID_SIZES):
        out["cases"].append(scored_serve_case(s, steps, warmup, dev))
        out["kernels"][s["name"]] = scored_kernel_cases(s, steps, warmup, dev)
    out["gpu_launches"] = _lib.kernel_launches() - before
    return out


# ---- Mumazen next to Vufasun (attention over the cache beside a recurrent mixer, looped layers, gated feed-forward) -----------
SSM_STATE, SSM_HEAD, SCAN_STATE = 128, 64, 16          # state-space heads of 128 x 64, selective scan of 16 states per channel


def mumazen_config(s: dict):
    from ..models.mumazen import MumazenConfig

    ff = {"kind": "dense", "ff": (2 * s["ff"] // 3 + 127) // 128 * 128, "limit": 7.0}
    inner = s["rec_heads"] * s["rec_vdim"]             # as wide as Vufasun's retention heads together
    par = {"left": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
                    "softcap": 30.0, "rot": {"base": 500000.0, "dims": s["dim"] // 2, "scaling": {"factor": 4.0}}},
           "right": {"heads": inner // SSM_HEAD, "vdim": SSM_HEAD, "state": SSM_STATE, "groups": 1, "conv": 4, "norm_groups": 1},
           "left_scale": 1.0, "right_scale": 1.0}
    scan = {"inner": s["width"], "state": SCAN_STATE, "dt_rank": s["width"] // 16, "conv": 4}
    return MumazenConfig.from_dict({
        "architecture": "Mumazen", "vocab": VOCAB, "width": s["width"], "embedding": {"scale": 1.0}, "residual_mult": 1.0,
        "norm": {"eps": 1e-6}, "layers": [{"type": "parallel", "mixer": par, "mlp": ff},
                                          {"type": "mamba1", "mixer": scan, "mlp": ff},
                                          {"type": "parallel", "mixer": par, "mlp": ff}]}, torch_dtype=torch.bfloat16)


def state_space_serve_case(s: dict, steps: int, warmup: int, dev) -> dict:
    from .hybrid import MumazenInferenceModel, VufasunInferenceModel

    timer = _Timer(dev)
    out = {"size": dict(s)}
    ic = dict(batch_size=s["decode_batch"], max_batch_size=s["decode_batch"], max_context_length=s["prompt"],
              seq_len=s["prompt"] + 64, is_continuous_batching=True, use_cuda_graphs=False)
    for name, make in (("mumazen", lambda: MumazenInferenceModel(mumazen_config(s), InferenceConfig(**ic), device=dev)),
                       ("vufasun", lambda: VufasunInferenceModel(vufasun_config(s), InferenceConfig(**ic), device=dev))):
        torch.manual_seed(0)
        model = make()
        model.init_kv_cache(device=dev)
        out[name] = _serve(model, s, timer, steps, warmup, dev)
        out[name]["parameters"] = sum(p.numel() for p in model.parameters())
        del model
        torch.cuda.empty_cache()
    out["mumazen_over_vufasun"] = {k: out["mumazen"][k] / out["vufasun"][k]
                                   for k in ("prefill_tokens_per_s", "decode_tokens_per_s")}
    return out


def state_space_kernel_cases(s: dict, steps: int, warmup: int, dev) -> List[dict]:
    """Mumazen's own kernels on the shapes of ``s``, alone, with roofline fractions, each next to the like kernel of the Vufasun
    family (of Gogalix where Vufasun has none).  The selective scan is as wide as in a layer of its own (twice the width)."""
    from ..ops import delta_rule as dr
    from ..ops import hyper_connection as hc_ops
    from ..ops import mlstm as ml
    from ..ops import retention as rt
    from ..ops import rope as rope_ops
    from ..ops import state_space as ss
    from ..ops import stream_norm as sn

    pk = peaks()
    timer = _Timer(dev)
    bf = torch.bfloat16
    B, T, H, G, D, W, Bd = s["prefill_batch"], s["prompt"], s["heads"], s["kv_heads"], s["dim"], s["width"], s["decode_batch"]
    rows = []

    def row(kernel, like, fn, flops=None, nbytes=None):
        ms = timer(fn, steps, warmup)
        r = {"kernel": kernel, "like": like, "ms": ms, "peak": pk["source"]}
        if flops is not None:
            r["tflops"] = flops / ms / 1e9
            r["of_peak"] = r["tflops"] / pk["bf16_tflops"]
        if nbytes is not None:
            r["gbs"] = nbytes / ms / 1e6
            r["of_peak"] = r["gbs"] / pk["hbm_gbs"]
        rows.append(r)

    S, N = T + 64, B * T
    lines = max(B, Bd)
    zero = torch.zeros(B, dtype=torch.int32, device=dev)
    pairs = T * (T + 1) // 2
    fl = 4.0 * D * pairs * H * B
    # attention with the cap, next to the same kernels without it
    q = torch.randn(B, T, H, D, device=dev, dtype=bf)
    kv = torch.randn(2, B, T, G, D, device=dev, dtype=bf)
    qp, kp, vp = q.permute(0, 2, 1, 3), kv[0].permute(0, 2, 1, 3), kv[1].permute(0, 2, 1, 3)
    gate = torch.randn(B, T, H * D, device=dev, dtype=bf)
    gd = gate.view(-1, H * D)[:Bd]
    row("capped attention prefill + gate per element, tcgen05", "prefill attention",
        lambda: wa.window_attention_tc(qp, kp, vp, D ** -0.5, softcap=30.0, gate=gate, gate_elements=True), flops=fl)
    row("causal attention prefill, tcgen05 (the like kernel)", "prefill attention",
        lambda: attn_ops.flash_attn_func(qp, kp, vp, softmax_scale=D ** -0.5, causal=True), flops=fl)
    ck = torch.randn(lines, G, S, D, device=dev, dtype=bf)
    cv = torch.randn(lines, G, S, D, device=dev, dtype=bf)
    for name, cap in (("capped attention prefill over the cache + gate per element, mma.sync", 30.0),
                      ("causal attention prefill over the cache (the like kernel)", None)):
        kw = dict(gate=gate, gate_elements=True) if cap else {}
        row(name, "prefill attention", lambda: wa.window_attention_prefill(q, ck, cv, zero, D ** -0.5, softcap=cap, **kw), flops=fl)
    qd = torch.randn(Bd, H, D, device=dev, dtype=bf)
    posd = torch.full((Bd,), T, dtype=torch.int32, device=dev)
    for name, cap in (("capped attention decode + gate per element", 30.0), ("causal attention decode (the like kernel)", None)):
        kw = dict(gate=gd, gate_elements=True) if cap else {}
        row(name, "decode attention", lambda: wa.window_attention_decode(qd, ck, cv, posd, D ** -0.5, softcap=cap, **kw),
            nbytes=2.0 * (T + 1) * G * 2 * D * Bd)
    del kv, ck, cv, gate, gd
    n_qkv = H * D + 2 * G * D
    wide = torch.randn(B, T, n_qkv, device=dev, dtype=bf)
    ckw, cvw = torch.zeros(B, G, S, D, device=dev, dtype=bf), torch.zeros(B, G, S, D, device=dev, dtype=bf)
    rope = rope_ops.build_interleaved_rope_cache(S, D // 2, 500000.0, device=dev, factor=4.0)
    for name, back in (("slowed rotation of halves + cache write + write-back", True), ("rotation of halves + cache write (the like kernel)", False)):
        row(name, "projection epilogue", lambda: wa.qk_norm_cache_write(wide, ckw, cvw, zero, H, G, D, D, 1e-6, normalize=False, rope=rope,
                                                                       rope_layout="halves", writeback=back),
            nbytes=2.0 * N * (2 * H * D + (5 if back else 4) * G * D))
    del wide, ckw, cvw, q
    # state-space heads next to retention
    Hr, Dk, Dvr = s["rec_heads"], s["rec_dim"], s["rec_vdim"]
    inner = Hr * Dvr
    Hs, Ns, P = inner // SSM_HEAD, SSM_STATE, SSM_HEAD
    C = inner + 2 * Ns
    xbc = torch.randn(B, T, C, device=dev, dtype=bf)
    cw, cb, cst = torch.randn(4, C, device=dev), torch.randn(C, device=dev), torch.zeros(lines, 3, C, device=dev)
    row("short convolution + bias + silu + state", "convolution", lambda: ss.conv_silu(xbc, cw, cb, cst, zero), nbytes=4.0 * N * C)
    Gd, Hd = max(1, C // (4 * Dk) // 2), max(1, C // 2 // Dvr)            # about as many channels
    Cd = 2 * Gd * Dk + (Hd // Gd * Gd or Gd) * Dvr
    Hd = Hd // Gd * Gd or Gd
    big = torch.randn(B, T, Cd, device=dev, dtype=bf)
    cwd, cstd = torch.randn(Cd, 4, device=dev), torch.zeros(lines, 3, Cd, device=dev)
    row("short convolution + silu + unit norm + state of the delta rule (the like kernel; fp32 output)", "convolution",
        lambda: dr.delta_prep(big, (0, Gd * Dk, 2 * Gd * Dk), cwd, cstd, zero, Hd, Gd, Dk, Dvr, 1.0), nbytes=6.0 * N * Cd)
    del big
    dt = torch.randn(B, T, Hs, device=dev)
    vec = [torch.randn(Hs, device=dev) for _ in range(3)]
    st = torch.zeros(lines, Hs, Ns, P, device=dev)
    offs = (0, inner, inner + Ns)
    row("state-space heads, prompt, chunks on tensor cores", "prefill recurrence",
        lambda: ss.state_space_heads(xbc, offs, dt, *vec, st, zero, 1), flops=4.0 * Ns * P * Hs * N)
    row("state-space heads, prompt, token by token", "prefill recurrence",
        lambda: ss.state_space_heads(xbc, offs, dt, *vec, st, zero, 1, impl="scan"), flops=4.0 * Ns * P * Hs * N)
    ld = 2 * Hr * Dk + 2 * Hr * Dvr
    pr = torch.randn(B, T, ld, device=dev, dtype=bf) * 0.3
    dec = torch.full((Hr,), 0.99, device=dev)
    rst = torch.zeros(lines, Hr, Dk, Dvr, device=dev)
    rrope = rope_ops.build_interleaved_rope_cache(S, Dk, 500000.0, device=dev)
    roffs = (0, Hr * Dk, 2 * Hr * Dk)
    row("retention prompt, chunk-wise (the like kernel)", "prefill recurrence",
        lambda: rt.retention_chunkwise(pr, roffs, dec, rst, zero, Hr, Dk, Dvr, Dk ** -0.5, rope=rrope), flops=4.0 * Dk * Dvr * Hr * N)
    xd, dtd = xbc[:1, :1].expand(Bd, 1, C).contiguous(), torch.randn(Bd, 1, Hs, device=dev)
    row("state-space heads, one token (state read + written)", "decode recurrence",
        lambda: ss.state_space_heads(xd, offs, dtd, *vec, st, posd, 1), nbytes=8.0 * Ns * P * Hs * Bd)
    prd = torch.randn(Bd, 1, ld, device=dev, dtype=bf) * 0.3
    row("retention, one token (the like kernel)", "decode recurrence",
        lambda: rt.retention_scan(prd, roffs, dec, rst, posd, Hr, Dk, Dvr, Dk ** -0.5, rope=rrope), nbytes=8.0 * Dk * Dvr * Hr * Bd)
    y, w = torch.randn(N, inner, device=dev), torch.ones(inner, device=dev)
    row("silu gate, then RMS norm over the row", "norm", lambda: ss.gate_norm(y, pr.view(N, ld)[:, :inner], w, 1, 1e-6), nbytes=8.0 * N * inner)
    yh = y.view(N, Hr, Dvr)
    row("unit head norm * silu gate (the like kernel)", "norm",
        lambda: ml.head_norm_gate(yh, pr.view(N, ld), 0, Hr, Dvr, None, 1e-6, True, bf, gate_act="silu"), nbytes=8.0 * N * inner)
    del xbc, pr, y, st, rst
    # selective scan
    Ci, n = 2 * W, SCAN_STATE
    x, z = torch.randn(B, T, Ci, device=dev, dtype=bf), torch.randn(B, T, Ci, device=dev, dtype=bf)
    dts, bc = torch.randn(B, T, Ci, device=dev), torch.randn(B, T, 2 * n, device=dev)
    a_log, dv = torch.rand(Ci, n, device=dev), torch.randn(2, Ci, device=dev)
    sst = torch.zeros(lines, Ci, n, device=dev)
    row("selective scan + gate, prompt", "prefill recurrence",
        lambda: ss.selective_scan(x, dts, dv[0], bc, 0, n, z, a_log, dv[1], sst, zero), nbytes=float(N * (10 * Ci + 8 * n)))
    rank = W // 16
    xd, zd = (t[:1, :1].expand(Bd, 1, Ci).contiguous() for t in (x, z))
    pd, dtw = torch.randn(Bd, 1, rank + 2 * n, device=dev), torch.randn(Ci, rank, device=dev, dtype=bf) * rank ** -0.5
    row("step sizes + selective scan + gate, one token (weights read, state read + written)", "decode recurrence",
        lambda: ss.selective_scan(xd, None, dv[0], pd, rank, rank + n, zd, a_log, dv[1], sst, posd, dt_w=dtw),
        nbytes=8.0 * Ci * n * Bd + 2.0 * Ci * rank)
    del x, z, dts, bc, sst
    # the stream
    x32 = torch.randn(N, W, device=dev)
    y1 = torch.randn(N, W, device=dev, dtype=bf)
    v = [torch.ones(W, device=dev) for _ in range(4)]
    table, ids = torch.randn(VOCAB, W, device=dev, dtype=bf), torch.randint(0, VOCAB, (N,), device=dev)
    row("layer-scaled residual + output bias + next norm", "norm",
        lambda: sn.stream_update_(x32, y1, v[0], v[1], w_next=v[2], out_dtype=bf), nbytes=float(N * W * 12))
    row("the same with the embedding and a pass vector added", "norm",
        lambda: sn.stream_update_(x32, y1, v[0], v[1], table, ids, 1.0, v[3], v[2], out_dtype=bf), nbytes=float(N * W * 14))
    xs = torch.randn(N, VUFASUN_STREAMS, W, device=dev)
    mix, ow = torch.eye(VUFASUN_STREAMS, device=dev), torch.ones(VUFASUN_STREAMS, device=dev)
    row(f"stream write + mixing + next read and norm, {VUFASUN_STREAMS} streams (the like kernel)", "norm",
        lambda: hc_ops.hc_step(xs, y1, mix, ow, ow, v[2], 1e-6, bf), nbytes=float(N * W * (8 * VUFASUN_STREAMS + 4)))
    del xs, x32
    F = (2 * s["ff"] // 3 + 127) // 128 * 128
    src, gb = torch.randn(N, 2 * F, device=dev, dtype=bf), torch.zeros(F, device=dev)
    row("clamped gated activation with biases", "activation",
        lambda: moe_sparse.glu_bias(src, 0, F, F, gb, gb, limit=7.0, alpha=moe_sparse.GLU_ALPHA, up_shift=1.0), nbytes=6.0 * N * F)
    row("gelu_tanh(gate) * up (the like kernel)", "activation", lambda: moe_sparse.glu_bias(src, 0, F, F, act="gelu_tanh"), nbytes=6.0 * N * F)
    del src
    # sparse feed-forward of token generation: 8 experts, two of them per token
    E, Fe = 8, W // 2
    h = torch.randn(Bd, W, device=dev, dtype=bf)
    wr, corr = torch.randn(E + 4, W, device=dev) * W ** -0.5, torch.zeros(E + 4, device=dev)
    row("router: normalised scores with identity experts", "router", lambda: moe_sparse.route(h, wr, corr, 2, 1.0, normalize=True), nbytes=4.0 * (E + 4) * W)
    row("router: sigmoid scores (the like kernel)", "router", lambda: moe_sparse.route(h, wr, None, 2, 1.0, score="sigmoid"), nbytes=4.0 * (E + 4) * W)
    idx = torch.stack([torch.arange(Bd, device=dev) % E, (torch.arange(Bd, device=dev) + 3) % E], dim=1).to(torch.int32).contiguous()
    wu, wg = torch.randn(E, W, Fe, device=dev, dtype=bf), torch.randn(E, W, 2 * Fe, device=dev, dtype=bf)
    row("expert up products + squared relu, per pair", "expert", lambda: moe_sparse.up_act(h, wu, idx), nbytes=2.0 * Bd * 2 * W * Fe)
    row("expert gate / up products + silu, per pair (the like kernel)", "expert",
        lambda: moe_sparse.gate_up_act(h, wg, idx, float("inf"), 1.0, 0.0), nbytes=2.0 * Bd * 2 * W * 2 * Fe)
    return rows


def run_state_space(steps: int = 10, warmup: int = 3, device=None, sizes=None) -> dict:
    dev = device or torch.device("cuda", torch.cuda.current_device())
    before = _lib.kernel_launches()
    out = {"metric": "Mumazen vs Vufasun, serving throughput at equal layer sizes", "dtype": "bf16",
           "data": "synthetic token ids, random-init weights", "steps": steps, "warmup": max(warmup, 3),
           "l2": "192 MB written between timed runs", "peaks": peaks(), "cases": [], "kernels": {}}
    for s in (sizes or HYBRID_SIZES):
        out["cases"].append(state_space_serve_case(s, steps, warmup, dev))
        out["kernels"][s["name"]] = state_space_kernel_cases(s, steps, warmup, dev)
    out["gpu_launches"] = _lib.kernel_launches() - before
    return out
