"""Tidavik family against the plain oracle of ``tests/tidavik_oracle.py``: every mechanism alone, then the model through the
framework's step function, cache manager and schedulers.  Every test runs on the CPU (the ops' PyTorch path) and, marked
``gpu``, on CUDA (the kernels) in fp32 and bf16."""
import json
import os
import subprocess
import sys

import pytest
import torch

import tidavik_oracle as O
from neuronx_distributed_llama3_2_b200.inference import InferenceConfig, TidavikInferenceModel
from neuronx_distributed_llama3_2_b200.inference.trace_replay import TraceReplayer
from neuronx_distributed_llama3_2_b200.models.tidavik import (TidavikConfig, convert_tidavik_state_dict,
                                                              export_tidavik_state_dict, in_proj_columns, tiny_tidavik)
from neuronx_distributed_llama3_2_b200.ops import latent_attention as la
from neuronx_distributed_llama3_2_b200.ops import stream_norm as sn
from neuronx_distributed_llama3_2_b200.ops import window_attention as wa

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F64 = torch.float64
CASES = [("cpu", torch.float32), pytest.param("cuda", torch.float32, marks=pytest.mark.gpu),
         pytest.param("cuda", torch.bfloat16, marks=pytest.mark.gpu)]
case = pytest.mark.parametrize("dev,dt", CASES)


def close(a, b, dt, scale=1.0):
    """Largest difference relative to the largest value (at least 1)."""
    tol = (2e-5 if dt == torch.float32 else 2e-2) * scale * max(1.0, float(b.abs().max()))
    err = (a.detach().to("cpu", F64) - b.to(F64)).abs().max().item()
    assert err <= tol, f"max error {err:.3e} above {tol:.1e}"


LAT = dict(heads=3, dim=16, vdim=24, q_rank=40, kv_rank=32, scale=0.25, mask={"size": 11})
SIG = dict(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.2, softcap=6.0, mask={"size": 19})
CAP = dict(heads=6, kv_heads=3, dim=16, vdim=8, scale=0.3, softcap=9.0, mask={"size": 7})
BASE = {"latent_attention": LAT, "attention": SIG, "attention_2": CAP}
FF = {"kind": "dense", "ff": 72}


def layer(kind, mlp=FF, **kw):
    return {"type": kind, "mixer": dict(BASE[kind], **kw), "mlp": mlp}


def config(layers=None, vocab=112, width=56, eps=1e-5):
    layers = layers or [layer("attention_2"), layer("latent_attention", mlp=None), layer("attention"),
                        layer("latent_attention", heads=2, mask={"size": 23}), layer("attention", heads=2, kv_heads=2, dim=16)]
    return {"architecture": "Tidavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# what the usual configurations make equal or 1: a single head, one key head for all and one for each, equal and odd key /
# value sizes, ranks smaller and larger than the width, a window of one token and of two, windows wider than the sequence, a
# tight and a wide cap, sizes that are no multiple of 8, a large eps, no feed-forward
ODD = config(layers=[
    layer("attention", heads=1, kv_heads=1, dim=5, vdim=7, scale=1.0, softcap=0.8, mask={"size": 2}, mlp={"kind": "dense", "ff": 11}),
    layer("latent_attention", heads=1, dim=9, vdim=9, q_rank=7, kv_rank=5, scale=0.7, mask={"size": 1}, mlp={"kind": "dense", "ff": 5}),
    layer("attention_2", heads=3, kv_heads=3, dim=6, vdim=6, scale=1.3, softcap=0.5, mask={"size": 3}, mlp=None),
    layer("latent_attention", heads=5, dim=33, vdim=3, q_rank=50, kv_rank=70, scale=0.1, mask={"size": 500}, mlp=None),
    layer("attention_2", heads=6, kv_heads=1, dim=40, vdim=34, scale=0.05, softcap=200.0, mask={"size": 64}, mlp={"kind": "dense", "ff": 30}),
    layer("attention", heads=6, kv_heads=3, dim=34, vdim=5, scale=0.3, softcap=2.0, mask={"size": 33}, mlp={"kind": "dense", "ff": 16}),
], vocab=50, width=30, eps=1e-2)


def build(cfg, dev, dt, lines=4, seq_len=96, seed=1, paged=False, pages=None, page_size=8, sd=None):
    sd = sd if sd is not None else O.random_weights(cfg, seed)
    tc = TidavikConfig.from_dict(cfg, torch_dtype=dt)
    ic = InferenceConfig(batch_size=lines, max_batch_size=lines, max_context_length=seq_len, seq_len=seq_len,
                         is_continuous_batching=True, use_cuda_graphs=False, paged_kv=paged, page_size=page_size,
                         num_kv_pages=pages)
    model = TidavikInferenceModel(tc, ic, device=torch.device(dev))
    missing, unexpected = model.load_state_dict(convert_tidavik_state_dict(sd, tc), strict=False)
    assert not unexpected and not missing, (missing, unexpected)
    model.init_kv_cache(device=torch.device(dev))
    return model, sd


def tokens_of(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def replay(model, steps):
    rp_ = TraceReplayer(model)
    got = {}
    for entries, end in steps:
        out = rp_.step(entries, end)
        r = 0
        for e in entries:
            for _ in e["want"]:
                got.setdefault(e["id"], []).append(out[r].cpu())
                r += 1
    return got


def rel_err(row, ref):
    d = row.to(F64) - ref
    d = d - d.mean()
    return float(d.pow(2).mean().sqrt() / ref.std())


def check_rows(rows, ref, places, dt, strict=1e-4):
    """Every position against the oracle: centred difference over the vocabulary, relative to the spread of the logits.
    fp32 is strict; bf16 rounding through the tiny layers reaches a few percent at single positions."""
    assert len(rows) == len(places)
    rels = [rel_err(row, ref[p]) for row, p in zip(rows, places)]
    worst = max(range(len(rels)), key=lambda i: rels[i])
    limit = strict if dt == torch.float32 else 0.12
    assert rels[worst] <= limit, f"position {places[worst]}: relative error {rels[worst]:.2e}"
    assert dt == torch.float32 or sum(rels) / len(rels) <= 0.04, f"mean relative error {sum(rels) / len(rels):.2e}"


# ---- mechanisms alone ------------------------------------------------------------------------------------------------------
@case
@pytest.mark.parametrize("W", [12, 56, 33, 1])
def test_embedding_with_position_vectors_and_the_first_norms(dev, dt, W):
    torch.manual_seed(W)
    table, we, wn = torch.randn(20, W).to(dt), torch.randn(W), torch.randn(W)
    ids = torch.tensor([[3, 19, 0], [7, 7, 7]])
    pos = torch.tensor([[0, 1, 2], [5, 1000, 123457]])
    e = table.to(F64)[ids] + torch.stack([O.position_vectors(p.tolist(), W) for p in pos])
    x_ref = O.rms(e, 1e-4) * we.to(F64)
    x, h = sn.embed_norm(table.to(dev), ids.to(dev), pos.to(dev), sn.position_frequencies(W, device=dev), we.to(dev), 1e-4,
                         wn.to(dev), dt)
    close(x, x_ref, torch.float32)
    close(h, O.rms(x_ref, 1e-4) * wn.to(F64), dt)
    x, h = sn.embed_norm(table.to(dev), ids.to(dev), pos.to(dev), None, we.to(dev), 1e-4)       # no position vectors
    assert h is None
    close(x, O.rms(table.to(F64)[ids], 1e-4) * we.to(F64), torch.float32)


@case
@pytest.mark.parametrize("W", [7, 40, 1024, 1100, 2052, 5000, 517])
def test_residual_add_with_bias_and_the_next_norm(dev, dt, W):
    torch.manual_seed(W)
    N, eps = 5, 1e-3
    x, y, b, w = torch.randn(N, W), (2 * torch.randn(N, W)).to(dt), torch.randn(W), torch.randn(W)
    for bias in (b, None):
        new = x.to(F64) + y.to(F64) + (b.to(F64) if bias is not None else 0.0)
        xd = x.clone().to(dev)
        _, h = sn.residual_norm_(xd, y.to(dev), bias.to(dev) if bias is not None else None, w.to(dev), eps, dt)
        close(xd, new, torch.float32)
        close(h, O.rms(new, eps) * w.to(F64), dt)
        xd = x.clone().to(dev)                                                         # the add alone
        assert sn.residual_norm_(xd, y.to(dev), bias.to(dev) if bias is not None else None)[1] is None
        close(xd, new, torch.float32)
    xd = x.clone().to(dev)                                                             # the norm alone leaves the stream
    _, h = sn.residual_norm_(xd, None, None, w.to(dev), eps, dt)
    assert torch.equal(xd.cpu(), x)
    close(h, O.rms(x.to(F64), eps) * w.to(F64), dt)


@case
@pytest.mark.parametrize("whole", [True, False])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 16, 8), (3, 3, 6, 7), (6, 1, 34, 33), (2, 2, 64, 64)])
def test_projection_bias_norms_and_cache_write(dev, dt, whole, H, G, D, Dv):
    """q | k | v columns of a wider row: bias first, then the norm over the whole q and the whole k projection (``whole``)
    or unit-RMS values per head; keys and values into the lines of a paged cache; padding rows write nothing.  With
    write-back the row then holds the keys and values as cached."""
    torch.manual_seed(D)
    B, T, eps, page = 2, 7, 1e-2, 4
    n = H * D + G * (D + Dv)
    big = torch.randn(B, T, n + 13).to(dt)
    bias = torch.randn(n)
    qw, kw = torch.randn(H * D), torch.randn(G * D)
    starts, cnt, lines = [0, 9], [7, 4], [2, 0]
    table = torch.tensor([[5, 1, 7, 0], [2, 9, 4, 8], [3, 6, 10, 11]], dtype=torch.int32)
    ckd = torch.full((12, G, page, D), 9.0, dtype=dt, device=dev)
    cvd = torch.full((12, G, page, Dv), 9.0, dtype=dt, device=dev)
    bigd = big.clone().to(dev)
    q = wa.qk_norm_cache_write(bigd[..., 5: 5 + n], ckd, cvd, torch.tensor(starts, device=dev), H, G, D, Dv, eps,
                               n_new=torch.tensor(cnt, device=dev), seq_ids=torch.tensor(lines, device=dev),
                               normalize=whole, whole_norm=whole, q_weight=qw.to(dev) if whole else None,
                               k_weight=kw.to(dev) if whole else None, bias=bias.to(dev), value_norm=not whole,
                               block_table=table.to(dev), page_size=page, writeback=True)
    row = big.to(F64)[..., 5: 5 + n] + bias.to(F64)
    qr, kr, vr = row[..., : H * D], row[..., H * D: (H + G) * D], row[..., (H + G) * D:]
    if whole:
        qr, kr = O.rms(qr, eps) * qw.to(F64), O.rms(kr, eps) * kw.to(F64)
    else:
        vr = O.rms(vr.reshape(B, T, G, Dv), eps).reshape(B, T, G * Dv)
    close(q, qr.reshape(B, T, H, D), dt)
    ck, cv = torch.full((12, G, page, D), 9.0, dtype=F64), torch.full((12, G, page, Dv), 9.0, dtype=F64)
    back = big.to(F64)
    for b in range(B):
        for t in range(cnt[b]):
            p = starts[b] + t
            pg, off = int(table[lines[b], p // page]), p % page
            ck[pg, :, off], cv[pg, :, off] = kr[b, t].reshape(G, D), vr[b, t].reshape(G, Dv)
            back[b, t, 5 + H * D: 5 + n] = torch.cat([kr[b, t], vr[b, t]])
    close(ckd, ck, dt)
    close(cvd, cv, dt)
    close(bigd, back, dt)


@case
@pytest.mark.parametrize("Q,R", [(24, 32), (7, 5), (130, 66), (256, 64)])
def test_latent_norms_and_cache_rows(dev, dt, Q, R):
    torch.manual_seed(Q)
    B, T, eps, page = 2, 6, 1e-2, 4
    ld = (Q + 7) // 8 * 8 + (R + 7) // 8 * 8 + 8
    qo, ko = 0, (Q + 7) // 8 * 8
    proj = torch.randn(B, T, ld).to(dt)
    qw, cw = torch.randn(Q), torch.randn(R)
    starts, cnt, lines = [3, 0], [6, 2], [1, 0]
    cq_ref = O.rms(proj.to(F64)[..., qo: qo + Q], eps) * qw.to(F64)
    c_ref = O.rms(proj.to(F64)[..., ko: ko + R], eps) * cw.to(F64)
    table = torch.tensor([[5, 1, 7], [2, 6, 4]], dtype=torch.int32)
    for paged in (False, True):
        cache = torch.full((8, 1, page, R) if paged else (2, 1, 12, R), 9.0, dtype=dt, device=dev)
        kw = dict(block_table=table.to(dev), page_size=page) if paged else {}
        cq, c = la.latent_norms(proj.to(dev), qo, ko, Q, R, cache, qw.to(dev), cw.to(dev), torch.tensor(starts, device=dev),
                                eps, n_new=torch.tensor(cnt, device=dev), seq_ids=torch.tensor(lines, device=dev),
                                rows=not paged, **kw)
        close(cq.reshape(B, T, Q), cq_ref, dt)
        assert (c is None) == paged
        if c is not None:
            close(c.reshape(B, T, R), c_ref, dt)
        ref = torch.full(tuple(cache.shape), 9.0, dtype=F64)
        for b in range(B):
            for t in range(cnt[b]):
                p = starts[b] + t
                if paged:
                    ref[int(table[lines[b], p // page]), 0, p % page] = c_ref[b, t]
                else:
                    ref[lines[b], 0, p] = c_ref[b, t]
        close(cache, ref, dt)


def oracle_attention(kind, q, k, v, scale, window, cap, r1, r2, pb, gate):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, Dv]``, ``gate [T, H]`` or None -> ``[T, H, Dv]``."""
    T = q.shape[0]
    vis = O.visible(T, window)
    if kind == "plain":
        p = O.softmax_weights(O.scores(q, k, scale), vis)
    elif kind == "sigmoid":
        p = O.sigmoid_weights(O.scores(q, k, scale, cap, r1, r2), vis, pb)
    else:
        p = O.softmax_weights(O.scores(q, k, scale, cap), vis, extra_one=True)
    o = O.weighted_values(p, v)
    return o * torch.sigmoid(gate).unsqueeze(-1) if gate is not None else o


def attention_kw(kind, cap, r1, r2, pb, H, dev):
    if kind == "plain":
        return {}
    if kind == "sigmoid":
        return dict(softcap=cap, log_bias=(r1.to(dev), r2.to(dev)), sigmoid_bias=pb.to(dev))
    return dict(softcap=cap, sinks=torch.zeros(H, device=dev))


def attention_inputs(T, H, G, D, Dv, dt, seed, big=False):
    """Random rows; ``big``: some scores lie far above the cap (and above the range of the tanh series)."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)                                         # noqa: E731
    q, k, v, gate = r(T, H, D), r(T, G, D), r(T, G, Dv), r(T, H)
    if big:
        q[T // 2] *= 6.0
        k[::5] *= 4.0
    return [t.to(dt) for t in (q, k, v, gate)] + [0.8 + 0.3 * r(H), 0.1 + torch.rand(H, generator=g), r(H) - 1.0]


SHAPES = [(4, 2, 16, 8), (3, 1, 33, 40), (4, 2, 32, 32), (4, 1, 64, 64), (6, 3, 96, 96), (2, 2, 128, 128), (4, 2, 64, 128),
          (2, 1, 128, 64), (2, 2, 32, 48)]


@case
@pytest.mark.parametrize("kind", ["plain", "sigmoid", "capped"])
@pytest.mark.parametrize("H,G,D,Dv", SHAPES)
def test_attention_over_the_cache(dev, dt, kind, H, G, D, Dv):
    """Prompt rows at different offsets of two lines, then one decoded row, against whole-sequence attention: windows that
    end inside a key tile, at its border and one beside it, and no window; a contiguous cache and pages; with and without
    the output gate; scores on both sides of the tanh series' range."""
    n, scale = 150, D ** -0.5
    big = kind != "plain"
    seqs = [attention_inputs(n, H, G, D, Dv, dt, 7 + D, big), attention_inputs(n, H, G, D, Dv, dt, 8 + D, big)]
    r1, r2, pb = seqs[0][4:]
    page = 16
    table = torch.randperm(20, generator=torch.Generator().manual_seed(1)).reshape(2, 10).to(torch.int32)
    for i, window in enumerate([64, 65, 63, 5, 1, None]):
        cap, paged, gated = [30.0, 2.5][i % 2], i % 2 == 1, i % 3 != 2
        starts, cnt = ([20, 0], [90, 131]) if i != 3 else ([0, 100], [3, 2])
        shape = (20, G, page) if paged else (2, G, 160)
        ck, cv = torch.full(shape + (D,), 3.0, dtype=dt), torch.full(shape + (Dv,), 3.0, dtype=dt)
        for b, (q, k, v, *_) in enumerate(seqs):
            for p in range(n):
                at = (int(table[b, p // page]), p % page) if paged else (b, p)
                ck[at[0], :, at[1]], cv[at[0], :, at[1]] = k[p], v[p]
        kw = attention_kw(kind, cap, r1, r2, pb, H, dev)
        if paged:
            kw.update(block_table=table.to(dev), page_size=page)
        Tn = max(cnt)
        qb, gb = torch.zeros(2, Tn, H, D, dtype=dt), torch.zeros(2, Tn, H + 3, dtype=dt)
        refs = []
        for b, (q, k, v, gate, *_) in enumerate(seqs):
            qb[b, :cnt[b]] = q[starts[b]: starts[b] + cnt[b]]
            gb[b, :cnt[b], :H] = gate[starts[b]: starts[b] + cnt[b]]
            refs.append(oracle_attention(kind, q.to(F64), k.to(F64), v.to(F64), scale, window, cap, r1.to(F64), r2.to(F64),
                                         pb.to(F64), gate.to(F64) if gated else None))
        ckd, cvd, gd = ck.to(dev), cv.to(dev), gb.to(dev)
        o = wa.window_attention_prefill(qb.to(dev), ckd, cvd, torch.tensor(starts, device=dev), scale, window,
                                        n_new=torch.tensor(cnt, device=dev), gate=gd[..., :H] if gated else None, **kw)
        for b in range(2):
            close(o[b, :cnt[b]], refs[b][starts[b]: starts[b] + cnt[b]], dt)
            assert not bool(o[b, cnt[b]:].any())                                # padding rows are zeros
        pos = [n - 1, 64]
        qd = torch.stack([seqs[b][0][pos[b]] for b in range(2)])
        gd = torch.stack([torch.cat([seqs[b][3][pos[b]], torch.zeros(5, dtype=dt)]) for b in range(2)]).to(dev)
        o = wa.window_attention_decode(qd.to(dev), ckd, cvd, torch.tensor(pos, device=dev), scale, window,
                                       gate=gd[:, :H] if gated else None, **kw)
        for b in range(2):
            close(o[b], refs[b][pos[b]], dt)


@case
@pytest.mark.parametrize("R,H", [(24, 3), (128, 5), (256, 20), (384, 2), (512, 16)])
def test_windowed_attention_over_latent_rows(dev, dt, R, H):
    """One decoded token per row over latent rows (values = the rows themselves): window edges inside and at tile borders,
    output gate, context split over CTAs, pages."""
    torch.manual_seed(R)
    n, scale, page = 200, R ** -0.5, 32
    rows = torch.randn(2, n, R).to(dt)
    table = torch.randperm(14, generator=torch.Generator().manual_seed(1)).reshape(2, 7).to(torch.int32)
    q, gate = torch.randn(2, H, R).to(dt), torch.randn(2, H + 2).to(dt)
    for window, pos, paged in [(64, [199, 63], False), (65, [64, 127], True), (1, [5, 128], False), (None, [199, 0], True),
                               (150, [198, 149], True)]:
        cache = torch.full((14, 1, page, R) if paged else (2, 1, n, R), 5.0, dtype=dt)
        for b in range(2):
            for p in range(n):
                if paged:
                    cache[int(table[b, p // page]), 0, p % page] = rows[b, p]
                else:
                    cache[b, 0, p] = rows[b, p]
        cache = cache.to(dev)
        kw = dict(block_table=table.to(dev), page_size=page) if paged else {}
        o = wa.window_attention_decode(q.to(dev), cache, cache[..., :R], torch.tensor(pos, device=dev), scale, window,
                                       gate=gate.to(dev)[:, :H], **kw)
        for b in range(2):
            lo = max(0, pos[b] - window + 1) if window else 0
            keys = rows[b, lo: pos[b] + 1].to(F64)
            ref = torch.softmax(q[b].to(F64) @ keys.T * scale, dim=-1) @ keys
            close(o[b], ref * torch.sigmoid(gate[b, :H].to(F64)).unsqueeze(-1), dt)


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["plain", "sigmoid", "capped"])
@pytest.mark.parametrize("D", [64, 128])
def test_tcgen05_prompt_attention(kind, D):
    """Prompts from position 0 on the tcgen05 kernel: several windows (inside a tile, at its border, one beside it, wider than
    the prompt, none), lengths that end inside tiles, strided q / k / v views, output gate; scores on both sides of the tanh
    series' range.  Compared with the oracle for every row."""
    dev, dt, H, G = "cuda", torch.bfloat16, 4, 2
    for i, (T, window) in enumerate([(300, 64), (257, 65), (190, 63), (128, 1), (320, 200), (130, 1000), (200, None)]):
        cap = [30.0, 2.5][i % 2]
        seqs = [attention_inputs(T, H, G, D, D, dt, 30 + i + b, kind != "plain") for b in range(2)]
        r1, r2, pb = seqs[0][4:]
        buf = torch.zeros(2, T, (H + 2 * G) * D + 16, dtype=dt)
        for b, (q, k, v, *_) in enumerate(seqs):
            buf[b, :, : (H + 2 * G) * D] = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=-1)
        buf = buf.to(dev)
        view = lambda a, n: buf[..., a * D: (a + n) * D].unflatten(-1, (n, D)).permute(0, 2, 1, 3)      # noqa: E731
        gate = torch.stack([s[3] for s in seqs]).to(dev)
        gated = i % 3 != 1
        o = wa.window_attention_tc(view(0, H), view(H, G), view(H + G, G), D ** -0.5, window,
                                   gate=gate if gated else None, **attention_kw(kind, cap, r1, r2, pb, H, dev))
        for b, (q, k, v, g, *_) in enumerate(seqs):
            ref = oracle_attention(kind, q.to(F64), k.to(F64), v.to(F64), D ** -0.5, window, cap, r1.to(F64), r2.to(F64),
                                   pb.to(F64), g.to(F64) if gated else None)
            close(o[b].permute(1, 0, 2), ref, dt)


@pytest.mark.gpu
def test_tcgen05_sigmoid_attention_over_more_distances_than_the_bias_table_holds():
    dev, dt, H, G, D, T = "cuda", torch.bfloat16, 2, 1, 64, 4400
    q, k, v, gate, r1, r2, pb = attention_inputs(T, H, G, D, D, dt, 3)
    pb = pb - 3.0
    for window in (None, 4200, 4096):
        o = wa.window_attention_tc(q.to(dev).permute(1, 0, 2)[None], k.to(dev).permute(1, 0, 2)[None],
                                   v.to(dev).permute(1, 0, 2)[None], D ** -0.5, window,
                                   **attention_kw("sigmoid", 8.0, r1, r2, pb, H, dev))[0].permute(1, 0, 2)
        for t in (0, 63, 4095, 4096, 4199, 4200, 4399):
            lo = max(0, t - window + 1) if window else 0
            kk, vv = k[lo: t + 1, 0].to(F64), v[lo: t + 1, 0].to(F64)
            dist = t - torch.arange(lo, t + 1, dtype=F64)
            for h in range(H):
                s = 8.0 * torch.tanh(kk @ q[t, h].to(F64) * D ** -0.5 / 8.0) - r1[h].to(F64) * torch.log(1 + r2[h].to(F64) * dist)
                close(o[t, h], torch.sigmoid(s + pb[h].to(F64)) @ vv, dt)


# ---- configuration, weights, cache -------------------------------------------------------------------------------------
def test_cache_holds_latent_rows_once_and_keys_and_values_of_their_own_sizes():
    cfg = tiny_tidavik()
    model = TidavikInferenceModel(cfg, InferenceConfig(batch_size=2, max_batch_size=2, seq_len=16, max_context_length=16))
    kc = model.init_kv_cache()
    a, m = cfg.layers[0].mixer, cfg.layers[1].mixer
    assert kc.layer(0)[0].shape == (2, a.kv_heads, 16, a.dim) and kc.layer(0)[1].shape == (2, a.kv_heads, 16, a.vdim)
    ck, cv = kc.layer(1)
    assert ck.shape == (2, 1, 16, m.kv_rank) and cv.data_ptr() == ck.data_ptr() and not kc.states
    n = sum(2 * 16 * (L.mixer.kv_rank if L.type == "latent_attention" else L.mixer.kv_heads * (L.mixer.dim + L.mixer.vdim))
            for L in cfg.layers)
    assert kc.bytes() == 4 * n


def test_checkpoint_names_round_trip_and_the_fused_projection_layout():
    cfg = tiny_tidavik()
    ic = InferenceConfig(batch_size=1, max_batch_size=1, seq_len=8, max_context_length=8)
    sd = O.random_weights(cfg.to_dict(), seed=4)
    model = TidavikInferenceModel(cfg, ic)
    missing, unexpected = model.load_state_dict(convert_tidavik_state_dict(sd, cfg), strict=False)
    assert not missing and not unexpected, (missing, unexpected)
    again = export_tidavik_state_dict(model)
    assert set(again) == set(sd) and "l2.mix.q.norm" in again and "l0.mix.r1" not in again and "l1.mlp.up" not in again
    for k in sd:
        assert torch.equal(again[k].float(), sd[k]), k
    assert TidavikConfig.from_dict(cfg.to_dict(), torch.float32).to_dict() == cfg.to_dict()
    for L in cfg.layers:                                            # every part of the fused projection starts aligned
        cols, n_out = in_proj_columns(L)
        assert n_out % 8 == 0 and all(at % 8 == 0 for at, _ in cols.values())
    with pytest.raises(ValueError):
        TidavikConfig.from_dict(config(layers=[layer("attention", heads=3, kv_heads=2)]))
    with pytest.raises(ValueError):
        TidavikConfig.from_dict(config(layers=[layer("attention", mlp={"kind": "moe"})]))
    with pytest.raises(ValueError):
        TidavikConfig.from_dict(config(layers=[{"type": "recurrent", "mixer": {}, "mlp": None}]))


# ---- the model through the framework -----------------------------------------------------------------------------------
@case
@pytest.mark.parametrize("kind", ["latent_attention", "attention", "attention_2"])
def test_each_mixer_as_the_only_layer(dev, dt, kind):
    """One layer without a feed-forward, whole prompt and token by token; the stream after the layer as well."""
    cfg = config(layers=[layer(kind, mlp=None)])
    toks = tokens_of(cfg, 40, 1)
    model, sd = build(cfg, dev, dt)
    streams, seen = [], []
    ref = O.forward(cfg, sd, toks, layer_outputs=streams)
    model.layer_probe = lambda i, x: seen.append(x.detach().to("cpu", F64)[0])
    check_rows(replay(model, [([{"id": "a", "tokens": toks, "want": list(range(40))}], ["a"])])["a"], ref, range(40), dt)
    close(seen[0], streams[0], dt, scale=2.0)
    model.layer_probe = None
    steps = [([{"id": "b", "tokens": [t], "want": [0]}], []) for t in toks]
    check_rows(replay(model, steps)["b"], ref, range(40), dt)


@case
@pytest.mark.parametrize("cfg", [config(), ODD], ids=["mixed", "odd"])
def test_prefill_matches_oracle_and_token_by_token_decoding(dev, dt, cfg):
    toks = tokens_of(cfg, 45, 1)
    model, sd = build(cfg, dev, dt, seed=2)
    streams, seen = [], []
    ref = O.forward(cfg, sd, toks, layer_outputs=streams)
    want = list(range(45))
    model.layer_probe = lambda i, x: seen.append(x.detach().to("cpu", F64))
    whole = replay(model, [([{"id": "a", "tokens": toks, "want": want}], ["a"])])["a"]
    model.layer_probe = None
    check_rows(whole, ref, want, dt)
    assert len(seen) == len(streams) == len(cfg["layers"])
    for got, exp in zip(seen, streams):
        close(got[0], exp, dt, scale=3.0)
    steps = [([{"id": "b", "tokens": toks[:1], "want": [0]}], [])]
    steps += [([{"id": "b", "tokens": [t], "want": [0]}], []) for t in toks[1:]]
    check_rows(replay(model, steps)["b"], ref, want, dt)


@case
@pytest.mark.parametrize("portion", [2, 5, 16, 70])
def test_portions_of_a_prompt(dev, dt, portion):
    cfg = config()
    n = 41 if portion < 70 else 150
    toks = tokens_of(cfg, n, 6)
    for paged in (False, True):
        model, sd = build(cfg, dev, dt, seq_len=160, paged=paged, pages=25 if paged else None, page_size=8)
        ref = O.forward(cfg, sd, toks)
        steps, places = [], []
        for lo in range(0, n, portion):
            part = toks[lo:lo + portion]
            steps.append(([{"id": "p", "tokens": part, "want": list(range(len(part)))}], []))
            places += list(range(lo, lo + len(part)))
        check_rows(replay(model, steps)["p"], ref, places, dt)


@case
def test_portions_of_requests_at_different_places(dev, dt):
    """Two requests continued in one step from different positions, by different numbers of tokens."""
    cfg = config()
    model, sd = build(cfg, dev, dt, lines=3, seq_len=96)
    a, b = tokens_of(cfg, 80, 3), tokens_of(cfg, 30, 4)
    ra, rb = O.forward(cfg, sd, a), O.forward(cfg, sd, b)
    steps = [([{"id": "a", "tokens": a[:50], "want": [49]}, {"id": "b", "tokens": b[:3], "want": [2]}], []),
             ([{"id": "b", "tokens": b[3:23], "want": [0, 19]}, {"id": "a", "tokens": a[50:57], "want": [0, 6]}], []),
             ([{"id": "a", "tokens": a[57:80], "want": [22]}, {"id": "b", "tokens": b[23:25], "want": [1]}], [])]
    got = replay(model, steps)
    check_rows(got["a"], ra, [49, 50, 56, 79], dt)
    check_rows(got["b"], rb, [2, 3, 22, 24], dt)


@case
def test_unequal_batch_equals_each_alone_and_lines_are_reused(dev, dt):
    cfg = config()
    model, sd = build(cfg, dev, dt, lines=3)
    lens = {"a": 1, "b": 30, "c": 13, "d": 22, "e": 2}
    toks = {k: tokens_of(cfg, n + 6, 10 + i) for i, (k, n) in enumerate(lens.items())}
    ref = {k: O.forward(cfg, sd, v) for k, v in toks.items()}
    first = [{"id": k, "tokens": toks[k][:lens[k]], "want": [lens[k] - 1]} for k in "abc"]
    steps = [(first, ["a"])]                                     # a one-token request ends at once: its line is free
    for s in range(3):
        steps.append(([{"id": k, "tokens": [toks[k][lens[k] + s]], "want": [0]} for k in "bc"], ["c"] if s == 2 else []))
    # two new requests take the lines that a and c gave back: stale keys lie in them
    steps.append(([{"id": k, "tokens": toks[k][:lens[k]], "want": [0, lens[k] - 1]} for k in "de"], []))
    for s in range(6):
        steps.append(([{"id": k, "tokens": [toks[k][lens[k] + s]], "want": [0]} for k in "de"], []))
    got = replay(model, steps)
    check_rows(got["a"], ref["a"], [0], dt)
    for k in "bc":
        check_rows(got[k], ref[k], [lens[k] - 1, lens[k], lens[k] + 1, lens[k] + 2], dt)
    for k in "de":
        check_rows(got[k], ref[k], [0, lens[k] - 1] + [lens[k] + s for s in range(6)], dt)


@case
def test_a_batch_of_many_rows_decodes_like_each_alone(dev, dt):
    """Nine and more rows take other projection kernels than a few rows do; a one-token prompt is part of the batch."""
    cfg = config(width=64)
    model, sd = build(cfg, dev, dt, lines=12, seq_len=48)
    lens = [1, 2, 30, 7, 8, 9, 19, 20, 11, 12, 23, 24]
    toks = [tokens_of(cfg, n + 4, 60 + i) for i, n in enumerate(lens)]
    ref = [O.forward(cfg, sd, t) for t in toks]
    steps = [([{"id": str(i), "tokens": t[:n], "want": [n - 1]} for i, (t, n) in enumerate(zip(toks, lens))], [])]
    for s in range(4):
        steps.append(([{"id": str(i), "tokens": [t[n + s]], "want": [0]} for i, (t, n) in enumerate(zip(toks, lens))], []))
    got = replay(model, steps)
    for i, n in enumerate(lens):
        check_rows(got[str(i)], ref[i], [n - 1] + [n + s for s in range(4)], dt)


@case
def test_long_decoding_over_a_small_page_pool(dev, dt):
    """85 decoded tokens after a prompt of 5 on pages of 8 rows from a pool that two lines could not both fill: every page
    border and every window's edge is crossed while decoding."""
    cfg = config()
    toks = tokens_of(cfg, 90, 4)
    model, sd = build(cfg, dev, dt, lines=2, paged=True, pages=14, page_size=8)
    ref = O.forward(cfg, sd, toks)
    steps = [([{"id": "x", "tokens": toks[:5], "want": [4]}], [])]
    steps += [([{"id": "x", "tokens": [t], "want": [0]}], []) for t in toks[5:]]
    check_rows(replay(model, steps)["x"], ref, list(range(4, 90)), dt)
    model.kv_cache.reset()                # the pages go back to the pool and a second request gets them in another order
    steps = [([{"id": "w", "tokens": toks[:9], "want": []}, {"id": "y", "tokens": toks[20:50], "want": [29]}], ["w"])]
    steps += [([{"id": "y", "tokens": [t], "want": [0]}], []) for t in toks[50:60]]
    check_rows(replay(model, steps)["y"], O.forward(cfg, sd, toks[20:60]), list(range(29, 40)), dt)


def planted(kind, size, **kw):
    """A one-layer model in which only token id 5 makes a key that every later query singles out: its embedding has a large
    entry in column W - 2, which the first key dimension reads; the first query dimension reads column W - 1, where the
    position vectors are nearly one for every token."""
    cfg = config(layers=[layer(kind, mlp=None, mask={"size": size}, **kw)])
    sd = O.random_weights(cfg, seed=3)
    W, m, x = cfg["width"], cfg["layers"][0]["mixer"], "l0.mix."
    sd["embed"] *= 0.2
    sd["embed"][:, W - 2:] = 0.0
    sd["embed"][:, W - 1] = 2.0
    sd["embed"][5, W - 2] = 8.0
    sd["embed.norm"][:], sd["l0.norm1"][:] = 1.0, 1.0
    D, H = m["dim"], m["heads"]
    if kind == "latent_attention":
        for n, col in (("dq", W - 1), ("dkv", W - 2)):
            sd[x + n] *= 0.3
            sd[x + n][0] = 0.0
            sd[x + n][0, col] = 4.0
        for h in range(H):
            for n in ("uq", "uk"):
                sd[x + n][h * D] = 0.0
                sd[x + n][h * D, 0] = 2.0
        sd[x + "uv"] *= 2.0
    else:
        sd[x + "q.b"][:], sd[x + "k.b"][:] = 0.0, 0.0
        for n, heads, col in (("q", H, W - 1), ("k", m["kv_heads"], W - 2)):
            sd[x + n] *= 0.3
            for h in range(heads):
                sd[x + n][h * D] = 0.0
                sd[x + n][h * D, col] = 4.0
        if kind == "attention":
            sd[x + "q.norm"][:], sd[x + "k.norm"][:] = 1.0, 1.0
            sd[x + "pb"][:] = -3.5
            sd[x + "r1"][:], sd[x + "r2"][:] = 0.25, 0.5
            sd[x + "v"] *= 3.0
    sd = {k: v.to(torch.bfloat16).float() for k, v in sd.items()}
    return cfg, sd


@case
@pytest.mark.parametrize("kind,size", [("latent_attention", 64), ("attention", 65), ("attention_2", 16), ("attention", 3)])
def test_a_key_just_inside_and_just_outside_the_window(dev, dt, kind, size):
    """The planted token moves the logits while it is inside the window (the oracle says by how much) and not at all from
    the first position behind it: in a prompt, in a portion at an offset, and while decoding, at places on both sides of
    tile and page borders."""
    kw = dict(scale=0.5) if kind == "latent_attention" else dict(scale=0.6, softcap=12.0)
    cfg, sd = planted(kind, size, **kw)
    n, at = 180, 63
    toks = [t if t != 5 else 6 for t in tokens_of(cfg, n, 9)]
    moved = list(toks)
    toks[at] = 5
    ref, other = O.forward(cfg, sd, toks), O.forward(cfg, sd, moved)
    inside, outside = at + size - 1, at + size
    assert rel_err(other[inside].float(), ref[inside]) > 0.3
    assert rel_err(other[outside], ref[outside]) < 1e-12
    places = sorted({0, 1, at, at + 1, inside - 1, inside, outside, outside + 1})
    for paged in (False, True):
        model, _ = build(cfg, dev, dt, sd=sd, seq_len=192, lines=2, paged=paged, pages=30 if paged else None, page_size=16)
        got = replay(model, [([{"id": "w", "tokens": toks, "want": places}], ["w"])])["w"]
        check_rows(got, ref, places, dt)
        cut = inside                                          # portions that end and start at the edge
        steps = [([{"id": "p", "tokens": toks[:cut], "want": []}], []),
                 ([{"id": "p", "tokens": toks[cut: cut + 4], "want": [0, 1, 2]}], ["p"])]
        check_rows(replay(model, steps)["p"], ref, [inside, outside, outside + 1], dt)
        start = inside - 2                                    # the window passes over the planted token while decoding
        steps = [([{"id": "d", "tokens": toks[:start], "want": []}], [])]
        steps += [([{"id": "d", "tokens": [t], "want": [0]}], []) for t in toks[start: start + 6]]
        check_rows(replay(model, steps)["d"], ref, range(start, start + 6), dt)


@case
def test_the_one_in_the_denominator_and_the_gate_show_at_the_first_token(dev, dt):
    """The first token sees only itself: without the added one its weight would be 1."""
    cfg = config(layers=[layer("attention_2", mlp=None)])
    sd = O.random_weights(cfg, seed=6)
    sd["l0.mix.q.b"][:], sd["l0.mix.k.b"][:] = 0.0, 0.0
    toks = tokens_of(cfg, 3, 2)
    ref = O.forward(cfg, sd, toks)
    m = cfg["layers"][0]["mixer"]
    x = O.embed({k: v.to(F64) for k, v in sd.items()}, toks, 1e-5)
    w = {k: v.to(F64) for k, v in sd.items()}
    h = O.rms(x, 1e-5)[:1] * w["l0.norm1"]
    v = O.rms((h @ w["l0.mix.v"].T + w["l0.mix.v.b"]).reshape(1, m["kv_heads"], m["vdim"]), 1e-5)
    full = v.repeat_interleave(m["heads"] // m["kv_heads"], dim=1).reshape(1, -1) @ w["l0.mix.o"].T + w["l0.mix.o.b"]
    no_one = (O.rms(x[:1] + full, 1e-5) * w["final.norm"]) @ w["head"].T
    assert rel_err(no_one[0], ref[0]) > 0.15
    model, _ = build(cfg, dev, dt, sd=sd)
    check_rows(replay(model, [([{"id": "a", "tokens": toks, "want": [0, 1, 2]}], ["a"])])["a"], ref, range(3), dt)
    steps = [([{"id": "b", "tokens": [t], "want": [0]}], []) for t in toks]
    check_rows(replay(model, steps)["b"], ref, range(3), dt)


BIG = config(layers=[
    layer("attention", mlp={"kind": "dense", "ff": 96}, heads=2, kv_heads=1, dim=128, vdim=128, scale=0.09, softcap=20.0, mask={"size": 70}),
    layer("latent_attention", mlp=None, heads=2, dim=64, vdim=64, q_rank=48, kv_rank=128, scale=0.125, mask={"size": 90}),
    layer("attention_2", mlp={"kind": "dense", "ff": 80}, heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125, softcap=50.0, mask={"size": 129}),
    layer("latent_attention", heads=3, dim=32, vdim=48, q_rank=64, kv_rank=256, scale=0.2, mask={"size": 64}),
    layer("attention", mlp=None, heads=4, kv_heads=2, dim=96, vdim=96, scale=0.1, softcap=30.0, mask={"size": 33}),
], width=64, vocab=80)


@case
def test_sizes_of_the_tensor_core_kernels_through_the_model(dev, dt):
    """Head sizes of the tensor-core kernels (in bf16: tcgen05 for prompts from position 0 with sizes 64 and 128, mma.sync
    for the others and for the portion, latent rows of 128 and 256), prompts of 70 and 200 tokens in one batch, a portion at
    an offset, decoding."""
    model, sd = build(BIG, dev, dt, lines=2, seq_len=256)
    a, b = tokens_of(BIG, 246, 51), tokens_of(BIG, 80, 52)
    ra, rb = O.forward(BIG, sd, a), O.forward(BIG, sd, b)
    pa = [0, 1, 47, 63, 64, 127, 128, 129, 199]
    steps = [([{"id": "a", "tokens": a[:200], "want": pa}, {"id": "b", "tokens": b[:70], "want": [0, 69]}], []),
             ([{"id": "a", "tokens": a[200:240], "want": [0, 39]}], [])]
    steps += [([{"id": "a", "tokens": [a[240 + s]], "want": [0]}, {"id": "b", "tokens": [b[70 + s]], "want": [0]}], [])
              for s in range(6)]
    got = replay(model, steps)
    check_rows(got["a"], ra, pa + [200, 239] + list(range(240, 246)), dt)
    check_rows(got["b"], rb, [0, 69] + list(range(70, 76)), dt)


@case
def test_greedy_generation_through_generate_and_the_continuous_batcher(dev, dt):
    cfg = config()
    sd = O.random_weights(cfg, seed=5)
    prompts = [tokens_of(cfg, n, 20 + n) for n in (7, 12, 3)]
    want = [O.greedy(cfg, sd, p, 6) for p in prompts]
    model, _ = build(cfg, dev, dt, lines=3, sd=sd)
    T = max(len(p) for p in prompts)
    ids = torch.zeros(3, T, dtype=torch.long)
    mask = torch.zeros(3, T, dtype=torch.long)
    for b, p in enumerate(prompts):
        ids[b, :len(p)], mask[b, :len(p)] = torch.tensor(p), 1
    out = model.generate(ids.to(dev), mask.to(dev), max_new_tokens=6)
    strict = dt == torch.float32
    best = [O.forward(cfg, sd, p)[-1].topk(3).indices.tolist() for p in prompts]      # bf16 may swap near-equal logits
    for b, p in enumerate(prompts):
        got = out[b, len(p):len(p) + 6].tolist()
        assert got == want[b] or not strict, (got, want[b])
        assert got[0] in best[b]
    from neuronx_distributed_llama3_2_b200.inference.continuous_batching import ContinuousBatcher

    model2, _ = build(cfg, dev, dt, lines=2, sd=sd, paged=True, pages=9, page_size=4, seq_len=32)
    cb = ContinuousBatcher(model2)
    rids = [cb.submit(torch.tensor(p), 6) for p in prompts]
    res = cb.run()
    for rid, w, top3 in zip(rids, want, best):
        assert res[rid][:6] == w or not strict, (res[rid], w)
        assert res[rid][0] in top3


@case
def test_runner_buckets_match_oracle_greedy(dev, dt):
    from neuronx_distributed_llama3_2_b200.inference import TidavikRunner

    cfg = config()
    sd = O.random_weights(cfg, seed=12)
    tc = TidavikConfig.from_dict(cfg, torch_dtype=dt)
    ic = InferenceConfig(batch_size=3, max_context_length=32, seq_len=64, buckets=[16, 32], max_new_tokens=5,
                         use_cuda_graphs=dev == "cuda")
    runner = TidavikRunner(tc, ic, checkpoint_loader=lambda: convert_tidavik_state_dict(sd, tc), device=torch.device(dev))
    runner.trace()
    prompts = [tokens_of(cfg, n, 40 + n) for n in (11, 5)]
    ids = torch.zeros(2, 11, dtype=torch.long)
    mask = torch.zeros(2, 11, dtype=torch.long)
    for b, p in enumerate(prompts):
        ids[b, :len(p)], mask[b, :len(p)] = torch.tensor(p), 1
    out = runner.generate(ids.to(dev), mask.to(dev), max_new_tokens=5)
    runner.close()
    for b, p in enumerate(prompts):
        w = O.greedy(cfg, sd, p, 5)
        got = out[b, len(p):len(p) + 5].tolist()
        assert got[0] in O.forward(cfg, sd, p)[-1].topk(3).indices.tolist()
        assert got == w or dt != torch.float32, (got, w)


def test_registry_and_command_line_replay(tmp_path):
    """``bin/trace_run`` on a model directory: family chosen from config.json, steps on stdin, logits in files."""
    from safetensors.torch import save_file

    from neuronx_distributed_llama3_2_b200.inference.registry import families

    assert "tidavik" in families()
    cfg = json.loads(json.dumps(ODD))
    sd = O.random_weights(cfg, seed=8)
    mdir = tmp_path / "model"
    mdir.mkdir()
    (mdir / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in sd.items()}, str(mdir / "model.safetensors"))
    toks = tokens_of(cfg, 20, 3)
    steps = [{"step": 0, "entries": [{"id": "r", "tokens": toks[:15], "want": [0, 14]}], "end": []},
             {"step": 1, "entries": [{"id": "r", "tokens": toks[15:16], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "r", "tokens": toks[16:17], "want": [0]}], "end": ["r"]}]
    out = tmp_path / "out"
    env = dict(os.environ, CUDA_VISIBLE_DEVICES="")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(mdir), "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, env=env, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [ln for ln in p.stdout.split("\n") if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (out / "1.f32").exists()
    ref = O.forward(cfg, sd, toks)
    import numpy as np

    a = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, cfg["vocab"]))
    b = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(1, cfg["vocab"]))
    check_rows([a[0], a[1], b[0]], ref, [0, 14, 16], torch.float32)
