"""A plain restatement of the Tidavik design, one function per mechanism, whole sequences at a time (float64 unless a
dtype is given).  It shares no code with the package: the tests compare the framework's step function, cache manager and
kernels with it.

Checkpoint names: ``embed``, ``embed.norm``, ``final.norm``, ``head`` and per layer ``l<i>.norm1 / norm2``,
``l<i>.mix.<name>`` (a bias is ``<name>.b``, a norm weight ``<name>.norm``), ``l<i>.mlp.<name>``.  Linear weights are
``[out, in]``.
"""
import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def position_vectors(positions, width, dtype=F64):
    """``[T, width]``: entry ``2 i`` is ``sin(p f_i)``, entry ``2 i + 1`` is ``cos(p f_i)`` with ``f_i = 10000 ** (-2 i / width)``."""
    out = torch.zeros(len(positions), width, dtype=dtype)
    for c in range(width):
        ang = torch.as_tensor(positions, dtype=dtype) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.sin(ang) if c % 2 == 0 else torch.cos(ang)
    return out


def visible(T, window):
    """``[T, T]`` (query, key): ``0 <= i - j < window`` (no window: all earlier keys and the query's own)."""
    d = torch.arange(T).reshape(-1, 1) - torch.arange(T).reshape(1, -1)
    return (d >= 0) & ((d < window) if window else torch.ones_like(d, dtype=torch.bool))


def scores(q, k, scale, softcap=None, r1=None, r2=None):
    """``q [T, H, D]``, ``k [T, G, D]`` -> ``[H, T, T]``: scaled products, soft cap, logarithmic distance bias."""
    T, H, _ = q.shape
    G = k.shape[1]
    dist = (torch.arange(T).reshape(-1, 1) - torch.arange(T).reshape(1, -1)).clamp(min=0).to(q.dtype)
    out = torch.zeros(H, T, T, dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if r1 is not None:
            s = s - r1[h] * torch.log(1.0 + r2[h] * dist)
        out[h] = s
    return out


def softmax_weights(s, vis, extra_one=False):
    """Softmax over the visible keys; ``extra_one``: one is added to the denominator."""
    s = s.masked_fill(~vis, float("-inf"))
    m = s.max(dim=-1, keepdim=True).values
    if extra_one:
        m = torch.clamp(m, min=0.0)
    e = torch.exp(s - m)
    den = e.sum(-1, keepdim=True)
    if extra_one:
        den = den + torch.exp(-m)
    return e / den


def sigmoid_weights(s, vis, pb):
    """Independent weights, not normalised over the keys: ``sigmoid(s + pb_h)``."""
    return torch.sigmoid(s + pb.reshape(-1, 1, 1)).masked_fill(~vis, 0.0)


def weighted_values(p, v):
    """``p [H, T, T]``, ``v [T, G, Dv]`` -> ``[T, H, Dv]``."""
    H, G = p.shape[0], v.shape[1]
    return torch.stack([p[h] @ v[:, h // (H // G)] for h in range(H)], dim=1)


def latent_mixer(h, w, m, eps):
    """Keys and values are up-projections of a small normalised row per token; queries go through a normalised row of
    their own; softmax in a window; one output gate number per head."""
    T = h.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    cq = rms(h @ w["dq"].T, eps) * w["dq.norm"]
    c = rms(h @ w["dkv"].T, eps) * w["dkv.norm"]
    q = (cq @ w["uq"].T).reshape(T, H, D)
    k, v = (c @ w["uk"].T).reshape(T, H, D), (c @ w["uv"].T).reshape(T, H, Dv)
    p = softmax_weights(scores(q, k, m["scale"]), visible(T, (m.get("mask") or {}).get("size")))
    o = weighted_values(p, v) * torch.sigmoid(h @ w["g"].T).unsqueeze(-1)
    return o.reshape(T, H * Dv) @ w["o"].T


def sigmoid_mixer(h, w, m, eps):
    """Biased projections, whole-projection norm of q and k, soft cap, logarithmic distance bias, sigmoid weights."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ w["q"].T + w["q.b"], eps) * w["q.norm"]
    k = rms(h @ w["k"].T + w["k.b"], eps) * w["k.norm"]
    v = h @ w["v"].T + w["v.b"]
    s = scores(q.reshape(T, H, D), k.reshape(T, G, D), m["scale"], m["softcap"], w["r1"], w["r2"])
    p = sigmoid_weights(s, visible(T, (m.get("mask") or {}).get("size")), w["pb"])
    return weighted_values(p, v.reshape(T, G, Dv)).reshape(T, H * Dv) @ w["o"].T + w["o.b"]


def capped_mixer(h, w, m, eps):
    """Biased projections, unit-RMS values per head, soft cap, softmax with one added to the denominator."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, D)
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, D)
    v = rms((h @ w["v"].T + w["v.b"]).reshape(T, G, Dv), eps)
    p = softmax_weights(scores(q, k, m["scale"], m["softcap"]), visible(T, (m.get("mask") or {}).get("size")),
                        extra_one=True)
    return weighted_values(p, v).reshape(T, H * Dv) @ w["o"].T + w["o.b"]


MIXERS = {"latent_attention": latent_mixer, "attention": sigmoid_mixer, "attention_2": capped_mixer}


def feed_forward(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def embed(sd, tokens, eps):
    x = sd["embed"][torch.as_tensor(tokens)]
    x = x + position_vectors(list(range(len(tokens))), x.shape[1], x.dtype)
    return rms(x, eps) * sd["embed.norm"]


def forward(config, sd, tokens, dtype=F64, layer_outputs=None):
    """Logits ``[T, vocab]`` of one sequence.  ``layer_outputs``: a list that receives the stream after every layer."""
    sd = {k: v.to(dtype) for k, v in sd.items() if v.is_floating_point()}
    eps = config["norm"]["eps"]
    x = embed(sd, tokens, eps)
    for i, L in enumerate(config["layers"]):
        w = sub(sd, f"l{i}.")
        x = x + MIXERS[L["type"]](rms(x, eps) * w["norm1"], sub(w, "mix."), L["mixer"], eps)
        if L.get("mlp"):
            x = x + feed_forward(rms(x, eps) * w["norm2"], sub(w, "mlp."))
        if layer_outputs is not None:
            layer_outputs.append(x)
    return (rms(x, eps) * sd["final.norm"]) @ sd["head"].T


def random_weights(cfg, seed=0, dtype=torch.float32):
    """A checkpoint of the design with weights that keep activations of order one through the layers (values that are
    exact in bfloat16, so that a bfloat16 model holds the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def bf(t):
        return t.to(torch.bfloat16).to(dtype)

    def mat(o, i, s=1.0):
        return bf(torch.randn(o, i, generator=g) * s * i ** -0.5)

    def vec(n, mean=0.0, s=0.1):
        return bf(mean + torch.randn(n, generator=g) * s)

    sd = {"embed": mat(V, W, W ** 0.5), "embed.norm": vec(W, 1.0), "final.norm": vec(W, 1.0), "head": mat(V, W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        sd[p + "norm1"] = vec(W, 1.0)
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        x = p + "mix."
        if L["type"] == "latent_attention":
            R, Q = m["kv_rank"], m["q_rank"]
            sd[x + "dq"], sd[x + "dq.norm"], sd[x + "uq"] = mat(Q, W), vec(Q, 1.0, 0.2), mat(H * D, Q, 1.5)
            sd[x + "dkv"], sd[x + "dkv.norm"] = mat(R, W), vec(R, 1.0, 0.2)
            sd[x + "uk"], sd[x + "uv"] = mat(H * D, R, 1.5), mat(H * Dv, R)
            sd[x + "g"], sd[x + "o"] = mat(H, W, 1.5), mat(W, H * Dv)
        else:
            G = m["kv_heads"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                sd[x + n], sd[x + n + ".b"] = mat(rows, W, 1.5 if n != "v" else 1.0), vec(rows, 0.0, 0.5)
            sd[x + "o"], sd[x + "o.b"] = mat(W, H * Dv), vec(W, 0.0, 0.3)
            if L["type"] == "attention":
                sd[x + "q.norm"], sd[x + "k.norm"] = vec(H * D, 1.0, 0.3), vec(G * D, 1.0, 0.3)
                sd[x + "r1"], sd[x + "r2"] = vec(H, 0.8, 0.3), bf(0.2 + torch.rand(H, generator=g))
                sd[x + "pb"] = vec(H, -1.5, 0.5)
        if L.get("mlp"):
            F = L["mlp"]["ff"]
            sd[p + "norm2"] = vec(W, 1.0)
            sd[p + "mlp.gate"], sd[p + "mlp.up"], sd[p + "mlp.down"] = mat(F, W), mat(F, W), mat(W, F)
    return sd


def greedy(cfg, sd, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, sd, toks)[-1].argmax()))
    return toks[len(prompt):]
