"""A plain restatement of the Mumazen design, one function per mechanism, whole sequences at a time (float64 unless a
dtype is given).  It shares no code with the package: the tests compare the framework's step function, cache / state
manager and kernels with it.

Checkpoint names: ``embed``, ``loop.step``, ``final.norm``, ``head`` and per layer ``l<i>.norm1 / norm2 / ls1 / ls2``,
``l<i>.mix.<name>``, ``l<i>.mlp.<name>``.  Linear weights are ``[out, in]``.
"""
import math

import torch

F64 = torch.float64
GLU_SLOPE = 1.702


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def rotate(x, pos, rot):
    """``x [T, heads, D]`` at positions ``pos [T]``: dimensions ``i`` and ``i + dims/2`` of the first ``dims`` turn by
    ``p * base ** (-2 i / dims) / factor``."""
    if not rot or not rot.get("dims"):
        return x
    dims = rot["dims"]
    half = dims // 2
    f = torch.as_tensor(float(rot["base"]), dtype=x.dtype) ** (-2.0 * torch.arange(half, dtype=x.dtype) / dims)
    if rot.get("scaling"):
        f = f / float(rot["scaling"]["factor"])
    ang = pos.to(x.dtype).reshape(-1, 1) * f.reshape(1, -1)
    c, s = torch.cos(ang).unsqueeze(1), torch.sin(ang).unsqueeze(1)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def capped_attention(q, k, v, scale, cap):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, Dv]`` -> ``[T, H, Dv]``: causal softmax of ``cap tanh(scale q k / cap)``."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for t in range(T):
            s = (k[: t + 1, g] @ q[t, h]) * scale
            if cap:
                s = cap * torch.tanh(s / cap)
            e = torch.exp(s - s.max())
            out[t, h] = (e / e.sum()) @ v[: t + 1, g]
    return out


def attention_heads(h, w, m):
    """Gated heads ``[T, H * Dv]`` ahead of the output projection."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rotate((h @ w["q"].T).reshape(T, H, D), pos, m.get("rot"))
    k = rotate((h @ w["k"].T).reshape(T, G, D), pos, m.get("rot"))
    v = (h @ w["v"].T).reshape(T, G, Dv)
    o = capped_attention(q, k, v, m["scale"], m.get("softcap")).reshape(T, H * Dv)
    return o * torch.sigmoid(h @ w["g"].T)


def causal_conv(x, w, b):
    """``x [T, C]``, ``w [C, taps]`` (last column: the current token), zeros ahead of the first token."""
    T, C = x.shape
    taps = w.shape[1]
    out = torch.zeros(T, C, dtype=x.dtype)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out + b


def state_space_heads(x, B, C, dt, a_log, d):
    """One decay per head: ``x [T, H, P]``, ``B, C [T, G, N]``, ``dt [T, H]`` (after softplus) ->
    ``y_t = S_t^T C_t + D x_t`` with ``S_t = exp(-exp(a_log) dt) S + dt B x^T``."""
    T, H, P = x.shape
    G = B.shape[1]
    y = torch.zeros(T, H, P, dtype=x.dtype)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros(B.shape[2], P, dtype=x.dtype)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + d[h] * x[t, h]
    return y


def gated_group_norm(y, z, w, groups, eps):
    T, n = y.shape
    v = (y * silu(z)).reshape(T, groups, n // groups)
    return rms(v, eps).reshape(T, n) * w


def mamba2_heads(h, w, m, eps):
    """Normed heads ``[T, heads * vdim]`` ahead of the output projection."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    n = H * P
    u = h @ w["in"].T
    z, xbc, dt = u[:, :n], u[:, n: 2 * n + 2 * G * N], u[:, 2 * n + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :n].reshape(T, H, P), xbc[:, n: n + G * N].reshape(T, G, N), xbc[:, n + G * N:].reshape(T, G, N)
    y = state_space_heads(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return gated_group_norm(y.reshape(T, n), z, w["norm"], m["norm_groups"], eps)


def parallel_mixer(h, w, m, eps):
    left = attention_heads(h, sub(w, "left."), m["left"]) @ w["left.o"].T
    right = mamba2_heads(h, sub(w, "right."), m["right"], eps) @ w["right.o"].T
    return m["left_scale"] * left + m["right_scale"] * right


def selective_scan(x, dt, B, C, a_log, d):
    """One decay per channel and state: ``x, dt [T, C]``, ``B, C [T, N]``, ``a_log [C, N]``."""
    T, ch = x.shape
    A = -torch.exp(a_log)
    S = torch.zeros(ch, B.shape[1], dtype=x.dtype)
    y = torch.zeros(T, ch, dtype=x.dtype)
    for t in range(T):
        S = torch.exp(dt[t].unsqueeze(1) * A) * S + (dt[t] * x[t]).unsqueeze(1) * B[t]
        y[t] = S @ C[t] + d * x[t]
    return y


def mamba1_mixer(h, w, m):
    n, N, r = m["inner"], m["state"], m["dt_rank"]
    u = h @ w["in"].T
    x, z = silu(causal_conv(u[:, :n], w["conv"], w["conv.b"])), u[:, n:]
    p = x @ w["x"].T
    dt = softplus(p[:, :r] @ w["dt"].T + w["dt.b"])
    y = selective_scan(x, dt, p[:, r: r + N], p[:, r + N:], w["A_log"], w["D"])
    return (y * silu(z)) @ w["o"].T


def dense_feed_forward(h, w, limit):
    g = torch.clamp(h @ w["gate"].T + w["gate.b"], max=limit)
    u = torch.clamp(h @ w["up"].T + w["up.b"], min=-limit, max=limit)
    return (g * torch.sigmoid(GLU_SLOPE * g) * (u + 1.0)) @ w["down"].T + w["down.b"]


def expert(h, w):
    return torch.clamp(h @ w["up"].T, min=0.0).pow(2) @ w["down"].T


def route(h, w, m):
    """Chosen indices ``[T, top]``, their weights and the choice scores ``[T, outputs]``."""
    z = h @ w["router"].T
    s = torch.exp(z - z.max(dim=-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    choice = s + w["correction"]
    idx = torch.topk(choice, m["router"]["top"], dim=-1).indices
    p = s.gather(1, idx)
    return idx, p / (p.sum(-1, keepdim=True) + 1e-20), choice


def moe(h, w, m, margins=None):
    E, top = m["router"]["experts"], m["router"]["top"]
    idx, p, choice = route(h, w, m)
    if margins is not None and top < choice.shape[1]:
        ranked = choice.sort(dim=-1, descending=True).values
        margins.append(ranked[:, top - 1] - ranked[:, top])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(top):
            e = int(idx[t, j])
            out[t] += p[t, j] * (h[t] if e >= E else expert(h[t], sub(w, f"e{e}.")))
    if m.get("shared"):
        out = out + torch.sigmoid(h @ w["shared.sg"].reshape(-1)).unsqueeze(1) * expert(h, sub(w, "shared."))
    return out


def feed_forward(h, w, m, margins=None):
    return dense_feed_forward(h, w, m["limit"]) if m["kind"] == "dense" else moe(h, w, m, margins)


def layer_runs(config):
    """``(layer, pass)`` of every layer run in order; ``pass`` is the number of the loop's pass when the run is the first
    of one, else ``None``."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, None) for i in range(a)]
    for t in range(times):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(config, sd, tokens, dtype=F64, layer_outputs=None, margins=None):
    """Logits ``[T, vocab]`` of one sequence.  ``layer_outputs``: a list that receives the stream after every layer run;
    ``margins``: a list that receives the routers' per-token gaps between the last chosen and the first rejected score."""
    sd = {k: v.to(dtype) for k, v in sd.items() if v.is_floating_point()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x0 = sd["embed"][torch.as_tensor(tokens)] * config["embedding"]["scale"]
    x = x0
    for i, t in layer_runs(config):
        L, w = config["layers"][i], sub(sd, f"l{i}.")
        if t is not None:
            x = (x + x0 if t > 0 else x) + sd["loop.step"][t]
        h, mw = rms(x, eps) * w["norm1"], sub(w, "mix.")
        y = parallel_mixer(h, mw, L["mixer"], eps) if L["type"] == "parallel" else mamba1_mixer(h, mw, L["mixer"])
        x = x + m * (w["ls1"] * y)
        if L.get("mlp"):
            x = x + m * (w["ls2"] * feed_forward(rms(x, eps) * w["norm2"], sub(w, "mlp."), L["mlp"], margins))
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

    def mat(o, i, s=None):
        return bf(torch.randn(o, i, generator=g) * (s if s is not None else i ** -0.5))

    def vec(n, mean=0.0, s=0.1):
        return bf(mean + torch.randn(n, generator=g) * s)

    def uni(shape, lo, hi):
        return bf(lo + (hi - lo) * torch.rand(shape, generator=g))

    sd = {"embed": mat(V, W, 1.0 / cfg["embedding"]["scale"]), "final.norm": vec(W, 1.0), "head": mat(V, W)}
    if cfg.get("loop"):
        sd["loop.step"] = mat(cfg["loop"]["times"], W, 0.3)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        sd[p + "norm1"], sd[p + "ls1"] = vec(W, 1.0), vec(W, 0.9, 0.2)
        x = p + "mix."
        if L["type"] == "mamba1":
            n, N, r = m["inner"], m["state"], m["dt_rank"]
            sd[x + "in"], sd[x + "o"] = mat(2 * n, W), mat(W, n, 1.5 * n ** -0.5)
            sd[x + "conv"], sd[x + "conv.b"] = mat(n, m["conv"], 0.6), vec(n)
            sd[x + "x"], sd[x + "dt"], sd[x + "dt.b"] = mat(r + 2 * N, n, 2.0 * n ** -0.5), mat(n, r), uni((n,), -3.0, 0.0)
            sd[x + "A_log"], sd[x + "D"] = uni((n, N), -2.0, 2.0), vec(n, 1.0, 0.3)
        else:
            a, r = m["left"], m["right"]
            H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = x + "left."
            sd[q + "q"], sd[q + "k"] = mat(H * D, W, 1.5 * W ** -0.5), mat(G * D, W, 1.5 * W ** -0.5)
            sd[q + "v"], sd[q + "g"], sd[q + "o"] = mat(G * Dv, W), mat(H * Dv, W), mat(W, H * Dv)
            H, P, N, G = r["heads"], r["vdim"], r["state"], r["groups"]
            q = x + "right."
            sd[q + "in"], sd[q + "o"] = mat(2 * H * P + 2 * G * N + H, W), mat(W, H * P)
            C = H * P + 2 * G * N
            sd[q + "conv"], sd[q + "conv.b"] = mat(C, r["conv"], 0.6), vec(C)
            sd[q + "dt_bias"], sd[q + "A_log"], sd[q + "D"] = uni((H,), -3.0, 0.5), uni((H,), -2.0, 2.0), vec(H, 1.0, 0.3)
            sd[q + "norm"] = vec(H * P, 1.0, 0.2)
        mlp = L.get("mlp")
        if not mlp:
            continue
        sd[p + "norm2"], sd[p + "ls2"] = vec(W, 1.0), vec(W, 0.9, 0.2)
        y = p + "mlp."
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            sd[y + "gate"], sd[y + "up"], sd[y + "down"] = mat(F, W, 1.5 * W ** -0.5), mat(F, W), mat(W, F)
            sd[y + "gate.b"], sd[y + "up.b"], sd[y + "down.b"] = vec(F, 0.0, 0.4), vec(F, 0.0, 0.4), vec(W, 0.0, 0.3)
            continue
        F, R = mlp["expert"]["ff"], mlp["router"]["experts"] + int(mlp["router"].get("identity") or 0)
        sd[y + "router"], sd[y + "correction"] = mat(R, W, 2.0 * W ** -0.5), vec(R, 0.0, 0.1)
        for e in range(mlp["router"]["experts"]):
            sd[y + f"e{e}.up"], sd[y + f"e{e}.down"] = mat(F, W), mat(W, F)
        if mlp.get("shared"):
            Fs = mlp["shared"]["ff"]
            sd[y + "shared.up"], sd[y + "shared.down"], sd[y + "shared.sg"] = mat(Fs, W), mat(W, Fs), mat(1, W)
    return sd


def greedy(cfg, sd, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, sd, toks)[-1].argmax()))
    return toks[len(prompt):]


def close_calls(config, sd, tokens, gap=0.02):
    """Positions at which some router's last chosen score and the first one left out lie within ``gap``: rounding the
    router's input to 16 bits may legitimately choose the other expert there."""
    margins = []
    forward(config, sd, tokens, margins=margins)
    if not margins:
        return set()
    return set(torch.nonzero(torch.stack(margins).min(dim=0).values < gap).reshape(-1).tolist())
