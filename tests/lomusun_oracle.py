"""Plain, slow restatement of the Lomusun design, one function per mechanism, straight from its equations.  It shares no code with the
package: dense tensors, whole sequences from their first token, Python loops over tokens, heads and experts; ``float64`` by default so that
it can serve as ground truth.

A model is ``(cfg, sd)``: ``cfg`` the parsed ``config.json`` (keys ``layers``, ``norm.eps``, ``max_positions``, ``vocab``, ``width``), ``sd`` a
dict name -> tensor.  ``forward(..., faults={...})`` plants a named mistake, so that a test can show that the mistake would be seen."""
import math

import torch


# ---------------------------------------------------------------------------------------------------------------- small pieces
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def unit(x, scale=1.0):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6) * scale


def sub(sd, prefix):
    return {k[len(prefix):]: v for k, v in sd.items() if k.startswith(prefix)}


def short_conv(u, w, lost_before=0):
    """``u`` [T, C], ``w`` [C, taps] (last column = the current token), no bias, zeros before the start.  ``lost_before``: a planted mistake,
    the inputs in front of this token are forgotten when it is reached."""
    T, C = u.shape
    K = w.shape[1]
    out = torch.zeros(T, C, dtype=u.dtype)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0 and not (lost_before and s < lost_before <= t):
                out[t] = out[t] + w[:, j] * u[s]
    return out


# ---------------------------------------------------------------------------------------------------------------- attention
def visible(T, size):
    """[query, key]: the last ``size`` positions up to the query's own (0: all of them)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (size == 0))


def slopes(H, dtype=torch.float64):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=dtype)


def bucket(n, rows, far):
    """Row of the distance table for a key ``n`` tokens back: one row per distance in the first half, logarithmically wider ones behind it."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def attend(q, k, v, scale, size, bias=None, sink=None):
    """``q`` [T, H, D], ``k`` [T, G, D], ``v`` [T, G, V]; ``bias`` [H, T] = what is added to the score of a key so many tokens back;
    ``sink`` [H] = score of a term without key and value.  Returns [T, H, V]."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = visible(T, size)
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias[h][back]
        s = s.masked_fill(~seen, float("-inf"))
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.clamp(top, min=float(sink[h]))
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - top)
        out[:, h] = (e / den) @ v[:, g]
    return out


def window_attention(h, p, m, eps, faults=()):
    """Sliding window with a slope per head, a sink, norms over the whole query and key rows, and a gate per element."""
    f = dict(faults)
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k = h @ p["q"].T, h @ p["k"].T
    if f.get("norm_per_head"):
        q, k = rms(q.view(T, H, D), eps).reshape(T, -1) * p["q.norm"], rms(k.view(T, G, D), eps).reshape(T, -1) * p["k.norm"]
    else:
        q, k = rms(q, eps) * p["q.norm"], rms(k, eps) * p["k.norm"]
    bias = -slopes(H)[:, None].to(h.dtype) * torch.arange(T, dtype=h.dtype)[None, :] * f.get("slope", 1.0)
    sink = None if f.get("no_sink") else p["sink"]
    o = attend(q.view(T, H, D), k.view(T, G, D), (h @ p["v"].T).view(T, G, V), float(m["scale"]), int(m["mask"]["size"]) if m.get("mask") else 0, bias, sink)
    return (o.reshape(T, H * V) * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def attention_mixer(h, p, m, kv=None, faults=()):
    """Convolved queries, keys and values, learned bias per distance bucket, a gate per head.  ``kv``: keys and values of another layer.
    Returns ``(mixer output, (keys, values))``."""
    f = dict(faults)
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    lost = f.get("conv_lost_before", 0)
    q = short_conv(h @ p["q"].T, p["q.conv"], lost)
    if kv is None:
        kv = short_conv(h @ p["k"].T, p["k.conv"], lost).view(T, G, D), short_conv(h @ p["v"].T, p["v.conv"], lost).view(T, G, V)
    rows, far = p["rel"].shape[0], int(m["bias_max"])
    bias = torch.stack([p["rel"][bucket(n + f.get("bucket_shift", 0), rows, far)] for n in range(T)]).T
    if f.get("no_bias"):
        bias = bias * 0.0
    o = attend(q.view(T, H, D), kv[0], kv[1], float(m["scale"]), int(m["mask"]["size"]) if m.get("mask") else 0, bias)
    o = o * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(T, H * V) @ p["o"].T, kv


# ---------------------------------------------------------------------------------------------------------------- gated delta rule
def delta_rule(q, k, v, beta, g, lost_before=0):
    """Per head ``S <- g S``, ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q``.  ``q, k`` [T, H, D], ``v`` [T, H, V], ``beta, g`` [T, H].
    ``lost_before``: a planted mistake, the state is set to zero before this token."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(D, v.shape[2], dtype=q.dtype)
        for t in range(T):
            if lost_before and t == lost_before:
                S = torch.zeros_like(S)
            S = g[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + torch.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
    return out


def delta_mixer(h, p, m, eps, faults=()):
    f = dict(faults)
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    lost = f.get("conv_lost_before", 0)
    q, k, v = (silu(short_conv(h @ p[n].T, p[n + ".conv"], lost)) for n in ("q", "k", "v"))
    q, k, v = unit(q.view(T, G, D), D ** -0.5), unit(k.view(T, G, D)), v.view(T, H, V)
    rep = H // G
    q, k = q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1)
    beta = torch.sigmoid(h @ p["b"].T)
    g = torch.exp(-torch.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    o = delta_rule(q, k, v, beta, g, f.get("lost_before", 0))
    o = rms(o, eps) * p["norm"] * silu(h @ p["g"].T).view(T, H, V)
    return o.reshape(T, H * V) @ p["o"].T


# ---------------------------------------------------------------------------------------------------------------- experts
def expert(h, p, limit):
    g = torch.clamp(h @ p["gate"].T, max=limit)
    u = torch.clamp(h @ p["up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ p["down"].T


def route(z, correction, top, scale):
    """Scores ``sigmoid(z)``; the ``top`` largest ``score + correction`` are chosen, weighted by their scores' share of their sum, times ``scale``.
    Returns ``(chosen experts per token, weights)``."""
    s = torch.sigmoid(z)
    idx = torch.argsort(s + correction, dim=-1, descending=True, stable=True)[:, :top]
    w = torch.gather(s, 1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20) * scale


def moe(h, p, mlp, faults=()):
    f = dict(faults)
    r, limit = mlp["router"], float(mlp["expert"]["limit"]) * f.get("limit", 1.0)
    corr = p["correction"] * f.get("correction", 1.0)
    idx, w = route(h @ p["router"].T, corr, int(r["top"]), float(r["scale"]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, x in zip(idx[t].tolist(), w[t]):
            out[t] = out[t] + x * expert(h[t:t + 1], sub(p, f"e{e}."), limit)[0]
    return out


# ---------------------------------------------------------------------------------------------------------------- the stack
def forward(cfg, sd, tokens, layers_out=None, dtype=torch.float64, faults=()):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` receives the residual after every layer.  ``faults``: planted mistakes by name
    (``norm_per_head``, ``slope``, ``no_sink``, ``conv_lost_before``, ``bucket_shift``, ``no_bias``, ``lost_before``, ``limit``, ``correction``,
    ``no_positions``, ``own_kv``, ``sequential``)."""
    f = dict(faults)
    w = {k: v.detach().cpu().to(dtype) for k, v in sd.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens)]
    if not f.get("no_positions"):
        x = x + w["pos"][:len(tokens)]
    kvs = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = sub(w, f"l{i}."), L["mixer"]
        mix = sub(p, "mix.")
        h = rms(x, eps) * p["norm1"]
        if L["type"] == "parallel":
            y = float(m["left_scale"]) * window_attention(h, sub(mix, "left."), m["left"], eps, faults) + \
                float(m["right_scale"]) * delta_mixer(h, sub(mix, "right."), m["right"], eps, faults)
        else:
            src = m.get("kv_from")
            y, kvs[i] = attention_mixer(h, mix, m, None if src is None else kvs[f.get("kv_from", src)], faults)
        if L.get("mlp"):
            if f.get("sequential"):
                x = x + y
                y, h = 0.0, rms(x, eps) * p["norm1"]
            y = y + moe(h, sub(p, "mlp."), L["mlp"], faults)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T
