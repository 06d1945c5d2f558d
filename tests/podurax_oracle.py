"""Plain, slow restatement of the Podurax design, one function per mechanism, straight from its equations.  It shares no code with the
package: dense tensors, whole sequences from their first token, Python loops over tokens and heads; ``float64`` by default so that it
can serve as ground truth.

A model is ``(cfg, sd)``: ``cfg`` the parsed ``config.json`` (keys ``layers``, ``norm.eps``, ``residual_mult``, ``embedding.scale``,
``vocab``, ``width``), ``sd`` a dict name -> tensor.  ``forward(..., faults={...})`` plants a named mistake, so that a test can show that
the mistake would be seen."""
import math

import torch


# ---------------------------------------------------------------------------------------------------------------- small pieces
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def sub(sd, prefix):
    return {k[len(prefix):]: v for k, v in sd.items() if k.startswith(prefix)}


# ---------------------------------------------------------------------------------------------------------------- selective scan
def short_conv_silu(u, w, b):
    """``u`` [T, C], ``w`` [C, taps] (last column = the current token), ``b`` [C]; zeros before the start."""
    T, C = u.shape
    K = w.shape[1]
    out = torch.zeros(T, C, dtype=u.dtype)
    for t in range(T):
        acc = b.clone()
        for j in range(K):
            if t - (K - 1) + j >= 0:
                acc = acc + w[:, j] * u[t - (K - 1) + j]
        out[t] = silu(acc)
    return out


def selective_scan(x, dt, A, B, C, D, lost_before=0):
    """``S <- exp(dt A) S + dt x B``, ``y = S C + D x`` per channel.  ``x, dt`` [T, inner], ``A`` [inner, N] (negative), ``B, C`` [T, N].
    ``lost_before``: a planted mistake, the state is set to zero before this token."""
    T, inner = x.shape
    S = torch.zeros(inner, A.shape[1], dtype=x.dtype)
    y = torch.zeros(T, inner, dtype=x.dtype)
    for t in range(T):
        if lost_before and t == lost_before:
            S = torch.zeros_like(S)
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba1_mixer(h, p, m, faults=()):
    inner, N, R = int(m["inner"]), int(m["state"]), int(m["dt_rank"])
    u = h @ p["in"].T
    x, z = u[:, :inner], u[:, inner:]
    x = short_conv_silu(x, p["conv"], p["conv.b"])
    dbc = x @ p["x"].T
    dt = softplus(dbc[:, :R] @ p["dt"].T + p["dt.b"])
    y = selective_scan(x, dt, -torch.exp(p["A_log"]), dbc[:, R:R + N], dbc[:, R + N:], p["D"], dict(faults).get("lost_before", 0))
    return (y * silu(z)) @ p["o"].T


# ---------------------------------------------------------------------------------------------------------------- attention
def yarn_freqs(rot):
    """Angles per position of the pairs of a partly rotated head, stretched between two rotation counts, and the factor on cos / sin."""
    n, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(f, dtype=torch.float64), 1.0
    where = lambda turns: n * math.log(float(s["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(float(s["fast"]))), 0), min(math.ceil(where(float(s["slow"]))), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / float(s["factor"]) * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(float(s["factor"])) + 1.0


def rotate_half(x, pos, freqs, mult):
    """Entry ``i`` is paired with ``i + n`` (``n`` = number of angles); the entries from ``2 n`` on stay.  ``x`` [T, heads, d]."""
    n = freqs.numel()
    a = pos.to(x.dtype)[:, None] * freqs.to(x.dtype)
    c, s = (torch.cos(a) * mult)[:, None, :], (torch.sin(a) * mult)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def visible(T, size, keep):
    """[query, key]: the last ``size`` positions up to the query's own and the first ``keep`` of the sequence."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep))


def attention_mixer(h, p, m, eps, v_first=None, faults=()):
    """Returns ``(mixer output, this layer's unmixed values)``."""
    f = dict(faults)
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ p["q"].T + p["q.b"]).view(T, H, D)
    k = (h @ p["k"].T + p["k.b"]).view(T, G, D)
    own = (h @ p["v"].T + p["v.b"]).view(T, G, V)
    pos = torch.arange(T)
    if m.get("rot"):
        fr, mult = yarn_freqs(m["rot"])
        q, k = rotate_half(q, pos, fr, f.get("rot_mult", mult)), rotate_half(k, pos, fr, f.get("rot_mult", mult))
    q, k = rms(q, eps), rms(k, eps)
    v = own
    if v_first is not None:
        lam = f.get("vmix", p["vmix"])
        v = (1.0 - lam) * own + lam * v_first
    mask = m.get("mask")
    seen = visible(T, int(mask["size"]), int(mask.get("keep_first", 0))) if mask else visible(T, T, 0)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = ((q[:, hd] @ k[:, g].T) * float(m["scale"])).masked_fill(~seen, float("-inf"))
        top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)                 # the sink's score is 0
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True) + torch.exp(-top) * f.get("sink", 1.0)
        out[:, hd] = (e / den) @ v[:, g]
    out = out * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return out.reshape(T, H * V) @ p["o"].T, own


# ---------------------------------------------------------------------------------------------------------------- the stack
def dense_ff(h, p):
    return (gelu_tanh(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def forward(cfg, sd, tokens, layers_out=None, dtype=torch.float64, faults=()):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` receives the residual after every layer.  ``faults``: planted mistakes by
    name (``vmix``, ``sink``, ``rot_mult``, ``lost_before``)."""
    w = {k: v.detach().cpu().to(dtype) for k, v in sd.items()}
    eps, m = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = w["embed"][torch.tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    v_first = None
    for i, L in enumerate(cfg["layers"]):
        p = sub(w, f"l{i}.")
        h = rms(x, eps) * p["norm1"]
        if L["type"] == "mamba1":
            y = mamba1_mixer(h, sub(p, "mix."), L["mixer"], faults)
        else:
            mixes = bool(L["mixer"].get("v_mix"))
            y, own = attention_mixer(h, sub(p, "mix."), L["mixer"], eps, v_first if mixes else None, faults)
            if mixes and v_first is None:
                v_first = own
        x = x + m * y
        if L.get("mlp"):
            x = x + m * dense_ff(rms(x, eps) * p["norm2"], sub(p, "mlp."))
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T
