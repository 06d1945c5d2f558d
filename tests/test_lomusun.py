"""Lomusun (parallel blocks: mixer and mixture of experts on one normed input, learned positions; windowed attention with a slope per head, a
sink, whole-row query / key norms and a gate per element BESIDE a gated delta rule with one decay per head; windowed attention with convolved
queries, keys and values, a learned bias per distance bucket, a gate per head, on keys and values of its own or of another layer) against the
plain oracle in ``lomusun_oracle.py``: every mechanism alone, prefill against token-by-token decoding, prompt portions down to two tokens,
ragged batches against each request alone, pages and state slots that are freed and used again, keys far away and just inside and just
outside the windows and the distance buckets, far tokens held only by the recurrent state, planted mistakes that must show, other sizes (one
key/value head and as many as query heads, values wider and narrower than keys, one to five convolution taps, no window, layers without
experts, all experts chosen), long decoding, and greedy generation through the engine.

Runs on the CPU with the unfused ops; the ``gpu`` variants run the same cases on the sm_100a kernels in fp32 and bf16.
"""
import copy
import json
import math
import os
import random
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import lomusun_oracle as oracle  # noqa: E402

from mlx_sharding_b200.config import ModelConfig  # noqa: E402
from mlx_sharding_b200.engine.core import LLMEngine  # noqa: E402
from mlx_sharding_b200.engine.sampler import SamplingParams  # noqa: E402
from mlx_sharding_b200.engine.trace import TraceSession  # noqa: E402
from mlx_sharding_b200.models import build_stage  # noqa: E402
from mlx_sharding_b200.models.lomusun import bucket_starts, distance_bias  # noqa: E402
from mlx_sharding_b200.ops import BatchMeta, LinearWeight, get_backend  # noqa: E402
from mlx_sharding_b200.parallel.pipeline import LocalPipeline, StageExecutor  # noqa: E402
from mlx_sharding_b200.utils.checkpoint import random_state_dict  # noqa: E402


def moe(experts, top, ff, scale=1.5, limit=0.8):
    return dict(kind="moe", router=dict(experts=experts, top=top, scale=scale), expert=dict(ff=ff, limit=limit))


def par(left, right, ls, rs, mlp):
    H, G, D, V, size, scale = left
    h, g, d, v, K = right
    m = dict(left=dict(dim=D, heads=H, kv_heads=G, scale=scale, vdim=V), left_scale=ls, right=dict(conv=K, dim=d, heads=h, kv_heads=g, vdim=v), right_scale=rs)
    if size:
        m["left"]["mask"] = dict(size=size)
    return dict(type="parallel", mixer=m, mlp=mlp)


def att(H, G, D, V, size, scale, K, far, mlp, kv_from=None):
    m = dict(bias_max=far, conv=K, dim=D, heads=H, kv_heads=G, scale=scale, vdim=V)
    if size:
        m["mask"] = dict(size=size)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m, mlp=mlp)


ROWS = {20: 8, 9: 6, 13: 5, 40: 16, 300: 32, 64: 12}        # distance-table rows by bias_max (a tensor shape, not configuration)
P_GQ = par((4, 2, 8, 12, 7, 0.8), (4, 2, 6, 10, 4), 1.2, 0.5, moe(6, 2, 24))              # two query heads per key/value head on both sides
P_ODD = par((3, 1, 10, 20, 9, 0.6), (3, 3, 5, 7, 1), -0.7, 2.0, None)                     # odd sizes, one key/value head, one tap, no experts
P_MH = par((2, 2, 16, 8, 16, 0.3), (6, 2, 16, 8, 2), 1.0, 1.0, moe(5, 5, 40, 0.7, 2.0))   # window = page, all experts, factors of 1
P_FREE = par((4, 4, 6, 5, 0, 0.5), (2, 1, 12, 4, 5), 0.8, 1.1, moe(3, 1, 21, 2.0, 0.4))   # no window
A_GQ = att(4, 2, 8, 12, 11, 0.5, 3, 20, moe(6, 3, 24, 1.0))
A_MQ = att(3, 1, 10, 20, 24, 0.4, 1, 9, None)                                             # one tap, table shorter than the window
A_FREE = att(2, 2, 16, 8, 0, 0.3, 5, 40, moe(4, 2, 33))                                   # no window
kv_of = lambda j, like, size, mlp=None, far=64, K=2, H=None: att(H or like["mixer"]["heads"], *(like["mixer"][k] for k in ("kv_heads", "dim", "vdim")), size, 0.6, K, far, mlp, j)
STACK = [A_GQ, P_GQ, kv_of(0, A_GQ, 5, moe(4, 1, 16)), P_ODD, A_MQ, kv_of(4, A_MQ, 30), kv_of(0, A_GQ, 26), P_MH]
CASES = {"par_gq": [P_GQ], "par_odd": [P_ODD], "par_mh": [P_MH], "par_free": [P_FREE], "att_gq": [A_GQ], "att_mq": [A_MQ], "att_free": [A_FREE],
         "att_shared": [A_GQ, kv_of(0, A_GQ, 4, moe(4, 2, 16)), kv_of(0, A_GQ, 17, None, 13, 1)], "stack": STACK}
DEVICES = [pytest.param("cpu", torch.float32, 2e-4, id="cpu"),
           pytest.param("cuda", torch.float32, 2e-4, id="b200-f32", marks=pytest.mark.gpu),
           pytest.param("cuda", torch.bfloat16, 6e-2, id="b200-bf16", marks=pytest.mark.gpu)]


def make_cfg(layers, width=48, vocab=96, eps=1e-3, positions=400):
    return dict(architecture="Lomusun", layers=copy.deepcopy(layers), max_positions=positions, norm=dict(eps=eps), vocab=vocab, width=width)


def make_model(cfgd, device="cpu", dtype=torch.float32, seed=3, edit=None):
    """In bf16 the corrections alone decide which experts are chosen (two units apart, scores lie in 0 .. 1), so no rounding flips a choice;
    the weights must still be the scores without them."""
    cfg = ModelConfig.from_dict(cfgd)
    sd = dict(random_state_dict(cfg, dtype=torch.bfloat16, seed=seed))
    g = torch.Generator().manual_seed(seed)
    for i, L in enumerate(cfg.layer_specs):
        if L["type"] == "attention":
            sd[f"l{i}.mix.rel"] = torch.randn(ROWS[int(L["mixer"]["bias_max"])], int(L["mixer"]["heads"]), generator=g).to(torch.bfloat16)
        if L["mlp"] and dtype == torch.bfloat16:
            sd[f"l{i}.mlp.correction"] = 2.0 * torch.randperm(int(L["mlp"]["router"]["experts"]), generator=g).to(torch.bfloat16)
    if edit:
        edit(sd)
    model = build_stage(cfg, None, dtype, device).load_state({k: v.clone() for k, v in sd.items()})
    return model, sd


def session(model, pages=12, page_size=16, live=4):
    return TraceSession(StageExecutor(model, pages, page_size, num_state_slots=live + 1), (pages - 1) * page_size, live)


def run_whole(model, tokens, **kw):
    return session(model, **kw).step([dict(id="a", tokens=tokens, want=list(range(len(tokens))))])


def toks(n, vocab=96, seed=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


SHOWS = 1e-2      # a fault must move the logits by this share of their largest: 50 times the exact-mode tolerance


def close(a, b, tol):
    a, b = a.float().cpu(), b.float().cpu()
    err = (a - b).abs().max().item() / max(1.0, b.abs().max().item())
    assert err < tol, f"relative error {err:.3e} >= {tol}"


def close_in_bf16(a, b, tol):
    """Stacks drawn at random: some amplify the rounding of bf16 at single positions (a short vector made a unit vector).  At most a tenth of the
    positions may be off by more than ``tol``, none by more than four times that."""
    a, b = a.float().cpu(), b.float().cpu()
    err = (a - b).abs().amax(-1) / max(1.0, b.abs().max().item())
    assert err.max() < 4 * tol and (err > tol).float().mean() <= 0.1, err.sort().values[-12:]


def in_portions(model, t, portions, **kw):
    s, at, got = session(model, **kw), 0, []
    for n in portions:
        got.append(s.step([dict(id="r", tokens=t[at:at + n], want=list(range(n)))]))
        at += n
    assert at == len(t)
    return torch.cat(got)


def decode_after(model, t, n_prompt, **kw):
    return in_portions(model, t, [n_prompt] + [1] * (len(t) - n_prompt), **kw)


def meta_of(lens, ctx, pages, page_size, device, slots=None):
    return BatchMeta.build(lens, ctx, pages, page_size, device=device, state_slots=slots)


def backend(device):
    return get_backend("b200" if device == "cuda" else "reference")


# ---------------------------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("case", list(CASES))
def test_mechanism_against_oracle(case, device, dtype, tol):
    """Each layer shape alone (and stacks): whole prompt, every position, the residual after every layer; 45 tokens span three pages."""
    cfgd = make_cfg(CASES[case])
    model, sd = make_model(cfgd, device, dtype)
    t = toks(45, seed=0)
    lo = []
    want = oracle.forward(cfgd, sd, t, layers_out=lo)
    got_layers = []
    s = session(model)
    tb = s.table
    tb.add(0), tb.reserve(0, len(t))
    meta = meta_of([len(t)], [0], [tb.pages[0]], 16, device, tb.state_slots([0]))
    got = model(torch.tensor(t, device=device), meta, s.stage.kv, all_logits=True, layer_out=got_layers)
    close(got, want, tol)
    for a, b in zip(got_layers, lo):
        close(a, b, tol)


@pytest.mark.parametrize("rows,far", [(8, 20), (16, 128), (32, 128), (2, 2), (6, 9), (5, 13), (16, 9), (12, 1000), (64, 33)])
def test_distance_buckets(rows, far):
    """Starts of the buckets (powers that are hit exactly, buckets without a distance of their own, odd numbers of rows, bias_max just above the
    linear half) against the oracle's logarithm at every distance; distances far behind the last bucket."""
    rel = torch.randn(rows, 3, generator=torch.Generator().manual_seed(rows))
    b = distance_bias(rel, far)
    starts = bucket_starts(rows, far)
    assert len(starts) == rows and starts[:rows // 2 + 1] == list(range(rows // 2 + 1)) and starts == sorted(starts) and b.shape[1] == starts[-1] + 1
    half, m = rows // 2, rows - rows // 2
    for n in range(far + 40):
        # the logarithm in doubles is off by parts in 1e16: where it is not that close to a whole number the bucket is certain
        x = 0.0 if n < half else math.log(n / half) / math.log(far / half) * m
        want = oracle.bucket(n, rows, far) if abs(x - round(x)) > 1e-9 else min(rows - 1, half + round(x)) if n >= half else n
        assert torch.equal(b[:, min(n, b.shape[1] - 1)], rel[want]), n
    with pytest.raises(ValueError):
        bucket_starts(8, 4)


def decays(dt, bias, A_log):
    return torch.exp(-torch.exp(A_log.double()) * oracle.softplus(dt.double() + bias.double()))


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("H,G,D,V,portions", [(4, 2, 6, 10, [13, 1, 9]), (3, 3, 5, 7, [2, 3, 1, 4, 5]), (2, 1, 128, 128, [40, 1, 2, 7]), (2, 2, 64, 40, [33, 1, 1]), (1, 1, 200, 16, [11, 1]),
                                              (4, 4, 33, 65, [1, 2, 30]), (8, 4, 16, 32, [70, 1, 5]), (2, 1, 300, 8, [9, 1]), (1, 1, 512, 4, [6, 1]), (1, 1, 530, 4, [6, 1]), (2, 1, 1, 3, [5, 1]),
                                              (64, 32, 24, 8, [17, 1]), (40, 8, 20, 128, [9, 1, 6]), (40, 4, 100, 131, [7, 2]), (40, 2, 130, 120, [6, 3]), (3, 1, 70, 6, [10])])
def test_delta_rule_alone(H, G, D, V, portions, device, dtype, tol):
    """The rule as an op: one sequence in portions that start inside a group of four tokens, the state carried in a dirty slot that must not be
    read at the first token; every lane layout of the kernels, sizes that are no multiple of 4, heads that share queries and keys."""
    O = backend(device)
    g = torch.Generator().manual_seed(H * 1000 + D)
    rn = lambda *s: torch.randn(*s, generator=g)
    T = sum(portions)
    qkv, bt, dt = rn(T, 2 * G * D + H * V).to(dtype), rn(T, H + 3).to(dtype), rn(T, H).to(dtype)
    bias, A_log = rn(H) - 1.0, torch.log(torch.rand(H, generator=g) + 0.02)
    x = qkv.double()
    q, k = oracle.unit(x[:, :G * D].view(T, G, D), D ** -0.5), oracle.unit(x[:, G * D:2 * G * D].view(T, G, D))
    want = oracle.delta_rule(q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1), x[:, 2 * G * D:].view(T, H, V), torch.sigmoid(bt[:, :H].double()),
                             decays(dt, bias, A_log)).view(T, H * V)
    dev = lambda v: v.to(device)
    st = torch.full((4, H, D, V), float("nan"), device=device)
    at, got = 0, []
    for n in portions:
        sl = slice(at, at + n)
        got.append(O.delta_scan(dev(qkv[sl]), dev(bt)[sl, :H], dev(dt[sl]), dev(bias), dev(A_log), st, meta_of([n], [at], [[1] * 10], 16, device, [2]), H, G, D, V, D ** -0.5))
        at += n
    close(torch.cat(got), want, 2e-5)
    assert torch.isnan(st[[0, 1, 3]]).all()          # other slots untouched


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 12, 16), (3, 1, 7, 9)])
def test_delta_rule_ragged(H, G, D, V, device, dtype, tol):
    """Sequences of 1, 7, 50, 0, 2 and 4 tokens in one step (some new, some with a state), then a step of single tokens; decays that underflow to
    zero in between; the states afterwards."""
    O = backend(device)
    g = torch.Generator().manual_seed(11)
    rn = lambda *s: torch.randn(*s, generator=g)
    lens, ctx0, slots = [1, 7, 50, 0, 2, 4], [0, 3, 0, 5, 9, 0], [2, 5, 1, 4, 3, 6]
    bias, A_log = rn(H) - 1.0, torch.log(torch.rand(H, generator=g) + 0.02)
    S0 = rn(7, H, D, V)
    st, ref = S0.clone().to(device), S0.double().clone()
    dev = lambda v: v.to(device)
    ctx = list(ctx0)
    for ln in (lens, [1] * 6):
        T = sum(ln)
        qkv, bt, dt = rn(T, 2 * G * D + H * V).to(dtype), rn(T, H).to(dtype), rn(T, H)
        dt[2::5] = 4e4                                # exp(-A softplus(4e4)) = 0
        dt = dt.to(dtype)
        got = O.delta_scan(dev(qkv), dev(bt), dev(dt), dev(bias), dev(A_log), st, meta_of(ln, ctx, [[1] * 12] * 6, 16, device, slots), H, G, D, V, D ** -0.5)
        x, gd, at, want = qkv.double(), decays(dt, bias, A_log), 0, []
        q, k = oracle.unit(x[:, :G * D].view(T, G, D), D ** -0.5), oracle.unit(x[:, G * D:2 * G * D].view(T, G, D))
        for n, c, sl in zip(ln, ctx, slots):
            S = ref[sl] if c > 0 else torch.zeros_like(ref[sl])
            for t in range(at, at + n):
                for h in range(H):
                    S[h] = gd[t, h] * S[h]
                    u = torch.sigmoid(bt[t, h].double()) * (x[t, 2 * G * D + h * V:2 * G * D + (h + 1) * V] - S[h].T @ k[t, h // (H // G)])
                    S[h] += torch.outer(k[t, h // (H // G)], u)
                want.append(torch.cat([S[h].T @ q[t, h // (H // G)] for h in range(H)]))
            if n:
                ref[sl] = S
            at += n
        close(got, torch.stack(want), 2e-5)
        close(st, ref, 2e-5)
        ctx = [c + n for c, n in zip(ctx, ln)]


@pytest.mark.parametrize("device,dtype,tol", DEVICES[:2])
def test_long_memory_keeps_its_precision(device, dtype, tol):
    """Decays close to 1 over 3000 tokens, orthogonal-ish keys: rounding must not add up."""
    O = backend(device)
    g = torch.Generator().manual_seed(2)
    T, H, D, V = 3000, 2, 32, 4
    qkv, bt, dt = torch.randn(T, 2 * H * D + H * V, generator=g), torch.full((T, H), -5.0), torch.full((T, H), -6.0)
    bias, A_log = torch.zeros(H), torch.tensor([-2.0, 0.0])
    x = qkv.double()
    q, k = oracle.unit(x[:, :H * D].view(T, H, D)), oracle.unit(x[:, H * D:2 * H * D].view(T, H, D))
    want = oracle.delta_rule(q, k, x[:, 2 * H * D:].view(T, H, V), torch.sigmoid(bt.double()), decays(dt, bias, A_log)).view(T, H * V)
    dev = lambda v: v.to(device)
    st = torch.zeros(2, H, D, V, device=device)
    got = O.delta_scan(dev(qkv), dev(bt), dev(dt), dev(bias), dev(A_log), st, meta_of([T], [0], [[1] * 200], 16, device, [1]), H, H, D, V, 1.0)
    close(got, want, 2e-5)


ATT_SIZES = [(4, 2, 8, 16, 10, [13, 14, 1, 2], 8), (3, 1, 10, 20, 9, [20, 3], 8), (6, 6, 56, 40, 40, [70, 1, 33, 16], 16), (2, 1, 6, 5, 0, [11, 5], 4),
             (10, 2, 128, 128, 100, [150, 66, 1], 64), (6, 2, 24, 136, 50, [60, 20], 16), (6, 1, 72, 104, 33, [120, 40, 1], 16), (4, 4, 192, 96, 64, [100, 64, 3], 64),
             (3, 3, 200, 16, 20, [40, 1], 16), (2, 2, 64, 64, 0, [300, 2, 1], 64), (8, 2, 16, 16, 1, [30, 1], 16)]


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("kind", ["slopes", "table", "both"])
@pytest.mark.parametrize("H,G,D,V,size,portions,page", ATT_SIZES)
def test_attention_alone(H, G, D, V, size, portions, page, kind, device, dtype, tol):
    """Prologue and attention as ops, portions into pages in scrambled order.  ``slopes``: whole-row norms, a slope per head, a sink, a gate per
    element, output into columns of a wider buffer; ``table``: convolved queries, keys and values, a bias table (shorter and longer than the
    window), a gate per head; ``both``: slopes and table together.  Sizes for every kernel form (vector form with 8, 16 and 32 lanes per key and 1,
    2, 4 heads per group, general form, tensor-core form of each size, split keys)."""
    O = backend(device)
    g = torch.Generator().manual_seed(H * 100 + D)
    rn = lambda *s: torch.randn(*s, generator=g)
    n, pad, C = sum(portions), 8, (H + G) * D + G * V
    rows = rn(n, pad + C).to(dtype)
    gate = rn(n, H if kind == "table" else H * V).to(dtype)
    slope = oracle.slopes(H).float() if kind != "table" else None
    sink = rn(H) if kind != "table" else None
    bias = rn(H, 7 if size == 10 else 60) if kind != "slopes" else None
    qn, kn, w = 1 + 0.3 * rn(H * D), 1 + 0.3 * rn(G * D), rn(C, 3)
    dev = lambda t: None if t is None else t.to(device)
    npg = (n + page - 1) // page
    pages = torch.randperm(npg, generator=g).add(1).tolist()
    kp, vp = torch.zeros(npg + 1, G, page, D, dtype=dtype, device=device), torch.zeros(npg + 1, G, page, V, dtype=dtype, device=device)
    cs = torch.full((3, 2, C), float("nan"), dtype=dtype, device=device)
    scale, outs, at = 2.0 * D ** -0.5, [], 0
    for m in portions:
        sl = slice(at, at + m)
        meta = meta_of([m], [at], [pages], page, device, [1])
        r = dev(rows[sl])
        if kind == "table":
            q = O.conv_qkv_append(r[:, pad:], dev(w), cs, H, D, kp, vp, meta)
        else:
            q = O.qk_norm_rope_append(r, pad, pad + H * D, pad + (H + G) * D, H, D, dev(qn), dev(kn), 1e-3, torch.zeros(0, device=device), kp, vp, meta, whole=True)
        buf = torch.zeros(m, 8 + H * V, dtype=dtype, device=device)
        O.sink_attention(q, kp, vp, dev(sink), meta, scale, 0, size, 1.3, dtype, buf, 8, gate=dev(gate[sl]), slopes=dev(slope), dist_bias=dev(bias))
        assert float(buf[:, :8].abs().max()) == 0.0
        outs.append(buf[:, 8:])
        at += m
    x = rows.double()[:, pad:]
    if kind == "table":
        x = oracle.short_conv(x, w.double())
        q, k = x[:, :H * D], x[:, H * D:(H + G) * D]
    else:
        q, k = oracle.rms(x[:, :H * D], 1e-3) * qn.double(), oracle.rms(x[:, H * D:(H + G) * D], 1e-3) * kn.double()
    back = torch.arange(n)
    b = torch.zeros(H, n, dtype=torch.float64)
    if slope is not None:
        b = b - oracle.slopes(H)[:, None] * back
    if bias is not None:
        b = b + bias.double()[:, back.clamp(max=bias.shape[1] - 1)]
    want = oracle.attend(q.view(n, H, D), k.view(n, G, D), x[:, (H + G) * D:].view(n, G, V), scale, size, b, None if sink is None else sink.double())
    want = 1.3 * want * torch.sigmoid(gate.double()).view(n, H, -1)
    close(torch.cat(outs), want.reshape(n, H * V), tol if dtype == torch.bfloat16 else 2e-5)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("K", [1, 2, 3, 5])
@pytest.mark.parametrize("with_kv", [True, False])
def test_convolution_into_the_pools(K, with_kv, device, dtype, tol):
    """Ragged steps (new and running sequences, one without tokens, then single tokens): queries in fp32, keys and values at their places in
    scrambled pages, histories in the slots; queries alone leave the pools as they are."""
    O = backend(device)
    g = torch.Generator().manual_seed(K)
    rn = lambda *s: torch.randn(*s, generator=g)
    H, G, D, V, page = 3, 2, 10, 5, 4
    C = H * D + (G * (D + V) if with_kv else 0)
    w = rn(C, K)
    slots, pages = [3, 1, 4, 2], [[3, 7, 1, 12], [5, 2, 13, 14], [8, 6, 15, 16], [9, 4, 10, 11]]
    seqs = [rn(n, C).to(dtype) for n in (9, 1, 14, 6)]
    kp, vp = torch.full((17, G, page, D), 7.0, dtype=dtype, device=device), torch.full((17, G, page, V), 7.0, dtype=dtype, device=device)
    cs = torch.full((5, K - 1, C), float("nan"), dtype=dtype, device=device)
    at, got = [0] * 4, [[] for _ in seqs]
    for take in ([3, 1, 11, 0], [5, 0, 2, 1], [1, 0, 1, 1], [0, 0, 0, 4]):
        ids = [i for i in range(4) if take[i] or take == [5, 0, 2, 1]]
        ln = [take[i] for i in ids]
        u = torch.cat([seqs[i][at[i]:at[i] + take[i]] for i in ids])
        q = O.conv_qkv_append(torch.nn.functional.pad(u, (8, 8)).to(device)[:, 8:-8], w.to(device), cs, H, D, kp, vp,
                              meta_of(ln, [at[i] for i in ids], [pages[i] for i in ids], page, device, [slots[i] for i in ids]))
        assert q.dtype == torch.float32
        o = 0
        for i, m in zip(ids, ln):
            got[i].append(q[o:o + m])
            o, at[i] = o + m, at[i] + m
    assert at == [len(s) for s in seqs]
    for i, s in enumerate(seqs):
        y = oracle.short_conv(s.double(), w.double())
        n = len(s)
        close(torch.cat(got[i]).view(n, -1), y[:, :H * D], 1e-5)
        rd = lambda pool, width: pool[pages[i]].transpose(1, 2).reshape(-1, G * width)[:n]
        if with_kv:
            close(rd(kp, D), y[:, H * D:H * D + G * D], tol)
            close(rd(vp, V), y[:, H * D + G * D:], tol)
    if not with_kv:
        assert float((kp - 7).abs().max()) == 0 and float((vp - 7).abs().max()) == 0


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("E,top,T", [(6, 2, 5), (12, 12, 3), (1, 1, 4), (70, 9, 300)])
def test_router_alone(E, top, T, device, dtype, tol):
    """Choice by score + correction, weights from the scores without it over their sum, times a factor; ties go to the lowest id."""
    O = backend(device)
    g = torch.Generator().manual_seed(E)
    z, corr = torch.randn(T, E, generator=g), torch.randn(E, generator=g)
    z[0] = 0.5
    idx, w = O.sigmoid_topk(z.to(device), E, top, corr.to(device), True, 1.7)
    iw, ww = oracle.route(z, corr, top, 1.7)
    assert torch.equal(idx.cpu().long(), iw)
    close(w, ww, 1e-5)
    flat = torch.zeros(T, E)
    assert O.sigmoid_topk(flat.to(device), E, top)[0][0].tolist() == list(range(top))
    idx, w = O.sigmoid_topk(z.to(device), E, top)                       # neither correction nor normalisation
    close(w, torch.sigmoid(z).sort(-1, descending=True).values[:, :top], 1e-5)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("T,K,F,E,top", [(7, 40, 24, 6, 2), (50, 40, 24, 6, 3), (9, 128, 128, 4, 2), (150, 128, 256, 5, 3), (3, 36, 21, 3, 1)])
def test_experts_alone(T, K, F, E, top, device, dtype, tol):
    """Clamped-GLU experts with the weight on the output: pair kernel, product per expert, grouped tensor-core products."""
    O = backend(device)
    g = torch.Generator().manual_seed(K)
    rn = lambda *s: torch.randn(*s, generator=g)
    x, wg, wu, wd = rn(T, K).to(dtype), (rn(E, F, K) * 2 * K ** -0.5).to(dtype), (rn(E, F, K) * 2 * K ** -0.5).to(dtype), (rn(E, K, F) * F ** -0.5).to(dtype)
    idx = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).int()
    w = torch.rand(T, top, generator=g) * 2
    lw = lambda t: LinearWeight(weight=t.to(device))
    got = O.moe_clamped_experts(x.to(device), idx.to(device), w.to(device), lw(wg), lw(wu), lw(wd), 0.9, on_input=False)
    want = torch.zeros(T, K, dtype=torch.float64)
    for t in range(T):
        for e, a in zip(idx[t].tolist(), w[t].double()):
            want[t] += a * oracle.expert(x[t:t + 1].double(), dict(gate=wg[e].double(), up=wu[e].double(), down=wd[e].double()), 0.9)[0]
    close(got, want, tol if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("C,groups", [(40, 4), (256, 2), (132, 1), (1024, 2), (21, 3), (1040, 2)])
def test_gated_norm_and_residual_alone(C, groups, device, dtype, tol):
    """Norm per head times weight times silu(gate), into columns of a wider buffer; two branches added to the residual with the norm behind
    them; embedding rows plus learned positions."""
    O = backend(device)
    g = torch.Generator().manual_seed(C)
    rn = lambda *s: torch.randn(*s, generator=g)
    T = 5
    y, gate, w = rn(T, C), rn(T, C).to(dtype), 1 + 0.2 * rn(C)
    buf = torch.zeros(T, C + 16, dtype=dtype, device=device)
    O.gated_rmsnorm(y.to(device), gate.to(device), w.to(device), 1e-3, groups, "silu_post", dtype, buf, 8)
    want = (oracle.rms(y.double().view(T, groups, -1), 1e-3).view(T, C)) * w.double() * oracle.silu(gate.double())
    close(buf[:, 8:-8], want, tol if dtype == torch.bfloat16 else 1e-5)
    assert float(buf[:, :8].abs().max()) == 0.0 and float(buf[:, -8:].abs().max()) == 0.0
    x, a, b = rn(T, C), rn(T, C), rn(T, C)
    xd = x.clone().to(device)
    ha = O.scaled_add_norm_(xd, a.to(device), None, w.to(device), 1e-3, dtype, extra=b.to(device))
    want = x.double() + a.double() + b.double()
    close(xd, want, 1e-5)
    close(ha, oracle.rms(want, 1e-3) * w.double(), tol if dtype == torch.bfloat16 else 1e-5)
    emb, pos = rn(11, C).to(dtype), rn(9, C).to(dtype)
    ids, p = torch.tensor([3, 0, 10, 3]), torch.tensor([8, 0, 4, 1], dtype=torch.int32)
    xs = O.stream_embed(emb.to(device), ids.to(device), 1.0, 1, pos.to(device), p.to(device))
    close(xs[:, 0], emb[ids].double() + pos[p.long()].double(), 1e-6)


# ---------------------------------------------------------------------------------------------------------------- schedules
@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_first_tokens_and_single_token(device, dtype, tol):
    cfgd = make_cfg(STACK)
    model, sd = make_model(cfgd, device, dtype)
    for t in ([5], toks(2, seed=4), toks(3, seed=5)):
        close(run_whole(model, t), oracle.forward(cfgd, sd, t), tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("portions", [[1] * 39, [2, 2, 2, 33], [16, 23], [15, 1, 1, 22], [3, 13, 7, 16], [38, 1], [8, 9, 6, 16], [2] * 19 + [1]])
def test_portions_equal_whole(portions, device, dtype, tol):
    """Prefill against token-by-token decoding and prompts cut anywhere (page edges at 16 and 32, windows of 5 to 30 that start inside an earlier
    portion, convolution histories that reach into the portions before, groups of the recurrence cut anywhere, 2-token portions)."""
    cfgd = make_cfg(STACK)
    model, sd = make_model(cfgd, device, dtype)
    t = toks(sum(portions), seed=1)
    close(in_portions(model, t, portions), oracle.forward(cfgd, sd, t), tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_ragged_batch_and_reuse_of_pages_and_slots(device, dtype, tol):
    """Unequal requests in one batch (portions beside single tokens) equal each alone; a pool of 5 pages and 2 state slots serves 4 requests
    one pair after another, so every page and slot is used again — by a request that must not see what the last one left."""
    cfgd = make_cfg(STACK)
    model, sd = make_model(cfgd, device, dtype)
    reqs = {n: toks(L, seed=10 + i) for i, (n, L) in enumerate([("a", 30), ("b", 9), ("c", 17), ("d", 33)])}
    want = {n: oracle.forward(cfgd, sd, t) for n, t in reqs.items()}
    s = session(model, pages=6, page_size=16, live=2)
    assert s.table.slots is not None and s.table.slots.num_free == 2
    got = {n: [] for n in reqs}

    def step(parts, end=()):
        entries = [dict(id=n, tokens=reqs[n][lo:hi], want=list(range(hi - lo))) for n, lo, hi in parts]
        out = s.step(entries)
        at = 0
        for n, lo, hi in parts:
            got[n].append(out[at:at + hi - lo])
            at += hi - lo
        s.end(end)

    step([("a", 0, 13), ("b", 0, 1)])
    step([("a", 13, 14), ("b", 1, 8)])
    step([("b", 8, 9), ("a", 14, 29)], end=["b"])
    step([("a", 29, 30)], end=["a"])
    assert s.table.alloc.num_free == 5 and s.table.slots.num_free == 2
    step([("d", 0, 2), ("c", 0, 16)])
    step([("c", 16, 17), ("d", 2, 33)], end=["c", "d"])
    for n in reqs:
        close(torch.cat(got[n]), want[n], tol)


def loud(layer, gain):
    """A larger share of a mixer in the residual, so that single keys count."""
    def edit(sd):
        for n in ("o", "left.o"):
            if f"l{layer}.mix.{n}" in sd:
                sd[f"l{layer}.mix.{n}"].mul_(gain)
    return edit


EDGES = [("parallel", 9, 1), ("parallel", 16, 4), ("parallel", 5, 2), ("attention", 9, 1), ("attention", 16, 5), ("attention", 4, 3), ("shared", 6, 1), ("shared", 16, 2)]


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("kind,size,seed", EDGES)
def test_window_edges_show(kind, size, seed, device, dtype, tol):
    """Sharp scores and a large share of the mixer in the residual make single keys count.  The oracle with a window one position off gives
    other logits from the position where the difference begins, so a wrong edge would show: in a prompt, in portions that start inside a
    window, and decoded one by one across edges and page borders (pages of 16)."""
    tol = min(tol, 3e-2)
    if kind == "parallel":
        layers, at = [par((4, 2, 8, 12, size, 0.8), (2, 1, 6, 4, 2), 1.0, 0.3, None)], 0
    elif kind == "attention":
        layers, at = [att(4, 2, 8, 12, size, 0.8, 2, 40, None)], 0
    else:
        layers, at = [att(4, 2, 8, 12, 20, 0.8, 2, 40, None), att(4, 2, 8, 12, size, 0.8, 1, 20, None, 0)], 1
    cfgd = make_cfg(layers)
    model, sd = make_model(cfgd, device, dtype, edit=loud(at, 4.0))
    t = toks(44, seed=seed)
    want = oracle.forward(cfgd, sd, t)
    for ds, first in ((-1, size - 1), (1, size)):
        other = copy.deepcopy(cfgd)
        m = other["layers"][at]["mixer"]
        (m["left"] if kind == "parallel" else m)["mask"] = dict(size=size + ds)
        diff = (oracle.forward(other, sd, t) - want).abs().max(-1).values
        assert diff[:first].max() == 0 and diff[first:].max() > 0.06 * want.abs().max(), ds
    close(run_whole(model, t), want, tol)
    close(decode_after(model, t, 4), want, tol)
    close(in_portions(model, t, [5, 6, 2, 14, 17]), want, tol)
    close(in_portions(model, t, [20, 24]), want, tol)          # tensor-core form: portions of 16 tokens and more


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("kind", ["parallel", "attention"])
def test_far_key_among_hundreds(kind, device, dtype, tol):
    """With sharp scores some late queries put their weight on single keys more than 200 tokens back: other tokens there move the late logits.
    Prompt, decode, portions (pages of 16: the keys lie many pages back)."""
    if kind == "parallel":
        layers = [par((8, 1, 16, 8, 300, 4.0), (2, 1, 6, 4, 2), 1.0, 0.0, None)]
    else:
        layers = [att(2, 1, 16, 8, 300, 4.0, 2, 300, None)]
    cfgd = make_cfg(layers)

    def edit(sd):
        if kind == "parallel":
            sd["l0.mix.left.sink"].sub_(3.0)
        loud(0, 3.0)(sd)

    model, sd = make_model(cfgd, device, dtype, edit=edit)
    t = toks(330, seed=17)
    want = oracle.forward(cfgd, sd, t)
    far = oracle.forward(cfgd, sd, [(x + 1 + i) % 96 if 40 <= i < 90 else x for i, x in enumerate(t)])
    gone = oracle.forward(cfgd, sd, [(x + 1 + i) % 96 if i < 9 else x for i, x in enumerate(t)])
    assert (far[300:] - want[300:]).abs().max() > 3 * SHOWS * want.abs().max()
    assert (gone[315:] - want[315:]).abs().max() < 1e-9                   # tokens behind the window
    kw = dict(pages=22)
    tol = min(tol, 4e-2)
    close(run_whole(model, t, **kw), want, tol)
    close(in_portions(model, t, [2, 120, 50, 128, 2, 20] + [1] * 8, **kw), want, tol)


FAULTS = [dict(no_sink=True), dict(slope=0.0), dict(slope=-1.0), dict(norm_per_head=True), dict(limit=5.0), dict(correction=0.0), dict(no_positions=True), dict(sequential=True),
          dict(no_bias=True), dict(bucket_shift=1), dict(conv_lost_before=16), dict(lost_before=16), dict(kv_from=2)]


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_planted_mistakes_show(device, dtype, tol):
    """Every planted mistake (a missing sink, slope, bias, correction, limit or position; norms per head; feed-forward behind the mixer; a bias
    table one distance off; a convolution history or a state lost between portions; another layer's keys) moves the logits."""
    layers = [A_GQ, P_GQ, A_GQ, kv_of(0, A_GQ, 9, None, 20), P_MH]
    layers[1] = par((4, 2, 8, 12, 12, 0.8), (4, 2, 6, 10, 4), 1.2, 1.5, moe(6, 2, 24, 1.5, 0.3))
    cfgd = make_cfg(layers)

    def edit(sd):
        sd["l1.mix.right.A_log"].fill_(-4.0)                              # slow decays: a lost state is missed
        if dtype == torch.float32:
            sd["l1.mlp.correction"].mul_(5.0)

    model, sd = make_model(cfgd, device, dtype, edit=edit)
    t = toks(30, seed=8)
    want = oracle.forward(cfgd, sd, t)
    for faults in FAULTS:
        assert (oracle.forward(cfgd, sd, t, faults=faults) - want).abs().max() > 2 * SHOWS * want.abs().max(), faults
    close(run_whole(model, t), want, tol)
    close(decode_after(model, t, 11), want, tol)
    close(in_portions(model, t, [16, 2, 12]), want, tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_far_token_lives_in_the_state(device, dtype, tol):
    """With slow decays and a window of 2 only the recurrent state carries the first tokens to position 60, four pages on: other tokens there and
    a state that is lost on the way move the late logits.  In a prompt, in decoding, and in portions."""
    cfgd = make_cfg([par((2, 1, 8, 4, 2, 0.5), (4, 2, 24, 10, 4), 0.1, 3.0, None)])
    edit = lambda sd: (sd["l0.mix.right.A_log"].fill_(-6.0), sd["l0.mix.right.b"].mul_(0.1))
    model, sd = make_model(cfgd, device, dtype, edit=edit)
    t = toks(70, seed=200)
    want = oracle.forward(cfgd, sd, t)
    other = [(x + 1 + i) % 96 if i < 8 else x for i, x in enumerate(t)]
    assert (oracle.forward(cfgd, sd, other)[60:] - want[60:]).abs().max() > SHOWS * want.abs().max()
    assert (oracle.forward(cfgd, sd, t, faults=dict(lost_before=40))[60:] - want[60:]).abs().max() > SHOWS * want.abs().max()
    close(run_whole(model, t, pages=8), want, tol)
    close(decode_after(model, t, 55, pages=8), want, tol)
    close(in_portions(model, t, (2, 31, 2, 30, 5), pages=8), want, tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_long_prompt_then_decode(device, dtype, tol):
    """A 290-token prompt over a window of 270 and without a window, then single tokens whose keys are split over CTAs and merged on the GPU."""
    cfgd = make_cfg([par((4, 2, 8, 16, 270, 0.5), (2, 2, 16, 8, 3), 0.9, 1.1, None), att(2, 1, 16, 40, 0, 0.4, 2, 300, None), kv_of(1, att(2, 1, 16, 40, 0, 0.4, 2, 300, None), 280, None, 300)])
    model, sd = make_model(cfgd, device, dtype)
    t = toks(296, seed=9)
    want = oracle.forward(cfgd, sd, t)
    close(decode_after(model, t, 290, pages=21), want, tol)
    close(in_portions(model, t, [40, 200, 3, 45, 2, 6], pages=21), want, tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_long_decode(device, dtype, tol):
    """Single-token steps after a 3-token prompt: states are read and written every step, windows move over page borders."""
    cfgd = make_cfg([A_GQ, P_GQ, kv_of(0, A_GQ, 20), P_ODD])
    model, sd = make_model(cfgd, device, dtype)
    t = toks(153, seed=5)
    close(decode_after(model, t, 3), oracle.forward(cfgd, sd, t), tol * (2 if dtype == torch.bfloat16 else 1))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-4), (torch.bfloat16, 6e-2)])
def test_tensor_core_sizes(dtype, tol):
    """Widths and expert sizes that are multiples of 128, head sizes of 64 and 128: bf16 takes the tensor-core GEMMs (grouped for the experts)
    and both sizes of the tensor-core attention with slopes and with tables; pages of 16 and 64."""
    cfgd = make_cfg([par((4, 2, 128, 128, 90, 0.1), (4, 2, 64, 64, 4), 0.8, 1.1, moe(4, 2, 128, 1.2, 3.0)), att(4, 2, 64, 64, 100, 0.12, 4, 64, moe(4, 2, 256)),
                     att(8, 2, 64, 64, 33, 0.15, 2, 20, None, 1), par((2, 1, 64, 128, 50, 0.2), (2, 2, 128, 128, 3), 1.0, 0.7, moe(3, 2, 128))], width=128)
    model, sd = make_model(cfgd, "cuda", dtype)
    t = toks(200, seed=2)
    want = oracle.forward(cfgd, sd, t)
    for kw in (dict(pages=14, page_size=16), dict(pages=5, page_size=64)):
        close(in_portions(model, t, [150, 2, 30, 10] + [1] * 8, **kw), want, tol)


def random_cfg(rng):
    """A configuration drawn at random: 2 to 6 layers of either mixer in any order, every size and constant drawn anew; layers that read another
    layer's keys and values take its sizes."""
    layers, own = [], []
    for i in range(rng.randint(2, 6)):
        mlp = None if rng.random() < 0.3 else moe(E := rng.choice([1, 3, 7, 9]), rng.randint(1, E), rng.choice([8, 21, 40]), rng.choice([0.5, 1.0, 2.5]), rng.choice([0.5, 1.0, 4.0]))
        G, size = rng.choice([1, 2, 3]), rng.choice([0, 1, 5, 16, 24, 33])
        H, D, V = G * rng.choice([1, 2, 3, 5]), rng.choice([5, 8, 16, 32, 72]), rng.choice([4, 8, 24, 41])
        if rng.random() < 0.45:
            g = rng.choice([1, 2, 3])
            layers.append(par((H, G, D, V, size, rng.choice([0.2, 0.5, 1.0])), (g * rng.choice([1, 2, 4]), g, rng.choice([3, 8, 16, 40]), rng.choice([4, 9, 16, 64]), rng.choice([1, 2, 3, 4, 6])),
                              rng.choice([1.0, 0.6, -1.1]), rng.choice([1.0, 0.4, 1.7]), mlp))
        elif own and rng.random() < 0.5:
            j = rng.choice(own)
            layers.append(kv_of(j, layers[j], size, mlp, rng.choice(list(ROWS)), rng.choice([1, 2, 4])))
        else:
            own.append(i)
            layers.append(att(H, G, D, V, size, rng.choice([0.2, 0.5, 1.0]), rng.choice([1, 2, 3, 5]), rng.choice(list(ROWS)), mlp))
    return make_cfg(layers, width=rng.choice([40, 64, 72, 51]), vocab=rng.choice([50, 77]), eps=rng.choice([1e-6, 1e-3]), positions=rng.choice([80, 333]))


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("seed", range(1, 11))
def test_random_configurations(seed, device, dtype, tol):
    """Configurations drawn at random, two requests stepped in portions of random sizes side by side, every position against the oracle."""
    rng = random.Random(seed)
    cfgd = random_cfg(rng)
    model, sd = make_model(cfgd, device, dtype, seed=seed)
    reqs = {"a": toks(rng.randint(50, 80), vocab=cfgd["vocab"], seed=seed), "b": toks(rng.randint(10, 40), vocab=cfgd["vocab"], seed=seed + 1)}
    want = {n: oracle.forward(cfgd, sd, t) for n, t in reqs.items()}
    s = session(model, pages=10)
    got, at = {"a": [], "b": []}, {"a": 0, "b": 0}
    while any(at[n] < len(reqs[n]) for n in reqs):
        entries = []
        for n, sizes in (("a", [1, 2, 5, 17, 33]), ("b", [1, 1, 2, 9])):
            if at[n] < len(reqs[n]) and (n == "a" or rng.random() < 0.7):
                k = min(len(reqs[n]) - at[n], rng.choice(sizes))
                entries.append(dict(id=n, tokens=reqs[n][at[n]:at[n] + k], want=list(range(k))))
        if not entries:
            continue
        out = s.step(entries)
        o = 0
        for e in entries:
            k = len(e["tokens"])
            got[e["id"]].append(out[o:o + k])
            o, at[e["id"]] = o + k, at[e["id"]] + k
    for n in reqs:
        (close_in_bf16 if dtype == torch.bfloat16 else close)(torch.cat(got[n]), want[n], tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_result_does_not_depend_on_the_batch(device, dtype, tol):
    """The last token of a request decoded alone, beside single tokens, and beside a long portion (which takes other kernel forms), from
    different pages and slots: the same logits up to rounding."""
    cfgd = make_cfg(STACK)
    model, _ = make_model(cfgd, device, dtype)
    t, long = toks(40, seed=31), toks(60, seed=32)
    rows = []
    for beside in (None, 1, 60):
        s = session(model, pages=16)
        if beside:
            s.step([dict(id="x", tokens=long[:20] if beside == 1 else long[:1], want=[])])
        s.step([dict(id="a", tokens=t[:39], want=[])])
        entries = [dict(id="a", tokens=t[39:], want=[0])]
        if beside:
            entries.insert(0, dict(id="x", tokens=long[20:21] if beside == 1 else long[1:], want=[]))
        rows.append(s.step(entries))
    tight = 1e-5 if dtype == torch.float32 else 2e-2
    close(rows[1], rows[0], tight)
    close(rows[2], rows[0], tight)


# ---------------------------------------------------------------------------------------------------------------- framework
def oracle_greedy(cfgd, sd, prompt, n):
    seq, gap = list(prompt), 1e9
    for _ in range(n):
        lg = oracle.forward(cfgd, sd, seq)[-1]
        top = lg.topk(2).values
        gap = min(gap, (top[0] - top[1]).item())
        seq.append(int(lg.argmax()))
    return seq[len(prompt):], gap


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_greedy_generation_through_engine(device, dtype, tol):
    """The engine's scheduler, sampler and (on the GPU) captured decode graphs: three requests of unequal length, more than there are slots,
    greedy tokens equal the oracle's argmax continuation (bf16: prompts whose best two logits never come close); pages and slots come back."""
    cfgd = make_cfg(STACK)
    model, sd = make_model(cfgd, device, dtype)
    eng = LLMEngine(LocalPipeline([StageExecutor(model, 16, 16, num_state_slots=3)]), 16, 16, num_groups=1, max_prefill_tokens=11)
    assert eng.table.slots is not None
    free0 = eng.table.slots.num_free
    need, found = (0.0 if dtype == torch.float32 else 0.5), []
    for i in range(60):
        p = toks((19, 4, 30)[len(found)], seed=21 + i)
        out, gap = oracle_greedy(cfgd, sd, p, 6)
        if gap > need:
            found.append((p, out))
        if len(found) == 3:
            break
    assert len(found) == 3
    rs = [eng.submit(p, SamplingParams(temperature=0.0), max_tokens=6) for p, _ in found]
    eng.drain()
    for (p, out), r in zip(found, rs):
        assert r.error is None
        assert r.output == out
    assert eng.table.alloc.num_free == 15 and eng.table.slots.num_free == free0


def test_no_request_passes_the_last_position():
    """The position table bounds a request: the engine and the trace session refuse longer ones, and one that just fits runs."""
    cfgd = make_cfg([A_GQ], positions=20)
    model, sd = make_model(cfgd)
    eng = LLMEngine(LocalPipeline([StageExecutor(model, 16, 16, num_state_slots=3)]), 16, 16, num_groups=1)
    assert eng.max_model_len == 20
    with pytest.raises(ValueError):
        eng.submit(toks(18), SamplingParams(temperature=0.0), max_tokens=3)
    assert len(eng.generate(toks(18), SamplingParams(temperature=0.0), max_tokens=2)) == 2
    s = session(model)
    t = toks(20, seed=3)
    close(s.step([dict(id="a", tokens=t, want=list(range(20)))]), oracle.forward(cfgd, sd, t), 2e-4)
    with pytest.raises(ValueError):
        s.step([dict(id="a", tokens=[1], want=[])])


def test_config_reader_takes_every_size_from_the_file():
    cfg = ModelConfig.from_dict(make_cfg([A_FREE, P_ODD, kv_of(0, A_FREE, 6)], width=40, vocab=50, eps=3e-3, positions=77))
    assert (cfg.model_type, cfg.hidden_size, cfg.vocab_size, cfg.num_hidden_layers, cfg.max_position_embeddings) == ("lomusun", 40, 50, 3, 77)
    assert cfg.rms_norm_eps == 3e-3 and cfg.tie_word_embeddings and cfg.layer_specs[1]["mlp"] is None and cfg.layer_specs[2]["mixer"]["kv_from"] == 0
    assert cfg.layer_specs[1]["mixer"]["left"]["mask"] == dict(size=9) and cfg.layer_specs[0]["mlp"]["expert"] == dict(ff=33, limit=0.8)
    bad = [dict(type="unknown", mixer=dict(heads=1), mlp=None)], [att(5, 2, 8, 8, 4, 1.0, 2, 20, None)], [dict(A_GQ, mlp=dict(kind="dense", ff=8))], [dict(A_GQ, mlp=moe(3, 4, 8))], \
        [kv_of(0, A_GQ, 5)], [P_GQ, kv_of(0, A_GQ, 5)], [A_GQ, kv_of(0, A_GQ, 5), kv_of(1, A_GQ, 5)], [A_MQ, kv_of(0, A_GQ, 5)], [A_GQ, kv_of(1, A_GQ, 5)], \
        [par((4, 2, 8, 8, 4, 1.0), (3, 2, 4, 4, 2), 1.0, 1.0, None)], [par((4, 2, 8, 8, 4, 1.0), (2, 2, 4, 4, 0), 1.0, 1.0, None)], [dict(A_GQ, mixer=dict(A_GQ["mixer"], mask=dict(size=0)))]
    for layers in bad:
        with pytest.raises(ValueError):
            ModelConfig.from_dict(make_cfg(layers))


def test_cache_layout_and_weights():
    model, sd = make_model(make_cfg(STACK))
    lay = model.cache_layout()
    assert lay[0][:5] == ("paged_kv", 2, 8, 12, torch.float32) and lay[0][5]["conv"][0] == (2, 72)
    assert lay[1][5]["S"] == ((4, 6, 10), torch.float32) and lay[1][5]["conv"][0] == (3, 64)
    assert lay[2] == ("alias", 0, {"conv": ((1, 32), torch.float32)}) and lay[5][:2] == ("alias", 4)
    kv = StageExecutor(model, 4, 16, num_state_slots=3).kv
    assert kv.num_slots == 3 and kv.k[2] is kv.k[0] and kv.v[6] is kv.v[0] and kv.state[2]["conv"].shape == (3, 1, 32) and kv.state[3]["conv"].shape == (3, 0, 51)
    build = lambda sd: build_stage(ModelConfig.from_dict(make_cfg(STACK)), None, torch.float32, "cpu").load_state(sd)
    with pytest.raises(ValueError):                       # a tensor the design does not have
        build(dict(sd, extra=torch.zeros(1)))
    for k in ("l0.mix.q", "l1.mix.left.q.norm", "l0.mlp.e1.up", "pos", "l2.mix.rel"):
        with pytest.raises(ValueError):                   # a tensor of another shape
            build({n: (v[..., :-1] if n == k else v) for n, v in sd.items()})


@pytest.mark.timeout(300)
def test_command_line_generation():
    """``generate.py`` on a synthetic model of the design: tokenizer, engine, sampler and the printed statistics."""
    repo = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(repo, "generate.py"), "--model", "synthetic:tiny-lomusun", "--prompt", "hello", "--max_tokens", "8",
                        "--device", "cpu", "--no_chat_template"], capture_output=True, text=True, timeout=240,
                       env=dict(os.environ, PYTHONPATH=repo, OMP_NUM_THREADS="1"))
    assert r.returncode == 0, r.stdout + r.stderr
    assert "Generation:" in r.stdout and "tokens-per-sec" in r.stdout


@pytest.mark.timeout(300)
def test_trace_replay_from_a_model_folder(tmp_path):
    """``bin/trace_run`` on a folder with config.json and safetensors: portions and single tokens of two requests, a pool of exactly the live
    pages, logits against the oracle."""
    import numpy as np
    from safetensors.torch import save_file

    repo = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfgd = make_cfg([A_GQ, P_GQ, kv_of(0, A_GQ, 8)], vocab=50)
    _, sd = make_model(cfgd)
    (tmp_path / "model").mkdir()
    (tmp_path / "model" / "config.json").write_text(json.dumps(cfgd))
    save_file({k: v.contiguous() for k, v in sd.items()}, str(tmp_path / "model" / "model.safetensors"))
    a, b = toks(70, vocab=50, seed=1), toks(5, vocab=50, seed=2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:60], want=[3, 59])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b, want=[4]), dict(id="a", tokens=a[60:61], want=[0])], end=["b"]),
             dict(step=2, entries=[dict(id="a", tokens=a[61:], want=[8])], end=["a"])]
    r = subprocess.run([sys.executable, os.path.join(repo, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "float32", "--out", str(tmp_path / "out"),
                        "--max-tokens", "192", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240,
                       env=dict(os.environ, OMP_NUM_THREADS="1"))
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    read = lambda n: torch.from_numpy(np.fromfile(str(tmp_path / "out" / f"{n}.f32"), dtype="<f4").reshape(-1, 50).copy())
    wa, wb = oracle.forward(cfgd, sd, a), oracle.forward(cfgd, sd, b)
    close(read(0), wa[[3, 59]], 2e-4)
    close(read(1), torch.stack([wb[4], wa[60]]), 2e-4)
    close(read(2), wa[69:], 2e-4)
