"""Podurax (selective scans with one step size per channel; sliding-window attention that keeps the first tokens visible, with rotary
positions stretched by YaRN, a 1 in the softmax denominator, values mixed with the first attention layer's, a gate per head; GELU-GLU
feed-forwards) against the plain oracle in ``podurax_oracle.py``: every mechanism alone, prefill against token-by-token decoding, prompt
portions down to two tokens, ragged batches against each request alone, pages and state slots that are freed and used again, keys just
inside and just outside the window and among the kept first tokens, far tokens held only by a recurrent state, the sink, the value
mixing, other sizes (one key/value head and as many as query heads, values wider and narrower than keys, one to five convolution taps,
states of 1 to 130 entries, rotation of all / some / no entries, no window, nothing kept, layers without feed-forward), long decoding, and
greedy generation through the engine.

Runs on the CPU with the unfused ops; the ``gpu`` variants run the same cases on the sm_100a kernels in fp32 and bf16.
"""
import copy
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import podurax_oracle as oracle  # noqa: E402

from mlx_sharding_b200.config import ModelConfig  # noqa: E402
from mlx_sharding_b200.engine.core import LLMEngine  # noqa: E402
from mlx_sharding_b200.engine.sampler import SamplingParams  # noqa: E402
from mlx_sharding_b200.engine.trace import TraceSession  # noqa: E402
from mlx_sharding_b200.models import build_stage  # noqa: E402
from mlx_sharding_b200.models.base import yarn_inv_freq  # noqa: E402
from mlx_sharding_b200.ops import BatchMeta, LinearWeight, get_backend  # noqa: E402
from mlx_sharding_b200.parallel.pipeline import LocalPipeline, StageExecutor  # noqa: E402
from mlx_sharding_b200.utils.checkpoint import random_state_dict  # noqa: E402


def scan(inner, state, dt_rank, conv, ff=40):
    return dict(type="mamba1", mixer=dict(conv=conv, dt_rank=dt_rank, inner=inner, state=state), mlp=dict(kind="dense", ff=ff) if ff else None)


def att(heads, kv_heads, dim, vdim, size, keep, rot, scale, v_mix=True, ff=40, base=50.0, factor=3.0, original=24, fast=4.0, slow=0.5):
    m = dict(dim=dim, heads=heads, kv_heads=kv_heads, scale=scale, v_mix=v_mix, vdim=vdim)
    if size:
        m["mask"] = dict(size=size, keep_first=keep)
    if rot:
        m["rot"] = dict(base=base, dims=rot)
        if factor:
            m["rot"]["scaling"] = dict(factor=factor, original=original, fast=fast, slow=slow)
    return dict(type="attention", mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None)


M_A = scan(24, 6, 3, 4)                                     # odd sizes: nothing is a multiple of 8 but the channels
M_B = scan(37, 1, 1, 1, ff=23)                              # one state entry, one step-size input, one tap (no history)
M_C = scan(16, 9, 5, 5, ff=None)                            # no feed-forward
A_GQ = att(4, 2, 8, 12, 7, 3, 4, 0.8)                       # two query heads per key/value head; window of 7, 3 kept; half the entries turn
A_GQ2 = att(4, 2, 16, 12, 16, 1, 16, 0.3, ff=None)          # window = page; all entries turn; another key size than the layer it mixes from
A_MQ = att(3, 1, 10, 20, 9, 0, 6, 0.6, v_mix=False, ff=33)  # one key/value head; nothing kept; no value mixing
A_FREE = att(2, 2, 6, 5, 0, 0, 0, 0.9, v_mix=False)         # no window, no rotation
A_PLAIN = att(2, 2, 8, 12, 11, 30, 8, 0.5, factor=None)     # more kept than the window; rotation without stretching
STACK = [M_A, A_GQ, A_GQ2, M_C, A_MQ, A_GQ]
CASES = {"scan": [M_A], "scan_small": [M_B], "scan_taps": [M_C], "att_gq": [A_GQ], "att_mix": [A_GQ, A_GQ2, A_PLAIN], "att_mq": [A_MQ], "att_free": [A_FREE],
         "stack": STACK}
DEVICES = [pytest.param("cpu", torch.float32, 2e-4, id="cpu"),
           pytest.param("cuda", torch.float32, 2e-4, id="b200-f32", marks=pytest.mark.gpu),
           pytest.param("cuda", torch.bfloat16, 6e-2, id="b200-bf16", marks=pytest.mark.gpu)]


def make_cfg(layers, width=48, vocab=96, eps=1e-3, mult=0.5, scale=3.0):
    return dict(architecture="Podurax", embedding=dict(scale=scale), layers=copy.deepcopy(layers), norm=dict(eps=eps), residual_mult=mult, vocab=vocab,
                width=width)


def make_model(cfgd, device="cpu", dtype=torch.float32, seed=3, edit=None):
    cfg = ModelConfig.from_dict(cfgd)
    sd = dict(random_state_dict(cfg, dtype=torch.bfloat16, seed=seed))
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


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [(16, 500.0, 4.0, 64, 32.0, 1.0), (8, 1e4, 8.0, 4096, 32.0, 1.0), (4, 50.0, 3.0, 24, 4.0, 0.5),
                                                                 (12, 1e6, 1.0, 100, 2.0, 2.0), (6, 20.0, 2.0, 1000, 500.0, 400.0)])
def test_yarn_frequencies(dims, base, factor, original, fast, slow):
    """Against the oracle's loop over pairs: ramps that start at 0, end at the last pair, are empty (both ends equal)."""
    want, mult = oracle.yarn_freqs(dict(dims=dims, base=base, scaling=dict(factor=factor, original=original, fast=fast, slow=slow)))
    close(yarn_inv_freq(dims, base, factor, original, fast, slow), want, 1e-6)
    assert abs(mult - (0.1 * math.log(factor) + 1.0)) < 1e-12


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("inner,state,portions,slots", [(24, 6, [13, 1, 9], [3]), (33, 1, [2, 20, 1], [1]), (40, 2, [23], [2]), (20, 16, [5, 18], [4]), (17, 30, [23], [1]),
                                                        (9, 61, [3, 20], [2]), (12, 130, [20, 1, 2], [1]), (8, 5, [300, 40], [2])])
def test_selective_scan_alone(inner, state, portions, slots, device, dtype, tol):
    """The scan as an op: one sequence in portions, the state carried in a dirty slot that must not be read at the first token; state sizes
    over every lane layout of the kernels, channels that do not fill a block, portions long enough for time slices; without a gate and with one."""
    O = get_backend("b200" if device == "cuda" else "reference")
    g = torch.Generator().manual_seed(inner * 1000 + state)
    rn = lambda *s: torch.randn(*s, generator=g)
    T = sum(portions)
    x, z, bc = rn(T, inner).to(dtype), (rn(T, inner) * 2).to(dtype), (rn(T, 3 + 2 * state) * state ** -0.5).to(dtype)
    dt, bias, D = rn(T, inner) * 1.5, rn(inner) - 1.0, rn(inner)
    A_log = torch.log(torch.rand(inner, state, generator=g) * 2 + 0.02)
    dd = torch.nn.functional.softplus(dt.double() + bias.double())
    y = oracle.selective_scan(x.double(), dd, -torch.exp(A_log.double()), bc[:, 3:3 + state].double(), bc[:, 3 + state:].double(), D.double())
    want = y * oracle.silu(z.double())
    dev = lambda v: v.to(device)
    st = torch.full((6, inner, state), float("nan"), device=device)
    for gate in (True, False):
        at, got = 0, []
        for n in portions:
            sl = slice(at, at + n)
            meta = meta_of([n], [at], [[1] * 30], 16, device, slots)
            got.append(O.selective_scan(dev(x[sl]), dev(dt[sl]), dev(bias), dev(A_log), dev(bc[sl]), 3, 3 + state, dev(D), dev(z[sl]) if gate else None, st, meta))
            at += n
        close(torch.cat(got), want if gate else y, tol if dtype == torch.bfloat16 else 2e-5)
        assert got[0].dtype == dtype and torch.isnan(st[0]).all() and torch.isnan(st[5]).all()          # other slots untouched


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_selective_scan_ragged(device, dtype, tol):
    """Sequences of 1, 7, 150, 0 and 2 tokens in one step (some new, some with a state), then a step of single tokens; the states afterwards."""
    O = get_backend("b200" if device == "cuda" else "reference")
    g = torch.Generator().manual_seed(11)
    rn = lambda *s: torch.randn(*s, generator=g)
    inner, N, lens = 44, 12, [1, 7, 150, 0, 2]
    bias, D, A_log = rn(inner) - 1.0, rn(inner), torch.log(torch.rand(inner, N, generator=g) * 2 + 0.02)
    A = -torch.exp(A_log.double())
    S0 = rn(6, inner, N)
    st = S0.clone().to(device)
    ref = S0.double().clone()
    dev = lambda v: v.to(device)
    for step, ln in enumerate((lens, [1] * 5)):
        T = sum(ln)
        x, bc, dt = rn(T, inner).to(dtype), (rn(T, 2 * N) * 0.3).to(dtype), rn(T, inner)
        ctx = [0, 3, 0, 5, 9] if step == 0 else [1, 10, 150, 0, 11]
        slots = [2, 5, 1, 4, 3]
        got = O.selective_scan(dev(x), dev(dt), dev(bias), dev(A_log), dev(bc), 0, N, dev(D), None, st, meta_of(ln, ctx, [[1] * 12] * 5, 16, device, slots))
        at, want = 0, []
        for n, c, sl in zip(ln, ctx, slots):
            S = ref[sl] if c > 0 else torch.zeros_like(ref[sl])
            for t in range(at, at + n):
                d = torch.nn.functional.softplus(dt[t].double() + bias.double())
                S = torch.exp(d[:, None] * A) * S + (d * x[t].double())[:, None] * bc[t, :N].double()
                want.append(S @ bc[t, N:].double() + D.double() * x[t].double())
            if n:
                ref[sl] = S
            at += n
        close(got, torch.stack(want), tol if dtype == torch.bfloat16 else 2e-5)
        close(st, ref, 2e-5)


@pytest.mark.parametrize("device,dtype,tol", DEVICES[:2])
def test_long_memory_keeps_its_precision(device, dtype, tol):
    """Decays close to 1 over 3000 tokens: the rounding of the factors must not add up (a last-bit error of one sign in every factor
    would)."""
    O = get_backend("b200" if device == "cuda" else "reference")
    g = torch.Generator().manual_seed(2)
    T, inner, N = 3000, 8, 4
    x, bc = torch.rand(T, inner, generator=g), torch.rand(T, 2 * N, generator=g)
    dt, bias, D = torch.full((T, inner), -6.0) + 0.1 * torch.randn(T, inner, generator=g), torch.zeros(inner), torch.zeros(inner)
    A_log = torch.linspace(-3.0, -1.0, inner * N).view(inner, N)
    dd = torch.nn.functional.softplus(dt.double())
    A = -torch.exp(A_log.double())
    S, want = torch.zeros(inner, N, dtype=torch.float64), []
    for t in range(T):
        S = torch.exp(dd[t][:, None] * A) * S + (dd[t] * x[t].double())[:, None] * bc[t, :N].double()
        want.append(S @ bc[t, N:].double())
    dev = lambda v: v.to(device)
    st = torch.zeros(2, inner, N, device=device)
    got = O.selective_scan(dev(x), dev(dt), dev(bias), dev(A_log), dev(bc), 0, N, dev(D), None, st, meta_of([T], [0], [[1] * 200], 16, device, [1]))
    close(got, torch.stack(want), 2e-5)


def attention_reference(q, k, v, ctx0, n, scale, size, keep, gate):
    """Oracle softmax of the last ``n`` queries (fp64) over all keys ``k`` ``[N, G, D]``, values ``v``; score 0 sink, gate per head."""
    N, H = k.shape[0], q.shape[1]
    rep = H // k.shape[1]
    seen = oracle.visible(N, size or N, keep)[ctx0:ctx0 + n]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T * scale).masked_fill(~seen, float("-inf"))
        e = torch.exp(s)
        out.append(e / (1.0 + e.sum(-1, keepdim=True)) @ v[:, h // rep] * torch.sigmoid(gate[:, h:h + 1]))
    return torch.cat(out, -1)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("H,G,D,V,rot,size,keep,portions,page", [
    (4, 2, 8, 16, 4, 10, 3, [13, 14, 1, 2], 8), (3, 1, 10, 20, 6, 9, 0, [20, 3], 8), (6, 6, 56, 40, 24, 40, 5, [70, 1, 33, 16], 16), (2, 1, 6, 5, 0, 0, 0, [11, 5], 4),
    (10, 2, 128, 128, 64, 100, 17, [150, 66, 1], 64), (6, 2, 24, 136, 8, 50, 7, [60, 20], 16), (6, 1, 72, 104, 72, 33, 70, [120, 40, 1], 16),
    (4, 4, 192, 96, 32, 64, 64, [100, 64, 3], 64), (3, 3, 200, 16, 8, 20, 2, [40, 1], 16)])
def test_attention_alone(H, G, D, V, rot, size, keep, portions, page, device, dtype, tol):
    """Prologue and attention as ops, portions into pages in scrambled order: rotation of all / some / no entries before a norm without
    weights, mixed values, window and kept tokens, gate per head, output into columns of a wider buffer; sizes for every kernel form
    (vector form with 8, 16 and 32 lanes per key and 1, 2, 4 heads per group, general form, tensor-core form)."""
    O = get_backend("b200" if device == "cuda" else "reference")
    g = torch.Generator().manual_seed(H * 100 + D)
    rn = lambda *s: torch.randn(*s, generator=g)
    n, pad = sum(portions), 8
    v0 = pad + (H + G) * D
    rows, vf, gate = rn(n, v0 + G * V + H).to(dtype), rn(n, G * V).to(dtype), None
    inv, mult = yarn_inv_freq(rot, 50.0, 3.0, 24.0, 4.0, 0.5) if rot else torch.zeros(0), 1.2 if rot else 1.0
    dev = lambda t: t.to(device)
    npg = (n + page - 1) // page
    pages = torch.randperm(npg, generator=g).add(1).tolist()
    kp, vp = torch.zeros(npg + 1, G, page, D, dtype=dtype, device=device), torch.zeros(npg + 1, G, page, V, dtype=dtype, device=device)
    scale, outs, at = (-2.0 if D == 72 else 2.0) * D ** -0.5, [], 0
    for m in portions:
        sl = slice(at, at + m)
        meta = meta_of([m], [at], [pages], page, device)
        r = dev(rows[sl])
        q = O.qk_norm_rope_append(r, pad, pad + H * D, v0, H, D, None, None, 1e-3, dev(inv), kp, vp, meta, half=True, norm_after=True, rot_mult=mult,
                                  v_first=dev(vf[sl]), v_lambda=0.3)
        buf = torch.zeros(m, 8 + H * V, dtype=dtype, device=device)
        O.sink_attention(q, kp, vp, torch.zeros(H, device=device), meta, scale, 0, size, 1.0, dtype, buf, 8, keep_first=keep, gate=r[:, v0 + G * V:])
        assert float(buf[:, :8].abs().max()) == 0.0
        outs.append(buf[:, 8:])
        at += m
    rd, pos = rows.double(), torch.arange(n)
    q, k = (oracle.rms(oracle.rotate_half(rd[:, c:c + h * D].view(n, h, D), pos, inv.double(), mult), 1e-3) for c, h in ((pad, H), (pad + H * D, G)))
    v = (0.7 * rd[:, v0:v0 + G * V] + 0.3 * vf.double()).view(n, G, V)
    want = attention_reference(q, k, v, 0, n, scale, size, keep, rd[:, v0 + G * V:])
    close(torch.cat(outs), want, tol if dtype == torch.bfloat16 else 2e-5)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("half,after,weights", [(False, False, True), (True, False, True), (False, True, False), (True, True, True), (True, False, False)])
def test_prologue_forms(half, after, weights, device, dtype, tol):
    """Every combination of pair layout, norm before / behind the rotation and norm weights the prologue offers."""
    O = get_backend("b200" if device == "cuda" else "reference")
    g = torch.Generator().manual_seed(4)
    rn = lambda *s: torch.randn(*s, generator=g)
    T, H, G, D, V, eps = 9, 3, 1, 40, 6, 1e-3
    rows, w = rn(T, (H + G) * D + G * V).to(dtype), (1 + 0.3 * rn(D)) if weights else None
    inv = torch.rand(12, generator=g)
    kp, vp = torch.zeros(3, G, 8, D, dtype=dtype, device=device), torch.zeros(3, G, 8, V, dtype=dtype, device=device)
    dw = w.to(device) if weights else None
    q = O.qk_norm_rope_append(rows.to(device), 0, H * D, (H + G) * D, H, D, dw, dw, eps, inv.to(device), kp, vp, meta_of([T], [0], [[2, 1]], 8, device), half=half,
                              norm_after=after, rot_mult=1.3)

    def rot(x):
        if half:
            return oracle.rotate_half(x, torch.arange(T), inv.double(), 1.3)
        a = torch.arange(T).double()[:, None, None] * inv.double()
        u, v = x[..., 0:24:2], x[..., 1:24:2]
        r = torch.stack([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)], -1).flatten(-2) * 1.3
        return torch.cat([r, x[..., 24:]], -1)

    nrm = lambda x: oracle.rms(x, eps) * (w.double() if weights else 1.0)
    x = rows.double()
    for got, c, h in ((q, 0, H), (kp[[2, 1], 0].reshape(16, 1, D)[:T], H * D, G)):
        r = x[:, c:c + h * D].view(T, h, D)
        close(got, nrm(rot(r)) if after else rot(nrm(r)), tol if dtype == torch.bfloat16 else 1e-5)
    assert torch.equal(vp[[2, 1], 0].reshape(16, V)[:T].cpu(), rows[:, (H + G) * D:])


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("K,F", [(40, 24), (128, 256), (36, 21)])
def test_feed_forward_and_residual_alone(K, F, device, dtype, tol):
    """GELU-GLU (fused product where the sizes allow it) and the residual step with a factor."""
    O = get_backend("b200" if device == "cuda" else "reference")
    g = torch.Generator().manual_seed(K)
    rn = lambda *s: torch.randn(*s, generator=g)
    x, wg, wu = rn(19, K).to(dtype), (rn(F, K) * 2 * K ** -0.5).to(dtype), (rn(F, K) * K ** -0.5).to(dtype)
    lw = lambda w: LinearWeight(weight=w.to(device))
    got = O.gelu_gated_up(x.to(device), lw(wg), lw(wu))
    close(got, oracle.gelu_tanh(x.double() @ wg.double().T) * (x.double() @ wu.double().T), tol if dtype == torch.bfloat16 else 1e-5)
    h, y, w = rn(5, K), rn(5, K), 1 + 0.2 * rn(K)
    hd = h.clone().to(device)
    ha = O.scaled_add_norm_(hd, y.to(device), None, w.to(device), 1e-3, dtype, mult=0.3)
    want = h.double() + 0.3 * y.double()
    close(hd, want, 1e-5)
    close(ha, oracle.rms(want, 1e-3) * w.double(), tol if dtype == torch.bfloat16 else 1e-5)


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
    """Prefill against token-by-token decoding and prompts cut anywhere (page edges at 16 and 32, windows of 7, 9 and 16 that start inside
    an earlier portion, convolution histories of 3 and 4 inputs that reach into the portions before, 2-token portions)."""
    cfgd = make_cfg(STACK)
    model, sd = make_model(cfgd, device, dtype)
    t = toks(sum(portions), seed=1)
    close(in_portions(model, t, portions), oracle.forward(cfgd, sd, t), tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_ragged_batch_and_reuse_of_pages_and_slots(device, dtype, tol):
    """Unequal requests in one batch (portions beside single tokens) equal each alone; a pool of 5 pages and 2 state slots serves 4
    requests one pair after another, so every page and slot is used again — by a request that must not see what the last one left."""
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


def sharp(sd, layer):
    """No query / key biases: nothing is common to all keys of a layer, so single keys stand out."""
    sd[f"l{layer}.mix.q.b"].zero_(), sd[f"l{layer}.mix.k.b"].zero_()


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("size,keep,seed", [(9, 4, 1), (16, 16, 4), (5, 1, 1)])
def test_window_and_kept_edges_show(size, keep, seed, device, dtype, tol):
    """Sharp scores and a large share of the mixer in the residual make single keys count.  The oracle with a window or a kept prefix that is one position off gives other logits at
    the positions where the difference begins, so a wrong edge would show: in a prompt, in portions that start inside a window, and decoded
    one by one across edges and page borders (pages of 16)."""
    tol = min(tol, 3e-2)
    cfgd = make_cfg([att(4, 2, 8, 12, size, keep, 4, 0.8, ff=None)], mult=4.0)
    model, sd = make_model(cfgd, device, dtype, edit=lambda sd: sharp(sd, 0))
    t = toks(44, seed=seed)
    want = oracle.forward(cfgd, sd, t)
    for ds, dk, first in ((-1, 0, size + keep - 1), (1, 0, size + keep), (0, -1, size + keep - 1), (0, 1, size + keep)):
        other = copy.deepcopy(cfgd)
        other["layers"][0]["mixer"]["mask"] = dict(size=size + ds, keep_first=keep + dk)
        wrong = oracle.forward(other, sd, t)
        diff = (wrong - want).abs().max(-1).values
        assert diff[:first].max() == 0 and diff[first:].max() > 0.06 * want.abs().max(), (ds, dk)
    close(run_whole(model, t), want, tol)
    close(decode_after(model, t, 4), want, tol)
    close(in_portions(model, t, [5, 6, 2, 14, 17]), want, tol)
    close(in_portions(model, t, [20, 24]), want, tol)          # tensor-core form: portions of 16 tokens and more


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_far_kept_key_among_hundreds(device, dtype, tol):
    """With a window of 30 over 330 tokens only the kept first tokens are far; one of them holds most of a query's weight.  Other tokens there
    move the late logits, tokens just behind the kept ones do not.  Prompt, decode, portions."""
    layer = att(2, 1, 16, 8, 30, 6, 4, 6.0, base=1e5, ff=None)
    cfgd = make_cfg([layer], mult=1.0)
    model, sd = make_model(cfgd, device, dtype, edit=lambda sd: sharp(sd, 0))
    t = toks(330, seed=17)
    want = oracle.forward(cfgd, sd, t)
    kept = oracle.forward(cfgd, sd, [(x + 1 + i) % 96 if i < 6 else x for i, x in enumerate(t)])
    behind = oracle.forward(cfgd, sd, [(x + 1 + i) % 96 if 6 <= i < 200 else x for i, x in enumerate(t)])
    assert (kept[300:] - want[300:]).abs().max() > 3 * SHOWS * want.abs().max() and (behind[300:] - want[300:]).abs().max() < 1e-9
    kw = dict(pages=22)
    close(run_whole(model, t, **kw), want, tol)
    close(in_portions(model, t, [2, 120, 50, 128, 2, 20] + [1] * 8, **kw), want, tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_sink_gate_and_value_mixing_show(device, dtype, tol):
    """Leaving out the 1 in the denominator, the value mixing, or cos / sin's factor moves the logits; lambda is taken per layer, the first
    mixing layer's own is not used, and its values are taken before mixing (three mixing layers, a layer without mixing between them)."""
    layers = [A_MQ, att(4, 2, 8, 12, 12, 2, 4, 1.0, ff=None), scan(16, 4, 2, 3, ff=None), att(2, 2, 16, 12, 20, 0, 8, 0.7, ff=None), A_GQ]
    cfgd = make_cfg(layers, mult=1.0)

    def edit(sd):
        for i, lam in ((1, 5.0), (3, 0.7), (4, -0.6)):
            sd[f"l{i}.mix.vmix"].fill_(lam)

    model, sd = make_model(cfgd, device, dtype, edit=edit)
    t = toks(30, seed=8)
    want = oracle.forward(cfgd, sd, t)
    for faults in (dict(sink=0.0), dict(vmix=0.0), dict(rot_mult=1.0)):
        assert (oracle.forward(cfgd, sd, t, faults=faults) - want).abs().max() > 2 * SHOWS * want.abs().max(), faults
    close(run_whole(model, t), want, tol)
    close(decode_after(model, t, 11), want, tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_far_token_lives_in_the_state(device, dtype, tol):
    """With slow decays and no attention only the recurrent state carries the first tokens to position 60, four pages on: other tokens there
    and a state that is lost on the way move the late logits.  In a prompt, in decoding, and in portions."""
    cfgd = make_cfg([scan(24, 6, 3, 4, ff=None)], mult=1.0)
    edit = lambda sd: (sd["l0.mix.A_log"].fill_(-6.0), sd["l0.mix.dt.b"].fill_(-1.0), sd["l0.mix.o"].mul_(3.0))
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
    """A 290-token prompt over windows of 270 and without a window, then single tokens whose keys are split over CTAs and merged on the GPU;
    prompts long enough for the scan's time slices and for the tensor-core attention."""
    cfgd = make_cfg([att(4, 2, 8, 16, 270, 9, 8, 0.5), scan(16, 5, 2, 4, ff=None), att(2, 1, 16, 40, 0, 0, 4, 0.4, v_mix=False, ff=None), scan(8, 20, 3, 2)])
    model, sd = make_model(cfgd, device, dtype)
    t = toks(296, seed=9)
    want = oracle.forward(cfgd, sd, t)
    close(decode_after(model, t, 290, pages=21), want, tol * (2 if dtype == torch.bfloat16 else 1))
    close(in_portions(model, t, [40, 200, 3, 45, 2, 6], pages=21), want, tol * (2 if dtype == torch.bfloat16 else 1))


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_long_decode(device, dtype, tol):
    """Single-token steps after a 3-token prompt: states are read and written every step, windows move over page borders."""
    cfgd = make_cfg([M_A, A_GQ, M_C, A_GQ2])
    model, sd = make_model(cfgd, device, dtype)
    t = toks(153, seed=5)
    close(decode_after(model, t, 3), oracle.forward(cfgd, sd, t), tol * (2 if dtype == torch.bfloat16 else 1))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-4), (torch.bfloat16, 6e-2)])
def test_tensor_core_sizes(dtype, tol):
    """Widths and feed-forwards that are multiples of 128, head sizes of 64 and 128: bf16 takes the tensor-core GEMMs (GELU-GLU in the
    two-weight epilogue, biases in the projection's) and both sizes of the tensor-core attention; pages of 16 and 64."""
    cfgd = make_cfg([scan(256, 16, 8, 4, ff=256), att(4, 2, 128, 128, 90, 20, 64, 0.1, ff=256), att(8, 2, 64, 128, 33, 2, 32, 0.15, ff=None), scan(128, 32, 16, 3, ff=128)], width=128)
    model, sd = make_model(cfgd, "cuda", dtype)
    t = toks(200, seed=2)
    want = oracle.forward(cfgd, sd, t)
    for kw in (dict(pages=14, page_size=16), dict(pages=5, page_size=64)):
        close(in_portions(model, t, [150, 2, 30, 10] + [1] * 8, **kw), want, tol)


def random_cfg(rng):
    """A configuration drawn at random: 2 to 5 layers of either mixer in any order, every size and constant drawn anew; value-mixing layers
    share their key/value heads and value width."""
    G, V = rng.choice([1, 2, 3]), rng.choice([5, 8, 24, 40])

    def layer():
        ff = rng.choice([None, 24, 40, 51])
        if rng.random() < 0.45:
            return scan(rng.choice([16, 31, 64]), rng.choice([1, 3, 8, 16, 20, 40]), rng.choice([1, 4, 7, 16]), rng.choice([1, 2, 3, 4, 6]), ff)
        mix = rng.random() < 0.7
        kv, dim = (G if mix else rng.choice([1, 2])), rng.choice([6, 8, 16, 32, 72])
        return att(kv * rng.choice([1, 2, 3, 5]), kv, dim, V if mix else rng.choice([8, 20]), rng.choice([0, 1, 5, 16, 24, 33]), rng.choice([0, 1, 4, 20]),
                   rng.choice([0, dim, dim // 2 // 2 * 2, 2]), rng.choice([0.2, 0.5, 1.0]), mix, ff, base=rng.choice([10000.0, 50.0]), factor=rng.choice([None, 1.0, 2.0, 8.0]),
                   original=rng.choice([16, 64, 1024]), fast=rng.choice([8.0, 32.0]), slow=rng.choice([1.0, 0.5]))

    return make_cfg([layer() for _ in range(rng.randint(2, 5))], width=rng.choice([40, 64, 72, 51]), vocab=rng.choice([50, 77]), eps=rng.choice([1e-6, 1e-3]),
                    mult=rng.choice([0.3, 0.5, 1.0]), scale=rng.choice([1.0, 4.0, 0.5]))


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("seed", range(1, 9))
def test_random_configurations(seed, device, dtype, tol):
    """Configurations drawn at random, two requests stepped in portions of random sizes side by side, every position against the oracle."""
    import random

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
        close(torch.cat(got[n]), want[n], tol)


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
    need, found = (0.0 if dtype == torch.float32 else 0.25), []
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


def test_stack_of_attention_layers_needs_no_slots():
    cfgd = make_cfg([A_GQ, A_MQ])
    model, sd = make_model(cfgd)
    s = session(model)
    assert s.table.slots is None
    t = toks(20, seed=2)
    close(run_whole(model, t), oracle.forward(cfgd, sd, t), 2e-4)


def test_config_reader_takes_every_size_from_the_file():
    cfg = ModelConfig.from_dict(make_cfg([M_C, A_GQ, A_FREE], width=40, vocab=50, eps=3e-3, mult=0.25, scale=7.0))
    assert (cfg.model_type, cfg.hidden_size, cfg.vocab_size, cfg.num_hidden_layers) == ("podurax", 40, 50, 3)
    assert cfg.rms_norm_eps == 3e-3 and cfg.residual_mult == 0.25 and cfg.embedding_scale == 7.0
    assert cfg.layer_specs[1]["mixer"]["mask"] == dict(size=7, keep_first=3) and cfg.layer_specs[0]["mixer"]["state"] == 9 and cfg.layer_specs[0]["mlp"] is None
    bad = [dict(type="unknown", mixer=dict(heads=1), mlp=None)], [att(5, 2, 8, 8, 4, 0, 4, 1.0)], [att(4, 2, 8, 8, 4, 0, 5, 1.0)], [att(4, 2, 8, 8, 4, 0, 10, 1.0)], \
        [A_GQ, att(3, 3, 8, 12, 7, 3, 4, 0.8)], [scan(8, 0, 1, 1)], [dict(M_A, mlp=dict(kind="moe", ff=8))]
    for layers in bad:
        with pytest.raises(ValueError):
            ModelConfig.from_dict(make_cfg(layers))


def test_cache_layout_and_weights():
    model, sd = make_model(make_cfg(STACK))
    lay = model.cache_layout()
    assert lay[0][0] == "state" and lay[0][1]["S"][0] == (24, 6) and lay[0][1]["conv"][0] == (3, 24)
    assert lay[1] == ("paged_kv", 2, 8, 12, torch.float32) and lay[2][:4] == ("paged_kv", 2, 16, 12)
    kv = StageExecutor(model, 4, 16, num_state_slots=3).kv
    assert kv.num_slots == 3 and kv.k[1].shape == (4, 2, 16, 8) and kv.v[2].shape == (4, 2, 16, 12) and kv.state[3]["S"].shape == (3, 16, 9) and kv.k[0] is None
    assert model.v_source == 1 and model.layer_weights[4]["vmix"] == 0.0 and model.layer_weights[5]["vmix"] != 0.0
    with pytest.raises(ValueError):                       # a tensor the design does not have
        build_stage(ModelConfig.from_dict(make_cfg(STACK)), None, torch.float32, "cpu").load_state(dict(sd, extra=torch.zeros(1)))
    with pytest.raises(ValueError):                       # a tensor of another shape
        build_stage(ModelConfig.from_dict(make_cfg(STACK)), None, torch.float32, "cpu").load_state({k: (v[:-1] if k == "l0.mix.in" else v) for k, v in sd.items()})


@pytest.mark.timeout(300)
def test_command_line_generation():
    """``generate.py`` on a synthetic model of the design: tokenizer, engine, sampler and the printed statistics."""
    import subprocess

    repo = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(repo, "generate.py"), "--model", "synthetic:tiny-podurax", "--prompt", "hello", "--max_tokens", "8",
                        "--device", "cpu", "--no_chat_template"], capture_output=True, text=True, timeout=240,
                       env=dict(os.environ, PYTHONPATH=repo, OMP_NUM_THREADS="1"))
    assert r.returncode == 0, r.stdout + r.stderr
    assert "Generation:" in r.stdout and "tokens-per-sec" in r.stdout


@pytest.mark.timeout(300)
def test_trace_replay_from_a_model_folder(tmp_path):
    """``bin/trace_run`` on a folder with config.json and safetensors: portions and single tokens of two requests, a pool of exactly the live
    pages, logits against the oracle."""
    import json
    import subprocess

    import numpy as np
    from safetensors.torch import save_file

    repo = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfgd = make_cfg([M_A, A_GQ, A_GQ2], vocab=50)
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
