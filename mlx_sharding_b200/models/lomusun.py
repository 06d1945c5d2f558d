"""Lomusun: a decoder stack of parallel blocks — in every layer the mixer and a mixture of experts read the SAME normed input and enter the
residual together — with learned positions.  A layer's mixer is windowed attention BESIDE a gated delta rule, or windowed attention with
convolved queries, keys and values.  No reference counterpart (the reference serves Llama / Gemma-2 / DeepSeek-V2 only).

Residual (``x = embed[token] + pos[p]``, fp32; ``rms(u) = u / sqrt(mean(u^2) + eps)``; logits = ``embed (rms(x) * final.norm)``):

    h = rms(x) * norm1        x <- x + (mixer(h) + experts(h))

Mixers (``h``: the layer's input):

* ``parallel``: ``left_scale * attention(h) + right_scale * delta(h)``.  Attention: ONE RMS norm over all heads' entries of the query row (and
  of the key row) with weights of that size; no rotation; scores ``q . k * scale - 2^(-8 (h + 1) / H) (i - j)``; the last ``mask.size``
  positions are visible; ``exp(sink_h)`` joins the softmax denominator; the heads' output times ``sigmoid(W_g h)`` per element.  Delta rule:
  ``q, k`` (``kv_heads x dim``) and ``v`` (``heads x vdim``) pass a short causal convolution and SiLU; ``q, k`` become unit vectors per head (``q``
  times ``dim^-1/2``); ``b = sigmoid(W_b h)``, ``g = exp(-exp(A_log) softplus(W_a h + dt_bias))``, one each per head; ``S <- g S``, ``u = b (v -
  S^T k)``, ``S <- S + k u^T``, ``o = S^T q``; ``o`` per head divided by its root mean square, times a weight shared by the heads, times
  ``silu(W_g h)``.
* ``attention``: ``q, k, v`` pass a short causal convolution without activation; scores ``q . k * scale + rel[bucket(i - j), h]`` with one table
  row per distance in its first half and logarithmically wider buckets up to ``bias_max`` behind it; the last ``mask.size`` positions are
  visible; ordinary softmax; every head's output times ``sigmoid(W_g h)_head``.  A layer with ``kv_from`` has queries alone and reads the named
  layer's cached keys and values.

Experts: sigmoid scores, the ``top`` largest ``score + correction`` are chosen, weights = scores over their sum, times ``router.scale``, on the
outputs of clamped-GLU experts (no biases).

Precision: residual, norms, scores / softmax, the router, and everything inside the recurrence (unit norms, decays, step sizes, state) are
fp32 in both dtypes; projections, short convolutions, cached rows and expert activations are bf16 on the serving path with fp32
accumulation.

Framework integration: layer order and every size come from ``ModelConfig.layer_specs``; a ``parallel`` layer keeps keys / values in its own
pair of paged pools AND the matrix state and convolution inputs in a slot, an ``attention`` layer pools and convolution inputs, a ``kv_from``
layer its query convolution's inputs beside aliased pools (``engine/kv_cache.py::HybridCache``).  The ops are ``ops/reference.py`` (unfused
PyTorch) / ``ops/b200.py`` (``ops/csrc/streams.cu``, ``sinkattn.cu``, ``attention_prefill.cu``, ``hybrid.cu``).
"""
from __future__ import annotations

from fractions import Fraction

import torch

from ..ops import BatchMeta, LinearWeight, RopeSpec
from .hybrid import HybridStage


def bucket_starts(rows: int, far: int):
    """Smallest distance of every row of a distance table with ``rows`` rows: row ``n`` for the distances ``n < half = rows // 2``, then ``half +
    floor(ln(n / half) / ln(far / half) * (rows - half))``, at most ``rows - 1``.  Exact: the step to ``half + k`` lies where ``(n / half)^(rows -
    half) >= (far / half)^k``, compared in integers."""
    half = rows // 2
    if half < 1 or far <= half:
        raise ValueError(f"distance table: {rows} rows need bias_max > {half} (got {far})")
    m, starts = rows - half, list(range(half + 1))
    for k in range(1, m):
        bound = Fraction(far, half) ** k
        lo, hi = starts[-1], far
        while lo < hi:                                     # smallest n with (n / half)^m >= bound
            mid = (lo + hi) // 2
            lo, hi = (lo, mid) if Fraction(mid, half) ** m >= bound else (mid + 1, hi)
        starts.append(lo)
    return starts


def distance_bias(rel: torch.Tensor, far: int) -> torch.Tensor:
    """Table ``[rows, heads]`` -> bias per head and distance, fp32 ``[heads, L]``; distances behind ``L - 1`` share the last row."""
    starts = bucket_starts(rel.shape[0], int(far))
    row = torch.bucketize(torch.arange(starts[-1] + 1), torch.tensor(starts), right=True) - 1
    return rel.float().cpu()[row].t().contiguous()


class LomusunStage(HybridStage):
    arch = "lomusun"
    UNIT_EPS = 1e-6            # inside the root of the unit vectors of the delta rule (fixed by the design)

    @property
    def max_positions(self) -> int:
        return int(self.cfg.max_position_embeddings)

    # ---- cache geometry ---------------------------------------------------------------------------------------------
    def cache_layout(self):
        out = []
        for L in self.specs:
            m = L["mixer"]
            a = m["left"] if L["type"] == "parallel" else m
            H, G, D, V = (int(a[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
            conv = lambda taps, rows: ((taps - 1, rows), self.dtype)
            if L["type"] == "parallel":
                h, g, d, v, K = (int(m["right"][k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
                out.append(("paged_kv", G, D, V, self.dtype, {"S": ((h, d, v), torch.float32), "conv": conv(K, 2 * g * d + h * v)}))
            elif m.get("kv_from") is None:
                out.append(("paged_kv", G, D, V, self.dtype, {"conv": conv(int(m["conv"]), H * D + G * (D + V))}))
            else:
                out.append(("alias", int(m["kv_from"]), {"conv": conv(int(m["conv"]), H * D)}))
        return out

    # ---- weights ----------------------------------------------------------------------------------------------------
    def _take(self, sd, key, *shape):
        w = sd.pop(key)
        if tuple(w.shape) != shape:
            raise ValueError(f"{key}: shape {tuple(w.shape)} does not fit the configuration ({shape})")
        return w

    def _vec32(self, sd, key, *shape):
        return self._take(sd, key, *shape).to(device=self.device, dtype=torch.float32).contiguous()

    def _qkv(self, sd, p, parts, taps):
        """Adjacent projections that pass one short convolution: ``parts`` = ``[(name, rows)]`` -> (weight, convolution weights)."""
        W = self.cfg.hidden_size
        w = torch.cat([self._take(sd, p + n, rows, W) for n, rows in parts])
        return w, torch.cat([self._vec32(sd, p + n + ".conv", rows, taps) for n, rows in parts]).contiguous()

    def _parallel_weights(self, sd, p, m):
        a, r, W = m["left"], m["right"], self.cfg.hidden_size
        H, G, D, V = (int(a[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        h, g, d, v, K = (int(r[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        w = {}
        parts = [("l" + n, self._take(sd, p + "left." + n, rows, W), None) for n, rows in (("q", H * D), ("k", G * D), ("v", G * V), ("g", H * V))]
        qkv, w["conv"] = self._qkv(sd, p + "right.", [("q", g * d), ("k", g * d), ("v", h * v)], K)
        parts += [("qkv", qkv, None)] + [(n, self._take(sd, p + "right." + n, rows, W), None) for n, rows in (("a", h), ("b", h), ("g", h * v))]
        w["proj"], w["seg"] = self._fused(parts)
        w["qn"], w["kn"] = self._vec32(sd, p + "left.q.norm", H * D), self._vec32(sd, p + "left.k.norm", G * D)
        w["sink"] = self._vec32(sd, p + "left.sink", H)
        w["slopes"] = torch.tensor([2.0 ** (-8.0 * (i + 1) / H) for i in range(H)], dtype=torch.float32, device=self.device)
        w["A_log"], w["dt_bias"] = self._vec32(sd, p + "right.A_log", h), self._vec32(sd, p + "right.dt_bias", h)
        # one weight vector for all heads; the branch's factor rides on it
        w["gnorm"] = (self._vec32(sd, p + "right.norm", v) * float(m.get("right_scale", 1.0))).repeat(h).contiguous()
        # both output projections as ONE product over [attention output | delta output] (each scaled by its branch factor where it is
        # written); the attention part is padded to a multiple of 8 columns, the whole likewise
        wl, wr = self._take(sd, p + "left.o", W, H * V), self._take(sd, p + "right.o", W, h * v)
        pad = lambda t: torch.cat([t, t.new_zeros(t.shape[0], (-t.shape[1]) % 8)], 1)
        wl, wr = pad(wl), pad(wr)
        w["o_split"], w["o_cols"] = wl.shape[1], wl.shape[1] + wr.shape[1]
        w["o"] = self._lw(torch.cat([wl, wr], 1))
        return w

    def _attention_weights(self, sd, p, m):
        H, G, D, V = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        W, w = self.cfg.hidden_size, {}
        qkv, w["conv"] = self._qkv(sd, p, [("q", H * D), ("k", G * D), ("v", G * V)][:3 if m.get("kv_from") is None else 1], int(m["conv"]))
        w["proj"], w["seg"] = self._fused([("qkv", qkv, None), ("g", self._take(sd, p + "g", H, W), None)])
        rel = sd.pop(p + "rel")
        if rel.dim() != 2 or rel.shape[1] != H:
            raise ValueError(f"{p}rel: shape {tuple(rel.shape)} does not fit the configuration")
        w["bias"] = distance_bias(rel, int(m["bias_max"])).to(self.device)
        w["o"] = self._lw(self._take(sd, p + "o", W, H * V))
        return w

    def _moe_weights(self, sd, p, mlp):
        E, F, W = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"]), self.cfg.hidden_size
        bank = lambda n, *shape: LinearWeight(weight=torch.stack([self._take(sd, f"{p}e{e}.{n}", *shape) for e in range(E)])
                                              .to(device=self.device, dtype=self.dtype).contiguous())
        return dict(e_gate=bank("gate", F, W), e_up=bank("up", F, W), e_down=bank("down", W, F), router=self._vec32(sd, p + "router", E, W),
                    correction=self._vec32(sd, p + "correction", E) if p + "correction" in sd else None)

    def load_state(self, sd, strict: bool = True):
        sd = dict(sd)
        W = self.cfg.hidden_size
        emb = self._take(sd, "embed", self.cfg.vocab_size, W)
        self.embed_tokens = LinearWeight(weight=emb.to(device=self.device, dtype=self.dtype).contiguous())
        self.lm_head = self._lw(emb) if emb.shape[0] % 8 else self.embed_tokens
        self.lm_head.n_real = emb.shape[0]
        self.pos_table = self._take(sd, "pos", self.max_positions, W).to(device=self.device, dtype=self.dtype).contiguous()
        for i, L in enumerate(self.specs):
            p = f"l{i}."
            w = (self._parallel_weights if L["type"] == "parallel" else self._attention_weights)(sd, p + "mix.", L["mixer"])
            w["norm1"] = self._vec32(sd, p + "norm1", W)
            if L["mlp"]:
                w.update(self._moe_weights(sd, p + "mlp.", L["mlp"]))
            self.layer_weights[i] = w
        self.norm_w = self._vec32(sd, "final.norm", W)
        if strict and sd:
            raise ValueError(f"unexpected checkpoint tensors: {sorted(sd)[:8]} ...")
        self.rope = RopeSpec(inv_freq=torch.zeros(0, device=self.device), rot_dim=0, interleaved=False)
        return self

    # ---- forward ----------------------------------------------------------------------------------------------------
    def _parallel(self, w, m, ha, meta, kpool, vpool, st):
        O, eps, seg, a, r = self.ops, self.cfg.rms_norm_eps, w["seg"], m["left"], m["right"]
        H, D, V = (int(a[k]) for k in ("heads", "dim", "vdim"))
        h, g, d, v = (int(r[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        u = O.linear_any(ha, w["proj"], self.dtype)                            # [lq | lk | lv | lg | qkv | a | b | g]
        padded = w["o_split"] != H * V or w["o_cols"] - w["o_split"] != h * v
        both = (torch.zeros if padded else torch.empty)(ha.shape[0], w["o_cols"], dtype=self.dtype, device=u.device)

        def delta():
            qkv = O.causal_conv_silu(self._cols(u, seg, "qkv"), w["conv"], None, st["conv"], meta)
            o = O.delta_scan(qkv, self._cols(u, seg, "b"), self._cols(u, seg, "a"), w["dt_bias"], w["A_log"], st["S"], meta, h, g, d, v, float(d) ** -0.5,
                             self.UNIT_EPS)
            O.gated_rmsnorm(o, self._cols(u, seg, "g"), w["gnorm"], eps, h, "silu_post", self.dtype, both, w["o_split"])

        join = O.run_aside(delta, 1)                                           # beside the attention: they meet in the output product
        q = O.qk_norm_rope_append(u, seg["lq"][0], seg["lk"][0], seg["lv"][0], H, D, w["qn"], w["kn"], eps, self.rope.inv_freq, kpool, vpool, meta, whole=True)
        O.sink_attention(q, kpool, vpool, w["sink"], meta, float(a["scale"]), 0, int((a.get("mask") or {}).get("size", 0) or 0),
                         float(m.get("left_scale", 1.0)), self.dtype, both, 0, gate=self._cols(u, seg, "lg"), slopes=w["slopes"])
        if join is not None:
            join.wait()
        return self._mm(both, w["o"], True)

    def _attention(self, w, m, ha, meta, kpool, vpool, st):
        O, seg = self.ops, w["seg"]
        u = O.linear_any(ha, w["proj"], self.dtype)                            # [q | k | v | g] or, on another layer's rows, [q | g]
        q = O.conv_qkv_append(self._cols(u, seg, "qkv"), w["conv"], st["conv"], int(m["heads"]), int(m["dim"]), kpool, vpool, meta)
        o = O.sink_attention(q, kpool, vpool, None, meta, float(m["scale"]), 0, int((m.get("mask") or {}).get("size", 0) or 0), 1.0, self.dtype,
                             gate=self._cols(u, seg, "g"), dist_bias=w["bias"])
        return self._mm(o, w["o"], True)

    def _experts(self, w, mlp, ha, out):
        O, r = self.ops, mlp["router"]
        idx, wts = O.sigmoid_router(ha, w["router"], int(r["experts"]), int(r["top"]), w["correction"], True, float(r.get("scale", 1.0)))
        O.moe_clamped_experts(ha, idx, wts, w["e_gate"], w["e_up"], w["e_down"], float(mlp["expert"]["limit"]), on_input=False, out=out)

    @torch.inference_mode()
    def forward(self, x, meta: BatchMeta, kv, all_logits: bool = False, layer_out=None):
        """``x``: token ids ``[T]``.  Returns fp32 logits ``[B, V]`` (``[T, V]`` with ``all_logits``).  ``layer_out``: optional list that
        receives a copy of the residual after every layer."""
        O, c, n = self.ops, self.cfg, len(self.specs)
        if meta.state_slots is None:
            raise ValueError("Lomusun needs state slots in the step metadata (BatchMeta.build(..., state_slots=...))")
        tokens = x.to(torch.int64).contiguous()
        h = O.stream_embed(self.embed_tokens.weight, tokens, 1.0, 1, self.pos_table, meta.positions).view(tokens.numel(), c.hidden_size)      # fp32 residual
        ha = O.rmsnorm_cast(h, self.layer_weights[0]["norm1"], c.rms_norm_eps, self.dtype)
        for i, L in enumerate(self.specs):
            w = self.layer_weights[i]
            mixer = self._parallel if L["type"] == "parallel" else self._attention
            ye, join = None, None
            if L["mlp"]:
                ye = torch.empty_like(h)
                join = O.run_aside(lambda: self._experts(w, L["mlp"], ha, ye))  # beside the mixer: they meet in the residual
            y = mixer(w, L["mixer"], ha, meta, kv.k[i], kv.v[i], kv.state[i])
            if join is not None:
                join.wait()
            nxt = self.layer_weights[i + 1]["norm1"] if i + 1 < n else self.norm_w
            ha = O.scaled_add_norm_(h, y, None, nxt, c.rms_norm_eps, self.dtype, extra=ye)
            if layer_out is not None:
                layer_out.append(h.clone())
        if not all_logits and meta.num_tokens != meta.num_seqs:
            ha = ha.index_select(0, meta.last_idx.long())
        return self._mm(ha, self.lm_head, True).contiguous()

    __call__ = forward


Model = LomusunStage
