"""Podurax: a pre-norm decoder stack whose layers have one *mixer* — a selective scan (Mamba with one step size per channel) or sliding-window
attention that keeps the first tokens visible — and an optional dense GELU-GLU feed-forward.  No reference counterpart (the reference
serves Llama / Gemma-2 / DeepSeek-V2 only).

Residual (``x = embed[token] * embedding_scale``, fp32; ``rms(u) = u / sqrt(mean(u^2) + eps)``; ``m = residual_mult``):

    x <- x + m * mixer(rms(x) * norm1)        x <- x + m * W_down(gelu_tanh(W_gate h) * (W_up h)),  h = rms(x) * norm2        logits = head(rms(x) * final.norm)

Mixers (``h``: the sublayer's input):

* ``mamba1``: ``[x | z] = W_in h``; ``x`` passes a short causal convolution and SiLU; ``[dt | B | C] = W_x x``; per channel ``c`` the step
  ``dt_c = softplus((W_dt dt)_c + b_c)``, the state ``S_c <- exp(-dt_c exp(A_log_c)) S_c + dt_c x_c B`` and ``y_c = S_c . C + D_c x_c``; output
  projection of ``y * silu(z)``.
* ``attention``: biased projections; queries and keys are rotated (first ``rot.dims`` entries, half-split pairs, YaRN frequencies, cos and sin
  times ``0.1 ln(factor) + 1``), then divided by their root mean square per head; values of the ``v_mix`` layers behind the first such layer
  are ``(1 - lambda) v + lambda v_first`` (the first such layer's values of the same token) before they are cached; a query sees the last
  ``mask.size`` positions and the first ``mask.keep_first`` of the sequence; softmax with a 1 added to the denominator; every head's
  output times ``sigmoid(W_g h)_head``; output projection.

Precision: residual, norms, positions and angles, scores / softmax, step sizes, decays and the recurrent state are fp32 in both dtypes;
projections, the short convolution and the feed-forward's activation run in the model dtype (bf16 on the serving path) with fp32
accumulation.

Framework integration: layer order and every size come from ``ModelConfig.layer_specs``; a ``mamba1`` layer keeps its state and the
convolution's last inputs in per-sequence state slots, an ``attention`` layer keeps keys and (mixed) values in its own pair of paged pools
(``engine/kv_cache.py::HybridCache``).  The ops are ``ops/reference.py`` (unfused PyTorch) / ``ops/b200.py`` (``ops/csrc/selscan.cu``,
``sinkattn.cu``, ``streams.cu``, ``hybrid.cu``).
"""
from __future__ import annotations

import math

import torch

from ..ops import BatchMeta, LinearWeight, RopeSpec
from .base import yarn_inv_freq
from .hybrid import HybridStage, pad_cols


class PoduraxStage(HybridStage):
    arch = "podurax"
    SINK_SCORE = 0.0           # the softmax has one keyless term of this score (fixed by the design)

    def __init__(self, cfg, spec=None, dtype=torch.bfloat16, device="cpu", backend=None):
        super().__init__(cfg, spec, dtype, device, backend)
        mixing = [i for i, L in enumerate(self.specs) if L["type"] == "attention" and L["mixer"].get("v_mix")]
        self.v_source = mixing[0] if mixing else None

    # ---- cache geometry ---------------------------------------------------------------------------------------------
    def cache_layout(self):
        out = []
        for L in self.specs:
            m = L["mixer"]
            if L["type"] == "mamba1":
                out.append(("state", {"S": ((int(m["inner"]), int(m["state"])), torch.float32), "conv": ((int(m["conv"]) - 1, int(m["inner"])), self.dtype)}))
            else:
                out.append(("paged_kv", int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), self.dtype))
        return out

    # ---- weights ----------------------------------------------------------------------------------------------------
    def _expect(self, key, w, rows, cols=None):
        if w.shape[0] != rows or (cols is not None and w.shape[1] != cols):
            raise ValueError(f"{key}: shape {tuple(w.shape)} does not fit the configuration")
        return w

    def _mamba1_weights(self, sd, p, m):
        I, N, R, K = (int(m[k]) for k in ("inner", "state", "dt_rank", "conv"))
        w = {}
        win = self._expect(p + "in", sd.pop(p + "in"), 2 * I)
        w["in"], w["seg"] = self._fused([("x", win[:I], None), ("z", win[I:], None)])
        w["conv"], w["conv_b"] = self._expect(p + "conv", self._f32(sd, p + "conv"), I, K), self._f32(sd, p + "conv.b")
        wx = self._expect(p + "x", sd.pop(p + "x"), R + 2 * N)
        # [dt | B | C], every segment at a multiple of 8 columns: the step-size product reads its segment in place (its weight has zero
        # columns for the padding)
        w["x"], w["xseg"] = self._fused([("dt", wx[:R], None), ("B", wx[R:R + N], None), ("C", wx[R + N:], None)])
        w["dt"] = self._lw(pad_cols(self._expect(p + "dt", sd.pop(p + "dt"), I, R)))
        w["dt_b"], w["A_log"], w["D"] = self._f32(sd, p + "dt.b"), self._expect(p + "A_log", self._f32(sd, p + "A_log"), I, N), self._f32(sd, p + "D")
        w["o"] = self._lw(self._expect(p + "o", sd.pop(p + "o"), self.cfg.hidden_size, I))
        return w

    def _attention_weights(self, sd, p, m):
        H, G, D, V = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        w = {}
        parts = [(n, self._expect(p + n, sd.pop(p + n), rows), sd.pop(p + n + ".b")) for n, rows in (("q", H * D), ("k", G * D), ("v", G * V))]
        w["proj"], w["seg"] = self._fused(parts + [("g", self._expect(p + "g", sd.pop(p + "g"), H), None)])
        lam = sd.pop(p + "vmix", None)
        w["vmix"] = float(lam.float()) if lam is not None else 0.0          # taken to the host once, at load
        w["o"] = self._lw(self._expect(p + "o", sd.pop(p + "o"), self.cfg.hidden_size, H * V))
        w["sink"] = torch.full((H,), self.SINK_SCORE, dtype=torch.float32, device=self.device)
        rot = m.get("rot") or {}
        n, base, sc = int(rot.get("dims", 0) or 0), float(rot.get("base", 10000.0)), rot.get("scaling")
        w["rot_mult"] = 1.0
        if n and sc:
            f = yarn_inv_freq(n, base, *(float(sc[k]) for k in ("factor", "original", "fast", "slow")))
            w["rot_mult"] = 0.1 * math.log(float(sc["factor"])) + 1.0
        else:
            f = (base ** (-2.0 * torch.arange(n // 2, dtype=torch.float64) / max(n, 1))).float()
        w["inv_freq"] = f.to(self.device)
        return w

    def load_state(self, sd, strict: bool = True):
        sd = dict(sd)
        self.embed_tokens = LinearWeight(weight=sd.pop("embed").to(device=self.device, dtype=self.dtype).contiguous())
        for i, L in enumerate(self.specs):
            p = f"l{i}."
            w = (self._mamba1_weights if L["type"] == "mamba1" else self._attention_weights)(sd, p + "mix.", L["mixer"])
            w["norm1"] = self._f32(sd, p + "norm1")
            if L["mlp"]:
                w["norm2"] = self._f32(sd, p + "norm2")
                w.update(gate=self._lw(sd.pop(p + "mlp.gate")), up=self._lw(sd.pop(p + "mlp.up")))
                w["down"] = self._lw(pad_cols(sd.pop(p + "mlp.down")))      # reads the padded gate / up rows
            self.layer_weights[i] = w
        self.norm_w = self._f32(sd, "final.norm")
        self.lm_head = self._lw(sd.pop("head"))
        if strict and sd:
            raise ValueError(f"unexpected checkpoint tensors: {sorted(sd)[:8]} ...")
        self.rope = RopeSpec(inv_freq=torch.zeros(1), rot_dim=0, interleaved=False)
        return self

    # ---- forward ----------------------------------------------------------------------------------------------------
    def _mamba1(self, w, m, ha, meta, st):
        O, I = self.ops, int(m["inner"])
        u = O.linear_any(ha, w["in"], self.dtype)                                    # [x | z]
        xc = O.causal_conv_silu(self._cols(u, w["seg"], "x"), w["conv"], w["conv_b"], st["conv"], meta)
        dbc = O.linear_any(xc, w["x"], self.dtype)                                   # [dt | B | C]
        dt = self._mm(dbc[:, :w["dt"].weight.shape[1]], w["dt"], True)               # fp32 raw step sizes [T, inner]
        y = O.selective_scan(xc, dt, w["dt_b"], w["A_log"], dbc, w["xseg"]["B"][0], w["xseg"]["C"][0], w["D"], self._cols(u, w["seg"], "z"),
                             st["S"], meta)
        return self._mm(y, w["o"], True)

    def _attention(self, i, w, m, ha, meta, kpool, vpool, v_first):
        """Returns ``(mixer output fp32, first mixing layer's value rows)``."""
        O, seg = self.ops, w["seg"]
        H, D, mask = int(m["heads"]), int(m["dim"]), m.get("mask") or {}
        u = O.linear_any(ha, w["proj"], self.dtype)                                   # [q | k | v | g], biases added
        mixes = bool(m.get("v_mix")) and i != self.v_source
        q = O.qk_norm_rope_append(u, seg["q"][0], seg["k"][0], seg["v"][0], H, D, None, None, self.cfg.rms_norm_eps, w["inv_freq"], kpool, vpool, meta,
                                  half=True, norm_after=True, rot_mult=w["rot_mult"], v_first=v_first if mixes else None, v_lambda=w["vmix"])
        if i == self.v_source:
            v_first = self._cols(u, seg, "v")
        o = O.sink_attention(q, kpool, vpool, w["sink"], meta, float(m["scale"]), 0, int(mask.get("size", 0) or 0), 1.0, self.dtype,
                             keep_first=int(mask.get("keep_first", 0) or 0), gate=self._cols(u, seg, "g"))
        return self._mm(o, w["o"], True), v_first

    @torch.inference_mode()
    def forward(self, x, meta: BatchMeta, kv, all_logits: bool = False, layer_out=None):
        """``x``: token ids ``[T]``.  Returns fp32 logits ``[B, V]`` (``[T, V]`` with ``all_logits``).  ``layer_out``: optional list that
        receives a copy of the residual after every layer."""
        O, c, n = self.ops, self.cfg, len(self.specs)
        if meta.state_slots is None and any(L["type"] == "mamba1" for L in self.specs):      # a stack of attention layers alone holds pages only
            raise ValueError("Podurax needs state slots in the step metadata (BatchMeta.build(..., state_slots=...))")
        tokens = x.to(torch.int64).contiguous()
        h = O.stream_embed(self.embed_tokens.weight, tokens, float(c.embedding_scale), 1).view(tokens.numel(), c.hidden_size)      # fp32 residual
        step = lambda y, w: O.scaled_add_norm_(h, y, None, w, c.rms_norm_eps, self.dtype, mult=float(c.residual_mult))
        ha = O.rmsnorm_cast(h, self.layer_weights[0]["norm1"], c.rms_norm_eps, self.dtype)
        v_first = None
        for i, L in enumerate(self.specs):
            w = self.layer_weights[i]
            if L["type"] == "mamba1":
                y = self._mamba1(w, L["mixer"], ha, meta, kv.state[i])
            else:
                y, v_first = self._attention(i, w, L["mixer"], ha, meta, kv.k[i], kv.v[i], v_first)
            nxt = self.layer_weights[i + 1]["norm1"] if i + 1 < n else self.norm_w
            if L["mlp"]:
                ha = step(y, w["norm2"])
                y = self._mm(O.gelu_gated_up(ha, w["gate"], w["up"]), w["down"], True)
            ha = step(y, nxt)
            if layer_out is not None:
                layer_out.append(h.clone())
        if not all_logits and meta.num_tokens != meta.num_seqs:
            ha = ha.index_select(0, meta.last_idx.long())
        return self._mm(ha, self.lm_head, True).contiguous()

    __call__ = forward


Model = PoduraxStage
