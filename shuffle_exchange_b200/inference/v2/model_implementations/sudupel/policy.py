"""Sudupel: a decoder-only stack with a norm before and after every sublayer (``hybrid_model.py``, block form ``"sandwich"``, norm
weights stored around zero): ``x += n1b(mixer(n1(x)))``, ``x += n2b(ff(n2(x)))``.  ``config.json`` lists every layer with its token
mixer, the mixer's sizes and its feed-forward (or none); embedding rows carry a factor, logits a soft cap, the head is a matrix of its
own.

Mixers.  ``lightning``: a matrix state per head that decays at a fixed rate and takes SiLU-activated outer products
(``lightning_mixer``).  ``parallel``: causal attention with whole-row q/k norms, scaled rotation in halves and one added to the
softmax denominator, beside a gated linear recurrent unit (``linear_recurrent_unit``).  ``parallel_2``: sliding-window attention on
filtered projections with per-head norms and rotation, beside gated linear attention (``gated_linear_mixer``).  The two halves of
a pair read the same input and are added with one factor each.

Feed-forwards.  ``dense``: ``W_down (a sigmoid(1.702 a) (1 + b))`` with ``a = min(W_gate h, L)``, ``b = max(-L, min(W_up h, L))``.
``moe``: SiLU-gated experts; sigmoid scores, the choice made by score + ``correction`` inside the ``groups.keep`` of ``groups.count``
blocks whose two best sums are largest, weights = the chosen experts' plain scores.

Checkpoint names: ``embed``, ``head``, ``final.norm``, per layer ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*`` (lightning: ``q``,
``k``, ``v``, ``g``, ``norm``, ``o``; attention under ``left.``: ``q``, ``k``, ``v`` with ``.norm`` and in ``parallel_2`` ``.conv``,
``o``; recurrent unit under ``right.``: ``y``, ``x`` with ``.b``, ``conv``, ``conv.b``, ``ra``, ``ri`` with ``.b``, ``lam``, ``o``;
gated linear attention under ``right.``: ``q``, ``k``, ``v``, ``g``, ``a1``, ``a2``, ``a2.b``, ``norm``, ``o``) and ``l<i>.mlp.*``
(dense: ``gate``, ``up``, ``down``; experts: ``router``, ``correction``, ``e<j>.gate|up|down``).  Linear weights are ``[out, in]``.
"""
from __future__ import annotations

from typing import Any, Dict, Optional, Tuple

import torch

from ..fomalix.policy import _cfg_dict
from ..hybrid_model import DSHybridModel, HybridLayerSpec, HybridSpec, pad_rows
from ..inference_policy_base import InferenceV2Policy
from ..inference_transformer_base import LayerWeights
from ..ridazen.policy import pad_cols

LRU_RATE = 8.0               # the recurrent unit's log decay is -LRU_RATE * r * softplus(lam)


def _rotary(m: Dict) -> Dict[str, Any]:
    rot = m.get("rot") or {"dims": 0}
    sc: Optional[Dict] = rot.get("scaling")
    scaling: Optional[Tuple[float, float, float, float]] = None
    if sc:
        scaling = (float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"]))
    return dict(rot_dims=int(rot.get("dims", m["dim"])), rot_base=float(rot.get("base", 10000.0)), rot_scaling=scaling,
                window=int((m.get("mask") or {}).get("size", 0)))


def _heads(m: Dict) -> Dict[str, int]:
    return dict(n_heads=int(m["heads"]), n_heads_kv=int(m.get("kv_heads", m["heads"])), key_dim=int(m["dim"]),
                value_dim=int(m["vdim"]))


def _feed_forward(mlp: Optional[Dict]) -> Dict[str, Any]:
    if mlp is None:
        return {}
    if mlp["kind"] == "dense":
        return dict(ff_dim=int(mlp["ff"]), ff_kind="gated", ff_activation="clamped_swish", ff_limit=float(mlp["limit"]))
    if mlp["kind"] == "moe":
        r = mlp["router"]
        groups = r.get("groups") or {}
        return dict(ff_dim=int(mlp["expert"]["ff"]), ff_kind="moe", ff_activation="silu", n_experts=int(r["experts"]),
                    top_k=int(r["top"]), moe_score="sigmoid", moe_correction=True, moe_groups=int(groups.get("count", 1)),
                    moe_keep_groups=int(groups.get("keep", groups.get("count", 1))), moe_group_rank="top2",
                    moe_plain_scores=True)
    raise ValueError(f"Unsupported feed-forward kind {mlp['kind']!r}")


class SudupelPolicy(InferenceV2Policy):

    def spec(self, model_config) -> HybridSpec:
        cfg = _cfg_dict(model_config)
        layers = []
        for L in cfg["layers"]:
            m, kind, ff = L["mixer"], L["type"], _feed_forward(L.get("mlp"))
            if kind == "lightning":
                layers.append(HybridLayerSpec(kind="lightning", head_decay=tuple(float(x) for x in m["decay"]), **_heads(m), **ff))
                continue
            if kind not in ("parallel", "parallel_2"):
                raise ValueError(f"Unknown mixer type {kind!r}")
            a, b = m["left"], m["right"]
            if kind == "parallel":
                if int(b["width"]) % int(b["blocks"]):
                    raise ValueError(f"a recurrent unit of {b['width']} channels has no {b['blocks']} equal blocks")
                left = HybridLayerSpec(kind="rotary_attention", attn_scale=float(a["scale"]), qk_row_norm=True, unit_sink=True,
                                       **_heads(a), **_rotary(a))
                right = HybridLayerSpec(kind="lru", n_heads=int(b["blocks"]), n_heads_kv=int(b["blocks"]),
                                        key_dim=int(b["width"]) // int(b["blocks"]),
                                        value_dim=int(b["width"]) // int(b["blocks"]), conv_taps=int(b["conv"]),
                                        decay_rate=LRU_RATE)
            else:
                left = HybridLayerSpec(kind="attention", attn_scale=float(a["scale"]), qk_norm_weight=True,
                                       conv_taps=int(a["conv"]), **_heads(a), **_rotary(a))
                right = HybridLayerSpec(kind="channel_decay", decay_tau=float(b["tau"]), **_heads(b))
            layers.append(HybridLayerSpec(kind="pair", n_heads=left.n_heads, n_heads_kv=left.n_heads_kv, key_dim=left.key_dim,
                                          value_dim=left.value_dim, parts=(left, right),
                                          pair_scales=(float(m["left_scale"]), float(m["right_scale"])), **ff))
        dt = getattr(model_config, "torch_dtype", None)
        return HybridSpec(vocab_size=int(cfg["vocab"]), model_dim=int(cfg["width"]), layers=layers,
                          norm_eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]), sinusoid_base=None,
                          block_form="sandwich", norm_weight_offset=1.0, logit_softcap=float(cfg.get("logit_softcap") or 0.0),
                          dtype=dt if dt in (torch.bfloat16, torch.float32) else torch.bfloat16)

    # ------------------------------------------------------------------------------------------ weights
    def load_weights(self) -> Dict:
        if self._weights is not None:
            return self._weights
        spec = self.resolved_spec()
        dev, dt, f32 = self._device(), spec.dtype, torch.float32
        raw = {name: t.detach() for name, t in self._checkpoint_engine.parameters()}
        used = set()

        def get(name, dtype=dt):
            used.add(name)
            return raw[name].to(dev, dtype).contiguous()

        def cat(*names):
            return torch.cat([get(n) for n in names], dim=0)

        def blocks(*groups):
            """Fused projection: every group of tensors is one block of rows, padded to whole 16-byte columns."""
            return torch.cat([pad_rows(cat(*names)) for names in groups], dim=0)

        def filter_of(name, rows, taps):
            w = get(name)
            if tuple(w.shape) != (rows, taps):
                raise ValueError(f"{name} is {tuple(w.shape)}, the configuration says {(rows, taps)}")
            return w

        weights: Dict[str, Any] = {"embed": get("embed"), "final_norm_w": get("final.norm"), "unembed": pad_rows(get("head")),
                                   "layers": []}
        for i, L in enumerate(spec.layers):
            p, lw = f"l{i}.", LayerWeights()
            m = p + "mix."
            lw["norm1"], lw["norm1b"] = get(p + "norm1"), get(p + "norm1b")
            if L.kind == "lightning":
                lw["w_in"] = blocks((m + "q",), (m + "k",), (m + "v",), (m + "g",))
                lw["norm"], lw["wo"] = get(m + "norm"), get(m + "o")
            else:
                a, b = m + "left.", m + "right."
                left, right = L.parts
                first = pad_rows(cat(a + "q", a + "k", a + "v"))
                la = LayerWeights(q_norm=get(a + "q.norm"), k_norm=get(a + "k.norm"))
                if left.kind == "attention":
                    rows = left.n_heads * left.key_dim, left.n_heads_kv * left.key_dim, left.n_heads_kv * left.value_dim
                    la["conv_w"] = torch.cat([filter_of(a + n + ".conv", r, left.conv_taps) for n, r in zip("qkv", rows)])
                if right.kind == "lru":
                    B, S, N = right.n_heads, right.key_dim, right.n_heads * right.key_dim
                    second = blocks((b + "y",), (b + "x",))
                    lb = LayerWeights(
                        conv_w=filter_of(b + "conv", N, right.conv_taps), conv_b=get(b + "conv.b"), x_bias=get(b + "x.b"),
                        y_bias=get(b + "y.b"),
                        gate_w=torch.stack([get(b + g).view(B, S, S).transpose(1, 2) for g in ("ra", "ri")]).contiguous(),
                        gate_b=torch.stack([get(b + g + ".b", f32).view(N) for g in ("ra", "ri")]).contiguous(),
                        rate=-right.decay_rate * torch.nn.functional.softplus(get(b + "lam", f32)), wo_width=N)
                else:
                    second = blocks((b + "q",), (b + "k",), (b + "v",), (b + "g",), (b + "a1",))
                    lb = LayerWeights(w2=get(b + "a2").t().contiguous(), decay_bias=get(b + "a2.b", f32), norm=get(b + "norm"),
                                      wo_width=right.n_heads * right.value_dim)
                la["wo_width"] = left.n_heads * left.value_dim
                lw["parts"], lw["cut"] = (la, lb), first.shape[0]
                lw["w_in"] = torch.cat([first, second], dim=0)
                wo = pad_cols(get(a + "o")), pad_cols(get(b + "o"))
                lw["wo"], lw["wo_cut"] = torch.cat(wo, dim=1).contiguous(), wo[0].shape[1]
            if L.ff_dim > 0:
                f = p + "mlp."
                lw["norm2"], lw["norm2b"] = get(p + "norm2"), get(p + "norm2b")
                if L.ff_kind == "moe":
                    lw["moe_gate"], lw["moe_correction"] = get(f + "router", f32), get(f + "correction", f32)
                    lw["moe_w1"] = torch.stack([cat(f"{f}e{e}.gate", f"{f}e{e}.up") for e in range(L.n_experts)])
                    lw["moe_w2"] = torch.stack([get(f"{f}e{e}.down") for e in range(L.n_experts)]).contiguous()
                else:
                    lw["w_gate_up"], lw["w_down"] = cat(f + "gate", f + "up"), get(f + "down")
            weights["layers"].append(lw)
        self.container_map.set_unmapped_params([n for n in raw if n not in used])
        self._weights = weights
        return weights

    def build_model(self, engine_config, mp_group=None, state_manager=None) -> DSHybridModel:
        self._engine_config = engine_config
        if mp_group is not None:
            self._mp_group = mp_group
        model = DSHybridModel(self.resolved_spec(), self.load_weights(), engine_config, state_manager, self._mp_group)
        model.model_config = self._model_config
        return model
