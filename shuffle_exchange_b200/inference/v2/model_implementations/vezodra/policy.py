"""Vezodra: a decoder-only stack whose layers add a mixer and a feed-forward of the same stream (``hybrid_model.py``, block
form ``"parallel"``): ``x += mixer(c(n1(x))) + ff(n2(x))`` with two RMS norms and ``c(h) = h + filter(h)``, a short causal filter
per channel whose last inputs are state of the sequence.  ``config.json`` lists every layer with its token mixer, the mixer's
sizes and its feed-forward; ``loop`` executes a span of layers several times in a row, every pass with its own caches and states.
The embedding table is also the head.

Mixers.  ``attention``: grouped heads whose values are the projected keys before rotation, interleaved rotation, a learned number
per query head on the scores, causal softmax with one added to its denominator, one sigmoid gate per head.  ``parallel``: two
mixers that read the same input, half the sum of their RMS-normed outputs.  Left: sliding-window attention, q and k rows normed
over all heads at once, rotation in halves with frequencies divided by ``rot.scaling.factor``.  Right: a delta rule that decays and
removes at separate rates per head and key channel (``removal_delta_mixer``).

Feed-forward: ``W_down (silu(W_gate h) * (W_up h))``.

Checkpoint names: ``embed``, ``final.norm``, per layer ``l<i>.norm1|norm2|canon1``, ``l<i>.mlp.gate|up|down`` and ``l<i>.mix.*``:
``q``, ``k``, ``temp``, ``g``, ``o`` (attention); ``left.q|k|v|q.norm|k.norm|o|out`` and ``right.r|k|v|a|a.b|g|w0|w1|w2|norm|o|out``
(parallel).  Linear weights are ``[out, in]``.
"""
from __future__ import annotations

import math
from typing import Any, Dict

import torch

from ..fomalix.policy import _cfg_dict
from ..hybrid_model import DSHybridModel, HybridLayerSpec, HybridSpec, pad_rows
from ..inference_policy_base import InferenceV2Policy
from ..inference_transformer_base import LayerWeights

DECAY_RATE = math.exp(-0.5)          # the delta rule's decay lies between exp(-DECAY_RATE) and 1


def _rotary(m: Dict) -> Dict[str, Any]:
    rot = m.get("rot") or {"dims": 0}
    return dict(rot_dims=int(rot.get("dims", m["dim"])), rot_base=float(rot.get("base", 10000.0)),
                rot_divisor=float((rot.get("scaling") or {}).get("factor", 1.0)),
                window=int((m.get("mask") or {}).get("size", 0)))


class VezodraPolicy(InferenceV2Policy):

    def spec(self, model_config) -> HybridSpec:
        cfg = _cfg_dict(model_config)
        layers = []
        for L in cfg["layers"]:
            m, kind = L["mixer"], L["type"]
            mlp = L.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"Unsupported feed-forward kind {mlp['kind']!r}")
            ff = dict(ff_dim=int(mlp["ff"]) if mlp is not None else 0, ff_kind="gated", ff_activation="silu")
            if kind == "attention":
                layers.append(HybridLayerSpec(
                    kind="rotary_attention", n_heads=int(m["heads"]), n_heads_kv=int(m["kv_heads"]), key_dim=int(m["dim"]),
                    value_dim=int(m["dim"]), attn_scale=float(m["scale"]), rot_interleaved=True, values_from_keys=True,
                    unit_sink=True, head_scale=True, out_gate=True, gate_per_head=True, **_rotary(m), **ff))
            elif kind == "parallel":
                a, b = m["left"], m["right"]
                left = HybridLayerSpec(
                    kind="rotary_attention", n_heads=int(a["heads"]), n_heads_kv=int(a["kv_heads"]), key_dim=int(a["dim"]),
                    value_dim=int(a["vdim"]), attn_scale=float(a["scale"]), qk_row_norm=True, **_rotary(a))
                right = HybridLayerSpec(
                    kind="removal_delta", n_heads=int(b["heads"]), n_heads_kv=int(b["heads"]), key_dim=int(b["dim"]),
                    value_dim=int(b["dim"]), decay_rate=DECAY_RATE)
                layers.append(HybridLayerSpec(kind="pair", n_heads=left.n_heads, n_heads_kv=left.n_heads_kv,
                                              key_dim=left.key_dim, value_dim=left.value_dim, parts=(left, right), **ff))
            else:
                raise ValueError(f"Unknown mixer type {kind!r}")
        loop = cfg.get("loop") or {}
        dt = getattr(model_config, "torch_dtype", None)
        return HybridSpec(vocab_size=int(cfg["vocab"]), model_dim=int(cfg["width"]), layers=layers,
                          norm_eps=float(cfg["norm"]["eps"]), sinusoid_base=None, block_form="parallel",
                          loop_start=int(loop.get("start", 0)), loop_stop=int(loop.get("stop", 0)),
                          loop_times=int(loop.get("times", 1)), input_conv_taps=int(cfg["canon"]["taps"]),
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

        def blocks(*groups):
            """Fused projection: every group of tensors is one block of rows, padded to whole 16-byte columns."""
            return torch.cat([pad_rows(torch.cat([get(n) for n in names], dim=0)) for names in groups], dim=0)

        embed = get("embed")
        weights: Dict[str, Any] = {"embed": embed, "final_norm_w": get("final.norm"), "unembed": pad_rows(embed), "layers": []}
        for i, L in enumerate(spec.layers):
            p, lw = f"l{i}.", LayerWeights()
            m = p + "mix."
            lw["norm1"] = get(p + "norm1")
            filt = get(p + "canon1")
            if filt.shape[1] != spec.input_conv_taps:
                raise ValueError(f"{p}canon1 has {filt.shape[1]} taps, the configuration says {spec.input_conv_taps}")
            lw["filter1"] = filt.t().contiguous()                       # [taps, width]
            if L.kind == "rotary_attention":
                lw["w_in"] = blocks((m + "q", m + "k"), (m + "g",))
                lw["q_head_scale"], lw["wo"] = get(m + "temp", f32), get(m + "o")
            else:
                a, b = m + "left.", m + "right."
                lw["w_in"] = blocks((a + "q", a + "k", a + "v"), (b + "r",), (b + "k",), (b + "v",), (b + "a",), (b + "g",),
                                    (b + "w1",))
                lw["parts"] = (
                    LayerWeights(q_norm=get(a + "q.norm"), k_norm=get(a + "k.norm"), wo=get(a + "o"), out_norm=get(a + "out")),
                    LayerWeights(w0=get(b + "w0", f32), a_bias=get(b + "a.b", f32), w2=get(b + "w2").t().contiguous(),
                                 norm=get(b + "norm"), wo=get(b + "o"), out_norm=get(b + "out")))
            if L.ff_dim > 0:
                f = p + "mlp."
                lw["norm2"] = get(p + "norm2")
                lw["w_gate_up"] = torch.cat([get(f + "gate"), get(f + "up")], dim=0).contiguous()
                lw["w_down"] = get(f + "down")
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
