"""Kulisun: a decoder-only language model whose every layer is latent attention over the whole sequence — direct queries, a compressed
key/value latent with one rotated key part shared by the heads, rotation frequencies rescaled for a longer context, a softmax with a
learned sink per head and a sigmoid output gate per coordinate (``modules/attention/latent_attention.py``) — followed by a dense gated
feed-forward with biases (``modules/gated_ffn.py``), a routed one (sigmoid scores, groups of experts of which the best are kept,
renormalised weights, a gated shared expert; ``modules/moe/routed_ffn.py``), or none.

Block shape: pre-norm with layer norms (gain and bias) and a learned scale per coordinate on every sublayer's result,
``x += m * ls1 * mixer(norm1(x))`` then ``x += m * ls2 * ff(norm2(x))`` with one residual multiplier ``m``.  The residual stream ``x`` is
float; each residual sum, the norm after it and — behind a routed feed-forward — the weighted sum of the experts are ONE kernel
(``ops.seqmix.residual_norm_``), so a layer hands the next one its normed input.  The sublayers compute in the model dtype; scores,
softmax, router, norms' statistics and angles are float.  ``config.json`` lists the layers in order (``mixer`` sizes, ``mlp`` or null),
so any order and any sizes load without code changes.

A sequence's cache is the latents and rotated key parts of ``max_seq_len`` tokens per layer.  Serving is the slot-based wrapper shared
with the other stateful families (``inference/slot_serving.py``)."""
from __future__ import annotations

import dataclasses
import json
import os
from typing import Any, Dict, List, Optional

import torch
import torch.nn.functional as F
from torch import nn

from ..inference.slot_serving import SlotServingModel
from ..inference.state_cache import SequenceStateManager, StepContext
from ..modules.attention.latent_attention import LatentWindowAttention
from ..modules.gated_ffn import GatedFFN
from ..modules.moe.routed_ffn import RoutedFFN
from ..modules.rms_norm import AffineLayerNorm
from ..ops import seqmix
from ..utils.sampling import Sampler


@dataclasses.dataclass
class KulisunConfig:
    vocab: int
    width: int
    layers: List[Dict[str, Any]]                    # [{"type", "mixer": {...}, "mlp": {...} | None}, ...] as in config.json
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    embedding_scale: float = 1.0
    dtype: torch.dtype = torch.bfloat16
    device: Any = None

    @classmethod
    def from_dict(cls, d: Dict[str, Any], **overrides) -> "KulisunConfig":
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), layers=list(d["layers"]), norm_eps=float(d["norm"]["eps"]),
                   residual_mult=float(d.get("residual_mult", 1.0)), embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   **overrides)

    @classmethod
    def from_pretrained(cls, path: str, **overrides) -> "KulisunConfig":
        with open(os.path.join(path, "config.json") if os.path.isdir(path) else path) as f:
            return cls.from_dict(json.load(f), **overrides)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)


def _mixer_sizes(m: Dict[str, Any]):
    return tuple(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))


def _build_mixer(cfg: KulisunConfig, spec: Dict[str, Any], max_seq_len: int) -> nn.Module:
    if spec["type"] != "latent_attention":
        raise ValueError(f"unknown mixer type {spec['type']!r}")
    m, rot = spec["mixer"], spec["mixer"]["rot"]
    heads, dim, rot_dim, vdim, kv_rank = _mixer_sizes(m)
    return LatentWindowAttention(cfg.width, heads, dim, rot_dim, vdim, kv_rank, 0, window=None, scale=float(m["scale"]),
                                 rot_base=float(rot["base"]), rot_dims=int(rot["dims"]), rot_scaling=rot.get("scaling"), eps=cfg.norm_eps,
                                 dtype=cfg.dtype, device=cfg.device, max_seq_len=max_seq_len, sink=True, out_gate=True, stacked=True)


def _build_ffn(cfg: KulisunConfig, f: Optional[Dict[str, Any]]) -> Optional[nn.Module]:
    if not f:
        return None
    if f["kind"] == "dense":
        return GatedFFN(cfg.width, int(f["ff"]), bias=True, dtype=cfg.dtype, device=cfg.device)
    if f["kind"] == "moe":
        r, g, sh = f["router"], f["router"].get("groups"), f.get("shared")
        return RoutedFFN(cfg.width, int(f["expert"]["ff"]), int(r["experts"]), int(r["top"]), shared_ff=int(sh["ff"]) if sh else 0,
                         router_act="sigmoid", gated=True, groups=(int(g["count"]), int(g["keep"])) if g else None, renormalise=True,
                         shared_gated=True, shared_gate=bool(sh), dtype=cfg.dtype, device=cfg.device)
    raise ValueError(f"unknown feed-forward kind {f['kind']!r}")


class KulisunLayer(nn.Module):
    def __init__(self, cfg: KulisunConfig, index: int, max_seq_len: int):
        super().__init__()
        spec = cfg.layers[index]
        scale = lambda: nn.Parameter(torch.ones(cfg.width, dtype=torch.float32, device=cfg.device), requires_grad=False)
        self.kind, self.dtype = spec["type"], cfg.dtype
        self.norm1 = AffineLayerNorm(cfg.width, cfg.norm_eps, cfg.device)
        self.mixer = _build_mixer(cfg, spec, max_seq_len)
        self.scale1 = scale()                                            # residual multiplier times the layer scale
        self.mlp = _build_ffn(cfg, spec.get("mlp"))
        if self.mlp is not None:
            self.norm2, self.scale2 = AffineLayerNorm(cfg.width, cfg.norm_eps, cfg.device), scale()

    def state_spec(self):
        return self.mixer.state_spec()

    def forward(self, x: torch.Tensor, h: torch.Tensor, ctx: StepContext, st: Dict[str, torch.Tensor],
                next_norm: Optional[AffineLayerNorm]) -> Optional[torch.Tensor]:
        """``x [B,S,width]`` float residual stream, updated in place; ``h``: its ``norm1`` in the model dtype.  Returns ``next_norm`` of the
        new stream, the next layer's input (None without one)."""
        B, S, W = x.shape
        rows = x.view(B * S, W)
        y, experts, scale = self.mixer(h.view(B, S, W), ctx, st).view(B * S, W), None, self.scale1
        if self.mlp is not None:
            h = self.norm2.after_sum(rows, y, scale)
            (y, experts), scale = self.mlp.pieces(h) if isinstance(self.mlp, RoutedFFN) else (self.mlp(h), None), self.scale2
        if next_norm is None:
            return seqmix.residual_norm_(rows, y, scale, None, None, 0.0, False, experts)
        return next_norm.after_sum(rows, y, scale, experts)


class KulisunForCausalLM(nn.Module):
    def __init__(self, cfg: KulisunConfig, max_seq_len: int = 2048):
        super().__init__()
        self.cfg = self.config = cfg
        mk = lambda *s: nn.Parameter(torch.zeros(*s, dtype=cfg.dtype, device=cfg.device), requires_grad=False)
        self.embed, self.head = mk(cfg.vocab, cfg.width), mk(cfg.vocab, cfg.width)
        self.layers = nn.ModuleList([KulisunLayer(cfg, i, max_seq_len) for i in range(len(cfg.layers))])
        self.final_norm = AffineLayerNorm(cfg.width, cfg.norm_eps, cfg.device)
        self.position_limit = max_seq_len                    # every layer keeps whole sequences

    def state_specs(self):
        return [layer.state_spec() for layer in self.layers]

    def body(self, input_ids: torch.Tensor, ctx: StepContext, states: SequenceStateManager, tap=None) -> torch.Tensor:
        x, _ = seqmix.embed_bigram(input_ids, self.embed, self.cfg.embedding_scale, None, 0, 0, None, ctx.slots, ctx.lens, ctx.fresh)
        n = len(self.layers)
        h = self.layers[0].norm1(x, self.cfg.dtype) if n else None
        for i, layer in enumerate(self.layers):
            h = layer(x, h, ctx, states.layer(i), self.layers[i + 1].norm1 if i + 1 < n else None)
            if tap is not None:
                tap(i, x)
        ctx.scratch.clear()
        return x

    def logits(self, rows: torch.Tensor) -> torch.Tensor:
        """Residual rows ``[n, width]`` float → float logits ``[n, vocab]``."""
        return F.linear(self.final_norm(rows, self.cfg.dtype), self.head).float()


# --------------------------------------------------------------------------------------------------------------- checkpoint names
def convert_state_dict(cfg: KulisunConfig, sd: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors (``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm2`` (+ ``.b``), ``l<i>.ls1|ls2``, ``l<i>.mix.*``,
    ``l<i>.mlp.*``; linear weights ``[out, in]``) → this module's parameters: the projections that read a mixer's input are stacked, gate
    and up projections are stacked, the shared expert's gate rides under the router's rows, experts are stacked, the residual multiplier
    is folded into the layer scales, and everything the kernels read as float is float."""
    out: Dict[str, torch.Tensor] = {"embed": sd["embed"], "head": sd["head"], "final_norm.weight": sd["final.norm"],
                                    "final_norm.bias": sd["final.norm.b"]}
    for i, spec in enumerate(cfg.layers):
        p, o, f = f"l{i}.", f"layers.{i}.", spec.get("mlp")
        for k in ("1", "2") if f else ("1",):
            out[o + f"norm{k}.weight"], out[o + f"norm{k}.bias"] = sd[p + f"norm{k}"], sd[p + f"norm{k}.b"]
            out[o + f"scale{k}"] = cfg.residual_mult * sd[p + f"ls{k}"].float()
        H, D, R, V, C = _mixer_sizes(spec["mixer"])
        x = lambda n: sd[p + "mix." + n]
        parts, rows = LatentWindowAttention.stacked_parts(H, D, R, V, C, True)
        stack = x("q").new_zeros(rows, cfg.width)
        for (at, n), name in zip(parts, ("q", "dkv", "g")):
            if x(name).shape[0] != n:
                raise ValueError(f"{p}mix.{name}: {x(name).shape[0]} rows, the configuration has {n}")
            stack[at:at + n] = x(name)
        a = o + "mixer."
        out.update({a + "in_proj": stack, a + "dkv_norm": x("dkv.norm"), a + "uk": x("uk").reshape(H, D, C), a + "uv": x("uv").reshape(H, V, C),
                    a + "sink": x("sink"), a + "o": x("o")})
        if not f:
            continue
        y = lambda n: sd[p + "mlp." + n]
        both = lambda n: torch.cat([y(n + "gate"), y(n + "up")], 0)
        m = o + "mlp."
        if f["kind"] == "dense":
            out.update({m + "up": both(""), m + "down": y("down"), m + "up_bias": torch.cat([y("gate.b"), y("up.b")], 0), m + "down_bias": y("down.b")})
            continue
        E = int(f["router"]["experts"])
        out[m + "router.linear_router.weight"] = torch.cat([y("router")] + ([y("shared.sg")] if f.get("shared") else []), 0)
        out[m + "up"] = torch.stack([both(f"e{e}.") for e in range(E)], 0)
        out[m + "down"] = torch.stack([y(f"e{e}.down") for e in range(E)], 0)
        if f.get("shared"):
            out[m + "shared_up"], out[m + "shared_down"] = both("shared."), y("shared.down")
    return out


def load_kulisun_weights(model: KulisunForCausalLM, sd: Dict[str, torch.Tensor]) -> None:
    conv = convert_state_dict(model.cfg, sd)
    params = dict(model.named_parameters())
    missing, extra = sorted(set(params) - set(conv)), sorted(set(conv) - set(params))
    if missing or extra:
        raise KeyError(f"checkpoint does not fit the model: missing {missing[:6]}, unexpected {extra[:6]}")
    with torch.no_grad():
        for k, v in conv.items():
            if tuple(params[k].shape) != tuple(v.shape):
                raise ValueError(f"{k}: checkpoint shape {tuple(v.shape)} != {tuple(params[k].shape)}")
            params[k].copy_(v.to(params[k].dtype))


# ------------------------------------------------------------------------------------------------------------------------ serving
class KulisunForInference(SlotServingModel):
    def __init__(self, cfg: KulisunConfig, batch_size: int = 1, max_seq_len: int = 2048, on_device_sampling: bool = True,
                 sampler: Optional[Sampler] = None):
        super().__init__(cfg, KulisunForCausalLM(cfg, max_seq_len=max_seq_len), batch_size=batch_size, max_seq_len=max_seq_len,
                         on_device_sampling=on_device_sampling, sampler=sampler)

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, device=None, **kw) -> "KulisunForInference":
        from ..utils.safetensors_utils import load_state_dict_safetensors

        sd = load_state_dict_safetensors(os.path.join(path, "model.safetensors"))
        model = cls(KulisunConfig.from_pretrained(path, dtype=dtype, device=device), **kw)
        load_kulisun_weights(model.lm, sd)
        return model.eval()

    def load_checkpoint_tensors(self, sd) -> None:
        load_kulisun_weights(self.lm, sd)
