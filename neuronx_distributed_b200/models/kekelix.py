"""Kekelix: a decoder-only language model of grouped-query attention layers of three kinds, each beside a routed feed-forward, with a stretch
of layers that runs several times.

Mixers (one module, ``modules/attention/window_attention.py``):
* ``attention`` — differential attention over the whole sequence, no rotation: two softmax maps per head over the same values, the second
  taken off times one learned number, the difference brought to unit root mean square;
* ``attention_2`` — biased projections, rotary positions with interpolated frequencies, every earlier position, one added to the softmax's
  denominator;
* ``attention_3`` — aligned chunks of positions, no value projection (the projected keys are the values), queries and keys brought to unit
  root mean square after the rotation.

Feed-forward (``modules/moe/routed_ffn.py``): sigmoid scores, the best experts' scores multiply what the experts read, clamped gated experts.

Block shape: parallel, ``x += mixer(norm1(x)) + ff(norm2(x))``, both norms of the same ``x``, RMS norms whose stored weight is the gain's
distance from one.  ``loop``: layers ``start .. stop-1`` run ``times`` times with the same weights and a cache of their own per pass; the
embedding output joins the stream before every pass but the first, a vector of its own (``loop.step``) before every pass.  The stream is
float; everything between one layer's sublayers and the next one's — the sum of the mixer's result and the experts' rows, what a pass adds,
both norms — is ONE kernel (``ops.seqmix.residual_norm_``).  The sublayers compute in the model dtype; scores, softmax, routers, norms'
statistics and angles are float.  The logits are the final norm times the embedding table.

``config.json`` lists the layers in order, so any order and any sizes load without code changes.  Serving is the slot-based wrapper shared
with the other stateful families (``inference/slot_serving.py``)."""
from __future__ import annotations

import dataclasses
import json
import os
from typing import Any, Dict, List, Optional, Tuple

import torch
import torch.nn.functional as F
from torch import nn

from ..inference.slot_serving import SlotServingModel
from ..inference.state_cache import SequenceStateManager, StepContext
from ..modules.attention.window_attention import GatedWindowAttention
from ..modules.moe.routed_ffn import RoutedFFN
from ..modules.rms_norm import OffsetRMSNorm
from ..ops import seqmix
from ..utils.sampling import Sampler

GLU_SLOPE = 1.702                                    # of the experts' gate, g sigmoid(slope g)


@dataclasses.dataclass
class KekelixConfig:
    vocab: int
    width: int
    layers: List[Dict[str, Any]]                    # [{"type", "mixer": {...}, "mlp": {...} | None}, ...] as in config.json
    norm_eps: float = 1e-6
    loop: Optional[Tuple[int, int, int]] = None     # (start, stop, times)
    dtype: torch.dtype = torch.bfloat16
    device: Any = None

    @classmethod
    def from_dict(cls, d: Dict[str, Any], **overrides) -> "KekelixConfig":
        lp = d.get("loop")
        loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
        if loop and not (0 <= loop[0] < loop[1] <= len(d["layers"]) and loop[2] >= 1):
            raise ValueError(f"layers {loop[0]} .. {loop[1] - 1} cannot run {loop[2]} times in a model of {len(d['layers'])} layers")
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), layers=list(d["layers"]), norm_eps=float(d["norm"]["eps"]), loop=loop, **overrides)

    @classmethod
    def from_pretrained(cls, path: str, **overrides) -> "KekelixConfig":
        with open(os.path.join(path, "config.json") if os.path.isdir(path) else path) as f:
            return cls.from_dict(json.load(f), **overrides)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """The layers in the order they run: ``(layer, number of the pass that starts right before it, or None)``."""
        n = len(self.layers)
        start, stop, times = self.loop or (n, n, 0)
        once = lambda a, b: [(i, None) for i in range(a, b)]
        return once(0, start) + [(i, t if i == start else None) for t in range(times) for i in range(start, stop)] + once(stop, n)


def _rotation(m: Dict[str, Any]) -> Dict[str, Any]:
    rot = m.get("rot") or {}
    return dict(rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), rot_scaling=rot.get("scaling"))


def _build_mixer(cfg: KekelixConfig, spec: Dict[str, Any], max_seq_len: int) -> GatedWindowAttention:
    kind, m = spec["type"], spec["mixer"]
    heads, kv_heads, dim, vdim = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    common = dict(window=None, scale=float(m["scale"]), eps=cfg.norm_eps, head_gate=False, dtype=cfg.dtype, device=cfg.device, max_seq_len=max_seq_len)
    if kind == "attention":
        return GatedWindowAttention(cfg.width, heads, kv_heads, dim, vdim, qk_norm=None, bias=False, diff=float(m["diff"]), **common)
    if kind == "attention_2":
        return GatedWindowAttention(cfg.width, heads, kv_heads, dim, vdim, qk_norm=None, bias=True, sink="zero", **_rotation(m), **common)
    if kind == "attention_3":
        return GatedWindowAttention(cfg.width, heads, kv_heads, dim, vdim, qk_norm="unit", bias=False, chunk=int(m["mask"]["size"]),
                                    values_are_keys=True, **_rotation(m), **common)
    raise ValueError(f"unknown mixer type {kind!r}")


def _build_ffn(cfg: KekelixConfig, f: Optional[Dict[str, Any]]) -> Optional[RoutedFFN]:
    if not f:
        return None
    if f["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
    r, e = f["router"], f["expert"]
    return RoutedFFN(cfg.width, int(e["ff"]), int(r["experts"]), int(r["top"]), router_act="sigmoid", gated=True, glu=(float(e["limit"]), GLU_SLOPE),
                     weigh_input=True, dtype=cfg.dtype, device=cfg.device)


class KekelixLayer(nn.Module):
    def __init__(self, cfg: KekelixConfig, index: int, max_seq_len: int):
        super().__init__()
        spec = cfg.layers[index]
        self.kind = spec["type"]
        self.norm1 = OffsetRMSNorm(cfg.width, cfg.norm_eps, cfg.device)
        self.mixer = _build_mixer(cfg, spec, max_seq_len)
        self.mlp = _build_ffn(cfg, spec.get("mlp"))
        self.norm2 = OffsetRMSNorm(cfg.width, cfg.norm_eps, cfg.device) if self.mlp is not None else None

    def state_spec(self):
        return self.mixer.state_spec()

    def normed(self, x: torch.Tensor, y: Optional[torch.Tensor], experts, inject, dtype: torch.dtype):
        """The stream ``x [rows, width]`` brought up to this layer in place (``y``, ``experts``: what the layer before left to add; ``inject``:
        what a pass that starts here adds) → this layer's one or two inputs."""
        h = self.norm1.after_sum(x, y, experts, self.norm2, inject, dtype)
        return h if self.norm2 is not None else (h, None)

    def forward(self, h1: torch.Tensor, h2: Optional[torch.Tensor], B: int, S: int, ctx: StepContext, st: Dict[str, torch.Tensor]):
        """``h1, h2 [B*S, width]`` → what the layer adds to the stream, as ``residual_norm_`` takes it: ``(rows, experts or None)``."""
        y = self.mixer(h1.view(B, S, -1), ctx, st).view(B * S, -1)
        if self.mlp is None:
            return y, None
        rows, (src, w, _, _) = self.mlp.pieces(h2)
        return rows, (src, w, y, None)


class KekelixForCausalLM(nn.Module):
    def __init__(self, cfg: KekelixConfig, max_seq_len: int = 2048):
        super().__init__()
        self.cfg = self.config = cfg
        self.embed = nn.Parameter(torch.zeros(cfg.vocab, cfg.width, dtype=cfg.dtype, device=cfg.device), requires_grad=False)
        self.layers = nn.ModuleList([KekelixLayer(cfg, i, max_seq_len) for i in range(len(cfg.layers))])
        self.loop_step = None
        if cfg.loop:
            self.loop_step = nn.Parameter(torch.zeros(cfg.loop[2], cfg.width, dtype=torch.float32, device=cfg.device), requires_grad=False)
        self.final_norm = OffsetRMSNorm(cfg.width, cfg.norm_eps, cfg.device)
        self.runs = cfg.runs()
        self.position_limit = max_seq_len if any(layer.mixer.whole_sequence for layer in self.layers) else None

    def state_specs(self):
        """One entry per layer RUN: every pass over the repeated layers has a cache of its own."""
        return [self.layers[i].state_spec() for i, _ in self.runs]

    def _inject(self, tokens: torch.Tensor, t: Optional[int]):
        """What joins the stream before pass ``t``: the embedding output (not before the first pass) and the pass's own vector."""
        if t is None:
            return None
        return (tokens, self.embed, self.loop_step[t]) if t > 0 else (None, None, self.loop_step[t])

    def body(self, input_ids: torch.Tensor, ctx: StepContext, states: SequenceStateManager, tap=None) -> torch.Tensor:
        tokens = input_ids.contiguous()
        B, S = tokens.shape
        stream, _ = seqmix.embed_bigram(tokens, self.embed, 1.0, None, 0, 0, None, ctx.slots, ctx.lens, ctx.fresh)
        x, y, experts = stream.view(B * S, -1), None, None
        for r, (i, t) in enumerate(self.runs):
            h1, h2 = self.layers[i].normed(x, y, experts, self._inject(tokens, t), self.cfg.dtype)
            y, experts = self.layers[i](h1, h2, B, S, ctx, states.layer(r))
            if tap is not None or r + 1 == len(self.runs):
                seqmix.residual_norm_(x, y, None, None, None, 0.0, False, experts)
                y = experts = None
            if tap is not None:
                tap(r, stream)
        ctx.scratch.clear()
        return stream

    def logits(self, rows: torch.Tensor) -> torch.Tensor:
        """Residual rows ``[n, width]`` float → float logits ``[n, vocab]``."""
        return F.linear(self.final_norm(rows, self.cfg.dtype), self.embed).float()


# --------------------------------------------------------------------------------------------------------------- checkpoint names
_PARTS = {"attention": ("q", "k", "v"), "attention_2": ("q", "k", "v"), "attention_3": ("q", "k")}


def convert_state_dict(cfg: KekelixConfig, sd: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors (``embed``, ``final.norm``, ``loop.step``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``; linear weights
    ``[out, in]``) → this module's parameters: a mixer's input projections (and biases) are stacked, norm weights become gains, the two
    inner products of a differential layer become its one number, gate over up projections and experts are stacked, and everything the
    kernels read as float is float."""
    gain = lambda n: 1.0 + sd[n].float()
    out: Dict[str, torch.Tensor] = {"embed": sd["embed"], "final_norm.weight": gain("final.norm")}
    if cfg.loop:
        out["loop_step"] = sd["loop.step"].float()
    for i, spec in enumerate(cfg.layers):
        p, o, f, m, kind = f"l{i}.", f"layers.{i}.", spec.get("mlp"), spec["mixer"], spec["type"]
        for k in ("1", "2") if f else ("1",):
            out[o + f"norm{k}.weight"] = gain(p + f"norm{k}")
        x = lambda n: sd[p + "mix." + n]
        maps = 2 if kind == "attention" else 1
        H, G, D, V = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        for n, want in zip(_PARTS[kind], (H * maps * D, G * maps * D, G * V)):
            if x(n).shape[0] != want:
                raise ValueError(f"{p}mix.{n}: {x(n).shape[0]} rows, the configuration has {want}")
        rows = GatedWindowAttention.stacked_rows(H, G, D, V if "v" in _PARTS[kind] else 0, False, 0, maps)
        stack = lambda parts: torch.cat(parts + [parts[0].new_zeros((rows - sum(t.shape[0] for t in parts),) + tuple(parts[0].shape[1:]))], 0)
        a = o + "mixer."
        out[a + "in_proj"], out[a + "o"] = stack([x(n) for n in _PARTS[kind]]), x("o")
        if kind == "attention_2":
            out[a + "in_bias"] = stack([x(n + ".b") for n in _PARTS[kind]])
        if kind == "attention":
            dot = lambda u, v: (x(u).double() * x(v).double()).sum()
            out[a + "lam"] = (torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2")) + float(m["diff"])).float().reshape(1)
        if f:
            y = lambda n: sd[p + "mlp." + n]
            E = range(int(f["router"]["experts"]))
            out[o + "mlp.router.linear_router.weight"] = y("router")
            out[o + "mlp.up"] = torch.stack([torch.cat([y(f"e{e}.gate"), y(f"e{e}.up")], 0) for e in E], 0)
            out[o + "mlp.down"] = torch.stack([y(f"e{e}.down") for e in E], 0)
    return out


def load_kekelix_weights(model: KekelixForCausalLM, sd: Dict[str, torch.Tensor]) -> None:
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
class KekelixForInference(SlotServingModel):
    def __init__(self, cfg: KekelixConfig, batch_size: int = 1, max_seq_len: int = 2048, on_device_sampling: bool = True,
                 sampler: Optional[Sampler] = None):
        super().__init__(cfg, KekelixForCausalLM(cfg, max_seq_len=max_seq_len), batch_size=batch_size, max_seq_len=max_seq_len,
                         on_device_sampling=on_device_sampling, sampler=sampler)

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, device=None, **kw) -> "KekelixForInference":
        from ..utils.safetensors_utils import load_state_dict_safetensors

        sd = load_state_dict_safetensors(os.path.join(path, "model.safetensors"))
        model = cls(KekelixConfig.from_pretrained(path, dtype=dtype, device=device), **kw)
        load_kekelix_weights(model.lm, sd)
        return model.eval()

    def load_checkpoint_tensors(self, sd) -> None:
        load_kekelix_weights(self.lm, sd)
