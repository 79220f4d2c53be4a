"""Rovurax decoder as an ONNX graph in packed serving form.

Parallel layers around one fp32 residual: the mixer and the feed-forward read the same norm, and their sum goes back.
The mixer is attention without positions over chunks of the sequence, whose values may be mixed with those of the first
such layer, or latent attention (keys and values as low-rank maps of one cached latent per token, a shared rotated key
part, a sink per head, an output gate per head).  config.json gives every size and constant; the graph is built from it
and from the checkpoint's tensors.

Mixer and feed-forward write into the columns of one tensor, so a layer's two output projections are one MatMul over
stacked columns whose fp32 accumulator is the parallel sum.  The projections that read the norm are one MatMul over
stacked rows for the mixer and one gated MatMul pair for the feed-forward.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch

from .decoder_cache import CacheTensor
from .packed_graph import TORCH_DT, PackedGraph, padded_head_widths

MIXERS = ("attention", "latent_attention")
GATE_SLOPE = 1.702       # of the feed-forward's sigmoid
UP_OFFSET = 1.0          # added to the feed-forward's clamped up branch


@dataclass
class RovuraxConfig:
    vocab_size: int
    width: int
    layers: List[Dict[str, Any]]
    norm_eps: float = 1e-6
    dtype: str = "bf16"
    max_seq_len: int = 2048               # rows of the rotary tables
    architecture: str = field(default="Rovurax", repr=False)

    @staticmethod
    def from_json(d: Mapping[str, Any], dtype: str = "bf16", max_seq_len: int = 2048) -> "RovuraxConfig":
        cfg = RovuraxConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), layers=list(d["layers"]), norm_eps=float(d["norm"]["eps"]),
                            dtype=dtype, max_seq_len=int(max_seq_len))
        cfg.validate()
        return cfg

    def to_json(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "layers": self.layers, "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size,
                "width": self.width}

    def validate(self) -> None:
        first = self.first_mixed()
        for i, layer in enumerate(self.layers):
            m = layer["mixer"]
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
            if layer.get("mlp") is not None and layer["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {layer['mlp']['kind']!r}")
            if layer["type"] == "attention":
                if m["heads"] % m["kv_heads"]:
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                if m.get("mask") and int(m["mask"]["size"]) <= 0:
                    raise ValueError(f"layer {i}: the chunk size must be positive")
                if m.get("v_mix") and any(m[k] != self.layers[first]["mixer"][k] for k in ("kv_heads", "vdim")):
                    raise ValueError(f"layer {i}: value sizes differ from those of layer {first}, whose values it mixes in")
            elif m.get("rot") and (m["rot"]["dims"] > m["rot_dim"] or m["rot"]["dims"] % 2):
                raise ValueError(f"layer {i}: rot.dims must be even and at most rot_dim")

    def first_mixed(self) -> Optional[int]:
        """The layer whose values later layers mix in."""
        return next((i for i, layer in enumerate(self.layers) if layer["type"] == "attention" and layer["mixer"].get("v_mix")), None)

    @property
    def has_latents(self) -> bool:
        return any(layer["type"] == "latent_attention" for layer in self.layers)

    def latent_widths(self, m: Mapping[str, Any]) -> Tuple[int, int]:
        """Stored widths of the latent and of the rotated key part: rows of the cache are read in 16-byte pieces."""
        unit = 4 if self.dtype == "fp32" else 8
        return -(-m["kv_rank"] // unit) * unit, -(-m["rot_dim"] // unit) * unit

    def cache_tensors(self, tp_size: int = 1) -> List[CacheTensor]:
        if tp_size != 1:
            raise ValueError("this graph is built for one device")
        dt = TORCH_DT[self.dtype]
        out: List[CacheTensor] = []
        for i, layer in enumerate(self.layers):
            m = layer["mixer"]
            if layer["type"] == "latent_attention":
                out.append(CacheTensor(f"latent_cache.{i}", f"latent_cache_out.{i}", "paged", (sum(self.latent_widths(m)),), dt))
            else:
                kw, vw = padded_head_widths(self.dtype, m["dim"], m["vdim"])
                out.append(CacheTensor(f"key_cache.{i}", f"key_cache_out.{i}", "paged", (m["kv_heads"], kw), dt))
                out.append(CacheTensor(f"value_cache.{i}", f"value_cache_out.{i}", "paged", (m["kv_heads"], vw), dt))
        return out

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Names and shapes of the checkpoint."""
        W, shapes = self.width, {"embed": (self.vocab_size, self.width)}
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}.", layer["mixer"]
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            x = p + "mix."
            shapes[p + "norm1"] = (W,)
            if layer["type"] == "latent_attention":
                rank, rot = m["kv_rank"], m["rot_dim"]
                shapes.update({x + "q": (H * (dk + rot), W), x + "dkv": (rank + rot, W), x + "dkv.norm": (rank,), x + "uk": (H * dk, rank),
                               x + "uv": (H * dv, rank), x + "sink": (H,), x + "g": (H, W)})
            else:
                shapes.update({x + "q": (H * dk, W), x + "k": (m["kv_heads"] * dk, W), x + "v": (m["kv_heads"] * dv, W)})
                if m.get("v_mix"):
                    shapes[x + "vmix"] = ()
            shapes[x + "o"] = (W, H * dv)
            if layer.get("mlp") is not None:
                ff = layer["mlp"]["ff"]
                shapes.update({p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
        shapes["final.norm"] = (W,)
        shapes["head"] = (self.vocab_size, W)
        return shapes


def random_weights(cfg: RovuraxConfig, seed: int = 0, device="cpu", dtype: torch.dtype = torch.bfloat16, gain: float = 1.0) -> Dict[str, torch.Tensor]:
    """Random tensors of the checkpoint's shapes, scaled so that activations stay in a useful range."""
    gen = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        t = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1"):
            t = 1 + 0.1 * t
        elif last == "vmix":
            t = torch.sigmoid(t)
        elif len(shape) == 2 and name != "embed":
            t = t * (gain / math.sqrt(shape[1]))
        out[name] = t.to(dtype)
    return out


def build_rovurax(cfg: RovuraxConfig, weights: Mapping[str, torch.Tensor], device: str = "cpu",
                  with_argmax: bool = True) -> Tuple[bytes, Dict[str, torch.Tensor]]:
    """Returns (ModelProto bytes, initializers); the initializers lie on ``device`` and are handed to
    ``SessionOptions.add_external_initializers``."""
    cfg.validate()
    g = PackedGraph(cfg, weights, device, key_starts=cfg.has_latents)
    eps, seq = cfg.norm_eps, ["cumulative_sequence_length", "past_seqlens", "block_table"]
    one = g.const32("plain.one", torch.ones(1))
    mix = g.const32("plain.mix", torch.ones(1, 1))
    residual, pending = g.embed("x0"), None       # pending: output of the layer before, still to be added

    def read(gamma: str, out: str, rows: str = "") -> str:
        """Add the pending output to the residual and return its norm."""
        nonlocal residual
        ins = [residual] + ([pending, mix, one] if pending else ["", "", ""]) + [one, gamma] + ([rows] if rows else [])
        outs = [out] + ([out + ".residual"] if pending and not rows else [])
        g.node("HyperConnectionNorm", ins, outs, streams=1, epsilon=eps)
        residual = outs[-1] if len(outs) > 1 else residual
        return out

    first = cfg.first_mixed()
    first_values = ("", 0)                        # tensor that holds the first mixed layer's values, and their first column
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer["mixer"]
        x, f, mlp = p + ".mix", p + ".mlp", layer.get("mlp")
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        h = read(g.const32(p + ".norm1"), p + ".h")
        base = ""
        if mlp is not None:    # its columns lie behind those the mixer fills
            gate = g.linear(h, f + ".gate", g.tensor(f + ".gate"), f + ".g")
            up = g.linear(h, f + ".up", g.tensor(f + ".up"), f + ".u")
            base = g.node("ClampedSwiGLU", [gate, up], [f + ".prod"], limit=float(mlp["limit"]), alpha=GATE_SLOPE, offset=UP_OFFSET,
                          lead_columns=H * dv)
        if layer["type"] == "latent_attention":
            packed = g.stacked(h, x + ".in", [g.tensor(x + n) for n in (".q", ".dkv", ".g")], x + ".packed")
            up = g.add(x + ".up", torch.cat([g.tensor(x + ".uk"), g.tensor(x + ".uv")]))
            att = g.node("LatentPagedAttention",
                         [packed, f"latent_cache.{i}"] + seq + g.rotary(m.get("rot")) +
                         [g.const32(x + ".dkv.norm"), up, g.const32(x + ".sink"), base, "key_starts"],
                         [x + ".mixed", f"latent_cache_out.{i}"], num_heads=H, head_size=dk, rotary_size=m["rot_dim"], v_head_size=dv,
                         latent_size=m["kv_rank"], latent_width=cfg.latent_widths(m)[0], scale=float(m["scale"]), epsilon=eps, gated=1)
        else:
            packed = g.stacked(h, x + ".in", [g.tensor(x + n) for n in (".q", ".k", ".v")], x + ".packed")
            ins = [packed, f"key_cache.{i}", f"value_cache.{i}"] + seq + [""] * 5
            if i == first:
                first_values = (packed, (H + m["kv_heads"]) * dk)
            mixes = bool(m.get("v_mix")) and i != first
            ins += [first_values[0], g.const32(x + ".vmix", g.tensor(x + ".vmix").reshape(1))] if mixes else ["", ""]
            ins.append(base)
            while not ins[-1]:
                ins.pop()
            att = g.node("GatedPagedAttention", ins, [x + ".mixed", f"key_cache_out.{i}", f"value_cache_out.{i}"], num_heads=H,
                         kv_num_heads=m["kv_heads"], head_size=dk, v_head_size=dv, scale=float(m["scale"]), epsilon=eps, kv_shared=0, gated=0,
                         chunk_size=int(m["mask"]["size"]) if m.get("mask") else 0, first_values_offset=first_values[1] if mixes else 0)
        out = [g.tensor(x + ".o")] + ([g.tensor(f + ".down")] if mlp is not None else [])
        pending = g.linear(att, p + ".out", torch.cat([w.to(g.dt) for w in out], 1), p + ".y")

    rows = read(g.const32("final.norm"), "final_rows", rows="logits_indices")
    g.linear(rows, "head", g.tensor("head"), "logits")
    return g.finish("rovurax", cfg.vocab_size, g.odt, with_argmax)
