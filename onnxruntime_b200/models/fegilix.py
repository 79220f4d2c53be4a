"""Fegilix decoder as an ONNX graph in packed serving form.

A decoder whose layers are of three kinds (softmax attention with a sink and an output gate, gated delta rule with
per-channel decay, mLSTM matrix memory) around hyper-connections: ``streams`` fp32 copies of the residual that every
sublayer reads through one weight vector and writes back through a mixing matrix.  config.json gives every size and
constant; the graph is built from it and from the checkpoint's tensors.

Inputs are those of the paged Llama graph (``input_ids``, ``cumulative_sequence_length``, ``past_seqlens``,
``block_table``, ``logits_indices``) plus ``state_slots`` when a layer is recurrent, and the cache tensors that
``FegilixConfig.cache_tensors`` lists.  A layer with ``kv_from`` reads the key / value cache that an earlier layer has
just written.

The projections of a sublayer that read the same input are one MatMul over stacked rows (padded to a multiple of eight);
the two low-rank maps of the delta rule share one down projection and one block-diagonal up projection.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch

from .. import onnx_lite as ol
from .decoder_cache import CacheTensor
from .packed_graph import TORCH_DT, PackedGraph, padded_head_widths
from .rotary import rotary_tables  # noqa: F401

T = ol.TensorProto

UNIT_EPS = 1e-6          # inside the root of the unit norms of the delta rule's q and k
DENOMINATOR_EPS = 1e-6   # added to the mLSTM denominator
MIXERS = ("attention", "channel_delta", "mlstm")


@dataclass
class FegilixConfig:
    vocab_size: int
    width: int
    layers: List[Dict[str, Any]]
    streams: Optional[int] = None         # None: one plain residual stream
    norm_eps: float = 1e-6
    logit_softcap: Optional[float] = None
    dtype: str = "bf16"
    max_seq_len: int = 2048               # rows of the rotary tables
    architecture: str = field(default="Fegilix", repr=False)

    @staticmethod
    def from_json(d: Mapping[str, Any], dtype: str = "bf16", max_seq_len: int = 2048) -> "FegilixConfig":
        cfg = FegilixConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), layers=list(d["layers"]),
                            streams=int(d["streams"]) if d.get("streams") is not None else None, norm_eps=float(d["norm"]["eps"]),
                            logit_softcap=float(d["logit_softcap"]) if d.get("logit_softcap") else None, dtype=dtype,
                            max_seq_len=int(max_seq_len))
        cfg.validate()
        return cfg

    def to_json(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "layers": self.layers, "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size,
                             "width": self.width}
        if self.streams is not None:
            d["streams"] = self.streams
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d

    def validate(self) -> None:
        for i, layer in enumerate(self.layers):
            m = layer["mixer"]
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
            if layer.get("mlp") is not None and layer["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {layer['mlp']['kind']!r}")
            j = m.get("kv_from")
            if j is not None:
                if layer["type"] != "attention" or not 0 <= j < i or self.layers[j]["type"] != "attention" \
                        or self.layers[j]["mixer"].get("kv_from") is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with keys of its own")
                src = self.layers[j]["mixer"]
                if any(m[k] != src[k] for k in ("kv_heads", "dim", "vdim")):
                    raise ValueError(f"layer {i}: key / value sizes differ from those of layer {j}")
            if layer["type"] != "mlstm" and m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")

    @property
    def is_recurrent(self) -> bool:
        return any(layer["type"] != "attention" for layer in self.layers)

    def cache_widths(self, m: Mapping[str, Any]) -> Tuple[int, int]:
        return padded_head_widths(self.dtype, m["dim"], m["vdim"])

    def cache_tensors(self, tp_size: int = 1) -> List[CacheTensor]:
        if tp_size != 1:
            raise ValueError("this graph is built for one device")
        dt = TORCH_DT[self.dtype]
        out: List[CacheTensor] = []
        for i, layer in enumerate(self.layers):
            m = layer["mixer"]
            if layer["type"] == "attention":
                if m.get("kv_from") is None:
                    kw, vw = self.cache_widths(m)
                    out.append(CacheTensor(f"key_cache.{i}", f"key_cache_out.{i}", "paged", (m["kv_heads"], kw), dt))
                    out.append(CacheTensor(f"value_cache.{i}", f"value_cache_out.{i}", "paged", (m["kv_heads"], vw), dt))
                continue
            if layer["type"] == "channel_delta":
                channels = 2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"]
                out.append(CacheTensor(f"conv_state.{i}", f"conv_state_out.{i}", "slot", (m["conv"], channels), dt))
            else:
                out.append(CacheTensor(f"aux_state.{i}", f"aux_state_out.{i}", "slot", (m["heads"], m["dim"] + 1), torch.float32))
            out.append(CacheTensor(f"state.{i}", f"state_out.{i}", "slot", (m["heads"], m["dim"], m["vdim"]), torch.float32))
        return out

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Names and shapes of the checkpoint, except the ranks of the low-rank maps, which only the tensors know (-1)."""
        W, shapes = self.width, {"embed": (self.vocab_size, self.width)}
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}.", layer["mixer"]
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            x = p + "mix."
            shapes[p + "norm1"] = (W,)
            shapes[x + "q"] = ((H if layer["type"] != "channel_delta" else m["kv_heads"]) * dk, W)
            shapes[x + "o"] = (W, H * dv)
            if layer["type"] == "attention":
                shapes.update({x + "q.norm": (dk,), x + "sink": (H,), x + "g": (H * dv, W)})
                if m.get("kv_from") is None:
                    shapes.update({x + "k": (m["kv_heads"] * dk, W), x + "v": (m["kv_heads"] * dv, W), x + "k.norm": (dk,)})
            elif layer["type"] == "channel_delta":
                G, taps = m["kv_heads"], m["conv"]
                shapes.update({x + "k": (G * dk, W), x + "v": (H * dv, W), x + "q.conv": (G * dk, taps), x + "k.conv": (G * dk, taps),
                               x + "v.conv": (H * dv, taps), x + "b": (H, W), x + "A_log": (H,), x + "norm": (dv,), x + "a1": (-1, W),
                               x + "a2": (H * dk, -1), x + "dt_bias": (H * dk,), x + "g1": (-1, W), x + "g2": (H * dv, -1)})
            else:
                shapes.update({x + "k": (H * dk, W), x + "v": (H * dv, W), x + "g": (H * dv, W), x + "norm": (H * dv,), x + "i": (H, W),
                               x + "i.b": (H,), x + "f": (H, W), x + "f.b": (H,)})
            subs = 1
            if layer.get("mlp") is not None:
                subs, ff = 2, layer["mlp"]["ff"]
                shapes.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
            if self.streams is not None:
                for q in range(1, subs + 1):
                    shapes.update({f"{p}hc{q}.in": (self.streams,), f"{p}hc{q}.out": (self.streams,), f"{p}hc{q}.mix": (self.streams, self.streams)})
        shapes["final.norm"] = (W,)
        shapes["head"] = (self.vocab_size, W)
        return shapes


def default_rank(cfg: FegilixConfig) -> int:
    """Rank of the low-rank maps for random weights: the key head size of the first delta-rule layer."""
    return next((layer["mixer"]["dim"] for layer in cfg.layers if layer["type"] == "channel_delta"), 16)


def random_weights(cfg: FegilixConfig, seed: int = 0, device="cpu", low_rank: int = 16, dtype: torch.dtype = torch.bfloat16,
                   gain: float = 1.0) -> Dict[str, torch.Tensor]:
    """Random tensors of the checkpoint's shapes, scaled so that activations and gates stay in a useful range."""
    gen = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        shape = tuple(low_rank if d < 0 else d for d in shape)
        last = name.rsplit(".", 1)[-1]
        t = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
        if last in ("norm", "norm1", "norm2"):
            t = 1 + 0.1 * t
        elif ".hc" in name:
            n = cfg.streams
            base = torch.eye(n, device=device) if last == "mix" else torch.full(shape, 1.0 / n if last == "in" else 1.0, device=device)
            t = base + 0.1 * t
        elif last == "conv":
            t = t / math.sqrt(shape[1])
        elif last == "A_log":
            t = 0.5 * t - 1
        elif last == "dt_bias":
            t = t - 2
        elif name.endswith("f.b"):
            t = t + 3
        elif len(shape) == 2 and name != "embed":
            t = t * (gain / math.sqrt(shape[1]))
        out[name] = t.to(dtype)
    return out


def build_fegilix(cfg: FegilixConfig, weights: Mapping[str, torch.Tensor], device: str = "cpu",
                  with_argmax: bool = True) -> Tuple[bytes, Dict[str, torch.Tensor]]:
    """Returns (ModelProto bytes, initializers); the initializers lie on ``device`` and are handed to
    ``SessionOptions.add_external_initializers``."""
    cfg.validate()
    g = PackedGraph(cfg, weights, device, state_slots=cfg.is_recurrent)
    tensor, const32, node, linear, stacked, rotary = g.tensor, g.const32, g.node, g.linear, g.stacked, g.rotary
    dt, eps = g.dt, cfg.norm_eps

    # ---- residual streams
    streams = cfg.streams if cfg.streams is not None else 1
    residual, pending = g.embed("x0"), None        # pending: (sublayer output, mix, w_out) still to be written back

    def hyper_weights(prefix: str) -> Tuple[str, str, str]:
        if cfg.streams is None:
            one = torch.ones(1)
            return const32("plain.in", one), const32("plain.mix", one.reshape(1, 1)), const32("plain.out", one)
        return const32(prefix + ".in"), const32(prefix + ".mix"), const32(prefix + ".out")

    def read(w_in: str, gamma: str, out: str, rows: str = "") -> str:
        """Write the pending sublayer output back and return the normed input of the next sublayer."""
        nonlocal residual, pending
        ins = [residual] + (list(pending) if pending else ["", "", ""]) + [w_in, gamma] + ([rows] if rows else [])
        outs = [out]
        if pending and not rows:
            outs.append(out + ".streams")
        node("HyperConnectionNorm", ins, outs, streams=streams, epsilon=eps)
        if len(outs) > 1:
            residual = outs[1]
        return out

    seq = ["cumulative_sequence_length", "past_seqlens"]
    kv_names: Dict[int, Tuple[str, str]] = {}
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer["mixer"]
        x = p + ".mix"
        w_in, mix, w_out = hyper_weights(p + ".hc1")
        h = read(w_in, const32(p + ".norm1"), p + ".h1")
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            src = m.get("kv_from")
            parts = [tensor(x + ".q")] + ([tensor(x + ".k"), tensor(x + ".v")] if src is None else []) + [tensor(x + ".g")]
            packed = stacked(h, x + ".qkvg", parts, x + ".packed")
            if src is None:
                caches, outs = [f"key_cache.{i}", f"value_cache.{i}"], [f"key_cache_out.{i}", f"value_cache_out.{i}"]
                kv_names[i] = (outs[0], outs[1])
            else:   # the tensors that layer src has just written: the edge orders the two nodes
                caches, outs = list(kv_names[src]), []
            att = node("GatedPagedAttention",
                       [packed] + caches + seq + ["block_table"] + rotary(m.get("rot")) +
                       [const32(x + ".q.norm"), const32(x + ".k.norm") if src is None else "", const32(x + ".sink")],
                       [x + ".mixed"] + outs, num_heads=H, kv_num_heads=m["kv_heads"], head_size=dk, v_head_size=dv, scale=float(m["scale"]),
                       epsilon=eps, kv_shared=int(src is not None), gated=1)
        elif layer["type"] == "channel_delta":
            packed = stacked(h, x + ".qkvb", [tensor(x + n) for n in (".q", ".k", ".v", ".b")], x + ".packed")
            a2, g2 = tensor(x + ".a2").to(dt), tensor(x + ".g2").to(dt)
            ra, rg = a2.shape[1], g2.shape[1]
            down = stacked(h, x + ".low1", [tensor(x + ".a1"), tensor(x + ".g1")], x + ".low")
            up = torch.zeros(a2.shape[0] + g2.shape[0], -(-(ra + rg) // 8) * 8, dtype=dt, device=device)
            up[:a2.shape[0], :ra] = a2
            up[a2.shape[0]:, ra:ra + rg] = g2
            low = linear(down, x + ".low2", up, x + ".low_out")
            conv = torch.cat([tensor(x + n).float() for n in (".q.conv", ".k.conv", ".v.conv")])
            att = node("PackedGatedDelta",
                       [packed, low, const32(x + ".conv", conv), const32(x + ".A_log"), const32(x + ".dt_bias"), const32(x + ".norm"),
                        f"conv_state.{i}", f"state.{i}"] + seq + ["state_slots"],
                       [x + ".mixed", f"conv_state_out.{i}", f"state_out.{i}"], num_heads=H, kv_num_heads=m["kv_heads"], head_size=dk,
                       v_head_size=dv, epsilon=eps, unit_epsilon=UNIT_EPS)
        else:
            packed = stacked(h, x + ".qkvgif", [tensor(x + n) for n in (".q", ".k", ".v", ".g", ".i", ".f")], x + ".packed")
            att = node("PackedMLstm",
                       [packed, const32(x + ".i.b"), const32(x + ".f.b"), const32(x + ".norm"), f"state.{i}", f"aux_state.{i}"] + seq +
                       ["state_slots"],
                       [x + ".mixed", f"state_out.{i}", f"aux_state_out.{i}"], num_heads=H, head_size=dk, v_head_size=dv,
                       gate_cap=float(m["gate_cap"]), epsilon=eps, denominator_epsilon=DENOMINATOR_EPS)
        pending = (linear(att, x + ".o", tensor(x + ".o"), x + ".out"), mix, w_out)
        if layer.get("mlp") is not None:
            f = p + ".mlp"
            w_in, mix, w_out = hyper_weights(p + ".hc2")
            h = read(w_in, const32(p + ".norm2"), p + ".h2")
            gate = linear(h, f + ".gate", tensor(f + ".gate"), f + ".g")
            up = linear(h, f + ".up", tensor(f + ".up"), f + ".u")
            act = node("FastGelu", [gate], [f + ".act"], domain="com.microsoft")
            prod = node("Mul", [act, up], [f + ".prod"], domain="")
            pending = (linear(prod, f + ".down", tensor(f + ".down"), f + ".out"), mix, w_out)

    rows = read(const32("streams.sum", torch.ones(streams)), const32("final.norm"), "final_rows", rows="logits_indices")
    logit_type = g.odt
    if cfg.logit_softcap is None:
        linear(rows, "head", tensor("head"), "logits")
    else:
        node("SoftCap", [linear(rows, "head", tensor("head"), "raw_logits")], ["logits"], cap=cfg.logit_softcap)
        logit_type = T.FLOAT
    return g.finish("fegilix", cfg.vocab_size, logit_type, with_argmax)
