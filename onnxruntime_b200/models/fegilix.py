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

T = ol.TensorProto
FUSED = "com.ortb200"

_TORCH_DT = {"bf16": torch.bfloat16, "fp16": torch.float16, "fp32": torch.float32}
_ONNX_DT = {"bf16": T.BFLOAT16, "fp16": T.FLOAT16, "fp32": T.FLOAT}

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
        """Stored widths of a key and a value head: 16-bit heads are padded to the sizes of the tensor-core kernels (zeros
        change neither a score nor an output), others to a multiple of four."""
        wide = max(m["dim"], m["vdim"])
        if self.dtype != "fp32" and wide <= 128:
            return (64, 64) if wide <= 64 else (128, 128)
        return -(-m["dim"] // 4) * 4, -(-m["vdim"] // 4) * 4

    def cache_tensors(self, tp_size: int = 1) -> List[CacheTensor]:
        if tp_size != 1:
            raise ValueError("this graph is built for one device")
        dt = _TORCH_DT[self.dtype]
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


def rotary_tables(rot: Mapping[str, Any], rows: int, device="cpu") -> Tuple[torch.Tensor, torch.Tensor]:
    """fp32 cos / sin [rows, dims / 2] of positions 0 .. rows - 1 (angles in float64), with the three-band frequency
    rescaling of long-context Llama models when ``rot`` has "scaling"."""
    half = rot["dims"] // 2
    f = float(rot["base"]) ** (-2.0 * torch.arange(half, dtype=torch.float64) / rot["dims"])
    sc = rot.get("scaling")
    if sc:
        wavelength = 2.0 * math.pi / f
        s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
        blend = (1.0 - s) * f / sc["factor"] + s * f
        f = torch.where(wavelength < sc["original"] / sc["high"], f, torch.where(wavelength > sc["original"] / sc["low"], f / sc["factor"], blend))
    angles = torch.outer(torch.arange(rows, dtype=torch.float64), f)
    return angles.cos().float().to(device), angles.sin().float().to(device)


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
    dt, odt = _TORCH_DT[cfg.dtype], _ONNX_DT[cfg.dtype]
    W, eps = cfg.width, cfg.norm_eps
    nodes: List[ol.Node] = []
    inits: List[ol.Tensor] = []
    store: Dict[str, torch.Tensor] = {}
    expected = cfg.tensor_shapes()

    def tensor(name: str) -> torch.Tensor:
        if name not in weights:
            raise KeyError(f"the checkpoint has no tensor {name!r}")
        w, want = weights[name], expected[name]
        if len(w.shape) != len(want) or any(e >= 0 and e != s for e, s in zip(want, w.shape)):
            raise ValueError(f"tensor {name!r} has shape {tuple(w.shape)}, the configuration wants {want}")
        return w.to(device)

    def add(name: str, w: torch.Tensor, dtype: Optional[torch.dtype] = None) -> str:
        if name not in store:
            w = w.to(dtype or dt).contiguous()
            store[name] = w
            inits.append(ol.make_external_tensor(name, odt if w.dtype == dt else T.FLOAT, w.shape))
        return name

    def const32(name: str, w: Optional[torch.Tensor] = None) -> str:
        return add(name, tensor(name) if w is None else w.to(device), torch.float32)

    def node(op: str, inputs: List[str], outputs: List[str], domain: str = FUSED, **attrs) -> str:
        nodes.append(ol.make_node(op, inputs, outputs, name=outputs[0] + "/" + op, domain=domain, **attrs))
        return outputs[0]

    def linear(x: str, name: str, rows: torch.Tensor, out: str) -> str:
        """out = x @ rows^T (rows [out, in] as in the checkpoint)."""
        add(name, rows.to(dt).t())
        return node("MatMul", [x, name], [out], domain="")

    def stacked(x: str, name: str, parts: List[torch.Tensor], out: str) -> str:
        rows = torch.cat([p.to(dt) for p in parts])
        pad = -rows.shape[0] % 8
        if pad:
            rows = torch.cat([rows, rows.new_zeros(pad, rows.shape[1])])
        return linear(x, name, rows, out)

    inputs = [ol.make_tensor_value_info("input_ids", T.INT64, ["tokens"]),
              ol.make_tensor_value_info("cumulative_sequence_length", T.INT32, ["batch_plus_1"]),
              ol.make_tensor_value_info("past_seqlens", T.INT32, ["batch"]),
              ol.make_tensor_value_info("block_table", T.INT32, ["batch", "max_blocks"]),
              ol.make_tensor_value_info("logits_indices", T.INT64, ["rows"])]
    if cfg.is_recurrent:
        inputs.append(ol.make_tensor_value_info("state_slots", T.INT32, ["batch"]))
    outputs = []
    for c in cfg.cache_tensors():
        lead = ["num_blocks", "block_size"] if c.kind == "paged" else ["num_slots"]
        elem = odt if c.dtype == dt else T.FLOAT
        inputs.append(ol.make_tensor_value_info(c.input, elem, lead + list(c.shape)))
        outputs.append(ol.make_tensor_value_info(c.output, elem, lead + list(c.shape)))

    tables: Dict[str, Tuple[str, str]] = {}

    def rotary(rot: Optional[Mapping[str, Any]]) -> List[str]:
        if not rot:
            return ["", ""]
        key = repr(sorted(rot.items(), key=lambda kv: kv[0]))
        if key not in tables:
            cos, sin = rotary_tables(rot, cfg.max_seq_len, device)
            k = len(tables)
            tables[key] = (const32(f"rotary.{k}.cos", cos), const32(f"rotary.{k}.sin", sin))
        return list(tables[key])

    # ---- residual streams
    streams = cfg.streams if cfg.streams is not None else 1
    add("embed", tensor("embed"))
    node("Gather", ["embed", "input_ids"], ["x0"], domain="", axis=0)
    residual, pending = "x0", None        # pending: (sublayer output, mix, w_out) still to be written back

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
    logit_type = odt
    if cfg.logit_softcap is None:
        linear(rows, "head", tensor("head"), "logits")
    else:
        node("SoftCap", [linear(rows, "head", tensor("head"), "raw_logits")], ["logits"], cap=cfg.logit_softcap)
        logit_type = T.FLOAT
    outputs.insert(0, ol.make_tensor_value_info("logits", logit_type, ["rows", cfg.vocab_size]))
    if with_argmax:
        node("ArgMax", ["logits"], ["next_tokens"], domain="", axis=-1, keepdims=0)
        outputs.insert(1, ol.make_tensor_value_info("next_tokens", T.INT64, ["rows"]))
    graph = ol.make_graph(nodes, "fegilix", inputs, outputs, inits)
    model = ol.make_model(graph, opset=17, metadata={"architecture": cfg.architecture}, extra_opsets={FUSED: 1})
    return model.serialize(), store
