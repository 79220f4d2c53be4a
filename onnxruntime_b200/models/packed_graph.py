"""Assembly of decoder graphs in packed serving form: what the model files that build such graphs share.

The inputs are those of every packed decoder (``input_ids``, ``cumulative_sequence_length``, ``past_seqlens``,
``block_table``, ``logits_indices``), ``state_slots`` when a layer is recurrent, ``key_starts`` when a layer expands
cached latents for prompts, and the cache tensors the configuration declares.
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional, Sequence, Tuple

import torch

from .. import onnx_lite as ol
from .rotary import rotary_tables

T = ol.TensorProto
FUSED = "com.ortb200"

TORCH_DT = {"bf16": torch.bfloat16, "fp16": torch.float16, "fp32": torch.float32}
ONNX_DT = {"bf16": T.BFLOAT16, "fp16": T.FLOAT16, "fp32": T.FLOAT}


def padded_head_widths(dtype: str, dim: int, vdim: int) -> Tuple[int, int]:
    """Stored widths of a key and a value head: 16-bit heads are padded to the sizes of the tensor-core kernels (zeros change
    neither a score nor an output), others to a multiple of four."""
    wide = max(dim, vdim)
    if dtype != "fp32" and wide <= 128:
        return (64, 64) if wide <= 64 else (128, 128)
    return -(-dim // 4) * 4, -(-vdim // 4) * 4


class PackedGraph:
    """Nodes, initializers and checked checkpoint tensors of one decoder.  ``cfg`` has ``dtype``, ``max_seq_len``,
    ``tensor_shapes()`` and ``cache_tensors()``; initializers lie on ``device``."""

    def __init__(self, cfg, weights: Mapping[str, torch.Tensor], device: str, state_slots: bool = False, key_starts: bool = False):
        self.cfg, self.weights, self.device = cfg, weights, device
        self.dt, self.odt = TORCH_DT[cfg.dtype], ONNX_DT[cfg.dtype]
        self.expected = cfg.tensor_shapes()
        self.nodes: List[ol.Node] = []
        self.inits: List[ol.Tensor] = []
        self.store: Dict[str, torch.Tensor] = {}
        self._tables: Dict[str, Tuple[str, str]] = {}
        info = ol.make_tensor_value_info
        self.inputs = [info("input_ids", T.INT64, ["tokens"]), info("cumulative_sequence_length", T.INT32, ["batch_plus_1"]),
                       info("past_seqlens", T.INT32, ["batch"]), info("block_table", T.INT32, ["batch", "max_blocks"]),
                       info("logits_indices", T.INT64, ["rows"])]
        if state_slots:
            self.inputs.append(info("state_slots", T.INT32, ["batch"]))
        if key_starts:
            self.inputs.append(info("key_starts", T.INT32, ["batch_plus_1"]))
        self.outputs = []
        for c in cfg.cache_tensors():
            lead = ["num_blocks", "block_size"] if c.kind == "paged" else ["num_slots"]
            elem = self.odt if c.dtype == self.dt else T.FLOAT
            self.inputs.append(info(c.input, elem, lead + list(c.shape)))
            self.outputs.append(info(c.output, elem, lead + list(c.shape)))

    def tensor(self, name: str) -> torch.Tensor:
        if name not in self.weights:
            raise KeyError(f"the checkpoint has no tensor {name!r}")
        w, want = self.weights[name], self.expected[name]
        if len(w.shape) != len(want) or any(e >= 0 and e != s for e, s in zip(want, w.shape)):
            raise ValueError(f"tensor {name!r} has shape {tuple(w.shape)}, the configuration wants {want}")
        return w.to(self.device)

    def add(self, name: str, w: torch.Tensor, dtype: Optional[torch.dtype] = None) -> str:
        if name not in self.store:
            w = w.to(dtype or self.dt).contiguous()
            self.store[name] = w
            self.inits.append(ol.make_external_tensor(name, self.odt if w.dtype == self.dt else T.FLOAT, w.shape))
        return name

    def const32(self, name: str, w: Optional[torch.Tensor] = None) -> str:
        return self.add(name, self.tensor(name) if w is None else w.to(self.device), torch.float32)

    def node(self, op: str, inputs: List[str], outputs: List[str], domain: str = FUSED, **attrs) -> str:
        self.nodes.append(ol.make_node(op, inputs, outputs, name=outputs[0] + "/" + op, domain=domain, **attrs))
        return outputs[0]

    def linear(self, x: str, name: str, rows: torch.Tensor, out: str) -> str:
        """out = x @ rows^T (rows [out, in] as in the checkpoint)."""
        self.add(name, rows.to(self.dt).t())
        return self.node("MatMul", [x, name], [out], domain="")

    def stacked(self, x: str, name: str, parts: Sequence[torch.Tensor], out: str) -> str:
        """One MatMul over stacked rows, padded to a multiple of eight."""
        rows = torch.cat([p.to(self.dt) for p in parts])
        pad = -rows.shape[0] % 8
        if pad:
            rows = torch.cat([rows, rows.new_zeros(pad, rows.shape[1])])
        return self.linear(x, name, rows, out)

    def rotary(self, rot: Optional[Mapping[str, Any]]) -> List[str]:
        """Names of the cos / sin tables of ``rot`` (shared by the layers that agree on it), or two absent inputs."""
        if not rot:
            return ["", ""]
        key = repr(sorted(rot.items(), key=lambda kv: kv[0]))
        if key not in self._tables:
            cos, sin = rotary_tables(rot, self.cfg.max_seq_len, self.device)
            k = len(self._tables)
            self._tables[key] = (self.const32(f"rotary.{k}.cos", cos), self.const32(f"rotary.{k}.sin", sin))
        return list(self._tables[key])

    def embed(self, out: str) -> str:
        self.add("embed", self.tensor("embed"))
        return self.node("Gather", ["embed", "input_ids"], [out], domain="", axis=0)

    def finish(self, name: str, vocab: int, logits_type: int, with_argmax: bool) -> Tuple[bytes, Dict[str, torch.Tensor]]:
        """(ModelProto bytes, initializers) of a graph whose "logits" have been produced."""
        outputs = [ol.make_tensor_value_info("logits", logits_type, ["rows", vocab])]
        if with_argmax:
            self.node("ArgMax", ["logits"], ["next_tokens"], domain="", axis=-1, keepdims=0)
            outputs.append(ol.make_tensor_value_info("next_tokens", T.INT64, ["rows"]))
        graph = ol.make_graph(self.nodes, name, self.inputs, outputs + self.outputs, self.inits)
        model = ol.make_model(graph, opset=17, metadata={"architecture": self.cfg.architecture}, extra_opsets={FUSED: 1})
        return model.serialize(), self.store
