"""Shared by the tests of packed decoders: single operators over bound tensors, and whole models through the registry against
an oracle module (``forward`` and ``rounding_noise``)."""
import pytest
import torch

import onnxruntime_b200 as ort
from onnxruntime_b200 import onnx_lite as ol
from onnxruntime_b200.models.registry import create_decoder

CPU, GPU = "CPUExecutionProvider", "CUDAExecutionProvider"
PROVIDERS = [pytest.param(CPU, id="cpu"), pytest.param(GPU, marks=pytest.mark.gpu, id="gpu")]
# (provider, type of activations)
KINDS = [pytest.param((CPU, torch.float32), id="cpu-fp32"), pytest.param((GPU, torch.float32), marks=pytest.mark.gpu, id="gpu-fp32"),
         pytest.param((GPU, torch.bfloat16), marks=pytest.mark.gpu, id="gpu-bf16")]
T = ol.TensorProto
ONNX = {torch.float32: T.FLOAT, torch.bfloat16: T.BFLOAT16, torch.int32: T.INT32, torch.int64: T.INT64}



def run_op(provider, op, inputs, outputs, domain="com.ortb200", **attrs):
    """One node over torch inputs (None = absent).  ``outputs``: tensors that receive the results; an output that is one of the
    inputs is updated in place.  Returns the outputs on the CPU."""
    dev = "cuda" if provider == GPU else "cpu"
    moved = {}
    def put(t):
        if id(t) not in moved:
            moved[id(t)] = t.to(dev)
        return moved[id(t)]
    names = [f"i{k}" if t is not None else "" for k, t in enumerate(inputs)]
    while names and not names[-1]:
        names.pop()
    info = [ol.make_tensor_value_info(f"i{k}", ONNX[t.dtype], list(t.shape)) for k, t in enumerate(inputs) if t is not None]
    outs = [ol.make_tensor_value_info(f"o{k}", ONNX[t.dtype], list(t.shape)) for k, t in enumerate(outputs)]
    graph = ol.make_graph([ol.make_node(op, names, [f"o{k}" for k in range(len(outputs))], name="n", domain=domain, **attrs)], "g", info, outs, [])
    sess = ort.InferenceSession(ol.make_model(graph, opset=17, extra_opsets={"com.ortb200": 1}).serialize(), providers=[provider],
                                **({"enable_fallback": False} if provider == GPU else {}))
    binding = sess.io_binding()
    for k, t in enumerate(inputs):
        if t is not None:
            binding.bind_torch_input(f"i{k}", put(t))
    results = [put(t) for t in outputs]
    for k, t in enumerate(results):
        binding.bind_torch_output(f"o{k}", t)
    sess.run_with_iobinding(binding)
    if provider == GPU:
        sess.check_device_status()
    for t in outputs:                       # in-place operands keep their identity for the next call of a test
        t.copy_(put(t).cpu())
    return list(outputs)


def close(got, want, dtype, tol=None):
    got, want = got.double(), want.double()
    tol = tol or (2e-5 if dtype == torch.float32 else 2e-2)
    scale = want.abs().max().clamp_min(1e-3)
    assert torch.isfinite(got).all()
    assert (got - want).abs().max() <= tol * scale, float((got - want).abs().max() / scale)


def i32(*v):
    return torch.tensor(v, dtype=torch.int32)


def tokens_of(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def decoder(cfg, w, kind, **kw):
    provider, dt = kind
    kw.setdefault("batch", 4)
    kw.setdefault("max_len", 96)
    kw.setdefault("block_size", 16 if provider == CPU else 128)
    return create_decoder(cfg, w, "bfloat16" if dt == torch.bfloat16 else "float32", provider=provider, **kw)


class Reference:
    """Logits of a token sequence, and what 16-bit projections alone would change at every place (its conditioning)."""

    def __init__(self, oracle, cfg, w, tokens, logits=None):
        self.oracle, self.args, self._noise = oracle, (cfg, w, tokens), None
        self.logits = oracle.forward(cfg, w, tokens) if logits is None else logits

    @property
    def noise(self):
        if self._noise is None:
            self._noise = self.oracle.rounding_noise(*self.args)
        return self._noise

    def __getitem__(self, rows):
        part = Reference(self.oracle, *self.args, logits=self.logits[rows])
        part.rows, part.whole = rows, self
        return part


def relative_error(diff, logits):
    diff = diff - diff.mean(-1, keepdim=True)
    return diff.pow(2).mean(-1).sqrt() / logits.pow(2).mean().sqrt()


def logits_close(got, want, dtype):
    got = got.double().cpu()
    assert got.shape == want.logits.shape and torch.isfinite(got).all()
    rel = relative_error(got - want.logits, want.logits)
    if dtype == torch.float32:
        assert rel.max() < 1e-4, float(rel.max())
    else:
        noise = want.whole.noise[want.rows] if hasattr(want, "whole") else want.noise
        limit = 0.06 + 2.5 * relative_error(noise, want.logits)
        assert (rel < limit).all(), float((rel / limit).max())


def feed(runner, seq, tokens, cuts):
    """The tokens of one sequence in portions; logits of every place."""
    out, at = [], 0
    for n in cuts:
        out.append(runner.step([(seq, tokens[at:at + n], list(range(n)))]))
        at += n
    assert at == len(tokens)
    return torch.cat(out)


def greedy_reference(oracle, cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
