"""Fegilix at sizes of real models' layers, beside the paged Llama decoder of equal width, depth, heads and feed-forward.

    python bench.py --workload fegilix [--sizes 2048,4096] [--steps K] [--warmup W]

Per size: prompt and decode throughput of both decoders through the registry's runner (random weights, bf16, greedy,
CUDA-graph decode), then the kernels that the designs do not share, each timed alone: ``us`` per launch, the bytes or
flops its job needs, and the fraction of the measured peak that makes (``of``: HBM bandwidth, bf16 tensor throughput, or
the nominal fp32 CUDA-core rate for the recurrences, whose arithmetic is 32-bit).  Kernel times are CUDA graphs of many
launches over rotating buffers larger than the L2.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..ops import _kernels as K
from .packed import KernelRows, graph_us, run_pair


def configs(width: int, layers: int = 8, vocab: int = 32000):
    """(fegilix, llama) config.json dicts of equal width, depth, heads and feed-forward."""
    heads, ff = width // 128, width * 7 // 2
    kv = heads // 4
    att = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"base": 500000.0, "dims": 128}}
    delta = {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": 4}
    mem = {"heads": heads // 2, "dim": 128, "vdim": 256, "gate_cap": 15.0}
    kinds = [("channel_delta", delta), ("mlstm", mem), ("channel_delta", delta), ("attention", att)]
    fegilix = {"architecture": "Fegilix", "vocab": vocab, "width": width, "streams": 4, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
               "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": {"kind": "dense", "ff": ff}} for i in range(layers)]}
    llama = {"architectures": ["LlamaForCausalLM"], "vocab_size": vocab, "hidden_size": width, "num_hidden_layers": layers,
             "num_attention_heads": heads, "num_key_value_heads": kv, "head_dim": 128, "intermediate_size": ff, "rope_theta": 500000.0}
    return fegilix, llama


def kernel_numbers(width: int, batch: int, prompt: int, context: int, streams: int = 4) -> List[Dict]:
    dev, bf, f32 = "cuda", torch.bfloat16, torch.float32
    heads, kv, H = width // 128, width // 512, 128
    torch.manual_seed(0)

    rows = KernelRows()
    row = rows.add

    for phase, T in (("decode", batch), ("prefill", batch * prompt)):
        n_buf = max(2, min(64, int(400e6 / (T * width * 4)))) if phase == "prefill" else 64
        n_buf = min(n_buf, 8) if phase == "prefill" else n_buf
        B = batch
        cu = (torch.arange(B + 1, dtype=torch.int32) * (T // B)).to(dev)
        past0 = torch.full((B,), 0 if phase == "prefill" else context, dtype=torch.int32, device=dev)
        # ---- residual + norm: hyper-connections beside the skip-norm
        ys = [torch.randn(T, width, dtype=bf, device=dev) for _ in range(n_buf)]
        xs = [torch.randn(T, streams, width, dtype=f32, device=dev) for _ in range(n_buf)]
        mix, wo, wi, gam = torch.eye(streams, device=dev), torch.ones(streams, device=dev), torch.full((streams,), 1 / streams, device=dev), \
            torch.ones(width, device=dev)
        us = graph_us([lambda x=x, y=y: K.hyper_norm(x, y, mix, wo, wi, gam, 1e-6) for x, y in zip(xs, ys)])
        row(f"hyper_norm {phase}", "fegilix", us, T * width * (8 * streams + 4))
        del xs
        g16 = torch.ones(width, dtype=bf, device=dev)
        rs = [torch.randn(T, width, dtype=bf, device=dev) for _ in range(n_buf)]
        us = graph_us([lambda x=x, y=y: K.norm(x, g16, skip=y, simplified=True, want_sum=True) for x, y in zip(rs, ys)])
        row(f"skip rms norm {phase}", "llama", us, T * width * 8)
        del rs, ys
        # ---- step 1 of attention
        bs = 128
        per = (context + prompt + bs) // bs + 1
        kc, vc = [torch.randn(B * per, bs, kv, H, dtype=bf, device=dev) for _ in range(2)]
        table = torch.arange(B * per, dtype=torch.int32, device=dev).view(per, B).t().contiguous()
        cos32, sin32 = torch.rand(per * bs, H // 2, device=dev), torch.rand(per * bs, H // 2, device=dev)
        cos16, sin16 = cos32.to(bf), sin32.to(bf)
        qn = torch.ones(H, device=dev)
        pk = [torch.randn(T, (2 * heads + 2 * kv) * H, dtype=bf, device=dev) for _ in range(n_buf)]
        us = graph_us([lambda x=x: K.qk_norm_rope(x, kc, vc, qn, qn, cos32, sin32, cu, past0, table, heads, H, H) for x in pk])
        row(f"qk_norm_rope {phase}", "fegilix", us, T * (heads + 2 * kv) * H * 4)
        qk = [p[:, :(heads + 2 * kv) * H].contiguous() for p in pk]
        us = graph_us([lambda x=x: K.paged_prep(x, kc, vc, cu, past0, table, heads, kv, cos16, sin16) for x in qk])
        row(f"paged_prep {phase}", "llama", us, T * (heads + 2 * kv) * H * 4)
        q = torch.randn(T, heads, H, dtype=bf, device=dev)
        sink = torch.zeros(heads, dtype=bf, device=dev)
        if phase == "prefill":
            fl = 4 * B * heads * H * prompt * (prompt + 1) / 2 * 1e-12
            calls = lambda split: [lambda: K.attn_prefill_paged(q, kc, vc, cu, past0, table, head_sink=sink if split else None, split_weights=split)] * 8
            row("attention prefill (split weights)", "fegilix", graph_us(calls(True)), tflop=fl)
            row("attention prefill", "llama", graph_us(calls(False)), tflop=fl)
        else:
            caches = [(torch.randn_like(kc), torch.randn_like(vc)) for _ in range(max(2, int(300e6 / (kc.numel() * 4))))]
            by = B * (context + 1) * kv * H * 4
            us = graph_us([lambda c=c: K.gqa_decode(q.view(B, heads, H), c[0], c[1], past0, head_sink=sink, block_table=table, split_weights=True) for c in caches] * 2)
            row("attention decode (fp32 weights)", "fegilix", us, by)
            us = graph_us([lambda c=c: K.gqa_decode(q.view(B, heads, H), c[0], c[1], past0, block_table=table, algo=2) for c in caches] * 2)
            row("attention decode", "llama", us, by)
            del caches
        us = graph_us([lambda x=x: K.head_gate(q, x[:, (heads + 2 * kv) * H:], x.shape[1], H) for x in pk])
        row(f"head_gate {phase}", "fegilix", us, T * heads * H * 6)
        del pk, qk, kc, vc
        # ---- recurrences
        slots = torch.arange(B, dtype=torch.int32, device=dev)
        G, dk, dv, taps = heads, 128, 128, 4
        C = 2 * G * dk + heads * dv
        conv, a_log, dtb, nrm = torch.randn(C, taps, device=dev), torch.zeros(heads, device=dev), torch.zeros(heads * dk, device=dev), torch.ones(dv, device=dev)
        nst = 2 if phase == "prefill" else max(2, int(300e6 / (B * heads * dk * dv * 4)))
        ring = torch.zeros(B, taps, C, dtype=bf, device=dev)
        states = [torch.zeros(B, heads, dk, dv, device=dev) for _ in range(nst)]
        x = torch.randn(T, C + heads, dtype=bf, device=dev)
        low = torch.randn(T, heads * (dk + dv), dtype=bf, device=dev)
        us = graph_us([lambda s=s: K.gated_delta(x, low, conv, a_log, dtb, nrm, ring, s, cu, past0, slots, G) for s in states])
        io = T * (C + heads + heads * (dk + dv) + heads * dv) * 2
        row(f"gated delta {phase}", "fegilix", us, 2 * B * heads * dk * dv * 4 + io, core_tflop=T * heads * dk * dv * 7e-12)
        hm, dvm = heads // 2, 256
        states = [torch.zeros(B, hm, dk, dvm, device=dev) for _ in range(nst)]
        aux = torch.zeros(B, hm, dk + 1, device=dev)
        xm = torch.randn(T, hm * (2 * dk + 2 * dvm + 2), dtype=bf, device=dev)
        zb, nm = torch.zeros(hm, device=dev), torch.ones(hm * dvm, device=dev)
        us = graph_us([lambda s=s: K.mlstm(xm, zb, zb, nm, s, aux, cu, past0, slots, 15.0) for s in states])
        io = T * hm * (2 * dk + 3 * dvm) * 2
        row(f"mlstm {phase}", "fegilix", us, 2 * B * hm * dk * dvm * 4 + io, core_tflop=T * hm * dk * dvm * 5e-12)
        del states, x, low, xm
        torch.cuda.empty_cache()
    return rows.rows


def run(sizes, batch: int = 8, prompt: int = 1024, steps: int = 64, warmup: int = 4) -> Dict:
    return run_pair("fegilix", configs, kernel_numbers, sizes, batch, prompt, steps, warmup)
