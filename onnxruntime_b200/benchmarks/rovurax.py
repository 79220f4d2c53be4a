"""Rovurax at sizes of real models' layers, beside the paged Llama decoder of equal width, depth, heads and feed-forward.

    python bench.py --workload rovurax [--sizes 2048,4096] [--steps K] [--warmup W]

Per size: prompt and decode throughput of both decoders through the registry's runner (random weights, bf16, greedy,
CUDA-graph decode), then the kernels that the designs do not share, each timed alone: ``us`` per launch, the bytes or
flops its job needs, and the fraction of the measured peak that makes (``of``: HBM bandwidth or bf16 tensor throughput).
Kernel times are CUDA graphs of many launches over rotating buffers larger than the L2.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..ops import _kernels as K
from .packed import KernelRows, graph_us, run_pair

H, ROT, RANK, CHUNK = 128, 64, 512, 512


def configs(width: int, layers: int = 8, vocab: int = 32000):
    """(rovurax, llama) config.json dicts of equal width, depth, heads and feed-forward."""
    heads, ff = width // H, width * 7 // 2
    att = {"heads": heads, "kv_heads": heads // 4, "dim": H, "vdim": H, "scale": H ** -0.5, "mask": {"size": CHUNK}, "v_mix": True}
    lat = {"heads": heads, "dim": H, "rot_dim": ROT, "vdim": H, "kv_rank": RANK, "scale": (H + ROT) ** -0.5,
           "rot": {"base": 500000.0, "dims": ROT, "scaling": {"factor": 4.0, "fast": 32.0, "slow": 1.0, "original": 8192}}}
    kinds = [("attention", att), ("latent_attention", lat)]
    rovurax = {"architecture": "Rovurax", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
               "layers": [{"type": kinds[i % 2][0], "mixer": kinds[i % 2][1], "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}} for i in range(layers)]}
    llama = {"architectures": ["LlamaForCausalLM"], "vocab_size": vocab, "hidden_size": width, "num_hidden_layers": layers,
             "num_attention_heads": heads, "num_key_value_heads": heads // 4, "head_dim": H, "intermediate_size": ff, "rope_theta": 500000.0}
    return rovurax, llama


def visible_keys(n: int, chunk: int) -> int:
    """Pairs of a query and a key it sees in a prompt of n tokens."""
    full, rest = divmod(n, chunk)
    return full * chunk * (chunk + 1) // 2 + rest * (rest + 1) // 2


def kernel_numbers(width: int, batch: int, prompt: int, context: int) -> List[Dict]:
    dev, bf, f32 = "cuda", torch.bfloat16, torch.float32
    rows = KernelRows()
    row = rows.add
    N, kv, ff, B = width // H, width // (4 * H), width * 7 // 2, batch
    torch.manual_seed(0)
    rand = lambda *s, dt=bf: torch.randn(*s, dtype=dt, device=dev)
    bs = 128
    per = (context + prompt + bs) // bs + 1
    table = torch.arange(B * per, dtype=torch.int32, device=dev).view(per, B).t().contiguous()
    one, mix1 = torch.ones(1, device=dev), torch.ones(1, 1, device=dev)
    for phase, T in (("decode", batch), ("prefill", batch * prompt)):
        n_buf = 64 if phase == "decode" else max(2, min(8, int(400e6 / (T * width * 4))))
        cu = (torch.arange(B + 1, dtype=torch.int32) * (T // B)).to(dev)
        past = torch.full((B,), 0 if phase == "prefill" else context - 1, dtype=torch.int32, device=dev)
        # ---- residual and norm
        ys = [rand(T, width) for _ in range(n_buf)]
        xs = [rand(T, 1, width, dt=f32) for _ in range(n_buf)]
        gam = torch.ones(width, device=dev)
        row(f"residual + norm {phase}", "rovurax", graph_us([lambda x=x, y=y: K.hyper_norm(x, y, mix1, one, one, gam, 1e-6) for x, y in zip(xs, ys)]),
            T * width * 12)
        g16, rs = gam.to(bf), [x.view(T, width).to(bf) for x in xs]
        row(f"skip rms norm {phase}", "llama", graph_us([lambda x=x, y=y: K.norm(x, g16, skip=y, simplified=True, want_sum=True) for x, y in zip(rs, ys)]),
            T * width * 8)
        del xs, ys, rs
        # ---- step 1 of attention
        kc, vc = [rand(B * per, bs, kv, H) for _ in range(2)]
        pk = [rand(T, (N + 2 * kv) * H) for _ in range(n_buf)]
        first = rand(T, kv * H)
        us = graph_us([lambda x=x: K.qk_norm_rope(x, kc, vc, None, None, None, None, cu, past, table, N, H, H, keep_q=True, first_values=first, v_mix=one)
                       for x in pk])
        row(f"append with mixed values {phase}", "rovurax", us, T * kv * H * 10)
        cos, sin = torch.rand(per * bs, H // 2, device=dev).to(bf), torch.rand(per * bs, H // 2, device=dev).to(bf)
        us = graph_us([lambda x=x: K.paged_prep(x, kc, vc, cu, past, table, N, kv, cos, sin) for x in pk])
        row(f"paged_prep {phase}", "llama", us, T * (N + 2 * kv) * H * 4)
        del pk
        q = rand(T, N, H)
        if phase == "prefill":
            fl = lambda pairs, size: 2 * B * N * size * pairs * 1e-12
            calls = lambda split, chunk: [lambda: K.attn_prefill_paged(q, kc, vc, cu, past, table, split_weights=split, chunk=chunk)] * 8
            row(f"attention prefill, chunks of {CHUNK}", "rovurax", graph_us(calls(True, CHUNK)), tflop=fl(visible_keys(prompt, CHUNK), 2 * H))
            row("attention prefill, one chunk", "rovurax", graph_us(calls(True, 1 << 20)), tflop=fl(visible_keys(prompt, prompt), 2 * H))
            row("attention prefill", "llama", graph_us(calls(False, 0)), tflop=fl(visible_keys(prompt, prompt), 2 * H))
        else:
            caches = [(torch.randn_like(kc), torch.randn_like(vc)) for _ in range(max(2, int(300e6 / (kc.numel() * 4))))]
            for chunk in (CHUNK, 1 << 20):
                seen = (context - 1) % chunk + 1
                us = graph_us([lambda c=c: K.gqa_decode(q.view(B, N, H), c[0], c[1], past, block_table=table, split_weights=True, chunk=chunk) for c in caches] * 2)
                row(f"attention decode, {seen} keys", "rovurax", us, B * seen * kv * H * 4)
            us = graph_us([lambda c=c: K.gqa_decode(q.view(B, N, H), c[0], c[1], past, block_table=table, algo=2) for c in caches] * 2)
            row("attention decode", "llama", us, B * context * kv * H * 4)
            del caches
        del kc, vc, q
        # ---- latent attention
        cols = N * (H + ROT) + RANK + ROT + N
        pk = [rand(T, cols + -cols % 8) for _ in range(min(n_buf, 8))]
        n_cache = 2 if phase == "prefill" else max(2, int(300e6 / (B * per * bs * (RANK + ROT) * 2)))
        caches = [rand(B * per, bs, RANK + ROT) for _ in range(n_cache)]
        norm, sink = torch.ones(RANK, device=dev), torch.zeros(N, device=dev)
        cos, sin = torch.rand(per * bs, ROT // 2, device=dev), torch.rand(per * bs, ROT // 2, device=dev)
        ups = [rand(N * 2 * H, RANK) * RANK ** -0.5 for _ in range(2 if phase == "prefill" else max(2, int(300e6 / (N * 2 * H * RANK * 2))))]
        scale = (H + ROT) ** -0.5
        if phase == "decode":
            us = graph_us([lambda u=u: K.latent_absorb(pk[0], caches[0], norm, cos, sin, cu, past, table, u, N, H, ROT, RANK) for u in ups])
            row("latent absorb + append decode", "rovurax", us, N * H * RANK * 2 + T * (N * (H + ROT) + N * (RANK + ROT) + 2 * (RANK + ROT)) * 2)
            qa = K.latent_absorb(pk[0], caches[0], norm, cos, sin, cu, past, table, ups[0], N, H, ROT, RANK)
            us = graph_us([lambda c=c: K.latent_decode(qa, c, cu, past, table, RANK, scale) for c in caches] * 2)
            row("latent attention decode", "rovurax", us, B * context * (RANK + ROT) * 2 + T * N * ((RANK + ROT) * 2 + RANK * 4),
                tflop=2 * B * N * context * (2 * RANK + ROT) * 1e-12)
            o, ml = K.latent_decode(qa, caches[0], cu, past, table, RANK, scale)
            us = graph_us([lambda u=u: K.latent_out(o, ml, sink, u[N * H:], pk[0][:, cols - N:], pk[0].shape[1], H) for u in ups])
            row("latent values + gate decode", "rovurax", us, N * H * RANK * 2 + T * N * (RANK * 4 + H * 2))
        else:
            us = graph_us([lambda x=x: K.latent_prep(x, caches[0], norm, cos, sin, cu, past, table, N, H, ROT, RANK) for x in pk])
            row("latent prep prefill", "rovurax", us, T * (N * ROT * 4 + (RANK + ROT) * 6))
            q_rot, c, kr = K.latent_prep(pk[0], caches[0], norm, cos, sin, cu, past, table, N, H, ROT, RANK)
            us = graph_us([lambda u=u: K.gemm(c, u) for u in ups] * 3)
            row("latent expansion GEMM prefill", "rovurax", us, tflop=2 * T * N * 2 * H * RANK * 1e-12, bytes_=T * (RANK + N * 2 * H) * 2)
            kvx = K.gemm(c, ups[0])
            s16 = sink.to(bf)
            us = graph_us([lambda: K.latent_prefill(pk[0], q_rot, kvx, kr, s16, pk[0][:, cols - N:], cu, past, N, H, ROT, H, scale)] * 8)
            row("latent attention prefill", "rovurax", us, tflop=2 * B * N * (2 * H + ROT) * visible_keys(prompt, prompt) * 1e-12)
            del q_rot, c, kr, kvx
        del pk, caches, ups
        torch.cuda.empty_cache()
        # ---- feed-forward: the gated epilogue (decode) or the streaming unit (prompts); output projections
        if phase == "decode":
            h, wg = rand(T, width), [rand(2 * ff, width) for _ in range(max(2, int(300e6 / (4 * ff * width))))]
            wide = torch.empty(T, N * H + ff, dtype=bf, device=dev)
            us = graph_us([lambda w=w: K.gemm(h, w, act="clamped_swiglu", gate=(7.0, 1.702, 1.0), out=wide[:, N * H:], n=ff, dual_offset=ff) for w in wg] * 2)
            row("gate / up GEMM, clamped, into columns decode", "rovurax", us, 2 * ff * width * 2)
            us = graph_us([lambda w=w: K.gemm(h, w, act="swiglu") for w in wg] * 2)
            row("gate / up GEMM decode", "llama", us, 2 * ff * width * 2)
            del wg
            wo = [rand(width, N * H + ff) for _ in range(max(2, int(300e6 / (2 * width * (N * H + ff)))))]
            us = graph_us([lambda w=w: K.gemm(wide, w) for w in wo] * 2)
            row("output + down GEMM decode", "rovurax", us, width * (N * H + ff) * 2)
            wd, prod = [w[:, N * H:].contiguous() for w in wo], wide[:, N * H:].contiguous()
            us = graph_us([lambda w=w: K.gemm(prod, w) for w in wd] * 2)
            row("down GEMM decode", "llama", us, width * ff * 2)
            del wo, wd, wide
        else:
            gu = [rand(T, 2 * ff) for _ in range(2)]
            wide = torch.empty(T, N * H + ff, dtype=bf, device=dev)
            us = graph_us([lambda g=g: K.gated_unit(g[:, :ff], g[:, ff:], "clamped_swiglu", 7.0, 1.702, 1.0, out=wide[:, N * H:]) for g in gu] * 3)
            row("clamped gated unit prefill", "rovurax", us, T * ff * 6)
            us = graph_us([lambda g=g: K.swiglu(g) for g in gu] * 3)
            row("swiglu unit prefill", "llama", us, T * ff * 6)
            del gu, wide
        torch.cuda.empty_cache()
    return rows.rows


def run(sizes, batch: int = 8, prompt: int = 1024, steps: int = 64, warmup: int = 4) -> Dict:
    return run_pair("rovurax", configs, kernel_numbers, sizes, batch, prompt, steps, warmup)
