"""Fegilix decoder against the plain restatement in fegilix_oracle.py: every mechanism alone, then whole models through the
registry, the pooled caches and the generation drivers.  Each case runs on the CPU provider and (marked gpu) on the GPU."""
import io
import json
import sys

import pytest
import torch

import fegilix_oracle as oracle
import packed_decoder
import onnxruntime_b200 as ort
from onnxruntime_b200 import onnx_lite as ol
from packed_decoder import CPU, GPU, KINDS, ONNX, PROVIDERS, close, decoder, feed, i32, logits_close, run_op, tokens_of
from onnxruntime_b200.models.decoder_cache import CacheFull, CachePool, CacheTensor
from onnxruntime_b200.models.fegilix import FegilixConfig, random_weights, rotary_tables
from onnxruntime_b200.models.generation import GenerationConfig, generate, generate_requests
from onnxruntime_b200.models.registry import create_decoder, load_decoder
from onnxruntime_b200.safetensors_lite import load_file, save_file


def Reference(*args):
    return packed_decoder.Reference(oracle, *args)


def greedy_reference(*args):
    return packed_decoder.greedy_reference(oracle, *args)


# ---------------------------------------------------------------------------------------------------- one operator alone
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("streams,width", [(1, 40), (2, 64), (3, 30), (5, 136), (8, 16)])
def test_hyper_connections(kind, streams, width):
    provider, dt = kind
    g = torch.Generator().manual_seed(streams)
    rand = lambda *s: torch.randn(*s, generator=g)
    N, eps = 7, 3e-3
    x, y, gamma = rand(N, streams, width), rand(N, width).to(dt), rand(width)
    mix, w_out, w_in = rand(streams, streams), rand(streams), rand(streams)
    out, xo = run_op(provider, "HyperConnectionNorm", [x, y, mix, w_out, w_in, gamma],
                     [torch.zeros(N, width, dtype=dt), torch.zeros(N, streams, width)], streams=streams, epsilon=eps)
    ref = oracle.hyper_write(x.double(), mix.double(), w_out.double(), y.double())
    close(xo, ref, torch.float32)
    close(out, oracle.rms_norm(oracle.hyper_read(ref, w_in.double()), gamma.double(), eps), dt)
    # all streams equal to one row, nothing to write back; and the rows of a selection
    row = rand(N, width).to(dt)
    (out,) = run_op(provider, "HyperConnectionNorm", [row, None, None, None, w_in, gamma], [torch.zeros(N, width, dtype=dt)], streams=streams,
                    epsilon=eps)
    same = row.double()[:, None, :].expand(N, streams, width)
    close(out, oracle.rms_norm(oracle.hyper_read(same, w_in.double()), gamma.double(), eps), dt)
    rows = torch.tensor([6, 0, 6], dtype=torch.int64)
    (out,) = run_op(provider, "HyperConnectionNorm", [row, y, mix, w_out, w_in, gamma, rows], [torch.zeros(3, width, dtype=dt)], streams=streams,
                    epsilon=eps)
    ref = oracle.hyper_write(same, mix.double(), w_out.double(), y.double())
    close(out, oracle.rms_norm(oracle.hyper_read(ref, w_in.double()), gamma.double(), eps)[rows], dt)


@pytest.mark.parametrize("kind", KINDS)
def test_gated_feed_forward_and_soft_cap(kind):
    provider, dt = kind
    g = torch.Generator().manual_seed(0)
    x = (4 * torch.randn(5, 33, generator=g)).to(dt)
    (y,) = run_op(provider, "SoftCap", [x], [torch.zeros(5, 33)], cap=2.5)
    close(y, 2.5 * torch.tanh(x.double() / 2.5), torch.float32)
    for tokens in (3, 80, 200):            # the three GEMM shapes of the gated epilogue
        h, wg, wu = [torch.randn(*s, generator=g).mul(0.3).to(dt) for s in ((tokens, 48), (72, 48), (72, 48))]
        dev = "cuda" if provider == GPU else "cpu"
        inits = [ol.make_external_tensor(n, ONNX[dt], (48, 72)) for n in ("wg", "wu")]
        nodes = [ol.make_node("MatMul", ["h", "wg"], ["a"]), ol.make_node("MatMul", ["h", "wu"], ["b"]),
                 ol.make_node("FastGelu", ["a"], ["c"], domain="com.microsoft"), ol.make_node("Mul", ["c", "b"], ["o"])]
        graph = ol.make_graph(nodes, "g", [ol.make_tensor_value_info("h", ONNX[dt], ["n", 48])], [ol.make_tensor_value_info("o", ONNX[dt], ["n", 72])], inits)
        so = ort.SessionOptions()
        so.add_external_initializers(["wg", "wu"], [wg.t().contiguous().to(dev), wu.t().contiguous().to(dev)])
        sess = ort.InferenceSession(ol.make_model(graph, opset=17).serialize(), so, providers=[provider])
        if dt == torch.bfloat16:
            assert [n["op_type"] for n in sess.graph_nodes()] == ["GemmSwiGLU"]
        out = torch.zeros(tokens, 72, dtype=dt, device=dev)
        b = sess.io_binding()
        b.bind_torch_input("h", h.to(dev))
        b.bind_torch_output("o", out)
        sess.run_with_iobinding(b)
        h, wg, wu = h.double(), wg.double(), wu.double()
        close(out.cpu(), oracle.gelu_tanh(h @ wg.T) * (h @ wu.T), dt)


class DeltaCase:
    def __init__(self, lengths, H, G, dk, dv, taps, dt, seed=0, decay_bias=-1.0):
        g = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=g)
        self.__dict__.update(locals())
        n, C = sum(lengths), 2 * G * dk + H * dv
        self.C = C
        pad = 3                                             # columns behind the projections are ignored
        self.x = rand(n, C + H + pad).to(dt)
        self.low = rand(n, H * (dk + dv)).to(dt)
        self.conv = rand(C, taps) / taps ** 0.5
        self.a_log, self.dt_bias, self.norm = 0.5 * rand(H), rand(H * dk) + decay_bias, 1 + 0.2 * rand(dv)

    def reference(self):
        H, G, dk, dv, C = self.H, self.G, self.dk, self.dv, self.C
        out, t0 = [], 0
        for n in self.lengths:
            x, low = self.x[t0:t0 + n].double(), self.low[t0:t0 + n].double()
            y = oracle.causal_conv_silu(x[:, :C], self.conv.double())
            q, k = y[:, :G * dk].reshape(n, G, dk), y[:, G * dk:2 * G * dk].reshape(n, G, dk)
            q, k = [t.repeat_interleave(H // G, 1) for t in (oracle.unit(q) * dk ** -0.5, oracle.unit(k))]
            z = low[:, :H * dk] + self.dt_bias.double()
            decay = torch.exp(-torch.exp(self.a_log.double())[None, :, None] * torch.log1p(torch.exp(z)).reshape(n, H, dk))
            o = oracle.gated_delta_scan(q, k, y[:, 2 * G * dk:].reshape(n, H, dv), torch.sigmoid(x[:, C:C + H]), decay)
            o = oracle.rms_norm(o, self.norm.double(), 1e-3) * torch.sigmoid(low[:, H * dk:]).reshape(n, H, dv)
            out.append(o.reshape(n, H * dv))
            t0 += n
        return torch.cat(out)

    def run(self, provider, cuts):
        """``cuts``: per call, how many tokens every sequence brings.  State lives in scattered slots filled with rubbish."""
        B, H, dk, dv = len(self.lengths), self.H, self.dk, self.dv
        slots = i32(*[2 * b + 1 for b in range(B)])
        ring = torch.full((2 * B + 1, self.taps, self.C), 7.0, dtype=self.dt)
        state = torch.full((2 * B + 1, H, dk, dv), 7.0)
        starts = [sum(self.lengths[:b]) for b in range(B)]
        past, out = [0] * B, [[] for _ in range(B)]
        for cut in cuts:
            idx = torch.cat([torch.arange(starts[b] + past[b], starts[b] + past[b] + cut[b]) for b in range(B)])
            cu = i32(0, *torch.tensor(cut).cumsum(0).tolist())
            y, _, _ = run_op(provider, "PackedGatedDelta",
                             [self.x[idx], self.low[idx], self.conv, self.a_log, self.dt_bias, self.norm, ring, state, cu, i32(*past), slots],
                             [torch.zeros(len(idx), H * dv, dtype=self.dt), ring, state], num_heads=H, kv_num_heads=self.G, head_size=dk,
                             v_head_size=dv, epsilon=1e-3, unit_epsilon=1e-6)
            at = 0
            for b in range(B):
                out[b].append(y[at:at + cut[b]])
                at += cut[b]
                past[b] += cut[b]
        assert past == list(self.lengths)
        assert (state[0] == 7).all() and (ring[0] == 7).all()      # slots of nobody stay as they are
        return torch.cat([torch.cat(o) for o in out])


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,G,dk,dv,taps", [(2, 2, 16, 16, 4), (4, 2, 40, 24, 3), (3, 1, 72, 130, 2), (1, 1, 8, 6, 1), (2, 1, 136, 20, 5)])
def test_gated_delta_rule(kind, H, G, dk, dv, taps):
    provider, dt = kind
    case = DeltaCase([9, 1, 20], H, G, dk, dv, taps, dt)
    ref = case.reference()
    tol = 2e-4 if dt == torch.float32 else 3e-2
    close(case.run(provider, [[9, 1, 20]]), ref, dt, tol)
    # portions, down to two tokens and to one token of each sequence
    case = DeltaCase([21, 8, 40], H, G, dk, dv, taps, dt, seed=1)
    ref = case.reference()
    close(case.run(provider, [[2, 2, 17], [1, 1, 1], [1, 1, 1], [2, 3, 17], [15, 1, 4]]), ref, dt, tol)


@pytest.mark.parametrize("kind", KINDS)
def test_gated_delta_rule_remembers_and_forgets(kind):
    """Slow decay: the first token still shows hundreds of tokens later, in prompts and in decoding.  Fast decay: it does not."""
    provider, dt = kind
    n = 260
    for bias, kept in ((-12.0, True), (3.0, False)):
        case = DeltaCase([n], 1, 1, 16, 8, 2, dt, seed=3, decay_bias=bias)
        case.x[1:n - 2, :32] = 0.001 * torch.randn(n - 3, 32).to(dt)      # unit keys of the middle tokens: noise
        case.x[1:n - 2, case.C:case.C + 1] = -30                          # and beta = 0: they write nothing
        case.x[n - 2:, :32] = case.x[:1, :32]                             # the last tokens ask for the first one
        ref = case.reference()
        tol = 2e-4 if dt == torch.float32 else 3e-2
        close(case.run(provider, [[n]]), ref, dt, tol)
        close(case.run(provider, [[n - 4], [1], [1], [2]]), ref, dt, tol)
        other = DeltaCase([n], 1, 1, 16, 8, 2, dt, seed=3, decay_bias=bias)
        other.x = case.x.clone()
        other.x[0, 32:] = -case.x[0, 32:]                                 # another value at the first token
        moved = (other.reference()[-1] - ref[-1]).abs().max() / ref[-1].abs().max()
        assert (moved > 0.1) == kept


class MLstmCase:
    def __init__(self, lengths, H, dk, dv, dt, seed=0, cap=9.0, f_bias=2.0, spread=1.0):
        g = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=g)
        self.__dict__.update(locals())
        n = sum(lengths)
        self.x = rand(n, H * (2 * dk + 2 * dv + 2) + 5).to(dt)
        self.x[:, H * (2 * dk + 2 * dv):] *= spread
        self.ib, self.fb, self.norm = rand(H), rand(H) + f_bias, 1 + 0.2 * rand(H * dv)

    def reference(self, floor=True):
        H, dk, dv, cap = self.H, self.dk, self.dv, self.cap
        out, t0 = [], 0
        for n in self.lengths:
            x = self.x[t0:t0 + n].double()
            q, k = x[:, :H * dk].reshape(n, H, dk) * dk ** -0.5, x[:, H * dk:2 * H * dk].reshape(n, H, dk)
            v, g = x[:, 2 * H * dk:H * (2 * dk + dv)].reshape(n, H, dv), x[:, H * (2 * dk + dv):H * (2 * dk + 2 * dv)]
            i, f = x[:, H * (2 * dk + 2 * dv):][:, :H], x[:, H * (2 * dk + 2 * dv):][:, H:2 * H]
            i = cap * torch.tanh((i + self.ib.double()) / cap)
            f = -torch.log1p(torch.exp(-cap * torch.tanh((f + self.fb.double()) / cap)))
            o = oracle.rms(oracle.mlstm_scan(q, k, v, i, f, floor), 1e-3).reshape(n, H * dv)
            out.append(o * self.norm.double() * torch.sigmoid(g))
            t0 += n
        return torch.cat(out)

    def run(self, provider, cuts):
        B, H, dk, dv = len(self.lengths), self.H, self.dk, self.dv
        slots = i32(*[2 * (B - b) for b in range(B)])
        state, aux = torch.full((2 * B + 1, H, dk, dv), 7.0), torch.full((2 * B + 1, H, dk + 1), 7.0)
        starts = [sum(self.lengths[:b]) for b in range(B)]
        past, out = [0] * B, [[] for _ in range(B)]
        for cut in cuts:
            idx = torch.cat([torch.arange(starts[b] + past[b], starts[b] + past[b] + cut[b]) for b in range(B)])
            cu = i32(0, *torch.tensor(cut).cumsum(0).tolist())
            y, _, _ = run_op(provider, "PackedMLstm", [self.x[idx], self.ib, self.fb, self.norm, state, aux, cu, i32(*past), slots],
                             [torch.zeros(len(idx), H * dv, dtype=self.dt), state, aux], num_heads=H, head_size=dk, v_head_size=dv,
                             gate_cap=self.cap, epsilon=1e-3, denominator_epsilon=1e-6)
            at = 0
            for b in range(B):
                out[b].append(y[at:at + cut[b]])
                at += cut[b]
                past[b] += cut[b]
        assert past == list(self.lengths) and (state[1] == 7).all() and (aux[1] == 7).all()
        return torch.cat([torch.cat(o) for o in out])


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,dk,dv", [(2, 16, 16), (3, 40, 26), (1, 72, 132), (2, 8, 5), (1, 140, 16)])
def test_mlstm(kind, H, dk, dv):
    provider, dt = kind
    tol = 2e-4 if dt == torch.float32 else 3e-2
    for spread in (1.0, 6.0):        # wide gates move the running maximum and reach the cap
        case = MLstmCase([9, 1, 20], H, dk, dv, dt, spread=spread)
        close(case.run(provider, [[9, 1, 20]]), case.reference(), dt, tol)
        case = MLstmCase([21, 8, 40], H, dk, dv, dt, seed=1, spread=spread)
        close(case.run(provider, [[2, 2, 17], [1, 1, 1], [1, 1, 1], [2, 3, 17], [15, 1, 4]]), case.reference(), dt, tol)


@pytest.mark.parametrize("kind", KINDS)
def test_mlstm_denominator_floor(kind):
    """All input gates strongly negative: the floor of the denominator decides, and outputs are small before their norm (whose
    eps makes that visible)."""
    provider, dt = kind
    case = MLstmCase([6], 2, 16, 8, dt, f_bias=30.0)
    case.x[:, 2 * (2 * 16 + 2 * 8):] = 0
    case.ib -= 5
    tol = 2e-4 if dt == torch.float32 else 3e-2
    ref = case.reference()
    close(case.run(provider, [[6]]), ref, dt, tol)
    close(case.run(provider, [[3], [1], [1], [1]]), ref, dt, tol)
    wrong = case.reference(floor=False)
    assert (wrong - ref).abs().max() > 0.3 * ref.abs().max()


class AttentionCase:
    def __init__(self, lengths, N, Nk, dk, dv, rot, dt, block, seed=0, sink=0.0, scale=None):
        g = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=g)
        self.__dict__.update(locals())
        n = sum(lengths)
        self.scale = scale if scale is not None else dk ** -0.5
        self.x = rand(n, N * dk + Nk * (dk + dv) + N * dv + 1).to(dt)
        self.qn, self.kn, self.sink = 1 + 0.2 * rand(dk), 1 + 0.2 * rand(dk), (2 * rand(N) + sink).to(dt).float()

    def heads(self, x):
        n, N, Nk, dk, dv = x.shape[0], self.N, self.Nk, self.dk, self.dv
        q, k, v, g = x[:, :-1].split([N * dk, Nk * dk, Nk * dv, N * dv], 1)
        return q.reshape(n, N, dk), k.reshape(n, Nk, dk), v.reshape(n, Nk, dv), g

    def reference(self, shared_queries=None):
        out, t0 = [], 0
        for n in self.lengths:
            x = self.x[t0:t0 + n].double()
            q, k, v, g = self.heads(x)
            pos = torch.arange(n)
            turn = (lambda t: oracle.rotate(t, pos, self.rot)) if self.rot else (lambda t: t)
            k = turn(oracle.rms_norm(k, self.kn.double(), 1e-3))
            if shared_queries is not None:
                y = shared_queries[t0:t0 + n].double()
                q, g = y[:, :self.N * self.dk].reshape(n, self.N, self.dk), y[:, self.N * self.dk:]
            q = turn(oracle.rms_norm(q, self.qn.double(), 1e-3))
            o = oracle.causal_attention(q, k, v, self.scale, self.sink.double()).reshape(n, -1)
            out.append(o * torch.sigmoid(g))
            t0 += n
        return torch.cat(out)

    def run(self, provider, cuts, shared_queries=None):
        B, N, Nk, dk, dv, block = len(self.lengths), self.N, self.Nk, self.dk, self.dv, self.block
        cfg = FegilixConfig(8, 8, [], dtype="bf16" if self.dt == torch.bfloat16 else "fp32")
        kw, vw = cfg.cache_widths({"dim": dk, "vdim": dv})
        per = max(-(-n // block) for n in self.lengths)
        kc, vc = [torch.full((B * per + 1, block, Nk, w), 3.0, dtype=self.dt) for w in (kw, vw)]
        order = torch.randperm(B * per, generator=torch.Generator().manual_seed(5)).to(torch.int32) + 1     # block 0 belongs to nobody
        table = order.reshape(B, per)
        cos, sin = rotary_tables(self.rot, per * block) if self.rot else (None, None)
        starts = [sum(self.lengths[:b]) for b in range(B)]
        past, out = [0] * B, [[] for _ in range(B)]
        attrs = dict(num_heads=N, kv_num_heads=Nk, head_size=dk, v_head_size=dv, scale=self.scale, epsilon=1e-3, gated=1)
        for cut in cuts:
            idx = torch.cat([torch.arange(starts[b] + past[b], starts[b] + past[b] + cut[b]) for b in range(B)])
            cu, pt = i32(0, *torch.tensor(cut).cumsum(0).tolist()), i32(*past)
            tail = [cu, pt, table, cos, sin, self.qn, self.kn, self.sink]
            y, _, _ = run_op(provider, "GatedPagedAttention", [self.x[idx], kc, vc] + tail, [torch.zeros(len(idx), N * dv, dtype=self.dt), kc, vc],
                             kv_shared=0, **attrs)
            if shared_queries is not None:      # another layer reads the same keys
                tail[6] = None
                (y,) = run_op(provider, "GatedPagedAttention", [shared_queries[idx], kc, vc] + tail,
                              [torch.zeros(len(idx), N * dv, dtype=self.dt)], kv_shared=1, **attrs)
            at = 0
            for b in range(B):
                out[b].append(y[at:at + cut[b]])
                at += cut[b]
                past[b] += cut[b]
        assert past == list(self.lengths) and (kc[0] == 3).all() and (vc[0] == 3).all()
        return torch.cat([torch.cat(o) for o in out])


SCALING = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("N,Nk,dk,dv,rot,block", [
    (2, 2, 16, 16, {"base": 100.0, "dims": 16}, 4), (4, 2, 40, 24, {"base": 1000.0, "dims": 20, "scaling": SCALING}, 16),
    (6, 2, 64, 64, {"base": 500.0, "dims": 64}, 128), (3, 1, 80, 128, {"base": 500.0, "dims": 2}, 128), (2, 1, 144, 20, {"base": 500.0, "dims": 144}, 8),
    (2, 2, 24, 136, None, 128)])
def test_gated_paged_attention(kind, N, Nk, dk, dv, rot, block):
    provider, dt = kind
    tol = 5e-5 if dt == torch.float32 else 2e-2
    case = AttentionCase([19, 1, 45], N, Nk, dk, dv, rot, dt, block)
    close(case.run(provider, [[19, 1, 45]]), case.reference(), dt, tol)
    close(case.run(provider, [[2, 1, 2], [15, 0, 15], [1, 0, 27], [1, 0, 1]]), case.reference(), dt, tol)
    case = AttentionCase([7, 5], N, Nk, dk, dv, rot, dt, block, seed=2, sink=4.0)
    close(case.run(provider, [[3, 1], [1, 1], [1, 1], [1, 1], [1, 1]]), case.reference(), dt, tol)
    queries = torch.randn(12, N * (dk + dv), generator=torch.Generator().manual_seed(9)).to(dt)
    close(case.run(provider, [[3, 1], [2, 2], [1, 1], [1, 1]], queries), case.reference(queries), dt, tol)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("block,dk", [(128, 64), (128, 96), (16, 48)])
def test_one_far_key_stands_out(kind, block, dk):
    """One key scores far above the rest: its value must come through whether it is the first token, sits at either side of a
    block border, or is the token itself - in prompts, across a portion's start, and in decoding."""
    provider, dt = kind
    n = 2 * block + 37
    asked = [0, 1, block - 1, block, block + 1, 2 * block - 1, 2 * block]
    case = AttentionCase([n], 1, 1, dk, dk, None, dt, block, seed=4, scale=0.6)
    q, k = case.x[:, :dk], case.x[:, dk:2 * dk]
    for j, key in enumerate(asked):
        pattern = torch.randn(dk, generator=torch.Generator().manual_seed(100 + j)).to(dt)
        k[key] = pattern
        q[n - len(asked) + j] = pattern
    case.qn, case.kn = torch.ones(dk), torch.ones(dk)
    ref = case.reference()
    tol = 5e-5 if dt == torch.float32 else 2e-2
    close(case.run(provider, [[n]]), ref, dt, tol)
    m = n - len(asked)
    close(case.run(provider, [[m]] + [[1]] * len(asked)), ref, dt, tol)
    close(case.run(provider, [[block], [2], [m - block - 2], [2], [len(asked) - 2]]), ref, dt, tol)
    # the case discriminates: without the asked key, the output at the asking token is another one
    weak = AttentionCase([n], 1, 1, dk, dk, None, dt, block, seed=4, scale=0.6)
    weak.x, weak.qn, weak.kn = case.x.clone(), case.qn, case.kn
    weak.x[block, dk:2 * dk] *= -1
    at = n - len(asked) + 3
    assert (weak.reference()[at] - ref[at]).abs().max() > 0.2 * ref[at].abs().max()


# -------------------------------------------------------------------------------------------------------- whole models
def small_config(name):
    att = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 24, "scale": 0.2, "rot": {"base": 300.0, "dims": 16, "scaling": dict(SCALING)}}
    delta = {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 20, "conv": 3}
    mem = {"heads": 3, "dim": 16, "vdim": 28, "gate_cap": 7.0}
    ff = lambda n: {"kind": "dense", "ff": n}
    layers = {
        "mixed": [("channel_delta", delta, None), ("attention", att, ff(56)), ("mlstm", mem, ff(40)), ("attention", dict(att, kv_from=1), None),
                  ("channel_delta", dict(delta, heads=2, kv_heads=2, conv=1), ff(64))],
        "attention": [("attention", dict(att, heads=2, kv_heads=2, dim=20, vdim=20, rot={"base": 50.0, "dims": 20}), None),
                      ("attention", dict(att, heads=6, kv_heads=1, dim=16, vdim=48, scale=1.0, rot={"base": 50.0, "dims": 4}), ff(24)),
                      ("attention", dict(att, heads=4, kv_heads=1, dim=16, vdim=48, scale=0.3, rot={"base": 50.0, "dims": 4}, kv_from=1), ff(24))],
        "recurrent": [("mlstm", mem, None), ("mlstm", dict(mem, heads=1, dim=8, vdim=8, gate_cap=2.0), ff(16)), ("channel_delta", delta, None)],
        # sizes that no tensor-core or vector path takes
        "odd": [("attention", dict(att, heads=3, kv_heads=1, dim=10, vdim=14, rot={"base": 30.0, "dims": 6}), ff(20)),
                ("channel_delta", dict(delta, heads=3, kv_heads=1, dim=9, vdim=7, conv=4), None), ("mlstm", dict(mem, heads=5, dim=11, vdim=6), ff(12))],
        "plain": [("attention", att, ff(24)), ("mlstm", mem, None), ("channel_delta", delta, ff(32))],
    }[name]
    cfg = {"architecture": "Fegilix", "vocab": 97 if name != "attention" else 120, "width": {"recurrent": 40, "odd": 36}.get(name, 48), "norm": {"eps": 1e-5},
           "layers": [{"type": t, "mixer": dict(m), "mlp": f} for t, m, f in layers]}
    if name != "plain":
        cfg.update(streams={"mixed": 3, "attention": 2, "recurrent": 1, "odd": 5}[name], logit_softcap=8.0)
    return cfg


def model_pair(name, seed=0):
    cfg = small_config(name)
    return cfg, random_weights(FegilixConfig.from_json(cfg), seed=seed, low_rank=6, gain=1.5)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", ["mixed", "attention", "recurrent", "plain", "odd"])
def test_model_matches_the_restatement(kind, name):
    """Whole prompt, portions down to two tokens, token by token, and a prompt followed by decoding."""
    cfg, w = model_pair(name)
    toks = tokens_of(cfg, 41, 1)
    ref = Reference(cfg, w, toks)
    runner = decoder(cfg, w, kind)
    for cuts in ([41], [2, 2, 15, 3, 2, 17], [1] * 41, [33] + [1] * 8, [16, 16, 9]):
        logits_close(feed(runner, "s", toks, cuts), ref, kind[1])
        runner.release("s")
    for n in (1, 2, 3):         # the shortest sequences
        logits_close(feed(runner, "s", toks[:n], [n]), ref[:n], kind[1])
        runner.release("s")


@pytest.mark.parametrize("kind", KINDS)
def test_residual_sums_reach_the_logits_in_every_layer_order(kind):
    """Layer order comes from the configuration: the same layers reversed are another model, and it matches too."""
    cfg, _ = model_pair("recurrent")
    cfg["layers"] = cfg["layers"][::-1]
    w = random_weights(FegilixConfig.from_json(cfg), seed=5, low_rank=6, gain=1.5)
    toks = tokens_of(cfg, 12, 3)
    logits_close(feed(decoder(cfg, w, kind), 0, toks, [5, 7]), Reference(cfg, w, toks), kind[1])


@pytest.mark.parametrize("kind", KINDS)
def test_unequal_requests_in_one_batch_equal_each_alone(kind):
    cfg, w = model_pair("mixed", seed=2)
    texts = {s: tokens_of(cfg, n, 10 + n) for s, n in (("a", 37), ("b", 5), ("c", 1), ("d", 22))}
    runner = decoder(cfg, w, kind)
    refs = {s: Reference(cfg, w, t) for s, t in texts.items()}
    got = {s: [] for s in texts}

    def step(portions):
        rows = runner.step([(s, texts[s][a:b], list(range(b - a))) for s, a, b in portions])
        at = 0
        for s, a, b in portions:
            got[s].append(rows[at:at + b - a])
            at += b - a
    step([("a", 0, 30), ("b", 0, 3), ("c", 0, 1), ("d", 0, 18)])
    runner.release("c")
    step([("d", 18, 19), ("a", 30, 31), ("b", 3, 4)])          # one token each, another order
    step([("b", 4, 5), ("a", 31, 36), ("d", 19, 22)])          # decoding and portions of prompts in one batch
    runner.release("b")
    runner.release("d")
    step([("a", 36, 37)])
    for s in texts:
        logits_close(torch.cat(got[s]), refs[s], kind[1])


@pytest.mark.parametrize("kind", KINDS)
def test_blocks_and_slots_are_reused(kind):
    """Many requests through a pool that holds few: every one finds blocks and slots that others have left full."""
    cfg, w = model_pair("mixed", seed=3)
    block = 16 if kind[0] == CPU else 128
    n = block + 9
    runner = decoder(cfg, w, kind, batch=2, max_len=2 * block, block_size=block)
    texts = [tokens_of(cfg, n if i % 2 else 7 + i, 50 + i) for i in range(6)]
    refs = [Reference(cfg, w, t) for t in texts]
    seen = set()
    for i in range(0, 6, 2):
        pair = [i + 1, i] if i == 2 else [i, i + 1]
        rows = runner.step([(j, texts[j][:-2], [len(texts[j]) - 3]) for j in pair])
        for k, j in enumerate(pair):
            logits_close(rows[k:k + 1], refs[j][-3:-2], kind[1])
        for back in (2, 1):
            rows = runner.step([(j, texts[j][-back:][:1], [0]) for j in pair])
            for k, j in enumerate(pair):
                logits_close(rows[k:k + 1], refs[j][len(texts[j]) - back:][:1], kind[1])
        for j in pair:
            entry = runner.pool.sequences[j]
            seen.add((entry.slot, tuple(entry.blocks)))
            runner.release(j)
    assert len({s for s, _ in seen}) == 2 and len(runner.pool.free_blocks) == 4 and len(runner.pool.free_slots) == 2


@pytest.mark.parametrize("kind", KINDS)
def test_decode_graphs_of_several_batch_sizes(kind):
    """Batch sizes come and go (each has its own captured step); state advances exactly once per step, the step that captures
    the graph included."""
    cfg, w = model_pair("mixed", seed=4)
    runner = decoder(cfg, w, kind, batch=9, max_len=64, block_size=16 if kind[0] == CPU else 128)
    texts = [tokens_of(cfg, 14, 200 + i) for i in range(9)]
    refs = [Reference(cfg, w, t) for t in texts]
    runner.step([(i, t[:2], []) for i, t in enumerate(texts)])
    at = [2] * 9
    for batch in (range(9), [4], range(9), [1, 7], [4], range(9), [7, 1], [4], [0, 2, 3, 5, 6, 8]):
        batch = list(batch)
        rows = runner.step([(i, [texts[i][at[i]]], [0]) for i in batch])
        for k, i in enumerate(batch):
            logits_close(rows[k:k + 1], refs[i][at[i]:at[i] + 1], kind[1])
            at[i] += 1


@pytest.mark.parametrize("kind", KINDS)
def test_long_decoding(kind):
    cfg, w = model_pair("mixed", seed=6)
    n = 300 if kind[0] == GPU else 70
    toks = tokens_of(cfg, n, 7)
    runner = decoder(cfg, w, kind, batch=1, max_len=n)
    logits_close(feed(runner, 0, toks, [3] + [1] * (n - 3)), Reference(cfg, w, toks), kind[1])


def test_capacity_errors_leave_the_pool_usable():
    cfg, w = model_pair("mixed")
    runner = decoder(cfg, w, (CPU, torch.float32), batch=2, max_len=32, block_size=16)
    toks = tokens_of(cfg, 40, 1)
    with pytest.raises(CacheFull):
        runner.step([("x", toks, [])])                       # longer than max_len
    assert not runner.pool.sequences and len(runner.pool.free_slots) == 2
    runner.step([("a", toks[:3], []), ("b", toks[:30], [])])
    with pytest.raises(CacheFull):
        runner.step([("c", toks[:1], [0])])                  # no slot
    with pytest.raises(ValueError):
        runner.step([("a", toks[:1], [1])])                  # a wanted place outside the tokens
    runner.release("b")
    assert runner.step([("c", toks[:1], [0])]).shape == (1, cfg["vocab"])
    assert runner.step([("c", toks[1:3], [])]).shape == (0, cfg["vocab"])


@pytest.mark.parametrize("provider", PROVIDERS)
def test_greedy_generation(provider, tmp_path, capsys):
    """The runner's own loop, ``generate``, ``generate_requests`` (more requests than fit at a time) and the command line."""
    cfg, w = model_pair("mixed", seed=8)
    kind = (provider, torch.float32)
    prompts = [tokens_of(cfg, n, 30 + n) for n in (9, 4, 13)]
    want = [greedy_reference(cfg, w, p, 6) for p in prompts]
    runner = decoder(cfg, w, kind, batch=3, max_len=64)
    assert runner.generate(prompts, 6).tolist() == want                     # unequal prompts, packed
    runner = decoder(cfg, w, kind, batch=2, max_len=64)
    assert generate_requests(runner, prompts, GenerationConfig(max_new_tokens=6)) == want
    assert not runner.pool.sequences
    eos = want[0][2]
    cut = [t[:t.index(eos) + 1] if eos in t else t for t in want]
    assert generate_requests(runner, prompts, GenerationConfig(max_new_tokens=6, eos_token_id=eos)) == cut
    a = generate_requests(runner, prompts, GenerationConfig(max_new_tokens=5, top_k=4, seed=3))
    assert a == generate_requests(runner, prompts, GenerationConfig(max_new_tokens=5, top_k=4, seed=3))
    block = torch.tensor([prompts[0], prompts[0][::-1]])
    out = generate(runner, block, GenerationConfig(max_new_tokens=5))
    assert out[:, 9:].tolist() == [greedy_reference(cfg, w, row, 5) for row in block.tolist()]
    beams = generate(runner, block[:1], GenerationConfig(max_new_tokens=4, num_beams=2, length_penalty=0.0))
    assert beams.shape == (1, 13)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    from onnxruntime_b200.tools import generate as cli
    args = ["--model", str(tmp_path), "--dtype", "float32", "--provider", "cuda" if provider == GPU else "cpu", "--max-new-tokens", "6"]
    for p in prompts:
        args += ["--prompt-ids", ",".join(map(str, p))]
    assert cli.main(args) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.splitlines() if x.startswith("{")]
    assert [x["generated"] for x in lines] == want


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(dtype, tmp_path, monkeypatch, capsys):
    from onnxruntime_b200.tools import trace_replay
    cfg, w = model_pair("mixed", seed=9)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    a, b = tokens_of(cfg, 20, 1), tokens_of(cfg, 8, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [17, 0]}, {"id": "b", "tokens": b[:7], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[18:19], "want": []}, {"id": "b", "tokens": b[7:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:], "want": [0]}], "end": ["a"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace_replay.main(["--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "40"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "1.f32").exists()
    ref = Reference(cfg, w, a)
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).reshape(-1, cfg["vocab"])
    logits_close(read(0), ref[[17, 0]], dt)
    logits_close(read(2), ref[[19]], dt)


# ------------------------------------------------------------------------------------- configuration, weights, registry
def test_configuration_is_checked():
    cfg = small_config("mixed")
    assert FegilixConfig.from_json(FegilixConfig.from_json(cfg).to_json()).layers == cfg["layers"]
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][1]["mlp"].update(kind="other"),
                   lambda c: c["layers"][3]["mixer"].update(kv_from=2), lambda c: c["layers"][3]["mixer"].update(vdim=16),
                   lambda c: c["layers"][1]["mixer"].update(heads=3)):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            FegilixConfig.from_json(bad)
    with pytest.raises(ValueError, match="unknown architecture"):
        create_decoder({"architecture": "Nothing"}, {}, "float32", provider=CPU)
    _, w = model_pair("mixed")
    short = dict(w)
    del short["l0.mix.a1"]
    with pytest.raises(KeyError, match="l0.mix.a1"):
        decoder(cfg, short, (CPU, torch.float32))
    wrong = dict(w, head=w["head"][:-1])
    with pytest.raises(ValueError, match="head"):
        decoder(cfg, wrong, (CPU, torch.float32))


def test_rotary_bands():
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 256}}
    cos, sin = rotary_tables(rot, 50)
    f = oracle.rotary_frequencies(rot)
    plain = oracle.rotary_frequencies({"base": 10000.0, "dims": 32})
    assert (f == plain).any() and (f == plain / 4).any() and ((f < plain) & (f > plain / 4)).any()      # all three bands occur
    a = torch.arange(50, dtype=torch.float64)[:, None] * f
    assert torch.allclose(cos.double(), a.cos(), atol=1e-6) and torch.allclose(sin.double(), a.sin(), atol=1e-6)


def test_safetensors_round_trip(tmp_path):
    tensors = {"a": torch.randn(3, 5).to(torch.bfloat16), "b.c": torch.arange(7, dtype=torch.int32), "e": torch.zeros(0, 4), "s": torch.tensor(2.5)}
    path = str(tmp_path / "x.safetensors")
    save_file(tensors, path)
    back = load_file(path)
    assert set(back) == set(tensors) and all(torch.equal(back[k], tensors[k]) and back[k].dtype == tensors[k].dtype for k in tensors)
    data = open(path, "rb").read()
    open(path, "wb").write(data[:-3])
    with pytest.raises(ValueError):
        load_file(path)


def test_cache_pool_accounting():
    pool = CachePool([CacheTensor("k", "k_out", "paged", (2,), torch.float32), CacheTensor("s", "s_out", "slot", (3,), torch.float32)], 4, 8, 2,
                     torch.device("cpu"))
    assert pool.tensors["k"].shape == (4, 8, 2) and pool.tensors["s"].shape == (2, 3)
    pool.open("a")
    assert pool.reserve("a", 8) and not pool.reserve("a", 8)
    pool.advance("a", 8)
    assert pool.reserve("a", 1) and len(pool.sequences["a"].blocks) == 2
    pool.open("b")
    with pytest.raises(CacheFull):
        pool.reserve("b", 17)
    assert pool.sequences["b"].blocks == []                 # all or nothing
    with pytest.raises(CacheFull):
        pool.open("c")
    first = list(pool.sequences["a"].blocks)
    pool.close("a")
    pool.open("c")
    pool.reserve("c", 9)
    assert pool.sequences["c"].blocks == first              # freed blocks go out first


@pytest.mark.parametrize("provider", PROVIDERS)
def test_llama_checkpoint_through_the_registry(provider, tmp_path):
    """The registry's other family: a Llama folder generates the same tokens in the packed form as in the contiguous-cache form."""
    from onnxruntime_b200.models.generation import DecoderRunner
    from onnxruntime_b200.models.llama import LlamaConfig, build_llama
    hf = {"architectures": ["LlamaForCausalLM"], "vocab_size": 64, "hidden_size": 32, "num_hidden_layers": 2, "num_attention_heads": 4,
          "num_key_value_heads": 2, "intermediate_size": 48, "rope_theta": 1000.0, "rms_norm_eps": 1e-5}
    g = torch.Generator().manual_seed(0)
    rand = lambda *s: 0.3 * torch.randn(*s, generator=g)
    state = {"model.embed_tokens.weight": rand(64, 32), "model.norm.weight": torch.ones(32), "lm_head.weight": rand(64, 32)}
    for i in range(2):
        p = f"model.layers.{i}."
        state.update({p + "input_layernorm.weight": torch.ones(32), p + "post_attention_layernorm.weight": 1 + rand(32),
                      p + "self_attn.q_proj.weight": rand(32, 32), p + "self_attn.k_proj.weight": rand(16, 32), p + "self_attn.v_proj.weight": rand(16, 32),
                      p + "self_attn.o_proj.weight": rand(32, 32), p + "mlp.gate_proj.weight": rand(48, 32), p + "mlp.up_proj.weight": rand(48, 32),
                      p + "mlp.down_proj.weight": rand(32, 48)})
    (tmp_path / "config.json").write_text(json.dumps(hf))
    save_file(state, str(tmp_path / "model.safetensors"))
    cfg = LlamaConfig.from_json(hf, "fp32", 64)
    model, _ = build_llama(cfg, state=state)
    ids = torch.randint(0, 64, (2, 9), generator=g)
    want = DecoderRunner(ort.InferenceSession(model, providers=[CPU]), cfg, 2, 64).generate(ids, 5)
    runner = load_decoder(str(tmp_path), "float32", batch=2, max_len=64, block_size=16, provider=provider, cuda_graph=False)
    assert torch.equal(runner.generate(ids, 5).cpu(), want)


@pytest.mark.gpu
@pytest.mark.parametrize("heads,kv,H", [(4, 1, 64), (2, 2, 128)])
@pytest.mark.parametrize("split", [False, True])
def test_packed_flash_attention_kernel(heads, kv, H, split):
    """Packed queries over a scattered paged cache, with cached keys in front, against float64; split weights are closer."""
    from onnxruntime_b200.ops import _kernels as K
    g = torch.Generator().manual_seed(H)
    lens, past, bs = [130, 1, 257, 0, 16], [0, 300, 128, 5, 127], 128
    per = max(-(-(p + n) // bs) for p, n in zip(past, lens))
    table = (torch.randperm(5 * per, generator=g).to(torch.int32)).reshape(5, per)
    kc, vc = [torch.randn(5 * per, bs, kv, H, generator=g).to(torch.bfloat16) for _ in range(2)]
    q = torch.randn(sum(lens), heads, H, generator=g).to(torch.bfloat16)
    sink = torch.randn(heads, generator=g).to(torch.bfloat16)
    cu = i32(0, *torch.tensor(lens).cumsum(0).tolist())
    status = torch.zeros(4, dtype=torch.int32, device="cuda")
    out = K.attn_prefill_paged(q.cuda(), kc.cuda(), vc.cuda(), cu.cuda(), i32(*past).cuda(), table.cuda(), scale=0.11, head_sink=sink.cuda(),
                               split_weights=split, status=status).cpu().double()
    assert status[0] == 0
    at = 0
    for b, n in enumerate(lens):
        total = past[b] + n
        kk, vv = [c[table[b].long()].reshape(per * bs, kv, H)[:total].double().repeat_interleave(heads // kv, 1) for c in (kc, vc)]
        s = torch.einsum("thd,lhd->htl", q[at:at + n].double(), kk) * 0.11
        hidden = torch.arange(total)[None, :] > torch.arange(n)[:, None] + past[b]
        w = oracle.softmax_with_sink(s.masked_fill(hidden, float("-inf")), sink.double())
        ref = torch.einsum("htl,lhv->thv", w, vv)
        if n:
            err = (out[at:at + n] - ref).abs() - 2.0 ** -8 * ref.abs()          # what rounding the result to bf16 costs
            assert err.max() < (1e-4 if split else 2e-2)
        at += n
