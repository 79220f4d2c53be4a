"""Rovurax decoder against the plain restatement in rovurax_oracle.py: every mechanism alone, then whole models through the
registry, the pooled caches and the generation drivers.  Each case runs on the CPU provider and (marked gpu) on the GPU."""
import copy
import io
import json
import sys

import pytest
import torch

import onnxruntime_b200 as ort
import packed_decoder
import rovurax_oracle as oracle
from onnxruntime_b200 import onnx_lite as ol
from onnxruntime_b200.models.generation import GenerationConfig, generate, generate_requests
from onnxruntime_b200.models.packed_graph import padded_head_widths
from onnxruntime_b200.models.registry import create_decoder
from onnxruntime_b200.models.rotary import rotary_tables
from onnxruntime_b200.models.rovurax import RovuraxConfig, random_weights
from onnxruntime_b200.safetensors_lite import save_file
from packed_decoder import CPU, GPU, KINDS, ONNX, PROVIDERS, close, decoder, feed, i32, logits_close, run_op, tokens_of


def Reference(*args):
    return packed_decoder.Reference(oracle, *args)


def greedy_reference(*args):
    return packed_decoder.greedy_reference(oracle, *args)


def tolerance(dt):
    return 5e-5 if dt == torch.float32 else 2e-2


class Packed:
    """Projections of several sequences behind one another, fed to one operator in portions over a scattered block table."""

    def feed(self, cuts, call):
        """``call(rows, cu, past)`` runs the tokens ``rows`` (indices into the projections) and returns their outputs."""
        B = len(self.lengths)
        starts = [sum(self.lengths[:b]) for b in range(B)]
        past, out = [0] * B, [[] for _ in range(B)]
        for cut in cuts:
            rows = torch.cat([torch.arange(starts[b] + past[b], starts[b] + past[b] + cut[b]) for b in range(B)])
            y = call(rows, i32(0, *torch.tensor(cut).cumsum(0).tolist()), i32(*past))
            at = 0
            for b in range(B):
                out[b].append(y[at:at + cut[b]])
                at += cut[b]
                past[b] += cut[b]
        assert past == list(self.lengths)
        return torch.cat([torch.cat(o) for o in out])

    def table(self, spare=0):
        """Blocks in random order; block 0 belongs to nobody.  ``spare``: columns behind what the sequences need."""
        B, per = len(self.lengths), max(-(-n // self.block) for n in self.lengths)
        order = torch.randperm(B * per, generator=torch.Generator().manual_seed(5)).to(torch.int32) + 1
        return torch.cat([order.reshape(B, per), torch.zeros(B, spare, dtype=torch.int32)], 1), B * per + 1

    def with_base(self, provider, op, inputs, at, cols, n, caches, extra, **attrs):
        """Runs the operator into the first columns of a wider tensor whose other columns have to stay."""
        base = torch.full((n, cols + extra), 0.5, dtype=self.dt) if extra else None
        inputs = inputs[:at] + [base] + inputs[at + 1:] if extra else inputs
        out = base if extra else torch.zeros(n, cols, dtype=self.dt)
        run_op(provider, op, inputs, [out] + caches, **attrs)
        if extra:
            assert (out[:, cols:] == 0.5).all()
        return out[:, :cols].clone()


# ---------------------------------------------------------------------------------------------------- chunked attention
class ChunkCase(Packed):
    def __init__(self, lengths, N, G, dk, dv, chunk, dt, block, seed=0, scale=None, mixed=True, extra=8):
        g = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=g)
        self.__dict__.update(locals())
        n = sum(lengths)
        self.scale = scale if scale is not None else dk ** -0.5
        cols = N * dk + G * (dk + dv)
        self.x = rand(n, cols + -cols % 8).to(dt)
        self.first_at = 5
        self.first, self.lam = rand(n, self.first_at + G * dv + 2).to(dt), torch.tensor([0.37])

    def reference(self):
        N, G, dk, dv = self.N, self.G, self.dk, self.dv
        out, t0 = [], 0
        for n in self.lengths:
            q, k, v, _ = self.x[t0:t0 + n].double().split([N * dk, G * dk, G * dv, self.x.shape[1] - N * dk - G * (dk + dv)], 1)
            v = v.reshape(n, G, dv)
            if self.mixed:
                v = oracle.mix_values(v, self.first[t0:t0 + n, self.first_at:self.first_at + G * dv].double().reshape(n, G, dv), self.lam.double())
            mask = oracle.chunk_mask(n, self.chunk) if self.chunk else oracle.causal_mask(n)
            out.append(oracle.attend(q.reshape(n, N, dk), k.reshape(n, G, dk), v, self.scale, mask).reshape(n, N * dv))
            t0 += n
        return torch.cat(out)

    def run(self, provider, cuts):
        N, G, dk, dv = self.N, self.G, self.dk, self.dv
        table, blocks = self.table()
        kc, vc = [torch.full((blocks, self.block, G, w), 3.0, dtype=self.dt) for w in padded_head_widths("bf16" if self.dt == torch.bfloat16 else "fp32", dk, dv)]
        attrs = dict(num_heads=N, kv_num_heads=G, head_size=dk, v_head_size=dv, scale=self.scale, chunk_size=self.chunk, first_values_offset=self.first_at)

        def call(rows, cu, past):
            mix = [self.first[rows], self.lam] if self.mixed else [None, None]
            ins = [self.x[rows], kc, vc, cu, past, table] + [None] * 5 + mix + [None]
            return self.with_base(provider, "GatedPagedAttention", ins, 13, N * dv, len(rows), [kc, vc], self.extra, **attrs)
        out = self.feed(cuts, call)
        assert (kc[0] == 3).all() and (vc[0] == 3).all()
        return out


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("N,G,dk,dv,chunk,block", [
    (2, 2, 16, 16, 7, 4), (4, 2, 40, 24, 16, 16), (6, 2, 64, 64, 20, 128), (3, 1, 128, 128, 33, 128), (4, 1, 128, 128, 1, 128), (4, 4, 64, 64, 500, 128),
    (2, 1, 144, 20, 10, 8), (3, 3, 10, 14, 9, 128), (2, 1, 64, 64, 0, 128), (3, 1, 80, 128, 128, 128)])
def test_chunked_attention_with_mixed_values(kind, N, G, dk, dv, chunk, block):
    provider, dt = kind
    case = ChunkCase([19, 1, 45], N, G, dk, dv, chunk, dt, block)
    close(case.run(provider, [[19, 1, 45]]), case.reference(), dt, tolerance(dt))
    close(case.run(provider, [[2, 1, 2], [15, 0, 15], [1, 0, 27], [1, 0, 1]]), case.reference(), dt, tolerance(dt))
    case = ChunkCase([23, 5], N, G, dk, dv, chunk, dt, block, seed=2, mixed=False, extra=0)
    close(case.run(provider, [[5, 1]] + [[1, 1]] * 4 + [[14, 0]]), case.reference(), dt, tolerance(dt))
    case = ChunkCase([14, 14], N, G, dk, dv, chunk, dt, block, seed=3, extra=3)       # rows of the result are not aligned
    close(case.run(provider, [[3, 3]] + [[1, 1]] * 11), case.reference(), dt, tolerance(dt))


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("block,dk,chunk", [(128, 64, 64), (128, 128, 96), (16, 48, 40), (128, 96, 256), (128, 64, 300)])
def test_one_key_stands_out_at_the_edge_of_its_chunk(kind, block, dk, chunk):
    """Every token of a stretch asks for one key whose score dwarfs the rest: it must come through up to its chunk's last token
    and not one token later, wherever blocks, tiles and portions begin."""
    provider, dt = kind
    n = 2 * chunk + 40
    asked = [chunk - 1, 0, chunk, chunk // 2, 2 * chunk - 1]
    case = ChunkCase([n], 1, 1, dk, dk, chunk, dt, block, seed=4, scale=0.6, mixed=False)
    q, k, v = case.x[:, :dk], case.x[:, dk:2 * dk], case.x[:, 2 * dk:3 * dk]
    patterns = [torch.randn(dk, generator=torch.Generator().manual_seed(100 + j)).to(dt) for j in range(len(asked))]
    for key, p in zip(asked, patterns):
        k[key] = p
        v[key] = 4 * v[key]
    for t in range(n):
        q[t] = patterns[t % len(asked)]
    ref = case.reference()
    close(case.run(provider, [[n]]), ref, dt, tolerance(dt))
    close(case.run(provider, [[chunk - 2]] + [[1]] * 5 + [[chunk - 6]] + [[1]] * 6 + [[n - 2 * chunk - 3]]), ref, dt, tolerance(dt))
    close(case.run(provider, [[2], [chunk - 3], [2], [chunk], [n - 2 * chunk - 1]]), ref, dt, tolerance(dt))
    # the case discriminates: with chunks that end one token later, the rows at the edge are other ones
    late = ChunkCase([n], 1, 1, dk, dk, chunk, dt, block, seed=4, scale=0.6, mixed=False)
    late.x, late.chunk = case.x, chunk + 1
    moved = (late.reference()[chunk] - ref[chunk]).abs().max()
    assert moved > 0.1 * ref.abs().max()


# ------------------------------------------------------------------------------------------------------ latent attention
class LatentCase(Packed):
    def __init__(self, lengths, N, dk, dr, dv, rank, rot, dt, block, seed=0, scale=None, sink=0.0, gated=True, extra=8):
        g = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=g)
        self.__dict__.update(locals())
        n = sum(lengths)
        self.scale = scale if scale is not None else (dk + dr) ** -0.5
        cols = N * (dk + dr) + rank + dr + (N if gated else 0)
        self.x = rand(n, cols + -cols % 8).to(dt)
        self.norm, self.up = 1 + 0.2 * rand(rank), (rand(N * (dk + dv), rank) * rank ** -0.5).to(dt)
        self.sink = (rand(N) + sink).to(dt).float()

    def reference(self):
        N, dk, dr, dv, rank = self.N, self.dk, self.dr, self.dv, self.rank
        up, out, t0 = self.up.double(), [], 0
        for n in self.lengths:
            x = self.x[t0:t0 + n].double()
            pos = torch.arange(n)
            q = x[:, :N * (dk + dr)].reshape(n, N, dk + dr)
            c = oracle.rms_norm(x[:, N * (dk + dr):][:, :rank], self.norm.double(), 1e-3)
            kr = x[:, N * (dk + dr) + rank:][:, None, :dr]
            qr = q[..., dk:]
            if self.rot:
                kr, qr = oracle.rotate_interleaved(kr, pos, self.rot), oracle.rotate_interleaved(qr, pos, self.rot)
            k = torch.cat([(c @ up[:N * dk].T).reshape(n, N, dk), kr.expand(n, N, dr)], -1)
            v = (c @ up[N * dk:].T).reshape(n, N, dv)
            o = oracle.attend(torch.cat([q[..., :dk], qr], -1), k, v, self.scale, oracle.causal_mask(n), self.sink.double())
            if self.gated:
                o = o * torch.sigmoid(x[:, N * (dk + dr) + rank + dr:][:, :N])[:, :, None]
            out.append(o.reshape(n, N * dv))
            t0 += n
        return torch.cat(out)

    def run(self, provider, cuts, spare=0):
        unit = 8 if self.dt == torch.bfloat16 else 4
        wide, rotw = -(-self.rank // unit) * unit, -(-self.dr // unit) * unit
        table, blocks = self.table(spare)
        cache = torch.full((blocks, self.block, wide + rotw), 3.0, dtype=self.dt)
        cache[1:] = 0
        cos, sin = rotary_tables(self.rot, max(self.lengths)) if self.rot else (None, None)
        attrs = dict(num_heads=self.N, head_size=self.dk, rotary_size=self.dr, v_head_size=self.dv, latent_size=self.rank, latent_width=wide,
                     scale=self.scale, epsilon=1e-3, gated=int(self.gated))

        def call(rows, cu, past):
            lengths = (cu[1:] - cu[:-1] + past).tolist()
            starts = i32(0, *torch.tensor(lengths).cumsum(0).tolist())
            ins = [self.x[rows], cache, cu, past, table, cos, sin, self.norm, self.up, self.sink, None, starts]
            return self.with_base(provider, "LatentPagedAttention", ins, 10, self.N * self.dv, len(rows), [cache], self.extra, **attrs)
        out = self.feed(cuts, call)
        assert (cache[0] == 3).all()
        return out


YARN = {"factor": 8.0, "fast": 4.0, "slow": 0.5, "original": 40}


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("N,dk,dr,dv,rank,rot,block", [
    (2, 16, 8, 16, 32, {"base": 100.0, "dims": 8}, 8), (6, 32, 16, 24, 72, {"base": 300.0, "dims": 16, "scaling": YARN}, 16),
    (16, 64, 64, 64, 128, {"base": 500.0, "dims": 64, "scaling": YARN}, 128), (17, 128, 64, 128, 512, {"base": 500.0, "dims": 64}, 128),
    (40, 24, 8, 72, 64, {"base": 50.0, "dims": 8}, 128), (1, 8, 24, 8, 200, {"base": 50.0, "dims": 24}, 256),
    (3, 10, 6, 14, 33, {"base": 30.0, "dims": 6, "scaling": YARN}, 128), (2, 40, 2, 144, 600, {"base": 30.0, "dims": 2}, 16),
    (5, 136, 40, 128, 320, {"base": 30.0, "dims": 40}, 128), (4, 48, 12, 40, 88, None, 32)])
def test_latent_attention(kind, N, dk, dr, dv, rank, rot, block):
    provider, dt = kind
    tol = tolerance(dt)
    case = LatentCase([19, 1, 45], N, dk, dr, dv, rank, rot, dt, block)
    close(case.run(provider, [[19, 1, 45]]), case.reference(), dt, tol)
    case = LatentCase([29, 1, 66], N, dk, dr, dv, rank, rot, dt, block, seed=1, sink=1.0)
    close(case.run(provider, [[2, 1, 2], [15, 0, 57], [11, 0, 6], [1, 0, 1]]), case.reference(), dt, tol)
    case = LatentCase([40, 5], N, dk, dr, dv, rank, rot, dt, block, seed=2, gated=False, extra=0)
    close(case.run(provider, [[36, 1], [1, 1], [1, 1], [1, 1], [1, 1]]), case.reference(), dt, tol)
    case = LatentCase([40], N, dk, dr, dv, rank, rot, dt, block, seed=3, extra=3)           # rows of the result are not aligned
    close(case.run(provider, [[30], [9], [1]]), case.reference(), dt, tol)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("N,rank,block", [(3, 64, 128), (33, 136, 64), (2, 96, 256)])
def test_latent_attention_over_many_tiles(kind, N, rank, block):
    """Long caches: several tiles per thread block, several parts per token, and capacities far beyond what a sequence holds."""
    provider, dt = kind
    n = 700 if provider == CPU else 2900
    case = LatentCase([n, 130, 257], N, 32, 16, 32, rank, {"base": 1000.0, "dims": 16}, dt, block, seed=6, scale=0.5)
    ref = case.reference()
    cuts = [[n - 3, 126, 255], [1, 1, 1], [1, 1, 1], [1, 2, 0]]
    close(case.run(provider, cuts), ref, dt, tolerance(dt))
    close(case.run(provider, cuts, spare=40), ref, dt, tolerance(dt))
    if provider == GPU:      # a lone token: the cache is cut into parts that are merged afterwards
        case = LatentCase([n], N, 32, 16, 32, rank, {"base": 1000.0, "dims": 16}, dt, block, seed=7, scale=0.5)
        close(case.run(provider, [[n - 12], [9], [1], [1], [1]], spare=20), case.reference(), dt, tolerance(dt))


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("block,rank,rotated", [(128, 64, False), (16, 40, False), (128, 48, True), (64, 128, True)])
def test_one_latent_stands_out(kind, block, rank, rotated):
    """One cached token scores far above the rest, through its latent or through the rotated part (positions matter then): the
    first token, either side of block and tile borders, or the token itself - in prompts, across portions and in decoding."""
    provider, dt = kind
    n, dr = 300, 8
    asked = [0, 1, 63, 64, 127, 128, 129, 255, 256]
    rot = {"base": 40.0, "dims": dr}
    case = LatentCase([n], 1, rank, dr, rank, rank, rot, dt, block, seed=4, scale=1.0, sink=-2.0)
    case.up[:rank], case.up[rank:] = torch.eye(rank).to(dt), torch.eye(rank).to(dt)    # keys and values are the latents
    case.norm = torch.ones(rank)
    q, qr, c, kr = case.x[:, :rank], case.x[:, rank:rank + dr], case.x[:, rank + dr:2 * rank + dr], case.x[:, 2 * rank + dr:2 * rank + 2 * dr]
    q *= 0.1
    qr *= 0.1
    for j, key in enumerate(asked):
        at = n - len(asked) + j
        if rotated:
            kr *= 0.1 if j == 0 else 1.0
            kr[key] = 4 * torch.randn(dr, generator=torch.Generator().manual_seed(100 + j)).to(dt)
            # rotated to its own position, the query points along the key that was rotated to the key's position
            want = oracle.rotate_interleaved(kr[key].double()[None, None], torch.tensor([key]), rot)
            qr[at] = 2 * oracle.rotate_interleaved(want, torch.tensor([-at]), rot)[0, 0].to(dt)
        else:
            pattern = torch.randn(rank, generator=torch.Generator().manual_seed(100 + j)).to(dt)
            c[key] = pattern
            q[at] = pattern
    ref = case.reference()
    tol = tolerance(dt) * (1 if dt == torch.float32 else 2)
    close(case.run(provider, [[n]]), ref, dt, tol)
    m = n - len(asked)
    close(case.run(provider, [[m]] + [[1]] * len(asked)), ref, dt, tol)
    close(case.run(provider, [[128], [2], [m - 130], [2], [len(asked) - 2]]), ref, dt, tol)
    other = copy.copy(case)
    other.x = case.x.clone()
    other.x[128, rank + dr:] *= -1
    at = n - len(asked) + asked.index(128)
    assert (other.reference()[at] - ref[at]).abs().max() > 0.2 * ref[at].abs().max()


@pytest.mark.parametrize("kind", KINDS)
def test_sink_takes_its_share_once(kind):
    """A sink far above the scores silences its head, one far below changes nothing; both next to each other."""
    provider, dt = kind
    case = LatentCase([70], 3, 16, 8, 16, 32, {"base": 50.0, "dims": 8}, dt, 128, seed=8, gated=False)
    case.sink = torch.tensor([12.0, -30.0, 3.0])
    ref = case.reference().reshape(70, 3, 16)
    assert ref[:, 0].abs().max() < 0.05 * ref[:, 1].abs().max() and 0.05 < ref[-1, 2].abs().max() / ref[-1, 1].abs().max()
    for cuts in ([[70]], [[40]] + [[1]] * 30, [[2]] * 35):
        close(case.run(provider, cuts), case.reference(), dt, tolerance(dt))
    other = copy.copy(case)
    other.sink = case.sink - torch.log(torch.tensor(2.0))         # counted half: another result
    assert (other.reference() - case.reference()).abs().max() > 0.02 * ref.abs().max()


@pytest.mark.gpu
def test_latent_kernels_take_the_tensor_cores():
    """Which sizes the tuned kernels serve: the prompt form, and the parts a decode step is cut into."""
    import ctypes
    from onnxruntime_b200.ops import _kernels as K
    f = K.lib().ortb200_latent_prefill_supported
    assert f(128, 64, 128, 1) and f(40, 24, 56, 1) and not f(30, 24, 56, 1) and not f(192, 64, 128, 1) and not f(64, 64, 64, 2)
    parts = ctypes.c_int(0)
    plan = K.lib().ortb200_latent_decode_plan
    assert plan(1, 16, 512, 576, 128, 256, 1, ctypes.byref(parts)) and parts.value > 4
    assert plan(64, 32, 512, 576, 128, 256, 1, ctypes.byref(parts)) and parts.value == 1
    assert not plan(1, 16, 600, 664, 128, 16, 1, ctypes.byref(parts)) and not plan(1, 16, 512, 576, 128, 16, 2, ctypes.byref(parts))


# ---------------------------------------------------------------------------------------------- rotation and feed-forward
@pytest.mark.parametrize("rot", [
    {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0, "fast": 32.0, "slow": 1.0, "original": 4096}},
    {"base": 100.0, "dims": 10, "scaling": {"factor": 2.5, "fast": 2000.0, "slow": 1e-9, "original": 64}},      # both ends clamped
    {"base": 500.0, "dims": 8, "scaling": {"factor": 16.0, "fast": 1.0, "slow": 1.0, "original": 628.3185307}},  # a step, no ramp
    {"base": 500.0, "dims": 12, "scaling": {"factor": 1.0, "fast": 8.0, "slow": 1.0, "original": 128}}, {"base": 500.0, "dims": 2}])
def test_yarn_tables(rot):
    cos, sin = rotary_tables(rot, 40)
    f, gain = oracle.yarn_frequencies(rot)
    a = torch.arange(40, dtype=torch.float64)[:, None] * f
    assert torch.allclose(cos.double(), gain * a.cos(), atol=1e-6) and torch.allclose(sin.double(), gain * a.sin(), atol=1e-6)


def test_yarn_has_a_ramp_between_two_bands():
    rot = {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0, "fast": 32.0, "slow": 1.0, "original": 4096}}
    f, gain = oracle.yarn_frequencies(rot)
    plain, one = oracle.yarn_frequencies({"base": 10000.0, "dims": 64})
    assert (f == plain).any() and torch.isclose(f, plain / 4).any() and ((f < 0.99 * plain) & (f > 1.01 * plain / 4)).any()
    assert one == 1.0 and 1.1 < gain < 1.2


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("width,ff,lead", [(48, 72, 0), (48, 72, 16), (40, 20, 6), (33, 9, 5)])
def test_clamped_feed_forward(kind, width, ff, lead):
    """Both clamps are reached; the product lies behind the lead columns; 16-bit models use the gated GEMM."""
    provider, dt = kind
    g = torch.Generator().manual_seed(ff)
    limit, alpha, offset = 1.5, 1.3, 0.75
    for tokens in (3, 80, 200):            # the three GEMM shapes of the gated epilogue
        h, wg, wu = [torch.randn(*s, generator=g).mul(0.6).to(dt) for s in ((tokens, width), (ff, width), (ff, width))]
        dev = "cuda" if provider == GPU else "cpu"
        inits = [ol.make_external_tensor(n, ONNX[dt], (width, ff)) for n in ("wg", "wu")]
        nodes = [ol.make_node("MatMul", ["h", "wg"], ["a"]), ol.make_node("MatMul", ["h", "wu"], ["b"]),
                 ol.make_node("ClampedSwiGLU", ["a", "b"], ["o"], domain="com.ortb200", limit=limit, alpha=alpha, offset=offset, lead_columns=lead)]
        graph = ol.make_graph(nodes, "g", [ol.make_tensor_value_info("h", ONNX[dt], ["n", width])],
                              [ol.make_tensor_value_info("o", ONNX[dt], ["n", lead + ff])], inits)
        so = ort.SessionOptions()
        so.add_external_initializers(["wg", "wu"], [wg.t().contiguous().to(dev), wu.t().contiguous().to(dev)])
        sess = ort.InferenceSession(ol.make_model(graph, opset=17, extra_opsets={"com.ortb200": 1}).serialize(), so, providers=[provider])
        if dt == torch.bfloat16 and width % 8 == 0:
            assert [n["op_type"] for n in sess.graph_nodes()] == ["GemmSwiGLU"]
        out = torch.zeros(tokens, lead + ff, dtype=dt, device=dev)
        b = sess.io_binding()
        b.bind_torch_input("h", h.to(dev))
        b.bind_torch_output("o", out)
        sess.run_with_iobinding(b)
        a, u = h.double() @ wg.double().T, h.double() @ wu.double().T
        assert (a > limit).any() and (u > limit).any() and (u < -limit).any() and (a < -limit).any()
        a, u = a.clamp(max=limit), u.clamp(-limit, limit)
        close(out.cpu()[:, lead:], a * torch.sigmoid(alpha * a) * (u + offset), dt, 3e-5 if dt == torch.float32 else 3e-2)
    z = torch.linspace(-4, 4, 41, dtype=torch.float64)
    gate = torch.minimum(z, torch.tensor(2.0, dtype=torch.float64))
    assert torch.allclose(oracle.clamped_gate(z, z, 2.0), gate * torch.sigmoid(1.702 * gate) * (z.clamp(-2, 2) + 1))


# -------------------------------------------------------------------------------------------------------- whole models
def small_config(name):
    att = {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 20, "scale": 0.25, "mask": {"size": 11}, "v_mix": True}
    lat = {"heads": 3, "dim": 24, "rot_dim": 8, "vdim": 16, "kv_rank": 40, "scale": 0.3, "rot": {"base": 300.0, "dims": 8, "scaling": dict(YARN)}}
    ff = lambda n, limit=1.0: {"kind": "dense", "ff": n, "limit": limit}
    layers = {
        "mixed": [("latent_attention", lat, ff(56)), ("attention", dict(att, v_mix=False, mask={"size": 5}), None), ("attention", att, ff(40, 0.6)),
                  ("latent_attention", dict(lat, heads=5, vdim=24, kv_rank=24, scale=0.2), None), ("attention", dict(att, heads=2, mask={"size": 16}), ff(24))],
        "chunks": [("attention", dict(att, dim=64, vdim=64, heads=2, kv_heads=1, mask={"size": 3}), ff(32)),
                   ("attention", dict(att, dim=128, vdim=64, heads=3, kv_heads=1, mask={"size": 19}), ff(24)),
                   ("attention", dict(att, dim=16, vdim=64, heads=2, kv_heads=1, mask={"size": 1}), None)],
        "latents": [("latent_attention", dict(lat, heads=17, dim=16, rot_dim=16, rot={"base": 90.0, "dims": 16}), None),
                    ("latent_attention", dict(lat, heads=1, kv_rank=64, vdim=64, rot={"base": 50.0, "dims": 8, "scaling": dict(YARN, factor=1.0)}), ff(16))],
        # sizes that no tensor-core or vector path takes
        "odd": [("attention", dict(att, heads=3, kv_heads=1, dim=10, vdim=14), ff(20)),
                ("latent_attention", dict(lat, heads=3, dim=9, rot_dim=6, vdim=7, kv_rank=21, rot={"base": 30.0, "dims": 6}), ff(10)),
                ("attention", dict(att, heads=2, kv_heads=1, dim=7, vdim=14), ff(9))],
        # the latent projections of a prompt reach the widest flash form; values of 128
        "wide": [("latent_attention", dict(lat, heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=192, scale=0.08, rot={"base": 900.0, "dims": 64, "scaling": dict(YARN)}),
                  ff(48)), ("attention", dict(att, dim=128, vdim=128, heads=4, kv_heads=1, scale=0.09, mask={"size": 40}), ff(48))],
    }[name]
    return {"architecture": "Rovurax", "vocab": 97 if name != "chunks" else 120, "width": {"odd": 36, "latents": 40}.get(name, 48), "norm": {"eps": 1e-5},
            "layers": [{"type": t, "mixer": copy.deepcopy(m), "mlp": f} for t, m, f in layers]}


NAMES = ["mixed", "chunks", "latents", "odd", "wide"]


def model_pair(name, seed=0):
    cfg = small_config(name)
    return cfg, random_weights(RovuraxConfig.from_json(cfg), seed=seed, gain=1.5)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", NAMES)
def test_model_matches_the_restatement(kind, name):
    """Whole prompt, portions down to two tokens, token by token, and a prompt followed by decoding."""
    cfg, w = model_pair(name)
    toks = tokens_of(cfg, 61, 1)
    ref = Reference(cfg, w, toks)
    runner = decoder(cfg, w, kind)
    for cuts in ([61], [2, 2, 15, 3, 2, 37], [1] * 61, [43] + [1] * 18, [16, 16, 29], [20, 1, 20, 20]):
        logits_close(feed(runner, "s", toks, cuts), ref, kind[1])
        runner.release("s")
    for n in (1, 2, 3):         # the shortest sequences
        logits_close(feed(runner, "s", toks[:n], [n]), ref[:n], kind[1])
        runner.release("s")


@pytest.mark.parametrize("kind", KINDS)
def test_layer_order_comes_from_the_configuration(kind):
    """The same layers reversed are another model (another layer is then the first whose values are mixed), and it matches too."""
    cfg, _ = model_pair("mixed")
    cfg["layers"] = cfg["layers"][::-1]
    w = random_weights(RovuraxConfig.from_json(cfg), seed=5, gain=1.5)
    toks = tokens_of(cfg, 30, 3)
    logits_close(feed(decoder(cfg, w, kind), 0, toks, [5, 25]), Reference(cfg, w, toks), kind[1])


@pytest.mark.parametrize("kind", KINDS)
def test_value_mixing_weight_matters_except_in_its_first_layer(kind):
    cfg, w = model_pair("chunks", seed=3)
    toks = tokens_of(cfg, 20, 4)
    for name, value in (("l0.mix.vmix", 0.9), ("l1.mix.vmix", 0.0), ("l2.mix.vmix", 1.0)):
        w = dict(w, **{name: torch.tensor(value).to(torch.bfloat16)})
        logits_close(feed(decoder(cfg, w, kind), 0, toks, [17, 1, 2]), Reference(cfg, w, toks), kind[1])
    base = oracle.forward(cfg, w, toks)
    assert torch.equal(base, oracle.forward(cfg, dict(w, **{"l0.mix.vmix": torch.tensor(0.1)}), toks))
    assert (base - oracle.forward(cfg, dict(w, **{"l1.mix.vmix": torch.tensor(0.8)}), toks)).abs().max() > 1e-2


@pytest.mark.parametrize("kind", KINDS)
def test_unequal_requests_in_one_batch_equal_each_alone(kind):
    cfg, w = model_pair("mixed", seed=2)
    texts = {s: tokens_of(cfg, n, 10 + n) for s, n in (("a", 77), ("b", 5), ("c", 1), ("d", 52))}
    runner = decoder(cfg, w, kind)
    refs = {s: Reference(cfg, w, t) for s, t in texts.items()}
    got = {s: [] for s in texts}

    def step(portions):
        rows = runner.step([(s, texts[s][a:b], list(range(b - a))) for s, a, b in portions])
        at = 0
        for s, a, b in portions:
            got[s].append(rows[at:at + b - a])
            at += b - a
    step([("a", 0, 60), ("b", 0, 3), ("c", 0, 1), ("d", 0, 8)])
    runner.release("c")
    step([("d", 8, 9), ("a", 60, 61), ("b", 3, 4)])            # one token each, another order
    step([("b", 4, 5), ("a", 61, 66), ("d", 9, 49)])           # decoding and portions of prompts in one batch
    runner.release("b")
    step([("a", 66, 76), ("d", 49, 52)])
    runner.release("d")
    step([("a", 76, 77)])
    for s in texts:
        logits_close(torch.cat(got[s]), refs[s], kind[1])


@pytest.mark.parametrize("kind", KINDS)
def test_blocks_are_reused(kind):
    """Many requests through a pool that holds few: every one finds blocks that others have left full."""
    cfg, w = model_pair("mixed", seed=3)
    block = 16 if kind[0] == CPU else 128
    n = block + 9
    runner = decoder(cfg, w, kind, batch=2, max_len=2 * block, block_size=block)
    texts = [tokens_of(cfg, n if i % 2 else 7 + i, 50 + i) for i in range(6)]
    refs = [Reference(cfg, w, t) for t in texts]
    held = []
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
            held += runner.pool.sequences[j].blocks
            runner.release(j)
    assert len(held) == 9 and len(set(held)) <= 4 and len(runner.pool.free_blocks) == 4


@pytest.mark.parametrize("kind", KINDS)
def test_decode_graphs_of_several_batch_sizes(kind):
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
    """Chunk after chunk and tile after tile passes over decoded tokens."""
    cfg, w = model_pair("mixed", seed=6)
    n = 300 if kind[0] == GPU else 70
    toks = tokens_of(cfg, n, 7)
    runner = decoder(cfg, w, kind, batch=1, max_len=n)
    logits_close(feed(runner, 0, toks, [3] + [1] * (n - 3)), Reference(cfg, w, toks), kind[1])


@pytest.mark.parametrize("provider", PROVIDERS)
def test_greedy_generation(provider, tmp_path, capsys):
    """The runner's own loop, ``generate``, ``generate_requests`` (more requests than fit at a time) and the command line."""
    cfg, w = model_pair("mixed", seed=8)
    kind = (provider, torch.float32)
    prompts = [tokens_of(cfg, n, 30 + n) for n in (9, 44, 13)]
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
    a, b = tokens_of(cfg, 60, 1), tokens_of(cfg, 8, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:58], "want": [57, 0]}, {"id": "b", "tokens": b[:7], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[58:59], "want": []}, {"id": "b", "tokens": b[7:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[59:], "want": [0]}], "end": ["a"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace_replay.main(["--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "80"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "1.f32").exists()
    ref = Reference(cfg, w, a)
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).reshape(-1, cfg["vocab"])
    logits_close(read(0), ref[[57, 0]], dt)
    logits_close(read(2), ref[[59]], dt)


@pytest.mark.gpu
def test_half_precision_model():
    """fp16 runs the same kernels as bfloat16."""
    cfg, w = model_pair("wide", seed=11)
    toks = tokens_of(cfg, 50, 2)
    ref = Reference(cfg, w, toks)
    runner = create_decoder(cfg, w, "float16", batch=2, max_len=96, block_size=128)
    logits_close(feed(runner, 0, toks, [41, 1, 1, 7]), ref, torch.bfloat16)


# --------------------------------------------------------------------------------------- configuration, weights, mistakes
def test_configuration_is_checked():
    cfg = small_config("mixed")
    assert RovuraxConfig.from_json(RovuraxConfig.from_json(cfg).to_json()).layers == cfg["layers"]
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][4]["mixer"].update(kv_heads=1), lambda c: c["layers"][2]["mixer"].update(vdim=16),
                   lambda c: c["layers"][1]["mixer"].update(heads=3), lambda c: c["layers"][1]["mixer"].update(mask={"size": 0}),
                   lambda c: c["layers"][0]["mixer"].update(rot={"base": 10.0, "dims": 10})):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            RovuraxConfig.from_json(bad)
    _, w = model_pair("mixed")
    short = dict(w)
    del short["l0.mix.uk"]
    with pytest.raises(KeyError, match="l0.mix.uk"):
        decoder(cfg, short, (CPU, torch.float32))
    wrong = dict(w, head=w["head"][:-1])
    with pytest.raises(ValueError, match="head"):
        decoder(cfg, wrong, (CPU, torch.float32))


@pytest.mark.parametrize("mistake", ["late chunk", "no sink", "rotate-half", "no gain", "plain up branch", "sequential block"])
def test_the_cases_show_mistakes(mistake, monkeypatch):
    """Planted in the restatement, each mistake moves the logits by far more than the tests allow."""
    cfg, w = model_pair("mixed", seed=12)
    toks = tokens_of(cfg, 40, 5)
    right = oracle.forward(cfg, w, toks)
    if mistake == "late chunk":
        mask = oracle.chunk_mask
        monkeypatch.setattr(oracle, "chunk_mask", lambda T, size: mask(T, size + 1))
    elif mistake == "no sink":
        soft = oracle.visible_softmax
        monkeypatch.setattr(oracle, "visible_softmax", lambda s, m, sink=None: soft(s, m))
    elif mistake == "rotate-half":
        turn = oracle.rotate_interleaved

        def halves(x, pos, rot):
            n = rot["dims"]
            order = torch.arange(n).reshape(2, n // 2).t().reshape(-1)
            y = turn(x[..., order], pos, rot)
            return y[..., torch.argsort(order)]
        # halves on the queries only: keys and queries no longer agree
        monkeypatch.setattr(oracle, "rotate_interleaved", lambda x, pos, rot: halves(x, pos, rot) if x.shape[1] > 1 else turn(x, pos, rot))
    elif mistake == "no gain":
        freq = oracle.yarn_frequencies
        monkeypatch.setattr(oracle, "yarn_frequencies", lambda rot: (freq(rot)[0], 1.0))
    elif mistake == "plain up branch":
        monkeypatch.setattr(oracle, "clamped_gate", lambda g, u, limit: torch.clamp(g, max=limit) * torch.sigmoid(1.702 * g.clamp(max=limit)) * u.clamp(-limit, limit))
    else:
        monkeypatch.setattr(oracle, "dense_ff", lambda h, w_, p, limit: 0.9 * h)
    wrong = oracle.forward(cfg, w, toks)
    assert packed_decoder.relative_error(wrong - right, right).max() > 1e-2


# ------------------------------------------------------------------------------------------------------- kernels alone
def rounded_close(got, want, tol=1e-4):
    """Equal up to rounding the result to bfloat16 and ``tol``: softmax weights in 16 bits would be a hundred times further off."""
    assert ((got.double() - want).abs() - 2.0 ** -8 * want.abs()).max() < tol


@pytest.mark.gpu
@pytest.mark.parametrize("N,G,chunk", [(4, 4, 0), (8, 2, 0), (16, 1, 100), (6, 2, 1), (8, 1, 300), (12, 4, 128)])
def test_decode_attention_keeps_its_weights(N, G, chunk):
    """Tensor-core decode kernel over a scattered paged cache: 32-bit weights, chunks that begin inside a tile."""
    from onnxruntime_b200.ops import _kernels as K
    g = torch.Generator().manual_seed(N)
    H, bs, lens = 128, 128, [1, 100, 101, 128, 129, 300, 301, 500, 777]
    B, per = len(lens), 7
    table = torch.randperm(B * per, generator=g).to(torch.int32).reshape(B, per)
    kc, vc = [torch.randn(B * per, bs, G, H, generator=g).to(torch.bfloat16) for _ in range(2)]
    q = torch.randn(B, N, H, generator=g).to(torch.bfloat16)
    past = i32(*[n - 1 for n in lens])
    out = [K.gqa_decode(q.cuda(), kc.cuda(), vc.cuda(), past.cuda(), block_table=table.cuda(), split_weights=True, chunk=chunk, scale=0.2, algo=2).cpu()
           for _ in range(3)]
    assert torch.equal(out[0], out[1]) and torch.equal(out[0], out[2])
    for b, n in enumerate(lens):
        lo = (n - 1) // chunk * chunk if chunk else 0
        k, v = [c[table[b].long()].reshape(per * bs, G, H)[lo:n].double().repeat_interleave(N // G, 1) for c in (kc, vc)]
        s = torch.einsum("hd,lhd->hl", q[b].double(), k)[:, None] * 0.2
        w = oracle.visible_softmax(s, torch.ones(1, n - lo, dtype=torch.bool))
        rounded_close(out[0][b].reshape(N, H), torch.einsum("htl,lhv->hv", w, v))


@pytest.mark.gpu
@pytest.mark.parametrize("H,chunk", [(64, 0), (128, 0), (128, 100)])
def test_prompt_attention_is_repeatable(H, chunk):
    """The same launch many times, on a machine full of other blocks: bit-equal, and right."""
    from onnxruntime_b200.ops import _kernels as K
    g = torch.Generator().manual_seed(H)
    N, G, bs, lens, past = 8, 2, 128, [700, 130, 1, 500], [0, 300, 77, 900]
    per = max(-(-(p + n) // bs) for p, n in zip(past, lens))
    table = torch.randperm(4 * per, generator=g).to(torch.int32).reshape(4, per)
    kc, vc = [torch.randn(4 * per, bs, G, H, generator=g).to(torch.bfloat16) for _ in range(2)]
    q = torch.randn(sum(lens), N, H, generator=g).to(torch.bfloat16)
    cu = i32(0, *torch.tensor(lens).cumsum(0).tolist()).cuda()
    args = [q.cuda(), kc.cuda(), vc.cuda(), cu, i32(*past).cuda(), table.cuda()]
    out = K.attn_prefill_paged(*args, scale=0.2, split_weights=True, chunk=chunk)
    for _ in range(40):
        assert torch.equal(K.attn_prefill_paged(*args, scale=0.2, split_weights=True, chunk=chunk), out)
    out, at = out.cpu(), 0
    for b, n in enumerate(lens):
        total = past[b] + n
        k, v = [c[table[b].long()].reshape(per * bs, G, H)[:total].double().repeat_interleave(N // G, 1) for c in (kc, vc)]
        mask = (oracle.chunk_mask(total, chunk) if chunk else oracle.causal_mask(total))[past[b]:]
        w = oracle.visible_softmax(torch.einsum("thd,lhd->htl", q[at:at + n].double(), k) * 0.2, mask)
        rounded_close(out[at:at + n], torch.einsum("htl,lhv->thv", w, v))
        at += n


@pytest.mark.gpu
@pytest.mark.parametrize("dk,dr,dv", [(32, 16, 32), (128, 64, 128), (64, 64, 128), (72, 8, 40)])
def test_latent_prompt_kernel_is_repeatable(dk, dr, dv):
    from onnxruntime_b200.ops import _kernels as K
    g = torch.Generator().manual_seed(dk)
    N, lens, past = 6, [300, 1, 600], [200, 5, 0]
    T, rows, cols = sum(lens), sum(lens) + sum(past), N * (dk + dr) + N
    rand = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    x, q_rot, kv, kr, sink = rand(T, cols + -cols % 8), rand(T, N, dr), rand(rows, N * (dk + dv)), rand(rows, dr + -dr % 8), rand(N)
    dev = [t.cuda() for t in (x, q_rot, kv, kr, sink)]
    cu = i32(0, *torch.tensor(lens).cumsum(0).tolist()).cuda()
    run = lambda: K.latent_prefill(dev[0], dev[1], dev[2], dev[3], dev[4], dev[0][:, cols - N:], cu, i32(*past).cuda(), N, dk, dr, dv, 0.15)
    out = run()
    for _ in range(40):
        assert torch.equal(run(), out)
    out, at, k0 = out.cpu(), 0, 0
    for b, n in enumerate(lens):
        total = past[b] + n
        q = torch.cat([x[at:at + n, :N * (dk + dr)].reshape(n, N, dk + dr)[..., :dk], q_rot[at:at + n]], -1).double()
        k = torch.cat([kv[k0:k0 + total, :N * dk].reshape(total, N, dk), kr[k0:k0 + total, None, :dr].expand(total, N, dr)], -1).double()
        v = kv[k0:k0 + total, N * dk:].reshape(total, N, dv).double()
        w = oracle.visible_softmax(torch.einsum("thd,lhd->htl", q, k) * 0.15, oracle.causal_mask(total)[past[b]:], sink.double())
        ref = torch.einsum("htl,lhv->thv", w, v) * torch.sigmoid(x[at:at + n, cols - N:cols].double())[:, :, None]
        rounded_close(out[at:at + n].reshape(n, N, dv), ref, 2e-4)
        at, k0 = at + n, k0 + total


@pytest.mark.gpu
@pytest.mark.parametrize("N,rank,dr,bs", [(16, 512, 64, 128), (40, 136, 16, 64), (3, 64, 8, 8)])
def test_latent_decode_kernel_is_repeatable(N, rank, dr, bs):
    from onnxruntime_b200.ops import _kernels as K
    g = torch.Generator().manual_seed(N)
    lens = [900, 33, 1, 129, 640]
    B, per = len(lens), -(-900 // bs)
    table = torch.randperm(B * per, generator=g).to(torch.int32).reshape(B, per)
    cache = torch.randn(B * per, bs, rank + dr, generator=g).to(torch.bfloat16)
    q = (0.3 * torch.randn(B, N, rank + dr, generator=g)).to(torch.bfloat16)
    args = [q.cuda(), cache.cuda(), torch.arange(B + 1, dtype=torch.int32).cuda(), i32(*[n - 1 for n in lens]).cuda(), table.cuda(), rank, 0.3]
    o, ml = K.latent_decode(*args)
    for _ in range(40):
        again = K.latent_decode(*args)
        assert torch.equal(again[0], o) and torch.equal(again[1], ml)
    for b, n in enumerate(lens):
        c = cache[table[b].long()].reshape(per * bs, -1)[:n].double()
        want = oracle.visible_softmax((q[b].double() @ c.T)[:, None] * 0.3, torch.ones(1, n, dtype=torch.bool))[:, 0] @ c[:, :rank]
        f = torch.exp2(ml[b, :, :, 0] - ml[b, :, :, 0].max(1, keepdim=True).values)
        got = (f[..., None] * o[b]).sum(1) / (f * ml[b, :, :, 1]).sum(1, keepdim=True)
        assert (got.double().cpu() - want).abs().max() < 1e-4
