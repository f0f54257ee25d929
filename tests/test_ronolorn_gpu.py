"""Ronolorn on the device against the plain implementation (tests/plain_ronolorn.py): each mechanism
alone through its kernel, then whole models through the step function: whole prompts, prompts against
token-by-token decoding, portions down to two tokens, mixed batches with pages and slots that are used
again, far keys and keys at page and window borders that the weights are made to show, long decoding,
other sizes, and greedy generation through the entry point."""
import math
import os
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_ronolorn as plain
from helpers import (collect_logits, lines_of, max_live_tokens, random_ids, schedule_mixed, schedule_portions,
                     schedule_tail_decode, schedule_whole)
from ronolorn_configs import (RONOLORN_TINY, _delta, _dense, _tied, _window, decisive, make_ronolorn_dir,
                              random_ronolorn_config_dict)

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
# Largest |logit difference|, and largest root-mean-square difference over the vocabulary at one position, over the
# largest plain |logit|.  float32: 32-bit sums against float64, the sharp test of every schedule.  bfloat16: products
# and activations rounded to 8 bits through tiny random layers; it catches a kernel that is wrong, not one that
# rounds elsewhere.
TOLERANCE = {"float32": 5e-5, "bfloat16": 1.5e-1}
RMS_TOLERANCE = {"float32": 1.7e-5, "bfloat16": 5e-2}
MEASURED = {}


def draws(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).bfloat16().double()


def on_device(x, dtype):
    return x.to(dtype).to(DEV).contiguous()


def close(got, want, tol):
    err = (got.double().cpu() - want).abs().max().item()
    assert err <= tol * max(want.abs().max().item(), 1e-30), (err, want.abs().max().item())


class Tables:
    """Rotary tables over ``dims`` elements."""

    def __init__(self, rot, interleaved=True, n=1024):
        from tinyserve_b200.parts.rotary import Rotary
        s = rot.get("scaling")
        self.rotary_dim, self.interleaved = rot["dims"], interleaved
        scaling = ("ramp", *(float(s[k]) for k in ("factor", "original", "fast", "slow"))) if s else None
        self.cos, self.sin = (t.to(DEV) for t in Rotary.tables(rot["dims"], float(rot["base"]), n, scaling))


# ----------------------------------------------------------------------------- streams
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 4e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("T,n,S", [(23, 41, 2), (7, 200, 1), (600, 1000, 3), (4, 2048, 2), (3, 5000, 4), (40, 1024, 4), (64, 8192, 1),
                                   (3, 12000, 2), (530, 1536, 2), (513, 4096, 2), (9, 96, 7), (2, 2000, 12), (5, 20000, 2), (3, 37, 32)])
def test_streams_take_in_an_output_and_are_read_through_a_norm(dtype, tol, T, n, S):
    """First read (all streams one row), two updates, a layer norm with and without bias and an RMS norm, and
    chosen rows of their sum, which leave the streams alone.  The rows sit far from zero: their mean is many times
    their deviation."""
    from tinyserve_b200.kernels import ops
    start = draws(T, n, seed=1) + draws(T, 1, seed=9, scale=20.0)
    y1, y2 = draws(T, n, seed=2, scale=3.0), draws(T, n, seed=3)
    mixes = [draws(S, S, seed=4, scale=0.6), draws(S, S, seed=5, scale=0.6)]
    outs = [draws(S, seed=6), draws(S, seed=7)]
    reads = [draws(S, seed=10 + i) for i in range(3)]
    w, b = (draws(n, seed=8, scale=0.3) + 1).bfloat16().double(), draws(n, seed=20)
    d = lambda x: on_device(x, dtype)
    streams = ops.Streams(on_device(start, torch.float32), S)
    X = start[None].repeat(S, 1, 1)

    def near(got, u, want):
        # (a sum of streams that cancels to nothing leaves the rounding of its parts)
        slack = max(1.0, 0.3 * X.abs().max().item() / u.std(-1).min().item())
        close(got, want, tol * slack if dtype == torch.float32 else max(tol, 3e-6 * slack))

    u = plain.streams_in(X, reads[0])
    near(ops.stream_norm(None, streams, d(reads[0]), d(w), 1e-5, dtype), u, plain.centred_norm(u, w, 1e-5))
    assert not streams.apart
    for i, y in enumerate((y1, y2)):
        X = plain.streams_out(X, y, mixes[i], outs[i])
        u = plain.streams_in(X, reads[1 + i])
        x = ops.StreamMix(d(y), d(mixes[i]), d(outs[i]))
        if i == 0:
            near(ops.stream_norm(x, streams, d(reads[1]), d(w), 1e-5, dtype, bias=d(b)), u, plain.centred_norm(u, w, 1e-5) + b)
        else:
            near(ops.stream_norm(x, streams, d(reads[2]), d(w), 1e-5, dtype, centred=False), u, plain.unit_rms(u, 1e-5) * w)
        close(streams.data, X.transpose(0, 1), 1e-6)
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device=DEV)
    before = streams.data.clone()
    x = ops.StreamMix(d(y1), d(mixes[0]), d(outs[0]))
    X = plain.streams_out(X, y1, mixes[0], outs[0])
    u = X.sum(0)
    got = ops.stream_norm(x, streams, None, d(w), 1e-5, dtype, rows=rows)
    near(got, u, plain.centred_norm(u, w, 1e-5)[rows.cpu().long()])
    assert torch.equal(streams.data, before)


@pytest.mark.parametrize("M,N,K,S", [(1, 2048, 512, 2), (8, 1024, 4096, 3), (16, 512, 72, 2), (13, 1000, 2048, 4), (33, 2048, 1024, 2),
                                     (64, 384, 512, 5), (20, 4096, 64, 1)])
@pytest.mark.parametrize("bias", [False, True])
def test_a_product_joins_the_streams_as_partial_tiles(M, N, K, S, bias):
    from tinyserve_b200.kernels import ops
    x, w, b = draws(M, K, seed=1), draws(N, K, seed=2, scale=K ** -0.5), draws(N, seed=3)
    start, mix, out, read = draws(M, N, seed=4), draws(S, S, seed=5), draws(S, seed=6), draws(S, seed=7)
    d = lambda t: on_device(t, torch.bfloat16)
    pending = ops.linear(d(x), d(w), d(b) if bias else None, allow_pending=True)
    assert isinstance(pending, ops.PendingProduct)
    streams = ops.Streams(on_device(start, torch.float32), S)
    h = ops.stream_norm(ops.StreamMix(pending, d(mix), d(out)), streams, d(read), d(draws(N, seed=8)), 1e-5, torch.bfloat16)
    X = plain.streams_out(start[None].repeat(S, 1, 1), x @ w.T + (b if bias else 0), mix, out)
    close(streams.data, X.transpose(0, 1), 1e-5 if pending.splits() > 1 else 6e-3)
    close(h, plain.centred_norm(plain.streams_in(X, read), draws(N, seed=8), 1e-5), 4e-2)


# ----------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("T,width,ff", [(1, 64, 72), (9, 128, 192), (70, 256, 384), (300, 96, 104), (5, 64, 37), (3, 2048, 256), (16, 256, 20000)])
def test_feed_forward_against_the_plain_one(dtype, tol, T, width, ff):
    from tinyserve_b200.kernels import ops
    from tinyserve_b200.parts.mlp import PlainMLP
    part = PlainMLP(width, ff)
    h, up, down = draws(T, width, seed=1), draws(ff, width, seed=2, scale=width ** -0.5), draws(width, ff, seed=3, scale=ff ** -0.5)
    part.bind({"up_proj.weight": on_device(up, dtype), "down_proj.weight": on_device(down, dtype)})
    close(ops.materialize(part.forward(on_device(h, dtype), None)), plain.feed_forward(h, {"up": up, "down": down}, ""), tol)
    close(ops.activated_linear(on_device(h, dtype), on_device(up, dtype), "relu_squared"), torch.relu(h @ up.T).pow(2), tol)
    z = draws(T, ff, seed=5)
    close(ops.plain_activation_(on_device(z, dtype), "relu_squared"), torch.relu(z).pow(2), 5e-3 if dtype == torch.bfloat16 else 1e-6)


# ----------------------------------------------------------------------------- the memory
def _memory_inputs(T, H, G, n, nv, seed):
    g = torch.Generator().manual_seed(seed)
    q, k, v, gate = (draws(T, m, seed=seed + i) for i, m in enumerate((G * n, G * n, H * nv, H * nv)))
    logits = torch.cat([torch.randn(T, H, generator=g) * 1.5, torch.randn(T, H, generator=g) * 2.0], -1).double()
    logits[::7, :H] += 6.0                     # (a token that makes the memory forget)
    return q, k, v, gate, logits


def _plain_memory(q, k, v, gate, logits, bias, rate, norm, eps, H, G, n, nv, states=None):
    T = q.shape[0]
    qu = plain.unit_length(q.view(T, G, n)) * n ** -0.5
    ku = plain.unit_length(k.view(T, G, n))
    decay = torch.exp(-torch.exp(rate) * torch.nn.functional.softplus(logits[:, :H] + bias, threshold=1e9))
    outs, ends = [], []
    for a in range(H):
        o, S = plain.delta_memory(qu[:, a // (H // G)], ku[:, a // (H // G)], v.view(T, H, nv)[:, a], decay[:, a],
                                  torch.sigmoid(logits[:, H + a]), states[a] if states is not None else None)
        outs.append(plain.unit_rms(o, eps) * norm * plain.silu(gate.view(T, H, nv)[:, a]))
        ends.append(S)
    return torch.cat(outs, -1), torch.stack(ends)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("H,G,n,nv", [(4, 2, 20, 12), (3, 3, 12, 40), (6, 2, 36, 10), (4, 1, 32, 48), (2, 2, 64, 80), (2, 1, 128, 128),
                                      (1, 1, 256, 300), (1, 1, 512, 18), (5, 1, 8, 1), (2, 2, 48, 33), (3, 1, 96, 64)])
@pytest.mark.parametrize("tile", [None, 0, 1, 16, 40])
def test_memory_under_the_delta_rule(dtype, tol, H, G, n, nv, tile):
    """Portions of every size (one token, shorter and longer than the staged chunk), requests beside one
    another, slots that held another request's memory before, in both forms of the kernel; outputs and the state
    that is left."""
    from tinyserve_b200.kernels import ops
    lengths = {0: 75, 1: 41, 2: 9}
    x = {r: _memory_inputs(L, H, G, n, nv, 10 * r + 1) for r, L in lengths.items()}
    bias, rate, norm = draws(H, seed=71), draws(H, seed=72) - 2.0, (draws(nv, seed=73, scale=0.3) + 1).bfloat16().double()
    want = {r: _plain_memory(*x[r], bias, rate, norm, 1e-5, H, G, n, nv) for r in lengths}
    state = torch.full((5, H, n, nv), 99.0, device=DEV)
    slot_of, done = {0: 3, 1: 0, 2: 4}, {r: 0 for r in lengths}
    for step in [{0: 1, 1: 2}, {0: 2}, {1: 33, 2: 3, 0: 40}, {2: 1, 0: 1, 1: 1}, {0: 29, 2: 5}, {1: 5, 0: 2}]:
        parts, cu = [[x[r][i][done[r]:done[r] + k] for r, k in step.items()] for i in range(5)], [0]
        for k in step.values():
            cu.append(cu[-1] + k)
        ctx = SimpleNamespace(state_slots=torch.tensor([slot_of[r] for r in step], dtype=torch.int32, device=DEV),
                              fresh=torch.tensor([int(done[r] == 0) for r in step], dtype=torch.int32, device=DEV),
                              cu_q=torch.tensor(cu, dtype=torch.int32, device=DEV), num_requests=len(step), max_q_len=max(step.values()))
        q, k, v, gate = (on_device(torch.cat(p), dtype) for p in parts[:4])
        got = ops.delta_rule(q, k, v, gate, on_device(torch.cat(parts[4]), torch.float32), on_device(bias, torch.float32),
                             on_device(rate, torch.float32), state, ctx, H, n, nv, on_device(norm, dtype), 1e-5, dtype, q_scale=n ** -0.5,
                             qk_group=H // G, tile=tile)
        for b, (r, c) in enumerate(step.items()):
            close(got[cu[b]:cu[b + 1]], want[r][0][done[r]:done[r] + c], tol)
            done[r] += c
    assert done == lengths
    for r, slot in slot_of.items():
        close(state[slot], want[r][1], 2e-5)
    assert (state[1] == 99).all() and (state[2] == 99).all()


def test_a_long_memory_neither_drifts_nor_depends_on_the_portions():
    """1,500 tokens that hardly fade: in one portion, in portions of 37, and from the wide form token by token."""
    from tinyserve_b200.kernels import ops
    H, G, n, nv, T = 2, 1, 64, 32, 1500
    q, k, v, gate, logits = _memory_inputs(T, H, G, n, nv, 5)
    logits[:, :H] = -4.0
    bias, rate, norm = torch.zeros(H).double(), torch.full((H,), -1.0).double(), torch.ones(nv).double()
    want, end = _plain_memory(q, k, v, gate, logits, bias, rate, norm, 1e-6, H, G, n, nv)
    f = lambda t: on_device(t, torch.float32)
    for size in (T, 37, 1):
        state = torch.full((1, H, n, nv), -7.0, device=DEV)
        outs = []
        for at in range(0, T, size):
            m = min(size, T - at)
            ctx = SimpleNamespace(state_slots=torch.zeros(1, dtype=torch.int32, device=DEV), num_requests=1, max_q_len=m,
                                  fresh=torch.tensor([int(at == 0)], dtype=torch.int32, device=DEV),
                                  cu_q=torch.tensor([0, m], dtype=torch.int32, device=DEV))
            s = slice(at, at + m)
            outs.append(ops.delta_rule(f(q[s]), f(k[s]), f(v[s]), f(gate[s]), f(logits[s]), f(bias), f(rate), state, ctx, H, n, nv, f(norm),
                                       1e-6, torch.float32, q_scale=n ** -0.5, qk_group=H))
        close(torch.cat(outs), want, 5e-5)
        close(state[0], end, 5e-5)


def test_requests_without_tokens_leave_their_memory_alone():
    from tinyserve_b200.kernels import ops
    H, n, nv = 2, 32, 16
    q, k, v, gate, logits = _memory_inputs(3, H, H, n, nv, 5)
    f = lambda t: on_device(t, torch.float32)
    for tile in (0, 16):
        state = torch.randn(3, H, n, nv, device=DEV)
        before = state.clone()
        ctx = SimpleNamespace(state_slots=torch.tensor([2, 0, 1], dtype=torch.int32, device=DEV), num_requests=3, max_q_len=3,
                              fresh=torch.tensor([0, 1, 0], dtype=torch.int32, device=DEV),
                              cu_q=torch.tensor([0, 0, 3, 3], dtype=torch.int32, device=DEV))
        ops.delta_rule(f(q), f(k), f(v), f(gate), f(logits), torch.zeros(H, device=DEV), torch.zeros(H, device=DEV), state, ctx, H, n, nv,
                       torch.ones(nv, device=DEV), 1e-6, torch.float32, tile=tile)
        assert torch.equal(state[1:], before[1:]) and not torch.equal(state[0], before[0])


# ----------------------------------------------------------------------------- attention
def _pages(lengths, page, seed):
    """A block table over shuffled pages for requests of these lengths, and every token's slot."""
    g = torch.Generator().manual_seed(seed)
    need = sum(-(-n // page) for n in lengths)
    order = (torch.randperm(need + 2, generator=g) + 1).tolist()
    table = torch.zeros(len(lengths), max(-(-n // page) for n in lengths) + 2, dtype=torch.int32)
    slots = []
    for b, n in enumerate(lengths):
        for i in range(-(-n // page)):
            table[b, i] = order.pop()
        slots += [int(table[b, j // page]) * page + j % page for j in range(n)]
    return table.to(DEV), torch.tensor(slots, dtype=torch.int32, device=DEV), need + 3


def _from_cache(cache, slots, D):
    return cache.permute(0, 2, 1, 3).reshape(-1, cache.shape[1], D)[slots.long()].double().cpu()


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 4e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("H,G,n,dims,page,interleaved,scaling", [
    (6, 2, 24, 24, 8, True, (3.0, 64, 8.0, 0.5)), (3, 1, 48, 20, 16, True, None), (8, 2, 64, 32, 64, True, (4.0, 256, 16.0, 2.0)),
    (5, 5, 22, 6, 4, True, None), (4, 2, 32, 0, 16, True, None), (4, 1, 40, 16, 16, False, None), (16, 4, 128, 64, 64, True, (4.0, 64, 32.0, 1.0)),
    (40, 8, 128, 128, 16, True, None), (80, 2, 128, 16, 16, True, None)])
@pytest.mark.parametrize("tied", [True, False])
def test_joint_norm_then_rotation_with_keys_that_are_values(dtype, tol, H, G, n, dims, page, interleaved, scaling, tied):
    from tinyserve_b200.kernels import ops
    T, D = 37, -(-n // 16) * 16
    x = draws(T, (H + 2 * G) * n, seed=1, scale=2.0)
    qw, kw = (draws(H * n, seed=2, scale=0.3) + 1).bfloat16().double(), (draws(G * n, seed=3, scale=0.3) - 1).bfloat16().double()
    rot = {"base": 500.0, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    q, k, v = x[:, :H * n], x[:, H * n:(H + G) * n], x[:, (H + G) * n:]
    q_want, k_want = (plain.unit_rms(a, 1e-5) * w for a, w in ((q, qw), (k, kw)))
    turn = lambda a, heads: plain.rotate_first(a.view(T, heads, n), rot)
    if not interleaved:            # the other pairing: halves of the rotated part, made neighbours and back
        order = torch.cat([torch.stack([torch.arange(dims // 2), torch.arange(dims // 2) + dims // 2], -1).flatten(), torch.arange(dims, n)])
        turn = lambda a, heads: plain.rotate_first(a.view(T, heads, n)[..., order], rot)[..., order.argsort()]
    table, slots, pages = _pages([T], page, seed=3)
    slots = slots.clone()
    slots[5] = -1                  # a token whose keys go nowhere
    kc, vc = torch.full((2, pages, G, page, D), 30.0).to(dtype).to(DEV)
    dx = on_device(x, dtype)
    dk = dx[:, H * n:(H + G) * n]
    got = ops.joint_norm_kvwrite(dx[:, :H * n], dk, dk if tied else dx[:, (H + G) * n:], H, G, n, n, D, on_device(qw, dtype), on_device(kw, dtype),
                                 1e-5, k_cache=kc, v_cache=vc, slot_mapping=slots, page_size=page,
                                 rotary=Tables(rot, interleaved) if dims else None, positions=torch.arange(T, dtype=torch.int32, device=DEV))
    close(got[..., :n], turn(q_want, H), tol)
    assert (got[..., n:] == 0).all()
    live = [i for i in range(T) if i != 5]
    kg, vg = (_from_cache(c, slots[live], D) for c in (kc, vc))
    close(kg[..., :n], turn(k_want, G)[live], tol)
    close(vg[..., :n], (k if tied else v).view(T, G, n)[live], 1e-9)
    assert (kg[..., n:] == 0).all() and (vg[..., n:] == 0).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D,page", [(32, 16), (64, 16), (96, 16), (128, 64)])
@pytest.mark.parametrize("one_more", [False, True])
def test_keys_at_the_edges_of_the_window(dtype, D, page, one_more):
    """One key stands out: where a query sees it the output is its value, where not the output does not hold it at
    all.  Just inside and just outside the window, at page borders; in a prompt and decoded alone."""
    from tinyserve_b200.kernels import ops
    H, G, n, size = 2, 1, 300, 100
    direction, last = torch.ones(D) / math.sqrt(D), n - 1
    for marked in (0, page - 1, page, last - size - 1, last - size, last - size + 1, last - size + 2, 12 * page - 1 if page < 20 else 255, last - 1, last):
        k, v = draws(n, G, D, seed=1, scale=0.02), draws(n, G, D, seed=2)
        k[marked] = (direction * 40).bfloat16().double()
        qrow = (direction * 40).bfloat16().double()
        table, slots, pages = _pages([n], page, seed=3)
        flat = torch.zeros(2, pages * page, G, D, dtype=dtype, device=DEV)
        flat[0, slots.long()], flat[1, slots.long()] = on_device(k, dtype), on_device(v, dtype)
        kc, vc = (f.view(pages, page, G, D).permute(0, 2, 1, 3).contiguous() for f in flat)
        view = SimpleNamespace(block_table=table, page_size=page)
        seen = plain.window_mask(n, size)
        for q_len in (1, 2, 150):
            ctx = SimpleNamespace(cu_q=torch.tensor([0, q_len], dtype=torch.int32, device=DEV),
                                  kv_lens=torch.tensor([n], dtype=torch.int32, device=DEV), num_requests=1, max_q_len=q_len,
                                  max_kv_len=n, host={}, tile_cache={}, positions=torch.arange(n - q_len, n, dtype=torch.int32, device=DEV))
            out = ops.paged_attention(on_device(qrow.repeat(q_len, H, 1), dtype), kc, vc, view, ctx, 1.0, size,
                                      sinks=torch.zeros(H, device=DEV) if one_more else None)
            for place in {0, q_len // 2, q_len - 1}:
                i = n - q_len + place
                miss = (out[place, 0].double().cpu() - v[marked, 0]).abs().max().item()
                assert (miss < 4e-2) == bool(seen[i, marked]), (marked, q_len, i, miss)


def _attention_layer(kind, m, width, dtype, seed):
    """The mixer part of a layer with random weights, bound; and the same weights for the plain one."""
    from tinyserve_b200.config import config_from_dict
    from tinyserve_b200.parts.base import build_mixer
    cfg = config_from_dict({"architecture": "Ronolorn", "vocab": 8, "width": width, "streams": 1, "norm": {"eps": 1e-5},
                            "layers": [{"type": kind, "mixer": m, "mlp": None}]})
    part = build_mixer(cfg.model_spec().layers[0].mixer)
    W, bound = {}, {}
    for j, (name, spec) in enumerate(part.param_specs().items()):
        whole = torch.zeros(spec.shape, dtype=torch.float64)
        for i, src in enumerate(spec.sources):
            shape = (src.row_end - src.row_start,) + tuple(spec.shape[1:])
            t = draws(*shape, seed=seed + 31 * j + i, scale=1.5 * width ** -0.5 if len(shape) == 2 else 0.5)
            if src.name.endswith("norm.weight"):
                t = (1 + 0.3 * t).bfloat16().double()
            whole[src.row_start:src.row_end] = t
            W[src.name.removesuffix(".weight").replace(".bias", ".b")] = t
        bound[name] = on_device(whole, dtype)
    part.bind(bound)
    return part, W


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("kind,m", [
    ("attention", _window(4, 2, 16, 32, 0.4, 1e4, 8, 20)), ("attention", _window(5, 5, 20, 12, 0.3, 300.0, 20, 33, (2.0, 64, 16.0, 1.0))),
    ("attention", _window(4, 4, 64, 40, 0.125, 1e4, 16, 48)), ("attention_2", _tied(6, 2, 24, 0.4, 50.0, 24, 9, (3.0, 64, 8.0, 0.5))),
    ("attention_2", _tied(4, 1, 64, 0.2, 1e4, 32, 40)), ("attention_2", _tied(3, 3, 30, 0.3, 1e3, 0, 1))])
def test_one_attention_layer_against_the_plain_one(dtype, tol, kind, m):
    """The mixer part alone: a whole prompt, and the same prompt in two portions."""
    width, T, page = 96, 130, 16
    part, W = _attention_layer(kind, m, width, dtype, 5)
    spec = part.cache_spec()
    h = draws(T, width, seed=77)
    want = plain.attention(h, W, "", m) if kind == "attention" else plain.attention_2(h, W, "", m, 1e-5)
    runtime = SimpleNamespace(device=DEV, dtype=dtype, max_positions=256, shared={})
    for p in part.named_parts():
        p.prepare(runtime)
    from tinyserve_b200.kernels import ops
    for cuts in ([0, T], [0, 77, 79, T]):
        table, slots, pages = _pages([T], page, seed=4)
        kc, vc = torch.full((2, pages, spec.num_kv_heads, page, spec.head_dim), 5.0).to(dtype).to(DEV)
        got = []
        for a, b in zip(cuts, cuts[1:]):
            view = SimpleNamespace(block_table=table, page_size=page, slot_mapping=slots[a:b].contiguous())
            ctx = SimpleNamespace(cu_q=torch.tensor([0, b - a], dtype=torch.int32, device=DEV), kv_lens=torch.tensor([b], dtype=torch.int32, device=DEV),
                                  num_requests=1, max_q_len=b - a, max_kv_len=b, host={}, tile_cache={}, dtype=dtype,
                                  positions=torch.arange(a, b, dtype=torch.int32, device=DEV),
                                  cache=lambda i: SimpleNamespace(k=kc, v=vc, group=0), group=lambda g: view)
            got.append(ops.materialize(part.forward(on_device(h[a:b], dtype), ctx, SimpleNamespace(cache=0, writes_cache=True))))
        close(torch.cat(got), want, tol)


# ----------------------------------------------------------------------------- whole models
LENGTHS = {"P": [5, 37, 40, 70, 2, 1, 33], "Q": [1, 9, 64, 100, 31, 48], "R": [150, 130, 57, 3, 129]}


@pytest.fixture(scope="module", params=sorted(RONOLORN_TINY))
def model(request, tmp_path_factory):
    name = request.param
    folder = make_ronolorn_dir(tmp_path_factory.mktemp(f"ronolorn{name}"), name, seed=41)
    cfg, weights = plain.load_folder(folder)
    reqs = {f"r{i}": random_ids(cfg["vocab"], n, seed=300 + i) for i, n in enumerate(LENGTHS[name])}
    ref = {rid: plain.logits(cfg, weights, ids) for rid, ids in reqs.items()}
    return {"name": name, "folder": folder, "cfg": cfg, "weights": weights, "requests": reqs, "ref": ref}


def run_replay(folder, dtype, steps, out_dir, page=16, max_live=4, graphs=False):
    from tinyserve_b200.engine import replay
    runner = replay.make_runner(folder, dtype, max_live_tokens(steps, max(64, page)), block_size=page,
                                max_live=max_live, use_cuda_graphs=graphs)
    done = []
    replay.replay(runner, lines_of(steps), str(out_dir), done.append)
    assert done == [f"done {s['step']}" for s in steps]
    runner.manager.check_invariants()
    assert not runner.manager.requests and all(p.num_free == p.num_usable for p in runner.manager.pools)
    outputs = {}
    for s in steps:
        wanted = sum(len(e["want"]) for e in s["entries"])
        if wanted:
            data = np.fromfile(os.path.join(str(out_dir), f"{s['step']}.f32"), dtype="<f4")
            outputs[s["step"]] = torch.from_numpy(data.reshape(wanted, runner.model.vocab_size))
    return outputs, runner


def check(model, dtype, steps, out_dir, slack=1.0, **kw):
    outputs, runner = run_replay(model["folder"], dtype, steps, out_dir, **kw)
    for rid, out in collect_logits(steps, outputs, model["cfg"]["vocab"]).items():
        ref = model["ref"][rid.rstrip("x")]
        assert out.shape == ref.shape
        scale = ref.abs().max().item()
        err = (out.double() - ref).abs().max(-1).values / scale
        rms = (out.double() - ref).pow(2).mean(-1).sqrt() / scale
        seen = MEASURED.setdefault((model["name"], dtype), [0.0, 0.0])
        seen[0], seen[1] = max(seen[0], err.max().item()), max(seen[1], rms.max().item())
        bad = ((err > slack * TOLERANCE[dtype]) | (rms > slack * RMS_TOLERANCE[dtype])).nonzero()
        if len(bad):
            i = int(bad[0])
            raise AssertionError(f"{model['name']} {dtype}: {len(bad)} of {len(err)} places of request {rid} differ; the first is {i} "
                                 f"(error {err[i].item():.3e}, rms {rms[i].item():.3e})")
    return runner


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts(model, dtype, tmp_path):
    check(model, dtype, schedule_whole(model["requests"]), tmp_path)


def test_streams_after_every_layer(model):
    """The sum of the 32-bit streams behind every layer, read off the model's own forward pass, against the plain one's."""
    from tinyserve_b200.engine import replay
    from tinyserve_b200.engine.batch import StepEntry
    from tinyserve_b200.kernels import ops
    ids = model["requests"]["r1"]
    with torch.no_grad():
        _, want = plain.forward(model["cfg"], model["weights"], ids, keep_layers=True)
    runner = replay.make_runner(model["folder"], "float32", 256)
    seen = []

    def watched(original):
        def forward(x, residual, ctx, call):
            out = original(x, residual, ctx, call)
            X = residual.data if residual.apart else residual.data[:, None].repeat(1, residual.count, 1)
            y = ops.materialize(out.y)
            seen.append(plain.streams_out(X.transpose(0, 1).double().cpu(), y.double().cpu(), out.mix.double().cpu(), out.out.double().cpu()).sum(0))
            return out
        return forward

    for b in runner.model.blocks:
        b.forward = watched(b.forward)
    runner.manager.begin("a")
    runner.step([StepEntry("a", ids, [len(ids) - 1])])
    runner.manager.free("a")
    assert len(seen) == want.shape[0]
    for i, got in enumerate(seen):
        assert (got - want[i]).abs().max() <= 2e-5 * want[i].abs().max(), f"layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_against_token_by_token(model, dtype, tmp_path):
    """The last 32 tokens one by one; and everything but the first token one by one (the first
    tokens of a sequence, a long run of decoding)."""
    check(model, dtype, schedule_tail_decode(model["requests"], 32), tmp_path / "tail")
    longest = max(model["requests"], key=lambda r: len(model["requests"][r]))
    one = {longest: model["requests"][longest]}
    check(model, dtype, schedule_tail_decode(one, len(one[longest]) - 1), tmp_path / "all", graphs=dtype == "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_down_to_two_tokens(model, dtype, tmp_path):
    check(model, dtype, schedule_portions(model["requests"]), tmp_path / "a")
    check(model, dtype, schedule_portions(model["requests"], sizes=(2,)), tmp_path / "twos")
    check(model, dtype, schedule_portions(model["requests"], sizes=(16, 1, 15, 17, 32, 3)), tmp_path / "edges", page=8)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [0, 1])
def test_mixed_batches_reuse_pages_and_slots(model, dtype, seed, tmp_path):
    reqs = dict(model["requests"])
    more = {f"{rid}x": ids for rid, ids in reqs.items()}
    steps = schedule_mixed({**reqs, **more}, max_live=4, seed=seed)
    assert max(len(s["entries"]) for s in steps) >= 3
    assert any(len({len(e["tokens"]) == 1 for e in s["entries"]}) == 2 for s in steps), "portions beside single tokens"
    runner = check(model, dtype, steps, tmp_path, max_live=4)
    assert len(reqs) + len(more) > runner.manager.slots.num_slots == 4, "slots are used again"
    total = sum(-(-len(i) // 16) for i in {**reqs, **more}.values())
    assert total > runner.manager.pools[0].num_usable, "the pool is too small to avoid reuse"


def test_batch_of_unequal_requests_equals_each_alone(model, tmp_path):
    reqs = model["requests"]
    together = [{"step": 0, "entries": [{"id": r, "tokens": ids, "want": list(range(len(ids)))} for r, ids in reqs.items()],
                 "end": list(reqs)}]
    out_a, _ = run_replay(model["folder"], "float32", together, tmp_path / "a", max_live=len(reqs))
    out_b, _ = run_replay(model["folder"], "float32", schedule_whole(reqs), tmp_path / "b")
    a = collect_logits(together, out_a, model["cfg"]["vocab"])
    b = collect_logits(schedule_whole(reqs), out_b, model["cfg"]["vocab"])
    for rid in reqs:
        # (the attention kernel cuts a request's keys into ranges by how full the batch is, and requests of a few tokens
        # take another form of the memory's kernel: the order of the sums, not what is summed, depends on the batch)
        assert (a[rid] - b[rid]).abs().max() <= 1e-5 * b[rid].abs().max()


@pytest.mark.parametrize("seed", range(16))
def test_drawn_configurations(seed, tmp_path):
    """Configurations drawn from a seed (odd head sizes, head counts, taps, streams, orders, layers without
    feed-forward, windows, rotation over all, a part or none of a head): whole prompts, portions and a mixed batch
    against the plain implementation."""
    from tinyserve_b200.config import config_from_dict
    from tinyserve_b200.weights import write_random_model
    raw = random_ronolorn_config_dict(seed)
    folder = decisive(write_random_model(config_from_dict(raw), str(tmp_path / "model"), seed=seed), seed, sharp=4.0)
    cfg, weights = plain.load_folder(folder)
    reqs = {f"r{i}": random_ids(cfg["vocab"], n, seed=700 + 10 * seed + i) for i, n in enumerate((37, 5, 66, 1))}
    ref = {rid: plain.logits(cfg, weights, ids) for rid, ids in reqs.items()}
    model = {"name": f"drawn{seed}", "folder": folder, "cfg": cfg, "requests": reqs, "ref": ref}
    check(model, "float32", schedule_whole(reqs), tmp_path / "whole", slack=2.0)
    check(model, "float32", schedule_portions(reqs, sizes=(17, 2, 16, 1, 3)), tmp_path / "portions", slack=2.0)
    check(model, "float32", schedule_mixed(reqs, max_live=3, seed=seed), tmp_path / "mixed", slack=2.0, max_live=3)
    check(model, "bfloat16", schedule_mixed(reqs, max_live=3, seed=seed), tmp_path / "mixed16", slack=2.0, max_live=3)


# ----------------------------------------------------------------------------- weights that show a fault
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["P", "R"])
def test_far_tokens_windows_sinks_and_what_the_memory_holds(name, dtype, tmp_path):
    """Sharp attention (a key at a window's or a page's border or a wrong position moves the logits) and memories that
    last (a far token, a lost state, a decay or a write strength that is left out move them too); long prompts, long
    decoding, portions, mixed."""
    folder = make_ronolorn_dir(tmp_path / "base", name, seed=43, sharp=12.0)
    cfg, weights = plain.load_folder(folder)
    ids = random_ids(cfg["vocab"], 210, seed=7)
    reqs = {"far": ids, "near": ids[:70]}
    ref = {rid: plain.logits(cfg, weights, t) for rid, t in reqs.items()}
    moved = lambda c, w, t=ids: (plain.logits(c, w, t) - ref["far"]).abs().max() / ref["far"].abs().max()
    other = list(ids)
    other[100] = (ids[100] + 1) % cfg["vocab"]
    changed = (plain.logits(cfg, weights, other) - ref["far"]).abs().max(-1).values / ref["far"].abs().max()
    assert changed[:100].max() < 1e-12 and changed[180:].max() > 1e-3, "a far token matters here, through the memory"
    for part, value in ((".dt_bias", -30.0), (".q.b", 0.0), (".v.b", 0.0), (".o.b", 0.0), (".k.norm", 1.0), (".mix.norm", 1.0), ("hc1.in", 1.0),
                        ("hc2.out", 1.0), (".mix.b", 0.0), (".mix.a", 0.0)):
        w2 = {k: (torch.full_like(v, value) if k.endswith(part) else v) for k, v in weights.items()}
        assert moved(cfg, w2) > 3e-3, f"{part} matters"
    turned = {k: (v.T if k.endswith((".hc1.mix", ".hc2.mix")) else v) for k, v in weights.items()}
    assert moved(cfg, turned) > 1e-2, "the direction of the mixing matters"
    newest = {k: (torch.cat([torch.zeros_like(v[:, :-1]), v[:, -1:]], -1) if k.endswith(".conv") else v) for k, v in weights.items()}
    assert moved(cfg, newest) > 1e-2, "the older taps matter"
    for kind in ("attention", "attention_2"):
        for by in (-1, 1):
            c2 = {**cfg, "layers": [{**l, "mixer": {**l["mixer"], "mask": {"size": l["mixer"]["mask"]["size"] + by}}} if l["type"] == kind else l
                                    for l in cfg["layers"]]}
            assert moved(c2, weights) > 3e-3, f"{kind}: a window off by {by} shows"
    keep, plain.softmax_over = plain.softmax_over, lambda s, seen, one_more: keep(s, seen, False)
    try:
        assert moved(cfg, weights) > 3e-3, "the one in the softmax sum matters"
    finally:
        plain.softmax_over = keep
    model = {"name": name + "sharp", "folder": folder, "cfg": cfg, "requests": reqs, "ref": ref}
    slack = 2.0 if dtype == "float32" else 3.0
    check(model, dtype, schedule_whole(reqs), tmp_path / "whole", slack=slack)
    check(model, dtype, schedule_tail_decode(reqs, 120), tmp_path / "tail", slack=slack)
    check(model, dtype, schedule_portions(reqs, sizes=(63, 2, 1, 64, 5, 16, 15)), tmp_path / "portions", slack=slack)
    check(model, dtype, schedule_mixed({**reqs, "farx": ids, "nearx": ids[:70]}, max_live=3, seed=5), tmp_path / "mixed",
          slack=slack, max_live=3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_head_sizes_of_real_models(dtype, tmp_path):
    """Heads of 128 and of 64, memories of 128 x 128, a width whose few rows are normed over a cluster, pages of 64: the
    kernels that real layer sizes reach (tcgen05 prefill, decode by whole pages, products cut along K), prompts longer
    than two key tiles of any kernel."""
    from tinyserve_b200.config import config_from_dict
    from tinyserve_b200.weights import write_random_model
    raw = {"architecture": "Ronolorn", "vocab": 1000, "width": 1024, "streams": 4, "norm": {"eps": 1e-6}, "embedding": {"scale": 3.0}, "layers": [
        {"type": "delta", "mlp": _dense(2048), "mixer": _delta(8, 4, 128, 128, 4)},
        {"type": "attention", "mlp": _dense(1024), "mixer": _window(8, 2, 128, 96, 0.09, 1e6, 64, 200)},
        {"type": "attention_2", "mlp": _dense(1536), "mixer": _tied(8, 2, 128, 0.09, 1e5, 128, 130, (8.0, 512, 32.0, 1.0))},
        {"type": "attention_2", "mlp": None, "mixer": _tied(8, 1, 64, 0.125, 1e4, 32, 300)},
    ]}
    folder = decisive(write_random_model(config_from_dict(raw), str(tmp_path / "model"), seed=5), 5, sharp=2.0)
    cfg, weights = plain.load_folder(folder)
    reqs = {"a": random_ids(1000, 420, seed=1), "b": random_ids(1000, 130, seed=2)}
    ref = {rid: plain.logits(cfg, weights, ids) for rid, ids in reqs.items()}
    model = {"name": "real", "folder": folder, "cfg": cfg, "requests": reqs, "ref": ref}
    check(model, dtype, schedule_tail_decode(reqs, 40), tmp_path / "tail", page=64)
    check(model, dtype, schedule_mixed(reqs, max_live=2, seed=1, chunk_sizes=(200, 2, 129, 64, 1)), tmp_path / "mixed", max_live=2)


def test_launches_of_a_step_of_few_tokens(tmp_path):
    """A decode step of a few requests: what lies between two sub-layers is one launch, a product hands it its partial
    tiles, and the feed-forward's activation is in its first product."""
    from tinyserve_b200.engine import replay
    from tinyserve_b200.engine.batch import StepEntry
    from tinyserve_b200.kernels import ops
    runner = replay.make_runner(make_ronolorn_dir(tmp_path, "R", seed=1), "bfloat16", 256)
    for rid in ("a", "b"):
        runner.manager.begin(rid)
        runner.step([StepEntry(rid, [1, 2, 3, 4, 5], [])])
    runner.cfg.check_indices = False         # (the index check has launches of its own)
    before = ops.launch_count()
    runner.step([StepEntry("a", [6], [0]), StepEntry("b", [7], [0])])
    # block tables 2 per cache group, embedding, last norm, logits; per layer: norm, inputs, heads or convolution, attention
    # or memory, output, norm, up, down
    assert ops.launch_count() - before <= 2 * 2 + 3 + 4 * 8, ops.launch_count() - before


# ----------------------------------------------------------------------------- the entry point
def test_greedy_generation_through_the_scheduler(tmp_path):
    """Five prompts of unequal length through LLM.generate with three slots and at most 48 tokens a
    step (prompts in portions beside decoding requests, slots and pages used again)."""
    from tinyserve_b200 import LLM, SamplingParams
    folder = make_ronolorn_dir(tmp_path, "P", seed=44)
    cfg, weights = plain.load_folder(folder)
    prompts = [random_ids(cfg["vocab"], n, seed=500 + n) for n in (3, 60, 17, 1, 90)]
    params = SamplingParams(temperature=0.0, max_tokens=12, repetition_penalty=1.0, ignore_eos=True)
    llm = LLM(folder, dtype="float32", max_model_len=128, block_size=16, max_num_seqs=3, max_num_batched_tokens=48,
              num_blocks=20, use_cuda_graphs=False)
    outs = llm.generate(prompts, params)
    for prompt, out in zip(prompts, outs):
        want, gaps = plain.greedy(cfg, weights, prompt, 12)
        assert out.finished and len(out.token_ids) == 12
        for j, (a, b, gap) in enumerate(zip(out.token_ids, want, gaps)):
            if gap < 1e-3:
                break                        # a near tie: either side is a right answer, the rest differs
            assert a == b, (len(prompt), j)
    outs16 = LLM(folder, dtype="bfloat16", max_model_len=128, block_size=16, max_num_seqs=3,
                 max_num_batched_tokens=48, num_blocks=20, use_cuda_graphs=True).generate(prompts, params)
    for prompt, out in zip(prompts, outs16):
        ids = list(prompt)
        for tok in out.token_ids:
            row = plain.logits(cfg, weights, ids)[-1]
            assert row[tok] >= row.max() - 0.05 * row.abs().max()
            ids.append(tok)


def test_programs_replay_and_generate(tmp_path):
    """bin/trace_run and ``python -m tinyserve_b200 generate`` as programs on a Ronolorn folder: the
    architecture is chosen by config.json; stdin to files, 'done' lines, exit code 0; greedy tokens."""
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    folder = make_ronolorn_dir(tmp_path / "m", "Q", seed=2)
    cfg, weights = plain.load_folder(folder)
    reqs = {"p": random_ids(cfg["vocab"], 45, seed=1), "q": random_ids(cfg["vocab"], 30, seed=2)}
    steps = schedule_mixed(reqs, max_live=2, seed=0)
    out = tmp_path / "out"
    proc = subprocess.run(
        [sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
         "--out", str(out), "--max-tokens", str(max_live_tokens(steps))],
        input="\n".join(lines_of(steps)) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.split("\n")[:-1] == [f"done {s['step']}" for s in steps]
    outputs = {}
    for s in steps:
        wanted = sum(len(e["want"]) for e in s["entries"])
        outputs[s["step"]] = torch.from_numpy(np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(wanted, cfg["vocab"]))
    got = collect_logits(steps, outputs, cfg["vocab"])
    for rid, ids in reqs.items():
        ref = plain.logits(cfg, weights, ids)
        assert (got[rid].double() - ref).abs().max().item() < TOLERANCE["float32"] * ref.abs().max().item()
    prompt = reqs["q"][:9]
    proc = subprocess.run(
        [sys.executable, "-m", "tinyserve_b200", "generate", "--model", folder, "--dtype", "float32", "--prompt-ids",
         ",".join(map(str, prompt)), "--max-tokens", "5", "--repetition-penalty", "1.0", "--ignore-eos", "--max-model-len", "64",
         "--max-num-seqs", "2", "--max-num-batched-tokens", "32", "--num-blocks", "16", "--block-size", "16"],
        capture_output=True, text=True, timeout=600, cwd=root)
    assert proc.returncode == 0, proc.stderr[-2000:]
    tokens = [int(t) for t in proc.stdout.strip().split("\n")[-1].split()]
    want, gaps = plain.greedy(cfg, weights, prompt, 5)
    for a, b, gap in zip(tokens, want, gaps):
        if gap < 1e-3:
            break
        assert a == b, (tokens, want)
    assert len(tokens) == 5


def test_measured_differences_are_reported():
    print({k: (f"{v[0]:.2e}", f"{v[1]:.2e}") for k, v in sorted(MEASURED.items())})
