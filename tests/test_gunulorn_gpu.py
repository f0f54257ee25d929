"""Gunulorn on the device against the plain implementation (tests/plain_gunulorn.py): each
mechanism alone through its kernel, then whole models through the step function: whole prompts,
prompts against token-by-token decoding, portions down to two tokens, mixed batches with pages and
slots that are used again, far keys and keys at page and window borders that the weights are made to
show, long decoding, other sizes, and greedy generation through the entry point."""
import json
import math
import os
from types import SimpleNamespace

import numpy as np
import pytest
import torch
from safetensors.torch import load_file, save_file

import plain_gunulorn as plain
from gunulorn_configs import (GUNULORN_TINY, _conv, _dense, _moe, _turned, decisive, make_gunulorn_dir,
                              random_gunulorn_config_dict)
from helpers import (collect_logits, lines_of, max_live_tokens, random_ids, schedule_mixed, schedule_portions,
                     schedule_tail_decode, schedule_whole)

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
# Largest |logit difference|, and largest root-mean-square difference over the vocabulary at one
# position, over the largest plain |logit|.  float32: 32-bit sums against float64, the sharp test of
# every schedule.  bfloat16: products and activations rounded to 8 bits through tiny random layers;
# it catches a kernel that is wrong, not one that rounds elsewhere.
TOLERANCE = {"float32": 5e-5, "bfloat16": 2e-1}
RMS_TOLERANCE = {"float32": 1.7e-5, "bfloat16": 6e-2}
MEASURED = {}


def draws(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).bfloat16().double()


def on_device(x, dtype):
    return x.to(dtype).to(DEV).contiguous()


class Tables:
    """Rotary tables of neighbouring pairs over ``dims`` elements."""

    def __init__(self, base, dims, n=1024):
        from tinyserve_b200.parts.rotary import Rotary
        self.rotary_dim, self.interleaved = dims, True
        self.cos, self.sin = (t.to(DEV) for t in Rotary.tables(dims, float(base), n))


def close(got, want, tol):
    err = (got.double().cpu() - want).abs().max().item()
    assert err <= tol * max(want.abs().max().item(), 1e-30), (err, want.abs().max().item())


# ----------------------------------------------------------------------------- two branches on one stream
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("T,n", [(23, 41), (23, 40), (7, 200), (600, 1000), (4, 2048), (3, 5000), (40, 2048), (64, 8192),
                                 (3, 12000), (530, 1536), (513, 4096), (2, 20000)])
def test_two_norms_of_one_stream_and_everything_that_joins_it(dtype, tol, T, n):
    """Two tensors, a multiple of a row per token and a vector for all rows join the 32-bit stream; one
    kernel writes both norms; chosen rows leave the stream alone."""
    from tinyserve_b200.kernels import ops
    x1, x2, rows_src, res = draws(T, n, seed=1), draws(T, n, seed=2), draws(T, n, seed=3), draws(T, n, seed=4, scale=2.0)
    factor = draws(T, seed=5)
    w1, w2 = draws(n, seed=6, scale=0.3) + 1, draws(n, seed=7, scale=0.3) - 1
    w1, w2 = w1.bfloat16().double(), w2.bfloat16().double()
    total = res + x1 + x2 + factor[:, None] * rows_src
    residual = on_device(res, torch.float32)
    fed = ops.RowsAdded(on_device(x2, dtype), on_device(factor, torch.float32), on_device(rows_src, dtype))
    a, b = ops.branch_norm(ops.BranchSum(on_device(x1, dtype), fed), residual, on_device(w1, dtype), on_device(w2, dtype), 1e-5, dtype)
    close(residual, total, 1e-6)
    close(a, plain.norm(total, w1, 1e-5), tol)
    close(b, plain.norm(total, w2, 1e-5), tol)
    pick = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device=DEV)
    before = residual.clone()
    only, none = ops.branch_norm(ops.BranchSum(on_device(x1, dtype), None), residual, on_device(w1, dtype), None, 1e-5, dtype, rows=pick)
    assert none is None and torch.equal(residual, before)
    close(only, plain.norm(total + x1, w1, 1e-5)[pick.cpu().long()], tol)
    close(ops.materialize(fed), x2 + factor[:, None] * rows_src, tol)
    close(ops.materialize(ops.BranchSum(on_device(x1, dtype), fed)), x1 + x2 + factor[:, None] * rows_src, 2 * tol)


@pytest.mark.parametrize("M,N,K1,K2", [(1, 2048, 512, 1024), (8, 2048, 1024, 5632), (16, 512, 72, 4096), (13, 1000, 200, 88),
                                       (5, 4096, 4096, 64), (33, 2048, 512, 1024), (64, 1024, 136, 2048), (20, 384, 64, 64)])
@pytest.mark.parametrize("bias", [False, True])
@pytest.mark.parametrize("second", [False, True])
def test_output_products_of_both_branches_in_one_launch(M, N, K1, K2, bias, second):
    """out = x1 W1^T + x2 W2^T (+ bias) with the residual add and two norm weights behind it: inside the
    product for up to 16 tokens (rows without their norm factor), through partial tiles above."""
    from tinyserve_b200.kernels import ops
    x1, w1, x2, w2 = draws(M, K1, seed=1), draws(N, K1, seed=2, scale=K1 ** -0.5), draws(M, K2, seed=3), draws(N, K2, seed=4, scale=K2 ** -0.5)
    bvec, res, src, factor = draws(N, seed=5), draws(M, N, seed=6), draws(M, N, seed=7), draws(M, seed=8)
    n1, n2 = (draws(N, seed=9, scale=0.2) + 1).bfloat16().double(), (draws(N, seed=10, scale=0.2) + 1).bfloat16().double()
    d = lambda t: on_device(t, torch.bfloat16)
    a = ops.linear(d(x1), d(w1), allow_pending=True)
    b = ops.linear(d(x2), d(w2), d(bvec) if bias else None, allow_pending=True)
    assert isinstance(a, ops.PendingProduct) and isinstance(b, ops.PendingProduct)
    b = ops.RowsAdded(b, on_device(factor, torch.float32), d(src))
    total = res + x1 @ w1.T
    if second:
        total = total + x2 @ w2.T + (bvec if bias else 0) + factor[:, None] * src
    residual = on_device(res, torch.float32)
    before = ops.launch_count()
    h1, h2 = ops.branch_norm(ops.BranchSum(a, b if second else None), residual, d(n1), d(n2), 1e-5, torch.bfloat16, scaled_ok=True)
    # (partial tiles are summed in 32-bit; a product that is not cut is rounded once)
    close(residual, total, 1e-5 if M <= 16 else 6e-3)
    assert isinstance(h1, ops.ScaledRows) == (M <= 16) and ops.launch_count() - before == (1 if M <= 16 else 2)
    close(ops.materialize(h1), plain.norm(total, n1, 1e-5), 1.2e-2)
    close(ops.materialize(h2), plain.norm(total, n2, 1e-5), 1.2e-2)


@pytest.mark.parametrize("M,K,Ns", [(8, 2048, (3072, 40, 5632)), (16, 64, (100, 7)), (1, 1024, (6144, 16, 2816)), (33, 256, (130, 130)),
                                    (64, 512, (1000, 13, 2000)), (5, 4096, (128,)), (3, 512, (64, 64, 64, 64))])
@pytest.mark.parametrize("scaled", [False, True])
def test_input_products_of_both_branches_in_one_launch(M, K, Ns, scaled):
    """Products of two inputs beside one another, 16-bit and 32-bit outputs, with and without biases, from
    finished rows and from rows that lack their norm factor."""
    from tinyserve_b200.kernels import ops
    d = lambda t: on_device(t, torch.bfloat16)
    xs = [draws(M, K, seed=1, scale=2.0), draws(M, K, seed=2)]
    ws = [draws(n, K, seed=10 + i, scale=K ** -0.5) for i, n in enumerate(Ns)]
    bs = [draws(n, seed=20 + i) if i % 2 == 0 else None for i, n in enumerate(Ns)]
    rstd = torch.ones(M, 1, dtype=torch.float64)
    hs = [d(x) for x in xs]
    if scaled and M <= 16:
        v = draws(M, K, seed=3, scale=3.0)
        sums = torch.zeros(-(-K // 128), 16)
        for t in range(sums.shape[0]):
            sums[t, :M] = v[:, 128 * t:128 * (t + 1)].pow(2).sum(-1).float()
        sums = sums.to(DEV)
        hs = [ops.ScaledRows(h, sums, sums.shape[0], 1e-5) for h in hs]
        rstd = 1 / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + 1e-5)
    groups = [(hs[0], [ops.InputProduct(d(ws[0]), d(bs[0]))]),
              (hs[1], [ops.InputProduct(d(w), d(b) if b is not None else None, out_float32=i % 2 == 0)
                       for i, (w, b) in enumerate(zip(ws[1:], bs[1:]))])]
    before = ops.launch_count()
    first, second = ops.linear_beside(groups)
    launches = ops.launch_count() - before
    if 1 < len(Ns) <= ops.BESIDE_MAX_PRODUCTS:
        assert launches == 1
    close(ops.materialize(first[0]), xs[0] @ ws[0].T * rstd + bs[0], 1e-2)
    for i, (w, b, got) in enumerate(zip(ws[1:], bs[1:], second)):
        assert got.dtype == (torch.float32 if i % 2 == 0 else torch.bfloat16)
        close(got, xs[1] @ w.T * rstd + (b if b is not None else 0), 2e-5 if i % 2 == 0 else 1e-2)


# ----------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("T,ff", [(1, 72), (9, 40), (3, 37), (70, 5632), (600, 1000), (513, 11264), (2, 20000), (600, 64)])
def test_polynomial_of_normed_powers(dtype, tol, T, ff):
    from tinyserve_b200.kernels import ops
    z = draws(T, ff, seed=1, scale=1.7)
    z[0, ff // 2] = 40.0             # one value that carries its row's higher powers
    for coef in ([0.5, -1.25, 2.0, 0.375], [0.0, 0.0, 1.0, 0.0], [1.0, 0.0, 0.0, 0.0], [0.0, 1.0, 0.0, -3.0]):
        c = torch.tensor(coef, dtype=torch.float64)
        close(ops.poly_norm(on_device(z, dtype), on_device(c, dtype), 1e-5), plain.poly_norm(z, c, 1e-5), tol)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("T,width,ff", [(1, 64, 72), (9, 128, 192), (70, 256, 384), (300, 96, 104), (5, 64, 37)])
def test_dense_feed_forward_against_the_plain_one(dtype, tol, T, width, ff):
    from tinyserve_b200.kernels import ops
    from tinyserve_b200.parts.mlp import PolyNormMLP
    part = PolyNormMLP(width, ff, 1e-5, names={"up": "up", "down": "down"})
    h = draws(T, width, seed=1)
    W = {"up": draws(ff, width, seed=2, scale=width ** -0.5), "up.b": draws(ff, seed=3), "down": draws(width, ff, seed=4, scale=ff ** -0.5),
         "down.b": draws(width, seed=5), "act": torch.tensor([0.75, -1.5, 0.5, 0.25], dtype=torch.float64)}
    part.bind({"up_proj.weight": on_device(W["up"], dtype), "up_proj.bias": on_device(W["up.b"], dtype),
               "down_proj.weight": on_device(W["down"], dtype), "down_proj.bias": on_device(W["down.b"], dtype), "act": on_device(W["act"], dtype)})
    close(ops.materialize(part.forward(on_device(h, dtype), None)), plain.dense_ff(h, W, "", 1e-5), tol)


@pytest.mark.parametrize("T,E,identity,top", [(1, 5, 0, 2), (50, 6, 3, 4), (9, 1, 4, 1), (300, 40, 24, 8), (7, 3, 2, 5)])
def test_router_of_corrected_softmax_scores(T, E, identity, top):
    from tinyserve_b200.kernels import ops
    R = E + identity
    z, corr = draws(T, R, seed=1, scale=2.0), draws(R, seed=2, scale=0.4)
    gates = ops.moe_route_scored(on_device(z, torch.float32), on_device(corr, torch.float32), top, softmax=True, renormalize=True,
                                 identity=identity)
    gates, rest = gates if identity else (gates, None)
    idx, w = plain.route(z, {"router": torch.eye(R, dtype=torch.float64), "correction": corr}, "", {"top": top})
    want = torch.zeros(T, R, dtype=torch.float64).scatter(1, idx, w)
    assert (torch.softmax(z, -1).topk(top, -1).indices.sort(-1).values != idx.sort(-1).values).any() or top == R or T < 5, "the correction moves a choice"
    close(gates, want[:, :E], 3e-6)
    if identity:
        close(rest, want[:, E:].sum(-1), 3e-6)


def _experts_part(width, ff, E, identity, top, dtype, seed=0):
    from tinyserve_b200.parts.moe import MixtureOfExperts
    W = {"router": draws(E + identity, width, seed=seed + 1, scale=1.5 * width ** -0.5), "correction": draws(E + identity, seed=seed + 2, scale=0.2)}
    for e in range(E):
        for i, (name, shape) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))):
            W[f"e{e}.{name}"] = draws(*shape, seed=seed + 10 * e + i + 3, scale=shape[1] ** -0.5)
    part = MixtureOfExperts(width, ff, E, top, activation="silu_gated", router="softmax_corrected", identity=identity)
    bound = {}
    for name, spec in part.param_specs().items():
        rows = torch.zeros(spec.shape, dtype=torch.float64)
        for src in (spec.sources or ()):
            rows[src.row_start:src.row_end] = W[src.name.removesuffix(".weight")]
        bound[name] = on_device(rows, dtype)
    part.bind(bound)
    return part, W


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("T,width,ff,E,identity,top", [(1, 64, 24, 3, 1, 4), (9, 128, 40, 6, 3, 2), (70, 64, 32, 2, 3, 1), (300, 96, 40, 8, 4, 3),
                                                      (600, 128, 64, 5, 0, 2), (520, 64, 16, 1, 5, 1), (300, 64, 24, 40, 2, 4)])
def test_experts_with_identity_experts_against_the_plain_ones(dtype, tol, T, width, ff, E, identity, top):
    from tinyserve_b200.kernels import ops
    part, W = _experts_part(width, ff, E, identity, top, dtype)
    h = draws(T, width, seed=99)
    want = plain.experts(h, W, "", {"router": {"experts": E, "identity": identity, "top": top}})
    got = ops.materialize(part.forward(on_device(h, dtype), None))
    # (in bfloat16 a token whose choice scores are a rounding apart may take another expert: one row in fifty may differ)
    err = (got.double().cpu() - want).abs().max(-1).values
    assert int((err > tol * want.abs().max()).sum()) <= (T // 50 if dtype == torch.bfloat16 else 0)
    if dtype == torch.bfloat16 and T >= ops.MOE_GROUPED_MIN_TOKENS and top < E:
        keep, ops.MOE_GROUPED_MIN_TOKENS = ops.MOE_GROUPED_MIN_TOKENS, 10 ** 9
        try:
            dense = ops.materialize(part.forward(on_device(h, dtype), None))
        finally:
            ops.MOE_GROUPED_MIN_TOKENS = keep
        assert (got.double() - dense.double()).abs().max() <= tol * want.abs().max(), "both forms route alike and agree to a rounding"


@pytest.mark.parametrize("T", [1, 7, 16])
def test_experts_on_rows_that_lack_their_norm_factor(T):
    """The identity experts' input is the normed row: its missing factor joins their weight."""
    from tinyserve_b200.kernels import ops
    width, ff, E, identity, top = 256, 32, 3, 5, 4
    part, W = _experts_part(width, ff, E, identity, top, torch.bfloat16, seed=5)
    v, w = draws(T, width, seed=1, scale=5.0), (draws(width, seed=2, scale=0.2) + 1).bfloat16().double()
    residual = on_device(v, torch.float32)
    x, wx = draws(T, 64, seed=3), draws(width, 64, seed=4, scale=0.125)
    pending = ops.linear(on_device(x, torch.bfloat16), on_device(wx, torch.bfloat16), allow_pending=True)
    rows, _ = ops.branch_norm(pending, residual, on_device(w, torch.bfloat16), None, 1e-6, torch.bfloat16, scaled_ok=True)
    assert isinstance(rows, ops.ScaledRows)
    h = plain.norm(v + x @ wx.T, w, 1e-6)
    (projected,) = ops.linear_beside([(rows, part.input_products())])
    got = ops.materialize(part.forward_projected(projected, rows, None))
    want = plain.experts(h, W, "", {"router": {"experts": E, "identity": identity, "top": top}})
    close(got, want, 3e-2)


def test_logits_are_scaled_then_capped():
    from tinyserve_b200.kernels import ops
    y = draws(9, 501, seed=1, scale=20.0)
    close(ops.softcap_(on_device(y, torch.float32), 7.5, 0.3), 7.5 * torch.tanh(y * 0.3 / 7.5), 1e-6)
    close(ops.softcap_(on_device(y, torch.float32), 0.0, 0.3), y * 0.3, 1e-6)


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


def _backends(dtype, D, page):
    from tinyserve_b200.kernels import ops
    return {"tcgen05": ["tcgen05", "mma", "simt"], "mma": ["mma", "simt"], "simt": ["simt"]}[ops.attention_backend(dtype, D, page)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("H,G,n,nv", [(4, 2, 24, 16), (3, 1, 7, 5), (2, 2, 16, 40), (6, 3, 64, 64), (1, 1, 12, 12)])
@pytest.mark.parametrize("taps", [1, 2, 4, 8])
@pytest.mark.parametrize("reader", [False, True])
def test_convolved_heads_and_their_state(dtype, tol, H, G, n, nv, taps, reader):
    """The convolution over portions of every size (down to one token, longer and shorter than the taps and
    the kernel's tile), requests beside one another, slots that held another request's rows before:
    query rows times the heads' factors, keys and values in the cache, zeros behind every head."""
    from tinyserve_b200.kernels import ops
    D, page = -(-max(n, nv) // 16) * 16, 8
    C = H * n if reader else H * n + G * (n + nv)
    lengths = {0: 75, 1: 41, 2: 9}
    u = {r: draws(L, C, seed=10 + r) for r, L in lengths.items()}
    w = draws(C, taps, seed=1)
    temp = draws(H, seed=2)
    want = {r: plain.past_convolution(x, w) for r, x in u.items()}
    table, slots, pages = _pages([lengths[r] for r in sorted(lengths)], page, seed=3)
    start = {0: 0, 1: 75, 2: 116}
    kc, vc = torch.full((2, pages, G, page, D), 30.0).to(dtype).to(DEV)
    state = torch.full((5, max(1, taps - 1), C), 99.0, device=DEV)
    slot_of = {0: 3, 1: 0, 2: 4}
    done = {r: 0 for r in lengths}
    steps = [{0: 1, 1: 2}, {0: 2}, {1: 33, 2: 3, 0: 40}, {2: 1, 0: 1, 1: 1}, {0: 29, 2: 5}, {1: 5, 0: 2}]
    for step in steps:
        rows, where, cu = [], [], [0]
        for r, k in step.items():
            rows.append(u[r][done[r]:done[r] + k])
            where.append(slots[start[r] + done[r]:start[r] + done[r] + k])
            cu.append(cu[-1] + k)
        ctx = SimpleNamespace(state_slots=torch.tensor([slot_of[r] for r in step], dtype=torch.int32, device=DEV),
                              fresh=torch.tensor([int(done[r] == 0) for r in step], dtype=torch.int32, device=DEV),
                              cu_q=torch.tensor(cu, dtype=torch.int32, device=DEV), num_requests=len(step), max_q_len=max(step.values()))
        q = ops.conv_heads_kvwrite(on_device(torch.cat(rows), dtype), ctx, H, G, n, nv, D, weight=on_device(w.T, dtype),
                                   state=state if taps > 1 else None, factor=on_device(temp, dtype), k_cache=kc, v_cache=vc,
                                   slot_mapping=None if reader else torch.cat(where), page_size=page)
        for b, (r, k) in enumerate(step.items()):
            y = want[r][done[r]:done[r] + k]
            got = q[cu[b]:cu[b + 1]]
            close(got[..., :n], y[:, :H * n].view(k, H, n) * temp[:, None], tol)
            assert (got[..., n:] == 0).all()
            done[r] += k
    assert done == lengths
    if reader:
        assert (kc == 30).all() and (vc == 30).all()
        return
    for r, L in lengths.items():
        at = slots[start[r]:start[r] + L].long().cpu()
        k_got = kc.permute(0, 2, 1, 3).reshape(-1, G, D).cpu()[at]
        v_got = vc.permute(0, 2, 1, 3).reshape(-1, G, D).cpu()[at]
        close(k_got[..., :n], want[r][:, H * n:(H + G) * n].view(L, G, n), tol)
        close(v_got[..., :nv], want[r][:, (H + G) * n:].view(L, G, nv), tol)
        assert (k_got[..., n:] == 0).all() and (v_got[..., nv:] == 0).all()


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("H,G,n,nv,dims,page", [(4, 2, 16, 32, 8, 8), (3, 1, 48, 16, 48, 16), (5, 5, 20, 10, 0, 4), (6, 3, 22, 40, 6, 16),
                                                (4, 1, 64, 64, 32, 32), (2, 1, 128, 128, 64, 64), (2, 2, 32, 128, 16, 16), (20, 1, 32, 64, 32, 32)])
@pytest.mark.parametrize("size,keep_first", [(40, 3), (1, 0), (17, 70), (500, 4)])
def test_turned_values_in_a_window(dtype, tol, H, G, n, nv, dims, page, size, keep_first):
    """Rotation of a part of q and k and of whole values, the window beside the first tokens, one more in
    every softmax sum, outputs turned back: a whole prompt, single tokens, a portion after a prefix, two
    tokens and a request of one token, on every attention kernel that takes the head size, with and
    without key ranges."""
    from tinyserve_b200.kernels import ops
    kv_lens, q_lens = [70, 24, 97, 9, 350, 1, 300], [70, 1, 29, 2, 1, 1, 150]
    rot, scale = {"base": 100.0, "dims": dims}, 1.2 / math.sqrt(n)
    width = (H + G) * n + G * nv
    T = sum(kv_lens)
    h = draws(T, width, seed=11)
    eye = torch.eye(width, dtype=torch.float64)
    W = {"q": eye[:H * n], "k": eye[H * n:(H + G) * n], "v": eye[(H + G) * n:], "o": torch.eye(H * nv, dtype=torch.float64)}
    m = {"heads": H, "kv_heads": G, "dim": n, "vdim": nv, "scale": scale, "rot": rot, "mask": {"size": size, "keep_first": keep_first}}
    want, at = [], 0
    for kv in kv_lens:
        want.append(plain.window_attention(h[at:at + kv], W, "", m))
        at += kv
    D = -(-max(n, nv) // 16) * 16
    table, slots, pages = _pages(kv_lens, page, seed=2)
    kc, vc = (torch.full((pages, G, page, D), 30.0).to(dtype).to(DEV) for _ in range(2))
    pos = torch.cat([torch.arange(kv) for kv in kv_lens]).to(torch.int32).to(DEV)
    x = on_device(h, dtype)
    turn = Tables(rot["base"], nv)
    rows = ops.rope_unit_kvwrite(x[:, :H * n], x[:, H * n:(H + G) * n], x[:, (H + G) * n:], pos, H, G, n, nv, D,
                                 rotary=Tables(rot["base"], dims) if dims else None, k_cache=kc, v_cache=vc, slot_mapping=slots,
                                 page_size=page, value_rotary=turn)
    alone = ops.rope_unit_kvwrite(x[:, :H * n], None, None, pos, H, G, n, nv, D, rotary=Tables(rot["base"], dims) if dims else None,
                                  page_size=page)
    assert torch.equal(rows, alone), "queries alone are the same rows"
    starts = np.concatenate([[0], np.cumsum(kv_lens)])
    take = torch.cat([torch.arange(starts[b] + kv - ql, starts[b] + kv) for b, (kv, ql) in enumerate(zip(kv_lens, q_lens))]).to(DEV)
    q = rows[take].contiguous()
    expect = torch.cat([w[kv - ql:] for w, kv, ql in zip(want, kv_lens, q_lens)])
    sinks = torch.zeros(H, dtype=torch.float32, device=DEV)
    lens = torch.tensor(kv_lens, dtype=torch.int32, device=DEV)
    ctx = SimpleNamespace(cu_q=torch.tensor([0] + list(np.cumsum(q_lens)), dtype=torch.int32, device=DEV), kv_lens=lens,
                          num_requests=len(q_lens), max_q_len=max(q_lens), max_kv_len=max(kv_lens), host={}, tile_cache={}, positions=pos[take])
    view = SimpleNamespace(block_table=table, page_size=page)
    cut = lambda out, k: out[..., :nv].reshape(k, H * nv)
    for backend in _backends(dtype, D, page):
        for splits in (None, 3):
            if splits and backend == "tcgen05":
                continue
            out = ops.paged_attention(q, kc, vc, view, ctx, scale, size, num_splits=splits, backend=backend, keep_first=keep_first,
                                      sinks=sinks, turn=turn)
            close(cut(out, q.shape[0]), expect, tol)
    # decoding alone (every request one token): the split-KV kernels, merged in a cluster and by a second launch
    one = torch.tensor([starts[b] + kv - 1 for b, kv in enumerate(kv_lens)], device=DEV)
    ctx1 = SimpleNamespace(cu_q=torch.arange(len(kv_lens) + 1, dtype=torch.int32, device=DEV), kv_lens=lens, num_requests=len(kv_lens),
                           max_q_len=1, max_kv_len=max(kv_lens), host={}, tile_cache={}, positions=pos[one])
    for splits in (None, 1, 5, 11):
        out = ops.paged_attention(rows[one].contiguous(), kc, vc, view, ctx1, scale, size, num_splits=splits, keep_first=keep_first,
                                  sinks=sinks, turn=turn)
        close(cut(out, len(kv_lens)), torch.stack([w[-1] for w in want]), tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D,page", [(32, 16), (64, 16), (128, 64)])
def test_keys_at_the_edges_of_the_window_and_of_the_first_tokens(dtype, D, page):
    """One key stands out: where a query sees it the output is its value, where not the output does not
    hold it at all.  Just inside and just outside the window, the last kept token and the next one, page
    borders; in a prompt and decoded alone."""
    from tinyserve_b200.kernels import ops
    H, G, n, size, keep = 2, 1, 300, 100, 5
    direction = torch.ones(D) / math.sqrt(D)
    last = n - 1
    turn = Tables(1e4, D)
    pos = torch.arange(n)
    for marked in (0, keep - 1, keep, page - 1, page, last - size - 1, last - size, last - size + 1, last - size + 2, 3 * page, last - 1, last):
        k, v = draws(n, G, D, seed=1, scale=0.02), draws(n, G, D, seed=2)
        k[marked] = (direction * 40).bfloat16().double()
        qrow = (direction * 40).bfloat16().double()
        table, slots, pages = _pages([n], page, seed=3)
        flat_k, flat_v = torch.zeros(pages * page, G, D, dtype=dtype, device=DEV), torch.zeros(pages * page, G, D, dtype=dtype, device=DEV)
        flat_k[slots.long()] = on_device(k, dtype)
        flat_v[slots.long()] = on_device(plain.rotate_values(v, pos, {"base": 1e4}), dtype)
        kc = flat_k.view(pages, page, G, D).permute(0, 2, 1, 3).contiguous()
        vc = flat_v.view(pages, page, G, D).permute(0, 2, 1, 3).contiguous()
        view = SimpleNamespace(block_table=table, page_size=page)
        seen = plain.window_mask(n, size, keep)
        for q_len in (1, 2, 150):
            q = on_device(qrow.repeat(q_len, H, 1), dtype)
            ctx = SimpleNamespace(cu_q=torch.tensor([0, q_len], dtype=torch.int32, device=DEV),
                                  kv_lens=torch.tensor([n], dtype=torch.int32, device=DEV), num_requests=1, max_q_len=q_len,
                                  max_kv_len=n, host={}, tile_cache={}, positions=torch.arange(n - q_len, n, dtype=torch.int32, device=DEV))
            out = ops.paged_attention(q, kc, vc, view, ctx, 1.0, size, keep_first=keep, sinks=torch.zeros(H, device=DEV), turn=turn)
            for place in {0, q_len // 2, q_len - 1}:
                i = n - q_len + place
                # (values turn relative to the query: by the distance i - marked)
                relative = plain.rotate_values(v[marked:marked + 1], torch.tensor([marked - i]), {"base": 1e4})[0, 0]
                miss = (out[place, 0].double().cpu() - relative).abs().max().item()
                assert (miss < 4e-2) == bool(seen[i, marked]), (marked, q_len, i, miss)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("D,page", [(16, 8), (64, 32), (128, 64)])
def test_sinks_learned_and_constant(dtype, tol, D, page):
    """Keys whose scores are all far below zero: a sink of zero leaves next to nothing of the values, no
    sink all of them; a learned sink of head 1 moves head 1 only."""
    from tinyserve_b200.kernels import ops
    H, n = 2, 170
    k, v, qrow = draws(n, 1, D, seed=1, scale=0.05), draws(n, 1, D, seed=2), torch.ones(D, dtype=torch.float64)
    k -= 6.0 / D                         # scores around -6
    k = k.bfloat16().double()
    table, slots, pages = _pages([n], page, seed=3)
    flat = torch.zeros(2, pages * page, 1, D, dtype=dtype, device=DEV)
    flat[0, slots.long()], flat[1, slots.long()] = on_device(k, dtype), on_device(v, dtype)
    kc, vc = (f.view(pages, page, 1, D).permute(0, 2, 1, 3).contiguous() for f in flat)
    view = SimpleNamespace(block_table=table, page_size=page)
    for q_len in (1, 3, 60):
        ctx = SimpleNamespace(cu_q=torch.tensor([0, q_len], dtype=torch.int32, device=DEV), kv_lens=torch.tensor([n], dtype=torch.int32, device=DEV),
                              num_requests=1, max_q_len=q_len, max_kv_len=n, host={}, tile_cache={})
        for sinks in ([0.0, 0.0], [-40.0, 5.0], None):
            out = ops.paged_attention(on_device(qrow.repeat(q_len, H, 1), dtype), kc, vc, view, ctx, 1.0,
                                      sinks=torch.tensor(sinks, device=DEV) if sinks else None)[-1]
            s = k[:, 0] @ qrow
            for a in range(H):
                den = s.exp().sum() + (math.exp(sinks[a]) if sinks else 0.0)
                want = (s.exp() / den) @ v[:, 0]
                assert (out[a].double().cpu() - want).abs().max() <= tol * v.abs().max(), (q_len, sinks, a)


# ----------------------------------------------------------------------------- whole models
LENGTHS = {"P": [5, 37, 40, 70, 2, 1, 33], "Q": [1, 9, 64, 100, 31, 48], "R": [150, 130, 57, 3, 129]}


@pytest.fixture(scope="module", params=sorted(GUNULORN_TINY))
def model(request, tmp_path_factory):
    name = request.param
    folder = make_gunulorn_dir(tmp_path_factory.mktemp(f"gunulorn{name}"), name, seed=41)
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
    got = collect_logits(steps, outputs, model["cfg"]["vocab"])
    # In bfloat16 a token whose router logits lie within a rounding of one another may take another
    # expert than the plain model does; one position in twenty may differ for that reason; none in
    # 32-bit, where every schedule is held to the plain model at every position.
    positions = sum(out.shape[0] for out in got.values())
    allowed = positions // 20 if dtype == "bfloat16" else 0
    over = []
    for rid, out in got.items():
        ref = model["ref"][rid.rstrip("x")]
        assert out.shape == ref.shape
        scale = ref.abs().max().item()
        err = (out.double() - ref).abs().max(-1).values / scale
        rms = (out.double() - ref).pow(2).mean(-1).sqrt() / scale
        bad = ((err > slack * TOLERANCE[dtype]) | (rms > slack * RMS_TOLERANCE[dtype]))
        seen = MEASURED.setdefault((model["name"], dtype), [0.0, 0.0])
        if (~bad).any():
            seen[0], seen[1] = max(seen[0], err[~bad].max().item()), max(seen[1], rms[~bad].max().item())
        over += [(rid, int(i), err[int(i)].item(), rms[int(i)].item()) for i in bad.nonzero()]
    assert len(over) <= allowed, (f"{model['name']} {dtype}: {len(over)} of {positions} positions differ; the first is place "
                                  f"{over[0][1]} of request {over[0][0]} (error {over[0][2]:.3e}, rms {over[0][3]:.3e})")
    return runner


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts(model, dtype, tmp_path):
    check(model, dtype, schedule_whole(model["requests"]), tmp_path)


def test_stream_after_every_layer_run(model):
    """The 32-bit stream behind every layer, read off the model's own forward pass, against the plain one's."""
    from tinyserve_b200.engine import replay
    from tinyserve_b200.engine.batch import StepEntry
    from tinyserve_b200.kernels import ops
    ids = model["requests"]["r1"]
    _, want = plain.forward(model["cfg"], model["weights"], ids, return_layers=True)
    runner = replay.make_runner(model["folder"], "float32", 256)
    seen = []
    blocks = runner.model.blocks
    originals = [b.forward for b in blocks]

    def watched(block, original):
        def forward(x, residual, ctx, call):
            out = original(x, residual, ctx, call)
            stream = residual.clone()
            ops.stream_add_(stream, out)
            seen.append(stream.double().cpu())
            return out
        return forward

    for b, original in zip(blocks, originals):
        b.forward = watched(b, original)
    runner.manager.begin("a")
    runner.step([StepEntry("a", ids, [len(ids) - 1])])
    runner.manager.free("a")
    assert len(seen) == want.shape[0]
    for i, got in enumerate(seen):
        assert (got - want[i]).abs().max() <= 2e-5 * want[i].abs().max(), f"layer run {i}"


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
        # (the attention kernel cuts a request's keys into ranges by how full the batch is: the
        # order of its sums, not what is summed, depends on the batch)
        assert (a[rid] - b[rid]).abs().max() <= 1e-5 * b[rid].abs().max()


@pytest.mark.parametrize("seed", range(16))
def test_drawn_configurations(seed, tmp_path):
    """Configurations drawn from a seed (odd head sizes, head counts, taps, orders, readers, layers without
    feed-forward, windows, rotation over all, a part or none of a head): whole prompts, portions and a
    mixed batch against the plain implementation."""
    from tinyserve_b200.config import config_from_dict
    from tinyserve_b200.weights import write_random_model
    raw = random_gunulorn_config_dict(seed)
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
def test_far_keys_sinks_factors_and_the_first_tokens(dtype, name, tmp_path):
    """Sharp attention (a far key, a key at a page's border or a wrong position moves the logits), sinks,
    factors, taps and corrections that move them too; long prompts, long decoding, portions, mixed."""
    folder = make_gunulorn_dir(tmp_path / "base", name, seed=43, sharp=14.0)
    cfg, weights = plain.load_folder(folder)
    ids = random_ids(cfg["vocab"], 210, seed=7)
    ids[130] = ids[-1] = ids[3]               # a token that comes back far behind
    reqs = {"far": ids, "near": ids[:70]}
    ref = {rid: plain.logits(cfg, weights, t) for rid, t in reqs.items()}
    moved = lambda c, w, t=ids: (plain.logits(c, w, t) - ref["far"]).abs().max() / ref["far"].abs().max()
    other = list(ids)
    other[3] = (ids[3] + 1) % cfg["vocab"]
    assert moved(cfg, weights, other) > 0.01, "a far token matters here"
    for part, value in ((".sink", -60.0), (".temp", 1.0), (".correction", 0.0), (".up.b", 0.0), (".down.b", 0.0)):
        changed = {k: (torch.full_like(v, value) if k.endswith(part) else v) for k, v in weights.items()}
        assert moved(cfg, changed) > 5e-3, f"{part} matters"
    newest = {k: (torch.cat([torch.zeros_like(v[:, :-1]), v[:, -1:]], -1) if k.endswith(".conv") else v) for k, v in weights.items()}
    assert moved(cfg, newest) > 1e-2, "the older taps matter"

    def with_mask(**change):
        return {**cfg, "layers": [{**l, "mixer": {**l["mixer"], "mask": {**l["mixer"]["mask"], **change}}} if "mask" in l["mixer"] else l
                                  for l in cfg["layers"]]}
    for change in ({"keep_first": 0}, {"size": 10}):
        assert moved(with_mask(**change), weights) > 1e-2, change
    model = {"name": name + "sharp", "folder": folder, "cfg": cfg, "requests": reqs, "ref": ref}
    slack = 2.0 if dtype == "float32" else 3.0
    check(model, dtype, schedule_whole(reqs), tmp_path / "whole", slack=slack)
    check(model, dtype, schedule_tail_decode(reqs, 120), tmp_path / "tail", slack=slack)
    check(model, dtype, schedule_portions(reqs, sizes=(63, 2, 1, 64, 5, 16, 15)), tmp_path / "portions", slack=slack)
    check(model, dtype, schedule_mixed({**reqs, "farx": ids, "nearx": ids[:70]}, max_live=3, seed=5), tmp_path / "mixed",
          slack=slack, max_live=3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_head_sizes_of_real_models(dtype, tmp_path):
    """Heads of 128 and of 64, a width whose few rows are normed over a cluster, pages of 64: the kernels
    that real layer sizes reach (tcgen05 prefill, decode by whole pages, products cut along K), prompts
    longer than two key tiles of any kernel."""
    from tinyserve_b200.config import config_from_dict
    from tinyserve_b200.weights import write_random_model
    raw = {"architecture": "Gunulorn", "vocab": 1000, "width": 1024, "norm": {"eps": 1e-6}, "logit_scale": 0.6, "logit_softcap": 25.0, "layers": [
        {"type": "attention", "mlp": _dense(2048), "mixer": _conv(8, 2, 128, 128, 0.09, 4)},
        {"type": "attention_2", "mlp": _moe(256, 8, 4, 2), "mixer": _turned(8, 2, 128, 128, 0.09, 1e6, 64, 200, 4)},
        {"type": "attention_2", "mlp": _moe(256, 16, 2, 3), "mixer": _turned(8, 1, 64, 64, 0.125, 1e4, 64, 130, 20)},
        {"type": "attention", "mlp": _moe(128, 4, 1, 2), "mixer": _conv(8, 2, 128, 128, 0.09, 3, kv_from=0)},
    ]}
    folder = decisive(write_random_model(config_from_dict(raw), str(tmp_path / "model"), seed=5), 5, sharp=2.0)
    cfg, weights = plain.load_folder(folder)
    reqs = {"a": random_ids(1000, 420, seed=1), "b": random_ids(1000, 130, seed=2)}
    ref = {rid: plain.logits(cfg, weights, ids) for rid, ids in reqs.items()}
    model = {"name": "real", "folder": folder, "cfg": cfg, "requests": reqs, "ref": ref}
    check(model, dtype, schedule_tail_decode(reqs, 40), tmp_path / "tail", page=64)
    check(model, dtype, schedule_mixed(reqs, max_live=2, seed=1, chunk_sizes=(200, 2, 129, 64, 1)), tmp_path / "mixed", max_live=2)


def test_steps_of_few_tokens_run_both_branches_products_together(tmp_path):
    """A decode step of a few requests: one launch for all input products of a layer, one for both output
    products with the residual add, none for a norm of its own between the layers."""
    from tinyserve_b200.engine import replay
    from tinyserve_b200.engine.batch import StepEntry
    from tinyserve_b200.kernels import ops
    runner = replay.make_runner(make_gunulorn_dir(tmp_path, "R", seed=1), "bfloat16", 256)
    for rid in ("a", "b"):
        runner.manager.begin(rid)
        runner.step([StepEntry(rid, [1, 2, 3, 4, 5], [])])
    runner.cfg.check_indices = False         # (the index check has launches of its own)
    before = ops.launch_count()
    runner.step([StepEntry("a", [6], [0]), StepEntry("b", [7], [0])])
    # block tables 2, embedding, first norm; per layer: inputs, heads, attention, activation, outputs; the last outputs
    # and the last norm are two; logits, cap
    assert ops.launch_count() - before == 4 + 5 * 5 - 1 + 2 + 2, ops.launch_count() - before


# ----------------------------------------------------------------------------- the entry point
def test_greedy_generation_through_the_scheduler(tmp_path):
    """Five prompts of unequal length through LLM.generate with three slots and at most 48 tokens a
    step (prompts in portions beside decoding requests, slots and pages used again)."""
    from tinyserve_b200 import LLM, SamplingParams
    folder = make_gunulorn_dir(tmp_path, "P", seed=44)
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
    """bin/trace_run and ``python -m tinyserve_b200 generate`` as programs on a Gunulorn folder: the
    architecture is chosen by config.json; stdin to files, 'done' lines, exit code 0; greedy tokens."""
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    folder = make_gunulorn_dir(tmp_path / "m", "Q", seed=2)
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
