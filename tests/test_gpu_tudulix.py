"""Tudulix on the GPU against the plain implementation: every mechanism alone, then whole models through every way of
cutting requests into steps, in 32-bit and in bfloat16, with pools so small that pages and slots are used again."""
import copy
import json
import math
import os

import pytest
import torch

import harness
import tiny
import tudulix_tiny as tt
from plain import tudulix_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
TOL = {torch.float32: (1e-4, 0.0), torch.bfloat16: (0.0, 8e-2)}


def _weights(folder):
    return {k: v for k, v in tiny.read_weights(folder).items()}


def _cfg(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def _reference(folder, reqs):
    cfg, w = _cfg(folder), _weights(folder)
    return {rid: plain.forward(cfg, w, toks, torch.float64) for rid, toks in reqs.items()}


def _compare(got, ref, dtype, loosen=1.0):
    """Every position within the bound, the median position well within it.  In bfloat16 one position in ten may be up to three
    times the bound off (these models are narrow and deep, and every sublayer's output is brought to unit size, so at some
    positions the rounding grows); the 32-bit runs of the same schedules are held to every position."""
    atol, rel = TOL[dtype]
    off, ratios = [], []
    for (rid, pos), row in got.items():
        want = ref[rid][pos]
        size = float(want.abs().max())
        bound = loosen * (atol * max(1.0, size) + rel * size)
        diff = float((row.double() - want).abs().max())
        ratios.append(diff / bound)
        if diff > bound:
            off.append(f"request {rid} position {pos}: max diff {diff:.3e} > {bound:.3e}")
    allowed = len(got) // 10 if dtype == torch.bfloat16 else 0
    assert len(off) <= allowed and max(ratios) <= (3.0 if allowed else 1.0), f"{len(off)} of {len(got)} positions off: " + "; ".join(off[:5])
    assert sorted(ratios)[len(ratios) // 2] <= 0.5, f"the median position is at {sorted(ratios)[len(ratios) // 2]:.2f} of the bound"


def _runner(folder, dtype, page_size, num_pages, max_slots=4, graphs=False):
    from prelude_b200.engine.loading import load_model, make_runner
    model = load_model(folder, dtype, DEV)
    runner = make_runner(model, page_size=page_size, num_pages=num_pages, max_slots=max_slots,
                         max_request_tokens=num_pages * page_size if graphs else None)
    if graphs:
        runner.enable_step_graphs()
    return runner


def _tensor(y, dtype):
    from prelude_b200.ops import kernels as K
    y = K.settled(y)
    return y.materialize(dtype) if isinstance(y, K.PartialSums) else y


def _steps_through(part, x, cuts, page, dtype):
    """x [T, width] through a mixer, cut into the steps ``cuts``; a step of one token is a decode step.  Pages that the window
    has passed are given back after every step."""
    from prelude_b200.cache.manager import CacheManager
    from prelude_b200.engine.batch import StepItem, build_step_batch
    dev = torch.device(DEV)
    T = x.shape[0]
    cache = CacheManager([part.cache_need()], page, -(-T // page) + 1, 2, dev, dtype)
    cache.add_request("a")
    got, at = [], 0
    for n in cuts:
        cache.grow("a", at + n)
        batch = build_step_batch([StepItem("a", [0] * n, at, [])], cache.block_tables(["a"]), [cache.slot_of("a")], dev, 10, 1 << 20)
        y = part.forward(x[at:at + n].to(DEV).contiguous(), batch, cache.layer_cache(0), True)
        got.append(_tensor(y, dtype).float().cpu())
        assert int(batch.status.item()) == 0
        at += n
        cache.trim("a")
    assert at == T
    return torch.cat(got).double()


def _cuts(T, head):
    return [head] + [1] * (T - head)


def _close(got, want, tol, what):
    assert float((got - want).abs().max()) < tol * float(want.abs().max()), (what, float((got - want).abs().max()), float(want.abs().max()))


def _load(part, w, dtype):
    from prelude_b200.parts.registry import RunContext
    part.load(lambda name: w[name], RunContext(torch.device(DEV), dtype))
    return part


def _reader(raw, where):
    from prelude_b200.config.reader import _Reader
    problems = []
    return _Reader(raw, where, problems), problems


def _mixer(kind, m, w, width, eps, dtype):
    from prelude_b200.config import tudulix as ct
    from prelude_b200.parts.registry import make_part
    rd, problems = _reader(m, "mixer")
    spec = ct._attention(rd, width) if kind == "attention" else ct._latent_attention(rd, width, eps)
    assert not problems
    return _load(make_part("mixer", spec, "mix"), w, dtype)


def _double(w, cut=4):
    return {k[cut:]: v.double() for k, v in w.items()}


# -- the residual add between two norms ---------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("T,width", [(1, 44), (9, 128), (300, 2048), (17, 33), (5, 7), (3, 4100), (2, 9000), (4, 8192)])
def test_residual_add_between_two_norms_takes_the_embedding_again(dtype, T, width):
    """The stream, normed addend and a second addend in one kernel, with the norm of the sum; without the second addend; and
    carried along as the model does (``joined``), for a pending norm and for a plain addend."""
    from prelude_b200.ops import kernels as K
    g = torch.Generator().manual_seed(T + width)
    res, plus = torch.randn(T, width, generator=g) * 3.0, torch.randn(T, width, generator=g) * 2.0
    x = torch.randn(T, width, generator=g).to(dtype)
    wx, w = torch.rand(width, generator=g) + 0.5, torch.rand(width, generator=g) + 0.5
    eps_x, eps = 0.3, 0.02                                     # large enough that one in the other's place would show
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    dev = [t.to(DEV) for t in (wx, w, plus)]
    for second in (None, plus):
        total = res.double() + plain.rms(x.double(), eps_x) * wx.double() + (0 if second is None else second.double())
        want = plain.rms(total, eps) * w.double()
        r = res.to(DEV)
        y = K.normed_add_rmsnorm(K.Normed(x.to(DEV), dev[0], eps_x, None if second is None else dev[2]), r, dev[1], eps, dtype)
        _close(r.cpu().double(), total, 1e-5, "stream")
        _close(y.cpu().double(), want, tol, "norm")
        r = res.to(DEV)
        assert K.normed_add_rmsnorm(K.Normed(x.to(DEV), dev[0], eps_x, None if second is None else dev[2]), r, None, 0.0, dtype) is None
        _close(r.cpu().double(), total, 1e-5, "stream alone")
    r = res.to(DEV)
    d = K.joined(K.Normed(x.to(DEV), dev[0], eps_x), dev[2], r)
    assert torch.equal(r.cpu(), res) and d.plus is dev[2]
    d = K.joined(x.to(DEV), dev[2], r)
    assert torch.equal(d.cpu(), x)
    _close(r.cpu().double(), res.double() + plus.double(), 1e-6, "joined")
    with pytest.raises(RuntimeError):                          # chosen rows are for the last norm, which nothing joins
        K.normed_add_rmsnorm(K.Normed(x.to(DEV), dev[0], eps_x, dev[2]), r, dev[1], eps, dtype, rows=torch.zeros(1, dtype=torch.int32, device=DEV))


@BOTH
@pytest.mark.parametrize("T,top,width,shared,places,y32", [
    (1, 1, 64, "none", False, True), (9, 3, 128, "tensor", True, True), (40, 6, 96, "parts", False, True), (7, 5, 264, "tensor", True, False),
    (300, 4, 2048, "parts", True, False), (5, 9, 4096, "none", True, True), (3, 2, 8192, "tensor", True, False), (6, 2, 30, "tensor", True, True),
    (2, 8, 16384, "tensor", True, True), (11, 7, 4096, "tensor", True, False)])
def test_the_experts_sum_with_the_norms_around_the_residual_add(dtype, T, top, width, shared, places, y32):
    """Weighted sum of a token's choices plus what every token adds, normed, added to the stream (with a second addend and
    without), the sum normed: in one kernel where it takes the width (all but two of the sizes), else in several; at chosen
    rows, one of which does not exist, the stream is left alone."""
    from prelude_b200.ops import kernels as K
    from prelude_b200.ops import library
    g = torch.Generator().manual_seed(T * 10 + top)
    y = torch.randn(T * top, width, generator=g).to(torch.float32 if y32 else dtype)
    place = torch.randperm(T * top, generator=g)
    weights = torch.rand(T, top, generator=g)
    at = place if places else torch.arange(T * top)
    v = (y.double()[at].reshape(T, top, width) * weights.double().unsqueeze(-1)).sum(1)
    sh = None
    if shared == "tensor":
        t = torch.randn(T, width, generator=g).to(dtype)
        sh, v = t.to(DEV), v + t.double()
    elif shared == "parts":
        t = torch.randn(3, T, width, generator=g)
        sh, v = K.PartialSums(t.to(DEV)), v + t.double().sum(0)
    pend = K.PendingExperts(y.to(DEV), place.int().to(DEV) if places else None, weights.to(DEV), sh, dtype)
    assert bool(library.library().pb_moe_sum_normed_supported(width, K.dtype_code(dtype))) == (width not in (30, 16384))
    res, plus = torch.randn(T, width, generator=g), torch.randn(T, width, generator=g)
    wv, w = torch.rand(width, generator=g) + 0.5, torch.rand(width, generator=g) + 0.5
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for second in (None, plus):
        total = res.double() + plain.rms(v, 0.2) * wv.double() + (0 if second is None else second.double())
        r = res.to(DEV)
        got = K.normed_add_rmsnorm(K.Normed(pend, wv.to(DEV), 0.2, None if second is None else second.to(DEV)), r, w.to(DEV), 0.03, dtype)
        _close(r.cpu().double(), total, 1e-5 if dtype == torch.float32 or width not in (30, 16384) else 1e-2, "stream")
        _close(got.cpu().double(), plain.rms(total, 0.03) * w.double(), tol, "norm")
    r = res.to(DEV)
    rows = torch.tensor([T - 1, 0, T, -1], dtype=torch.int32, device=DEV)[:4 if width not in (30, 16384) else 2]
    got = K.normed_add_rmsnorm(K.Normed(pend, wv.to(DEV), 0.2), r, w.to(DEV), 0.03, dtype, rows=rows).cpu().double()
    want = plain.rms(res.double() + plain.rms(v, 0.2) * wv.double(), 0.03) * w.double()
    assert torch.equal(r.cpu(), res) and float(got[2:].abs().sum()) == 0.0
    _close(got[:2], want[[T - 1, 0]], tol, "chosen rows")


@BOTH
@pytest.mark.parametrize("T,cols,pad", [(1, 42, 3), (9, 256, 8), (300, 2048, 0), (17, 33, 1), (5, 4104, 16)])
def test_gate_per_element_in_place(dtype, T, cols, pad):
    from prelude_b200.ops import kernels as K
    g = torch.Generator().manual_seed(T + cols)
    y = torch.randn(T, cols, generator=g).to(dtype)
    gate = (torch.randn(T, cols + pad, generator=g) * 6.0).to(dtype)
    want = y.double() * torch.sigmoid(gate[:, pad:].double())
    got = y.to(DEV)
    assert K.sigmoid_gate_(got, gate.to(DEV)[:, pad:]) is got
    _close(got.cpu().double(), want, 1e-6 if dtype == torch.float32 else 5e-3, "gate")


# -- attention over a window ------------------------------------------------------------------------------------------------
def _gqa_weights(g, width, H, G, dim, vdim, dtype):
    w = {"mix.q": torch.randn(H * dim, width, generator=g) * 0.3, "mix.k": torch.randn(G * dim, width, generator=g) * 0.3,
         "mix.v": torch.randn(G * vdim, width, generator=g) * 0.3, "mix.o": torch.randn(width, H * vdim, generator=g) * 0.2}
    return {k: v.to(dtype) for k, v in w.items()}


@BOTH
@pytest.mark.parametrize("H,G,dim,vdim,dims,window,page", [
    (6, 2, 10, 7, 6, 9, 4), (4, 2, 64, 64, 32, 24, 16), (8, 1, 32, 48, 32, 70, 16), (1, 1, 16, 16, 16, 1, 8), (3, 3, 9, 9, 4, 21, 4), (6, 2, 128, 128, 64, 33, 16),
    (12, 3, 64, 64, 2, 128, 64), (5, 5, 16, 32, 8, 130, 8), (8, 2, 128, 64, 128, 40, 16), (4, 4, 80, 80, 48, None, 16), (16, 1, 48, 48, 16, 500, 32)])
def test_window_attention_equals_the_plain_one(dtype, H, G, dim, vdim, dims, window, page):
    """Whole, with a decoded tail across page borders, in portions and token by token."""
    width, T = 48, 160
    g = torch.Generator().manual_seed(H * 100 + dim)
    m = tt.attention_mixer(H, G, dim, vdim, 1.5 / math.sqrt(dim), 3000.0, dims, window)
    w = _gqa_weights(g, width, H, G, dim, vdim, dtype)
    x = torch.randn(T, width, generator=g).to(dtype)
    want = plain.grouped_attention(x.double(), _double(w), m)
    part = _mixer("attention", m, w, width, 1e-5, dtype)
    tol = 5e-5 if dtype == torch.float32 else 4e-2
    for cuts in ([T], _cuts(T, 75), [2, 30, 3, 26, 2, 97], [1] * T):
        _close(_steps_through(part, x, cuts, page, dtype), want, tol, cuts[:3])


def _latent_weights(g, width, H, dim, rot_dim, vdim, rank, dtype):
    w = {"mix.q": torch.randn(H * (dim + rot_dim), width, generator=g) * 0.25, "mix.uk": torch.randn(H * dim, rank, generator=g) / math.sqrt(rank),
         "mix.uv": torch.randn(H * vdim, rank, generator=g) / math.sqrt(rank), "mix.g": torch.randn(H * vdim, width, generator=g) * 0.3,
         "mix.o": torch.randn(width, H * vdim, generator=g) * 0.2, "mix.dkv": torch.randn(rank + rot_dim, width, generator=g) * 0.3,
         "mix.dkv.norm": 1.0 + 0.3 * torch.randn(rank, generator=g)}
    return {k: v.to(dtype) for k, v in w.items()}


@BOTH
@pytest.mark.parametrize("H,dim,rot_dim,vdim,rank,window,page", [
    (3, 10, 6, 7, 13, 13, 4), (4, 32, 16, 32, 64, 40, 16), (2, 12, 6, 10, 13, 1, 8), (1, 8, 8, 8, 8, 64, 8), (8, 64, 32, 48, 96, 33, 16), (5, 6, 4, 9, 11, None, 4),
    (16, 128, 64, 128, 512, 50, 16), (32, 16, 16, 16, 32, 17, 64), (6, 32, 32, 32, 128, 96, 16), (3, 40, 24, 96, 64, 70, 16)])
def test_latent_attention_over_a_window_with_a_gate_per_element_equals_the_plain_one(dtype, H, dim, rot_dim, vdim, rank, window, page):
    width, T, eps = 48, 160, 1e-2
    g = torch.Generator().manual_seed(H * 100 + dim)
    m = tt.latent_mixer(H, dim, rot_dim, vdim, rank, 2.0 / math.sqrt(dim + rot_dim), 3000.0, window)
    w = _latent_weights(g, width, H, dim, rot_dim, vdim, rank, dtype)
    x = torch.randn(T, width, generator=g).to(dtype)
    wd = _double(w)
    want = plain.latent_attention(x.double(), wd, m, plain.cached_rows(x.double(), wd, m, eps))
    part = _mixer("latent_attention", m, w, width, eps, dtype)
    tol = 5e-5 if dtype == torch.float32 else 4e-2
    for cuts in ([T], _cuts(T, 75), [2, 30, 3, 26, 2, 97], [1] * T):
        _close(_steps_through(part, x, cuts, page, dtype), want, tol, cuts[:3])


@BOTH
@pytest.mark.parametrize("kind,window,page", [("attention", 75, 16), ("attention", 128, 16), ("attention", 33, 8), ("attention", 200, 64),
                                              ("latent_attention", 75, 16), ("latent_attention", 128, 16), ("latent_attention", 33, 8),
                                              ("latent_attention", 200, 64)])
def test_a_key_is_seen_until_it_leaves_the_window(dtype, kind, window, page):
    """One early token's key stands out by so much that every query that sees it sees nothing else: the last position that
    sees it and the first that does not differ outright, in prompts (also long ones, on the prompt kernels), in portions that
    end right at the edge, and in decoding."""
    width, T, eps, at = 64, 330, 1e-5, 21
    g = torch.Generator().manual_seed(window)
    x = torch.randn(T, width, generator=g) * 0.5
    x[:, 0], x[:, 1] = 1.0, 0.0                                # column 0: every token asks; column 1: one token answers
    x[at, 1] = 8.0
    x = x.to(dtype)
    if kind == "attention":
        H, G, dim = 4, 2, 64
        m = tt.attention_mixer(H, G, dim, dim, 0.125, 3000.0, 32, window)
        w = _gqa_weights(g, width, H, G, dim, dim, torch.float32)
        w["mix.q"][dim - 1::dim, 0] = 16.0                     # the last element of every head, which is not turned
        w["mix.k"][dim - 1::dim, 1] = 3.0
        w = {k: v.to(dtype) for k, v in w.items()}
        run = lambda mm: plain.grouped_attention(x.double(), _double(w), mm)
    else:
        H, dim, rot_dim, rank = 4, 48, 16, 64
        m = tt.latent_mixer(H, dim, rot_dim, 32, rank, 0.125, 3000.0, window)
        w = _latent_weights(g, width, H, dim, rot_dim, 32, rank, torch.float32)
        w["mix.dkv"][0, 1] = 12.0                              # the answering token's latent is nearly its first element alone
        w["mix.uk"][dim - 1::dim, 0] = 4.0
        w["mix.q"][dim - 1::dim + rot_dim, 0] = 16.0
        w = {k: v.to(dtype) for k, v in w.items()}
        run = lambda mm: plain.latent_attention(x.double(), _double(w), mm, plain.cached_rows(x.double(), _double(w), mm, eps))
    want = run(m)
    for other in (window - 1, window + 1):                     # a window one token off shows at the edge
        wrong = (run(dict(m, mask={"size": other})) - want).abs().amax(dim=1)
        edge = at + min(window, other)
        assert float(wrong[edge]) > 0.3 * float(want.abs().max()), "the test would not see a window that is one token off"
    part = _mixer(kind, m, w, width, eps, dtype)
    tol = 2e-4 if dtype == torch.float32 else 5e-2
    last = at + window - 1                                     # the last position that sees the key
    for cuts in ([T], _cuts(T, 60), _cuts(T, last), [last, 1, 2, T - last - 3], [last + 1, T - last - 1], [last - 1, 2, T - last - 1], [150, 2, 178]):
        _close(_steps_through(part, x, cuts, page, dtype), want, tol, cuts[:3])


@pytest.mark.parametrize("heads,dim,rot_dim,vdim,rank,window,page", [
    (4, 128, 64, 128, 512, 100, 16), (3, 64, 32, 64, 96, 300, 16), (2, 32, 16, 32, 64, 128, 64), (2, 112, 16, 128, 128, 129, 8), (3, 40, 24, 96, 64, 1, 16),
    (1, 80, 16, 8, 40, 640, 16), (8, 16, 16, 120, 32, 255, 128)])
def test_long_portions_with_keys_and_values_made_per_head_inside_a_window(heads, dim, rot_dim, vdim, rank, window, page):
    """bfloat16.  One step holds a portion of 300 tokens behind 470 cached ones (of which the window has passed pages, which
    were given back), a decoded token behind 500, a fresh portion of 330 and one of 20: the long ones go through keys and
    values made per head, the others stay in the latent's space.  The same step with that way turned off, and the plain
    implementation, say what must come out."""
    from prelude_b200.cache.manager import CacheManager
    from prelude_b200.engine.batch import StepItem, build_step_batch
    width, eps, dtype = 64, 1e-5, torch.bfloat16
    g = torch.Generator().manual_seed(heads * 100 + dim)
    m = tt.latent_mixer(heads, dim, rot_dim, vdim, rank, 2.0 / math.sqrt(dim + rot_dim), 3000.0, window)
    w = _latent_weights(g, width, heads, dim, rot_dim, vdim, rank, dtype)
    part = _mixer("latent_attention", m, w, width, eps, dtype)
    assert part.w_rows is not None
    before, step = {"a": 470, "b": 500, "c": 0, "d": 0}, {"a": 300, "b": 1, "c": 330, "d": 20}
    xs = {r: torch.randn(before[r] + n, width, generator=g).to(dtype) for r, n in step.items()}
    dev = torch.device(DEV)
    cache = CacheManager([part.cache_need()], page, sum(-(-x.shape[0] // page) for x in xs.values()), 4, dev, dtype)
    cache.layer_cache(0).k_pages.fill_(float("nan"))           # what no one wrote must not be read
    outs = {}
    for way in ("per head", "latent"):
        rows = part.w_rows
        if way == "latent":
            part.w_rows = None
        for r in step:
            cache.add_request(r)
        for counts in ({r: n for r, n in before.items() if n}, step):
            rids = list(counts)
            at = {r: (before[r] if counts is step else 0) for r in rids}
            for r in rids:
                cache.grow(r, at[r] + counts[r])
            batch = build_step_batch([StepItem(r, [0] * counts[r], at[r], []) for r in rids], cache.block_tables(rids), [cache.slot_of(r) for r in rids],
                                     dev, 10, 1 << 20)
            x = torch.cat([xs[r][at[r]:at[r] + counts[r]] for r in rids]).to(DEV)
            got = _tensor(part.forward(x, batch, cache.layer_cache(0), True), dtype).float().cpu().double()
            assert int(batch.status.item()) == 0
            for r in rids:
                cache.trim(r)
        plan = batch.extras.get(("rows_plan", window))
        assert (plan is not None) == (way == "per head")
        if plan is not None:
            assert plan.n_blocks == 7 - max(0, 470 - window + 1) // 128 + 3
        outs[way] = got
        for r in step:
            cache.release(r)
        part.w_rows = rows
    o = 0
    wd = _double(w)
    for r, n in step.items():
        want = plain.latent_attention(xs[r].double(), wd, m, plain.cached_rows(xs[r].double(), wd, m, eps))[before[r]:]
        for way in outs:
            _close(outs[way][o:o + n], want, 3e-2 if n > 1 else 6e-2, (r, way))      # (one row: its own largest element is the measure)
        o += n


# -- the router and the experts -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("experts,top", [(6, 2), (5, 3), (16, 2), (4, 1), (2, 2), (1, 1), (64, 6), (40, 5), (9, 9), (160, 8), (7, 1), (250, 32), (300, 4)])
def test_router_chooses_by_biased_logits_and_weighs_the_chosen_alone(experts, top):
    """The kernels' experts and weights against the plain router's, from logits (a prompt step) and from rows and matrix in
    one kernel (a decode step), logits spread from nearly equal to hundreds apart; the bias decides many choices."""
    from prelude_b200.ops import kernels as K
    g = torch.Generator().manual_seed(experts * 7 + top)
    bias = torch.randn(experts, generator=g) * 2.0
    args = (top, 1, 1, 2, False, None, False, 0.0, 1.0, bias.to(DEV), True)
    T = 200
    logits = torch.randn(T, experts, generator=g) * torch.logspace(-1, 2.5, T).unsqueeze(1)
    biased = logits + bias
    keep = plain.route_margin(biased.double(), top) > 1e-4
    logits, biased = logits[keep], biased[keep]
    want_ids, want_w = plain.route(biased.double(), top)
    ids, w = K.moe_route(logits.to(DEV), *args)
    dense = torch.zeros(logits.shape, dtype=torch.float64)
    want, got = dense.scatter(1, want_ids, want_w), dense.scatter(1, ids.cpu().long(), w.cpu().double())
    assert torch.equal(ids.cpu().long().sort(dim=1).values, want_ids.sort(dim=1).values)
    assert float((got - want).abs().max()) < 1e-4 and float((w.cpu().double().sum(1) - 1.0).abs().max()) < 1e-5
    if 1 < top < experts:
        assert float((plain.route(logits.double(), top)[0].sort(dim=1).values != want_ids.sort(dim=1).values).double().mean()) > 0.1
    if experts > 256:
        return
    for dtype in (torch.float32, torch.bfloat16):
        for width, pad, rows in ((64, 0, 1), (200, 8, 32), (1024, 0, 9)):
            x = torch.randn(rows, width + pad, generator=g).to(dtype).to(DEV)[:, :width]
            m = (torch.randn(experts, width, generator=g) / math.sqrt(width)).to(dtype).to(DEV)
            assert K.moe_route_few_takes(x, m)
            ids, w = K.moe_route_few(x, m, *args)
            z = x.cpu().double() @ m.cpu().double().T + bias.double()
            ok = plain.route_margin(z, top) > 1e-4
            want_ids, want_w = plain.route(z, top)
            assert torch.equal(ids.cpu()[ok].long().sort(dim=1).values, want_ids[ok].sort(dim=1).values)
            dense = torch.zeros(z.shape, dtype=torch.float64)
            assert float((dense.scatter(1, ids.cpu().long(), w.cpu().double()) - dense.scatter(1, want_ids, want_w))[ok].abs().max()) < 1e-5


@BOTH
@pytest.mark.parametrize("experts,top,ff,limit,shared,T,width", [
    (6, 2, 10, 0.8, (14, 0.4), 37, 48), (5, 3, 14, 1.5, None, 1, 48), (8, 4, 64, 0.7, (96, 1.2), 300, 64), (2, 1, 16, 1.0, (16, 1.0), 9, 48),
    (16, 2, 32, 2.0, (64, 0.5), 70, 128), (2, 2, 64, 0.6, (128, 0.9), 400, 64), (4, 2, 128, 1.1, (256, 0.7), 900, 128), (32, 4, 64, 0.9, (64, 2.0), 8, 256),
    (3, 1, 7, 0.5, (5, 0.8), 6, 33), (4, 1, 24, 1.0, (8, 0.3), 50, 40), (1, 1, 96, 1.3, (48, 0.9), 800, 64), (14, 3, 88, 1.7, (112, 1.2), 16, 96)])
def test_experts_with_the_clamped_unit_equal_the_plain_ones(dtype, experts, top, ff, limit, shared, T, width):
    """A decode step's few tokens, prompt steps on every tile height, and steps long enough for the paired-block kernel; many
    gate and up sums lie beyond the limits, on both sides, and the shared expert has a limit of its own."""
    from prelude_b200.config.tudulix import _experts
    from prelude_b200.parts.registry import make_part
    g = torch.Generator().manual_seed(experts + T)
    mlp = tt.moe(experts, top, ff, limit, shared)
    w = {"mlp.router": torch.randn(experts, width, generator=g) * 0.5, "mlp.router.b": torch.randn(experts, generator=g) * 2.0}
    for e in [f"e{i}" for i in range(experts)] + (["shared"] if shared else []):
        n = shared[0] if e == "shared" else ff
        w.update({f"mlp.{e}.gate": torch.randn(n, width, generator=g) * 0.3, f"mlp.{e}.up": torch.randn(n, width, generator=g) * 0.3,
                  f"mlp.{e}.down": torch.randn(width, n, generator=g) * 0.3})
    w = {k: v.to(dtype) for k, v in w.items()}
    x = torch.randn(T, width, generator=g).to(dtype)
    wd = _double(w)
    want = plain.routed_ff(x.double(), wd, mlp)
    size = float(want.abs().max())
    assert float((plain.routed_ff(x.double(), wd, dict(mlp, expert={"ff": ff, "limit": 100.0})) - want).abs().max()) > 0.05 * size
    if shared:
        for other in (None, {"ff": shared[0], "limit": shared[1] * 2}):
            assert float((plain.routed_ff(x.double(), wd, dict(mlp, shared=other)) - want).abs().max()) > 0.03 * size
    rd, problems = _reader(mlp, "mlp")
    part = _load(make_part("feed_forward", _experts(rd, width), "mlp"), w, dtype)
    assert not problems
    got = _tensor(part.forward(x.to(DEV)), dtype).float().cpu().double()
    if dtype == torch.float32:
        _close(got, want, 5e-5, "routed")
    else:
        ok = plain.route_margin(plain.router_logits(x.double(), wd), top) > 1e-4
        _close(got[ok], want[ok], 3e-2, "routed")
        assert int(ok.sum()) >= T - 1 - T // 50
    # a token's result does not depend on who else is in the step
    alone = torch.cat([_tensor(part.forward(x[t:t + 1].to(DEV)), dtype) for t in range(min(T, 5))]).float().cpu().double()
    _close(alone, got[:alone.shape[0]], 1e-5 if dtype == torch.float32 else 2e-2, "alone")


# -- whole models ----------------------------------------------------------------------------------------------------
REQUESTS = {"A": {"a1": 1, "a2": 2, "a19": 19, "a70": 70, "a33": 33}, "B": {"b3": 3, "b150": 150, "b64": 64, "b41": 41, "b97": 97},
            "C": {"c1": 1, "c9": 9, "c40": 40, "c17": 17}, "D": {"d5": 5, "d80": 80, "d31": 31, "d2": 2}}


def _requests(which):
    v = tt.PARAMS[which][0]["vocab"]
    return {rid: tiny.random_ids(n, v, sum(map(ord, rid))) for rid, n in REQUESTS[which].items()}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("tudulix")
    return {(w, d): tt.make_folder(root, w, d) for w in "ABCD" for d in (torch.float32, torch.bfloat16)}


@pytest.fixture(scope="module")
def references(folders):
    return {d: {w: _reference(folders[(w, d)], _requests(w)) for w in "ABCD"} for d in (torch.float32, torch.bfloat16)}


def test_the_stream_after_every_layer_run_equals_the_plain_one(folders):
    """Layer run by layer run in 32-bit: the first that differs names the mechanism."""
    from prelude_b200.engine.batch import StepItem, build_step_batch
    from prelude_b200.engine.loading import load_model, make_runner
    from prelude_b200.engine.runner import StepEntry
    from prelude_b200.ops import kernels as K
    from prelude_b200.ops.linear import step_status
    for which in "ABCD":
        folder = folders[(which, torch.float32)]
        cfg, w = _cfg(folder), _weights(folder)
        toks = tiny.random_ids(45, cfg["vocab"], 4)
        want = []
        plain.forward(cfg, w, toks, torch.float64, layers_out=want)
        model = load_model(folder, torch.float32, DEV)
        assert len(model.order) == len(want)
        runner = make_runner(model, page_size=tt.PARAMS[which][2], num_pages=16, max_slots=1)
        runner.reserve([StepEntry("x", toks, [])])
        batch = build_step_batch([StepItem("x", toks, 0, [])], runner.cache.block_tables(["x"]), [runner.cache.slot_of("x")], runner.device,
                                 model.spec.vocab_size, model.spec.max_positions)
        with step_status(batch.status):
            res = model.embedding.forward(batch)
            start, delta = res.clone(), None
            for i, call in enumerate(model.order):
                if call.adds_embedding:
                    delta = K.joined(delta, start, res)
                delta = model.blocks[call.block].forward(delta, res, batch, runner.caches[call.cache], call.writes_cache)
                assert isinstance(delta, K.Normed)            # the block leaves its last norm to the add that follows
                got = res.clone()
                K.normed_add_rmsnorm(K.Normed(_tensor(delta.x, torch.float32), delta.weight, delta.eps), got, None, 0.0, torch.float32)
                assert float((got.cpu().double() - want[i]).abs().max()) < 5e-5 * max(1.0, float(want[i].abs().max())), f"{which}: layer run {i}"
        assert int(batch.status.item()) == 0


@BOTH
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
@pytest.mark.parametrize("cut", ["whole", "tail_decode", "portions", "mixed", "mixed_graphs"])
def test_cuts_match_plain(folders, references, which, dtype, cut):
    """Whole prompts, a decoded tail that crosses page borders, portions down to two tokens, and mixed batches in a pool
    that holds less than all requests (pages and slots used again), launched and captured."""
    reqs = _requests(which)
    ref = references[dtype][which]
    page = tt.PARAMS[which][2]
    make = {"whole": harness.whole, "tail_decode": lambda r: harness.tail_decode(r, 40), "portions": harness.portions,
            "mixed": lambda r: harness.mixed(r, max_live=3), "mixed_graphs": lambda r: harness.mixed(r, max_live=3, seed=5)}[cut]
    schedule = make(reqs)
    num_pages = harness.peak_tokens(schedule, page) // page
    if cut.startswith("mixed"):
        assert num_pages < sum(-(-len(t) // page) for t in reqs.values())
    runner = _runner(folders[(which, dtype)], dtype, page, num_pages, max_slots=3 if cut.startswith("mixed") else 1,
                     graphs=cut == "mixed_graphs")
    got = harness.run_schedule(runner, schedule)
    assert len(got) == sum(len(t) for t in reqs.values())
    _compare(got, ref, dtype)
    runner.cache.check()
    assert runner.cache.used_pages() == 0
    if cut == "mixed_graphs":
        assert runner.graph_steps_run > 0


@pytest.mark.parametrize("which", ["A", "B"])
def test_batched_requests_equal_each_alone_in_32_bit(folders, which):
    reqs = _requests(which)
    page = tt.PARAMS[which][2]
    folder = folders[(which, torch.float32)]
    alone = harness.run_schedule(_runner(folder, torch.float32, page, 64), harness.whole(reqs))
    together = harness.run_schedule(_runner(folder, torch.float32, page, 64, max_slots=5),
                                    [([(rid, toks, list(range(len(toks)))) for rid, toks in reqs.items()], list(reqs))])
    for key, row in alone.items():
        assert float((row - together[key]).abs().max()) <= 2e-5 * float(row.abs().max()), key


def test_cuts_agree_in_32_bit(folders):
    """However a request is cut, its logits agree to rounding of the last bits."""
    reqs = {"a70": _requests("A")["a70"]}
    folder = folders[("A", torch.float32)]
    a = harness.run_schedule(_runner(folder, torch.float32, 4, 20), harness.whole(reqs))
    b = harness.run_schedule(_runner(folder, torch.float32, 4, 20), harness.portions(reqs))
    c = harness.run_schedule(_runner(folder, torch.float32, 4, 20), harness.tail_decode(reqs, 50))
    for key, row in a.items():
        bound = 2e-5 * float(row.abs().max())
        assert float((row - b[key]).abs().max()) <= bound and float((row - c[key]).abs().max()) <= bound, key


def test_every_pass_of_the_loop_reads_its_own_cache(folders):
    """The plain implementation with the first pass's keys in the later passes' place gives other logits: what the cuts above
    compare would show a cache shared between passes.  And the embedding's output is not added once too often or too seldom."""
    cfg, w = copy.deepcopy(tt.TUDULIX_A), _weights(folders[("A", torch.float32)])
    toks = tiny.random_ids(40, cfg["vocab"], 6)
    want = plain.forward(cfg, w, toks)
    for times in (2, 4):
        other = copy.deepcopy(cfg)
        other["loop"]["times"] = times
        assert float((plain.forward(other, w, toks) - want).abs().max()) > 0.05 * float(want.abs().max())
    once = [(i, False) for i, _ in plain.run_order(cfg)]
    order, plain.run_order = plain.run_order, lambda c: once
    try:
        assert float((plain.forward(cfg, w, toks) - want).abs().max()) > 0.02 * float(want.abs().max())
    finally:
        plain.run_order = order
    runner = _runner(folders[("A", torch.float32)], torch.float32, 4, 16, max_slots=1)
    assert len({id(c) for c in runner.caches if c is not None}) == 11
    pages = [runner.cache.layer_cache(n).k_pages.data_ptr() for n in range(11)]
    assert len(set(pages)) == 11


@BOTH
def test_prompts_and_decoding_far_beyond_every_window(folders, dtype):
    """A prompt of several times the longest window in one step, in portions of hundreds and with a long decoded tail: most
    keys have left the windows of the first layers and their pages been given back, while the layer without a window sees all."""
    cfg = tt.TUDULIX_B
    reqs = {"long": tiny.random_ids(420, cfg["vocab"], 5)}
    folder = folders[("B", dtype)]
    ref = _reference(folder, reqs)
    for schedule in (harness.whole(reqs), harness.portions(reqs, (137, 2, 200, 3, 29)), harness.tail_decode(reqs, 90)):
        runner = _runner(folder, dtype, 16, 27, max_slots=1)
        _compare(harness.run_schedule(runner, schedule), ref, dtype)
        runner.cache.check()


def test_sharp_attention_finds_keys_at_every_distance(tmp_path):
    """Scales turned up make every softmax pick few keys, wherever they lie, up to hundreds of positions back.  32-bit, prompt in
    one step, in portions, and with a long decoded tail."""
    cfg = copy.deepcopy(tt.TUDULIX_D)
    for layer, window in zip(cfg["layers"], (260, None)):
        layer["mixer"]["scale"] *= 5.0
        layer["mixer"]["mask"] = None if window is None else {"size": window}
    tensors = tt.tensors_of(cfg, seed=21, std=0.25, norm_jitter=0.3)
    folder = tt.make_folder_from_tensors(tmp_path, "sharp", cfg, tensors)
    reqs = {"s": tiny.random_ids(300, cfg["vocab"], 77)}
    ref = _reference(folder, reqs)
    near = copy.deepcopy(cfg)
    for layer in near["layers"]:
        layer["mixer"]["mask"] = {"size": 64}
    cut = plain.forward(near, tensors, reqs["s"])
    assert float((cut - ref["s"])[200:].abs().max()) > 0.1 * float(ref["s"].abs().max())                    # the far keys found matter
    for schedule in (harness.whole(reqs), harness.portions(reqs, (37, 2, 64, 3, 29)), harness.tail_decode(reqs, 70)):
        got = harness.run_schedule(_runner(folder, torch.float32, 16, 19), schedule)
        _compare(got, ref, torch.float32, loosen=5.0)        # scores of tens: their 32-bit rounding shows in the weights


@BOTH
@pytest.mark.parametrize("keep,loop", [((0,), None), ((1,), (0, 1, 3)), ((4,), None), ((2, 3), (1, 2, 2)), ((0, 1, 2, 3, 4), (0, 5, 2))])
def test_other_orders_and_loops(tmp_path, dtype, keep, loop):
    """Models of one layer, with and without a feed-forward, a single layer run three times, a loop at the end, and one over
    everything."""
    cfg = copy.deepcopy(tt.TUDULIX_A)
    cfg["layers"] = [cfg["layers"][i] for i in keep]
    cfg.pop("loop")
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    folder = tt.make_folder_from_tensors(tmp_path, "m", cfg, tt.tensors_of(cfg, dtype, seed=31, std=0.25, norm_jitter=0.3))
    reqs = {"a": tiny.random_ids(40, cfg["vocab"], 1), "b": tiny.random_ids(9, cfg["vocab"], 2)}
    ref = _reference(folder, reqs)
    for schedule in (harness.whole(reqs), harness.tail_decode(reqs, 6), harness.mixed(reqs, max_live=2)):
        _compare(harness.run_schedule(_runner(folder, dtype, 4, 16), schedule), ref, dtype, loosen=1.5)


def test_long_decoding_through_freed_and_reused_pages(folders):
    """Two requests decoded token by token for 120 steps side by side after short prompts, then a third takes the slot and the
    pages that the first gave back."""
    cfg = tt.TUDULIX_A
    reqs = {"a": tiny.random_ids(130, cfg["vocab"], 1), "b": tiny.random_ids(127, cfg["vocab"], 2), "c": tiny.random_ids(60, cfg["vocab"], 3)}
    ref = _reference(folders[("A", torch.float32)], reqs)
    steps = [([("a", reqs["a"][:10], list(range(10))), ("b", reqs["b"][:7], list(range(7)))], [])]
    for i in range(120):
        steps.append(([("a", reqs["a"][10 + i:11 + i], [0]), ("b", reqs["b"][7 + i:8 + i], [0])], ["a", "b"] if i == 119 else []))
    steps.append(([("c", reqs["c"], list(range(60)))], ["c"]))
    runner = _runner(folders[("A", torch.float32)], torch.float32, 4, 66, max_slots=2)
    _compare(harness.run_schedule(runner, steps), ref, torch.float32)
    runner.cache.check()


@pytest.mark.parametrize("which,lens,new", [("A", [1, 5, 17], 20), ("B", [9, 64, 2, 31], 12), ("C", [4, 11], 15), ("D", [3, 40], 10)])
def test_greedy_generation_through_the_engine_equals_the_plain_one(folders, which, lens, new):
    from prelude_b200 import Engine
    folder = folders[(which, torch.float32)]
    cfg, w = _cfg(folder), _weights(folder)
    prompts = [tiny.random_ids(n, cfg["vocab"], 50 + n) for n in lens]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(new):
            seq.append(int(plain.forward(cfg, w, seq, torch.float64)[-1].argmax()))
        want.append(seq[len(p):])
    eng = Engine(folder, dtype="f32", page_size=tt.PARAMS[which][2], num_pages=64, max_running_requests=4)
    assert eng.caps.cuda_graph and eng.caps.kv_cache and not eng.caps.state_slots
    got = eng.generate(prompts, temperature=0.0, max_new_tokens=new, ignore_eos=True)
    assert [r.token_ids for r in got] == want
    # portions of a few tokens beside decoding requests, launched kernel by kernel: the same tokens
    eng2 = Engine(folder, dtype="f32", page_size=tt.PARAMS[which][2], num_pages=64, max_running_requests=4,
                  max_num_batched_tokens=7, long_prefill_token_threshold=3, cuda_graph=False)
    assert [r.token_ids for r in eng2.generate(prompts, temperature=0.0, max_new_tokens=new, ignore_eos=True)] == want
    assert eng.cache.used_pages() == 0 and eng2.cache.used_pages() == 0


def test_generation_in_bfloat16_runs_captured_steps(folders):
    from prelude_b200 import Engine
    folder = folders[("B", torch.bfloat16)]
    prompts = [tiny.random_ids(n, tt.TUDULIX_B["vocab"], 50 + n) for n in (40, 7, 90)]
    eng = Engine(folder, dtype="bf16", page_size=16, num_pages=64, max_running_requests=4)
    got = eng.generate(prompts, temperature=0.0, max_new_tokens=16, ignore_eos=True)
    eng2 = Engine(folder, dtype="bf16", page_size=16, num_pages=64, max_running_requests=4, cuda_graph=False)
    got2 = eng2.generate(prompts, temperature=0.0, max_new_tokens=16, ignore_eos=True)
    assert all(len(r.token_ids) == 16 for r in got)
    # captured and launched steps run the same kernels on the same numbers
    assert [r.token_ids for r in got] == [r.token_ids for r in got2]


def test_trace_replay_of_a_tudulix_folder(folders, tmp_path):
    import subprocess
    import sys
    import numpy as np
    folder = folders[("A", torch.float32)]
    cfg = _cfg(folder)
    toks = tiny.random_ids(30, cfg["vocab"], 9)
    ref = plain.forward(cfg, _weights(folder), toks, torch.float64)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:11], "want": [0, 10]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[11:13], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[13:], "want": [16]}], "end": ["x"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64"], input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (out / "1.f32").exists()
    a = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    b = np.fromfile(out / "2.f32", dtype="<f4").reshape(1, -1)
    for row, pos in ((a[0], 0), (a[1], 10), (b[0], 29)):
        assert float(np.abs(row - ref[pos].numpy()).max()) < 1e-4 * max(1.0, float(ref[pos].abs().max()))


def test_command_line_generates_from_a_tudulix_folder(folders):
    import subprocess
    import sys
    folder = folders[("B", torch.float32)]
    cfg, w = _cfg(folder), _weights(folder)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = subprocess.run([sys.executable, os.path.join(root, "bin", "prelude"), "--model", folder, "--dtype", "f32", "--prompt-ids", "5,17,3,200",
                          "--max-new-tokens", "5", "--temperature", "0", "--num-pages", "16", "--page-size", "16", "--ignore-eos"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    seq = [5, 17, 3, 200]
    for _ in range(5):
        seq.append(int(plain.forward(cfg, w, seq, torch.float64)[-1].argmax()))
    assert json.loads(out.stdout.strip().splitlines()[0])["token_ids"] == seq[4:]
