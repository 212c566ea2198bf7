"""The Dokulix design and its kernels on the GPU against the plain CPU implementation: every mechanism alone, then whole
models: prompts, token-by-token decoding, portions, reuse, loops, greedy generation."""

import pytest
import torch

from oracle import dokulix_oracle as O
from quickdraw_b200 import synthetic
from quickdraw_b200.engine import Engine
from quickdraw_b200.loader import assemble_hybrid, save_hybrid_checkpoint
from quickdraw_b200.state import HybridState, LayerHistory
from quickdraw_b200.weights import ChunkAttnWeights, LatentAttnWeights, LoopConfig
from tests import dokulix_cases as cases

pytestmark = pytest.mark.gpu
BF16, F32, F64 = torch.bfloat16, torch.float32, torch.float64


def rnd(*shape, seed=0, std=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std


def bf(*shape, seed=0, std=1.0):
    return rnd(*shape, seed=seed, std=std).to(BF16)


def error(got, want):
    got, want = got.detach().to("cpu", F64), want.to(F64)
    return float((got - want).norm() / want.norm().clamp(min=1e-30))


def status():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


@pytest.fixture(scope="module")
def M(cuda_device):
    from quickdraw_b200 import mixers
    return mixers


# ------------------------------------------------------------------------------- products
SHAPES = [(1, 200, 256), (1, 6000, 1032), (2, 34, 1032), (7, 5000, 64), (8, 76, 24), (9, 80, 64), (300, 264, 72), (513, 1000, 128), (40, 38, 50), (5, 20, 7),
          (2600, 4160, 40)]


@pytest.mark.parametrize("tokens,rows,width", SHAPES)
@pytest.mark.parametrize("x_type,y_type", [(BF16, BF16), (BF16, F32), (F32, F32), (F32, BF16)])
def test_products_with_what_follows_them(M, tokens, rows, width, x_type, y_type):
    """Bias; bias onto what the output holds; the gated unit over pairs of rows: in the few-row, tensor-core and any-shape forms."""
    if x_type == F32 and tokens > 600:
        tokens = 600
    x, w, bias = rnd(tokens, width, seed=1).to(x_type), bf(rows, width, seed=2, std=width ** -0.5), rnd(rows, seed=3)
    dev, stat = [t.cuda() for t in (x, w, bias)], status()
    plain = x.double() @ w.double().T + bias.double()
    tolerance = 1e-5 if y_type == F32 else 6e-3
    held = rnd(tokens, rows, seed=4).to(y_type)
    out = held.cuda()
    M.linear(dev[0], 0, width, dev[1], out, tokens=tokens, status=stat, bias=dev[2], add=True)
    assert error(out, plain + held.double()) < tolerance
    M.linear(dev[0], 0, width, dev[1], out, tokens=tokens, status=stat, bias=dev[2])
    assert error(out, plain) < tolerance
    half = torch.full((tokens, rows // 2), 7.0, dtype=y_type, device="cuda")
    M.linear(dev[0], 0, width, dev[1], half, tokens=tokens, status=stat, bias=dev[2], glu=True)
    assert error(half, torch.relu(plain[:, 0::2]) * plain[:, 1::2]) < tolerance
    assert int(stat.item()) == 0


@pytest.mark.parametrize("tokens,rows,width", [(1, 33, 64), (1, 5000, 264), (1, 40, 5000), (2, 17, 1032), (5, 40, 2056), (8, 24, 72)])
@pytest.mark.parametrize("x_type,y_type", [(BF16, BF16), (F32, F32), (F32, BF16)])
@pytest.mark.parametrize("offset", [0.0, 1.0])
def test_products_that_norm_their_input(M, tokens, rows, width, x_type, y_type, offset):
    x, w, norm = rnd(tokens, width + 8, seed=1, std=3.0).to(x_type), bf(rows, width, seed=2, std=width ** -0.5), bf(width, seed=3, std=0.5)
    out, stat = torch.empty(tokens, rows, dtype=y_type, device="cuda"), status()
    x_d, w_d, norm_d = x.cuda(), w.cuda(), norm.cuda()
    M.linear(x_d, 8, width + 8, w_d, out, tokens=tokens, status=stat, norm=norm_d, norm_offset=offset, eps=0.2)
    want = O.rms_norm(x[:, 8:].double(), offset + norm.double(), 0.2) @ w.double().T
    assert error(out, want) < (1e-5 if y_type == F32 else 4e-3)


# ------------------------------------------------------------------------- residual stream
@pytest.mark.parametrize("width", [64, 256, 320, 100, 33, 2048, 1280, 4096])
@pytest.mark.parametrize("tokens", [1, 5, 70])
@pytest.mark.parametrize("dtype", [BF16, F32])
def test_stream_rows_and_norm(M, width, tokens, dtype):
    """Embedding rows or stream rows, with and without a sublayer's result, a vector, the sum, the norm, an index."""
    from quickdraw_b200._lib import call_hybrid, ptr, stream_of
    table, step, w = bf(50, width), bf(width, seed=1), bf(width, seed=2, std=0.3)
    ids = torch.randint(0, 50, (tokens,), generator=torch.Generator().manual_seed(4))
    x, y, eps = rnd(tokens, width, seed=5), rnd(tokens, width, seed=6).to(dtype), 1e-2
    index = torch.randint(0, tokens, (tokens,), generator=torch.Generator().manual_seed(7), dtype=torch.int32)
    d = {n: t.cuda() for n, t in dict(table=table, step=step, w=w, ids=ids, x=x, y=y, index=index).items()}
    out, normed = torch.empty(tokens, width, device="cuda"), torch.empty(tokens, width, dtype=dtype, device="cuda")

    def run(token_ids=None, source=None, rows=None, y=None, step=None, out=None, norm=None):
        call_hybrid("qd_stream_norm", ptr(token_ids), ptr(d["table"]) if token_ids is not None else None, 50, ptr(source), ptr(rows), ptr(y), ptr(step),
                    ptr(out), ptr(norm), 1.0, ptr(normed), tokens, width, eps, M.DTYPE_CODE[dtype], stream_of(normed))
    close = lambda want: error(normed, O.rms_norm_around_one(want, w.double(), eps)) < (1e-6 if dtype == F32 else 4e-3)
    rows = table[ids].double()
    run(token_ids=d["ids"], out=out)
    assert torch.equal(out.cpu(), table[ids].float())
    run(token_ids=d["ids"], step=d["step"], out=out, norm=d["w"])
    assert error(out, rows + step.double()) < 1e-6 and close(rows + step.double())
    run(source=d["x"], y=d["y"], step=d["step"], out=out, norm=d["w"])
    want = x.double() + y.double() + step.double()
    assert error(out, want) < 1e-6 and close(want)
    run(source=d["x"], y=d["y"], out=out)
    assert error(out, x.double() + y.double()) < 1e-6
    run(source=d["x"], rows=d["index"], norm=d["w"])
    assert close(x.double()[index.long()])


# ------------------------------------------------------------------------------- mixers alone
def stacked(parts, tokens, dtype, seed=0):
    """Random projection rows laid out as the model does, and each part as float64."""
    at, total = {}, 0
    for name, width in parts.items():
        at[name] = total
        total += width + (-width) % 8
    proj = rnd(tokens, total, seed=seed).to(dtype)
    return proj, at, lambda: {name: proj[:, at[name]:at[name] + width].double() for name, width in parts.items()}


def drive(mixer, proj, at, history, cuts, start=0):
    """The mixer over the rows in portions of the given sizes (1: the one-token form)."""
    out, done, stat = [], 0, status()
    for cut in cuts:
        rows = proj[done:done + cut]
        if cut == 1:
            out.append(mixer.step(rows, at, history, torch.tensor(start + done, dtype=torch.int32, device="cuda"), stat))
        else:
            out.append(mixer.chunk(rows, at, history, start + done, stat))
        done += cut
    assert done == proj.shape[0] and int(stat.item()) == 0
    return torch.cat(out)


CUTS = {"whole": lambda n: [n], "one by one": lambda n: [1] * n, "pairs": lambda n: [2] * (n // 2) + [1] * (n % 2),
        "portions": lambda n: [3, 17, 2, 1, 1, 20] + [n - 44]}
nan_rows = lambda dtype, *shape: torch.full(shape, float("nan"), dtype=dtype, device="cuda")
on_gpu = lambda w: type(w)(**{n: None if t is None else t.cuda() for n, t in vars(w).items()})


def latent_case(m, tokens, dtype, sharp, seed=0):
    """Projections, weights, and the oracle as a function of the window."""
    proj, at, parts = stacked({"dq": m.q_rank, "dkv": m.kv_rank + m.rot_dim, "g": m.heads * m.vdim}, tokens, dtype, seed)
    w = LatentAttnWeights(dq=None, dkv=None, g=None, o=None, dq_norm=bf(m.q_rank, seed=seed + 1, std=0.3) + 1, dkv_norm=bf(m.kv_rank, seed=seed + 2, std=0.3) + 1,
                          uq=bf(m.heads * (m.dim + m.rot_dim), m.q_rank, seed=seed + 3, std=sharp * m.q_rank ** -0.5),
                          uk=bf(m.heads * m.dim, m.kv_rank, seed=seed + 4, std=m.kv_rank ** -0.5),
                          uv=bf(m.heads * m.vdim, m.kv_rank, seed=seed + 5, std=m.kv_rank ** -0.5))
    eps = 1e-3

    def want(window=m.window, heads=True):
        p = parts()
        cfg = dict(heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, kv_rank=m.kv_rank, scale=m.scale, mask={"size": window},
                   rot={"base": m.rotary_base, "dims": m.rot_dim})
        weights = {"dq.norm": w.dq_norm, "dkv.norm": w.dkv_norm, "uq": w.uq, "uk": w.uk, "uv": w.uv}
        out = O.latent_heads(p["dq"], p["dkv"], {n: t.double() for n, t in weights.items()}, "", cfg, eps).flatten(1)
        return out * torch.sigmoid(p["g"]) if heads else out
    return w, eps, proj, at, want


LATENTS = {
    "small": cases.latent(), "one head": cases.latent(heads=1, dim=16, rot_dim=32, vdim=24, window=33), "two row blocks": cases.latent(heads=19, window=40),
    "window of one": cases.latent(window=1), "window beyond the prompt": cases.latent(window=1000, scale=-0.3), "tile edges": cases.latent(window=64),
    "wide": cases.latent(heads=2, dim=128, rot_dim=64, vdim=136, q_rank=200, kv_rank=512, window=33, scale=0.06),
    "rank of 264": cases.latent(heads=3, kv_rank=264, rot_dim=24, vdim=48, window=45), "rank of 1024": cases.latent(heads=2, kv_rank=1024, window=9),
    "rank of 1536": cases.latent(heads=2, kv_rank=1536, window=37),
    "no vectors": cases.latent(heads=3, dim=14, rot_dim=6, vdim=9, q_rank=21, kv_rank=19, window=11), "value 300": cases.latent(heads=1, vdim=300, dim=264),
}


@pytest.mark.parametrize("cut", CUTS)
@pytest.mark.parametrize("name", LATENTS)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_latent_attention(M, name, cut, dtype):
    """Scores stand out, so a key too many or too few at the window's edge moves the result beyond the tolerance; the
    ring is smaller than the prompt and wraps, and starts as NaN."""
    m, tokens = LATENTS[name], 130
    w, eps, proj, at, want = latent_case(m, tokens, dtype, sharp=2.5)
    exact = want()
    if m.window < tokens:
        assert error(want(window=m.window + 1), exact) > 0.08 and (m.window == 1 or error(want(window=m.window - 1), exact) > 0.08)
    mixer = M.LatentAttention(on_gpu(w), m, eps, torch.device("cuda"))
    cuts = CUTS[cut](tokens)
    history = LayerHistory(latent=nan_rows(dtype, min(tokens, m.window - 1 + max(cuts)), m.row))
    got = drive(mixer, proj.cuda(), at, history, cuts)
    assert error(got, exact) < (2e-5 if dtype == F32 else 2.5e-2)


@pytest.mark.parametrize("splits", [1, 2, 5])
@pytest.mark.parametrize("name", ["small", "two row blocks", "window beyond the prompt", "rank of 1536", "no vectors"])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_latent_decoding_with_long_splits(M, name, splits, dtype):
    """Splits of several key tiles, as a large window has them."""
    m, tokens = LATENTS[name], 230
    w, eps, proj, at, want = latent_case(m, tokens, dtype, sharp=2.5)
    mixer = M.LatentAttention(on_gpu(w), m, eps, torch.device("cuda"))
    mixer.splits = min(splits, mixer.splits)
    history = LayerHistory(latent=nan_rows(dtype, min(tokens, m.window - 1 + 60), m.row))
    got = drive(mixer, proj.cuda(), at, history, [60, 60, 60] + [1] * 50)
    assert error(got[180:], want()[180:]) < (2e-5 if dtype == F32 else 2.5e-2)


def chunk_case(m, tokens, dtype, sharp, seed=0):
    """Projections, weights, and the oracle with other spans, slopes, denominators."""
    parts_of = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
    proj, at, parts = stacked(parts_of, tokens, dtype, seed)
    w = ChunkAttnWeights(q=None, k=None, v=None, o=None, q_b=None, k_b=None, v_b=None, o_b=None, q_norm=bf(m.dim, seed=seed + 1, std=0.3) + sharp,
                         k_norm=bf(m.dim, seed=seed + 2, std=0.3) + 1)
    eps = 1e-3

    def want(span=m.span, slopes=True, extra_one=True):
        p = parts()
        q = O.rms_norm(p["q"].view(tokens, m.heads, m.dim), w.q_norm.double(), eps)
        k = O.rms_norm(p["k"].view(tokens, m.kv_heads, m.dim), w.k_norm.double(), eps)
        return O.masked_attention(q, k, p["v"].view(tokens, m.kv_heads, m.vdim), m.scale, lambda i, j: O.sees_chunk(i, j, span),
                                  O.distance_slopes(m.heads) if slopes else None, extra_one).flatten(1)
    return w, eps, proj, at, want


CHUNKS = {
    "shared heads": cases.chunked(), "one kv head": cases.chunked(heads=5, kv_heads=1, dim=32, vdim=16, span=33), "one head": cases.chunked(heads=1, kv_heads=1),
    "own heads": cases.chunked(heads=3, kv_heads=3, dim=16, vdim=64, span=7), "chunk of one": cases.chunked(span=1),
    "chunk beyond the prompt": cases.chunked(span=1000, scale=-0.2), "wide": cases.chunked(heads=2, kv_heads=1, dim=136, vdim=200, span=64, scale=0.1),
    "no vectors": cases.chunked(heads=3, kv_heads=3, dim=13, vdim=9, span=11), "tile edges": cases.chunked(heads=4, kv_heads=4, span=64),
    "value 300": cases.chunked(heads=2, kv_heads=1, vdim=300, span=50),
}


@pytest.mark.parametrize("cut", CUTS)
@pytest.mark.parametrize("name", CHUNKS)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_chunked_attention(M, name, cut, dtype):
    m, tokens = CHUNKS[name], 150
    w, eps, proj, at, want = chunk_case(m, tokens, dtype, sharp=1.5)
    exact = want()
    if m.span < tokens:
        assert error(want(span=m.span + 1), exact) > 0.1
    assert error(want(extra_one=False), exact) > 0.04 and (m.span == 1 or error(want(slopes=False), exact) > (0.04 if m.heads > 1 else 0.004))
    mixer = M.ChunkAttention(on_gpu(w), m, eps, torch.device("cuda"))
    cuts = CUTS[cut](tokens)
    capacity = min(tokens, m.span - 1 + max(cuts))
    history = LayerHistory(k=nan_rows(dtype, capacity, m.kv_heads, m.dim), v=nan_rows(dtype, capacity, m.kv_heads, m.vdim))
    got = drive(mixer, proj.cuda(), at, history, cuts)
    assert error(got, exact) < (2e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("splits", [1, 3])
@pytest.mark.parametrize("name", ["wide", "chunk beyond the prompt", "no vectors"])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_chunked_decoding_with_long_splits(M, name, splits, dtype):
    m, tokens = CHUNKS[name], 230
    w, eps, proj, at, want = chunk_case(m, tokens, dtype, sharp=1.5)
    mixer = M.ChunkAttention(on_gpu(w), m, eps, torch.device("cuda"))
    mixer.splits = min(splits, mixer.splits)
    capacity = min(tokens, m.span - 1 + 60)
    history = LayerHistory(k=nan_rows(dtype, capacity, m.kv_heads, m.dim), v=nan_rows(dtype, capacity, m.kv_heads, m.vdim))
    got = drive(mixer, proj.cuda(), at, history, [60, 60, 60] + [1] * 50)
    assert error(got[180:], want()[180:]) < (2e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_more_heads_to_a_key_than_one_launch_holds(M, dtype):
    m, tokens = cases.chunked(heads=70, kv_heads=1, dim=256, vdim=256, span=14, scale=0.08), 32
    w, eps, proj, at, want = chunk_case(m, tokens, dtype, sharp=1.5)
    mixer = M.ChunkAttention(on_gpu(w), m, eps, torch.device("cuda"))
    history = LayerHistory(k=nan_rows(dtype, 30, 1, 256), v=nan_rows(dtype, 30, 1, 256))
    got = drive(mixer, proj.cuda(), at, history, [17] + [1] * 15)
    assert error(got, want()) < (2e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("norm,sink,gate,mask", [(0, 0, 0, 1), (1, 1, 2, 1), (2, 0, 1, 0), (0, 2, 2, 0), (2, 1, 0, 1)])
@pytest.mark.parametrize("vdim", [24, 21])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_kinds_combine_freely(M, norm, sink, gate, mask, vdim, dtype):
    """Norm none / row / head, sink none / learned / zero, gate none / head / value, window or chunk, with a rotation and slopes."""
    m = cases.chunked(heads=4, kv_heads=2, dim=16, vdim=vdim, span=23)
    tokens, eps, rot = 70, 1e-3, 8
    gates = {0: 8, 1: m.heads, 2: m.heads * vdim}[gate]
    proj, at, parts = stacked({"q": 64, "k": 32, "v": 2 * vdim, "g": gates}, tokens, dtype)
    size = {0: 64, 1: 64, 2: 16}[norm], {0: 32, 1: 32, 2: 16}[norm]
    qn, kn, sinks, slopes = bf(size[0], seed=1) + 2, bf(size[1], seed=2) + 1, bf(4, seed=3), torch.tensor([0.5, 0.0, 0.01, 0.1])
    p = parts()
    q, k = p["q"].view(tokens, 4, 16), p["k"].view(tokens, 2, 16)
    if norm == 1:
        q, k = O.rms_norm(p["q"], qn.double(), eps).view(tokens, 4, 16), O.rms_norm(p["k"], kn.double(), eps).view(tokens, 2, 16)
    elif norm == 2:
        q, k = O.rms_norm(q, qn.double(), eps), O.rms_norm(k, kn.double(), eps)
    # interleaved pairs: the rotation by halves on a permuted head
    order = torch.tensor([0, 2, 4, 6, 1, 3, 5, 7, *range(8, 16)])
    q, k = (O.rotate_half(x[..., order], torch.arange(tokens), 300.0, rot)[..., order.argsort()] for x in (q, k))
    v, exact = p["v"].view(tokens, 2, vdim), torch.zeros(tokens, 4, vdim, dtype=F64)
    for i in range(tokens):
        lo = i - i % m.span if mask else max(0, i - m.span + 1)
        for h in range(4):
            e = torch.exp(k[lo:i + 1, h // 2] @ q[i, h] * m.scale - slopes[h] * (i - torch.arange(lo, i + 1)))
            exact[i, h] = e @ v[lo:i + 1, h // 2] / (e.sum() + (0, float(torch.exp(sinks.double()[h])), 1)[sink])
    if gate:
        exact = exact * torch.sigmoid(p["g"].view(tokens, 4, vdim if gate == 2 else 1))
    dev = dict(q_norm=qn.cuda(), k_norm=kn.cuda(), sink=sinks.cuda(), slopes=slopes.cuda(), freq=M.frequencies(300.0, rot, "cuda"))
    mixer = M.GroupedAttention(m, eps, torch.device("cuda"), dev, rot=rot, norm=norm, sink_kind=sink, gate_kind=gate, mask=mask)
    for cuts in ([30, 2, 38], [40] + [1] * 30):
        history = LayerHistory(k=nan_rows(dtype, 62, 2, 16), v=nan_rows(dtype, 62, 2, vdim))
        got = drive(mixer, proj.cuda(), at, history, cuts)
        assert error(got, exact.flatten(1)) < (2e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("inside", [True, False])
@pytest.mark.parametrize("decoded", [True, False])
def test_a_single_far_latent_at_the_edge_of_a_long_window(M, inside, decoded, dtype):
    """One query is made of one key at the far end of a window of 300 (or one position beyond it)."""
    m = cases.latent(heads=2, dim=32, rot_dim=2, vdim=16, q_rank=72, kv_rank=48, window=300, base=1e9, scale=0.6)
    m.q_rank = m.heads * (m.dim + m.rot_dim) + 4
    tokens, query = 420, 417
    w, eps, proj, at, want = latent_case(m, tokens, dtype, sharp=1.0, seed=5)
    w.uq = torch.eye(m.q_rank)[:m.heads * (m.dim + m.rot_dim)].to(BF16)
    w.dq_norm = torch.ones_like(w.dq_norm)
    key = query - (m.window - 1) - (0 if inside else 1)
    proj[:, at["dkv"] + 24:at["dkv"] + 48] = 0                     # ordinary latents live in the first half, the special one in the second
    proj[:, at["dkv"] + 48:at["dkv"] + 50] = 0
    proj[key, at["dkv"]:at["dkv"] + 24] = 0
    proj[key, at["dkv"] + 24:at["dkv"] + 48] = rnd(24, seed=8).to(dtype)
    special = O.rms_norm(proj[key, at["dkv"]:at["dkv"] + 48].double(), w.dkv_norm.double(), eps)
    aim = torch.cat([(w.uk.double().view(2, 32, 48) @ special), torch.zeros(2, 2)], 1).flatten()
    proj[query, at["dq"]:at["dq"] + m.q_rank] = torch.cat([aim, torch.zeros(4)]).to(dtype)
    exact, other = want()[query], want(window=m.window + (-1 if inside else 1))[query]
    assert error(other, exact) > 0.5
    mixer = M.LatentAttention(on_gpu(w), m, eps, torch.device("cuda"))
    history = LayerHistory(latent=nan_rows(dtype, m.window - 1 + 128, m.row))
    got = drive(mixer, proj.cuda(), at, history, [128, 128, 128, 33] + ([1] * 3 if decoded else [3]))[query]
    assert error(got, exact) < (1e-4 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("inside", [True, False])
@pytest.mark.parametrize("decoded", [True, False])
def test_a_single_far_key_at_the_start_of_a_long_chunk(M, inside, decoded, dtype):
    """One query equals the first key of its chunk of 300 (or the last one of the chunk before)."""
    m = cases.chunked(heads=8, kv_heads=1, dim=32, vdim=16, span=300, scale=1.0)
    tokens, query = 640, 597
    w, eps, proj, at, want = chunk_case(m, tokens, dtype, sharp=1.0, seed=5)
    key, special = 300 - (0 if inside else 1), rnd(32, seed=9).to(dtype)
    proj[key, at["k"]:at["k"] + 32] = special
    proj[query, at["q"]:at["q"] + 256] = special.repeat(8)
    exact = want()[query].view(8, 16)
    without = proj[key].clone()
    proj[key, at["v"]:at["v"] + 16] += 5.0                          # only what sees the key notices
    moved = error(want()[query].view(8, 16)[7], exact[7])
    assert moved > 0.5 if inside else moved < 1e-9
    proj[key] = without
    mixer = M.ChunkAttention(on_gpu(w), m, eps, torch.device("cuda"))
    history = LayerHistory(k=nan_rows(dtype, 299 + 128, 1, 32), v=nan_rows(dtype, 299 + 128, 1, 16))
    got = drive(mixer, proj.cuda(), at, history, [128, 128, 128, 128, 83] + ([1] * 45 if decoded else [45]))[query]
    assert error(got.view(8, 16), exact) < (1e-4 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_rotation_far_from_the_start(M, dtype):
    from quickdraw_b200._lib import call_hybrid, ptr, stream_of
    x, freq = rnd(6, 3, 20, seed=2).to(dtype), M.frequencies(1.0e5, 8, "cuda")
    for position in (0, 77, 1_000_003):
        got = x.cuda()
        call_hybrid("qd_rotate_half", ptr(got), ptr(freq), None, position, 6, 3, 20, 8, M.DTYPE_CODE[dtype], stream_of(got))
        want = torch.cat([x[..., :12].double(), O.rotate_half(x[..., 12:].double(), position + torch.arange(6), 1.0e5, 8)], -1)
        assert error(got, want) < (5e-7 if dtype == F32 else 4e-3)


# -------------------------------------------------------------------------------- whole models
def build(name, seed=3):
    cfg = cases.MODELS[name]()
    tensors = cases.tensors(cfg, seed)
    return cfg, tensors, assemble_hybrid(cfg, lambda n: tensors[n].cuda())


def engine_of(ckpt, dtype, max_context=256, chunk=64, graph=True):
    return Engine(ckpt, max_context=max_context, device="cuda", dtype=dtype, prefill_chunk_size=chunk, cuda_graph=graph)


def run_portions(engine, tokens, cuts):
    rows, done = [], 0
    for cut in cuts:
        rows.append(engine.extend(tokens[done:done + cut], list(range(cut))))
        done += cut
    assert done == len(tokens) and engine.fused.check() == 0
    return torch.cat(rows)


LOGITS = {F32: 1e-4, BF16: 6e-2}


@pytest.mark.parametrize("name", cases.MODELS)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prompts_portions_and_decoding_give_the_oracle_s_logits(cuda_device, name, dtype):
    """One prompt whole (longer than a chunk), token by token, in portions down to two tokens: the same logits; every
    run follows another request on the same engine."""
    cfg, tensors, ckpt = build(name)
    tokens = cases.prompt(cfg, 90)
    want, _ = O.forward(cfg.to_dict(), tensors, tokens)
    engine = engine_of(ckpt, dtype)
    scale = float(want.std())
    runs = {}
    for cut, sizes in (("whole", [90]), ("one by one", [1] * 90), ("portions", [2, 3, 31, 1, 2, 1, 1, 47, 2]), ("prompt and decoding", [70] + [1] * 20)):
        engine.reset()
        engine.extend(cases.prompt(cfg, 40, seed=9))           # another request leaves its rows behind
        engine.reset()
        runs[cut] = run_portions(engine, tokens, sizes).cpu().double()
        worst = float((runs[cut] - want).pow(2).mean(1).sqrt().max()) / scale
        assert worst < LOGITS[dtype], (cut, worst)
    for cut, got in runs.items():
        assert float((got - runs["whole"]).pow(2).mean(1).sqrt().max()) / scale < LOGITS[dtype], cut


@pytest.mark.parametrize("name", ["middle loop", "one layer again", "odd sizes"])
def test_the_stream_after_every_layer_run(cuda_device, name):
    from quickdraw_b200.hybrid import DokulixModel
    cfg, tensors, ckpt = build(name)
    tokens = cases.prompt(cfg, 30)
    _, want = O.forward(cfg.to_dict(), tensors, tokens)
    record = []
    DokulixModel(ckpt, F32).run(torch.tensor(tokens, device="cuda"), 0, HybridState(cfg, 64, "cuda", dtype=F32), [29], record)
    assert len(record) == len(want)
    for got, layer in zip(record, want):
        assert error(got, layer) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding_wraps_the_rings(cuda_device, dtype):
    """300 tokens through rings of a few rows, decoded one by one in the graph; every pass of the loop keeps its own."""
    cfg = cases.config([(cases.latent(window=9), 64), (cases.chunked(span=10), None)], loop=(0, 2, 2))
    tensors = cases.tensors(cfg)
    engine = engine_of(assemble_hybrid(cfg, lambda n: tensors[n].cuda()), dtype, max_context=512, chunk=4)
    assert engine.state.layers[0].latent.shape[0] == 12 and engine.state.layers[3].k.shape[0] == 13
    tokens = cases.prompt(cfg, 300)
    want, _ = O.forward(cfg.to_dict(), tensors, tokens)
    got = run_portions(engine, tokens, [20] + [1] * 280).cpu().double()
    assert float((got - want).pow(2).mean(1).sqrt().max() / want.std()) < LOGITS[dtype]


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_graph_replay_and_eager_step_agree(cuda_device, dtype):
    cfg, tensors, ckpt = build("middle loop")
    tokens = cases.prompt(cfg, 25)
    eager, graph = engine_of(ckpt, dtype, graph=False), engine_of(ckpt, dtype)
    assert eager.graph is None and graph.graph is not None
    a, b = (run_portions(e, tokens, [20] + [1] * 5) for e in (eager, graph))
    assert torch.equal(a, b)


@pytest.mark.parametrize("name", ["middle loop", "loop over everything", "odd sizes"])
def test_greedy_generation_follows_the_oracle(cuda_device, name):
    cfg, tensors, ckpt = build(name)
    prompt = cases.prompt(cfg, 17)
    want, gap = O.greedy(cfg.to_dict(), tensors, prompt, 12)
    engine = engine_of(ckpt, F32)
    assert gap > 1e-3 and engine.generate(prompt, 12) == want
    assert engine.generate(prompt, 12) == want                    # and again after its own request
    engine.eos_token_ids = {want[4]}
    stop = want.index(want[4])
    assert engine.generate(prompt, 12) == want[:stop + 1]


def test_requests_of_unequal_length_on_one_engine_do_not_touch_one_another(cuda_device):
    cfg, tensors, ckpt = build("middle loop")
    shared = engine_of(ckpt, BF16)
    for seed, count in enumerate((70, 3, 41, 90, 1)):
        tokens = cases.prompt(cfg, count, seed=seed)
        shared.reset()
        alone = engine_of(ckpt, BF16)
        cuts = [count] if count < 20 else [count - 9] + [1] * 9
        assert torch.equal(run_portions(shared, tokens, cuts), run_portions(alone, tokens, cuts))


def test_snapshots_and_prefix_reuse(cuda_device):
    cfg, tensors, ckpt = build("middle loop")
    prompt = cases.prompt(cfg, 60)
    engine = engine_of(ckpt, F32)
    engine.prefill_reuse(prompt[:40])
    snap = engine.snapshot()
    engine.prefill(cases.prompt(cfg, 50, seed=4))
    engine.restore(snap)
    got = engine.extend(prompt[40:], [19])[0]
    fresh = engine.prefill(prompt)
    torch.testing.assert_close(got, fresh, rtol=1e-4, atol=1e-4)
    engine.prefill_reuse(prompt[:40])
    again = engine.prefill_reuse(prompt)
    assert engine.reused_tokens == 40
    torch.testing.assert_close(again, fresh, rtol=1e-4, atol=1e-4)


def test_from_pretrained_reads_the_directory(cuda_device, tmp_path):
    cfg, tensors, ckpt = build("odd sizes")
    save_hybrid_checkpoint(cfg, tensors, tmp_path)
    engine = Engine.from_pretrained(str(tmp_path), max_context=64, dtype=F32)
    prompt = cases.prompt(cfg, 9)
    want, _ = O.forward(cfg.to_dict(), tensors, prompt)
    assert error(engine.prefill(prompt), want[-1]) < 1e-4


def test_sizes_of_a_real_layer(cuda_device):
    """Widths of a real model's layers (tensor-core tiles, vectorised epilogues, several splits): a chunk against
    token-by-token decoding in fp32, and bf16 against fp32 in both."""
    cfg = synthetic.dokulix_config(3, 512, hidden=512, heads=20, kv_heads=4, window=70, chunk=90, loop=LoopConfig(1, 3, 2))
    ckpt = synthetic.make_dokulix(cfg, 1, "cuda")
    tokens = cases.prompt(cfg, 140)
    exact = run_portions(engine_of(ckpt, F32), tokens, [140]).cpu()
    assert error(run_portions(engine_of(ckpt, F32), tokens, [1] * 140), exact) < 1e-4
    assert error(run_portions(engine_of(ckpt, BF16, chunk=140), tokens, [140]), exact) < 6e-2
    assert error(run_portions(engine_of(ckpt, BF16), tokens, [64] + [1] * 76), exact) < 6e-2
