"""Each mechanism of the Milozen decoder alone, on the device, against its plain function: the kernel that writes, reads
and norms parallel residual streams (streams all equal and different, with and without an output pending, on chosen
rows); the rotation of neighbouring pairs in cached rows and queries; latent attention with a window, an output gate and
rows of an earlier layer, over a paged cache (pages scattered, stale numbers in unused slots), in portions and batches of
unequal requests, with keys made to stand out just inside and just outside the window, at page borders, at the borders of
the kernels' tiles and at the start, in prompts and in decoding; the softmax over a window's rows of scores; the sigmoid
router, the bounded gated unit and the weight on the experts' inputs, on each of the expert paths."""
import math

import pytest
import torch

from helpers import rel_err
from plain import milozen_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)


def _weights(part, dtype, std, seed, overrides=None):
    g = torch.Generator().manual_seed(seed)
    w = {}
    for t in part.tensor_specs():
        x = std * torch.randn(t.concrete_shape(), generator=g)
        w[t.name] = (1.0 + x if t.init == "norm" else x).to(dtype)
    for k, v in (overrides or {}).items():
        w[k] = v.to(dtype)
    part.load({k: v.to(DEV) for k, v in w.items()})
    return {k: v.double() for k, v in w.items()}


# ----------------------------------------------------------------------------- parallel residual streams

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["layer_norm", "rms_norm"])
@pytest.mark.parametrize("S,H", [(1, 64), (2, 72), (3, 50), (4, 2048), (5, 33), (8, 4096), (16, 20), (6, 11000)])
def test_streams_are_written_read_and_normed_in_one_kernel(dtype, kind, S, H):
    from photon_infer_b200.parts.base import Connected
    from photon_infer_b200.parts.registry import create_part
    g = torch.Generator().manual_seed(S * 1000 + H)
    T = 6
    params = {"size": H, "eps": 1e-5, "weight_name": "w"}
    if kind == "layer_norm":
        params["bias_name"] = None
    norm = create_part("norm", kind, params)
    nw = (1 + 0.3 * torch.randn(H, generator=g)).to(dtype)
    norm.load({"w": nw.to(DEV)})
    ref = plain.layer_norm if kind == "layer_norm" else plain.rms_norm
    conns, ws = [], []
    for i in range(2):
        c = create_part("connection", "hyper", {"streams": S})
        ws.append(_weights(c, dtype, 0.5, 10 * S + i))
        conns.append(c)
    tol = 5e-6 if dtype == torch.float32 else 8e-3
    x0 = 3 + 2 * torch.randn(T, H, generator=g)                     # a mean that is not zero
    ys = [(2 * torch.randn(T, H, generator=g)).to(dtype) for _ in range(3)]
    X = torch.stack([x0.double()] * S)
    # the first read: all streams equal, nothing pending
    h, streams = norm.read_streams(None, x0.to(DEV), conns[0].w_in, dtype)
    assert streams.dim() == 2 and h.dtype == dtype
    assert rel_err(h.float().cpu(), ref(plain.streams_read(X, ws[0]["in"]), nw.double(), 1e-5)) < tol
    # then write and read in turn: the first write spreads the equal streams out, the others work in place
    for i, y in enumerate(ys[:2]):
        before = streams
        h, streams = norm.read_streams(Connected(y.to(DEV), conns[i % 2]), streams, conns[(i + 1) % 2].w_in, dtype)
        X = plain.streams_write(X, ws[i % 2]["mix"], ws[i % 2]["out"], y.double())
        assert streams.shape == (T, S, H) and (i == 0 or streams.data_ptr() == before.data_ptr())
        assert rel_err(streams.cpu().transpose(0, 1), X) < 3e-6
        assert rel_err(h.float().cpu(), ref(plain.streams_read(X, ws[(i + 1) % 2]["in"]), nw.double(), 1e-5)) < tol
    # nothing pending on streams that differ
    h, same = norm.read_streams(None, streams, conns[0].w_in, dtype)
    assert same is streams and rel_err(h.float().cpu(), ref(plain.streams_read(X, ws[0]["in"]), nw.double(), 1e-5)) < tol
    # the model's last norm: the sum of the streams on chosen rows, with an output pending; nothing is written back
    kept = streams.clone()
    out = norm.add_forward_rows(Connected(ys[2].to(DEV), conns[0]), streams, i32([4, 1, 4]), dtype)
    X = plain.streams_write(X, ws[0]["mix"], ws[0]["out"], ys[2].double())
    assert torch.equal(kept, streams)
    assert rel_err(out.float().cpu(), ref(X.sum(0)[[4, 1, 4]], nw.double(), 1e-5)) < tol


def test_the_mix_matrix_is_indexed_from_to():
    """One stream sent to another one only: the transposed matrix would leave it where it was."""
    from photon_infer_b200.kernels import ops
    X = torch.arange(3.0).view(1, 3, 1).expand(2, 3, 8).contiguous().to(DEV) + 1
    mix = torch.zeros(3, 3, device=DEV)
    mix[0, 2] = 1.0
    new = torch.empty_like(X)
    out = torch.empty(2, 8, device=DEV)
    ops.stream_norm(X, 3, torch.zeros(2, 8, device=DEV), mix, torch.ones(3, device=DEV), torch.ones(3, device=DEV), torch.ones(8, device=DEV),
                    None, 1e-5, out, center=False, new_streams=new)
    assert torch.equal(new.cpu()[:, :, 0], torch.tensor([[0.0, 0.0, 1.0]]).expand(2, 3))


def test_sizes_that_the_stream_kernel_refuses():
    from photon_infer_b200.errors import PhotonError
    from photon_infer_b200.kernels import ops
    out, w = torch.empty(1, 8, device=DEV), torch.ones(8, device=DEV)
    with pytest.raises(PhotonError):
        ops.stream_norm(torch.zeros(1, 17, 8, device=DEV), 17, None, None, None, torch.ones(17, device=DEV), w, None, 1e-5, out)
    with pytest.raises(PhotonError):
        ops.stream_norm(torch.zeros(1, 2, 8, device=DEV), 2, torch.zeros(1, 8, device=DEV), None, None, None, w, None, 1e-5, out)


# ----------------------------------------------------------------------------- rotation and cache write

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rot,dims", [(8, 8), (12, 6), (64, 64), (2, 2)])
def test_neighbours_turn_in_rows_and_queries(dtype, rot, dims):
    from photon_infer_b200.kernels import ops
    g = torch.Generator().manual_seed(rot)
    T, qr, kr, heads, dim, base = 9, 20, 24, 3, 10, 500.0
    pos = torch.tensor([0, 1, 2, 15, 16, 17, 100, 599, 1200])
    down = torch.randn(T, qr + kr + rot + 7, generator=g).to(dtype)             # a section behind belongs to someone else
    qw, kw = (1 + 0.2 * torch.randn(qr, generator=g)).to(dtype), (1 + 0.2 * torch.randn(kr, generator=g)).to(dtype)
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)]).float().to(DEV)
    cache = torch.full((3, 1, 8, kr + rot), 7.0, dtype=dtype, device=DEV)
    slots = [5, 0, 23, 8, 7, -1, 16, 1, 12]
    cq = torch.empty(T, qr, dtype=dtype, device=DEV)
    err = torch.zeros(4, dtype=torch.int32, device=DEV)
    ops.latent_prep(down.to(DEV), qr, kr, rot, dims, qw.to(DEV), kw.to(DEV), 1e-5, pos.int().to(DEV), freq, i32(slots), cq, cache, err,
                    interleaved=True)
    tol = 1e-4 if dtype == torch.float32 else 1e-2              # position 1,200 times a frequency that is rounded to 32-bit
    d = down.double()
    assert rel_err(cq.float().cpu(), plain.rms_norm(d[:, :qr], qw.double(), 1e-5)) < tol
    flat = cache.view(-1, kr + rot).float().cpu()
    c = plain.rms_norm(d[:, qr:qr + kr], kw.double(), 1e-5)
    k = plain.rotate_neighbours(d[:, qr + kr:qr + kr + rot], pos, dims, base)
    for t, s in enumerate(slots):
        if s >= 0:
            assert rel_err(flat[s], torch.cat([c[t], k[t]])) < tol
    unused = [s for s in range(24) if s not in slots]
    assert torch.all(flat[unused] == 7.0) and err.cpu().tolist()[0] == 0
    # a layer that reads another one's rows: the query latent alone, nothing is stored
    cq2 = torch.empty_like(cq)
    ops.latent_prep(down.to(DEV)[:, :qr + 7], qr, kr, rot, dims, qw.to(DEV), None, 1e-5, pos.int().to(DEV), freq, None, cq2, None, err,
                    interleaved=True)
    assert torch.equal(cq2, cq)
    q = torch.randn(T, heads * (dim + rot), generator=g).to(dtype)
    out = torch.zeros(T, heads, kr + rot, dtype=dtype, device=DEV)
    ops.latent_q_rope(q.to(DEV), heads, dim, rot, dims, pos.int().to(DEV), freq, out, kr, interleaved=True)
    want = plain.rotate_neighbours(q.double().view(T, heads, dim + rot)[..., dim:], pos, dims, base)
    assert rel_err(out[:, :, kr:].float().cpu(), want) < tol and torch.all(out[:, :, :kr] == 0)


# ----------------------------------------------------------------------------- the mixer

class Pages:
    """Scattered pages for several requests, in a pool that is filled with stale numbers."""

    def __init__(self, requests, pages_each, page_size, width, dtype, seed):
        g = torch.Generator().manual_seed(seed)
        n = requests * pages_each
        self.perm = torch.randperm(n, generator=g).view(requests, pages_each).tolist()
        self.ps, self.n = page_size, n
        self.cache = (50 * torch.randn(n, 1, page_size, width, generator=g)).to(dtype).to(DEV)

    def fill(self, request, rows):
        """Stores the rows of positions 0 .. of a request."""
        idx = torch.tensor([self.perm[request][p // self.ps] * self.ps + p % self.ps for p in range(len(rows))], device=DEV)
        self.cache.view(-1, rows.shape[1])[idx] = rows.to(self.cache.dtype).to(DEV)

    def context(self, cut, starts, dtype, window=None, order=None):
        """A step of the given requests; pages behind the window are taken away from the tables, as the manager does."""
        from photon_infer_b200.parts.base import GroupView, StepContext
        order = list(range(len(cut))) if order is None else order
        pos, seq, sm, tables = [], [], [], []
        for s, r in enumerate(order):
            first = 0 if window is None else max(0, starts[r] + 1 - window) // self.ps
            tables.append([p if i >= first else -1 for i, p in enumerate(self.perm[r])])
            for p in range(starts[r], starts[r] + cut[r]):
                pos.append(p); seq.append(s); sm.append(self.perm[r][p // self.ps] * self.ps + p % self.ps)
        lens, st = [cut[r] for r in order], [starts[r] for r in order]
        ends = [a + b for a, b in zip(lens, st)]
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        return StepContext(sum(lens), len(lens), dtype, i32([0] * sum(lens)), i32(pos), i32(seq), i32(cu), i32(ends), i32(list(range(len(lens)))),
                           [GroupView(i32(tables), i32(sm), self.ps, self.n, len(tables[0]))], lens, ends, st, max(lens), max(ends),
                           torch.zeros(4, dtype=torch.int32, device=DEV))


def _mixer(dtype, heads, dim, rot, vdim, kv_rank, q_rank, window, H=48, base=300.0, own=True, seed=5, std=0.3):
    from photon_infer_b200.parts.registry import create_part
    m = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=0.8 * (dim + rot) ** -0.5,
             rot=dict(base=base, dims=rot))
    if window:
        m["mask"] = dict(size=window)
    att = create_part("mixer", "latent_attention", dict(hidden_size=H, heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank,
                                                        q_rank=q_rank, scale=m["scale"], eps=1e-5, rot_base=base, rot_dims=rot,
                                                        rot_interleaved=True, window=window, output_gate=True, own_kv=own))
    return att, m, _weights(att, dtype, std, seed)


SHAPES = [dict(heads=3, dim=16, rot=8, vdim=20, kv_rank=24, q_rank=40),            # general kernel
          dict(heads=5, dim=16, rot=16, vdim=24, kv_rank=32, q_rank=24),           # tensor-core decoding, half a tile of heads
          dict(heads=18, dim=8, rot=32, vdim=8, kv_rank=64, q_rank=16),            # more heads than a tile
          dict(heads=2, dim=7, rot=6, vdim=9, kv_rank=13, q_rank=11)]              # multiples of nothing


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [None, 1, 2, 16, 33, 100])
@pytest.mark.parametrize("expand", [False, True])
def test_owner_and_reader_in_portions(monkeypatch, dtype, shape, window, expand):
    """A layer with its own latent and one that reads its rows with other heads and another window, two unequal requests
    in portions (from 90 tokens down to one), against whole-sequence attention.  In bfloat16 the long portions take the
    products-and-softmax path or (``expand``) keys and values formed from the rows, beside short ones in the same step."""
    from photon_infer_b200.parts import latent_attention
    if expand and (dtype == torch.float32 or shape["vdim"] % 8 or shape["dim"] % 8):
        pytest.skip("only bfloat16 with sizes of 8s expands rows")
    if expand:                                  # whatever the arithmetic says: small latents would not be worth it
        def every_long(self, ctx, lens, dtype):
            assert self._prompt_defines(dtype) is not None
            starts = ctx.host_start_positions
            return {i: (starts[i], starts[i] + n - self._first_seen(starts[i])) for i, n in enumerate(lens) if n >= 32}
        monkeypatch.setattr(latent_attention.LatentAttention, "_expanded_requests", every_long)
    else:
        monkeypatch.setattr(latent_attention, "USE_EXPANDED_PROMPTS", False)
    from photon_infer_b200.parts.base import LayerCache
    own, m, w = _mixer(dtype, window=window, **shape)
    rshape = dict(shape, heads=shape["heads"] + 1, dim=shape["dim"] + (8 if expand else 3), vdim=shape["vdim"] + (8 if expand else 4), q_rank=shape["q_rank"] + 5)
    rwindow = None if window is None else max(1, window - 7)
    reader, rm, rw = _mixer(dtype, window=rwindow, own=False, seed=9, **rshape)
    lens, ps = [150, 77], 8
    g = torch.Generator().manual_seed(6)
    hs = [torch.randn(L, 48, generator=g).to(dtype) for L in lens]
    want, rwant = [], []
    for h in hs:
        pos = torch.arange(len(h))
        rows = plain.latent_rows(h.double(), w, m, pos, 1e-5)
        want.append(plain.latent_attention(h.double(), w, m, pos, 1e-5, rows))
        rwant.append(plain.latent_attention(h.double(), rw, rm, pos, 1e-5, rows))
    pages = Pages(2, 20, ps, own.width, dtype, seed=3)
    got, rgot, starts = [[], []], [[], []], [0, 0]
    for k, cut in enumerate([(33, 2), (2, 40), (1, 1), (90, 3), (1, 1), (23, 30)]):
        order = [1, 0] if k % 2 else [0, 1]
        ctx = pages.context(cut, starts, dtype, window, order)
        h = torch.cat([hs[r][starts[r]:starts[r] + cut[r]] for r in order]).to(DEV)
        out = own.forward(h, ctx, LayerCache(group=0, k=pages.cache)).float().cpu()
        snap = pages.cache.clone()
        rout = reader.forward(h, ctx, LayerCache(group=0, k=pages.cache, shared=True)).float().cpu()
        assert torch.equal(snap, pages.cache)                       # a reader stores nothing
        assert ctx.error_flag.cpu().tolist()[0] == 0
        a = 0
        for r in order:
            got[r].append(out[a:a + cut[r]]); rgot[r].append(rout[a:a + cut[r]])
            a += cut[r]
        starts = [starts[r] + cut[r] for r in range(2)]
    for r in range(2):
        tol = 2e-5 if dtype == torch.float32 else 3e-2
        assert rel_err(torch.cat(got[r]), want[r]) < tol
        assert rel_err(torch.cat(rgot[r]), rwant[r]) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [1, 5, 16, 64, 65, 129])
@pytest.mark.parametrize("phase", ["decode", "portion", "short"])
def test_a_key_just_inside_and_just_outside_the_window(dtype, window, phase):
    """One cached row is made to fit every query (its score stands out by far), at each distance around the window's edge
    and with the asking token at several places of a page and of the kernels' tiles of 32 and 64 rows: inside it takes
    nearly all of the weight, one further it takes none."""
    from photon_infer_b200.parts.base import LayerCache
    heads, kr, rot, ps = 4, 32, 16, 8
    att, m, _ = _mixer(dtype, heads, 16, rot, 16, kr, 24, window)
    att.scale = 1.0
    width = kr + rot
    g = torch.Generator().manual_seed(window)
    n = 330
    rows = torch.randn(n, width, generator=g)
    rows = 0.5 * rows / rows.norm(dim=1, keepdim=True)
    special = torch.randn(width, generator=g)
    special = special / special.norm()
    pages = Pages(1, 48, ps, width, dtype, seed=window)
    for asking in (window + 3, 191, 192, 200, 255, 256, 257, 300, 319, 320, 329):
        for back in sorted({0, 1, window - 1, window, window + 1}):
            target = asking - back
            if target < 0 or asking >= n or back < 0:
                continue
            keys = rows.clone()
            keys[target] = special
            count = {"decode": 1, "portion": 40, "short": 3}[phase]
            first = max(0, asking + 1 - count)
            count = asking + 1 - first
            pages.fill(0, keys)
            ctx = pages.context([count], [first], dtype, window)
            q = torch.zeros(count, heads, width)
            q[-1] = 14.0 * special
            out = torch.empty(count, heads * kr, dtype=dtype, device=DEV)
            att.attend(q.to(dtype).to(DEV), out, ctx, LayerCache(group=0, k=pages.cache))
            assert ctx.error_flag.cpu().tolist()[0] == 0
            kd = keys.to(dtype).double()
            lo = max(0, asking + 1 - window)
            s = (q[-1].to(dtype).double() @ kd.T)[:, lo:asking + 1]
            p = torch.softmax(s, dim=-1)
            if back < window:
                assert float(p[:, target - lo].min()) > 0.5
            want = p @ kd[lo:asking + 1, :kr]
            assert rel_err(out[-1].float().cpu().view(heads, kr), want) < (2e-5 if dtype == torch.float32 else 2e-2), (asking, back)


@pytest.mark.parametrize("sizes", [(64, 16, 64), (128, 64, 128), (16, 16, 24), (72, 8, 80), (136, 40, 104), (192, 64, 8)])
@pytest.mark.parametrize("window", [None, 1, 63, 64, 65, 200])
@pytest.mark.parametrize("gated", [False, True])
def test_long_portions_over_expanded_rows(sizes, window, gated):
    """The tensor-core kernel alone: three requests of unequal length and start in one call, heads whose sizes fill 64-wide
    chunks, do not fill them, or need several; for some queries one key is made to stand out, at the window's inner edge,
    just outside it, at the first visible key and at the query's own position.  Tokens that belong to nobody stay as they
    are."""
    from photon_infer_b200.kernels import ops
    d, r, v = sizes
    heads = 3
    g = torch.Generator().manual_seed(d + (window or 0))
    reqs = [(40, 0), (300, 517), (129, 130)]                        # (tokens, position of the first)
    gap = 5
    T = sum(n for n, _ in reqs) + gap * len(reqs)
    q = torch.randn(T, heads, d + r, generator=g)
    seqs, kus, krs, vs, t, row = [], [], [], [], 0, 0
    for n, start in reqs:
        base = 0 if window is None else max(0, start + 1 - window)
        L = start + n - base
        ku, kr, vv = torch.randn(L, heads, d, generator=g), torch.randn(L, r, generator=g), torch.randn(L, heads, v, generator=g)
        ku, kr = 0.3 * ku, 0.3 * kr
        for i in range(0, n, 7):
            pos = start + i
            lo = 0 if window is None else max(0, pos + 1 - window)
            back = [0, pos - lo, pos - lo + 1, (window or 40) - 1, (window or 40)][(i // 7) % 5]
            k = pos - back - base
            if 0 <= k < L:
                q[t + i, :, :d] = ku[k] / 0.3 * (5.0 / d ** 0.5)
                q[t + i, :, d:] = kr[k] / 0.3 * (5.0 / r ** 0.5)
        seqs.append((t, n, start, base, row))
        kus.append(ku); krs.append(kr); vs.append(vv)
        t += n + gap
        row += L
    b16 = lambda x: x.bfloat16()
    q, kus, krs, vs = b16(q), [b16(x) for x in kus], [b16(x) for x in krs], [b16(x) for x in vs]
    kv = torch.cat([torch.cat([a.reshape(len(a), -1), c.reshape(len(c), -1)], 1) for a, c in zip(kus, vs)])
    wide = torch.cat([torch.randn(row, 24, generator=g).bfloat16(), torch.cat(krs)], 1).to(DEV)        # the part lies in wider rows
    gate = (2 * torch.randn(T, heads * v + 16, generator=g)).bfloat16()
    out = torch.full((T, heads * v), 9.0, dtype=torch.bfloat16, device=DEV)
    err = torch.zeros(4, dtype=torch.int32, device=DEV)
    scale = 0.8
    ops.latent_prompt_attention(q.reshape(T, -1).to(DEV), q[:, :, d:].contiguous().to(DEV), kv.to(DEV), wide[:, 24:], out, seqs, heads, d, r, v,
                                window, scale, err, gate=gate.to(DEV)[:, 16:] if gated else None)
    assert err.cpu().tolist()[0] == 0
    out = out.float().cpu()
    for (t, n, start, base, row), ku, kr, vv in zip(seqs, kus, krs, vs):
        p, k = start + torch.arange(n)[:, None], base + torch.arange(len(ku))[None, :]
        ok = (k <= p) & (p - k < (window or 10 ** 9))
        qq = q[t:t + n].double()
        want = plain.attend(qq[..., :d], qq[..., d:], ku.double(), kr.double(), vv.double(), ok, scale)
        if gated:
            want = want * torch.sigmoid(gate[t:t + n, 16:].double()).view(n, heads, v)
        assert rel_err(out[t:t + n].view(n, heads, v), want) < 1.5e-2
        assert torch.all(out[t + n:t + n + gap] == 9.0)


def test_what_the_kernel_of_expanded_rows_refuses():
    from photon_infer_b200.errors import PhotonError
    from photon_infer_b200.kernels import ops
    z = lambda *s: torch.zeros(*s, dtype=torch.bfloat16, device=DEV)
    call = lambda seqs, d=64, r=16, v=64, rows=64, window=None: ops.latent_prompt_attention(
        z(40, 2 * (d + r)), z(40, 2, r), z(rows, 2 * (d + v)), z(rows, r), z(40, 2 * v), seqs, 2, d, r, v, window, 1.0, None)
    call([(0, 40, 24, 0, 0)])
    for bad in ([(0, 41, 0, 0, 0)], [(0, 40, 25, 0, 0)], [(0, 40, 0, 1, 0)], [(8, 33, 0, 0, 0)], [(0, 40, 0, 0, 25)]):
        with pytest.raises(PhotonError):
            call(bad)                           # rows or tokens that do not exist, or a first row behind the first visible one
    with pytest.raises(PhotonError):
        call([(0, 40, 0, 0, 0)], d=60)
    with pytest.raises(PhotonError):
        call([(0, 40, 0, 0, 0)], v=136)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_far_keys_without_a_window_and_pages_used_again(dtype):
    """No window: the row that stands out lies hundreds of tokens back, at the start and at page borders.  Then the pages
    go to another, shorter request: nothing of the first one shows."""
    from photon_infer_b200.parts.base import LayerCache
    att, m, w = _mixer(dtype, 3, 16, 16, 16, 32, 24, None)
    att.scale = 1.0
    ps, n, width, heads, kr = 16, 700, 48, 3, 32
    g = torch.Generator().manual_seed(2)
    rows = torch.randn(n, width, generator=g)
    rows = 0.5 * rows / rows.norm(dim=1, keepdim=True)
    special = rows[0] / rows[0].norm()
    pages = Pages(1, 48, ps, width, dtype, seed=8)
    for target in (0, 1, 15, 16, 63, 64, 65, 320, 640, 698, 699):
        keys = rows.clone()
        keys[target] = special
        pages.fill(0, keys)
        for count in (1, 50):
            ctx = pages.context([count], [n - count], dtype)
            q = torch.zeros(count, heads, width)
            q[-1] = 14.0 * special
            out = torch.empty(count, heads * kr, dtype=dtype, device=DEV)
            att.attend(q.to(dtype).to(DEV), out, ctx, LayerCache(group=0, k=pages.cache))
            kd = keys.to(dtype).double()
            p = torch.softmax(q[-1].to(dtype).double() @ kd.T, dim=-1)
            assert float(p[:, target].min()) > 0.5
            assert rel_err(out[-1].float().cpu().view(heads, kr), p @ kd[:, :kr]) < (2e-5 if dtype == torch.float32 else 2e-2)
    att, m, w = _mixer(dtype, 3, 16, 16, 16, 32, 24, None)
    h = torch.randn(41, 48, generator=g).to(dtype)
    pos = torch.arange(41)
    want = plain.latent_attention(h.double(), w, m, pos, 1e-5, plain.latent_rows(h.double(), w, m, pos, 1e-5))
    got, start = [], 0
    for cut in (37, 1, 2, 1):
        got.append(att.forward(h[start:start + cut].to(DEV), pages.context([cut], [start], dtype), LayerCache(group=0, k=pages.cache)).float().cpu())
        start += cut
    assert rel_err(torch.cat(got), want) < (2e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("rows_per_step", [1, 3, 8, 9, 40])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_products_per_head(dtype, rows_per_step):
    from photon_infer_b200.kernels import ops
    g = torch.Generator().manual_seed(rows_per_step)
    heads, K, N, T = 3, 40, 20, rows_per_step
    x = torch.randn(T, heads, K, generator=g).to(dtype)
    w = (0.3 * torch.randn(heads, N, K, generator=g)).to(dtype)
    wide = (3 * torch.randn(T, heads * N + 8, generator=g)).to(dtype)               # the gate is a section of a wider row
    out = torch.empty(T, heads, N, dtype=dtype, device=DEV)
    ops.head_linear(x.to(DEV), w.to(DEV), out, gate=wide.to(DEV)[:, 8:])
    want = torch.einsum("thk,hnk->thn", x.double(), w.double()) * torch.sigmoid(wide[:, 8:].double()).view(T, heads, N)
    assert rel_err(out.float().cpu(), want) < (5e-6 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window,first_pos,first_key", [(None, 5, 0), (3, 5, 0), (3, 40, 32), (300, 500, 200), (1, 17, 16), (64, 20, 0)])
def test_softmax_over_a_window_s_scores(dtype, window, first_pos, first_key):
    from photon_infer_b200.kernels import ops
    g = torch.Generator().manual_seed(first_pos)
    heads, tokens = 3, 21
    cols = first_pos + tokens - first_key + 4
    s = 3 * torch.randn(tokens * heads, cols, generator=g)
    probs = torch.full(s.shape, float("nan"), dtype=dtype, device=DEV)
    ops.causal_softmax_rows(s.to(DEV), probs, heads, first_pos, 0.7, first_key=first_key, window=window)
    q = first_pos + torch.arange(tokens * heads)[:, None] // heads
    k = first_key + torch.arange(cols)[None, :]
    ok = (k <= q) & (q - k < (window or 10 ** 9))
    want = torch.softmax((0.7 * s.double()).masked_fill(~ok, -math.inf), dim=-1)
    assert rel_err(probs.float().cpu(), want) < (3e-6 if dtype == torch.float32 else 5e-3)
    assert torch.all(probs.cpu()[~ok] == 0)


# ----------------------------------------------------------------------------- experts

@pytest.mark.parametrize("E,top", [(6, 2), (8, 1), (4, 4), (32, 5), (40, 3), (1, 1)])
@pytest.mark.parametrize("rows", [1, 5, 70])
def test_sigmoid_router(E, top, rows):
    from photon_infer_b200.kernels import ops
    g = torch.Generator().manual_seed(E + rows)
    h, wr = torch.randn(rows, 48, generator=g), 0.3 * torch.randn(E, 48, generator=g)
    ids, weights, counts = ops.moe_route(h.to(DEV), wr.to(DEV), None, top, "sigmoid")
    want_ids, want_w = plain.route(h.double(), wr.double(), top)
    assert torch.equal(ids.cpu().long(), want_ids) and rel_err(weights.cpu(), want_w) < 1e-5
    assert torch.equal(counts.cpu().long(), torch.bincount(want_ids.flatten(), minlength=E))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,top,ff,H,rows", [(6, 2, 32, 64, 5), (8, 1, 24, 48, 3), (4, 4, 14, 50, 40), (5, 3, 64, 96, 400), (3, 1, 40, 64, 90),
                                              (40, 2, 16, 56, 200), (2, 2, 128, 256, 1)])
@pytest.mark.parametrize("limit", [0.4, 1.7, 50.0])
def test_clamped_experts_with_weighted_inputs(dtype, E, top, ff, H, rows, limit):
    """Each of the expert paths (pair by pair, own grouped product, the library's grouped product), with a bound that most
    sums pass, one that some pass and one that none does, both signs; the plain side gets the router's choice."""
    from photon_infer_b200.kernels import ops
    from photon_infer_b200.parts.registry import create_part
    part = create_part("feed_forward", "moe", dict(hidden_size=H, experts=E, top=top, expert_size=ff, activation="clamped_swish",
                                                   act_limit=limit, act_slope=1.702, router_bias=False, scoring="sigmoid", weight_input=True))
    w = _weights(part, dtype, 0.35, E + rows)
    h = torch.randn(rows, H, generator=torch.Generator().manual_seed(rows)).to(dtype)
    chosen, route = [], ops.moe_route
    ops.moe_route = lambda *a, **k: chosen.append(route(*a, **k)) or chosen[-1]
    try:
        got = part.forward(h.to(DEV), None).float().cpu()
    finally:
        ops.moe_route = route
    m = dict(router=dict(top=top), expert=dict(limit=limit))
    if limit < 1:
        gate = torch.cat([h.double() @ w[f"e{e}.gate"].T for e in range(E)], 1)
        assert float((gate.abs() > limit).double().mean()) > 0.3            # the bound matters
    want = plain.moe_ff(h.double(), w, m, chosen[0][0].long().cpu())
    assert rel_err(got, want) < (1e-5 if dtype == torch.float32 else 2.5e-2)


def test_the_weight_sits_on_the_input():
    """With bounds in the unit the weight on the input and the weight on the output give different numbers: the result is
    the former."""
    from photon_infer_b200.parts.registry import create_part
    make = lambda on_input: create_part("feed_forward", "moe", dict(
        hidden_size=64, experts=3, top=2, expert_size=32, activation="clamped_swish", act_limit=1.0, act_slope=1.702, router_bias=False,
        scoring="sigmoid", weight_input=on_input))
    h = torch.randn(6, 64, generator=torch.Generator().manual_seed(3))
    outs = []
    for on_input in (True, False):
        part = make(on_input)
        w = _weights(part, torch.float32, 0.4, 1)
        outs.append(part.forward(h.to(DEV), None).cpu())
    want = plain.moe_ff(h.double(), w, dict(router=dict(top=2), expert=dict(limit=1.0)))
    ids, scores = plain.route(h.double(), w["router"], 2)
    behind = torch.stack([sum(s * plain.expert(h[t].double()[None], w, int(e), 1.0)[0] for e, s in zip(ids[t], scores[t])) for t in range(6)])
    assert rel_err(outs[0], want) < 1e-5 and rel_err(outs[1], behind) < 1e-5 and rel_err(outs[0], outs[1].double()) > 0.05


def test_what_the_experts_do_not_combine_with():
    from photon_infer_b200.parts.registry import create_part
    base = dict(hidden_size=16, experts=2, top=1, expert_size=8)
    for bad in (dict(activation="clamped_swish"), dict(activation="clamped_swish", act_limit=1.0, gated=False),
                dict(activation="clamped_swish", act_limit=1.0, shared_size=8), dict(weight_input=True, gated=False, activation="gelu")):
        with pytest.raises(ValueError):
            create_part("feed_forward", "moe", dict(base, **bad))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows", [2, 60])
def test_dense_feed_forward(dtype, rows):
    from photon_infer_b200.parts.registry import create_part
    ff = create_part("feed_forward", "gated", dict(hidden_size=56, intermediate_size=88, activation="silu", names=("gate", "up", "down")))
    w = _weights(ff, dtype, 0.2, 1)
    h = torch.randn(rows, 56, generator=torch.Generator().manual_seed(2)).to(dtype)
    assert rel_err(ff.forward(h.to(DEV), None).float().cpu(), plain.dense_ff(h.double(), w)) < (5e-6 if dtype == torch.float32 else 2e-2)
