"""What the tests of the model families share: the fixture that makes sure a GPU case launched this package's kernels,
comparisons against a float64 oracle, and feeding of a cached decoder."""
import pytest
import torch

F32 = torch.float32
CPU = "cpu"


@pytest.fixture(autouse=True)
def _native(request):
    """A ``gpu`` case must launch this package's kernels.  The small host products run fastest on one thread."""
    threads = torch.get_num_threads()
    torch.set_num_threads(1)
    try:
        yield from _checked(request)
    finally:
        torch.set_num_threads(threads)


def _checked(request):
    if request.node.get_closest_marker("gpu") is None:
        yield
        return
    if not torch.cuda.is_available():
        pytest.skip("needs a CUDA device")
    from ferrl_b200.ops import cuda as C
    before = C.launches()
    yield
    torch.cuda.synchronize()
    assert C.launches() > before and C.kernel_status() == 0


def near(got, want, tol, what=""):
    """Largest difference against ``tol`` times the reference's root mean square (float64 on the host)."""
    g, w = got.detach().double().cpu(), want.double()
    assert g.shape == w.shape, (what, g.shape, w.shape)
    err = float((g - w).abs().max() / w.pow(2).mean().sqrt().clamp(min=1e-30))
    assert err < tol, (what, err, tol)
    return err


def rand(*shape, seed=0, std=1.0, dtype=F32, device=CPU):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * std).to(dtype).to(device)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def prefill_all(dec, prompts, device):
    """Every position's logits of every prompt, through one padded batch."""
    lens = torch.tensor([len(p) for p in prompts], device=device)
    ids = torch.zeros(len(prompts), int(lens.max()), dtype=torch.int64)
    for i, p in enumerate(prompts):
        ids[i, :len(p)] = torch.tensor(p)
    at = [(i, t) for i, p in enumerate(prompts) for t in range(len(p))]
    out = dec.prefill(ids.to(device), lens, at=tuple(torch.tensor([a[k] for a in at], device=device) for k in (0, 1)))
    return list(out.split([len(p) for p in prompts]))


def feed(dec, toks, device, active=None):
    return dec.decode(torch.tensor(toks, device=device), None if active is None else torch.tensor(active, device=device))


def row_errors(got, want):
    g = got.detach().double().cpu()
    assert g.shape == want.shape
    return (g - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def rms_near(got, want, tol):
    err = float(row_errors(got, want).max())
    assert err < tol, (err, tol)


def adapters(model, value=0.02, seed=4):
    g = torch.Generator().manual_seed(seed)
    with torch.no_grad():
        for p in model.trainable_params():
            p.copy_((torch.randn(p.shape, generator=g) * value).to(p.device))
