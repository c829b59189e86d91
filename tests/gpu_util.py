"""What the GPU tests of the layered decoders share: uploads, comparisons, rounding."""
import numpy as np
import torch

F32, BF16 = torch.float32, torch.bfloat16


def cu(a, dtype=F32):
    return torch.from_numpy(np.ascontiguousarray(a)).to("cuda:0").to(dtype)


def f64(t):
    return t.double().cpu().numpy()


def close(got, ref, tol):
    """Largest difference over the reference's largest magnitude."""
    got = f64(got) if isinstance(got, torch.Tensor) else got
    assert got.shape == ref.shape and np.isfinite(got).all()
    err = np.abs(got - ref).max() / max(np.abs(ref).max(), 1e-30)
    assert err <= tol, err


def rounded(a, dtype):
    """The values a tensor of `dtype` holds, as float64."""
    return f64(torch.from_numpy(np.asarray(a)).to(dtype))


TOL = {F32: 3e-6, BF16: 2.0 ** -7}


def rounding(ref, ref32, tol):
    """Limit of an fp32 result: eight times what the oracle itself loses in fp32 (or `tol`, if that is more)."""
    return max(tol, 8 * np.abs(ref32 - ref).max() / np.abs(ref).max())


def rel(got, ref):
    """Root mean square of the difference over that of the reference, mean over the vocabulary taken off, worst position."""
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    return float(np.sqrt((d * d).mean(-1)).max() / np.sqrt(((ref - ref.mean(-1, keepdims=True)) ** 2).mean()))
