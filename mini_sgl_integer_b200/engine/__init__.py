from .engine import Engine  # noqa: F401
from .scheduler import GenerationRequest, SamplingParams, Scheduler  # noqa: F401
