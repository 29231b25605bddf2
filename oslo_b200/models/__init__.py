from .gpt2 import *  # noqa: F401,F403
from .gpt_neo import *  # noqa: F401,F403
from .gptj import *  # noqa: F401,F403
from .moronex import *  # noqa: F401,F403
from .begovik import *  # noqa: F401,F403
from .dekutar import *  # noqa: F401,F403
from .masezen import *  # noqa: F401,F403
from .registry import MODELS, find_model, load_causal_lm  # noqa: F401
